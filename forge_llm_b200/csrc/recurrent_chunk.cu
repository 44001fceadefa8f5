// Recurrent mixers over segments of a prompt, bfloat16 models, on the tensor cores: chunks of 64 tokens.
//
// With G_t the sum of a chunk's log decays up to and including token t, and S the state in front of the chunk,
//   delta rule    (I + L) U = R,  R_t = beta_t (v_t - S^T (e^{G_t} k_t)),  L_ts = beta_t sum_c k_tc k_sc e^{G_tc - G_sc}  (s < t)
//                 o_t = S^T (e^{G_t} q_t) + sum_{s <= t} P_ts u_s,         P_ts = sum_c q_tc k_sc e^{G_tc - G_sc}
//                 S <- e^{G_end} S + sum_s (e^{G_end - G_s} k_s) u_s^T
//   time mixing   U = V, o_t reads with e^{G_(t-1)} instead of e^{G_t}, and P_tt = sum_c q_tc bonus_c k_tc.
// chunk_prep_kernel (every chunk and head at once) forms T = (I + L)^-1 and P, and for decays per channel the decayed q and k;
// chunk_scan_kernel walks a sequence's chunks with a block of the state's columns in registers.
//
// Precision: q, k and v are the model's bf16 values; every factor that is not (decays, unit norms, T, P, U, the state) enters a product as a
// bf16 pair hi + lo, three products with f32 sums for two such factors.  Exponents are differences <= 0, so strong decays
// underflow to zero and nothing overflows: for decays per channel the pairs of a 16-token block are formed directly, and earlier
// blocks are reached through the sum at the block's start.
#include <algorithm>
#include <type_traits>

#include "mma.cuh"
#include "recurrent.cuh"

namespace forge {

namespace {

using bf16 = __nv_bfloat16;

constexpr int C = kRecurChunk;          // tokens of a chunk
constexpr int LDT = C + 8;
enum Mode { HEAD_DELTA = 0, CHANNEL_DELTA = 1, TIME_MIX = 2 };

__device__ __forceinline__ uint32_t smem_addr(const void* p) { return uint32_t(__cvta_generic_to_shared(p)); }

// per (chunk, head): bf16 [2][64][64] T and P (hi, lo); f32 scal[4][64]; f32 end[dim] = e^{G_end}; decays per channel also
// bf16 [3][2][64][DK]: k with e^G (delta rule only), q with e^G, k with e^{G_end - G}
struct ChunkPtr {
    bf16* T; bf16* P; float* scal; float* end; bf16* dec;
};
__device__ __forceinline__ ChunkPtr chunk_ptr(const ChunkScratch& s, int chunk, int heads, int h, int DK) {
    const size_t i = size_t(chunk) * heads + h;
    return {s.tp + i * 4 * C * C, s.tp + i * 4 * C * C + 2 * C * C, s.scal + i * 4 * C, s.end + i * DK, s.dec + i * 6 * C * DK};
}
constexpr int kScalKin = 0, kScalQin = C, kScalKout = 2 * C, kScalBeta = 3 * C;   // scal: e^G |k|^-1, e^G q scale, e^{G_end - G} |k|^-1, beta

// t = (I + L)^-1 for the strictly lower L in l (what l holds on and above the diagonal is ignored); 64 rows of LDL floats each, the blocks
// above t's diagonal blocks are not written; tmp: 3 x 16 x 17 floats
constexpr int LDL = C + 1;
template <int NT>
__device__ __forceinline__ void invert_unit_lower(float* t, const float* l, float* tmp, int tid) {
    if (tid < C) {   // the four 16 x 16 blocks on the diagonal, a column per thread
        const int b = (tid >> 4) * 16 * (LDL + 1), c = tid & 15;
        float x[16];
#pragma unroll
        for (int r = 0; r < 16; ++r) {
            float s = r == c ? 1.f : 0.f;
#pragma unroll
            for (int m = 0; m < r; ++m) s = fmaf(-l[b + r * LDL + m], x[m], s);   // x[m] = 0 above the column's one
            x[r] = s;
            t[b + r * LDL + c] = s;
        }
    }
    __syncthreads();
    for (int lev = 1; lev < 4; ++lev) {   // block (i, j = i - lev): -T_ii sum_{j <= k < i} L_ik T_kj
        const int nb = 4 - lev;
        for (int e = tid; e < nb * 256; e += NT) {
            const int i = lev + (e >> 8), j = i - lev, r = (e >> 4) & 15, c = e & 15;
            const float* lr = l + (i * 16 + r) * LDL;
            float s = 0.f;
            for (int k = j * 16; k < i * 16; ++k) s = fmaf(lr[k], t[k * LDL + j * 16 + c], s);
            tmp[(e >> 8) * 272 + r * 17 + c] = s;
        }
        __syncthreads();
        for (int e = tid; e < nb * 256; e += NT) {
            const int i = lev + (e >> 8), j = i - lev, r = (e >> 4) & 15, c = e & 15;
            const float* tr = t + (i * 16 + r) * LDL + i * 16;
            float s = 0.f;
#pragma unroll
            for (int k = 0; k < 16; ++k) s = fmaf(-tr[k], tmp[(e >> 8) * 272 + k * 17 + c], s);
            t[(i * 16 + r) * LDL + j * 16 + c] = s;
        }
        __syncthreads();
    }
}

// lower triangle of an f32 matrix (LDL apart) -> [2][64][64] hi, lo with zeros above
template <int NT>
__device__ __forceinline__ void store_lower(bf16* dst, const float* src, int tid) {
    for (int e = tid; e < C * C / 2; e += NT) {
        const int r = e / (C / 2), c = (e % (C / 2)) * 2;
        uint32_t hi, lo;
        split_bf16x2(c <= r ? src[r * LDL + c] : 0.f, c + 1 <= r ? src[r * LDL + c + 1] : 0.f, hi, lo);
        reinterpret_cast<uint32_t*>(dst)[e] = hi;
        reinterpret_cast<uint32_t*>(dst + C * C)[e] = lo;
    }
}

template <int DK, int MODE> struct Prep {
    static constexpr int NT = MODE == HEAD_DELTA ? 256 : 512, LDK = DK + 8;
    static constexpr bool CH = MODE != HEAD_DELTA;
    static constexpr size_t tiles = size_t(2) * C * LDK * 2;                          // q, k
    static constexpr size_t mats = size_t(2) * C * LDL * 4 + 3 * 272 * 4;             // L / T, P, tmp
    static constexpr size_t chan = CH ? size_t(C) * DK * 4 + size_t(5) * DK * 4 + size_t(2) * (32 + 48) * LDK * 2 : 0;   // sums, block sums, operands of one block row
    static constexpr size_t smem = tiles + mats + chan;
};

template <int DK, int MODE>
__global__ void __launch_bounds__(Prep<DK, MODE>::NT) chunk_prep_kernel(const RecurDims d, const RecurArgs a, const RecurScratch sc, const ScanSeg* __restrict__ segs, int n_segs) {
    using L = Prep<DK, MODE>;
    constexpr int NT = L::NT, LDK = L::LDK, NW = NT / 32;
    extern __shared__ __align__(16) unsigned char sm_raw[];
    bf16* sq = reinterpret_cast<bf16*>(sm_raw);
    bf16* sk = sq + C * LDK;
    float* sl = reinterpret_cast<float*>(sm_raw + L::tiles);
    float* sp = sl + C * LDL;
    float* tmp = sp + C * LDL;
    float* sg = tmp + 3 * 272;                 // [64][DK] sums of the log decays inside their 16-token block
    float* sb = sg + C * DK;                   // [5][DK] sums in front of each block, and the chunk's
    bf16* sa = reinterpret_cast<bf16*>(sb + 5 * DK);   // [2][32][LDK] rows k, then q, of a block row
    bf16* so = sa + 2 * 32 * LDK;              // [2][48][LDK] keys in front of it
    __shared__ float s_scal[4][C], s_gt[C];
    __shared__ int s_find[3];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int chunk = blockIdx.x, h = blockIdx.y, g = h / (d.heads / d.groups);
    if (tid < n_segs && segs[tid].chunk0 <= chunk && chunk < segs[tid].chunk0 + (segs[tid].n + C - 1) / C) s_find[0] = tid;
    for (int i = tid + NT; i < n_segs; i += NT) if (segs[i].chunk0 <= chunk && chunk < segs[i].chunk0 + (segs[i].n + C - 1) / C) s_find[0] = i;
    __syncthreads();
    const ScanSeg s = segs[s_find[0]];
    const int t0 = (chunk - s.chunk0) * C, n = min(C, s.n - t0), row0 = s.row0 + t0;
    const ChunkPtr out = chunk_ptr(sc.chunk, chunk, d.heads, h, DK);
    const bf16* x = MODE == TIME_MIX ? static_cast<const bf16*>(a.x) : static_cast<const bf16*>(sc.conv);
    const size_t ld = MODE == TIME_MIX ? a.x_ld : d.channels();
    for (int i = tid; i < 2 * C * (DK / 8); i += NT) {
        const int which = i / (C * (DK / 8)), t = i / (DK / 8) % C, c = (i % (DK / 8)) * 8;
        const bool ok = t < n && c < d.dim;
        cp_async16(smem_addr((which ? sk : sq) + t * LDK + c), ok ? x + size_t(row0 + t) * ld + which * d.qk() + g * d.dim + c : x, ok);
    }
    cp_commit();
    if (tid < C) {
        const bool ok = tid < n;
        if constexpr (MODE != TIME_MIX) {
            s_scal[0][tid] = ok ? sc.unit[size_t(row0 + tid) * 2 * d.groups + d.groups + g] : 0.f;   // |k|^-1
            s_scal[1][tid] = ok ? sc.unit[size_t(row0 + tid) * 2 * d.groups + g] : 0.f;              // q scale
            s_scal[3][tid] = ok ? a.beta[size_t(row0 + tid) * d.heads + h] : 0.f;
        } else { s_scal[0][tid] = s_scal[1][tid] = 1.f; }
        if constexpr (MODE == HEAD_DELTA) s_gt[tid] = ok ? a.decay[size_t(row0 + tid) * a.decay_ld + h] : 0.f;
    }
    if constexpr (L::CH) {
        for (int i = tid; i < C * DK; i += NT) {
            const int t = i / DK, c = i % DK;
            sg[i] = t < n && c < d.dim ? a.decay[size_t(row0 + t) * a.decay_ld + h * d.dim + c] : 0.f;
        }
    }
    cp_wait<0>();
    __syncthreads();
    const SmemMat mk{smem_addr(sk), LDK}, mq{smem_addr(sq), LDK};
    const int lr = lane >> 2, lc = (lane & 3) * 2;

    if constexpr (MODE == HEAD_DELTA) {
        if (warp == 0) {   // sums of the log decays
            const float v0 = s_gt[2 * lane], v1 = s_gt[2 * lane + 1];
            float sum = v0 + v1;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) { const float y = __shfl_up_sync(0xffffffffu, sum, o); if (lane >= o) sum += y; }
            __syncwarp();
            s_gt[2 * lane] = sum - v1;
            s_gt[2 * lane + 1] = sum;
        }
        // K K^T (warps 0..3) and Q K^T (4..7), 16 rows each, blocks up to the diagonal
        const int mt = warp & 3, is_q = warp >> 2;
        float acc[8][4];
#pragma unroll
        for (int i = 0; i < 8; ++i)
#pragma unroll
            for (int e = 0; e < 4; ++e) acc[i][e] = 0.f;
#pragma unroll
        for (int kt = 0; kt < DK / 16; ++kt) {
            uint32_t fa[4];
            (is_q ? mq : mk).a(fa, mt * 16, kt * 16, lane);
#pragma unroll
            for (int nb = 0; nb < 4; ++nb)
                if (nb <= mt) {
                    uint32_t fb[4];
                    mk.b(fb, nb * 16, kt * 16, lane);
                    mma(acc[2 * nb], fa, fb[0], fb[1]);
                    mma(acc[2 * nb + 1], fa, fb[2], fb[3]);
                }
        }
        __syncthreads();
        float* dst = is_q ? sp : sl;
#pragma unroll
        for (int i = 0; i < 8; ++i)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int t = mt * 16 + lr + (e >> 1) * 8, c = i * 8 + lc + (e & 1);
                if (i / 2 > mt) continue;
                float v = 0.f;
                if (is_q ? c <= t : c < t) v = acc[i][e] * s_scal[0][c] * expf(s_gt[t] - s_gt[c]) * (is_q ? s_scal[1][t] : s_scal[0][t] * s_scal[3][t]);
                dst[t * LDL + c] = v;
            }
        __syncthreads();
        if (tid < C) {
            const float e = expf(s_gt[tid]);
            out.scal[kScalKin + tid] = e * s_scal[0][tid];
            out.scal[kScalQin + tid] = e * s_scal[1][tid];
            out.scal[kScalKout + tid] = expf(s_gt[C - 1] - s_gt[tid]) * s_scal[0][tid];
            out.scal[kScalBeta + tid] = s_scal[3][tid];
        }
        if (tid < DK) out.end[tid] = expf(s_gt[C - 1]);
    } else {
        // sums inside the blocks, then in front of them
        for (int i = tid; i < 4 * DK; i += NT) {
            const int b = i / DK, c = i % DK;
            float sum = 0.f;
#pragma unroll
            for (int t = 0; t < 16; ++t) { sum += sg[(b * 16 + t) * DK + c]; sg[(b * 16 + t) * DK + c] = sum; }
        }
        __syncthreads();
        for (int c = tid; c < DK; c += NT) {
            float sum = 0.f;
#pragma unroll
            for (int b = 0; b < 4; ++b) { sb[b * DK + c] = sum; sum += sg[(b * 16 + 15) * DK + c]; }
            sb[4 * DK + c] = sum;
            out.end[c] = expf(sum);
        }
        __syncthreads();
        // exponent of a query row inside its block: up to and including its own decay, or for time mixing without it
        auto sum_q = [&](int t, int c) { return MODE == TIME_MIX ? (t & 15 ? sg[(t - 1) * DK + c] : 0.f) : sg[t * DK + c]; };
        // pairs inside a block: a warp per row, lanes share the channels
        for (int t = warp; t < C; t += NW) {
            constexpr int PL = DK / 32;
            float qv[PL], kv[PL], eq[PL], ek[PL];
#pragma unroll
            for (int i = 0; i < PL; ++i) {
                const int c = lane + 32 * i;
                qv[i] = __bfloat162float(sq[t * LDK + c]); kv[i] = __bfloat162float(sk[t * LDK + c]);
                eq[i] = sum_q(t, c); ek[i] = sg[t * DK + c];
            }
            for (int u = t & ~15; u <= t; ++u) {
                float pq = 0.f, pk = 0.f;
#pragma unroll
                for (int i = 0; i < PL; ++i) {
                    const int c = lane + 32 * i;
                    const float ku = __bfloat162float(sk[u * LDK + c]), gu = sg[u * DK + c];
                    if constexpr (MODE == TIME_MIX) pq = fmaf(qv[i] * ku, u < t ? expf(eq[i] - gu) : c < d.dim ? a.bonus[h * d.dim + c] : 0.f, pq);
                    else { const float e = expf(ek[i] - gu) * ku; pq = fmaf(qv[i], e, pq); pk = fmaf(kv[i], e, pk); }
                }
                pq = warp_sum(pq);
                if constexpr (MODE != TIME_MIX) pk = warp_sum(pk);
                if (lane == 0) {
                    sp[t * LDL + u] = pq * s_scal[1][t] * s_scal[0][u];
                    if constexpr (MODE != TIME_MIX) sl[t * LDL + u] = pk * s_scal[3][t] * s_scal[0][t] * s_scal[0][u];
                }
            }
        }
        // earlier blocks, reached through the sum at the block's start
        for (int b = 1; b < 4; ++b) {
            __syncthreads();
            for (int i = tid; i < (32 + 16 * b) * (DK / 2); i += NT) {
                const int r = i / (DK / 2), c = (i % (DK / 2)) * 2;
                float v[2];
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    if (r < 16) v[e] = __bfloat162float(sk[(b * 16 + r) * LDK + c + e]) * expf(sg[(b * 16 + r) * DK + c + e]);
                    else if (r < 32) v[e] = __bfloat162float(sq[(b * 16 + r - 16) * LDK + c + e]) * expf(sum_q(b * 16 + r - 16, c + e));
                    else {
                        const int u = r - 32;
                        v[e] = __bfloat162float(sk[u * LDK + c + e]) * expf(sb[b * DK + c + e] - sb[(u >> 4) * DK + c + e] - sg[u * DK + c + e]);
                    }
                }
                uint32_t hi, lo;
                split_bf16x2(v[0], v[1], hi, lo);
                bf16* dst = r < 32 ? sa + r * LDK + c : so + (r - 32) * LDK + c;
                *reinterpret_cast<uint32_t*>(dst) = hi;
                *reinterpret_cast<uint32_t*>(dst + (r < 32 ? 32 : 48) * LDK) = lo;
            }
            __syncthreads();
            const SmemMat ah{smem_addr(sa), LDK}, al{smem_addr(sa + 32 * LDK), LDK}, bh{smem_addr(so), LDK}, bl{smem_addr(so + 48 * LDK), LDK};
            for (int w = warp; w < 2 * b; w += NW) {   // (k or q) x 16 earlier keys
                const int is_q = w & 1, nb = w >> 1;
                if (MODE == TIME_MIX && !is_q) continue;
                float acc[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
#pragma unroll
                for (int kt = 0; kt < DK / 16; ++kt) {
                    uint32_t fh[4], fl[4], gh[4], gl[4];
                    ah.a(fh, is_q * 16, kt * 16, lane); al.a(fl, is_q * 16, kt * 16, lane);
                    bh.b(gh, nb * 16, kt * 16, lane); bl.b(gl, nb * 16, kt * 16, lane);
#pragma unroll
                    for (int j = 0; j < 2; ++j) {
                        mma(acc[j], fl, gh[2 * j], gh[2 * j + 1]);
                        mma(acc[j], fh, gl[2 * j], gl[2 * j + 1]);
                        mma(acc[j], fh, gh[2 * j], gh[2 * j + 1]);
                    }
                }
                float* dst = is_q ? sp : sl;
#pragma unroll
                for (int j = 0; j < 2; ++j)
#pragma unroll
                    for (int e = 0; e < 4; ++e) {
                        const int t = b * 16 + lr + (e >> 1) * 8, u = nb * 16 + j * 8 + lc + (e & 1);
                        dst[t * LDL + u] = acc[j][e] * s_scal[0][u] * (is_q ? s_scal[1][t] : s_scal[0][t] * s_scal[3][t]);
                    }
            }
        }
        // q and k with their decays, for the walk over the state
        for (int i = tid; i < C * (DK / 2); i += NT) {
            const int t = i / (DK / 2), c = (i % (DK / 2)) * 2, b = t >> 4;
            const __nv_bfloat162 q2 = *reinterpret_cast<const __nv_bfloat162*>(sq + t * LDK + c), k2 = *reinterpret_cast<const __nv_bfloat162*>(sk + t * LDK + c);
            const float2 q = __bfloat1622float2(q2), k = __bfloat1622float2(k2);
            const float f0 = sb[b * DK + c], f1 = sb[b * DK + c + 1], g0 = sg[t * DK + c], g1 = sg[t * DK + c + 1];
            const float ks = s_scal[0][t], qs = s_scal[1][t];
            uint32_t hi, lo;
            uint32_t* dst = reinterpret_cast<uint32_t*>(out.dec) + i;
            constexpr int M = C * DK / 2;
            if constexpr (MODE != TIME_MIX) {
                split_bf16x2(k.x * ks * expf(f0 + g0), k.y * ks * expf(f1 + g1), hi, lo);
                dst[0] = hi; dst[M] = lo;
            }
            split_bf16x2(q.x * qs * expf(f0 + sum_q(t, c)), q.y * qs * expf(f1 + sum_q(t, c + 1)), hi, lo);
            dst[2 * M] = hi; dst[3 * M] = lo;
            split_bf16x2(k.x * ks * expf(sb[4 * DK + c] - f0 - g0), k.y * ks * expf(sb[4 * DK + c + 1] - f1 - g1), hi, lo);
            dst[4 * M] = hi; dst[5 * M] = lo;
        }
        if constexpr (MODE != TIME_MIX) if (tid < C) out.scal[kScalBeta + tid] = s_scal[3][tid];
        __syncthreads();
    }
    store_lower<NT>(out.P, sp, tid);
    if constexpr (MODE != TIME_MIX) {
        __syncthreads();
        invert_unit_lower<NT>(sp, sl, tmp, tid);   // P is stored: its place takes T
        store_lower<NT>(out.T, sp, tid);
    }
}

// ------------------------------------------------------------------------------------------------ walk over the chunks
constexpr int NB = 32, LDN = NB + 8;   // value columns of a CTA

template <int DK, int MODE> struct Scan {
    static constexpr int LDK = DK + 8;
    static constexpr int KT = C * LDK, TT = C * LDT, VT = C * LDN;            // elements of the tiles
    // k (two buffers for exact k; hi and lo otherwise), q (one; hi, lo), k for the update (hi, lo)
    static constexpr int nk = MODE == TIME_MIX ? 0 : 2, nq = MODE == HEAD_DELTA ? 1 : 2, no = MODE == HEAD_DELTA ? 0 : 2;
    static constexpr int oq = nk * KT, oo = oq + nq * KT, ot = oo + no * KT, op = ot + (MODE == TIME_MIX ? 0 : 2 * TT), ov = op + 2 * TT, os = ov + VT,
                         orr = os + 2 * DK * LDN, ou = orr + (MODE == TIME_MIX ? 0 : 2 * VT), ow = ou + (MODE == TIME_MIX ? 0 : 2 * VT), total = ow + (MODE == HEAD_DELTA ? 2 * VT : 0);
    static constexpr size_t smem = size_t(total) * 2 + 2 * (4 * C + DK) * 4;
};

template <int DK, int MODE>
__global__ void __launch_bounds__(256) chunk_scan_kernel(const RecurDims d, const RecurArgs a, const RecurScratch sc, const ScanSeg* __restrict__ segs) {
    using L = Scan<DK, MODE>;
    constexpr int LDK = L::LDK, NT = 256;
    extern __shared__ __align__(16) unsigned char sm_raw[];
    bf16* sm = reinterpret_cast<bf16*>(sm_raw);
    float* s_scal = reinterpret_cast<float*>(sm + L::total);   // [2][4 * 64]
    float* s_end = s_scal + 2 * 4 * C;                         // [2][DK]
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, lr = lane >> 2, lc = (lane & 3) * 2;
    const ScanSeg s = segs[blockIdx.z];
    const int h = blockIdx.y, g = h / (d.heads / d.groups), c0 = blockIdx.x * NB;
    const int chunks = (s.n + C - 1) / C;
    const bf16* x = MODE == TIME_MIX ? static_cast<const bf16*>(a.x) : static_cast<const bf16*>(sc.conv);
    const size_t ld = MODE == TIME_MIX ? a.x_ld : d.channels();
    auto mat = [&](int off, int l) { return SmemMat{smem_addr(sm + off), l}; };

    // [64][cols] bf16 rows of a dense scratch matrix
    auto copy_rows = [&](int off, int l, const bf16* src, int cols) {
        for (int i = tid; i < C * (cols / 8); i += NT) {
            const int r = i / (cols / 8), c = (i % (cols / 8)) * 8;
            cp_async16(smem_addr(sm + off + r * l + c), src + size_t(r) * cols + c, true);
        }
    };
    // [64][DK] rows of the step's q or k (which = 0, 1), or [64][NB] of v (2)
    auto copy_x = [&](int off, int l, int ch, int which) {
        const int cols = which == 2 ? NB : DK, valid = which == 2 ? min(NB, d.vdim - c0) : d.dim;
        const int col0 = which == 2 ? 2 * d.qk() + h * d.vdim + c0 : which * d.qk() + g * d.dim;
        for (int i = tid; i < C * (cols / 8); i += NT) {
            const int r = i / (cols / 8), c = (i % (cols / 8)) * 8;
            const bool ok = ch * C + r < s.n && c < valid;
            cp_async16(smem_addr(sm + off + r * l + c), ok ? x + size_t(s.row0 + ch * C + r) * ld + col0 + c : x, ok);
        }
    };
    auto fetch1 = [&](int ch) {   // read by the first products
        if (ch < chunks) {
            const ChunkPtr p = chunk_ptr(sc.chunk, s.chunk0 + ch, d.heads, h, DK);
            if constexpr (MODE == HEAD_DELTA) { copy_x((ch & 1) * L::KT, LDK, ch, 1); copy_x(L::oq, LDK, ch, 0); }
            else {
                if constexpr (MODE == CHANNEL_DELTA) for (int i = 0; i < 2; ++i) copy_rows(i * L::KT, LDK, p.dec + i * C * DK, DK);
                for (int i = 0; i < 2; ++i) copy_rows(L::oq + i * L::KT, LDK, p.dec + (2 + i) * C * DK, DK);
            }
            if constexpr (MODE != TIME_MIX) {
                copy_x(L::ov, LDN, ch, 2);
                if (tid < C) cp_async16(smem_addr(s_scal + (ch & 1) * 4 * C + tid * 4), p.scal + tid * 4, true);
            }
            if (tid < DK / 4) cp_async16(smem_addr(s_end + (ch & 1) * DK + tid * 4), p.end + tid * 4, true);
        }
        cp_commit();
    };
    auto fetch2 = [&](int ch) {
        if (MODE != TIME_MIX && ch < chunks) {
            const ChunkPtr p = chunk_ptr(sc.chunk, s.chunk0 + ch, d.heads, h, DK);
            for (int i = 0; i < 2; ++i) copy_rows(L::ot + i * L::TT, LDT, p.T + i * C * C, C);
        }
        cp_commit();
    };
    auto fetch3 = [&](int ch) {   // read by the last products
        if (ch < chunks) {
            const ChunkPtr p = chunk_ptr(sc.chunk, s.chunk0 + ch, d.heads, h, DK);
            for (int i = 0; i < 2; ++i) copy_rows(L::op + i * L::TT, LDT, p.P + i * C * C, C);
            if constexpr (MODE != HEAD_DELTA) for (int i = 0; i < 2; ++i) copy_rows(L::oo + i * L::KT, LDK, p.dec + (4 + i) * C * DK, DK);
            if constexpr (MODE == TIME_MIX) copy_x(L::ov, LDN, ch, 2);
        }
        cp_commit();
    };

    // the state: 16 rows and NI times 16 columns per warp
    constexpr int MW = DK / 16 < 8 ? DK / 16 : 8, NI = NB / 16 / (8 / MW), MI = DK / 16 / MW;
    static_assert(MI == 1 && NI >= 1, "one row tile per warp");
    const int sm0 = (warp % MW) * 16, sn0 = (warp / MW) * NI * 16;
    float st[NI][2][4];
    float* S = a.state + (size_t(s.slot) * d.heads + h) * d.dim * d.vdim + c0;
#pragma unroll
    for (int i = 0; i < NI; ++i)
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const int r = sm0 + lr + e * 8, c = sn0 + i * 16 + j * 8 + lc;
                float2 v = make_float2(0.f, 0.f);
                if (s.pos0 > 0 && r < d.dim && c0 + c < d.vdim) v = *reinterpret_cast<const float2*>(S + size_t(r) * d.vdim + c);
                st[i][j][2 * e] = v.x; st[i][j][2 * e + 1] = v.y;
            }
    auto put_pair = [&](int off, int tile, int r, int c, float vx, float vy) {   // hi at off, lo `tile` elements behind
        uint32_t hi, lo;
        split_bf16x2(vx, vy, hi, lo);
        *reinterpret_cast<uint32_t*>(sm + off + r * LDN + c) = hi;
        *reinterpret_cast<uint32_t*>(sm + off + tile + r * LDN + c) = lo;
    };
    auto put_state = [&]() {
#pragma unroll
        for (int i = 0; i < NI; ++i)
#pragma unroll
            for (int j = 0; j < 2; ++j)
#pragma unroll
                for (int e = 0; e < 2; ++e) put_pair(L::os, DK * LDN, sm0 + lr + e * 8, sn0 + i * 16 + j * 8 + lc, st[i][j][2 * e], st[i][j][2 * e + 1]);
    };
    fetch1(0); fetch2(0); fetch3(0);
    put_state();
    cp_wait<2>();
    __syncthreads();

    const SmemMat sh = mat(L::os, LDN), slo = mat(L::os + DK * LDN, LDN), vt = mat(L::ov, LDN);
    const SmemMat rh = mat(L::orr, LDN), rl = mat(L::orr + L::VT, LDN), uh = mat(L::ou, LDN), ul = mat(L::ou + L::VT, LDN), wh = mat(L::ow, LDN), wl = mat(L::ow + L::VT, LDN);
    const SmemMat th = mat(L::ot, LDT), tl = mat(L::ot + L::TT, LDT), ph = mat(L::op, LDT), pl = mat(L::op + L::TT, LDT);
    // tiles of the products with 64 rows: warps 0..3 k, 4..7 q, two 16-column blocks each; time mixing: a block per warp
    constexpr int NQ = MODE == TIME_MIX ? 1 : 2;
    const int mt = warp & 3, half = warp >> 2, qn0 = MODE == TIME_MIX ? half * 16 : 0;
    const bool is_q = MODE == TIME_MIX || half == 1;
    for (int ch = 0; ch < chunks; ++ch) {
        const float* scal = s_scal + (ch & 1) * 4 * C;
        const int rows = min(C, s.n - ch * C);
        // decayed k and q against the state
        float acc[NQ][2][4];
#pragma unroll
        for (int i = 0; i < NQ; ++i)
#pragma unroll
            for (int j = 0; j < 2; ++j)
#pragma unroll
                for (int e = 0; e < 4; ++e) acc[i][j][e] = 0.f;
        {
            const SmemMat ah = is_q ? mat(L::oq, LDK) : mat(MODE == HEAD_DELTA ? (ch & 1) * L::KT : 0, LDK), al = is_q ? mat(L::oq + L::KT, LDK) : mat(L::KT, LDK);
#pragma unroll
            for (int kt = 0; kt < DK / 16; ++kt) {
                uint32_t fh[4], fl[4];
                ah.a(fh, mt * 16, kt * 16, lane);
                if constexpr (MODE != HEAD_DELTA) al.a(fl, mt * 16, kt * 16, lane);
#pragma unroll
                for (int i = 0; i < NQ; ++i) {
                    uint32_t gh[4], gl[4];
                    sh.b_t(gh, kt * 16, qn0 + i * 16, lane);
                    slo.b_t(gl, kt * 16, qn0 + i * 16, lane);
#pragma unroll
                    for (int j = 0; j < 2; ++j) {
                        if constexpr (MODE != HEAD_DELTA) mma(acc[i][j], fl, gh[2 * j], gh[2 * j + 1]);
                        mma(acc[i][j], fh, gl[2 * j], gl[2 * j + 1]);
                        mma(acc[i][j], fh, gh[2 * j], gh[2 * j + 1]);
                    }
                }
            }
        }
        if constexpr (MODE != TIME_MIX) {
            if (!is_q) {   // R = beta (v - decayed k against the state)
#pragma unroll
                for (int i = 0; i < NQ; ++i)
#pragma unroll
                    for (int j = 0; j < 2; ++j)
#pragma unroll
                        for (int e = 0; e < 2; ++e) {
                            const int t = mt * 16 + lr + e * 8, c = i * 16 + j * 8 + lc;
                            const float2 v = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(sm + L::ov + t * LDN + c));
                            const float k = MODE == HEAD_DELTA ? scal[kScalKin + t] : 1.f, b = scal[kScalBeta + t];
                            put_pair(L::orr, L::VT, t, c, b * (v.x - k * acc[i][j][2 * e]), b * (v.y - k * acc[i][j][2 * e + 1]));
                        }
            }
            cp_wait<1>();          // T
            __syncthreads();
            fetch1(ch + 1);
            // U = T R, a 16 x 16 block per warp
            float u[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
#pragma unroll
            for (int kt = 0; kt < C / 16; ++kt)
                if (kt <= mt) {
                    uint32_t fh[4], fl[4], gh[4], gl[4];
                    th.a(fh, mt * 16, kt * 16, lane); tl.a(fl, mt * 16, kt * 16, lane);
                    rh.b_t(gh, kt * 16, half * 16, lane); rl.b_t(gl, kt * 16, half * 16, lane);
#pragma unroll
                    for (int j = 0; j < 2; ++j) {
                        mma(u[j], fl, gh[2 * j], gh[2 * j + 1]);
                        mma(u[j], fh, gl[2 * j], gl[2 * j + 1]);
                        mma(u[j], fh, gh[2 * j], gh[2 * j + 1]);
                    }
                }
#pragma unroll
            for (int j = 0; j < 2; ++j)
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    const int t = mt * 16 + lr + e * 8, c = half * 16 + j * 8 + lc;
                    put_pair(L::ou, L::VT, t, c, u[j][2 * e], u[j][2 * e + 1]);
                    if constexpr (MODE == HEAD_DELTA) { const float k = scal[kScalKout + t]; put_pair(L::ow, L::VT, t, c, k * u[j][2 * e], k * u[j][2 * e + 1]); }
                }
            cp_wait<1>();          // P and the update's k
            __syncthreads();
            fetch2(ch + 1);
        } else {
            cp_wait<0>();
            __syncthreads();
            fetch1(ch + 1);
            fetch2(ch + 1);
        }
        // the state's update
        {
            const float* end = s_end + (ch & 1) * DK;
            const float e0 = end[sm0 + lr], e1 = end[sm0 + lr + 8];
#pragma unroll
            for (int i = 0; i < NI; ++i)
#pragma unroll
                for (int j = 0; j < 2; ++j) { st[i][j][0] *= e0; st[i][j][1] *= e0; st[i][j][2] *= e1; st[i][j][3] *= e1; }
            const SmemMat kh = MODE == HEAD_DELTA ? mat((ch & 1) * L::KT, LDK) : mat(L::oo, LDK), kl = mat(L::oo + L::KT, LDK);
#pragma unroll
            for (int kt = 0; kt < C / 16; ++kt) {
                uint32_t fh[4], fl[4];
                kh.a_t(fh, kt * 16, sm0, lane);
                if constexpr (MODE != HEAD_DELTA) kl.a_t(fl, kt * 16, sm0, lane);
#pragma unroll
                for (int i = 0; i < NI; ++i) {
                    uint32_t gh[4], gl[4];
                    (MODE == TIME_MIX ? vt : MODE == HEAD_DELTA ? wh : uh).b_t(gh, kt * 16, sn0 + i * 16, lane);
                    if constexpr (MODE != TIME_MIX) (MODE == HEAD_DELTA ? wl : ul).b_t(gl, kt * 16, sn0 + i * 16, lane);
#pragma unroll
                    for (int j = 0; j < 2; ++j) {
                        if constexpr (MODE != HEAD_DELTA) mma(st[i][j], fl, gh[2 * j], gh[2 * j + 1]);
                        if constexpr (MODE != TIME_MIX) mma(st[i][j], fh, gl[2 * j], gl[2 * j + 1]);
                        mma(st[i][j], fh, gh[2 * j], gh[2 * j + 1]);
                    }
                }
            }
            put_state();   // read again behind the next barrier only
        }
        if (is_q) {        // read-out
            if constexpr (MODE == HEAD_DELTA) {
                const float q0 = scal[kScalQin + mt * 16 + lr], q1 = scal[kScalQin + mt * 16 + lr + 8];
#pragma unroll
                for (int i = 0; i < NQ; ++i)
#pragma unroll
                    for (int j = 0; j < 2; ++j) { acc[i][j][0] *= q0; acc[i][j][1] *= q0; acc[i][j][2] *= q1; acc[i][j][3] *= q1; }
            }
#pragma unroll
            for (int kt = 0; kt < C / 16; ++kt)
                if (kt <= mt) {
                    uint32_t fh[4], fl[4];
                    ph.a(fh, mt * 16, kt * 16, lane); pl.a(fl, mt * 16, kt * 16, lane);
#pragma unroll
                    for (int i = 0; i < NQ; ++i) {
                        uint32_t gh[4], gl[4];
                        (MODE == TIME_MIX ? vt : uh).b_t(gh, kt * 16, qn0 + i * 16, lane);
                        if constexpr (MODE != TIME_MIX) ul.b_t(gl, kt * 16, qn0 + i * 16, lane);
#pragma unroll
                        for (int j = 0; j < 2; ++j) {
                            mma(acc[i][j], fl, gh[2 * j], gh[2 * j + 1]);
                            if constexpr (MODE != TIME_MIX) mma(acc[i][j], fh, gl[2 * j], gl[2 * j + 1]);
                            mma(acc[i][j], fh, gh[2 * j], gh[2 * j + 1]);
                        }
                    }
                }
#pragma unroll
            for (int i = 0; i < NQ; ++i)
#pragma unroll
                for (int j = 0; j < 2; ++j)
#pragma unroll
                    for (int e = 0; e < 2; ++e) {
                        const int t = mt * 16 + lr + e * 8, c = c0 + qn0 + i * 16 + j * 8 + lc;
                        if (t < rows && c < d.vdim) *reinterpret_cast<float2*>(sc.o + (size_t(s.row0 + ch * C + t) * d.heads + h) * d.vdim + c) = make_float2(acc[i][j][2 * e], acc[i][j][2 * e + 1]);
                    }
        }
        cp_wait<1>();              // the next chunk's first operands
        __syncthreads();
        fetch3(ch + 1);
    }
    cp_wait<0>();
#pragma unroll
    for (int i = 0; i < NI; ++i)
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const int r = sm0 + lr + e * 8, c = sn0 + i * 16 + j * 8 + lc;
                if (r < d.dim && c0 + c < d.vdim) *reinterpret_cast<float2*>(S + size_t(r) * d.vdim + c) = make_float2(st[i][j][2 * e], st[i][j][2 * e + 1]);
            }
}

template <int DK, int MODE>
int32_t launch(const RecurDims& d, const RecurArgs& a, const RecurScratch& sc, const ScanSeg* segs, int n_segs, int n_chunks, cudaStream_t st) {
    auto prep = chunk_prep_kernel<DK, MODE>;
    FORGE_CUDA(cudaFuncSetAttribute(prep, cudaFuncAttributeMaxDynamicSharedMemorySize, int(Prep<DK, MODE>::smem)));
    prep<<<dim3(n_chunks, d.heads), Prep<DK, MODE>::NT, Prep<DK, MODE>::smem, st>>>(d, a, sc, segs, n_segs);
    FORGE_LAUNCH_CHECK();
    auto scan = chunk_scan_kernel<DK, MODE>;
    FORGE_CUDA(cudaFuncSetAttribute(scan, cudaFuncAttributeMaxDynamicSharedMemorySize, int(Scan<DK, MODE>::smem)));
    scan<<<dim3((d.vdim + NB - 1) / NB, d.heads, n_segs), 256, Scan<DK, MODE>::smem, st>>>(d, a, sc, segs);
    FORGE_LAUNCH_CHECK();
    return FORGE_OK;
}

int padded_dim(const RecurDims& d) { return d.dim <= 64 ? 64 : 128; }

}  // namespace

bool recur_chunked_supported(const RecurDims& d) { return d.dim <= 128 && d.dim % 8 == 0 && d.vdim % 8 == 0; }

ChunkBytes recur_chunk_bytes(const RecurDims& d) {
    const size_t h = size_t(d.heads), dk = size_t(padded_dim(d));
    return {h * 4 * C * C * 2, h * 4 * C * 4, h * dk * 4, d.channel ? h * 6 * C * dk * 2 : 0};
}

int32_t recur_chunked(const RecurDims& d, const RecurArgs& a, const RecurScratch& sc, const ScanSeg* segs, int n_segs, int n_chunks, cudaStream_t st) {
    if (n_segs <= 0) return FORGE_OK;
    auto go = [&](auto dk) -> int32_t {
        constexpr int DK = decltype(dk)::value;
        if (!d.delta) return launch<DK, TIME_MIX>(d, a, sc, segs, n_segs, n_chunks, st);
        return d.channel ? launch<DK, CHANNEL_DELTA>(d, a, sc, segs, n_segs, n_chunks, st) : launch<DK, HEAD_DELTA>(d, a, sc, segs, n_segs, n_chunks, st);
    };
    return padded_dim(d) == 64 ? go(std::integral_constant<int, 64>{}) : go(std::integral_constant<int, 128>{});
}

}  // namespace forge
