// Recurrent mixers over segments of a prompt, bfloat16 models, on the tensor cores: chunks of 64 tokens.
//
// With G_t the sum of a chunk's log decays up to and including token t, and S the state in front of the chunk,
//   delta rule    (I + L) U = R,  R_t = beta_t (v_t - S^T (e^{G_t} k_t)),  L_ts = beta_t sum_c k_tc k_sc e^{G_tc - G_sc}  (s < t)
//                 o_t = S^T (e^{G_t} q_t) + sum_{s <= t} P_ts u_s,         P_ts = sum_c q_tc k_sc e^{G_tc - G_sc}
//                 S <- e^{G_end} S + sum_s (e^{G_end - G_s} k_s) u_s^T
//   time mixing   U = V, o_t reads with e^{G_(t-1)} instead of e^{G_t}, and P_tt = sum_c q_tc bonus_c k_tc;
//   linear        U = V.
// chunk_prep_kernel (every chunk and head at once) inverts I + L and leaves P, U0 = (I + L)^-1 diag(beta) V and
// W = (I + L)^-1 diag(beta) e^G K, so that U = U0 - W S; chunk_scan_kernel walks a sequence's chunks with a block of 32 columns of
// the state in registers: two dependent products per chunk (U, then S), the read-out beside them.  What the walk reads lies in
// memory as the tiles its shared memory holds, so a tile is one bulk copy of a producer warp.
//
// Precision: q, k and v are the model's bf16 values; every factor that is not (decays, unit norms, W, P, U, the state) enters a product as
// a bf16 pair hi + lo, three products with f32 sums for two such factors.  Exponents are differences <= 0, so strong decays
// underflow to zero and nothing overflows: for decays per channel the pairs of a 16-token block are formed directly, and earlier
// blocks are reached through the sum at the block's start.
#include <algorithm>
#include <type_traits>

#include "mma.cuh"
#include "recurrent.cuh"
#include "tc5.cuh"

namespace forge {

namespace {

using bf16 = __nv_bfloat16;
using tc5::bulk_load;
using tc5::mbar_arrive;
using tc5::mbar_expect_tx;
using tc5::mbar_fence_init;
using tc5::mbar_init;
using tc5::mbar_wait;

constexpr int C = kRecurChunk;          // tokens of a chunk
constexpr int NB = 32;                  // value columns of a CTA of the walk
constexpr int LDT = C + 8, LDN = NB + 8, TT = C * LDT, VT = C * LDN;
enum Mode { HEAD_DELTA = 0, CHANNEL_DELTA = 1, TIME_MIX = 2, LINEAR = 3 };
__host__ __device__ constexpr bool writes_v(int mode) { return mode == TIME_MIX || mode == LINEAR; }   // U = V
constexpr float kLog2e = 1.4426950408889634f;

__device__ __forceinline__ uint32_t smem_addr(const void* p) { return uint32_t(__cvta_generic_to_shared(p)); }
__device__ __forceinline__ float ex2(float x) {   // 2^x
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

// What one chunk of one head leaves for the walk.  bf16 tiles: W hi, lo (delta rules); q (hi, lo where decays are per channel); k (the same);
// P hi, lo; v in blocks of 32 columns (time mixing).  f32: U0 in blocks [64][32] (delta rules), scale of q and of k's update per
// token (decay per head), e^{G_end} per channel.
template <int DK, int MODE> struct Rec {
    static constexpr bool PLAIN = writes_v(MODE);
    static constexpr int LDK = DK + 8, KT = C * LDK;
    static constexpr int nw = PLAIN ? 0 : 2, nx = MODE == HEAD_DELTA ? 1 : 2;
    static constexpr int oq = nw * KT, ok = oq + nx * KT, op = ok + nx * KT, ov = op + 2 * TT;
    static __host__ __device__ size_t halves(int nb) { return size_t(ov) + (PLAIN ? size_t(nb) * VT : 0); }
    static __host__ __device__ size_t floats(int nb) { return (PLAIN ? 0 : size_t(nb) * C * NB) + 2 * C + DK; }
    bf16* h; float* f;
    float *scal, *end;
    __device__ __forceinline__ Rec(const ChunkScratch& s, int chunk, int heads, int head, int nb) {
        const size_t i = size_t(chunk) * heads + head;
        h = s.half + i * halves(nb);
        f = s.f32 + i * floats(nb);
        scal = f + (PLAIN ? 0 : size_t(nb) * C * NB);
        end = scal + 2 * C;
    }
};

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

// lower triangle of an f32 matrix (LDL apart), its columns times `col` -> bf16 hi and lo tiles with zeros above
template <int NT>
__device__ __forceinline__ void put_lower(bf16* dst, const float* src, const float* col, int tid) {
    for (int e = tid; e < C * C / 2; e += NT) {
        const int r = e / (C / 2), c = (e % (C / 2)) * 2;
        uint32_t hi, lo;
        split_bf16x2(c <= r ? src[r * LDL + c] * (col ? col[c] : 1.f) : 0.f, c + 1 <= r ? src[r * LDL + c + 1] * (col ? col[c + 1] : 1.f) : 0.f, hi, lo);
        *reinterpret_cast<uint32_t*>(dst + r * LDT + c) = hi;
        *reinterpret_cast<uint32_t*>(dst + TT + r * LDT + c) = lo;
    }
}

template <int DK, int MODE> struct Prep {
    static constexpr int NT = MODE == HEAD_DELTA ? 256 : 512, LDK = DK + 8;
    static constexpr bool CH = MODE != HEAD_DELTA;
    static constexpr size_t tiles = size_t(2) * C * LDK * 2;                          // q (later v), k
    static constexpr size_t mats = size_t(2) * C * LDL * 4 + 3 * 272 * 4;             // L (later (I + L)^-1 as hi, lo), P (later (I + L)^-1), tmp
    static constexpr size_t chan = CH ? size_t(C) * DK * 4 + size_t(5) * DK * 4 + size_t(2) * (32 + 48) * LDK * 2 : 0;   // sums, block sums, operands of one block row (later decayed k)
    static constexpr size_t smem = tiles + mats + chan;
    static_assert(size_t(2) * TT * 2 <= size_t(C) * LDL * 4 + 3 * 272 * 4, "hi and lo fit where L and tmp lay");
};

template <int DK, int MODE>
__global__ void __launch_bounds__(Prep<DK, MODE>::NT) chunk_prep_kernel(const RecurDims d, const RecurArgs a, const RecurScratch sc, const ScanSeg* __restrict__ segs, int n_segs) {
    constexpr bool PLAIN = writes_v(MODE), TIME = MODE == TIME_MIX;
    using L = Prep<DK, MODE>;
    using R = Rec<DK, MODE>;
    constexpr int NT = L::NT, LDK = L::LDK, NW = NT / 32, KT = R::KT;
    extern __shared__ __align__(16) unsigned char sm_raw[];
    bf16* sq = reinterpret_cast<bf16*>(sm_raw);
    bf16* sk = sq + C * LDK;
    float* sp = reinterpret_cast<float*>(sm_raw + L::tiles);
    float* sl = sp + C * LDL;
    float* tmp = sl + C * LDL;                 // behind sl: both give way to the inverse's bf16 tiles
    float* sg = tmp + 3 * 272;                 // [64][DK] sums of the log decays inside their 16-token block (base 2)
    float* sb = sg + C * DK;                   // [5][DK] sums in front of each block, and the chunk's
    bf16* sa = reinterpret_cast<bf16*>(sb + 5 * DK);   // [2][32][LDK] rows k, then q, of a block row
    bf16* so = sa + 2 * 32 * LDK;              // [2][48][LDK] keys in front of it
    bf16* st = reinterpret_cast<bf16*>(sl);    // [2][64][LDT]
    __shared__ float s_ks[C], s_qs[C], s_beta[C], s_gt[C], s_col[C];
    __shared__ int s_seg;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int chunk = blockIdx.x, h = blockIdx.y, g = h / (d.heads / d.groups), nb = (d.vdim + NB - 1) / NB;
    for (int i = tid; i < n_segs; i += NT) if (segs[i].chunk0 <= chunk && chunk < segs[i].chunk0 + (segs[i].n + C - 1) / C) s_seg = i;
    __syncthreads();
    const ScanSeg s = segs[s_seg];
    const int t0 = (chunk - s.chunk0) * C, n = min(C, s.n - t0), row0 = s.row0 + t0;
    const R out(sc.chunk, chunk, d.heads, h, nb);
    const bf16* x = PLAIN ? static_cast<const bf16*>(a.x) : static_cast<const bf16*>(sc.conv);
    const size_t ld = PLAIN ? a.x_ld : d.channels();
    // [64] rows of the step, `cols` of its columns from col0 (zeros past `valid`)
    auto fetch = [&](bf16* dst, int l, int col0, int cols, int valid) {
        for (int i = tid; i < C * (cols / 8); i += NT) {
            const int t = i / (cols / 8), c = (i % (cols / 8)) * 8;
            const bool ok = t < n && c < valid;
            cp_async16(smem_addr(dst + t * l + c), ok ? x + size_t(row0 + t) * ld + col0 + c : x, ok);
        }
    };
    fetch(sq, LDK, g * d.dim, DK, d.dim);
    fetch(sk, LDK, d.qk() + g * d.dim, DK, d.dim);
    cp_commit();
    if (tid < C) {
        const bool ok = tid < n;
        s_ks[tid] = s_beta[tid] = 1.f;
        s_qs[tid] = d.q_scale;
        if constexpr (!PLAIN) {
            s_ks[tid] = ok ? sc.unit[size_t(row0 + tid) * 2 * d.groups + d.groups + g] : 0.f;   // |k|^-1
            s_qs[tid] = ok ? sc.unit[size_t(row0 + tid) * 2 * d.groups + g] : 0.f;              // q scale
            s_beta[tid] = ok ? a.beta[size_t(row0 + tid) * d.heads + h] : 0.f;
        }
        if constexpr (MODE == HEAD_DELTA) s_gt[tid] = ok ? a.decay[size_t(row0 + tid) * a.decay_ld + h] * kLog2e : 0.f;
    }
    if constexpr (L::CH) {
        // sums inside the blocks: a thread per block and channel
        for (int i = tid; i < 4 * DK; i += NT) {
            const int b = i / DK, c = i % DK;
            float v[16], sum = 0.f;
#pragma unroll
            for (int t = 0; t < 16; ++t) v[t] = b * 16 + t < n && c < d.dim ? a.decay[size_t(row0 + b * 16 + t) * a.decay_ld + h * d.dim + c] : 0.f;
#pragma unroll
            for (int t = 0; t < 16; ++t) { sum = fmaf(v[t], kLog2e, sum); sg[(b * 16 + t) * DK + c] = sum; }
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
            for (int b = 0; b < 4; ++b)
                if (b <= mt) {
                    uint32_t fb[4];
                    mk.b(fb, b * 16, kt * 16, lane);
                    mma(acc[2 * b], fa, fb[0], fb[1]);
                    mma(acc[2 * b + 1], fa, fb[2], fb[3]);
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
                dst[t * LDL + c] = c <= t ? acc[i][e] * s_ks[c] * ex2(s_gt[t] - s_gt[c]) * (is_q ? s_qs[t] : s_ks[t] * s_beta[t]) : 0.f;
            }
        if (tid < C) {
            const float e = ex2(s_gt[tid]);
            s_col[tid] = e * s_ks[tid];
            out.scal[tid] = e * s_qs[tid];
            out.scal[C + tid] = ex2(s_gt[C - 1] - s_gt[tid]) * s_ks[tid];
        }
        if (tid < DK) out.end[tid] = ex2(s_gt[C - 1]);
        for (int i = tid; i < 2 * KT / 8; i += NT) reinterpret_cast<uint4*>(out.h + R::oq)[i] = reinterpret_cast<const uint4*>(sq)[i];   // q, k as they are (padding columns too)
        __syncthreads();
    } else {
        for (int c = tid; c < DK; c += NT) {
            float sum = 0.f;
#pragma unroll
            for (int b = 0; b < 4; ++b) { sb[b * DK + c] = sum; sum += sg[(b * 16 + 15) * DK + c]; }
            sb[4 * DK + c] = sum;
            out.end[c] = ex2(sum);
        }
        // exponents of a query row inside its block: up to and including its own decay, or for time mixing without it
        auto sum_q = [&](int t) { return TIME ? sg + (t - 1) * DK : sg + t * DK; };
        auto first = [](int t) { return TIME && !(t & 15); };   // then they are zero
        // pairs inside a block: a warp per row, DK / 32 neighbouring channels per lane, sixteen partners at once
        constexpr int PL = DK / 32;
        for (int t = warp; t < C; t += NW) {
            float qv[PL], kv[PL], eq[PL];
            const int c = lane * PL;
#pragma unroll
            for (int i = 0; i < PL; ++i) {
                qv[i] = __bfloat162float(sq[t * LDK + c + i]); kv[i] = __bfloat162float(sk[t * LDK + c + i]);
                eq[i] = first(t) ? 0.f : sum_q(t)[c + i];
            }
            float part[32];   // P of the sixteen partners, then L
#pragma unroll
            for (int j = 0; j < 16; ++j) {
                const int u = (t & ~15) + j;
                part[j] = part[16 + j] = 0.f;
                if (u > t) continue;
#pragma unroll
                for (int i = 0; i < PL; ++i) {
                    const float ku = __bfloat162float(sk[u * LDK + c + i]), gu = sg[u * DK + c + i];
                    if constexpr (TIME) part[j] = fmaf(qv[i] * ku, u < t ? ex2(eq[i] - gu) : c + i < d.dim ? a.bonus[h * d.dim + c + i] : 0.f, part[j]);
                    else { const float e = ex2(eq[i] - gu) * ku; part[j] = fmaf(qv[i], e, part[j]); if (!PLAIN) part[16 + j] = fmaf(kv[i], e, part[16 + j]); }
                }
            }
            // lane l ends with the sum of part[l]
#pragma unroll
            for (int w = 16; w > 0; w >>= 1)
#pragma unroll
                for (int i = 0; i < w; ++i) {
                    const bool up = lane & w;
                    const float send = up ? part[i] : part[i + w], mine = up ? part[i + w] : part[i];
                    part[i] = mine + __shfl_xor_sync(0xffffffffu, send, w);
                }
            const int j = lane & 15, u = (t & ~15) + j;
            if (u <= t) {
                if (lane < 16) sp[t * LDL + u] = part[0] * s_qs[t] * s_ks[u];
                else if (!PLAIN) sl[t * LDL + u] = part[0] * s_beta[t] * s_ks[t] * s_ks[u];
            }
        }
        __syncthreads();
        // earlier blocks, reached through the sum at the block's start
        for (int b = 1; b < 4; ++b) {
            for (int i = tid; i < (32 + 16 * b) * (DK / 2); i += NT) {
                const int r = i / (DK / 2), c = (i % (DK / 2)) * 2, t = b * 16 + (r & 15), u = r - 32;
                const float2 v = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>((r < 16 ? sk + t * LDK : r < 32 ? sq + t * LDK : sk + u * LDK) + c));
                float2 e;
                if (r < 16) e = *reinterpret_cast<const float2*>(sg + t * DK + c);
                else if (r < 32) e = first(t) ? make_float2(0.f, 0.f) : *reinterpret_cast<const float2*>(sum_q(t) + c);
                else {
                    const float2 f = *reinterpret_cast<const float2*>(sb + b * DK + c), o = *reinterpret_cast<const float2*>(sb + (u >> 4) * DK + c), w = *reinterpret_cast<const float2*>(sg + u * DK + c);
                    e = make_float2(f.x - o.x - w.x, f.y - o.y - w.y);
                }
                uint32_t hi, lo;
                split_bf16x2(v.x * ex2(e.x), v.y * ex2(e.y), hi, lo);
                bf16* dst = r < 32 ? sa + r * LDK + c : so + u * LDK + c;
                *reinterpret_cast<uint32_t*>(dst) = hi;
                *reinterpret_cast<uint32_t*>(dst + (r < 32 ? 32 : 48) * LDK) = lo;
            }
            __syncthreads();
            const SmemMat ah{smem_addr(sa), LDK}, al{smem_addr(sa + 32 * LDK), LDK}, bh{smem_addr(so), LDK}, bl{smem_addr(so + 48 * LDK), LDK};
            for (int w = warp; w < 4 * b; w += NW) {   // (k or q) x 8 earlier keys
                const int is_q = w & 1, n8 = w >> 1;
                if (PLAIN && !is_q) continue;
                float acc[3][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
#pragma unroll
                for (int kt = 0; kt < DK / 16; ++kt) {
                    uint32_t fh[4], fl[4], gh[4], gl[4];
                    ah.a(fh, is_q * 16, kt * 16, lane); al.a(fl, is_q * 16, kt * 16, lane);
                    bh.b(gh, (n8 >> 1) * 16, kt * 16, lane); bl.b(gl, (n8 >> 1) * 16, kt * 16, lane);
                    const int j = (n8 & 1) * 2;
                    mma(acc[0], fl, j ? gh[2] : gh[0], j ? gh[3] : gh[1]);
                    mma(acc[1], fh, j ? gl[2] : gl[0], j ? gl[3] : gl[1]);
                    mma(acc[2], fh, j ? gh[2] : gh[0], j ? gh[3] : gh[1]);
                }
                float* dst = is_q ? sp : sl;
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const int t = b * 16 + lr + (e >> 1) * 8, u = n8 * 8 + lc + (e & 1);
                    dst[t * LDL + u] = (acc[0][e] + acc[1][e] + acc[2][e]) * s_ks[u] * (is_q ? s_qs[t] : s_ks[t] * s_beta[t]);
                }
            }
            __syncthreads();
        }
        // q and k with their decays: for the walk, and k as an operand of W
        for (int i = tid; i < C * (DK / 2); i += NT) {
            const int t = i / (DK / 2), c = (i % (DK / 2)) * 2, b = t >> 4;
            const float2 q = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(sq + t * LDK + c)), k = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(sk + t * LDK + c));
            const float2 f = *reinterpret_cast<const float2*>(sb + b * DK + c), w = *reinterpret_cast<const float2*>(sg + t * DK + c), end = *reinterpret_cast<const float2*>(sb + 4 * DK + c);
            const float2 wq = first(t) ? make_float2(0.f, 0.f) : *reinterpret_cast<const float2*>(sum_q(t) + c);
            const float ks = s_ks[t], qs = s_qs[t];
            uint32_t hi, lo;
            split_bf16x2(q.x * qs * ex2(f.x + wq.x), q.y * qs * ex2(f.y + wq.y), hi, lo);
            uint32_t* dst = reinterpret_cast<uint32_t*>(out.h + R::oq + t * LDK + c);
            dst[0] = hi; dst[KT / 2] = lo;
            split_bf16x2(k.x * ks * ex2(end.x - f.x - w.x), k.y * ks * ex2(end.y - f.y - w.y), hi, lo);
            dst = reinterpret_cast<uint32_t*>(out.h + R::ok + t * LDK + c);
            dst[0] = hi; dst[KT / 2] = lo;
            if constexpr (!PLAIN) {
                split_bf16x2(k.x * ks * ex2(f.x + w.x), k.y * ks * ex2(f.y + w.y), hi, lo);
                dst = reinterpret_cast<uint32_t*>(sa + t * LDK + c);
                dst[0] = hi; dst[KT / 2] = lo;
            }
        }
        if constexpr (PLAIN) {   // v as the walk's tiles
            for (int i = tid; i < nb * C * (NB / 8); i += NT) {
                const int blk = i / (C * (NB / 8)), t = i / (NB / 8) % C, c = (i % (NB / 8)) * 8;
                const bool ok = t < n && blk * NB + c < d.vdim;
                *reinterpret_cast<uint4*>(out.h + R::ov + size_t(blk) * VT + t * LDN + c) =
                    ok ? *reinterpret_cast<const uint4*>(x + size_t(row0 + t) * ld + 2 * d.qk() + h * d.vdim + blk * NB + c) : make_uint4(0, 0, 0, 0);
            }
        }
    }
    put_lower<NT>(out.h + R::op, sp, nullptr, tid);
    if constexpr (!PLAIN) {
        __syncthreads();
        fetch(sq, LDK, 2 * d.qk() + h * d.vdim, DK, d.vdim);   // q gives way to the first columns of v
        cp_commit();
        invert_unit_lower<NT>(sp, sl, tmp, tid);               // P is stored: its place takes the inverse
        put_lower<NT>(st, sp, s_beta, tid);
        cp_wait<0>();
        __syncthreads();
        const SmemMat th{smem_addr(st), LDT}, tl{smem_addr(st + TT), LDT};
        // [64][cols] = (I + L)^-1 diag(beta) B in blocks of 16 x 16, B as one bf16 matrix or as hi and lo
        auto product = [&](const bf16* B, bool pair, int cols, auto store) {
            const SmemMat bh{smem_addr(B), LDK}, bl{smem_addr(B + KT), LDK};
            for (int w = warp; w < 4 * (cols / 16); w += NW) {
                const int mt = 3 - (w & 3), n0 = (w >> 2) * 16;
                float acc[2][2][4];
#pragma unroll
                for (int i = 0; i < 16; ++i) acc[i >> 3][(i >> 2) & 1][i & 3] = 0.f;
#pragma unroll
                for (int kt = 0; kt < C / 16; ++kt)
                    if (kt <= mt) {
                        uint32_t fh[4], fl[4], gh[4], gl[4];
                        th.a(fh, mt * 16, kt * 16, lane); tl.a(fl, mt * 16, kt * 16, lane);
                        bh.b_t(gh, kt * 16, n0, lane);
                        if (pair) bl.b_t(gl, kt * 16, n0, lane);
#pragma unroll
                        for (int j = 0; j < 2; ++j) {
                            mma(acc[0][j], fl, gh[2 * j], gh[2 * j + 1]);
                            if (pair) mma(acc[0][j], fh, gl[2 * j], gl[2 * j + 1]);
                            mma(acc[1][j], fh, gh[2 * j], gh[2 * j + 1]);
                        }
                    }
#pragma unroll
                for (int j = 0; j < 2; ++j)
#pragma unroll
                    for (int e = 0; e < 2; ++e) store(mt * 16 + lr + e * 8, n0 + j * 8 + lc, acc[0][j][2 * e] + acc[1][j][2 * e], acc[0][j][2 * e + 1] + acc[1][j][2 * e + 1]);
            }
        };
        for (int c0 = 0; c0 < d.vdim; c0 += DK) {   // U0
            if (c0) {
                __syncthreads();
                fetch(sq, LDK, 2 * d.qk() + h * d.vdim + c0, DK, d.vdim - c0);
                cp_commit();
                cp_wait<0>();
                __syncthreads();
            }
            product(sq, false, min(DK, (d.vdim - c0 + 15) / 16 * 16), [&](int t, int c, float vx, float vy) {
                *reinterpret_cast<float2*>(out.f + size_t((c0 + c) / NB) * C * NB + t * NB + (c0 + c) % NB) = make_float2(vx, vy);
            });
        }
        if constexpr (MODE == HEAD_DELTA) {         // W: the decay of k goes into the inverse's columns
            __syncthreads();
            if (tid < C) s_col[tid] *= s_beta[tid];
            __syncthreads();
            put_lower<NT>(st, sp, s_col, tid);
            __syncthreads();
        }
        product(MODE == HEAD_DELTA ? sk : sa, MODE != HEAD_DELTA, DK, [&](int t, int c, float vx, float vy) {
            uint32_t hi, lo;
            split_bf16x2(vx, vy, hi, lo);
            uint32_t* dst = reinterpret_cast<uint32_t*>(out.h + t * LDK + c);
            dst[0] = hi; dst[KT / 2] = lo;
        });
    }
}

// ------------------------------------------------------------------------------------------------ walk over the chunks
template <int DK, int MODE> struct Scan {
    static constexpr bool PLAIN = writes_v(MODE);
    using R = Rec<DK, MODE>;
    static constexpr int SS = DK * LDN;                              // one half of a state buffer
    static constexpr int ST = DK <= 64 ? 2 : 1;                      // buffers of every tile
    static constexpr int ow = 0, oq = R::nw * R::KT, ok = oq + R::nx * R::KT, op = ok + R::nx * R::KT, ov = op + 2 * TT, stage = ov + (PLAIN ? VT : 0), os = ST * stage,
                         ou = os + 4 * SS, ox = ou + (PLAIN ? 0 : 2 * VT), total = ox + (MODE == HEAD_DELTA ? 2 * VT : 0);
    static constexpr size_t smem = size_t(total) * 2 + 16;
};

constexpr int kScanThreads = 288;   // eight warps of products and a producer
__device__ __forceinline__ void walk_sync() { asm volatile("bar.sync 1, 256;" ::: "memory"); }

template <int DK, int MODE>
__global__ void __launch_bounds__(kScanThreads, 1) chunk_scan_kernel(const RecurDims d, const RecurArgs a, const RecurScratch sc, const ScanSeg* __restrict__ segs, int* err) {
    constexpr bool PLAIN = writes_v(MODE);
    using L = Scan<DK, MODE>;
    using R = Rec<DK, MODE>;
    constexpr int LDK = R::LDK, KT = R::KT, ST = L::ST;
    extern __shared__ __align__(16) unsigned char sm_raw[];
    bf16* sm = reinterpret_cast<bf16*>(sm_raw);
    enum { BW, BK, BQ, BP, BUFS };
    __shared__ uint64_t full[ST][BUFS], empty[ST][BUFS];
    __shared__ int s_err;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, lr = lane >> 2, lc = (lane & 3) * 2;
    const ScanSeg s = segs[blockIdx.z];
    const int h = blockIdx.y, c0 = blockIdx.x * NB, nb = gridDim.x, chunks = (s.n + C - 1) / C;
    if (tid == 0) {
        for (int i = 0; i < ST * BUFS; ++i) { mbar_init(&full[0][i], 1); mbar_init(&empty[0][i], 8); }
        s_err = 0;
        mbar_fence_init();
    }
    __syncthreads();
    if (warp == 8) {
        if (lane == 0) {
            bool ok = true;
            for (int ch = 0; ch < chunks && ok; ++ch) {
                const R r(sc.chunk, s.chunk0 + ch, d.heads, h, nb);
                auto load = [&](int buf, int dst, const bf16* src, int elems, const bf16* more = nullptr, int more_dst = 0, int more_elems = 0) {
                    if (!ok) return;
                    const int b = ch % ST;
                    if (ch >= ST && !mbar_wait(&empty[b][buf], (ch / ST - 1) & 1, &s_err)) { atomicExch(&s_err, 1); ok = false; return; }
                    mbar_expect_tx(&full[b][buf], uint32_t(elems + more_elems) * 2);
                    bulk_load(sm + b * L::stage + dst, src, uint32_t(elems) * 2, &full[b][buf]);
                    if (more_elems) bulk_load(sm + b * L::stage + more_dst, more, uint32_t(more_elems) * 2, &full[b][buf]);
                };
                if constexpr (!PLAIN) load(BW, L::ow, r.h, 2 * KT);
                load(BK, L::ok, r.h + R::ok, R::nx * KT, r.h + R::ov + size_t(blockIdx.x) * VT, L::ov, PLAIN ? VT : 0);
                load(BQ, L::oq, r.h + R::oq, R::nx * KT);
                load(BP, L::op, r.h + R::op, 2 * TT);
            }
        }
    } else {
        auto mat = [&](int off, int l) { return SmemMat{smem_addr(sm + off), l}; };
        // every warp meets at the barriers below, so a wait that gave up must not leave the loop alone
        auto take = [&](int buf, int ch) { if (!mbar_wait(&full[ch % ST][buf], (ch / ST) & 1, &s_err)) atomicExch(&s_err, 1); };
        auto give = [&](int buf, int ch) { __syncwarp(); if (lane == 0) mbar_arrive(&empty[ch % ST][buf]); };
        // the state: 16 rows and NI times 16 columns per warp
        constexpr int MW = DK / 16 < 8 ? DK / 16 : 8, NI = NB / 16 / (8 / MW);
        static_assert(DK / 16 / MW == 1 && NI >= 1, "one row tile per warp");
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
        auto put_pair = [&](int off, int half, int r, int c, float vx, float vy) {   // hi at off, lo `half` elements behind
            uint32_t hi, lo;
            split_bf16x2(vx, vy, hi, lo);
            *reinterpret_cast<uint32_t*>(sm + off + r * LDN + c) = hi;
            *reinterpret_cast<uint32_t*>(sm + off + half + r * LDN + c) = lo;
        };
        auto put_state = [&](int buf) {
#pragma unroll
            for (int i = 0; i < NI; ++i)
#pragma unroll
                for (int j = 0; j < 2; ++j)
#pragma unroll
                    for (int e = 0; e < 2; ++e) put_pair(L::os + buf * 2 * L::SS, L::SS, sm0 + lr + e * 8, sn0 + i * 16 + j * 8 + lc, st[i][j][2 * e], st[i][j][2 * e + 1]);
        };
        put_state(0);
        walk_sync();
        // products with 64 rows: 16 rows and 16 columns per warp
        const int mt = warp & 3, n0 = (warp >> 2) * 16, t_lo = mt * 16 + lr;
        const SmemMat xh = mat(L::ox, LDN), xl = mat(L::ox + VT, LDN), ul = mat(L::ou + VT, LDN);
        // what a thread reads of a chunk by itself, one chunk ahead
        struct Own { float2 u0[2][2]; float end[2], qd[2], ko[2]; };
        auto own = [&](int ch) {
            Own o;
            const R r(sc.chunk, s.chunk0 + min(ch, chunks - 1), d.heads, h, nb);
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                o.end[e] = r.end[sm0 + lr + 8 * e];
                if constexpr (MODE == HEAD_DELTA) { o.qd[e] = r.scal[t_lo + 8 * e]; o.ko[e] = r.scal[C + t_lo + 8 * e]; }
                if constexpr (!PLAIN)
#pragma unroll
                    for (int j = 0; j < 2; ++j) o.u0[j][e] = *reinterpret_cast<const float2*>(r.f + size_t(blockIdx.x) * C * NB + (t_lo + 8 * e) * NB + n0 + j * 8 + lc);
            }
            return o;
        };
        Own now = own(0);
        for (int ch = 0; ch < chunks; ++ch) {
            const Own next = own(ch + 1);
            const int at = ch % ST * L::stage;
            const SmemMat uh = mat(PLAIN ? at + L::ov : L::ou, LDN), ph = mat(at + L::op, LDT), pl = mat(at + L::op + TT, LDT);
            const SmemMat wh = mat(at + L::ow, LDK), wl = mat(at + L::ow + KT, LDK), qh = mat(at + L::oq, LDK), ql = mat(at + L::oq + KT, LDK), kh = mat(at + L::ok, LDK), kl = mat(at + L::ok + KT, LDK);
            const SmemMat sh = mat(L::os + (ch & 1) * 2 * L::SS, LDN), slo = mat(L::os + (ch & 1) * 2 * L::SS + L::SS, LDN);
            // the state in front of the chunk as B operands of two products (shared-memory reads bound this kernel)
            uint32_t gh[DK / 16][4], gl[DK / 16][4];
#pragma unroll
            for (int kt = 0; kt < DK / 16; ++kt) { sh.b_t(gh[kt], kt * 16, n0, lane); slo.b_t(gl[kt], kt * 16, n0, lane); }
            if constexpr (!PLAIN) {   // U = U0 - W S
                take(BW, ch);
                float acc[3][2][4];
#pragma unroll
                for (int i = 0; i < 24; ++i) acc[i / 8][(i >> 2) & 1][i & 3] = 0.f;
#pragma unroll
                for (int kt = 0; kt < DK / 16; ++kt) {
                    uint32_t fh[4], fl[4];
                    wh.a(fh, mt * 16, kt * 16, lane); wl.a(fl, mt * 16, kt * 16, lane);
#pragma unroll
                    for (int j = 0; j < 2; ++j) {
                        mma(acc[0][j], fl, gh[kt][2 * j], gh[kt][2 * j + 1]);
                        mma(acc[1][j], fh, gl[kt][2 * j], gl[kt][2 * j + 1]);
                        mma(acc[2][j], fh, gh[kt][2 * j], gh[kt][2 * j + 1]);
                    }
                }
                give(BW, ch);
#pragma unroll
                for (int j = 0; j < 2; ++j)
#pragma unroll
                    for (int e = 0; e < 2; ++e) {
                        const float ux = now.u0[j][e].x - (acc[0][j][2 * e] + acc[1][j][2 * e] + acc[2][j][2 * e]);
                        const float uy = now.u0[j][e].y - (acc[0][j][2 * e + 1] + acc[1][j][2 * e + 1] + acc[2][j][2 * e + 1]);
                        put_pair(L::ou, VT, t_lo + 8 * e, n0 + j * 8 + lc, ux, uy);
                        if constexpr (MODE == HEAD_DELTA) put_pair(L::ox, VT, t_lo + 8 * e, n0 + j * 8 + lc, now.ko[e] * ux, now.ko[e] * uy);
                    }
                walk_sync();
            }
            take(BK, ch);
            // the state's update
#pragma unroll
            for (int i = 0; i < NI; ++i)
#pragma unroll
                for (int j = 0; j < 2; ++j)
#pragma unroll
                    for (int e = 0; e < 4; ++e) st[i][j][e] *= now.end[e >> 1];
#pragma unroll
            for (int kt = 0; kt < C / 16; ++kt) {
                uint32_t fh[4], fl[4];
                kh.a_t(fh, kt * 16, sm0, lane);
                if constexpr (MODE != HEAD_DELTA) kl.a_t(fl, kt * 16, sm0, lane);
#pragma unroll
                for (int i = 0; i < NI; ++i) {
                    uint32_t gh[4], gl[4];
                    (MODE == HEAD_DELTA ? xh : uh).b_t(gh, kt * 16, sn0 + i * 16, lane);
                    if constexpr (!PLAIN) (MODE == HEAD_DELTA ? xl : ul).b_t(gl, kt * 16, sn0 + i * 16, lane);
#pragma unroll
                    for (int j = 0; j < 2; ++j) {
                        if constexpr (MODE != HEAD_DELTA) mma(st[i][j], fl, gh[2 * j], gh[2 * j + 1]);
                        if constexpr (!PLAIN) mma(st[i][j], fh, gl[2 * j], gl[2 * j + 1]);
                        mma(st[i][j], fh, gh[2 * j], gh[2 * j + 1]);
                    }
                }
            }
            if constexpr (!PLAIN) give(BK, ch);
            put_state((ch + 1) & 1);
            // the read-out: q against the state in front of the chunk, then P U
            take(BQ, ch);
            float acc[3][2][4];
#pragma unroll
            for (int i = 0; i < 24; ++i) acc[i / 8][(i >> 2) & 1][i & 3] = 0.f;
#pragma unroll
            for (int kt = 0; kt < DK / 16; ++kt) {
                uint32_t fh[4], fl[4];
                qh.a(fh, mt * 16, kt * 16, lane);
                if constexpr (MODE != HEAD_DELTA) ql.a(fl, mt * 16, kt * 16, lane);
#pragma unroll
                for (int j = 0; j < 2; ++j) {
                    if constexpr (MODE != HEAD_DELTA) mma(acc[0][j], fl, gh[kt][2 * j], gh[kt][2 * j + 1]);
                    mma(acc[1][j], fh, gl[kt][2 * j], gl[kt][2 * j + 1]);
                    mma(acc[2][j], fh, gh[kt][2 * j], gh[kt][2 * j + 1]);
                }
            }
            give(BQ, ch);
            if constexpr (MODE == HEAD_DELTA) {
#pragma unroll
                for (int i = 1; i < 3; ++i)
#pragma unroll
                    for (int j = 0; j < 2; ++j)
#pragma unroll
                        for (int e = 0; e < 4; ++e) acc[i][j][e] *= now.qd[e >> 1];
            }
            take(BP, ch);
#pragma unroll
            for (int kt = 0; kt < C / 16; ++kt)
                if (kt <= mt) {
                    uint32_t fh[4], fl[4], gh[4], gl[4];
                    ph.a(fh, mt * 16, kt * 16, lane); pl.a(fl, mt * 16, kt * 16, lane);
                    uh.b_t(gh, kt * 16, n0, lane);
                    if constexpr (!PLAIN) ul.b_t(gl, kt * 16, n0, lane);
#pragma unroll
                    for (int j = 0; j < 2; ++j) {
                        mma(acc[0][j], fl, gh[2 * j], gh[2 * j + 1]);
                        if constexpr (!PLAIN) mma(acc[1][j], fh, gl[2 * j], gl[2 * j + 1]);
                        mma(acc[2][j], fh, gh[2 * j], gh[2 * j + 1]);
                    }
                }
            give(BP, ch);
            if constexpr (PLAIN) give(BK, ch);   // v lies with k
            const int rows = s.n - ch * C;
#pragma unroll
            for (int j = 0; j < 2; ++j)
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    const int t = t_lo + 8 * e, c = c0 + n0 + j * 8 + lc;
                    if (t < rows && c < d.vdim)
                        *reinterpret_cast<float2*>(sc.o + (size_t(s.row0 + ch * C + t) * d.heads + h) * d.vdim + c) =
                            make_float2(acc[0][j][2 * e] + acc[1][j][2 * e] + acc[2][j][2 * e], acc[0][j][2 * e + 1] + acc[1][j][2 * e + 1] + acc[2][j][2 * e + 1]);
                }
            now = next;
            walk_sync();   // the new state is complete, U and the old state are read
        }
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
    __syncthreads();
    if (tid == 0 && s_err && err) atomicExch(err, 1);
}

template <int DK, int MODE>
int32_t launch(const RecurDims& d, const RecurArgs& a, const RecurScratch& sc, const ScanSeg* segs, int n_segs, int n_chunks, cudaStream_t st) {
    auto prep = chunk_prep_kernel<DK, MODE>;
    FORGE_CUDA(cudaFuncSetAttribute(prep, cudaFuncAttributeMaxDynamicSharedMemorySize, int(Prep<DK, MODE>::smem)));
    prep<<<dim3(n_chunks, d.heads), Prep<DK, MODE>::NT, Prep<DK, MODE>::smem, st>>>(d, a, sc, segs, n_segs);
    FORGE_LAUNCH_CHECK();
    auto scan = chunk_scan_kernel<DK, MODE>;
    FORGE_CUDA(cudaFuncSetAttribute(scan, cudaFuncAttributeMaxDynamicSharedMemorySize, int(Scan<DK, MODE>::smem)));
    scan<<<dim3((d.vdim + NB - 1) / NB, d.heads, n_segs), kScanThreads, Scan<DK, MODE>::smem, st>>>(d, a, sc, segs, sc.err);
    FORGE_LAUNCH_CHECK();
    return FORGE_OK;
}

template <typename F> auto dispatch(const RecurDims& d, F f) {
    auto mode = [&](auto dk) {
        if (d.rule == Rule::TimeMix) return f(dk, std::integral_constant<int, TIME_MIX>{});
        if (d.rule == Rule::Linear) return f(dk, std::integral_constant<int, LINEAR>{});
        return d.channel ? f(dk, std::integral_constant<int, CHANNEL_DELTA>{}) : f(dk, std::integral_constant<int, HEAD_DELTA>{});
    };
    return d.dim <= 64 ? mode(std::integral_constant<int, 64>{}) : mode(std::integral_constant<int, 128>{});
}

}  // namespace

bool recur_chunked_supported(const RecurDims& d) { return d.dim <= 128 && d.dim % 8 == 0 && d.vdim % 8 == 0; }

ChunkBytes recur_chunk_bytes(const RecurDims& d) {
    const size_t h = size_t(d.heads);
    const int nb = (d.vdim + NB - 1) / NB;
    return dispatch(d, [&](auto dk, auto mode) {
        using R = Rec<decltype(dk)::value, decltype(mode)::value>;
        return ChunkBytes{h * R::halves(nb) * 2, h * R::floats(nb) * 4};
    });
}

int32_t recur_chunked(const RecurDims& d, const RecurArgs& a, const RecurScratch& sc, const ScanSeg* segs, int n_segs, int n_chunks, cudaStream_t st) {
    if (n_segs <= 0) return FORGE_OK;
    return dispatch(d, [&](auto dk, auto mode) { return launch<decltype(dk)::value, decltype(mode)::value>(d, a, sc, segs, n_segs, n_chunks, st); });
}

}  // namespace forge
