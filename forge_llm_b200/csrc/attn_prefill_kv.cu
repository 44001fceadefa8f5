// Prompt attention of the layer-list models, bfloat16, tcgen05: over keys and values formed for this call (latent attention) or over
// the pages of the cache (a page is one key tile).  The structure is that of attn_prefill_tc5.cu - S = Q K^T in tensor memory,
// lazy running maximum, probabilities back into tensor memory as the operand of O += P V, three overlapped stages - with these
// differences: the query / key width (a part per head plus, optionally, a part whose keys all heads share) and the value width
// are independent run-time sizes, several query heads may share a key head, the scores may be capped and the keys limited to the
// query's chunk or window (with the first tokens kept: their key tiles come first; or blocks in front of it seen as one key: then tiles of
// those come first, gathered into rows by sequence), scores may have a bias by distance, a sink may stand in the denominator, several sequences'
// tiles run in one launch (a table gives each tile's rows, position and context), and the epilogue applies an output gate per value or per
// head.  Joint values: a CTA meets up to four 64-column pieces of all groups' values, so that heads' weights can be mixed behind it.
// Warp roles (192 threads): 0 = TMA producer, 1 = TMEM allocation and MMA issue, 2..5 = softmax, rescale, store.  Where a bound of the scores is known
// (BOUND, 320 threads) it stands in for the maximum: nothing is ever rescaled, and eight warps, two per 32 rows, take half of a tile's columns each.
// Tensor memory: S [0, 64), P0 [64, 96), P1 [96, 128), O from 128.
#include <algorithm>

#include "attn_prompt.cuh"
#include "tc5.cuh"

namespace forge {

namespace {

using namespace tc5;

constexpr int BM = 128, BN = 64;
constexpr uint32_t kColS = 0, kColP = 64, kColO = 128;
constexpr float kLazy = 8.f;
constexpr float kMostBound = 35.f;   // weights from exp(-2 * 35) on are far from the smallest numbers

struct Params {
    PromptDims d;
    PromptAttnArgs a;
    float scale2;
    int stages;
    int pieces;          // 64-column pieces of values per CTA, at most
};

__host__ __device__ __forceinline__ int first_visible(const PromptDims& d, int pos) { return d.chunk > 0 ? pos / d.chunk * d.chunk : d.window > 0 && pos >= d.window ? pos - d.window + 1 : 0; }
// key tiles: `head` tiles of kept first tokens or of blocks, then from jb, the first one that anybody's chunk or window reaches
__host__ __device__ __forceinline__ int head_tiles(const PromptDims& d, const PromptTile& t, int jb) {
    if (d.pool > 0) return (first_visible(d, t.pos0 + t.rows - 1) / d.pool + BN - 1) / BN;
    const int k = (d.keep + BN - 1) / BN;
    return d.window > 0 ? (jb < k ? jb : k) : 0;
}
__host__ __device__ __forceinline__ int value_pieces(const PromptDims& d) { return d.vdim_p / 64 * (d.joint ? d.heads / d.share : 1); }
constexpr int kBiasRow = 4096;     // longest bias row that is kept in shared memory
__host__ __device__ __forceinline__ int bias_row(const PromptDims& d) { return d.bias_n <= kBiasRow ? d.bias_n : 0; }

__device__ __forceinline__ float ex2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

template <uint32_t COLS, bool BOUND>
__global__ void __launch_bounds__(BOUND ? 320 : 192, COLS <= 256 ? 2 : 1) attn_prefill_kv_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_k,
                                                                   const __grid_constant__ CUtensorMap map_r, const __grid_constant__ CUtensorMap map_v, const __grid_constant__ CUtensorMap map_bk,
                                                                   const __grid_constant__ CUtensorMap map_bv, const __grid_constant__ Params p) {
    constexpr int WARPS = BOUND ? 8 : 4, kThreads = 64 + 32 * WARPS, NC = BOUND ? 32 : 64;   // softmax warps; columns of a tile per thread
    constexpr int Q_CHUNK = BM * 128, KV_CHUNK = BN * 128, kMaxStages = 3;
    const PromptDims& d = p.d;
    const int h = int(blockIdx.x) % d.heads, vp0 = int(blockIdx.x) / d.heads * p.pieces;   // first piece of the values
    const int kch = d.dim_p / 64, rch = d.rot_p / 64, vch = min(p.pieces, value_pieces(d) - vp0), qch = kch + rch;
    const int stage_bytes = (qch + p.pieces) * KV_CHUNK, KVS = p.stages;
    extern __shared__ __align__(1024) unsigned char smem_raw[];
    unsigned char* sQ = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
    unsigned char* sKV = sQ + qch * Q_CHUNK;
    float* sBias = reinterpret_cast<float*>(sKV + KVS * stage_bytes);
    __shared__ uint64_t q_full, kv_full[kMaxStages], kv_empty[kMaxStages], s_full, s_free, p_full[2], pv_done[2];
    __shared__ uint32_t s_tmem;
    __shared__ int s_err;
    __shared__ float s_sum[BOUND ? 2 : 1][BM];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const PromptTile t = p.a.tiles[blockIdx.y];
    auto first_key = [&](int pos) { return first_visible(d, pos); };
    const int jb = first_key(t.pos0) / BN, head = head_tiles(d, t, jb);
    const int nblk = head + (t.pos0 + t.rows - 1) / BN + 1 - jb;
    auto key_tile = [&](int j) { return j < head ? j : jb + j - head; };

    if (tid == 0) {
        mbar_init(&q_full, 1);
        for (int s = 0; s < kMaxStages; ++s) { mbar_init(&kv_full[s], 1); mbar_init(&kv_empty[s], 1); }
        mbar_init(&s_full, 1);
        mbar_init(&s_free, WARPS);
        for (int s = 0; s < 2; ++s) { mbar_init(&p_full[s], WARPS); mbar_init(&pv_done[s], 1); }
        s_err = 0;
        mbar_fence_init();
    }
    if (warp == 1) tmem_alloc<COLS>(&s_tmem);
    if (p.a.bias) for (int i = tid; i < bias_row(d); i += kThreads) sBias[i] = p.a.bias[size_t(h) * d.bias_n + i] * 1.4426950408889634f;
    fence_before();
    __syncthreads();
    fence_after();
    const uint32_t tmem = s_tmem;

    if (warp == 0) {
        if (lane == 0) {
            mbar_expect_tx(&q_full, uint32_t(qch * Q_CHUNK));
            for (int c = 0; c < qch; ++c) tma_3d(sQ + c * Q_CHUNK, &map_q, c * 64, h, t.row0, &q_full);
            for (int j = 0; j < nblk; ++j) {
                const int s = j % KVS, use = j / KVS;
                if (use > 0 && !mbar_wait(&kv_empty[s], (use - 1) & 1, &s_err)) { atomicExch(&s_err, 1); break; }
                const bool blocks = d.pool > 0 && j < head;
                const int row = blocks ? t.pool0 + j * BN : p.a.pages ? p.a.pages[t.ctx0 / BN + key_tile(j)] * BN : t.ctx0 + key_tile(j) * BN, hk = h / d.share;
                unsigned char* dst = sKV + size_t(s) * stage_bytes;
                mbar_expect_tx(&kv_full[s], uint32_t((qch + vch) * KV_CHUNK));
                for (int c = 0; c < kch; ++c) tma_3d(dst + c * KV_CHUNK, blocks ? &map_bk : &map_k, c * 64, hk, row, &kv_full[s]);
                for (int c = 0; c < rch; ++c) tma_2d(dst + (kch + c) * KV_CHUNK, &map_r, c * 64, row, &kv_full[s]);
                for (int c = 0; c < vch; ++c) {
                    const int per = d.vdim_p / 64, piece = vp0 + c;
                    tma_3d(dst + (qch + c) * KV_CHUNK, blocks ? &map_bv : &map_v, piece % per * 64, d.joint ? piece / per : hk, row, &kv_full[s]);
                }
            }
        }
    } else if (warp == 1) {
        if (lane == 0) {
            bool ok = mbar_wait(&q_full, 0, &s_err);
            const uint32_t q_base = smem_u32(sQ);
            const int ks = (d.dim + 15) / 16, rs = (d.rot + 15) / 16;   // sixteen-wide steps that hold anything
            auto issue_s = [&](int j) {
                const uint32_t k_base = smem_u32(sKV + size_t(j % KVS) * stage_bytes);
                for (int i = 0; i < ks + rs; ++i) {
                    const int step = i < ks ? i : kch * 4 + (i - ks);
                    const uint32_t off = uint32_t(step / 4), in = uint32_t((step % 4) * 32);
                    umma_ss(tmem + kColS, desc_kmajor(q_base + off * Q_CHUNK + in), desc_kmajor(k_base + off * KV_CHUNK + in), idesc_bf16(BN), i > 0 ? 1u : 0u);
                }
                umma_commit(&s_full);
            };
            if (ok && mbar_wait(&kv_full[0], 0, &s_err)) { fence_after(); issue_s(0); }
            else ok = false;
            const uint32_t id_v = idesc_bf16(vch * 64, true);
            for (int j = 0; j < nblk && ok; ++j) {
                if (j + 1 < nblk) {
                    if (!mbar_wait(&kv_full[(j + 1) % KVS], ((j + 1) / KVS) & 1, &s_err) || !mbar_wait(&s_free, j & 1, &s_err)) { ok = false; break; }
                    fence_after();
                    issue_s(j + 1);
                }
                if (!mbar_wait(&p_full[j & 1], (j >> 1) & 1, &s_err)) { ok = false; break; }
                fence_after();
                const uint32_t v_base = smem_u32(sKV + size_t(j % KVS) * stage_bytes) + qch * KV_CHUNK;
#pragma unroll
                for (int k16 = 0; k16 < BN / 16; ++k16)
                    umma_ts(tmem + kColO, tmem + kColP + uint32_t((j & 1) * 32 + k16 * 8), desc_mnmajor(v_base + k16 * 2048, KV_CHUNK), id_v, (j > 0 || k16 > 0) ? 1u : 0u);
                umma_commit(&pv_done[j & 1]);
                umma_commit(&kv_empty[j % KVS]);
            }
            if (!ok) atomicExch(&s_err, 1);
        }
    } else {
        const int quad = warp & 3, half = BOUND ? (warp - 2) / 4 : 0, col0 = half * NC;   // of the tile
        const int r = quad * 32 + lane;
        const int pq = t.pos0 + r, lo = first_key(pq), keep = d.window > 0 ? d.keep : 0;
        const int lo_last = first_key(t.pos0 + t.rows - 1);   // of the tile's last row
        const float* bias = !p.a.bias ? nullptr : bias_row(d) ? sBias : p.a.bias + size_t(h) * d.bias_n;
        const float bias2 = bias == sBias ? 1.f : 1.4426950408889634f;
        const float own2 = d.softcap > 0.f ? d.softcap * 1.4426950408889634f : p.scale2, scale2 = bias ? 1.f : own2, cap2 = d.softcap > 0.f ? 2.f * p.scale2 / d.softcap : 0.f;
        const uint32_t lane_addr = tmem + (uint32_t(quad * 32) << 16);
        const uint32_t masked = scale2 < 0.f ? 0x7f800000u : 0xff800000u;   // -inf behind the scale
        float m_ref = BOUND ? d.bound * 1.4426950408889634f : -INFINITY, l_run = 0.f;
        bool ok = true;
        for (int j = 0; j < nblk; ++j) {
            const int t0 = key_tile(j) * BN + col0;
            if (ok && !mbar_wait(&s_full, j & 1, &s_err)) { atomicExch(&s_err, 1); ok = false; }
            fence_after();
            uint32_t sv[NC / 32][32];
#pragma unroll
            for (int c = 0; c < NC / 32; ++c) tmem_ld32(lane_addr + kColS + col0 + 32 * c, sv[c]);
            wait_ld();
            fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(&s_free);
            if (d.softcap > 0.f) {   // tanh(x) = 1 - 2 / (1 + exp(2 x)); own2 then holds the cap
#pragma unroll
                for (int c = 0; c < NC; ++c) sv[c >> 5][c & 31] = __float_as_uint(1.f - __fdividef(2.f, 1.f + ex2(fminf(__uint_as_float(sv[c >> 5][c & 31]) * cap2, 120.f))));
            }
            if (bias) {   // scores and biases in the logarithm's base: scale2 is one
#pragma unroll
                for (int c = 0; c < NC; ++c)
                    sv[c >> 5][c & 31] = __float_as_uint(fmaf(__uint_as_float(sv[c >> 5][c & 31]), own2, bias[max(0, min(pq - t0 - c, d.bias_n - 1))] * bias2));
            }
            if (d.pool > 0 && j < head) {
                const int seen = lo / d.pool;
#pragma unroll
                for (int c = 0; c < NC; ++c) if (t0 + c >= seen) sv[c >> 5][c & 31] = masked;
            } else if (t0 + NC - 1 > t.pos0 || (t0 < lo_last && t0 + NC > keep)) {
#pragma unroll
                for (int c = 0; c < NC; ++c)
                    if (t0 + c > pq || (t0 + c < lo && t0 + c >= keep)) sv[c >> 5][c & 31] = masked;
            }
            float alpha = 1.f;
            if constexpr (!BOUND) {
                float mx4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
                for (int c = 0; c < NC; ++c) mx4[c & 3] = fmaxf(mx4[c & 3], __uint_as_float(sv[c >> 5][c & 31]) * scale2);   // the scale may have either sign
                const float mx = fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3]));
                if (m_ref == -INFINITY) m_ref = mx;
                else if (mx > m_ref + kLazy) { alpha = ex2(m_ref - mx); m_ref = mx; }
            }
            const float m_use = m_ref == -INFINITY ? 0.f : m_ref;
            float sum4[4] = {0.f, 0.f, 0.f, 0.f};
            uint32_t ph[NC / 2];
#pragma unroll
            for (int c = 0; c < NC; c += 2) {
                const float p0 = ex2(fmaf(__uint_as_float(sv[c >> 5][c & 31]), scale2, -m_use));
                const float p1 = ex2(fmaf(__uint_as_float(sv[c >> 5][(c & 31) + 1]), scale2, -m_use));
                sum4[(c >> 1) & 3] += p0 + p1;
                ph[c >> 1] = pack_bf2(p0, p1);
            }
            l_run = l_run * alpha + ((sum4[0] + sum4[1]) + (sum4[2] + sum4[3]));
            if (j >= 2 && ok && !mbar_wait(&pv_done[j & 1], ((j >> 1) - 1) & 1, &s_err)) { atomicExch(&s_err, 1); ok = false; }
            if (!BOUND && j > 0 && __any_sync(0xffffffffu, alpha != 1.f)) {
                if (ok && !mbar_wait(&pv_done[(j - 1) & 1], ((j - 1) >> 1) & 1, &s_err)) { atomicExch(&s_err, 1); ok = false; }
                fence_after();
                for (int c0 = 0; c0 < vch * 64; c0 += 32) {
                    uint32_t o[32];
                    tmem_ld32(lane_addr + kColO + c0, o);
                    wait_ld();
#pragma unroll
                    for (int i = 0; i < 32; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * alpha);
                    tmem_st32(lane_addr + kColO + c0, o);
                }
            }
            fence_after();
            if constexpr (BOUND) tmem_st16(lane_addr + kColP + uint32_t((j & 1) * 32 + half * 16), ph);
            else tmem_st32(lane_addr + kColP + uint32_t((j & 1) * 32), ph);
            wait_st();
            fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(&p_full[j & 1]);
        }
        if (ok && !mbar_wait(&pv_done[(nblk - 1) & 1], ((nblk - 1) >> 1) & 1, &s_err)) { atomicExch(&s_err, 1); ok = false; }
        fence_after();
        if constexpr (BOUND) {   // both halves of a row
            s_sum[half][r] = l_run;
            asm volatile("bar.sync 1, %0;" ::"n"(32 * WARPS) : "memory");
            l_run += s_sum[half ^ 1][r];
        }
        const bool per_value = p.a.gate != nullptr;
        if (p.a.sink) {
            const float own = p.a.sink[h] * 1.4426950408889634f;
            l_run += m_ref == -INFINITY ? 1.f : ex2(own - m_ref);
        }
        const float head_gate = per_value || r >= t.rows || !p.a.head_gate ? 1.f : p.a.head_gate[size_t(t.row0 + r) * d.heads + h];
        const float inv = l_run > 0.f ? head_gate / l_run : 0.f;
        const __nv_bfloat16* gate = static_cast<const __nv_bfloat16*>(p.a.gate) + size_t(t.row0 + r) * p.a.gate_ld + h * d.vdim;
        const int width = d.joint ? vch * 64 : d.vdim;
        __nv_bfloat16* out = static_cast<__nv_bfloat16*>(p.a.out) + size_t(t.row0 + r) * p.a.out_ld + (d.joint ? h * value_pieces(d) * 64 + vp0 * 64 : h * d.vdim);
        const bool vec = !(width & 7) && !(p.a.gate_ld & 7) && !(p.a.out_ld & 7);   // 16-byte pieces stay aligned
        for (int c0 = half * 32; c0 < width; c0 += 32 * (WARPS / 4)) {
            uint32_t o[32];
            tmem_ld32(lane_addr + kColO + c0, o);
            wait_ld();
            if (r < t.rows && ok) {
                const int nc = min(32, width - c0);
                if (vec) {
#pragma unroll
                    for (int i = 0; i < 32; i += 8)
                        if (i < nc) {
                            const uint4 g4 = per_value ? *reinterpret_cast<const uint4*>(gate + c0 + i) : make_uint4(0x3f803f80u, 0x3f803f80u, 0x3f803f80u, 0x3f803f80u);   // ones
                            const __nv_bfloat162* g2 = reinterpret_cast<const __nv_bfloat162*>(&g4);
                            uint32_t w[4];
#pragma unroll
                            for (int e = 0; e < 4; ++e) {
                                const float2 g = __bfloat1622float2(g2[e]);
                                w[e] = pack_bf2(__uint_as_float(o[i + 2 * e]) * inv * g.x, __uint_as_float(o[i + 2 * e + 1]) * inv * g.y);
                            }
                            *reinterpret_cast<uint4*>(out + c0 + i) = make_uint4(w[0], w[1], w[2], w[3]);
                        }
                } else {
#pragma unroll
                    for (int i = 0; i < 32; ++i)
                        if (i < nc) out[c0 + i] = __float2bfloat16_rn(__uint_as_float(o[i]) * inv * (per_value ? __bfloat162float(gate[c0 + i]) : 1.f));
                }
            }
        }
        fence_before();
    }
    __syncthreads();
    if (warp == 1) {
        fence_after();
        tmem_free<COLS>(tmem);
    }
    if (tid == 0 && s_err && p.a.err) atomicExch(p.a.err, 1);
}

int pieces_of(const PromptDims& d) { return std::min(4, value_pieces(d)); }
size_t smem_bytes(const PromptDims& d, int stages) {
    const int qch = (d.dim_p + d.rot_p) / 64, vch = pieces_of(d);
    return size_t(qch) * BM * 128 + size_t(stages) * (qch + vch) * BN * 128 + size_t(bias_row(d)) * 4 + 1024;
}

}  // namespace

bool attn_prefill_kv_supported(const PromptDims& d) { return (d.joint || d.vdim_p <= 256) && smem_bytes(d, 2) <= 220 * 1024; }

int32_t attn_prefill_kv(const PromptDims& d, const PromptAttnArgs& a, cudaStream_t st) {
    if (a.n_tiles <= 0) return FORGE_OK;
    if (!attn_prefill_kv_supported(d)) { set_error("prompt attention: head sizes %d + %d / %d unsupported", d.dim, d.rot, d.vdim); return FORGE_ERR_SHAPE; }
    CUtensorMap mq, mk, mr, mv, bk, bv;
    const uint64_t qd = uint64_t(d.dim_p + d.rot_p), H = uint64_t(d.heads), G = H / d.share;
    const uint64_t k_row = a.pages ? uint64_t(a.page_row) * 2 : G * d.dim_p * 2, v_row = a.pages ? k_row : G * d.vdim_p * 2;
    FORGE_TRY(make_map_3d(&mq, a.q, qd, H, uint64_t(a.q_rows), qd * 2, H * qd * 2, BM));
    FORGE_TRY(make_map_3d(&mk, a.k, uint64_t(d.dim_p), G, uint64_t(a.ctx_rows), uint64_t(d.dim_p) * 2, k_row, BN));
    if (d.rot_p == 0) mr = mk;   // no rotated part: never read
    else FORGE_TRY(make_map_2d(&mr, a.krot, uint64_t(d.rot_p), uint64_t(a.ctx_rows), uint64_t(d.rot_p) * 2, BN));
    FORGE_TRY(make_map_3d(&mv, a.v, uint64_t(d.vdim_p), G, uint64_t(a.ctx_rows), uint64_t(d.vdim_p) * 2, v_row, BN));
    if (d.pool > 0 && a.block_rows > 0) {
        FORGE_TRY(make_map_3d(&bk, a.blocks, uint64_t(d.dim_p), G, uint64_t(a.block_rows), uint64_t(d.dim_p) * 2, k_row, BN));
        FORGE_TRY(make_map_3d(&bv, static_cast<const __nv_bfloat16*>(a.blocks) + G * d.dim_p, uint64_t(d.vdim_p), G, uint64_t(a.block_rows), uint64_t(d.vdim_p) * 2, v_row, BN));
    } else { bk = mk; bv = mv; }
    // three stages, or two where that lets two CTAs share an SM: if the work of an SM, not the longest tile, decides
    auto fit = [&](int stages, size_t ctas) { return ctas * (smem_bytes(d, stages) + 2048) <= 226 * 1024; };
    long long total = 0, longest = 0;
    for (int i = 0; i < a.n_tiles && a.host_tiles; ++i) {
        const PromptTile& t = a.host_tiles[i];
        const int jb = first_visible(d, t.pos0) / BN;
        const long long n = head_tiles(d, t, jb) + (t.pos0 + t.rows - 1) / BN + 1 - jb;
        total += n * d.heads;
        longest = std::max(longest, n);
    }
    const int pieces = pieces_of(d), parts = (value_pieces(d) + pieces - 1) / pieces;
    const bool share = longest * 148 < total * parts && pieces <= 2;
    Params p{d, a, d.scale * 1.4426950408889634f, fit(3, share ? 2 : 1) ? 3 : fit(2, share ? 2 : 1) ? 2 : fit(3, 1) ? 3 : 2, pieces};
    const size_t smem = smem_bytes(d, p.stages);
    const bool bound = d.bound > 0.f && d.bound <= kMostBound;
    auto go = [&](auto kern) -> int32_t {
        FORGE_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, int(smem)));
        kern<<<dim3(d.heads * parts, a.n_tiles), bound ? 320 : 192, smem, st>>>(mq, mk, mr, mv, bk, bv, p);
        FORGE_LAUNCH_CHECK();
        return FORGE_OK;
    };
    if (bound) return pieces <= 2 ? go(attn_prefill_kv_kernel<256, true>) : go(attn_prefill_kv_kernel<512, true>);
    return pieces <= 2 ? go(attn_prefill_kv_kernel<256, false>) : go(attn_prefill_kv_kernel<512, false>);
}

}  // namespace forge
