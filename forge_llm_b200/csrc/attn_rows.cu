// Attention of single rows (decode, short portions, float32 prompts) over a paged cache.
//
// One CTA = some query heads of one key / value head, one row, one of up to eight ranges of its keys; the CTAs of a row form a
// cluster and merge their sums through distributed shared memory.
//   float32 (and value heads beyond 256)  up to four heads; a warp takes 32 keys at a time: eight keys by four lanes for the scores, then
//                                         a lane per pair of value columns for the sums.  Everything behind the loads is f32.
//   bfloat16                              up to sixteen heads are the rows of a tensor-core tile; a warp takes sixteen keys at a time, whose
//                                         keys and values it copies into its own two buffers in shared memory.  The tiles of earlier
//                                         steps' keys are requested before the dependency wait.  Probabilities enter their product as bf16 pairs.
#include <cooperative_groups.h>

#include <algorithm>

#include "attn_rows.cuh"
#include "mma.cuh"

namespace forge {

namespace {

namespace cg = cooperative_groups;

constexpr int kWarps = 8, kThreads = kWarps * 32;
constexpr float kLog2e = 1.4426950408889634f;

__device__ __forceinline__ float2 load_pair(const float* p) { return *reinterpret_cast<const float2*>(p); }
__device__ __forceinline__ float2 load_pair(const __nv_bfloat16* p) { return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p)); }

// The warps' maxima and sums (sml [warp][hs][2]) and unnormalised outputs (so, `stride` values per warp, [head][vdim_p]) of a CTA become one, then those of
// the cluster's CTAs: nh heads from h0, hs the stride of sml in heads, cml [nh][2].
template <typename T>
__device__ __forceinline__ void merge_rows(const AttnDims& d, float* so, int stride, float* sml, float* cml, int hs, int nh, int h0, int r, const float* gate, const float* sink, T* out, int out_ld) {
    const int split = blockIdx.x, splits = gridDim.x;
    __syncthreads();
    if (int(threadIdx.x) < nh) {   // maximum and sum of the CTA
        const int h = threadIdx.x;
        float mt = -INFINITY, lt = 0.f;
        for (int w = 0; w < kWarps; ++w) mt = fmaxf(mt, sml[(w * hs + h) * 2]);
        for (int w = 0; w < kWarps; ++w) {
            const float f = mt == -INFINITY ? 0.f : exp2f(sml[(w * hs + h) * 2] - mt);
            lt += sml[(w * hs + h) * 2 + 1] * f;
            sml[(w * hs + h) * 2] = f;     // the warp's factor
        }
        cml[2 * h] = mt; cml[2 * h + 1] = lt;
    }
    __syncthreads();
    for (int i = threadIdx.x; i < nh * d.vdim_p; i += kThreads) {   // own element of every warp: read, then written over warp 0's
        const int h = i / d.vdim_p;
        float v = 0.f;
#pragma unroll
        for (int w = 0; w < kWarps; ++w) v += so[w * stride + i] * sml[(w * hs + h) * 2];
        so[i] = v;
    }
    cg::cluster_group cl = cg::this_cluster();
    if (splits > 1) cl.sync();
    else __syncthreads();
    const int items = nh * d.vdim, share = (items + splits - 1) / splits;
    for (int i = split * share + threadIdx.x; i < min(items, (split + 1) * share); i += kThreads) {
        const int h = i / d.vdim, c = i % d.vdim;
        const float own = sink ? sink[h0 + h] * kLog2e : -INFINITY;
        float mt = own, lt = 0.f, v = 0.f;
        for (int s = 0; s < splits; ++s) mt = fmaxf(mt, splits > 1 ? cl.map_shared_rank(cml, s)[2 * h] : cml[2 * h]);
        for (int s = 0; s < splits; ++s) {
            const float* o = splits > 1 ? cl.map_shared_rank(cml, s) : cml;
            const float* x = splits > 1 ? cl.map_shared_rank(so, s) : so;
            const float f = o[2 * h] == -INFINITY ? 0.f : exp2f(o[2 * h] - mt);
            lt = fmaf(o[2 * h + 1], f, lt);
            v = fmaf(x[h * d.vdim_p + c], f, v);
        }
        if (sink) lt += exp2f(own - mt);
        v /= lt;
        if (gate) v *= gate[size_t(r) * d.heads + h0 + h];
        out[size_t(r) * out_ld + (h0 + h) * d.vdim + c] = to_t<T>(v);
    }
    if (splits > 1) cl.sync();   // nobody leaves while its shared memory is read
}

// (What a kernel in front writes is not __restrict__: loads of it may not be moved above the dependency wait.)
// GQ: query heads per CTA; VP: pairs of value columns per lane
template <typename T, int GQ, int VP>
__global__ void __launch_bounds__(kThreads) attn_rows_kernel(const AttnDims d, const T* q, const T* cache, const float* gate, const float* __restrict__ sink,
                                                             const float* __restrict__ bias, T* __restrict__ out, int out_ld, const StepRows rows) {
    extern __shared__ float sm[];
    const int gq = d.heads / d.groups, blocks = (gq + GQ - 1) / GQ;
    const int split = blockIdx.x, splits = gridDim.x, g = blockIdx.y / blocks, h0 = g * gq + (blockIdx.y % blocks) * GQ, nh = min(GQ, (g + 1) * gq - h0), r = blockIdx.z;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    float* sq = sm;                                    // [GQ][dim_p]
    float* sp = sq + GQ * d.dim_p + warp * GQ * 32;    // [warp][GQ][32]
    float* so = sq + GQ * d.dim_p + kWarps * GQ * 32;  // [warp][GQ][vdim_p]; in the end [GQ][vdim_p] of the CTA
    float* sml = so + kWarps * GQ * d.vdim_p;          // [warp][GQ][2], then [GQ][2] of the CTA
    float* cml = sml + kWarps * GQ * 2;
    pdl_trigger();
    // positions and page tables are written in front of the step's first kernel, which is launched without overlap
    const int pos = rows.pos[r], seq = rows.seq ? rows.seq[r] : r;
    const int lo = d.first_key(pos), front = d.front(pos), n = front + pos - lo + 1;
    const int per = ((n + splits - 1) / splits + 31) & ~31;
    const int k_begin = split * per, k_end = min(n, k_begin + per);
    const int32_t* pt = rows.page_table + size_t(seq) * rows.pages_per_seq;
    const size_t W = d.row();
    pdl_wait();
    for (int i = threadIdx.x; i < GQ * d.dim_p; i += kThreads) {
        const int h = i / d.dim_p, c = i % d.dim_p;
        sq[i] = h < nh && c < d.dim ? to_f(q[(size_t(r) * d.heads + h0 + h) * d.dim_p + c]) : 0.f;
    }
    __syncthreads();
    float m[GQ], l[GQ], acc[GQ][2 * VP];
#pragma unroll
    for (int h = 0; h < GQ; ++h) {
        m[h] = -INFINITY; l[h] = 0.f;
#pragma unroll
        for (int c = 0; c < 2 * VP; ++c) acc[h][c] = 0.f;
    }
    const float inv_cap = d.softcap > 0.f ? 1.0f / d.softcap : 0.f;
    const T* kbase = cache + size_t(g) * d.dim_p;
    const T* vbase = cache + size_t(d.groups) * d.dim_p + size_t(g) * d.vdim_p;
    auto row_of = [&](int i) { return d.key_row(pt, i, front, lo); };
    for (int key0 = k_begin + warp * 32; key0 < k_end; key0 += kThreads) {
        const int nk = min(32, k_end - key0);
        const size_t my_row = row_of(key0 + min(lane, nk - 1));
        __syncwarp();
#pragma unroll
        for (int b = 0; b < 4; ++b) {   // eight keys by four lanes
            const int key = b * 8 + (lane >> 2), part = (lane & 3) * 8;
            const size_t row = __shfl_sync(0xffffffffu, my_row, key);
            const T* kr = kbase + row * W;
            float s[GQ];
#pragma unroll
            for (int h = 0; h < GQ; ++h) s[h] = 0.f;
#pragma unroll 4
            for (int c = part; c < d.dim_p; c += 32) {
                float kv[8];
                load8(kv, kr + c);
#pragma unroll
                for (int h = 0; h < GQ; ++h) {
                    float qv[8];
                    load8(qv, sq + h * d.dim_p + c);
#pragma unroll
                    for (int e = 0; e < 8; ++e) s[h] = fmaf(kv[e], qv[e], s[h]);
                }
            }
#pragma unroll
            for (int h = 0; h < GQ; ++h) {
                s[h] += __shfl_xor_sync(0xffffffffu, s[h], 1);
                s[h] += __shfl_xor_sync(0xffffffffu, s[h], 2);
                float v = s[h] * d.scale;
                if (d.softcap > 0.f) v = d.softcap * tanhf(v * inv_cap);
                if (bias && h < nh) {
                    const int i = min(key0 + key, n - 1), dist = pos - (i < front ? i : lo + i - front);
                    v += bias[size_t(h0 + h) * d.bias_n + min(dist, d.bias_n - 1)];
                }
                if ((lane & 3) == 0) sp[h * 32 + key] = key < nk ? v * kLog2e : -INFINITY;
            }
        }
        __syncwarp();
#pragma unroll
        for (int h = 0; h < GQ; ++h) {
            const float s = sp[h * 32 + lane];
            float mx = s;
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
            const float mn = fmaxf(m[h], mx), alpha = exp2f(m[h] - mn), p = exp2f(s - mn);   // a tile holds a visible key
            l[h] = l[h] * alpha + p;      // lanes are added at the end
            m[h] = mn;
#pragma unroll
            for (int c = 0; c < 2 * VP; ++c) acc[h][c] *= alpha;
            sp[h * 32 + lane] = p;
        }
        __syncwarp();
#pragma unroll 4
        for (int k = 0; k < nk; ++k) {
            const T* vr = vbase + __shfl_sync(0xffffffffu, my_row, k) * W;
            float2 v[VP];
#pragma unroll
            for (int c = 0; c < VP; ++c) v[c] = 2 * lane + 64 * c < d.vdim_p ? load_pair(vr + 2 * lane + 64 * c) : make_float2(0.f, 0.f);
#pragma unroll
            for (int h = 0; h < GQ; ++h) {
                const float p = sp[h * 32 + k];
#pragma unroll
                for (int c = 0; c < VP; ++c) { acc[h][2 * c] = fmaf(p, v[c].x, acc[h][2 * c]); acc[h][2 * c + 1] = fmaf(p, v[c].y, acc[h][2 * c + 1]); }
            }
        }
    }
#pragma unroll
    for (int h = 0; h < GQ; ++h) {
        const float ls = warp_sum(l[h]);
        if (lane == 0) { sml[(warp * GQ + h) * 2] = m[h]; sml[(warp * GQ + h) * 2 + 1] = ls; }
#pragma unroll
        for (int c = 0; c < VP; ++c)
            if (2 * lane + 64 * c < d.vdim_p) *reinterpret_cast<float2*>(so + (warp * GQ + h) * d.vdim_p + 2 * lane + 64 * c) = make_float2(acc[h][2 * c], acc[h][2 * c + 1]);
    }
    merge_rows(d, so, GQ * d.vdim_p, sml, cml, GQ, nh, h0, r, gate, sink, out, out_ld);
}

size_t smem_bytes(const AttnDims& d, int gq) { return sizeof(float) * (size_t(gq) * d.dim_p + kWarps * gq * 32 + size_t(kWarps) * gq * d.vdim_p + kWarps * gq * 2 + gq * 2); }

template <typename T, int GQ, int VP>
int32_t launch(const AttnDims& d, const void* q, const void* cache, const float* gate, const float* sink, const float* bias, void* out, int out_ld, const StepRows& rows, int splits, cudaStream_t st) {
    auto kern = attn_rows_kernel<T, GQ, VP>;
    const size_t smem = smem_bytes(d, GQ);
    if (smem > 48 * 1024) FORGE_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, int(smem)));
    const int gq = d.heads / d.groups, blocks = (gq + GQ - 1) / GQ;
    FORGE_CUDA(launch_pdl_cluster(kern, dim3(splits, d.groups * blocks, rows.n), dim3(kThreads), splits, smem, st, d, static_cast<const T*>(q), static_cast<const T*>(cache), gate, sink, bias, static_cast<T*>(out), out_ld, rows));
    FORGE_LAUNCH_CHECK();
    return FORGE_OK;
}

template <typename T>
int32_t run(const AttnDims& d, const void* q, const void* cache, const float* gate, const float* sink, const float* bias, void* out, int out_ld, const StepRows& rows, int splits, cudaStream_t st) {
    const int gq = d.heads / d.groups, vp = d.vdim_p / 64;
    auto with_vp = [&](auto gqc) -> int32_t {
        constexpr int GQ = decltype(gqc)::value;
        if (vp <= 1) return launch<T, GQ, 1>(d, q, cache, gate, sink, bias, out, out_ld, rows, splits, st);
        if (vp <= 2) return launch<T, GQ, 2>(d, q, cache, gate, sink, bias, out, out_ld, rows, splits, st);
        return launch<T, GQ, 8>(d, q, cache, gate, sink, bias, out, out_ld, rows, splits, st);
    };
    if (gq == 1) return with_vp(std::integral_constant<int, 1>{});
    if (gq == 2) return with_vp(std::integral_constant<int, 2>{});
    return with_vp(std::integral_constant<int, 4>{});
}

// ------------------------------------------------------------------------------------------------ bfloat16
using bf16 = __nv_bfloat16;
constexpr int kTileKeys = 16, kRowHeads = 16;
struct TileBytes {   // of shared memory, in elements
    int ldk, ldv, stage;
    __host__ __device__ explicit TileBytes(const AttnDims& d) : ldk(d.dim_p + 8), ldv(d.vdim_p + 8), stage(kTileKeys * (d.dim_p + 8 + d.vdim_p + 8)) {}
};
size_t mma_smem(const AttnDims& d) { return (size_t(kWarps) * 2 * TileBytes(d).stage + kRowHeads * TileBytes(d).ldk) * 2 + (kWarps * kRowHeads * 2 + kRowHeads * 2) * 4; }

// VC: blocks of 64 value columns at most; KP, VP: 16-byte pieces of a row's key and values (0: any number)
template <int VC, int KP, int VP>
__global__ void __launch_bounds__(kThreads, 1) attn_rows_mma_kernel(const AttnDims d, const bf16* q, const bf16* cache, const float* gate, const float* __restrict__ sink, const float* __restrict__ bias,
                                                                    bf16* out, int out_ld, const StepRows rows) {
    extern __shared__ __align__(16) unsigned char sm_raw[];
    const TileBytes L(d);
    bf16* tiles = reinterpret_cast<bf16*>(sm_raw);              // [warp][2]: keys, values
    bf16* sq = tiles + size_t(kWarps) * 2 * L.stage;            // [16][ldk]
    float* sml = reinterpret_cast<float*>(sq + kRowHeads * L.ldk);
    float* cml = sml + kWarps * kRowHeads * 2;
    const int gq = d.heads / d.groups, blocks = (gq + kRowHeads - 1) / kRowHeads;
    const int split = blockIdx.x, splits = gridDim.x, g = blockIdx.y / blocks, h0 = g * gq + (blockIdx.y % blocks) * kRowHeads, nh = min(kRowHeads, (g + 1) * gq - h0), r = blockIdx.z;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, lr = lane >> 2, lc = (lane & 3) * 2;
    pdl_trigger();
    // positions and page tables are written in front of the step's first kernel, which is launched without overlap
    const int pos = rows.pos[r], seq = rows.seq ? rows.seq[r] : r;
    const int lo = d.first_key(pos), front = d.front(pos), n = front + pos - lo + 1;
    const int per = ((n + splits - 1) / splits + kTileKeys - 1) & ~(kTileKeys - 1);
    const int k_begin = split * per, k_end = min(n, k_begin + per);
    const int32_t* pt = rows.page_table + size_t(seq) * rows.pages_per_seq;
    const size_t W = d.row();
    const bf16* kbase = cache + size_t(g) * d.dim_p;
    const bf16* vbase = cache + size_t(d.groups) * d.dim_p + size_t(g) * d.vdim_p;
    bf16* mine = tiles + size_t(warp) * 2 * L.stage;
    const int kp = KP ? KP : d.dim_p / 8, vp = VP ? VP : d.vdim_p / 8;
    auto fetch = [&](int i) {   // the warp's i-th tile
        const int key0 = k_begin + (warp + kWarps * i) * kTileKeys;
        if (key0 < k_end) {
            const uint32_t row = uint32_t(d.key_row(pt, key0 + min(lane & (kTileKeys - 1), k_end - key0 - 1), front, lo));
            const uint32_t sk = uint32_t(__cvta_generic_to_shared(mine + (i & 1) * L.stage)), sv = sk + kTileKeys * L.ldk * 2;
            auto copy = [&](uint32_t dst, int ld, const bf16* src, int pieces) {
#pragma unroll
                for (int p = lane; p < kTileKeys * pieces; p += 32) {
                    const int k = p / pieces, c = (p % pieces) * 8;
                    cp_async16(dst + (k * ld + c) * 2, src + __shfl_sync(0xffffffffu, row, k) * W + c, true);
                }
            };
            copy(sk, L.ldk, kbase, kp);
            copy(sv, L.ldv, vbase, vp);
        }
        cp_commit();
    };
    // a tile all of whose keys earlier steps have written (a block that this step completes is seen by rows a window behind it)
    const int written = d.pool > 0 && rows.fresh > d.window ? 0 : n - rows.fresh;
    auto old = [&](int i) { return min(k_end, k_begin + (warp + kWarps * i + 1) * kTileKeys) <= written; };
    int ahead = 0;
    while (ahead < 2 && old(ahead)) fetch(ahead++);
    pdl_wait();
    while (ahead < 2) fetch(ahead++);
    for (int i = threadIdx.x; i < kRowHeads * kp; i += kThreads) {
        const int h = i / kp, c = (i % kp) * 8;
        uint4 v = make_uint4(0, 0, 0, 0);
        if (h < nh) v = *reinterpret_cast<const uint4*>(q + (size_t(r) * d.heads + h0 + h) * d.dim_p + c);
        *reinterpret_cast<uint4*>(sq + h * L.ldk + c) = v;
    }
    __syncthreads();
    const SmemMat mq{uint32_t(__cvta_generic_to_shared(sq)), L.ldk};
    const int ksteps = (d.dim + 15) / 16, vsteps = (d.vdim + 15) / 16;
    const float scale2 = d.scale * kLog2e, inv_cap = d.softcap > 0.f ? d.scale / d.softcap : 0.f;
    float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f}, o[VC * 4][2][4];
#pragma unroll
    for (int v = 0; v < VC * 4; ++v)
#pragma unroll
        for (int e = 0; e < 8; ++e) o[v][e >> 2][e & 3] = 0.f;
    for (int i = 0;; ++i) {
        const int key0 = k_begin + (warp + kWarps * i) * kTileKeys;
        if (key0 >= k_end) break;
        float far[2][4];   // biases
        if (bias)
#pragma unroll
            for (int j = 0; j < 2; ++j)
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const int idx = min(key0 + j * 8 + lc + (e & 1), k_end - 1), dist = pos - (idx < front ? idx : lo + idx - front);
                    far[j][e] = bias[size_t(h0 + min(lr + (e >> 1) * 8, nh - 1)) * d.bias_n + min(dist, d.bias_n - 1)];
                }
        cp_wait<1>();
        __syncwarp();
        const uint32_t at = uint32_t(__cvta_generic_to_shared(mine + (i & 1) * L.stage));
        const SmemMat mk{at, L.ldk}, mv{at + uint32_t(kTileKeys * L.ldk) * 2, L.ldv};
        float s[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
#pragma unroll 4
        for (int k = 0; k < ksteps; ++k) {
            uint32_t fa[4], fb[4];
            mq.a(fa, 0, k * 16, lane);
            mk.b(fb, 0, k * 16, lane);
            mma(s[0], fa, fb[0], fb[1]);
            mma(s[1], fa, fb[2], fb[3]);
        }
        float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                float v = d.softcap > 0.f ? d.softcap * kLog2e * tanhf(s[j][e] * inv_cap) : s[j][e] * scale2;
                if (bias) v = fmaf(far[j][e], kLog2e, v);
                if (key0 + j * 8 + lc + (e & 1) >= k_end) v = -INFINITY;
                s[j][e] = v;
                mx[e >> 1] = fmaxf(mx[e >> 1], v);
            }
        float alpha[2];
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            mx[e] = fmaxf(mx[e], __shfl_xor_sync(0xffffffffu, mx[e], 1));
            mx[e] = fmaxf(fmaxf(mx[e], __shfl_xor_sync(0xffffffffu, mx[e], 2)), m[e]);
            alpha[e] = exp2f(m[e] - mx[e]);
            m[e] = mx[e];
            l[e] *= alpha[e];
        }
        uint32_t ph[4], pl[4];
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const float p0 = exp2f(s[j][2 * e] - m[e]), p1 = exp2f(s[j][2 * e + 1] - m[e]);
                l[e] += p0 + p1;
                split_bf16x2(p0, p1, ph[2 * j + e], pl[2 * j + e]);
            }
#pragma unroll
        for (int v = 0; v < VC * 4; ++v) {
            if (v >= vsteps) break;
            uint32_t fb[4];
            mv.b_t(fb, 0, v * 16, lane);
#pragma unroll
            for (int j = 0; j < 2; ++j) {
#pragma unroll
                for (int e = 0; e < 4; ++e) o[v][j][e] *= alpha[e >> 1];
                mma(o[v][j], pl, fb[2 * j], fb[2 * j + 1]);
                mma(o[v][j], ph, fb[2 * j], fb[2 * j + 1]);
            }
        }
        __syncwarp();   // the buffer is read
        fetch(i + 2);
    }
    cp_wait<0>();
    __syncwarp();
    float* so = reinterpret_cast<float*>(mine);                 // [nh][vdim_p]: fits the warp's buffers
#pragma unroll
    for (int e = 0; e < 2; ++e) {
        l[e] += __shfl_xor_sync(0xffffffffu, l[e], 1);
        l[e] += __shfl_xor_sync(0xffffffffu, l[e], 2);
        const int h = lr + 8 * e;
        if (h >= nh) continue;
        if ((lane & 3) == 0) { sml[(warp * kRowHeads + h) * 2] = m[e]; sml[(warp * kRowHeads + h) * 2 + 1] = l[e]; }
#pragma unroll
        for (int v = 0; v < VC * 4; ++v)
            if (v < vsteps)
#pragma unroll
                for (int j = 0; j < 2; ++j) *reinterpret_cast<float2*>(so + h * d.vdim_p + v * 16 + j * 8 + lc) = make_float2(o[v][j][2 * e], o[v][j][2 * e + 1]);
    }
    merge_rows(d, reinterpret_cast<float*>(tiles), L.stage, sml, cml, kRowHeads, nh, h0, r, gate, sink, out, out_ld);
}

bool mma_supported(const AttnDims& d) { return d.vdim_p <= 256 && mma_smem(d) <= 220 * 1024; }

int32_t run_mma(const AttnDims& d, const void* q, const void* cache, const float* gate, const float* sink, const float* bias, void* out, int out_ld, const StepRows& rows, int max_keys, cudaStream_t st) {
    const int gq = d.heads / d.groups, blocks = (gq + kRowHeads - 1) / kRowHeads;
    const size_t smem = mma_smem(d);
    auto go = [&](auto kern) -> int32_t {
        FORGE_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, int(smem)));
        // the most splits whose clusters all run at once, none shorter than one round of its warps
        static int fits[9] = {0};   // one CTA per SM
        if (!fits[1])
            for (int c = 1; c <= 8; ++c) {
                cudaLaunchConfig_t cfg{};
                cudaLaunchAttribute at[1];
                cfg.gridDim = dim3(unsigned(c * 148)); cfg.blockDim = dim3(kThreads); cfg.dynamicSmemBytes = std::max(smem, size_t(120) * 1024);
                at[0].id = cudaLaunchAttributeClusterDimension;
                at[0].val.clusterDim.x = unsigned(c); at[0].val.clusterDim.y = 1; at[0].val.clusterDim.z = 1;
                cfg.attrs = at; cfg.numAttrs = 1;
                FORGE_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, int(std::max(smem, size_t(120) * 1024))));
                FORGE_CUDA(cudaOccupancyMaxActiveClusters(&fits[c], kern, &cfg));
            }
        int splits = 1;
        for (int c = 2; c <= 8; ++c)
            if ((long long)rows.n * d.groups * blocks <= fits[c] && max_keys > (c - 1) * kWarps * kTileKeys) splits = c;
        FORGE_CUDA(launch_pdl_cluster(kern, dim3(splits, d.groups * blocks, rows.n), dim3(kThreads), splits, smem, st, d, static_cast<const bf16*>(q), static_cast<const bf16*>(cache), gate, sink, bias,
                                      static_cast<bf16*>(out), out_ld, rows));
        FORGE_LAUNCH_CHECK();
        return FORGE_OK;
    };
    if (d.dim_p == 64 && d.vdim_p == 64) return go(attn_rows_mma_kernel<1, 8, 8>);
    if (d.dim_p == 128 && d.vdim_p == 128) return go(attn_rows_mma_kernel<2, 16, 16>);
    return d.vdim_p <= 64 ? go(attn_rows_mma_kernel<1, 0, 0>) : d.vdim_p <= 128 ? go(attn_rows_mma_kernel<2, 0, 0>) : go(attn_rows_mma_kernel<4, 0, 0>);
}

// ------------------------------------------------------------------------------------------------ queries and keys
// One CTA = eight heads (queries first, then keys) of one row, a warp per head.
constexpr int kQkDims = 16;   // values per lane at most
template <typename T>
__global__ void __launch_bounds__(256) qk_post_kernel(const AttnDims d, const QkPost p, const float* proj, int ldp, int k_col, const float* __restrict__ q_norm,
                                                      const float* __restrict__ k_norm, const float2* __restrict__ rope, T* q, T* cache, const int32_t* place, const StepRows rows, const RouteBeside route, const ConvBeside conv) {
    extern __shared__ float sm[];
    __shared__ float red[2][8];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, r = blockIdx.y, h = blockIdx.x * 8 + warp;
    if (conv.blocks && int(blockIdx.x) >= int(gridDim.x) - conv.blocks) {
        conv_one<T>(conv.d, conv.a, rows, r, (int(blockIdx.x) - int(gridDim.x) + conv.blocks) * 256 + int(threadIdx.x));
        return;
    }
    if (route.logits && blockIdx.x == gridDim.x - 1) {
        if (r > 0) return;
        pdl_trigger();
        route_few_clear(route.d, sm);
        pdl_wait();
        route_few_rows(route.d, route.logits, rows.n, route.t, sm);
        return;
    }
    const bool on = h < d.heads + d.groups, is_q = h < d.heads;
    const int g = is_q ? h : h - d.heads, half = p.rot_dims / 2;
    const float* w = is_q ? q_norm : k_norm;
    if (p.norm == QkPost::WHOLE) w += size_t(g) * d.dim;
    pdl_trigger();
    const float2* turn = rope + size_t(rows.pos[r]) * half;
    float nw[kQkDims], v[kQkDims];
#pragma unroll
    for (int i = 0; i < kQkDims; ++i) nw[i] = on && lane + 32 * i < d.dim ? w[lane + 32 * i] : 0.f;
    pdl_wait();
    const float* row = proj + size_t(r) * ldp;
    const float* src = is_q ? row + size_t(g) * d.dim : row + k_col + size_t(g) * d.dim;
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < kQkDims; ++i) {
        v[i] = on && lane + 32 * i < d.dim ? src[lane + 32 * i] : 0.f;
        ss = fmaf(v[i], v[i], ss);
    }
    ss = warp_sum(ss);
    float n = float(d.dim);
    if (p.norm == QkPost::WHOLE) {   // this CTA sums up the rows that its heads belong to
        const int last = min(d.heads + d.groups, int(blockIdx.x) * 8 + 8) - 1;
        const int nq = int(blockIdx.x) * 8 < d.heads ? d.heads * d.dim : 0, nk = last >= d.heads ? d.groups * d.dim : 0;
        float sq = 0.f, sk = 0.f;
        for (int i = threadIdx.x; i < nq; i += 256) sq = fmaf(row[i], row[i], sq);
        for (int i = threadIdx.x; i < nk; i += 256) sk = fmaf(row[k_col + i], row[k_col + i], sk);
        sq = warp_sum(sq); sk = warp_sum(sk);
        if (lane == 0) { red[0][warp] = sq; red[1][warp] = sk; }
        __syncthreads();
        ss = 0.f;
        for (int i = 0; i < 8; ++i) ss += red[is_q ? 0 : 1][i];
        n = float(is_q ? d.heads : d.groups) * d.dim;
    }
    const float inv = 1.0f / sqrtf(ss / n + p.eps);
    float* s = sm + warp * d.dim_p;
#pragma unroll
    for (int i = 0; i < kQkDims; ++i) if (lane + 32 * i < d.dim) s[lane + 32 * i] = v[i] * inv * nw[i];
    __syncwarp();
    if (!on) return;
    T* dst = is_q ? q + (size_t(r) * d.heads + g) * d.dim_p : cache + size_t(place[r]) * d.row() + size_t(g) * d.dim_p;
    for (int i = lane; i < d.dim; i += 32) {
        float x = s[i];
        if (i < 2 * half) {
            const bool second = p.interleaved ? i & 1 : i >= half;
            const int pair = p.interleaved ? i >> 1 : second ? i - half : i;
            const float y = s[p.interleaved ? i ^ 1 : second ? i - half : i + half];
            const float2 t = turn[pair];
            x = second ? fmaf(x, t.x, y * t.y) : fmaf(x, t.x, -y * t.y);
        }
        dst[i] = to_t<T>(x);
    }
}

// The same for sizes in whole pieces of four values: a lane holds up to four pieces of its head, its rotation partners come through shared
// memory for halves and lie in the same piece for interleaved pairs.
__device__ __forceinline__ void store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void store4(__nv_bfloat16* p, float4 v) {
    const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
}
__device__ __forceinline__ float sum4(float4 v) { return fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, v.w * v.w))); }
template <typename T, int P, int R>   // R: rows per CTA, whose loads are in flight together
__global__ void __launch_bounds__(256) qk_post4_kernel(const AttnDims d, const QkPost p, const float* proj, int ldp, int k_col, const float* __restrict__ q_norm,
                                                       const float* __restrict__ k_norm, const float2* __restrict__ rope, T* q, T* cache, const int32_t* place, const StepRows rows, const RouteBeside route, const ConvBeside conv) {
    extern __shared__ __align__(16) float sm[];
    __shared__ float red[R][2][8];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, r0 = blockIdx.y * R, h = blockIdx.x * 8 + warp;
    if (conv.blocks && int(blockIdx.x) >= int(gridDim.x) - conv.blocks) {
        for (int r = r0; r < min(r0 + R, rows.n); ++r) conv_one<T>(conv.d, conv.a, rows, r, (int(blockIdx.x) - int(gridDim.x) + conv.blocks) * 256 + int(threadIdx.x));
        return;
    }
    if (route.logits && blockIdx.x == gridDim.x - 1) {
        if (r0 > 0) return;
        pdl_trigger();
        route_few_clear(route.d, sm);
        pdl_wait();
        route_few_rows(route.d, route.logits, rows.n, route.t, sm);
        return;
    }
    const bool on = h < d.heads + d.groups, is_q = h < d.heads;
    const int g = is_q ? h : h - d.heads, half = p.rot_dims / 2, pieces = d.dim / 4;
    const float* w = is_q ? q_norm : k_norm;
    if (p.norm == QkPost::WHOLE) w += size_t(g) * d.dim;
    pdl_trigger();
    float4 nw[P], v[R][P], t0[R][P], t1[R][P];
#pragma unroll
    for (int i = 0; i < P; ++i) {
        const int c = (lane + 32 * i) * 4;
        nw[i] = on && c < d.dim ? *reinterpret_cast<const float4*>(w + c) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
#pragma unroll
    for (int j = 0; j < R; ++j) {
        const float2* turn = rope + size_t(rows.pos[min(r0 + j, rows.n - 1)]) * half;
#pragma unroll
        for (int i = 0; i < P; ++i) {
            const int c = (lane + 32 * i) * 4;
            t0[j][i] = t1[j][i] = make_float4(1.f, 0.f, 1.f, 0.f);
            if (on && c < d.dim && c < 2 * half) {   // {cos, sin} of the piece's pairs
                const int pair = p.interleaved ? c / 2 : c < half ? c : c - half;
                t0[j][i] = *reinterpret_cast<const float4*>(turn + pair);
                if (!p.interleaved) t1[j][i] = *reinterpret_cast<const float4*>(turn + pair + 2);
            }
        }
    }
    pdl_wait();
    float ss[R];
    int to[R];
#pragma unroll
    for (int j = 0; j < R; ++j) {
        const int r = min(r0 + j, rows.n - 1);
        const float* row = proj + size_t(r) * ldp;
        const float* src = is_q ? row + size_t(g) * d.dim : row + k_col + size_t(g) * d.dim;
        to[j] = place[r];
        ss[j] = 0.f;
#pragma unroll
        for (int i = 0; i < P; ++i) v[j][i] = on && lane + 32 * i < pieces ? reinterpret_cast<const float4*>(src)[lane + 32 * i] : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    float n = float(d.dim);
    if (p.norm == QkPost::WHOLE) {   // this CTA sums up the rows that its heads belong to
        const int last = min(d.heads + d.groups, int(blockIdx.x) * 8 + 8) - 1;
        const int nq = int(blockIdx.x) * 8 < d.heads ? d.heads * pieces : 0, nk = last >= d.heads ? d.groups * pieces : 0;
#pragma unroll
        for (int j = 0; j < R; ++j) {
            const float* row = proj + size_t(min(r0 + j, rows.n - 1)) * ldp;
            float sq = 0.f, sk = 0.f;
#pragma unroll 4
            for (int i = threadIdx.x; i < nq; i += 256) sq += sum4(reinterpret_cast<const float4*>(row)[i]);
#pragma unroll 2
            for (int i = threadIdx.x; i < nk; i += 256) sk += sum4(reinterpret_cast<const float4*>(row + k_col)[i]);
            sq = warp_sum(sq); sk = warp_sum(sk);
            if (lane == 0) { red[j][0][warp] = sq; red[j][1][warp] = sk; }
        }
        __syncthreads();
#pragma unroll
        for (int j = 0; j < R; ++j)
            for (int i = 0; i < 8; ++i) ss[j] += red[j][is_q ? 0 : 1][i];
        n = float(is_q ? d.heads : d.groups) * d.dim;
    } else {
#pragma unroll
        for (int j = 0; j < R; ++j) {
#pragma unroll
            for (int i = 0; i < P; ++i) ss[j] += sum4(v[j][i]);
            ss[j] = warp_sum(ss[j]);
        }
    }
    float* s = sm + warp * d.dim_p;
#pragma unroll
    for (int j = 0; j < R; ++j) {
        const int r = r0 + j;
        const float inv = 1.0f / sqrtf(ss[j] / n + p.eps);
        __syncwarp();
#pragma unroll
        for (int i = 0; i < P; ++i) {
            float4& x = v[j][i];
            x = make_float4(x.x * inv * nw[i].x, x.y * inv * nw[i].y, x.z * inv * nw[i].z, x.w * inv * nw[i].w);
            if (!p.interleaved && (lane + 32 * i) * 4 < 2 * half) store4(s + (lane + 32 * i) * 4, x);
        }
        __syncwarp();
        if (!on || r >= rows.n) continue;
        T* dst = is_q ? q + (size_t(r) * d.heads + g) * d.dim_p : cache + size_t(to[j]) * d.row() + size_t(g) * d.dim_p;
#pragma unroll
        for (int i = 0; i < P; ++i) {
            const int c = (lane + 32 * i) * 4;
            if (c >= d.dim) continue;
            float4 x = v[j][i];
            const float4 a = t0[j][i], b = t1[j][i];
            if (c < 2 * half) {
                if (p.interleaved) {
                    x = make_float4(fmaf(x.x, a.x, -x.y * a.y), fmaf(x.y, a.x, x.x * a.y), fmaf(x.z, a.z, -x.w * a.w), fmaf(x.w, a.z, x.z * a.w));
                } else {
                    const float4 y = *reinterpret_cast<const float4*>(s + (c < half ? c + half : c - half));
                    const float sign = c < half ? -1.f : 1.f;
                    x = make_float4(fmaf(x.x, a.x, sign * y.x * a.y), fmaf(x.y, a.z, sign * y.y * a.w), fmaf(x.z, b.x, sign * y.z * b.y), fmaf(x.w, b.z, sign * y.w * b.w));
                }
            }
            store4(dst + c, x);
        }
    }
}

}  // namespace

int32_t qk_post(const AttnDims& d, const QkPost& p, int dtype, const float* proj, int ldp, int k_col, const float* q_norm, const float* k_norm, const float* rope, void* q, void* cache,
                const int32_t* place, const StepRows& rows, const RouteBeside* route, const ConvBeside* conv, cudaStream_t st) {
    if (rows.n <= 0) return FORGE_OK;
    if (route && (rows.n > kScaleRows || route->d.choices() > kMaxExperts)) { set_error("routing: %d rows, %d experts", rows.n, route->d.experts); return FORGE_ERR_SHAPE; }
    if ((route && conv) || (conv && rows.n > 65535)) { set_error("queries and keys: nothing more fits beside them"); return FORGE_ERR_SHAPE; }
    if (d.dim > kQkDims * 32 || p.rot_dims > d.dim || p.rot_dims % 2) { set_error("attention: head size %d with %d rotated dimensions", d.dim, p.rot_dims); return FORGE_ERR_SHAPE; }
    auto go = [&](auto t) -> int32_t {
        using T = decltype(t);
        const RouteBeside beside = route ? *route : RouteBeside{};
        ConvBeside scan = conv ? *conv : ConvBeside{};
        if (conv) scan.blocks = (conv->d.inner + 255) / 256;
        for (int r0 = 0; r0 < rows.n; r0 += 65535) {
            StepRows part = rows;
            part.n = std::min(65535, rows.n - r0);
            part.pos += r0;
            const bool four = d.dim % 4 == 0 && ldp % 4 == 0 && k_col % 4 == 0 && p.rot_dims % (p.interleaved ? 4 : 8) == 0;
            const int per = four && d.dim <= 128 && part.n >= 512 && p.norm == QkPost::PER_HEAD ? 4 : 1;
            auto kern = !four ? qk_post_kernel<T> : per == 4 ? qk_post4_kernel<T, 1, 4> : d.dim <= 128 ? qk_post4_kernel<T, 1, 1> : d.dim <= 256 ? qk_post4_kernel<T, 2, 1> : qk_post4_kernel<T, 4, 1>;
            const size_t smem = std::max(size_t(8) * d.dim_p * 4, route ? route_few_smem(route->d) : 0);
            if (smem > 48 * 1024) FORGE_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, int(smem)));
            FORGE_CUDA(launch_pdl(kern, dim3((d.heads + d.groups + 7) / 8 + (route ? 1 : 0) + scan.blocks, (part.n + per - 1) / per), dim3(256), smem, st, d, p, proj + size_t(r0) * ldp, ldp, k_col, q_norm, k_norm,
                                  reinterpret_cast<const float2*>(rope), static_cast<T*>(q) + size_t(r0) * d.heads * d.dim_p, static_cast<T*>(cache), place + r0, part, beside, scan));
            FORGE_LAUNCH_CHECK();
        }
        return FORGE_OK;
    };
    return dtype == FORGE_F32 ? go(float{}) : go(__nv_bfloat16{});
}

bool attn_rows_supported(const AttnDims& d) { return d.vdim_p <= 512 && smem_bytes(d, 4) <= 200 * 1024; }

int32_t attn_rows(const AttnDims& d, int dtype, const void* q, const void* cache, const float* gate, const float* sink, const float* bias, void* out, int out_ld, const StepRows& rows, int max_keys,
                  cudaStream_t st) {
    if (rows.n <= 0) return FORGE_OK;
    if (!attn_rows_supported(d)) { set_error("row attention: head sizes %d / %d unsupported", d.dim, d.vdim); return FORGE_ERR_SHAPE; }
    if (dtype == FORGE_BF16 && mma_supported(d)) return run_mma(d, q, cache, gate, sink, bias, out, out_ld, rows, max_keys, st);
    const int gq = d.heads / d.groups, blocks = (gq + 3) / 4;
    int splits = 1;   // about two CTAs per SM, no split shorter than one round of its warps
    while (splits < 8 && rows.n * d.groups * blocks * splits * 2 <= 296 && max_keys > splits * kThreads) splits *= 2;
    return dtype == FORGE_F32 ? run<float>(d, q, cache, gate, sink, bias, out, out_ld, rows, splits, st) : run<__nv_bfloat16>(d, q, cache, gate, sink, bias, out, out_ld, rows, splits, st);
}

}  // namespace forge
