// Attention of single rows (decode, short portions, float32 prompts) over a paged cache.
//
// One CTA = up to eight query heads of one key / value head, one row, one of up to eight ranges of its keys; the CTAs of a row form a
// cluster and merge their sums through distributed shared memory.  A warp takes 32 keys at a time: eight keys by four lanes for
// the scores, then a lane per pair of value columns for the sums.  Everything behind the loads is f32.
#include <cooperative_groups.h>

#include <algorithm>

#include "attn_rows.cuh"

namespace forge {

namespace {

namespace cg = cooperative_groups;

constexpr int kWarps = 8, kThreads = kWarps * 32;
constexpr float kLog2e = 1.4426950408889634f;

__device__ __forceinline__ float2 load_pair(const float* p) { return *reinterpret_cast<const float2*>(p); }
__device__ __forceinline__ float2 load_pair(const __nv_bfloat16* p) { return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p)); }

// (What a kernel in front writes is not __restrict__: loads of it may not be moved above the dependency wait.)
// GQ: query heads per CTA; VP: pairs of value columns per lane
template <typename T, int GQ, int VP>
__global__ void __launch_bounds__(kThreads) attn_rows_kernel(const AttnDims d, const T* q, const T* cache, const float* gate, const float* __restrict__ sink,
                                                             T* __restrict__ out, int out_ld, const StepRows rows) {
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
    // the visible keys are numbered: the kept first ones, then those from lo
    const int lo = d.first_key(pos), kept = d.kept(pos), n = kept + pos - lo + 1;
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
    auto row_of = [&](int i) { const int key = i < kept ? i : lo + i - kept; return size_t(pt[key / FORGE_KV_PAGE]) * FORGE_KV_PAGE + key % FORGE_KV_PAGE; };
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
    __syncthreads();
    if (threadIdx.x < GQ) {   // maximum and sum of the CTA
        const int h = threadIdx.x;
        float mt = -INFINITY, lt = 0.f;
        for (int w = 0; w < kWarps; ++w) mt = fmaxf(mt, sml[(w * GQ + h) * 2]);
        for (int w = 0; w < kWarps; ++w) {
            const float f = mt == -INFINITY ? 0.f : exp2f(sml[(w * GQ + h) * 2] - mt);
            lt += sml[(w * GQ + h) * 2 + 1] * f;
            sml[(w * GQ + h) * 2] = f;     // the warp's factor
        }
        cml[2 * h] = mt; cml[2 * h + 1] = lt;
    }
    __syncthreads();
    for (int i = threadIdx.x; i < GQ * d.vdim_p; i += kThreads) {   // own element of every warp: read, then written over warp 0's
        const int h = i / d.vdim_p;
        float v = 0.f;
#pragma unroll
        for (int w = 0; w < kWarps; ++w) v += so[w * GQ * d.vdim_p + i] * sml[(w * GQ + h) * 2];
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

size_t smem_bytes(const AttnDims& d, int gq) { return sizeof(float) * (size_t(gq) * d.dim_p + kWarps * gq * 32 + size_t(kWarps) * gq * d.vdim_p + kWarps * gq * 2 + gq * 2); }

template <typename T, int GQ, int VP>
int32_t launch(const AttnDims& d, const void* q, const void* cache, const float* gate, const float* sink, void* out, int out_ld, const StepRows& rows, int splits, cudaStream_t st) {
    auto kern = attn_rows_kernel<T, GQ, VP>;
    const size_t smem = smem_bytes(d, GQ);
    if (smem > 48 * 1024) FORGE_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, int(smem)));
    const int gq = d.heads / d.groups, blocks = (gq + GQ - 1) / GQ;
    FORGE_CUDA(launch_pdl_cluster(kern, dim3(splits, d.groups * blocks, rows.n), dim3(kThreads), splits, smem, st, d, static_cast<const T*>(q), static_cast<const T*>(cache), gate, sink, static_cast<T*>(out), out_ld, rows));
    FORGE_LAUNCH_CHECK();
    return FORGE_OK;
}

template <typename T>
int32_t run(const AttnDims& d, const void* q, const void* cache, const float* gate, const float* sink, void* out, int out_ld, const StepRows& rows, int splits, cudaStream_t st) {
    const int gq = d.heads / d.groups, vp = d.vdim_p / 64;
    auto with_vp = [&](auto gqc) -> int32_t {
        constexpr int GQ = decltype(gqc)::value;
        if (vp <= 1) return launch<T, GQ, 1>(d, q, cache, gate, sink, out, out_ld, rows, splits, st);
        if (vp <= 2) return launch<T, GQ, 2>(d, q, cache, gate, sink, out, out_ld, rows, splits, st);
        return launch<T, GQ, 8>(d, q, cache, gate, sink, out, out_ld, rows, splits, st);
    };
    if (gq == 1) return with_vp(std::integral_constant<int, 1>{});
    if (gq == 2) return with_vp(std::integral_constant<int, 2>{});
    return with_vp(std::integral_constant<int, 4>{});
}

// ------------------------------------------------------------------------------------------------ queries and keys
// One CTA = eight heads (queries first, then keys) of one row, a warp per head.
constexpr int kQkDims = 16;   // values per lane at most
template <typename T>
__global__ void __launch_bounds__(256) qk_post_kernel(const AttnDims d, const QkPost p, const float* proj, int ldp, int k_col, const float* __restrict__ q_norm,
                                                      const float* __restrict__ k_norm, const float2* __restrict__ rope, T* q, T* cache, const int32_t* place, const StepRows rows) {
    extern __shared__ float sm[];
    __shared__ float red[2][8];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, r = blockIdx.y, h = blockIdx.x * 8 + warp;
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

}  // namespace

int32_t qk_post(const AttnDims& d, const QkPost& p, int dtype, const float* proj, int ldp, int k_col, const float* q_norm, const float* k_norm, const float* rope, void* q, void* cache,
                const int32_t* place, const StepRows& rows, cudaStream_t st) {
    if (rows.n <= 0) return FORGE_OK;
    if (d.dim > kQkDims * 32 || p.rot_dims > d.dim || p.rot_dims % 2) { set_error("attention: head size %d with %d rotated dimensions", d.dim, p.rot_dims); return FORGE_ERR_SHAPE; }
    auto go = [&](auto t) -> int32_t {
        using T = decltype(t);
        const size_t smem = size_t(8) * d.dim_p * 4;
        for (int r0 = 0; r0 < rows.n; r0 += 65535) {
            StepRows part = rows;
            part.n = std::min(65535, rows.n - r0);
            part.pos += r0;
            FORGE_CUDA(launch_pdl(qk_post_kernel<T>, dim3((d.heads + d.groups + 7) / 8, part.n), dim3(256), smem, st, d, p, proj + size_t(r0) * ldp, ldp, k_col, q_norm, k_norm,
                                  reinterpret_cast<const float2*>(rope), static_cast<T*>(q) + size_t(r0) * d.heads * d.dim_p, static_cast<T*>(cache), place + r0, part));
            FORGE_LAUNCH_CHECK();
        }
        return FORGE_OK;
    };
    return dtype == FORGE_F32 ? go(float{}) : go(__nv_bfloat16{});
}

bool attn_rows_supported(const AttnDims& d) { return d.vdim_p <= 512 && smem_bytes(d, 4) <= 200 * 1024; }

int32_t attn_rows(const AttnDims& d, int dtype, const void* q, const void* cache, const float* gate, const float* sink, void* out, int out_ld, const StepRows& rows, int max_keys, cudaStream_t st) {
    if (rows.n <= 0) return FORGE_OK;
    if (!attn_rows_supported(d)) { set_error("row attention: head sizes %d / %d unsupported", d.dim, d.vdim); return FORGE_ERR_SHAPE; }
    const int gq = d.heads / d.groups, blocks = (gq + 3) / 4;
    int splits = 1;   // about two CTAs per SM, no split shorter than one round of its warps
    while (splits < 8 && rows.n * d.groups * blocks * splits * 2 <= 296 && max_keys > splits * kThreads) splits *= 2;
    return dtype == FORGE_F32 ? run<float>(d, q, cache, gate, sink, out, out_ld, rows, splits, st) : run<__nv_bfloat16>(d, q, cache, gate, sink, out, out_ld, rows, splits, st);
}

}  // namespace forge
