// Latent attention, the parts around the score product: append to the cache, queries into the latent space, attention of
// single rows on the CUDA cores (float32 models, and bfloat16 sizes the tensor-core kernel does not take), merge of the
// splits with the value projection and the output gate.  T is the model's type (bfloat16 or float32); everything is
// computed in f32.
#include <algorithm>

#include "mla.cuh"

namespace forge {

namespace {

__device__ __forceinline__ float2 load2(const float* p) { return *reinterpret_cast<const float2*>(p); }
__device__ __forceinline__ float2 load2(const __nv_bfloat16* p) { return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p)); }

constexpr int kThreads = 256;

__device__ __forceinline__ float block_sum(float v, float* red) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    __syncthreads();
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
    __syncthreads();
    float s = 0.f;
    for (int w = 0; w < int(blockDim.x >> 5); ++w) s += red[w];
    return s;
}

// entry i of a rotated vector of n values whose first `dims` turn in the pairs (i, i + dims/2); cs = the position's table row
__device__ __forceinline__ float rotated(const float* x, int i, int dims, const float2* cs) {
    const int half = dims >> 1;
    if (i >= dims) return x[i];
    if (i < half) { const float2 t = cs[i]; return x[i] * t.x - x[i + half] * t.y; }
    const float2 t = cs[i - half];
    return x[i] * t.x + x[i - half] * t.y;
}

template <typename T>
__device__ void append_row(const LatentDims& d, const float* down, const float* kv_norm, const float2* cs, T* dst, float* red) {
    float ss = 0.f;
    for (int i = threadIdx.x; i < d.rank; i += blockDim.x) ss += down[i] * down[i];
    ss = block_sum(ss, red);
    const float inv = 1.0f / sqrtf(ss / float(d.rank) + d.eps);
    for (int i = threadIdx.x; i < d.rank_p; i += blockDim.x) dst[i] = to_t<T>(i < d.rank ? down[i] * inv * kv_norm[i] : 0.f);
    for (int i = threadIdx.x; i < d.rot_p; i += blockDim.x) dst[d.rank_p + i] = to_t<T>(i < d.rot ? rotated(down + d.rank, i, d.rot_dims, cs) : 0.f);
}

constexpr int kAbsorbCols = 128;   // latent columns per CTA

// blockIdx.x: group of RB rows.  blockIdx.y < heads * col blocks: queries of one head into 128 latent columns; the last RB
// values of blockIdx.y append one row each to the cache.
// Eight consecutive constant weights held in registers from in front of the dependency wait.  bf16 and one row per CTA only: a
// float32 model loads them where they are used, and with several rows the registers are worth more (the weights are then
// only asked towards L2).
template <typename T> struct Held { static constexpr bool on = false; __device__ __forceinline__ void fetch(const T*) {} __device__ __forceinline__ void get(float (&)[8]) const {} };
template <> struct Held<__nv_bfloat16> {
    static constexpr bool on = true;
    uint4 u;
    __device__ __forceinline__ void fetch(const __nv_bfloat16* p) { u = *reinterpret_cast<const uint4*>(p); }
    __device__ __forceinline__ void get(float (&v)[8]) const {
        const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&u);
#pragma unroll
        for (int i = 0; i < 4; ++i) { const float2 f = __bfloat1622float2(h[i]); v[2 * i] = f.x; v[2 * i + 1] = f.y; }
    }
};

template <typename T, int RB>
__global__ void __launch_bounds__(kThreads) latent_post_kernel(const LatentDims d, const float* proj, int ldp, int dkv_col, const float* __restrict__ kv_norm,
                                                               const float2* __restrict__ rope, const T* __restrict__ uk, int uk_ld, T* __restrict__ qabs, T* __restrict__ cache,
                                                               const StepRows rows) {
    extern __shared__ float sm[];   // queries [RB][dim], then partial sums [8][RB][128]
    __shared__ float red[32];
    const int nrb = (d.rank_p + kAbsorbCols - 1) / kAbsorbCols;
    const int r0 = blockIdx.x * RB, nr = min(RB, rows.n - r0);
    if (int(blockIdx.y) >= d.heads * nrb) {
        const int r = r0 + int(blockIdx.y) - d.heads * nrb;
        pdl_trigger();
        pdl_wait();
        if (r < rows.n) {
            const int pos = rows.pos[r];
            append_row<T>(d, proj + size_t(r) * ldp + dkv_col, kv_norm, rope + size_t(pos) * (d.rot_dims / 2), cache + cache_row(rows, r, pos) * d.row(), red);
        }
        return;
    }
    const int h = blockIdx.y / nrb, c0 = (blockIdx.y % nrb) * kAbsorbCols;
    const T* w = uk + size_t(h) * d.dim * uk_ld + c0;
    // sixteen threads cover the columns, sixteen groups of them share the dimensions; the weights are constant: the first
    // kHeld rows of every thread are fetched while the kernel in front runs
    constexpr int kHeld = 8;
    constexpr bool kHold = Held<T>::on && RB == 1;
    const int col = (threadIdx.x & 15) * 8, group = threadIdx.x >> 4;
    const bool col_ok = c0 + col < d.rank_p;
    Held<T> held[kHeld];
    if (!kHold)
        for (int i = threadIdx.x; i < d.dim * 2; i += kThreads)
            asm volatile("prefetch.global.L2 [%0];" ::"l"(reinterpret_cast<const char*>(w + size_t(i >> 1) * uk_ld) + (i & 1) * 128));
    if (kHold && col_ok)
#pragma unroll
        for (int i = 0; i < kHeld; ++i) if (group + 16 * i < d.dim) held[i].fetch(w + size_t(group + 16 * i) * uk_ld + col);
    pdl_trigger();
    pdl_wait();
    float* sq = sm;
    float* sp = sm + RB * d.dim;
    const int qd = d.dim + d.rot;
    for (int i = threadIdx.x; i < RB * d.dim; i += kThreads) {
        const int j = i / d.dim, e = i % d.dim;
        sq[i] = j < nr ? proj[size_t(r0 + j) * ldp + h * qd + e] : 0.f;
    }
    __syncthreads();
    float a[RB][8];
#pragma unroll
    for (int j = 0; j < RB; ++j)
#pragma unroll
        for (int c = 0; c < 8; ++c) a[j][c] = 0.f;
    if (col_ok) {
        auto add = [&](int e, const float (&v)[8]) {
#pragma unroll
            for (int j = 0; j < RB; ++j) {
                const float q = sq[j * d.dim + e];
#pragma unroll
                for (int c = 0; c < 8; ++c) a[j][c] = fmaf(q, v[c], a[j][c]);
            }
        };
        float v[8];
        if (kHold)
#pragma unroll
            for (int i = 0; i < kHeld; ++i) if (group + 16 * i < d.dim) { held[i].get(v); add(group + 16 * i, v); }
#pragma unroll 8
        for (int e = group + (kHold ? 16 * kHeld : 0); e < d.dim; e += 16) { load8(v, w + size_t(e) * uk_ld + col); add(e, v); }
    }
#pragma unroll
    for (int j = 0; j < RB; ++j) {   // lanes l and l + 16 hold the same columns
#pragma unroll
        for (int c = 0; c < 8; ++c) a[j][c] += __shfl_xor_sync(0xffffffffu, a[j][c], 16);
        if (!(threadIdx.x & 16))
#pragma unroll
            for (int c = 0; c < 8; ++c) sp[((threadIdx.x >> 5) * RB + j) * 128 + col + c] = a[j][c];
    }
    __syncthreads();
    for (int i = threadIdx.x; i < RB * 128; i += kThreads) {
        const int j = i >> 7, c = i & 127;
        if (j < nr && c0 + c < d.rank_p) {
            float s = 0.f;
#pragma unroll
            for (int q = 0; q < 8; ++q) s += sp[(q * RB + j) * 128 + c];
            qabs[(size_t(r0 + j) * d.heads + h) * d.row() + c0 + c] = to_t<T>(s);
        }
    }
    if (c0 == 0)
        for (int i = threadIdx.x; i < nr * d.rot_p; i += kThreads) {
            const int j = i / d.rot_p, e = i % d.rot_p;
            const float2* cs = rope + size_t(rows.pos[r0 + j]) * (d.rot_dims / 2);
            const float* x = proj + size_t(r0 + j) * ldp + h * qd + d.dim;
            qabs[(size_t(r0 + j) * d.heads + h) * d.row() + d.rank_p + e] = to_t<T>(e < d.rot ? rotated(x, e, d.rot_dims, cs) : 0.f);
        }
}

// prompt rows: one CTA per row
__global__ void __launch_bounds__(kThreads) latent_prompt_kernel(const LatentDims d, const float* __restrict__ proj, int ldp, int dkv_col, const float* __restrict__ kv_norm,
                                                                 const float2* __restrict__ rope, __nv_bfloat16* __restrict__ q, __nv_bfloat16* __restrict__ cache, const StepRows rows) {
    __shared__ float red[32];
    const int r = blockIdx.x, pos = rows.pos[r];
    const float* src = proj + size_t(r) * ldp;
    const float2* cs = rope + size_t(pos) * (d.rot_dims / 2);
    append_row<__nv_bfloat16>(d, src + dkv_col, kv_norm, cs, cache + cache_row(rows, r, pos) * d.row(), red);
    const int qd = d.dim + d.rot, qp = d.dim_p + d.rot_p;
    __nv_bfloat16* dst = q + size_t(r) * d.heads * qp;
    const int lane = threadIdx.x & 31;
    for (int h = threadIdx.x >> 5; h < d.heads; h += kThreads / 32) {   // a warp per head
        const float* x = src + h * qd;
        __nv_bfloat162* out = reinterpret_cast<__nv_bfloat162*>(dst + h * qp);
#pragma unroll 4
        for (int e = 2 * lane; e < d.dim_p; e += 64) out[e >> 1] = __floats2bfloat162_rn(e < d.dim ? x[e] : 0.f, e + 1 < d.dim ? x[e + 1] : 0.f);
        for (int t = 2 * lane; t < d.rot_p; t += 64)
            out[(d.dim_p + t) >> 1] = __floats2bfloat162_rn(t < d.rot ? rotated(x + d.dim, t, d.rot_dims, cs) : 0.f, t + 1 < d.rot ? rotated(x + d.dim, t + 1, d.rot_dims, cs) : 0.f);
    }
}

// one (row, head, split) per CTA; four warps take its pages' 32-key halves in turn
template <typename T>
__global__ void __launch_bounds__(128) latent_attn_kernel(const LatentDims d, const T* qabs, const T* cache, const StepRows rows, float scale2,
                                                          float* __restrict__ part, float2* __restrict__ ml) {
    extern __shared__ float sm[];   // query [row], then per warp the running sums [rank_p]
    __shared__ float sml[4][2];
    const int split = blockIdx.x, splits = gridDim.x, h = blockIdx.y, r = blockIdx.z;
    const int W = d.row(), warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int pos = rows.pos[r], seq = rows.seq ? rows.seq[r] : r;
    float* sq = sm;
    float* so = sm + W + warp * d.rank_p;
    const T* q = qabs + (size_t(r) * d.heads + h) * W;
    for (int i = threadIdx.x; i < W; i += 128) sq[i] = to_f(q[i]);
    for (int i = lane; i < d.rank_p; i += 32) so[i] = 0.f;
    __syncthreads();
    float m = -INFINITY, l = 0.f;
    const int halves = pos / 32 + 1;   // 32-key halves that hold a visible key
    int turn = 0;
    for (int pg = split; pg * 2 < halves; pg += splits)
        for (int hf = 0; hf < 2 && pg * 2 + hf < halves; ++hf) {
            if ((turn++ & 3) != warp) continue;
            const int key0 = pg * FORGE_KV_PAGE + hf * 32;
            const T* base = cache + (size_t(rows.page_table[size_t(seq) * rows.pages_per_seq + pg]) * FORGE_KV_PAGE + hf * 32) * W;
            const T* kr = base + size_t(lane) * W;
            float s0 = 0.f, s1 = 0.f;
            for (int e = 0; e < W; e += 4) {
                const float2 a = load2(kr + e), b = load2(kr + e + 2);
                s0 = fmaf(a.x, sq[e], s0); s1 = fmaf(a.y, sq[e + 1], s1);
                s0 = fmaf(b.x, sq[e + 2], s0); s1 = fmaf(b.y, sq[e + 3], s1);
            }
            const float s = key0 + lane <= pos ? (s0 + s1) * scale2 : -INFINITY;
            float mx = s;
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
            const float mn = fmaxf(m, mx);
            const float alpha = exp2f(m - mn), p = exp2f(s - mn);
            float sum = p;
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
            l = l * alpha + sum;
            m = mn;
            const int keys = min(32, pos - key0 + 1);
            for (int c = lane; c < d.rank_p; c += 32) {
                float acc = so[c] * alpha;
                // (all lanes stay together: rank_p is a multiple of 64)
                for (int k = 0; k < keys; ++k) acc = fmaf(__shfl_sync(0xffffffffu, p, k), to_f(base[size_t(k) * W + c]), acc);
                so[c] = acc;
            }
        }
    if (lane == 0) { sml[warp][0] = m; sml[warp][1] = l; }
    __syncthreads();
    float mt = -INFINITY, lt = 0.f, f[4];
#pragma unroll
    for (int w = 0; w < 4; ++w) mt = fmaxf(mt, sml[w][0]);
#pragma unroll
    for (int w = 0; w < 4; ++w) { f[w] = sml[w][0] == -INFINITY ? 0.f : exp2f(sml[w][0] - mt); lt += sml[w][1] * f[w]; }
    const size_t o = (size_t(r) * d.heads + h) * splits + split;
    for (int c = threadIdx.x; c < d.rank_p; c += 128) {
        float v = 0.f;
#pragma unroll
        for (int w = 0; w < 4; ++w) v += sm[W + w * d.rank_p + c] * f[w];
        part[o * d.rank_p + c] = v;
    }
    if (threadIdx.x == 0) ml[o] = make_float2(mt, lt);
}

constexpr int kValueRows = 32;   // rows of W_uv per CTA

template <typename T, int RB>
__global__ void __launch_bounds__(kThreads) latent_value_kernel(const LatentDims d, const float* part, const float2* ml, int splits,
                                                                const T* __restrict__ uv, int uv_ld, const T* gate, int gate_ld, T* __restrict__ out, int out_ld, int rows, const int32_t* __restrict__ rows_pos) {
    extern __shared__ __align__(16) float sm[];   // merged latents [RB][rank_p], split factors [RB][splits]
    const int h = blockIdx.y, v0 = blockIdx.z * kValueRows, r0 = blockIdx.x * RB, nr = min(RB, rows - r0);
    const int nv = min(kValueRows, d.vdim - v0);
    const T* w = uv + (size_t(h) * d.vdim + v0) * uv_ld;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    // four rows of W_uv per warp; their first kHeld pieces are fetched while the kernel in front runs
    constexpr int VR = kValueRows / (kThreads / 32), kHeld = 2, kUnroll = RB == 1 ? 16 : 4;
    constexpr bool kHold = Held<T>::on && RB == 1;
    Held<T> held[VR][kHeld];
    if (!kHold) {
        const int lines = int((size_t(d.rank_p) * sizeof(T) + 127) / 128);
        for (int i = threadIdx.x; i < nv * lines; i += kThreads)
            asm volatile("prefetch.global.L2 [%0];" ::"l"(reinterpret_cast<const char*>(w + size_t(i / lines) * uv_ld) + (i % lines) * 128));
    }
    if (kHold)
#pragma unroll
    for (int v = 0; v < VR; ++v)
#pragma unroll
        for (int i = 0; i < kHeld; ++i) if (lane * 8 + 256 * i < d.rank_p) held[v][i].fetch(w + size_t(min(warp * VR + v, nv - 1)) * uv_ld + lane * 8 + 256 * i);
    pdl_trigger();
    pdl_wait();
    float* lat = sm;
    float* fac = sm + RB * d.rank_p;
    if (warp < nr) {   // RB <= 8 warps: one row each
        const float2* p = ml + (size_t(r0 + warp) * d.heads + h) * splits;
        float mt = -INFINITY;
        for (int s = lane; s < splits; s += 32) mt = fmaxf(mt, p[s].x);
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) mt = fmaxf(mt, __shfl_xor_sync(0xffffffffu, mt, o));
        float lt = 0.f;
        for (int s = lane; s < splits; s += 32) {
            const float2 a = p[s];
            const float f = a.x == -INFINITY ? 0.f : exp2f(a.x - mt);
            fac[warp * splits + s] = f;
            lt += a.y * f;
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) lt += __shfl_xor_sync(0xffffffffu, lt, o);
        __syncwarp();
        const float inv = 1.0f / lt;
        for (int s = lane; s < splits; s += 32) fac[warp * splits + s] *= inv;
    }
    __syncthreads();
    {
        // four latents per thread; with room to spare two threads share a quad's splits (rank_p / 4 is a multiple of 16)
        const int quads = d.rank_p / 4, halves = nr * quads * 2 <= kThreads ? 2 : 1;
        for (int i = threadIdx.x; i < nr * quads * halves; i += kThreads) {
            const int hf = halves == 2 ? (i >> 4) & 1 : 0, q = halves == 2 ? (i >> 5) * 16 + (i & 15) : i;
            const int j = q / quads, c = (q % quads) * 4;
            const int n = min(splits, rows_pos[r0 + j] / FORGE_KV_PAGE + 1);   // splits that own a page
            const float* p = part + (size_t(r0 + j) * d.heads + h) * splits * d.rank_p + c;
            float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll kUnroll
            for (int s = hf; s < n; s += halves) {
                const float f = fac[j * splits + s];
                const float4 x = *reinterpret_cast<const float4*>(p + size_t(s) * d.rank_p);
                v.x = fmaf(x.x, f, v.x); v.y = fmaf(x.y, f, v.y); v.z = fmaf(x.z, f, v.z); v.w = fmaf(x.w, f, v.w);
            }
            if (halves == 2) {   // whole warps are in the loop (a multiple of 32 items)
                v.x += __shfl_xor_sync(0xffffffffu, v.x, 16); v.y += __shfl_xor_sync(0xffffffffu, v.y, 16);
                v.z += __shfl_xor_sync(0xffffffffu, v.z, 16); v.w += __shfl_xor_sync(0xffffffffu, v.w, 16);
            }
            if (!hf) *reinterpret_cast<float4*>(lat + j * d.rank_p + c) = v;
        }
        for (int i = nr * d.rank_p + threadIdx.x; i < RB * d.rank_p; i += kThreads) lat[i] = 0.f;
    }
    __syncthreads();
    float acc[VR][RB];
#pragma unroll
    for (int v = 0; v < VR; ++v)
#pragma unroll
        for (int j = 0; j < RB; ++j) acc[v][j] = 0.f;
    auto add = [&](int c, const float (&a)[VR][8]) {
#pragma unroll
        for (int j = 0; j < RB; ++j) {
            float x[8];
            load8(x, lat + j * d.rank_p + c);
#pragma unroll
            for (int v = 0; v < VR; ++v)
#pragma unroll
                for (int e = 0; e < 8; ++e) acc[v][j] = fmaf(a[v][e], x[e], acc[v][j]);
        }
    };
    float a[VR][8];
    if (kHold)
#pragma unroll
        for (int i = 0; i < kHeld; ++i)
            if (lane * 8 + 256 * i < d.rank_p) {
#pragma unroll
                for (int v = 0; v < VR; ++v) held[v][i].get(a[v]);
                add(lane * 8 + 256 * i, a);
            }
    for (int c = lane * 8 + (kHold ? 256 * kHeld : 0); c < d.rank_p; c += 256) {
#pragma unroll
        for (int v = 0; v < VR; ++v) load8(a[v], w + size_t(min(warp * VR + v, nv - 1)) * uv_ld + c);
        add(c, a);
    }
#pragma unroll
    for (int v = 0; v < VR; ++v)
#pragma unroll
        for (int j = 0; j < RB; ++j) {
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) acc[v][j] += __shfl_xor_sync(0xffffffffu, acc[v][j], o);
            if (lane == 0 && j < nr && warp * VR + v < nv) {
                const int col = h * d.vdim + v0 + warp * VR + v;
                out[size_t(r0 + j) * out_ld + col] = to_t<T>(acc[v][j] * to_f(gate[size_t(r0 + j) * gate_ld + col]));
            }
        }
}

__global__ void __launch_bounds__(128) latent_gather_kernel(const LatentDims d, const uint4* __restrict__ cache, const int32_t* __restrict__ pages, uint4* __restrict__ c, uint4* __restrict__ krot) {
    const int r = blockIdx.x, W = d.row() / 8, R = d.rank_p / 8;
    const uint4* src = cache + (size_t(pages[r / FORGE_KV_PAGE]) * FORGE_KV_PAGE + r % FORGE_KV_PAGE) * W;
    for (int i = threadIdx.x; i < W; i += 128) {
        if (i < R) c[size_t(r) * R + i] = src[i];
        else krot[size_t(r) * (W - R) + i - R] = src[i];
    }
}

template <typename T>
int32_t post_t(const LatentDims& d, const float* proj, int ldp, int dkv_col, const float* kv_norm, const float* rope, const void* uk, int uk_ld, void* qabs, void* cache,
               const StepRows& rows, cudaStream_t st) {
    const int nrb = (d.rank_p + kAbsorbCols - 1) / kAbsorbCols;
    auto go = [&](auto kern, int rb) -> int32_t {
        const size_t smem = sizeof(float) * size_t(rb) * (d.dim + 8 * 128);
        if (smem > 48 * 1024) FORGE_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, int(smem)));
        FORGE_CUDA(launch_pdl(kern, dim3((rows.n + rb - 1) / rb, d.heads * nrb + rb), dim3(kThreads), smem, st, d, proj, ldp, dkv_col, kv_norm, reinterpret_cast<const float2*>(rope),
                              static_cast<const T*>(uk), uk_ld, static_cast<T*>(qabs), static_cast<T*>(cache), rows));
        FORGE_LAUNCH_CHECK();
        return FORGE_OK;
    };
    if (rows.n <= 2) return go(latent_post_kernel<T, 1>, 1);
    return go(latent_post_kernel<T, 4>, 4);
}

template <typename T>
int32_t value_t(const LatentDims& d, const float* part, const float2* ml, int splits, const void* uv, int uv_ld, const void* gate, int gate_ld, void* out, int out_ld, const StepRows& sr, cudaStream_t st) {
    const int rows = sr.n;
    auto go = [&](auto kern, int rb) -> int32_t {
        const size_t smem = sizeof(float) * size_t(rb) * (d.rank_p + splits);
        if (smem > 48 * 1024) FORGE_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, int(smem)));
        FORGE_CUDA(launch_pdl(kern, dim3((rows + rb - 1) / rb, d.heads, (d.vdim + kValueRows - 1) / kValueRows), dim3(kThreads), smem, st, d, part, ml, splits,
                              static_cast<const T*>(uv), uv_ld, static_cast<const T*>(gate), gate_ld, static_cast<T*>(out), out_ld, rows, sr.pos));
        FORGE_LAUNCH_CHECK();
        return FORGE_OK;
    };
    if (rows <= 2) return go(latent_value_kernel<T, 1>, 1);
    return go(latent_value_kernel<T, 4>, 4);
}

template <typename T>
int32_t attn_t(const LatentDims& d, const void* qabs, const void* cache, const StepRows& rows, int splits, float* part, float2* ml, cudaStream_t st) {
    const size_t smem = sizeof(float) * (size_t(d.row()) + 4 * size_t(d.rank_p));
    auto kern = latent_attn_kernel<T>;
    if (smem > 48 * 1024) FORGE_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, int(smem)));
    kern<<<dim3(splits, d.heads, rows.n), 128, smem, st>>>(d, static_cast<const T*>(qabs), static_cast<const T*>(cache), rows, d.scale * 1.4426950408889634f, part, ml);
    FORGE_LAUNCH_CHECK();
    return FORGE_OK;
}

}  // namespace

int32_t latent_post(const LatentDims& d, int dtype, const float* proj, int ldp, int dkv_col, const float* kv_norm, const float* rope, const void* uk, int uk_ld, void* qabs, void* cache,
                    const StepRows& rows, cudaStream_t st) {
    if (rows.n <= 0) return FORGE_OK;
    if (dtype == FORGE_F32) return post_t<float>(d, proj, ldp, dkv_col, kv_norm, rope, uk, uk_ld, qabs, cache, rows, st);
    return post_t<__nv_bfloat16>(d, proj, ldp, dkv_col, kv_norm, rope, uk, uk_ld, qabs, cache, rows, st);
}
int32_t latent_post_prompt(const LatentDims& d, const float* proj, int ldp, int dkv_col, const float* kv_norm, const float* rope, void* q, void* cache, const StepRows& rows, cudaStream_t st) {
    if (rows.n <= 0) return FORGE_OK;
    latent_prompt_kernel<<<rows.n, kThreads, 0, st>>>(d, proj, ldp, dkv_col, kv_norm, reinterpret_cast<const float2*>(rope), static_cast<__nv_bfloat16*>(q), static_cast<__nv_bfloat16*>(cache), rows);
    FORGE_LAUNCH_CHECK();
    return FORGE_OK;
}
int32_t latent_attn_rows(const LatentDims& d, int dtype, const void* qabs, const void* cache, const StepRows& rows, int splits, float* part, float2* ml, cudaStream_t st) {
    if (rows.n <= 0) return FORGE_OK;
    return dtype == FORGE_F32 ? attn_t<float>(d, qabs, cache, rows, splits, part, ml, st) : attn_t<__nv_bfloat16>(d, qabs, cache, rows, splits, part, ml, st);
}
int32_t latent_value(const LatentDims& d, int dtype, const float* part, const float2* ml, int splits, const void* uv, int uv_ld, const void* gate, int gate_ld, void* out, int out_ld,
                     const StepRows& rows, cudaStream_t st) {
    if (rows.n <= 0) return FORGE_OK;
    return dtype == FORGE_F32 ? value_t<float>(d, part, ml, splits, uv, uv_ld, gate, gate_ld, out, out_ld, rows, st)
                              : value_t<__nv_bfloat16>(d, part, ml, splits, uv, uv_ld, gate, gate_ld, out, out_ld, rows, st);
}
int32_t latent_gather_context(const LatentDims& d, const void* cache, const int32_t* pages, int rows, void* c, void* krot, cudaStream_t st) {
    if (rows <= 0) return FORGE_OK;
    latent_gather_kernel<<<rows, 128, 0, st>>>(d, static_cast<const uint4*>(cache), pages, static_cast<uint4*>(c), static_cast<uint4*>(krot));
    FORGE_LAUNCH_CHECK();
    return FORGE_OK;
}

}  // namespace forge
