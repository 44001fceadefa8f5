// Latent attention of single rows (decode, short portions) on the tensor cores, bfloat16.  All heads of a row share the
// cached latents, so sixteen heads form one MMA tile: S[head][key] = Q_abs C^T over the whole cache row (latent and rotated
// part), O[head][latent] += P C with the SAME page as the value operand - a page is read once for both.
//
// One CTA = sixteen heads of one row and one split of its pages.  A producer warp requests a page (one box of 64-column chunks,
// SWIZZLE_128B) per stage of a two-stage ring; eight consumer warps form the scores (four groups of sixteen keys x two halves
// of the columns, the query fragments stay in registers), the running softmax (two heads per warp) and the sums (sixteen
// latent columns at a time per warp).  mma.sync m16n8k16: sixteen heads are an eighth of a tcgen05 tile, and the kernel is
// bound by the cache stream.  The partial results are merged by the value projection's kernel.
#include <algorithm>
#include <cstring>

#include "mla.cuh"
#include "mma.cuh"
#include "tc5.cuh"

namespace forge {

namespace {

using namespace tc5;

constexpr int kConsumers = 256, kThreads = kConsumers + 32;
constexpr int kStages = 2;
constexpr int kPage = FORGE_KV_PAGE;
constexpr int kSLd = 68, kPLd = 72;

__device__ __forceinline__ void consumer_sync() { asm volatile("bar.sync 1, 256;" ::: "memory"); }

// byte offset of (key, col) in a page stage: 64-column chunks of 64 swizzled 128-byte rows
__device__ __forceinline__ uint32_t page_off(int key, int col) {
    return uint32_t((col >> 6) * (kPage * 128) + key * 128 + ((((col & 63) >> 3) ^ (key & 7)) << 4));
}

// NCH: most 64-column chunks of a cache row
template <int NCH>
__global__ void __launch_bounds__(kThreads, 1) latent_decode_kernel(const __grid_constant__ CUtensorMap map, const LatentDims d, const __nv_bfloat16* __restrict__ qabs,
                                                                    const StepRows rows, float scale2, float* __restrict__ part, float2* __restrict__ ml, int* err) {
    extern __shared__ __align__(1024) unsigned char smem_raw[];
    const int W = d.row(), stage_bytes = W * kPage * 2, ldq = W + 8;
    unsigned char* ring = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
    __nv_bfloat16* sQ = reinterpret_cast<__nv_bfloat16*>(ring + kStages * stage_bytes);
    float* sS = reinterpret_cast<float*>(sQ + 16 * ldq);
    __nv_bfloat16* sP = reinterpret_cast<__nv_bfloat16*>(sS + 2 * 16 * kSLd);
    __shared__ uint64_t full[kStages], empty[kStages];
    __shared__ float s_alpha[16];
    __shared__ int s_err;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int split = blockIdx.x, splits = gridDim.x, h0 = blockIdx.y * 16, r = blockIdx.z;
    if (tid == 0) {
        for (int s = 0; s < kStages; ++s) { mbar_init(&full[s], 1); mbar_init(&empty[s], 8); }
        s_err = 0;
        mbar_fence_init();
    }
    __syncthreads();
    pdl_trigger();
    // positions and page tables are written in front of the step's first kernel, which is launched without overlap
    const int pos = rows.pos[r], seq = rows.seq ? rows.seq[r] : r;
    const int pages = pos / kPage + 1;
    const int n = pages > split ? (pages - split + splits - 1) / splits : 0;

    if (warp == 8) {
        // the warp reads 32 entries of the page table at a time; lane 0 requests the pages
        const int32_t* pt = rows.page_table + size_t(seq) * rows.pages_per_seq;
        int entry = lane < n ? pt[split + lane * splits] : 0;
        auto request = [&](int i) {
            const int s = i % kStages, y = __shfl_sync(0xffffffffu, entry, i & 31) * kPage;
            if (lane == 0) {
                mbar_expect_tx(&full[s], uint32_t(stage_bytes));
                tma_3d(ring + size_t(s) * stage_bytes, &map, 0, y, 0, &full[s]);
            }
            __syncwarp();
        };
        // pages that hold no row of this step are complete already: the first ones are requested before the wait
        const int complete = (pos - rows.fresh + 1) / kPage;   // (rounds towards zero: 0 if nothing is older than the step)
        int i = 0;
        for (; i < n && i < kStages && split + i * splits < complete; ++i) request(i);
        pdl_wait();
        for (; i < n; ++i) {
            if ((i & 31) == 0 && i > 0) entry = i + lane < n ? pt[split + (i + lane) * splits] : 0;
            const bool ok = i < kStages || mbar_wait(&empty[i % kStages], (i / kStages - 1) & 1, &s_err);
            if (!__all_sync(0xffffffffu, ok)) { atomicExch(&s_err, 1); break; }
            request(i);
        }
    } else {
        pdl_wait();
        // queries into shared memory (heads past the last are zero), then this warp's half of them into registers
        {
            const uint4* src = reinterpret_cast<const uint4*>(qabs + (size_t(r) * d.heads + h0) * W);
            const int per = W / 8, have = min(16, d.heads - h0) * per;
            uint4 v[5];   // every load before the first store; a row has at most nine chunks of eight pieces
#pragma unroll
            for (int u = 0; u < 5; ++u) v[u] = tid + u * kConsumers < have ? src[tid + u * kConsumers] : make_uint4(0, 0, 0, 0);
#pragma unroll
            for (int u = 0; u < 5; ++u) {
                const int i = tid + u * kConsumers;
                if (i < 16 * per) *reinterpret_cast<uint4*>(sQ + (i / per) * ldq + (i % per) * 8) = v[u];
            }
        }
        consumer_sync();
        const int kg = warp & 3, kh = warp >> 2;
        const int half = W / 32;                 // sixteen-column steps of one half
        const int j = lane >> 3, jr = lane & 7;
        uint32_t qf[NCH * 2][4];
#pragma unroll
        for (int i = 0; i < NCH * 2; ++i)
            if (i < half) ldsm4(qf[i], smem_u32(sQ + ((j & 1) * 8 + jr) * ldq + (kh * half + i) * 16 + (j >> 1) * 8));
        float acc[4][2][4];
#pragma unroll
        for (int t = 0; t < 4; ++t)
#pragma unroll
            for (int b = 0; b < 2; ++b)
#pragma unroll
                for (int e = 0; e < 4; ++e) acc[t][b][e] = 0.f;
        const int nt = d.rank_p / 16;            // sixteen-column tiles of the latent; this warp: warp, warp + 8, ...
        float m_run = -INFINITY, l_run = 0.f;    // of head 2 warp + (lane >> 4), kept by sixteen lanes
        const int sh = 2 * warp + (lane >> 4), sl = lane & 15;
        for (int i = 0; i < n; ++i) {
            const int s = i % kStages;
            // every warp of the CTA meets at the barriers below, so a wait that gave up must not leave the loop alone
            if (!mbar_wait(&full[s], (i / kStages) & 1, &s_err)) atomicExch(&s_err, 1);
            const uint32_t page = smem_u32(ring + size_t(s) * stage_bytes);
            float sc[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
#pragma unroll
            for (int k = 0; k < NCH * 2; ++k)
                if (k < half) {
                    uint32_t b[4];
                    ldsm4(b, page + page_off(kg * 16 + (j >> 1) * 8 + jr, (kh * half + k) * 16 + (j & 1) * 8));
                    mma(sc[0], qf[k], b[0], b[1]);
                    mma(sc[1], qf[k], b[2], b[3]);
                }
            {
                float* dst = sS + kh * 16 * kSLd + (lane >> 2) * kSLd + kg * 16 + (lane & 3) * 2;
#pragma unroll
                for (int b = 0; b < 2; ++b) {
                    *reinterpret_cast<float2*>(dst + b * 8) = make_float2(sc[b][0], sc[b][1]);
                    *reinterpret_cast<float2*>(dst + 8 * kSLd + b * 8) = make_float2(sc[b][2], sc[b][3]);
                }
            }
            consumer_sync();
            {
                const int key0 = (split + i * splits) * kPage;
                const float4 a = *reinterpret_cast<const float4*>(sS + sh * kSLd + sl * 4), b = *reinterpret_cast<const float4*>(sS + (16 + sh) * kSLd + sl * 4);
                float v[4] = {(a.x + b.x) * scale2, (a.y + b.y) * scale2, (a.z + b.z) * scale2, (a.w + b.w) * scale2};
                float mx = -INFINITY;
#pragma unroll
                for (int e = 0; e < 4; ++e) { if (key0 + sl * 4 + e > pos) v[e] = -INFINITY; mx = fmaxf(mx, v[e]); }
#pragma unroll
                for (int o = 8; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
                const float mn = fmaxf(m_run, mx), alpha = exp2f(m_run - mn);   // a page of the split holds at least one visible key
                float sum = 0.f;
#pragma unroll
                for (int e = 0; e < 4; ++e) { v[e] = exp2f(v[e] - mn); sum += v[e]; }
#pragma unroll
                for (int o = 8; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
                l_run = l_run * alpha + sum;
                m_run = mn;
                *reinterpret_cast<uint2*>(sP + sh * kPLd + sl * 4) = make_uint2(pack_bf2(v[0], v[1]), pack_bf2(v[2], v[3]));
                if (sl == 0) s_alpha[sh] = alpha;
            }
            consumer_sync();
            const float al0 = s_alpha[lane >> 2], al1 = s_alpha[(lane >> 2) + 8];
            uint32_t pf[4][4];
#pragma unroll
            for (int k = 0; k < 4; ++k) ldsm4(pf[k], smem_u32(sP + ((j & 1) * 8 + jr) * kPLd + k * 16 + (j >> 1) * 8));
#pragma unroll
            for (int t = 0; t < 4; ++t) {
                const int tile = warp + t * 8;
                if (tile < nt) {
#pragma unroll
                    for (int b = 0; b < 2; ++b) { acc[t][b][0] *= al0; acc[t][b][1] *= al0; acc[t][b][2] *= al1; acc[t][b][3] *= al1; }
#pragma unroll
                    for (int k = 0; k < 4; ++k) {
                        uint32_t b[4];
                        ldsm4t(b, page + page_off(k * 16 + (j & 1) * 8 + jr, tile * 16 + (j >> 1) * 8));
                        mma(acc[t][0], pf[k], b[0], b[1]);
                        mma(acc[t][1], pf[k], b[2], b[3]);
                    }
                }
            }
            __syncwarp();
            if (lane == 0) mbar_arrive(&empty[s]);
        }
#pragma unroll
        for (int t = 0; t < 4; ++t) {
            const int tile = warp + t * 8;
            if (n > 0 && tile < nt)
#pragma unroll
                for (int b = 0; b < 2; ++b)
#pragma unroll
                    for (int hf = 0; hf < 2; ++hf) {
                        const int h = h0 + (lane >> 2) + hf * 8;
                        if (h < d.heads)
                            *reinterpret_cast<float2*>(part + ((size_t(r) * d.heads + h) * splits + split) * d.rank_p + tile * 16 + b * 8 + (lane & 3) * 2) =
                                make_float2(acc[t][b][2 * hf], acc[t][b][2 * hf + 1]);
                    }
        }
        if (sl == 0 && h0 + sh < d.heads) ml[(size_t(r) * d.heads + h0 + sh) * splits + split] = make_float2(m_run, l_run);
    }
    __syncthreads();
    if (tid == 0 && s_err && err) atomicExch(err, 1);
}

size_t decode_smem(const LatentDims& d) {
    return size_t(kStages) * d.row() * kPage * 2 + size_t(16) * (d.row() + 8) * 2 + sizeof(float) * 2 * 16 * kSLd + size_t(16) * kPLd * 2 + 1024;
}

template <int NCH>
int32_t launch(const LatentDims& d, const void* qabs, const void* map, const StepRows& rows, int splits, float* part, float2* ml, int* err, cudaStream_t st) {
    CUtensorMap m;
    memcpy(&m, map, sizeof(m));
    auto kern = latent_decode_kernel<NCH>;
    const size_t smem = decode_smem(d);
    FORGE_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, int(smem)));
    FORGE_CUDA(launch_pdl(kern, dim3(splits, (d.heads + 15) / 16, rows.n), dim3(kThreads), smem, st, m, d, static_cast<const __nv_bfloat16*>(qabs), rows,
                          d.scale * 1.4426950408889634f, part, ml, err));
    FORGE_LAUNCH_CHECK();
    return FORGE_OK;
}

}  // namespace

bool latent_decode_tc_supported(const LatentDims& d) { return d.row() <= 9 * 64 && d.rank_p <= 512; }
int latent_decode_head_groups(const LatentDims& d) { return (d.heads + 15) / 16; }

int32_t latent_cache_map(void* map_out, const void* cache, const LatentDims& d, size_t rows) {
    CUtensorMap m;
    // {64 columns, rows, chunks}: one box brings a whole page as chunks of swizzled 128-byte rows
    const uint64_t dims[3] = {64, rows, uint64_t(d.row() / 64)}, strides[2] = {uint64_t(d.row()) * 2, 128};
    const uint32_t box[3] = {64, kPage, uint32_t(d.row() / 64)};
    FORGE_TRY(make_map(&m, cache, 3, dims, strides, box));
    memcpy(map_out, &m, sizeof(m));
    return FORGE_OK;
}

int32_t latent_decode_tc(const LatentDims& d, const void* qabs, const void* map, const StepRows& rows, int splits, float* part, float2* ml, int* err, cudaStream_t st) {
    if (rows.n <= 0) return FORGE_OK;
    if (!latent_decode_tc_supported(d)) { set_error("latent decode: rows of %d values unsupported", d.row()); return FORGE_ERR_SHAPE; }
    const int nch = d.row() / 64;
    if (nch <= 3) return launch<3>(d, qabs, map, rows, splits, part, ml, err, st);
    if (nch <= 5) return launch<5>(d, qabs, map, rows, splits, part, ml, err, st);
    return launch<9>(d, qabs, map, rows, splits, part, ml, err, st);
}

}  // namespace forge
