// Latent attention of single rows (decode, short portions) on the tensor cores (tcgen05 + TMEM), bfloat16.  All heads of a row
// share the cached latents, and a page is the operand of both products, read once:
//   S[key][head]    = C Q_abs^T   the page as the K-major A operand (M = keys), the queries of N = 16 or 32 heads as B;
//   O[latent][head] += C^T P      the same page as the MN-major A operand (M = 128 latent columns), the probabilities as B.
// The few heads are the N side of the products, so a decode step does not pay for a 128-row query tile (an mma.sync form of
// this kernel was bound by the tensor pipe at 16 heads).  A page has 64 rows, the MMA 128: the upper half of S is formed
// from whatever follows in shared memory (always inside the CTA's allocation) and never read.
//
// One CTA = N heads of one row and one split of its pages.  Warp roles (224 threads): 0 = TMA producer (a page is one box of
// 64-column chunks, SWIZZLE_128B, a two-stage ring; pages of earlier steps are requested before the dependency wait), 1 = TMEM allocation and
// the products of S, 2..5 = softmax, 6 = the products of O (two issuing threads: with one, a page's O would wait for the
// arrival of the next page).  S is turned in shared memory so that 128 / N lanes share a head's 64 scores; the
// probabilities go to shared memory as the next B operand.  The running maximum is lazy (as in attn_prefill_tc5.cu): O is
// rescaled in tensor memory only when a maximum has grown by more than 2^8.  The partial results of the splits are merged by
// the value projection's kernel.
#include <algorithm>
#include <cstring>

#include "mla.cuh"
#include "tc5.cuh"

namespace forge {

namespace {

using namespace tc5;

constexpr int kThreads = 224, kStages = 2, kPage = FORGE_KV_PAGE;
constexpr int kChunk = kPage * 128;      // bytes of one 64-column chunk of a page
constexpr int kSLd = 68;
constexpr float kLazy = 8.f;

// A MN-major (bit 15), B K-major
__device__ __forceinline__ constexpr uint32_t idesc_a_mn(int n) { return idesc_bf16(n) | (1u << 15); }

__device__ __forceinline__ void softmax_sync() { asm volatile("bar.sync 1, 128;" ::: "memory"); }
__device__ __forceinline__ bool softmax_sync_or(bool v) {
    uint32_t r;
    asm volatile("{\n.reg .pred p, q;\nsetp.ne.u32 p, %1, 0;\nbar.red.or.pred q, 1, 128, p;\nselp.u32 %0, 1, 0, q;\n}" : "=r"(r) : "r"(uint32_t(v)) : "memory");
    return r != 0;
}
template <int N> __device__ __forceinline__ void tmem_ld(uint32_t addr, uint32_t (&v)[N]) {
    if constexpr (N == 16) tmem_ld16(addr, v);
    else tmem_ld32(addr, v);
}
__device__ __forceinline__ void tmem_st16(uint32_t taddr, const uint32_t (&v)[16]) {
    asm volatile("tcgen05.st.sync.aligned.32x32b.x16.b32 [%0], {%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16};"
                 ::"r"(taddr), "r"(v[0]), "r"(v[1]), "r"(v[2]), "r"(v[3]), "r"(v[4]), "r"(v[5]), "r"(v[6]), "r"(v[7]), "r"(v[8]),
                   "r"(v[9]), "r"(v[10]), "r"(v[11]), "r"(v[12]), "r"(v[13]), "r"(v[14]), "r"(v[15]) : "memory");
}
template <int N> __device__ __forceinline__ void tmem_st(uint32_t addr, const uint32_t (&v)[N]) {
    if constexpr (N == 16) tmem_st16(addr, v);
    else tmem_st32(addr, v);
}

template <int N, uint32_t COLS>
__global__ void __launch_bounds__(kThreads, 1) latent_decode_kernel(const __grid_constant__ CUtensorMap map, const __grid_constant__ CUtensorMap map_q, const LatentDims d, const StepRows rows,
                                                                    float scale2, float* __restrict__ part, float2* __restrict__ ml, int* err) {
    extern __shared__ __align__(1024) unsigned char smem_raw[];
    const int W = d.row(), nch = W / 64, stage_bytes = nch * kChunk, tiles = (d.rank_p + 127) / 128;
    unsigned char* ring = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
    unsigned char* sQ = ring + kStages * stage_bytes;          // [chunk][head][64 columns], swizzled
    unsigned char* sP = sQ + nch * N * 128;                    // [2][head][64 keys], swizzled
    float* sS = reinterpret_cast<float*>(sP + 2 * N * 128);    // [head][key]
    __shared__ uint64_t full[kStages], empty[kStages], q_full, s_full[2], s_free[2], p_full[2], pv_done[2];
    __shared__ float s_alpha[N];
    __shared__ uint32_t s_tmem;
    __shared__ int s_err;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int split = blockIdx.x, splits = gridDim.x, h0 = blockIdx.y * N, r = blockIdx.z;
    if (tid == 0) {
        mbar_init(&q_full, 1);
        for (int s = 0; s < kStages; ++s) { mbar_init(&full[s], 1); mbar_init(&empty[s], 1); }
        for (int s = 0; s < 2; ++s) { mbar_init(&s_full[s], 1); mbar_init(&s_free[s], 2); mbar_init(&p_full[s], 4); mbar_init(&pv_done[s], 1); }
        s_err = 0;
        mbar_fence_init();
    }
    if (warp == 1) tmem_alloc<COLS>(&s_tmem);
    fence_before();
    __syncthreads();
    fence_after();
    const uint32_t tmem = s_tmem, t_o = tmem + 2 * N;
    pdl_trigger();
    // positions and page tables are written in front of the step's first kernel, which is launched without overlap
    const int pos = rows.pos[r], seq = rows.seq ? rows.seq[r] : r;
    const int pages = pos / kPage + 1;
    const int n = pages > split ? (pages - split + splits - 1) / splits : 0;

    if (warp == 0) {
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
            // the row's queries (heads past the last read the next row's, or zero past the end: their columns are not used)
        if (n > 0 && lane == 0) {
            mbar_expect_tx(&q_full, uint32_t(nch * N * 128));
            tma_3d(sQ, &map_q, 0, r * d.heads + h0, 0, &q_full);
        }
        for (; i < n; ++i) {
            if ((i & 31) == 0 && i > 0) entry = i + lane < n ? pt[split + (i + lane) * splits] : 0;
            const bool ok = i < kStages || mbar_wait(&empty[i % kStages], (i / kStages - 1) & 1, &s_err);
            if (!__all_sync(0xffffffffu, ok)) { atomicExch(&s_err, 1); break; }
            request(i);
        }
    }
    if (warp == 1) {
        if (lane == 0 && n > 0) {
            const uint64_t q_desc = desc_kmajor(smem_u32(sQ));
            if (!mbar_wait(&q_full, 0, &s_err)) atomicExch(&s_err, 1);
            for (int j = 0; j < n; ++j) {
                if (!mbar_wait(&full[j % kStages], (j / kStages) & 1, &s_err) || (j >= 2 && !mbar_wait(&s_free[j & 1], ((j >> 1) - 1) & 1, &s_err))) { atomicExch(&s_err, 1); break; }
                fence_after();
                uint64_t a = desc_kmajor(smem_u32(ring + size_t(j % kStages) * stage_bytes)), b = q_desc;
                const uint32_t t_s = tmem + uint32_t((j & 1) * N);
                for (int c = 0; c < nch; ++c, a += kChunk >> 4, b += (N * 128) >> 4)
#pragma unroll
                    for (int k = 0; k < 4; ++k) umma_ss(t_s, a + uint64_t(k * 2), b + uint64_t(k * 2), idesc_bf16(N), (c > 0 || k > 0) ? 1u : 0u);
                umma_commit(&s_full[j & 1]);
            }
        }
    } else if (warp == 6) {
        if (lane == 0) {
            for (int j = 0; j < n; ++j) {
                if (!mbar_wait(&p_full[j & 1], (j >> 1) & 1, &s_err)) { atomicExch(&s_err, 1); break; }
                fence_after();
                uint64_t a = desc_mnmajor(smem_u32(ring + size_t(j % kStages) * stage_bytes), kChunk);
                const uint64_t b = desc_kmajor(smem_u32(sP) + uint32_t((j & 1) * N * 128));
                for (int t = 0; t < tiles; ++t, a += (2 * kChunk) >> 4)
#pragma unroll
                    for (int k16 = 0; k16 < kPage / 16; ++k16)
                        umma_ss(t_o + uint32_t(t * N), a + uint64_t(k16 * 2048 >> 4), b + uint64_t(k16 * 2), idesc_a_mn(N), (j > 0 || k16 > 0) ? 1u : 0u);
                umma_commit(&pv_done[j & 1]);
                umma_commit(&empty[j % kStages]);
            }
        }
    } else if (warp >= 2) {
        pdl_wait();   // the results overwrite what an earlier layer's merge reads
        const int quad = warp & 3, tt = tid - 64;
        const uint32_t lane_addr = uint32_t(quad * 32) << 16;
        constexpr int HL = 128 / N, KL = kPage / HL;   // lanes of one head, keys per lane
        const int sh = tt / HL, sl = tt % HL;
        float m_ref = -INFINITY, l_run = 0.f;
        // (a wait that gave up must not leave the loop alone: the four warps meet at barriers)
        for (int j = 0; j < n; ++j) {
            if (!mbar_wait(&s_full[j & 1], (j >> 1) & 1, &s_err)) atomicExch(&s_err, 1);
            fence_after();
            if (quad < 2) {   // the quadrants that hold the page's 64 keys
                uint32_t v[N];
                tmem_ld<N>(tmem + lane_addr + uint32_t((j & 1) * N), v);
                wait_ld();
                fence_before();
                __syncwarp();
                if (lane == 0) mbar_arrive(&s_free[j & 1]);
#pragma unroll
                for (int h = 0; h < N; ++h) sS[h * kSLd + quad * 32 + lane] = __uint_as_float(v[h]);
            }
            softmax_sync();
            const int key0 = (split + j * splits) * kPage;
            float v[KL], mx = -INFINITY;
#pragma unroll
            for (int e = 0; e < KL; e += 4) {
                const float4 x = *reinterpret_cast<const float4*>(sS + sh * kSLd + sl * KL + e);
                v[e] = x.x * scale2; v[e + 1] = x.y * scale2; v[e + 2] = x.z * scale2; v[e + 3] = x.w * scale2;
            }
#pragma unroll
            for (int e = 0; e < KL; ++e) { if (key0 + sl * KL + e > pos) v[e] = -INFINITY; mx = fmaxf(mx, v[e]); }
#pragma unroll
            for (int o = HL / 2; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
            float alpha = 1.f;
            if (j == 0) m_ref = mx;   // a page of the split holds at least one visible key
            else if (mx > m_ref + kLazy) { alpha = exp2f(m_ref - mx); m_ref = mx; }
            if (sl == 0) s_alpha[sh] = alpha;
            // this buffer of probabilities was last read by the product of page j - 2
            if (j >= 2 && !mbar_wait(&pv_done[j & 1], ((j >> 1) - 1) & 1, &s_err)) atomicExch(&s_err, 1);
            float sum = 0.f;
            unsigned char* prow = sP + (j & 1) * (N * 128) + sh * 128;
#pragma unroll
            for (int e = 0; e < KL; e += 8) {
                uint32_t w[4];
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    const float p0 = exp2f(v[e + 2 * i] - m_ref), p1 = exp2f(v[e + 2 * i + 1] - m_ref);
                    sum += p0 + p1;
                    w[i] = pack_bf2(p0, p1);
                }
                const int piece = (sl * KL + e) >> 3;
                *reinterpret_cast<uint4*>(prow + ((piece ^ (sh & 7)) << 4)) = make_uint4(w[0], w[1], w[2], w[3]);
            }
#pragma unroll
            for (int o = HL / 2; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
            l_run = l_run * alpha + sum;
            asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
            if (softmax_sync_or(alpha != 1.f)) {
                // O changes scale: every product issued so far must be complete (the next one waits for this page's probabilities)
                if (!mbar_wait(&pv_done[(j - 1) & 1], ((j - 1) >> 1) & 1, &s_err)) atomicExch(&s_err, 1);
                fence_after();
                for (int t = 0; t < tiles; ++t) {
                    uint32_t o[N];
                    tmem_ld<N>(t_o + lane_addr + uint32_t(t * N), o);
                    wait_ld();
#pragma unroll
                    for (int h = 0; h < N; ++h) o[h] = __float_as_uint(__uint_as_float(o[h]) * s_alpha[h]);
                    tmem_st<N>(t_o + lane_addr + uint32_t(t * N), o);
                }
                wait_st();
                fence_before();
            }
            __syncwarp();
            if (lane == 0) mbar_arrive(&p_full[j & 1]);
        }
        if (n > 0) {
            if (!mbar_wait(&pv_done[(n - 1) & 1], ((n - 1) >> 1) & 1, &s_err)) atomicExch(&s_err, 1);
            fence_after();
            for (int t = 0; t < tiles; ++t) {
                uint32_t o[N];
                tmem_ld<N>(t_o + lane_addr + uint32_t(t * N), o);
                wait_ld();
                const int col = t * 128 + quad * 32 + lane;
                float* dst = part + ((size_t(r) * d.heads + h0) * splits + split) * d.rank_p + col;
                const size_t step = size_t(splits) * d.rank_p;
                const int nh = col < d.rank_p ? min(N, d.heads - h0) : 0;
#pragma unroll
                for (int h = 0; h < N; ++h, dst += step)
                    if (h < nh) *dst = __uint_as_float(o[h]);
            }
            fence_before();
        }
        if (sl == 0 && h0 + sh < d.heads) ml[(size_t(r) * d.heads + h0 + sh) * splits + split] = make_float2(m_ref, l_run);
    }
    __syncthreads();
    if (warp == 1) {
        fence_after();
        tmem_free<COLS>(tmem);
    }
    if (tid == 0 && s_err && err) atomicExch(err, 1);
}

int head_tile(const LatentDims& d) { return d.heads > 16 ? 32 : 16; }
size_t decode_smem(const LatentDims& d, int n) {
    const size_t extra = size_t(d.row() / 64) * n * 128 + size_t(2) * n * 128 + sizeof(float) * n * kSLd;
    return size_t(kStages) * d.row() * 128 + std::max<size_t>(extra, kChunk) + 1024;   // at least a chunk behind the ring: see the header
}

// {64 columns, rows, chunks}: one box brings `box_rows` whole rows as chunks of swizzled 128-byte rows
int32_t chunked_map(CUtensorMap* m, const void* base, const LatentDims& d, uint64_t rows, uint32_t box_rows) {
    const uint32_t nch = uint32_t(d.row() / 64);
    const uint64_t dims[3] = {64, rows, nch}, strides[2] = {uint64_t(d.row()) * 2, 128};
    const uint32_t box[3] = {64, box_rows, nch};
    return make_map(m, base, 3, dims, strides, box);
}

template <int N, uint32_t COLS>
int32_t launch(const LatentDims& d, const void* qabs, const void* map, const StepRows& rows, int splits, float* part, float2* ml, int* err, cudaStream_t st) {
    CUtensorMap m, mq;
    memcpy(&m, map, sizeof(m));
    FORGE_TRY(chunked_map(&mq, qabs, d, uint64_t(rows.n) * d.heads, N));
    auto kern = latent_decode_kernel<N, COLS>;
    const size_t smem = decode_smem(d, N);
    FORGE_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, int(smem)));
    FORGE_CUDA(launch_pdl(kern, dim3(splits, (d.heads + N - 1) / N, rows.n), dim3(kThreads), smem, st, m, mq, d, rows,
                          d.scale * 1.4426950408889634f, part, ml, err));
    FORGE_LAUNCH_CHECK();
    return FORGE_OK;
}

}  // namespace

bool latent_decode_tc_supported(const LatentDims& d) { return decode_smem(d, head_tile(d)) <= 224 * 1024; }
int latent_decode_head_groups(const LatentDims& d) { return (d.heads + head_tile(d) - 1) / head_tile(d); }

int32_t latent_cache_map(void* map_out, const void* cache, const LatentDims& d, size_t rows) {
    CUtensorMap m;
    FORGE_TRY(chunked_map(&m, cache, d, rows, kPage));
    memcpy(map_out, &m, sizeof(m));
    return FORGE_OK;
}

int32_t latent_decode_tc(const LatentDims& d, const void* qabs, const void* map, const StepRows& rows, int splits, float* part, float2* ml, int* err, cudaStream_t st) {
    if (rows.n <= 0) return FORGE_OK;
    if (!latent_decode_tc_supported(d)) { set_error("latent decode: rows of %d values unsupported", d.row()); return FORGE_ERR_SHAPE; }
    const int n = head_tile(d), cols = (2 + (d.rank_p + 127) / 128) * n;
    if (n == 16) return cols <= 128 ? launch<16, 128>(d, qabs, map, rows, splits, part, ml, err, st) : launch<16, 256>(d, qabs, map, rows, splits, part, ml, err, st);
    return cols <= 256 ? launch<32, 256>(d, qabs, map, rows, splits, part, ml, err, st) : launch<32, 512>(d, qabs, map, rows, splits, part, ml, err, st);
}

}  // namespace forge
