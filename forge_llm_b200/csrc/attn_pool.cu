// Blocks of tokens seen as one key and value: the mean of the rows that the cache holds of them, formed when the last of them is written.
#include "attn_rows.cuh"

namespace forge {

namespace {

// A CTA per eight rows of the step; eight columns per thread.
constexpr int kPoolRows = 8;
template <typename T>
__global__ void __launch_bounds__(128) pool_blocks_kernel(const AttnDims d, T* cache, const StepRows rows) {
    pdl_trigger();
    pdl_wait();
    const int r0 = blockIdx.x * kPoolRows;
    int at[kPoolRows];
#pragma unroll
    for (int i = 0; i < kPoolRows; ++i) at[i] = r0 + i < rows.n ? rows.pos[r0 + i] : 0;
#pragma unroll
    for (int i = 0; i < kPoolRows; ++i) {
        const int r = r0 + i, pos = at[i];
        if (r >= rows.n || (pos + 1) % d.pool) continue;
        const int seq = rows.seq ? rows.seq[r] : r;
        const int32_t* pt = rows.page_table + size_t(seq) * rows.pages_per_seq;
        for (int c = 0; c < d.row(); c += 128 * 8) pool_columns(d, cache, pt, pos, c, min(128, (d.row() - c) / 8));
    }
}

// Rows that are no block yet become zeros: their weights are zero, so they must be finite.
__global__ void __launch_bounds__(128) gather_blocks_kernel(const AttnDims d, int pieces, uint4* __restrict__ dst, const uint4* __restrict__ cache, const int32_t* __restrict__ pages, const PoolChunk* __restrict__ chunks) {
    const PoolChunk ch = chunks[blockIdx.x];
    const int n = ch.len / d.pool;
    for (int i = blockIdx.y; i < FORGE_KV_PAGE; i += gridDim.y) {
        const int b = ch.block0 + i;
        const uint4* src = b < n ? cache + d.block_row(pages + ch.pages0, b) * pieces : nullptr;
        uint4* to = dst + (size_t(blockIdx.x) * FORGE_KV_PAGE + i) * pieces;
        for (int p = threadIdx.x; p < pieces; p += 128) to[p] = src ? src[p] : make_uint4(0, 0, 0, 0);
    }
}

}  // namespace

int32_t pool_blocks(const AttnDims& d, int dtype, void* cache, const StepRows& rows, cudaStream_t st) {
    if (rows.n <= 0) return FORGE_OK;
    if (dtype == FORGE_F32) FORGE_CUDA(launch_pdl(pool_blocks_kernel<float>, dim3((rows.n + kPoolRows - 1) / kPoolRows), dim3(128), 0, st, d, static_cast<float*>(cache), rows));
    else FORGE_CUDA(launch_pdl(pool_blocks_kernel<__nv_bfloat16>, dim3((rows.n + kPoolRows - 1) / kPoolRows), dim3(128), 0, st, d, static_cast<__nv_bfloat16*>(cache), rows));
    FORGE_LAUNCH_CHECK();
    return FORGE_OK;
}

int32_t gather_blocks(const AttnDims& d, int dtype, void* dst, const void* cache, const int32_t* pages, const PoolChunk* chunks, int n_chunks, cudaStream_t st) {
    if (n_chunks <= 0) return FORGE_OK;
    const int pieces = int(size_t(d.row()) * dense_size(dtype) / 16);
    gather_blocks_kernel<<<dim3(n_chunks, 16), 128, 0, st>>>(d, pieces, static_cast<uint4*>(dst), static_cast<const uint4*>(cache), pages, chunks);
    FORGE_LAUNCH_CHECK();
    return FORGE_OK;
}

}  // namespace forge
