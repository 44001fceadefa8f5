// Softmax attention over a paged cache of keys and values, grouped heads, optional cap on the scores, optional chunks (position i
// sees the keys of its own chunk of positions only) or a sliding window, in front of which first tokens are kept or blocks of tokens are
// seen as the mean of their keys and values, optional learned biases by distance, optional sinks (a learned score per head that enters
// the denominator only), optional mixing of the heads' weights; and what stands in front of it: norms and rotation of queries and keys.
#pragma once

#include "dense.cuh"
#include "moe.cuh"
#include "selective.cuh"

namespace forge {

struct AttnDims {
    int heads = 0, groups = 0, dim = 0, vdim = 0;   // query head h uses key / value head h / (heads / groups)
    int dim_p = 0, vdim_p = 0;                      // padded to 64: a cache row is [groups][dim_p] keys, then [groups][vdim_p] values
    float scale = 1.f, softcap = 0.f;               // softcap > 0: score <- softcap * tanh(score / softcap)
    int chunk = 0;                                  // > 0: key j is visible to i only if j / chunk == i / chunk
    int window = 0, keep = 0;                       // window > 0: key j is visible to i only if i - j < window or j < keep
    // pool > 0 (keep is 0): of the blocks of `pool` tokens those that lie wholly in front of the window are seen, a block as one key and value.  A block's
    // row belongs to the page of its first token; these rows follow those of the pages, from cache row pool_row0.
    int pool = 0, pool_row0 = 0;
    int bias_n = 0;                                 // > 0: scores get bias[head][min(i - j, bias_n - 1)]
    __host__ __device__ int row() const { return groups * (dim_p + vdim_p); }
    __host__ __device__ int pool_slots() const { return pool > 0 ? (FORGE_KV_PAGE + pool - 1) / pool : 0; }   // block rows of a page
    __host__ __device__ int blocks(int pos) const { return pool > 0 ? first_key(pos) / pool : 0; }
    // cache row of block b; pt: the sequence's pages
    __device__ size_t block_row(const int32_t* pt, int b) const {
        const int page = b * pool / FORGE_KV_PAGE, first = (page * FORGE_KV_PAGE + pool - 1) / pool;
        return size_t(pool_row0) + size_t(pt[page]) * pool_slots() + (b - first);
    }
    // The keys that a position sees are numbered: `front` blocks or kept tokens, then the tokens from `lo` on.
    __host__ __device__ int front(int pos) const { return pool > 0 ? blocks(pos) : kept(pos); }
    __device__ size_t key_row(const int32_t* pt, int i, int front, int lo) const {
        if (pool > 0 && i < front) return block_row(pt, i);
        const int key = i < front ? i : lo + i - front;
        return size_t(pt[key / FORGE_KV_PAGE]) * FORGE_KV_PAGE + key % FORGE_KV_PAGE;
    }
    // position pos sees the keys first_key(pos) .. pos, and the first kept(pos) in front of them
    __host__ __device__ int first_key(int pos) const { return chunk > 0 ? pos / chunk * chunk : window > 0 && pos >= window ? pos - window + 1 : 0; }
    __host__ __device__ int kept(int pos) const { const int lo = first_key(pos); return window > 0 ? (keep < lo ? keep : lo) : 0; }
    int most_keys(int n) const { return chunk > 0 ? (n < chunk ? n : chunk) : window > 0 && (long long)window + keep + (pool > 0 ? n / pool : 0) < n ? window + keep + (pool > 0 ? n / pool : 0) : n; }
};

// Queries and keys of a step's rows: rms norm (per head, or over all heads at once), rotary positions on the first rot_dims dimensions,
// queries to q, keys to the cache.
struct QkPost {
    enum Scope { PER_HEAD, WHOLE } norm = PER_HEAD;
    bool interleaved = false;                       // dimension 2 i turns with 2 i + 1; else i with i + rot_dims / 2
    int rot_dims = 0;
    float eps = 0.f;
};
// proj: f32 rows [q of all heads | ... | k of all groups from k_col | ...] of ldp floats; rope: {cos, sin} by position and pair; place: cache row of each row
// route (may be null): a routing of the step's rows (route_few) done by one more CTA of the launch
// conv (may be null): the convolution of single tokens of a scan beside the attention, by further CTAs
struct RouteBeside { RouterDims d; const float* logits = nullptr; RouteTables t; };
struct ConvBeside { SelectiveDims d; SelectiveArgs a; int blocks = 0; };
int32_t qk_post(const AttnDims& d, const QkPost& p, int dtype, const float* proj, int ldp, int k_col, const float* q_norm, const float* k_norm, const float* rope, void* q, void* cache,
                const int32_t* place, const StepRows& rows, const RouteBeside* route, const ConvBeside* conv, cudaStream_t st);

bool attn_rows_supported(const AttnDims& d);
// q: T rows [heads][dim_p]; out[row][head * vdim + i] = gate[row][head] * attention, T (gate null: ungated).  sink: score per head, or null.
// bias: f32 [heads][bias_n], or null.  max_keys: most keys a row sees.
int32_t attn_rows(const AttnDims& d, int dtype, const void* q, const void* cache, const float* gate, const float* sink, const float* bias, void* out, int out_ld, const StepRows& rows, int max_keys,
                  cudaStream_t st);

// ---- blocks seen as one key (attn_pool.cu)
// The means of the blocks that the step's rows complete.
#ifdef __CUDACC__
// columns of the block that position pos completes, if it does: `pieces` pieces of eight from `col`, piece i by thread i
template <typename T>
__device__ __forceinline__ void pool_columns(const AttnDims& d, T* cache, const int32_t* pt, int pos, int col, int pieces) {
    if ((pos + 1) % d.pool || int(threadIdx.x) >= pieces) return;
    const int b = pos / d.pool, c = col + int(threadIdx.x) * 8;
    const size_t W = d.row();
    float sum[8];
#pragma unroll
    for (int e = 0; e < 8; ++e) sum[e] = 0.f;
#pragma unroll 16
    for (int t = b * d.pool; t <= pos; ++t) {
        float v[8];
        load8(v, cache + (size_t(pt[t / FORGE_KV_PAGE]) * FORGE_KV_PAGE + t % FORGE_KV_PAGE) * W + c);
#pragma unroll
        for (int e = 0; e < 8; ++e) sum[e] += v[e];
    }
    const float inv = 1.0f / float(d.pool);
    T* dst = cache + d.block_row(pt, b) * W + c;
    put4(dst, make_float4(sum[0] * inv, sum[1] * inv, sum[2] * inv, sum[3] * inv));
    put4(dst + 4, make_float4(sum[4] * inv, sum[5] * inv, sum[6] * inv, sum[7] * inv));
}
#endif
int32_t pool_blocks(const AttnDims& d, int dtype, void* cache, const StepRows& rows, cudaStream_t st);
// For prompts: block rows of sequences in a row, 64 per table entry.  dst: rows like the cache's.
struct PoolChunk { int32_t pages0, block0, len, unused; };   // first entry of the sequence in `pages`, first block, positions of the sequence
int32_t gather_blocks(const AttnDims& d, int dtype, void* dst, const void* cache, const int32_t* pages, const PoolChunk* chunks, int n_chunks, cudaStream_t st);

// ---- mixed heads (attn_talk.cu): the weight of head h becomes the sum over heads g of talk[h][g] times the weight of g
bool talk_rows_supported(const AttnDims& d);
size_t talk_rows_bytes(const AttnDims& d, int rows, int max_keys);
// out[row][head * vdim + i] = factor * attention, T; scratch: talk_rows_bytes of at most max_bytes (more rows go in turn).  pools: the rows' sequences have one row
// each, and the blocks that they complete (which nobody sees yet) are formed here.
int32_t talk_rows(const AttnDims& d, int dtype, const void* q, void* cache, bool pools, const float* talk, float factor, void* scratch, size_t max_bytes, void* out, int out_ld, const StepRows& rows, int max_keys,
                  cudaStream_t st);
// out[row][h * vdim + i] = factor * sum over g of talk[h][g] o[row][g][group of h][i]: o bf16 [rows][heads][groups][vdim_p], every head's weights on all groups' values
int32_t talk_heads(const AttnDims& d, const void* o, const float* talk, float factor, void* out, int out_ld, int rows, cudaStream_t st);

}  // namespace forge
