// Latent attention: per token the cache holds one normed latent c (kv_rank values) and one rotated key part shared by all
// heads (rot_dim values); keys and values of the heads are linear in c.
#pragma once

#include "dense.cuh"

namespace forge {

struct LatentDims {
    int heads = 0, dim = 0, rot = 0, vdim = 0, rank = 0;
    int rot_dims = 0;              // rotated dimensions (<= rot)
    int rank_p = 0, rot_p = 0;     // padded to 64: a cache row is [c | zeros | rotated key | zeros], rank_p + rot_p values
    int dim_p = 0, vdim_p = 0;     // padded to 64: rows of the expanded keys and values of a prompt
    float scale = 1.f, eps = 0.f;
    __host__ __device__ int row() const { return rank_p + rot_p; }
};

// proj: f32 rows [q | ... | dkv | ...] of ldp floats; q at column 0, W_dkv h at column dkv_col.
// The latent is normed, the key part rotated, and both are appended to the cache; the queries are rotated and carried into
// the latent space, qabs[row][head] = [W_uk^T q_unrotated | zeros | q_rotated | zeros] as T.
int32_t latent_post(const LatentDims& d, int dtype, const float* proj, int ldp, int dkv_col, const float* kv_norm, const float* rope, const void* uk, int uk_ld,
                    void* qabs, void* cache, const StepRows& rows, cudaStream_t st);
// Prompt rows: the same append, and the rotated queries as bf16 q[row][head] = [unrotated | zeros | rotated | zeros]
// (dim_p + rot_p values).
int32_t latent_post_prompt(const LatentDims& d, const float* proj, int ldp, int dkv_col, const float* kv_norm, const float* rope, void* q,
                           void* cache, const StepRows& rows, cudaStream_t st);
// Attention of single rows over the latent cache: unnormalised sums part[row][head][split][rank_p] and ml[row][head][split] =
// {maximum, sum} in the base-2 domain; split s owns the pages s, s + splits, ...
int32_t latent_attn_rows(const LatentDims& d, int dtype, const void* qabs, const void* cache, const StepRows& rows, int splits, float* part, float2* ml, cudaStream_t st);
// the same on the tensor cores (bfloat16); map: tensor map of the layer's cache rows, see latent_cache_map
bool latent_decode_tc_supported(const LatentDims& d);
int latent_decode_head_groups(const LatentDims& d);   // CTAs per row and split
int32_t latent_cache_map(void* map_out, const void* cache, const LatentDims& d, size_t rows);
int32_t latent_decode_tc(const LatentDims& d, const void* qabs, const void* map, const StepRows& rows, int splits, float* part, float2* ml, int* err, cudaStream_t st);
// out[row][head * vdim + v] = gate * (W_uv (sum of the splits)) as T
int32_t latent_value(const LatentDims& d, int dtype, const float* part, const float2* ml, int splits, const void* uv, int uv_ld, const void* gate, int gate_ld,
                     void* out, int out_ld, const StepRows& rows, cudaStream_t st);

// ---- prompts (bfloat16): keys and values of the heads are formed once per prompt portion, then a tcgen05 flash attention (attn_prompt.cuh)
// c[r] = latents of context row r, krot[r] = its rotated key part (rows gathered through page list `pages`)
int32_t latent_gather_context(const LatentDims& d, const void* cache, const int32_t* pages, int rows, void* c, void* krot, cudaStream_t st);

}  // namespace forge
