// Softmax attention over a paged cache of keys and values, grouped heads, optional cap on the scores and optional chunks (position i
// sees the keys of its own chunk of positions only).
#pragma once

#include "dense.cuh"

namespace forge {

struct AttnDims {
    int heads = 0, groups = 0, dim = 0, vdim = 0;   // query head h uses key / value head h / (heads / groups)
    int dim_p = 0, vdim_p = 0;                      // padded to 64: a cache row is [groups][dim_p] keys, then [groups][vdim_p] values
    float scale = 1.f, softcap = 0.f;               // softcap > 0: score <- softcap * tanh(score / softcap)
    int chunk = 0;                                  // > 0: key j is visible to i only if j / chunk == i / chunk
    __host__ __device__ int row() const { return groups * (dim_p + vdim_p); }
    __host__ __device__ int first_key(int pos) const { return chunk > 0 ? pos / chunk * chunk : 0; }
};

bool attn_rows_supported(const AttnDims& d);
// q: T rows [heads][dim_p]; out[row][head * vdim + i] = gate[row][head] * attention, T.  max_keys: most keys a row sees.
int32_t attn_rows(const AttnDims& d, int dtype, const void* q, const void* cache, const float* gate, void* out, int out_ld, const StepRows& rows, int max_keys, cudaStream_t st);

}  // namespace forge
