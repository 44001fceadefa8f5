// Softmax attention over a paged cache of keys and values, grouped heads, optional cap on the scores, optional chunks (position i
// sees the keys of its own chunk of positions only) or a sliding window with kept first tokens, optional sinks (a learned score per
// head that enters the denominator only); and what stands in front of it: norms and rotation of queries and keys.
#pragma once

#include "dense.cuh"
#include "moe.cuh"

namespace forge {

struct AttnDims {
    int heads = 0, groups = 0, dim = 0, vdim = 0;   // query head h uses key / value head h / (heads / groups)
    int dim_p = 0, vdim_p = 0;                      // padded to 64: a cache row is [groups][dim_p] keys, then [groups][vdim_p] values
    float scale = 1.f, softcap = 0.f;               // softcap > 0: score <- softcap * tanh(score / softcap)
    int chunk = 0;                                  // > 0: key j is visible to i only if j / chunk == i / chunk
    int window = 0, keep = 0;                       // window > 0: key j is visible to i only if i - j < window or j < keep
    __host__ __device__ int row() const { return groups * (dim_p + vdim_p); }
    // position pos sees the keys first_key(pos) .. pos, and the first kept(pos) in front of them
    __host__ __device__ int first_key(int pos) const { return chunk > 0 ? pos / chunk * chunk : window > 0 && pos >= window ? pos - window + 1 : 0; }
    __host__ __device__ int kept(int pos) const { const int lo = first_key(pos); return window > 0 ? (keep < lo ? keep : lo) : 0; }
    int most_keys(int n) const { return chunk > 0 ? (n < chunk ? n : chunk) : window > 0 && (long long)window + keep < n ? window + keep : n; }
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
struct RouteBeside { RouterDims d; const float* logits = nullptr; RouteTables t; };
int32_t qk_post(const AttnDims& d, const QkPost& p, int dtype, const float* proj, int ldp, int k_col, const float* q_norm, const float* k_norm, const float* rope, void* q, void* cache,
                const int32_t* place, const StepRows& rows, const RouteBeside* route, cudaStream_t st);

bool attn_rows_supported(const AttnDims& d);
// q: T rows [heads][dim_p]; out[row][head * vdim + i] = gate[row][head] * attention, T (gate null: ungated).  sink: score per head, or null.
// max_keys: most keys a row sees.
int32_t attn_rows(const AttnDims& d, int dtype, const void* q, const void* cache, const float* gate, const float* sink, void* out, int out_ld, const StepRows& rows, int max_keys, cudaStream_t st);

}  // namespace forge
