// Recurrent mixers: per head a state S [dim][vdim] in f32 that every token decays, extends and reads.
//   delta rule     S <- diag(g) S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q
//   time mixing    o = S^T q + (sum_c q_c bonus_c k_c) v;  S <- diag(g) S + k v^T
//   linear         S <- diag(g) S + k v^T;  o = S^T q
// g is one decay per head or one per head and key channel, given by its logarithm.  The delta rule's q, k, v come from a short
// causal convolution per channel with silu behind it, q and k as unit vectors; its last inputs are kept in a ring of `taps` rows,
// the input of position p in row p % taps.  A sequence's state counts as zero when its first row of a step is at position 0, so
// a slot that is used again needs no clearing.
#pragma once

#include "dense.cuh"

namespace forge {

enum class Rule { TimeMix, Delta, Linear };
struct RecurDims {
    int heads = 0, groups = 0, dim = 0, vdim = 0;   // groups: heads of q and k (head h uses h / (heads / groups))
    int taps = 0;                                   // 0: no convolution
    Rule rule = Rule::TimeMix;
    bool channel = false;                           // a decay per key channel
    float eps = 0.f, q_scale = 1.f;
    __host__ __device__ int qk() const { return groups * dim; }
    __host__ __device__ int channels() const { return 2 * groups * dim + heads * vdim; }
    size_t state_values() const { return size_t(heads) * dim * vdim; }
    __host__ __device__ size_t ring_values() const { return size_t(taps) * channels(); }
};

constexpr int kRecurChunk = 64;     // tokens of a chunk (recurrent_chunk.cu)
constexpr int kChunkedRows = 16;    // segments of fewer tokens go token by token
// consecutive rows of one sequence: rows [row0, row0 + n) of the step at positions pos0, pos0 + 1, ... of state slot `slot`; chunk0: number
// of its first chunk among all chunks of the step (segments of at least kChunkedRows)
struct ScanSeg { int32_t row0, n, slot, pos0, chunk0, unused[3]; };
// a step's segments (device table), the n_short short ones first; together they are the rows [row0, row0 + rows)
struct SegTable { const ScanSeg* segs = nullptr; int n = 0, n_short = 0, max_n = 0, n_chunks = 0, row0 = 0, rows = 0; };

struct RecurArgs {
    const void* x = nullptr; int x_ld = 0;               // T rows [q | k | v]: in front of the convolution, if there is one
    const float* decay = nullptr; int decay_ld = 0;      // logarithms, [row][heads] or [row][heads * dim]
    const float* beta = nullptr;                         // [row][heads]
    const float* bonus = nullptr;                        // [heads][dim]
    const float* conv = nullptr; void* ring = nullptr;   // [taps][channels]; T [slot][taps][channels]
    float* state = nullptr;                              // [slot][heads][dim][vdim]
    // second step of two-step decays and gates, for single tokens (then decay, and gate if gate_w is set, are not read): T rows of low_k values per
    // key channel and per value over the inner values low[row], the gate's from column gate_col; a decay's logarithm is
    // -mul softplus(z + add), for time mixing -exp(z + add)
    const void* decay_w = nullptr; const void* gate_w = nullptr; const void* low = nullptr;
    int low_ld = 0, low_k = 0, gate_col = 0;
    const float* decay_mul = nullptr; const float* decay_add = nullptr;
    const float* norm = nullptr; int norm_head = 0;      // weight of the output's norm, and its step per head
    const void* gate = nullptr; int gate_ld = 0;         // T rows [heads * vdim]
    void* out = nullptr; int out_ld = 0;                 // T rows [heads * vdim]: rms norm(o) * norm * gate
};

// per chunk and head, see recurrent_chunk.cu
struct ChunkScratch { __nv_bfloat16* half = nullptr; float* f32 = nullptr; };
struct ChunkBytes { size_t half, f32; };   // of one chunk, all heads
// scratch of a step with segments
struct RecurScratch {
    void* conv = nullptr;         // T [rows][channels]: behind convolution and silu
    float* unit = nullptr;        // [rows][2 * groups]: what q and k are multiplied with to be unit vectors (q: times q_scale)
    float* o = nullptr;           // [rows][heads * vdim]
    ChunkScratch chunk;
    int* err = nullptr;           // set when a bounded wait gave up
};

bool recur_supported(const RecurDims& d);
// single tokens: row r of `rows` is one token of its sequence
int32_t recur_decode(const RecurDims& d, int dtype, const RecurArgs& a, const StepRows& rows, cudaStream_t st);
// segments of any length
int32_t recur_segments(const RecurDims& d, int dtype, const RecurArgs& a, const RecurScratch& sc, const SegTable& t, cudaStream_t st);
// the walk of the long segments by chunks (bfloat16; called by recur_segments): leaves o and the state
bool recur_chunked_supported(const RecurDims& d);
ChunkBytes recur_chunk_bytes(const RecurDims& d);
int32_t recur_chunked(const RecurDims& d, const RecurArgs& a, const RecurScratch& sc, const ScanSeg* segs, int n_segs, int n_chunks, cudaStream_t st);

// Token shift: dst rows get, next to h in columns [0, width_p), `n_mix` blocks of width_p columns h + (h' - h) mu[i], h' being the
// sequence's row before (prev [slot][width], zeros at position 0).  h lies in dst's first block already.  prev is left at the
// sequence's last row.
int32_t token_shift(void* dst, int ld, int width, int width_p, int n_mix, const float* mu, void* prev, int dtype, const StepRows& rows, int n_single, const SegTable& t, cudaStream_t st);

// x += (rms norm(a) wa + rms norm(b) wb) / 2 over rows of `width` values, then `after`; ab: f32 rows [a | b]
int32_t add_normed_pair(float* x, const float* ab, int rows, int width, float eps, const float* wa, const float* wb, const After& after, int dtype, cudaStream_t st);

}  // namespace forge
