// Dense (bfloat16 or float32) linear layers: out[token][row] = act[token][K] . W[row][K]^T with an epilogue per row range.
#pragma once

#include <cuda_bf16.h>

#include "common.cuh"

namespace forge {

// A model runs either in bfloat16 (weights, activations and cache; f32 accumulation, residual, norms and scores) or in
// float32 throughout.
inline size_t dense_size(int dtype) { return dtype == FORGE_BF16 ? 2 : 4; }

constexpr int kDensePad = 64;    // K and activation rows are padded to whole 128-byte bf16 swizzle rows
constexpr int kSegAlign = 32;    // output segments start at multiples of a warp's rows
inline int pad_to(int x, int a) { return (x + a - 1) / a * a; }

struct DenseWeight {
    void* w = nullptr;           // [N][K] of the model's type, padding columns and rows are zero (f32 products, and where a kernel reads rows)
    void* tiles = nullptr;       // bf16: the same matrix as dense_tile_image
    int N = 0, K = 0;            // K: padded
    int dtype = FORGE_BF16;
};

// What becomes of the rows [row0, row0 + rows) of a product.  T: the model's activation type; v: the value.
enum SegKind {
    SEG_F32 = 0,      // f32 dst[token * ld + r]
    SEG_CAST,         // T   dst[token * ld + (r / group) * group_ld + r % group]   (group = 0: dst[token * ld + r])
    SEG_SIGMOID,      // T   dst[token * ld + r] = sigmoid
    SEG_CLAMPED_GLU,  // rows 2j = gate_j, 2j + 1 = up_j: T dst[token * ld + j] = g sigmoid(1.702 g) (u + 1) with
                      // g = min(gate, limit), u = clamp(up, -limit, limit)
    SEG_SILU_GLU,     // the same rows: T dst[token * ld + j] = silu(gate) * up
    SEG_SILU,         // T   silu(v)
    SEG_TANH,         // T   tanh(v)
    SEG_SIGMOID_F32,  // f32 sigmoid(v)
    SEG_DECAY,        // f32 -mul[r] * softplus(v + add[r]): the logarithm of a decay
    SEG_EXP_DECAY,    // f32 -exp(v + add[r]): the same
    SEG_RESID         // f32 dst[token * ld + r] (+)= value + add[r]; then what `after` asks for
};
// What the epilogue that finishes a row of the residual stream leaves for its next reader, as T dst[token * ld + r]:
// tanh(alpha * x) * w[r] + b[r] (the Dynamic Tanh norm, which needs no statistics of the row), or x itself.
enum AfterKind { AFTER_NONE = 0, AFTER_DYT, AFTER_CAST };
struct After {
    int kind = AFTER_NONE;
    float alpha = 0.f;
    const float* w = nullptr; const float* b = nullptr;
    void* dst = nullptr; int ld = 0;
};
struct OutSeg {
    int kind = SEG_F32, row0 = 0, rows = 0, ld = 0;
    void* dst = nullptr;
    int group = 0, group_ld = 0;
    float limit = 0.f;
    const float* mul = nullptr; const float* add = nullptr;   // per row
    const int32_t* place = nullptr;   // SEG_CAST: row of dst that token goes to (null: the token's own number)
    bool fresh = false;               // SEG_RESID: dst is written, not added to
    int act_col = 0;                  // first column of the activations these rows are multiplied with (segments that differ in it start at multiples of 128 rows)
    After after;
};
constexpr int kMaxSegs = 12;
struct DenseOut {
    int nseg = 0; OutSeg seg[kMaxSegs];
    OutSeg& add(int kind, int row0, int rows, void* dst, int ld) { OutSeg& g = seg[nseg++]; g.kind = kind; g.row0 = row0; g.rows = rows; g.dst = dst; g.ld = ld; return g; }
};

// partial tiles of products whose K steps are dealt to several CTAs, and one self-resetting ticket per output tile
struct DenseScratch { float* part = nullptr; int* tickets = nullptr; size_t tickets_cap = 0; };
constexpr size_t kDensePartFloats = size_t(148) * 2 * 256 * 128;

inline size_t dense_tile_bytes(int N, int K) { return size_t((N + 127) / 128) * 128 * K * 2; }
void dense_tile_image(void* dst, const void* rows, int N, int K);
// act: [m][w.K] of the model's type, rows act_ld values apart.
int32_t dense_gemm(const DenseWeight& w, const void* act, int act_ld, int m, const DenseOut& out, const DenseScratch& sc, int* err, cudaStream_t st);

// Rows of a step and where their sequence lives.  Row r belongs to sequence seq[r] (null: sequence r) at position pos[r].
struct StepRows {
    int n = 0;
    const int32_t* pos = nullptr; const int32_t* seq = nullptr;   // device
    const int32_t* page_table = nullptr; int pages_per_seq = 0;
    int fresh = 1;                 // most rows one sequence has in this step
    int slot0 = 0;                 // added to a row's sequence where its recurrent state is addressed
};

// ---- row-wise operators (elementwise.cu)
// x[r] = table[tokens[r]] as f32, its `after` (padding columns written as zero) and, if given, a copy x0[r] as T; place[r] = the
// cache row of the row's position
struct EmbedArgs {
    float* x = nullptr; const void* table = nullptr; const uint32_t* tokens = nullptr;
    int width = 0, width_p = 0;
    After after;
    void* x0 = nullptr; int x0_ld = 0;
    int32_t* place = nullptr; StepRows rows;
    uint32_t* hist = nullptr; const int32_t* step = nullptr;
};
int32_t embed_rows(const EmbedArgs& a, int dtype, cudaStream_t st);
// dst[i] = src[idx[i]], rows of ld elements of the model's type
int32_t gather_act_rows(void* dst, const void* src, const int32_t* idx, int rows, int ld, int dtype, cudaStream_t st);
int32_t rope_half_table(float* table_host, int n_pos, int dims, double base);

#ifdef __CUDACC__
// ---- shared by the kernels of the layer-list models
template <typename T> __device__ __forceinline__ T to_t(float v);
template <> __device__ __forceinline__ float to_t<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 to_t<__nv_bfloat16>(float v) { return __float2bfloat16_rn(v); }
__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(__nv_bfloat16 v) { return __bfloat162float(v); }
// eight consecutive values
__device__ __forceinline__ void load8(float (&v)[8], const float* p) {
    const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
    v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
}
__device__ __forceinline__ void load8(float (&v)[8], const __nv_bfloat16* p) {
    const uint4 u = *reinterpret_cast<const uint4*>(p);
    const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&u);
#pragma unroll
    for (int i = 0; i < 4; ++i) { const float2 f = __bfloat1622float2(h[i]); v[2 * i] = f.x; v[2 * i + 1] = f.y; }
}
__device__ __forceinline__ float sigmoid(float v) { return 1.0f / (1.0f + expf(-v)); }
__device__ __forceinline__ float silu(float v) { return v / (1.0f + expf(-v)); }
__device__ __forceinline__ float softplus(float v) { return fmaxf(v, 0.f) + log1pf(expf(-fabsf(v))); }
__device__ __forceinline__ float dynamic_tanh(float x, float alpha, float w, float b) { return tanhf(alpha * x) * w + b; }
__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}
__device__ __forceinline__ size_t cache_row(const StepRows& rows, int r, int pos) {
    const int seq = rows.seq ? rows.seq[r] : r;
    return size_t(rows.page_table[size_t(seq) * rows.pages_per_seq + pos / FORGE_KV_PAGE]) * FORGE_KV_PAGE + pos % FORGE_KV_PAGE;
}
__device__ __forceinline__ int state_slot(const StepRows& rows, int r) { return (rows.seq ? rows.seq[r] : r) + rows.slot0; }
#endif

}  // namespace forge
