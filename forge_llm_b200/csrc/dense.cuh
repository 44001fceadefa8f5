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

// What becomes of the rows [row0, row0 + rows) of a product.  T: the model's activation type.
enum SegKind {
    SEG_F32 = 0,      // f32 dst[token * ld + r]
    SEG_CAST,         // T   dst[token * ld + (r / group) * group_ld + r % group]   (group = 0: dst[token * ld + r])
    SEG_SIGMOID,      // T   dst[token * ld + r] = sigmoid
    SEG_CLAMPED_GLU,  // rows 2j = gate_j, 2j + 1 = up_j: T dst[token * ld + j] = g sigmoid(1.702 g) (u + 1) with
                      // g = min(gate, limit), u = clamp(up, -limit, limit)
    SEG_RESID         // f32 dst[token * ld + r] += value; then, if `next` is set, T next[token * next_ld + r] =
                      // tanh(alpha * dst) * norm_w[r] + norm_b[r], the Dynamic Tanh norm of whatever reads the stream next
};
struct OutSeg {
    int kind = SEG_F32, row0 = 0, rows = 0, ld = 0;
    void* dst = nullptr;
    int group = 0, group_ld = 0;
    float limit = 0.f, alpha = 0.f;
    const float* norm_w = nullptr; const float* norm_b = nullptr;
    void* next = nullptr; int next_ld = 0;
};
constexpr int kMaxSegs = 6;
struct DenseOut { int nseg = 0; OutSeg seg[kMaxSegs]; };

// partial tiles of products whose K steps are dealt to several CTAs, and one self-resetting ticket per output tile
struct DenseScratch { float* part = nullptr; int* tickets = nullptr; size_t tickets_cap = 0; };
constexpr size_t kDensePartFloats = size_t(148) * 2 * 256 * 128;

inline size_t dense_tile_bytes(int N, int K) { return size_t((N + 127) / 128) * 128 * K * 2; }
void dense_tile_image(void* dst, const void* rows, int N, int K);
// act: [m][w.K] of the model's type (rows w.K apart unless act_ld says otherwise).  max_rows: rows the buffer holds.
int32_t dense_gemm(const DenseWeight& w, const void* act, int act_ld, int m, const DenseOut& out, const DenseScratch& sc, int* err, cudaStream_t st);

// ---- row-wise operators (elementwise.cu)
// x[r] = table[tokens[r]] as f32; h[r] = Dynamic Tanh of x[r] as T (rows h_ld apart, padding written as zero)
int32_t embed_dyt(float* x, void* h, int h_ld, const void* table, int dtype, const uint32_t* tokens, int rows, int width, float alpha,
                  const float* w, const float* b, uint32_t* hist, const int32_t* step, cudaStream_t st);
// dst[i] = src[idx[i]], rows of ld elements of the model's type
int32_t gather_act_rows(void* dst, const void* src, const int32_t* idx, int rows, int ld, int dtype, cudaStream_t st);
int32_t rope_half_table(float* table_host, int n_pos, int dims, double base);

}  // namespace forge
