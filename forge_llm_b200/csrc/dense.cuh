// Dense (bfloat16 or float32) linear layers: out[token][row] = act[token][K] . W[row][K]^T with an epilogue per row range.
#pragma once

#include <cuda_bf16.h>

#include <vector>

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
    // a view of some columns: K columns from col0 of rows of ld (0: K) columns; col0 and ld are multiples of 64
    int ld = 0, col0 = 0;
    int pitch() const { return ld ? ld : K; }
    // a view of n rows from row `from` (a multiple of 128)
    DenseWeight rows(int from, int n) const {
        DenseWeight v = *this;
        v.N = n;
        if (w) v.w = static_cast<char*>(w) + size_t(from) * pitch() * dense_size(dtype);
        if (tiles) v.tiles = static_cast<char*>(tiles) + size_t(from) * pitch() * 2;
        return v;
    }
    DenseWeight columns(int from, int n) const { DenseWeight v = *this; v.ld = pitch(); v.col0 = col0 + from; v.K = n; return v; }
};

// What becomes of the rows [row0, row0 + rows) of a product.  T: the model's activation type; v: the value, which is the product
// times the token's scale (RowScale) plus add[r].
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
    SEG_DECAY,        // f32 -mul[r] * softplus(v): the logarithm of a decay
    SEG_EXP_DECAY,    // f32 -exp(v): the same
    SEG_RESID         // f32 dst[token * ld + r] (+)= v; then what `after` asks for
};
// What the kernel that finishes a row of the residual stream leaves for its next reader, as T dst[token * ld + r]:
// tanh(alpha * x) * w[r] + b[r] (the Dynamic Tanh norm, which needs no statistics of the row), x itself, or for an RMS norm
// x * w[r] (and for a second one x * w2[r], col2 columns on) and the sums of x^2 over each 32 columns, sums[token * parts + r / 32],
// from which the product that reads it forms the token's scale.
enum AfterKind { AFTER_NONE = 0, AFTER_DYT, AFTER_CAST, AFTER_RMS };
struct After {
    int kind = AFTER_NONE;
    float alpha = 0.f;
    const float* w = nullptr; const float* b = nullptr; const float* w2 = nullptr;
    void* dst = nullptr; int ld = 0, col2 = 0;
    float* sums = nullptr; int parts = 0;
    // first, the entry of a pass of a loop: x += plus[r] + again[token * stride of x + r]; keep: the stream in front of it
    const float* plus = nullptr; const float* again = nullptr;
    float* keep = nullptr;
    bool enters() const { return plus || again; }
};
// a token's products are multiplied with mul / sqrt(sum over parts of sums[row * parts ..] * inv_n + eps); row: row[token] or the token
struct RowScale {
    const float* sums = nullptr; int parts = 0;
    float inv_n = 0.f, eps = 0.f, mul = 1.f;
    const int32_t* row = nullptr;
};
inline int scale_parts(int width) { return pad_to((width + 31) / 32, 4); }   // (the padding stays zero)
constexpr int kScaleRows = 32;   // products of more tokens take one sum per row (row_sums)
struct OutSeg {
    int kind = SEG_F32, row0 = 0, rows = 0, ld = 0;
    void* dst = nullptr;
    int group = 0, group_ld = 0;
    float limit = 0.f;
    const float* mul = nullptr; const float* add = nullptr;   // per row (add: not with gated pairs)
    const int32_t* place = nullptr;   // SEG_CAST: row of dst that token goes to (null: the token's own number)
    // SEG_CAST, blending: what is stored is own * v + other * blend[row of dst * blend_ld + column of dst], blend being T rows
    const void* blend = nullptr; int blend_ld = 0; float own = 1.f, other = 0.f;
    bool fresh = false;               // SEG_RESID: dst is written, not added to
    int act_col = 0;                  // first column of the activations these rows are multiplied with (segments that differ in it start at multiples of 128 rows)
    After after;
};
constexpr int kMaxSegs = 12;
struct DenseOut {
    RowScale scale;
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

// ---- products in groups: a matrix per group of tokens (mixtures of experts)
// A tile of tokens: rows [row0, row0 + rows) of the activations meet the matrix of `group`; w0: where its tokens' weights begin.
struct GroupTile { int32_t group, row0, rows, w0; };
struct GroupTable {
    const GroupTile* tiles = nullptr; const int32_t* n = nullptr;   // device
    int max_tiles = 0;               // host: at most so many
    int tile_rows = 0;               // rows of a tile at most: 16, 32, 64, 128 or 256
    const float* weight = nullptr;   // gated pairs: multiplied with weight[w0 + row in tile]
};
inline int group_tile_rows(int rows_per_group) { return rows_per_group <= 16 ? 16 : rows_per_group <= 32 ? 32 : rows_per_group <= 64 ? 64 : rows_per_group <= 128 ? 128 : 256; }
// `w` holds every group's matrix: group_rows > 0: rows [g * group_rows, + rows) (group_rows a multiple of 128), group_cols > 0: columns
// [g * group_cols, + w.K); rows: of one group.  Outputs of group g go group_dst elements of its segment's type further each.
struct GroupShape { int rows = 0, group_rows = 0, group_cols = 0; size_t group_dst = 0; };
int32_t dense_gemm_groups(const DenseWeight& w, const GroupShape& s, const GroupTable& t, const void* act, int act_ld, int act_rows, const DenseOut& out, int* err, cudaStream_t st);
// One product over the first k_fixed columns and the k_group columns of every group that the table names (of k_fixed + groups * k_group);
// bfloat16, at most 32 tokens.
bool dense_listed_supported(const DenseWeight& w, int m);
int32_t dense_gemm_listed(const DenseWeight& w, int k_fixed, int k_group, const GroupTable& t, const void* act, int act_ld, int m, const DenseOut& out, int* err, cudaStream_t st);

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
    float* x0_f32 = nullptr;          // the same as f32 rows of `width`
    float scale = 1.f;                // of the table's rows
    // a second table, its row (previous token * mul_prev + token * mul_cur) % buckets, `buckets` for a sequence's first token; prev: last token by state slot
    const void* bigram = nullptr; uint32_t buckets = 0, mul_prev = 0, mul_cur = 0;
    const uint32_t* prev = nullptr;
    int32_t* place = nullptr; StepRows rows;
    uint32_t* hist = nullptr; const int32_t* step = nullptr;
};
int32_t embed_rows(const EmbedArgs& a, int dtype, cudaStream_t st);
// prev[slot] = the last token each sequence has in this step
int32_t keep_tokens(uint32_t* prev, const uint32_t* tokens, const StepRows& rows, cudaStream_t st);
// dst[r] = sum of sums[r * parts ..]
int32_t row_sums(float* dst, const float* sums, int rows, int parts, cudaStream_t st);
// dst[i] = src[idx[i]], rows of `cols` elements of the model's type (src's src_ld apart)
int32_t gather_act_rows(void* dst, const void* src, int src_ld, const int32_t* idx, int rows, int cols, int dtype, cudaStream_t st);
// {cos, sin} * factor of p * freq[i]
int32_t rope_table(float* table_host, int n_pos, const std::vector<double>& freq, double factor);

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
// Warp-wide leavings of a stream value x (lane: column 32 * part + lane of row t, ok: there is one); returns what x becomes.  For
// writers whose warps hold 32 neighbouring columns.
template <typename T>
__device__ __forceinline__ float leave_value(const After& a, float x, size_t t, size_t stride, int col, bool ok) {
    if (ok) {
        if (a.keep) a.keep[t * stride + col] = x;
        if (a.plus) x += a.plus[col];
        if (a.again) x += a.again[t * stride + col];
        T* dst = static_cast<T*>(a.dst) + t * a.ld + col;
        if (a.kind == AFTER_DYT) *dst = to_t<T>(dynamic_tanh(x, a.alpha, a.w[col], a.b[col]));
        else if (a.kind == AFTER_CAST) *dst = to_t<T>(x);
        else if (a.kind == AFTER_RMS) { *dst = to_t<T>(x * a.w[col]); if (a.w2) dst[a.col2] = to_t<T>(x * a.w2[col]); }
    }
    if (a.kind == AFTER_RMS) {
        const float s = warp_sum(ok ? x * x : 0.f);
        if ((threadIdx.x & 31) == 0 && ok) a.sums[t * a.parts + col / 32] = s;
    }
    return x;
}
// The same with four neighbouring columns from `col` per lane, eight lanes per part; sizes and strides are multiples of four.
__device__ __forceinline__ void put4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void put4(__nv_bfloat16* p, float4 v) {
    const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
}
__device__ __forceinline__ float4 get4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 get4(const __nv_bfloat16* p) {
    const uint2 u = *reinterpret_cast<const uint2*>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.x)), b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.y));
    return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ float4 add4(float4 a, float4 b) { return make_float4(a.x + b.x, a.y + b.y, a.z + b.z, a.w + b.w); }
__device__ __forceinline__ float4 mul4(float4 a, float4 b) { return make_float4(a.x * b.x, a.y * b.y, a.z * b.z, a.w * b.w); }
template <typename T>
__device__ __forceinline__ float4 leave_four(const After& a, float4 x, size_t t, size_t stride, int col, bool ok) {
    if (ok) {
        if (a.keep) put4(a.keep + t * stride + col, x);
        if (a.plus) x = add4(x, get4(a.plus + col));
        if (a.again) x = add4(x, get4(a.again + t * stride + col));
        T* dst = static_cast<T*>(a.dst) + t * a.ld + col;
        if (a.kind == AFTER_DYT) {
            const float4 w = get4(a.w + col), b = get4(a.b + col);
            put4(dst, make_float4(dynamic_tanh(x.x, a.alpha, w.x, b.x), dynamic_tanh(x.y, a.alpha, w.y, b.y), dynamic_tanh(x.z, a.alpha, w.z, b.z), dynamic_tanh(x.w, a.alpha, w.w, b.w)));
        } else if (a.kind == AFTER_CAST) put4(dst, x);
        else if (a.kind == AFTER_RMS) { put4(dst, mul4(x, get4(a.w + col))); if (a.w2) put4(dst + a.col2, mul4(x, get4(a.w2 + col))); }
    }
    if (a.kind == AFTER_RMS) {
        float s = ok ? fmaf(x.x, x.x, fmaf(x.y, x.y, fmaf(x.z, x.z, x.w * x.w))) : 0.f;
#pragma unroll
        for (int o = 4; o > 0; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
        if ((threadIdx.x & 7) == 0 && ok) a.sums[t * a.parts + col / 32] = s;
    }
    return x;
}
__device__ __forceinline__ size_t cache_row(const StepRows& rows, int r, int pos) {
    const int seq = rows.seq ? rows.seq[r] : r;
    return size_t(rows.page_table[size_t(seq) * rows.pages_per_seq + pos / FORGE_KV_PAGE]) * FORGE_KV_PAGE + pos % FORGE_KV_PAGE;
}
__device__ __forceinline__ int state_slot(const StepRows& rows, int r) { return (rows.seq ? rows.seq[r] : r) + rows.slot0; }
#endif

}  // namespace forge
