// Mixtures of experts: which experts a token uses, and the tables by which the products in groups (dense.cuh) find their tokens.
#pragma once

#include "dense.cuh"

namespace forge {

constexpr int kMaxExperts = 512;

// Choices behind the experts pass a token's input on (identity).  correction (device, null: none): the `top` largest of softmax(logits) +
// correction are chosen and weighted with their softmax over all choices; without it the largest logits, weighted by the softmax over the chosen.
// always: groups of the products in front of the experts that every token uses with weight one (pieces of a shared expert).
struct RouterDims {
    int experts = 0, top = 0, identity = 0, always = 0;
    const float* correction = nullptr;
    __host__ __device__ int choices() const { return experts + identity; }
    __host__ __device__ int groups() const { return always + experts; }
};
// Device tables of one routing.  A pair is (row, k), k = 0 .. top - 1; pairs are dealt to slots expert by expert, in the order of
// rows within an expert.
struct RouteTables {
    int32_t* expert = nullptr; float* weight = nullptr; int32_t* slot = nullptr;   // [rows][top]
    int32_t* row = nullptr; float* slot_weight = nullptr;                          // [rows * top], by slot
    float* row_weight = nullptr;                                                   // few rows: [groups][kScaleRows], zero where the group is not used
    float* passed = nullptr;                                                       // [rows]: weight of the choices that pass the input on
    GroupTile* tiles = nullptr; int32_t* n_tiles = nullptr;
    GroupTile* listed = nullptr; int32_t* n_listed = nullptr;                      // few rows: the experts among them, numbered without the groups in front
};
size_t route_bytes(const RouterDims& d, int rows);
RouteTables route_tables(void* p, const RouterDims& d, int rows);

GroupTable few_table(const RouterDims& d, int rows, const RouteTables& t);   // of route_few
GroupTable listed_table(const RouterDims& d, int rows, const RouteTables& t);   // the same for a listed product whose fixed columns are those of the groups in front
inline size_t route_few_smem(const RouterDims& d) { return size_t(d.groups()) * (kScaleRows + 1) * 4; }
// logits: f32 [rows][choices].
// Few rows (at most kScaleRows): a tile of all rows per expert that any of them uses.
int32_t route_few(const RouterDims& d, const float* logits, int rows, const RouteTables& t, GroupTable* out, cudaStream_t st);
// Any number: tiles of slots.
int32_t route_slots(const RouterDims& d, const float* logits, int rows, const RouteTables& t, GroupTable* out, cudaStream_t st);
// x[r] += sum over k of y[slot(r, k)], f32 rows of `width`, then `after`
int32_t add_experts(float* x, const float* y, const RouterDims& d, const RouteTables& t, int rows, int width, const After& after, int dtype, cudaStream_t st);
// x += gain * y / rms(y), then `after`.  y: f32 rows; with a mixture first y[r] += passed[r] x[r], and with expert outputs e (f32 rows by slot) += those of the
// row's slots.
struct MixtureSum { const float* passed = nullptr; const float* e = nullptr; const int32_t* slot = nullptr; int top = 0; };
// Few rows: the finished rows of the stream are routed, too (route_few's tables): w: T rows [choices][ld]; ticket: one self-resetting word.
struct RouteBehind { RouterDims d; const void* w = nullptr; int ld = 0; RouteTables t; int* ticket = nullptr; };
bool route_behind_supported(const RouterDims& d, int width, int rows);
int32_t add_normed(float* x, const float* y, int rows, int width, float eps, float gain, const MixtureSum& mix, const After& after, const RouteBehind* route, int dtype, cudaStream_t st);

#ifdef __CUDACC__
constexpr int kPerLane = kMaxExperts / 32;

// The warp chooses a row's experts (lower numbers win ties); expert[k] and weight[k] by lane 0.  PER: choices per lane.
template <int PER = kPerLane>
__device__ __forceinline__ void choose(const float* z, const RouterDims& d, int32_t* expert, float* weight) {
    constexpr int kPerLane = PER;
    const int lane = threadIdx.x & 31, experts = d.choices(), top = d.top;
    float v[kPerLane];
    uint32_t taken = 0;
#pragma unroll
    for (int i = 0; i < kPerLane; ++i) v[i] = lane + 32 * i < experts ? z[lane + 32 * i] : 0.f;
    float first = 0.f, sum = 0.f;
    if (d.correction) {
        float mx = -INFINITY;
#pragma unroll
        for (int i = 0; i < kPerLane; ++i) if (lane + 32 * i < experts) mx = fmaxf(mx, v[i]);
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
        float s = 0.f;
#pragma unroll
        for (int i = 0; i < kPerLane; ++i) if (lane + 32 * i < experts) s += v[i] = expf(v[i] - mx);
        s = warp_sum(s);
        first = mx; sum = s;
#pragma unroll
        for (int i = 0; i < kPerLane; ++i) if (lane + 32 * i < experts) v[i] = v[i] / s + d.correction[lane + 32 * i];
    }
    for (int k = 0; k < top; ++k) {
        float best = 0.f;
        int at = -1;
#pragma unroll
        for (int i = 0; i < kPerLane; ++i)
            if (lane + 32 * i < experts && !(taken >> i & 1) && (at < 0 || v[i] > best)) { best = v[i]; at = lane + 32 * i; }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            const float other = __shfl_xor_sync(0xffffffffu, best, o);
            const int whose = __shfl_xor_sync(0xffffffffu, at, o);
            if (whose >= 0 && (at < 0 || other > best || (other == best && whose < at))) { best = other; at = whose; }
        }
        at = __shfl_sync(0xffffffffu, at, 0);      // (values that are no numbers compare differently in different lanes)
        best = __shfl_sync(0xffffffffu, best, 0);
        if ((at & 31) == lane) taken |= 1u << (at >> 5);
        if (d.correction) { if (lane == 0) { expert[k] = at; weight[k] = expf(z[at] - first) / sum; } continue; }
        if (k == 0) first = best;
        const float e = expf(best - first);
        sum += e;
        if (lane == 0) { expert[k] = at; weight[k] = e; }
    }
    if (lane == 0 && !d.correction) for (int k = 0; k < top; ++k) weight[k] /= sum;
    __syncwarp();
}

// Routing of few rows by one CTA of whole warps; s_w: route_few_smem(d) bytes, cleared before.  (Also run by a kernel that stands beside it in a step.)
__device__ __forceinline__ void route_few_clear(const RouterDims& d, float* s_w) {
    for (int i = threadIdx.x; i < d.groups() * (kScaleRows + 1); i += blockDim.x) s_w[i] = 0.f;
    __syncthreads();
}
// the tables of rows whose choices lie in expert and weight, [rows][top]
__device__ __forceinline__ void route_few_tables(const RouterDims& d, int rows, const RouteTables& t, const int32_t* expert, const float* weight, float* s_w) {
    const int G = d.groups();
    int* used = reinterpret_cast<int*>(s_w + G * kScaleRows);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    for (int i = threadIdx.x; i < d.always * kScaleRows; i += blockDim.x) {
        s_w[i] = 1.f;
        if (i % kScaleRows == 0) used[i / kScaleRows] = 1;
    }
    for (int r = threadIdx.x; r < rows; r += blockDim.x) {
        float passed = 0.f;
#pragma unroll 4
        for (int k = 0; k < d.top; ++k) {
            const int e = expert[r * d.top + k];
            const float w = weight[r * d.top + k];
            if (e >= d.experts) { passed += w; continue; }
            s_w[(d.always + e) * kScaleRows + r] = w;
            used[d.always + e] = 1;
        }
        t.passed[r] = passed;
    }
    __syncthreads();
    for (int i = threadIdx.x; i < G * kScaleRows; i += blockDim.x) t.row_weight[i] = s_w[i];
    if (warp == 0) {
        int n = 0;
        for (int g0 = 0; g0 < G; g0 += 32) {
            const int g = g0 + lane;
            const bool on = g < G && used[g];
            const uint32_t mask = __ballot_sync(0xffffffffu, on);
            const int at = n + __popc(mask & ((1u << lane) - 1));
            if (on) t.tiles[at] = GroupTile{g, 0, rows, g * kScaleRows};
            if (on && g >= d.always) t.listed[at - d.always] = GroupTile{g - d.always, 0, rows, g * kScaleRows};
            n += __popc(mask);
        }
        if (lane == 0) { *t.n_tiles = n; *t.n_listed = n - d.always; }
    }
}
__device__ __forceinline__ void route_few_rows(const RouterDims& d, const float* logits, int rows, const RouteTables& t, float* s_w) {
    for (int r = threadIdx.x >> 5; r < rows; r += blockDim.x / 32) choose(logits + size_t(r) * d.choices(), d, t.expert + r * d.top, t.weight + r * d.top);
    __threadfence_block();
    __syncthreads();
    route_few_tables(d, rows, t, t.expert, t.weight, s_w);
}
#endif

}  // namespace forge
