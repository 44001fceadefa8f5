// Mixtures of experts: which experts a token uses, and the tables by which the products in groups (dense.cuh) find their tokens.
#pragma once

#include "dense.cuh"

namespace forge {

constexpr int kMaxExperts = 512;

struct RouterDims { int experts = 0, top = 0; };
// Device tables of one routing.  A pair is (row, k), k = 0 .. top - 1; pairs are dealt to slots expert by expert, in the order of
// rows within an expert.
struct RouteTables {
    int32_t* expert = nullptr; float* weight = nullptr; int32_t* slot = nullptr;   // [rows][top]
    int32_t* row = nullptr; float* slot_weight = nullptr;                          // [rows * top], by slot
    float* row_weight = nullptr;                                                   // few rows: [experts][kScaleRows], zero where the expert is not used
    GroupTile* tiles = nullptr; int32_t* n_tiles = nullptr;
};
size_t route_bytes(const RouterDims& d, int rows);
RouteTables route_tables(void* p, const RouterDims& d, int rows);

// logits: f32 [rows][experts].  The `top` largest of a row, weighted by the softmax over them.
// Few rows (at most kScaleRows): a tile of all rows per expert that any of them uses.
int32_t route_few(const RouterDims& d, const float* logits, int rows, const RouteTables& t, GroupTable* out, cudaStream_t st);
// Any number: tiles of slots.
int32_t route_slots(const RouterDims& d, const float* logits, int rows, const RouteTables& t, GroupTable* out, cudaStream_t st);
// x[r] += sum over k of y[slot(r, k)], f32 rows of `width`, then `after`
int32_t add_experts(float* x, const float* y, const RouterDims& d, const RouteTables& t, int rows, int width, const After& after, int dtype, cudaStream_t st);

}  // namespace forge
