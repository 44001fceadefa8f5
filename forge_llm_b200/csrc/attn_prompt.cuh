// Prompt attention of the layer-list models (bfloat16): query tiles of several sequences over their contexts.
#pragma once

#include "attn_rows.cuh"
#include "mla.cuh"

namespace forge {

struct PromptDims {
    int heads = 0, share = 1;                 // query head h uses key / value head h / share
    int dim = 0, rot = 0, vdim = 0;           // query / key part of the head, part whose keys all heads share, values
    int dim_p = 0, rot_p = 0, vdim_p = 0;     // padded to 64
    float scale = 1.f, softcap = 0.f;
    int chunk = 0, window = 0, keep = 0, pool = 0, bias_n = 0;   // as in AttnDims
    float bound = 0.f;                        // > 0: no score (bias included) is larger or smaller than this
    bool joint = false;                       // every head meets the values of all groups: out [row][head][group][vdim_p]
    PromptDims() = default;
    explicit PromptDims(const LatentDims& d) : heads(d.heads), dim(d.dim), rot(d.rot), vdim(d.vdim), dim_p(d.dim_p), rot_p(d.rot_p), vdim_p(d.vdim_p), scale(d.scale) {}
    explicit PromptDims(const AttnDims& d)
        : heads(d.heads), share(d.heads / d.groups), dim(d.dim), vdim(d.vdim), dim_p(d.dim_p), vdim_p(d.vdim_p), scale(d.scale), softcap(d.softcap), chunk(d.chunk), window(d.window), keep(d.keep), pool(d.pool), bias_n(d.bias_n) {}
};
// query rows of the step, position of the first, first context row of its sequence, first row of its blocks
struct PromptTile { int32_t row0, rows, pos0, ctx0, pool0, unused[3]; };
struct PromptAttnArgs {
    // [q_rows][heads][dim_p + rot_p], [ctx][heads / share][dim_p], [ctx][rot_p], [ctx][heads / share][vdim_p]
    const void* q = nullptr; const void* k = nullptr; const void* krot = nullptr; const void* v = nullptr;
    const void* gate = nullptr; int gate_ld = 0;      // out[row][head * vdim + i] = gate * attention: bf16 per value,
    const float* head_gate = nullptr;                 // or, without gate, f32 per head, or none
    const float* sink = nullptr;                      // score per head that enters the denominator
    void* out = nullptr; int out_ld = 0;
    int q_rows = 0, ctx_rows = 0;
    const PromptTile* tiles = nullptr; int n_tiles = 0;   // device
    const PromptTile* host_tiles = nullptr;               // the same on the host, if they are at hand
    // k and v are the pool of the cache: rows of page_row values, context rows 64 i .. lie in page pages[i] (device)
    const int32_t* pages = nullptr; int page_row = 0;
    const float* bias = nullptr;                      // [heads][bias_n]
    const void* blocks = nullptr; int block_rows = 0; // rows like the cache's
    int* err = nullptr;
};
bool attn_prefill_kv_supported(const PromptDims& d);
int32_t attn_prefill_kv(const PromptDims& d, const PromptAttnArgs& a, cudaStream_t st);

}  // namespace forge
