// Handles behind the session calls and what the host files of the library share.
#pragma once

#include <algorithm>
#include <string>
#include <vector>

#include "gemv_core.cuh"

namespace forge {
struct StackModel;   // layer-list models (stack_model.cu)
struct StackCache;
}  // namespace forge

using namespace forge;

// ------------------------------------------------------------------------------ structures
struct ForgeLayer {
    float* attn_norm = nullptr;
    QWeight qkv;           // rows: [q ; k ; v] of this rank (row-major split layout: prefill GEMM)
    QTiled qkv_t;          // the same matrix in the tiled streaming layout (decode GEMV)
    QTiled v_t;            // only when v_proj is stored in another format than q/k: qkv holds [q ; k], this holds v
    float* qkv_bias = nullptr;
    QWeight o;
    QTiled o_t;
    float* ffn_norm = nullptr;
    QWeight gateup;        // rows interleaved: 2j = gate_j, 2j+1 = up_j
    QTiled gateup_t;
    QWeight down;
    QTiled down_t;
};

struct ForgeModel {
    ForgeModelConfig cfg;
    int device = 0;
    cudaStream_t stream = nullptr;
    // local (per tensor-parallel rank) sizes
    int h = 0, qk = 0, kv = 0, ff = 0, V = 0, hd = 0, nq = 0, nkv = 0;
    float* embed = nullptr;
    std::vector<ForgeLayer> layers;
    float* final_norm = nullptr;
    QWeight lm_head;
    QTiled lm_head_t;
    int* d_err = nullptr;  // set by a kernel whose bounded wait gave up
    GemvSplit split;       // split-K scratch shared by the decode GEMVs (one launch at a time on the stream)
    GemvSplit bsplit;      // the same for the batched decode products
    uint2* d_bact = nullptr;  // packed activations of one batched product (sixteen rows)
    float* rope = nullptr;  // [max_seq][hd/2]{cos,sin}
    int max_seq = 0;
    std::vector<void*> allocs;
    StackModel* stack = nullptr;   // set for a layer-list model (stack_model.cu); the quantised-decoder fields above and below then stay empty
    // prefill scratch (grown on demand)
    int scratch_rows = 0, tok_cap = 0;
    float* p_hidden = nullptr; __half* p_normed = nullptr; float* p_qkv = nullptr; __half* p_q16 = nullptr; __half* p_q16_lo = nullptr;
    __half* p_attn16 = nullptr; float* p_gu = nullptr; __half* p_act16 = nullptr; uint32_t* p_tokens = nullptr;
    __half* p_normed_lo = nullptr; __half* p_attn16_lo = nullptr; __half* p_act16_lo = nullptr;
    float* p_parts = nullptr;   // [4][rows][h] partial products of the K-sliced o / down projections
    float* p_qkv_parts = nullptr;   // [4][rows][qk + 2 kv] the same for the QKV projection
    int gemm_passes = 3;  // 3: split-precision prefill GEMMs (default); 1: single fp16 pass
    std::vector<struct ForgeKV*> caches;   // live caches of this model (released with it if the caller did not)
    int pq[8] = {0, 0, 0, 0, 0, 0, 0, 0};  // storage format of q, k, v, o, gate, up, down, lm_head (cfg.proj_quant or cfg.quant)
    bool uniform_basic = true;             // every projection is stored in cfg.quant (Q8_0 / Q4_0): what the whole-step kernel takes
    bool per_token_prefill = false;        // no batched layout for this mix of formats: the prompt always runs token by token
    bool any_kquant = false;               // a projection is stored as Q4_K / Q6_K
    bool kquant_batched = false;           // K-quant models: prompt through the batched GEMMs (forge_model_set_prefill_mode)
    TpComm* tp = nullptr;  // tensor-parallel communicator (cfg.tp_world > 1)
    // peer-memory exchange of the decode step (forge_model_tp_exchange_*): local buffer, peers' mappings, device tables
    void* tpx_local = nullptr; std::vector<void*> tpx_peer; bool tpx_ready = false;
    uint2** d_tpx_ll = nullptr; uint32_t* d_tpx_step = nullptr;  // peers' buffers (device table), decode step counter
    float* p_part = nullptr; float* d_part = nullptr;  // this rank's partial sums of a row-sliced projection
    uint32_t wait_limit = 1u << 20;     // polls per device-side peer wait (forge_model_set_wait_limit)
    // decode scratch (per batch row).  Growing it moves every buffer: scratch_gen counts the moves, and whatever holds the
    // old addresses (a cache's captured decode graph) is rebuilt when its generation differs.
    int dec_batch = 0; int scratch_gen = 0;
    float* d_hidden2 = nullptr;
    float* d_hidden = nullptr; float* d_q = nullptr; float* d_attn = nullptr; float* d_act = nullptr; float* d_logits = nullptr;
    uint32_t* d_tok = nullptr; uint32_t* d_hist = nullptr; int hist_cap = 0; int32_t* d_step = nullptr;
    float* d_amax_val = nullptr; int* d_amax_idx = nullptr; int* d_amax_ticket = nullptr;
    // parity trace
    bool trace_on = false; float* trace = nullptr; size_t trace_cap = 0; int trace_rows = 0;
    // timing of the last generate call
    cudaEvent_t ev[3] = {nullptr, nullptr, nullptr};
    float prefill_ms = 0.f, decode_ms = 0.f; long long last_launches = 0;
};

struct ForgeKV {
    ForgeModel* model = nullptr;
    int max_seq = 0, batch = 0, pages_per_seq = 0, num_pages = 0;
    __half* k_pool = nullptr; __half* v_pool = nullptr;
    size_t layer_stride = 0;  // halfs per layer pool
    int32_t* d_page_table = nullptr; int32_t* d_seq_len = nullptr;
    std::vector<int32_t> h_page_table; std::vector<int> free_pages; std::vector<int> pages_used; std::vector<int> len;
    float* attn_ws = nullptr; int* attn_counters = nullptr; int splits = 1;
    StackCache* stack = nullptr;   // cache rows and states of a layer-list model (then k_pool and v_pool stay empty)
    int slot0 = 0;                 // of a view of single sequences: the first one's state slot
    std::vector<char> lost;        // sequences whose recurrent state a failed step has left undefined
    alignas(64) unsigned char k_map[128], v_map[128];   // CUtensorMap of the two pools (all layers), for the decode attention's page copies
    cudaGraphExec_t graph = nullptr; int graph_batch = 0; bool graph_greedy = false; int graph_gen = -1;  // scratch generation the graph was captured with
    long long graph_kernels = 0;   // kernels of one replay
};

namespace forge {

template <typename T>
int32_t dev_alloc(ForgeModel* m, T** p, size_t count) {
    void* q = nullptr;
    FORGE_CUDA(cudaMalloc(&q, std::max<size_t>(count, 1) * sizeof(T)));
    m->allocs.push_back(q);
    *p = static_cast<T*>(q);
    return FORGE_OK;
}


// hand out pages so that sequence `seq` can hold `new_len` positions; uploads the table row if it changed
int32_t ensure_pages(ForgeKV* kv, int seq, int new_len);
int32_t upload_len(ForgeKV* kv);
// The synchronisation point of a session call.  Also reads the word the bounded device-side waits raise when they give
// up (a pipeline stage, a peer's contribution or another CTA's result never arrived): the call then fails with
// FORGE_ERR_TIMEOUT, the word is cleared and the device-side positions are put back to the host's (`kv`, may be null).
int32_t sync_and_check(ForgeModel* m, ForgeKV* kv);
int32_t ensure_decode_scratch(ForgeModel* m, int batch);
int32_t ensure_trace(ForgeModel* m, int rows);
int32_t check_seq(const ForgeKV* kv, int seq);
// a failed step of a model with recurrent state: the sequences that hold one must start over (or be loaded)
void mark_lost(ForgeKV* kv);

// ------------------------------------------------------------------ layer-list models (stack_model.cu)
void stack_destroy(ForgeModel* m);
int32_t stack_cache_create(ForgeKV* kv);
void stack_cache_destroy(ForgeKV* kv);
// One forward pass of the step's entries as one batch, from the cache that earlier steps left.  tokens / want: the entries'
// tokens and wanted places (within the entry) one after another; the wanted logits are left in *d_logits [wants][V].
// Pages are reserved by the caller; kv->len is not advanced.  trace_rows > 0 (one entry): the residual stream after every
// layer goes to the model's trace, rows [trace_row0, trace_row0 + n) of trace_rows.
int32_t stack_step(ForgeModel* m, ForgeKV* kv, const ForgeStepEntry* entries, int n_entries, const uint32_t* tokens, const int32_t* want, float** d_logits,
                   int trace_rows = 0, int trace_row0 = 0);
// prompt portion of one sequence (any length): as stack_step in bounded portions, the last row's logits in m->d_logits
int32_t stack_prefill(ForgeModel* m, ForgeKV* kv, int seq, const uint32_t* tokens_host, int n);
// decode step of `batch` sequences from device-side tokens and positions (captured into the cache's graph)
int32_t stack_ensure_decode(ForgeModel* m, ForgeKV* kv, int batch);
int32_t stack_decode_launches(ForgeModel* m, ForgeKV* kv, int batch, bool greedy, bool record);
bool stack_has_state(const ForgeModel* m);
int stack_kv_width(const ForgeKV* kv, int run, int which);
int32_t stack_kv_read(ForgeKV* kv, int seq, int run, int which, float* out_host);
size_t stack_state_values(const ForgeKV* kv, int run);
int32_t stack_state_read(ForgeKV* kv, int seq, int run, float* out_host);
size_t stack_kv_bytes_per_token(const ForgeKV* kv);
size_t stack_kv_bytes(const ForgeKV* kv, int len);   // of a sequence
int32_t stack_kv_copy(ForgeKV* kv, int seq, int len, char* host, bool to_host);

}  // namespace forge
