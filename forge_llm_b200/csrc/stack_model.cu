// Layer-list models: a checkpoint's config.json names an architecture and lists layers, each with a mixer, the mixer's sizes
// and a feed-forward.  This file holds the registry, the reader of the configuration, the loader, the cache rows and the
// launch sequences; the session calls (model.cu) - cache, prompt, decode graph, greedy loop, sampling, mixed steps - take
// such a model like a quantised decoder.
//
// One layer of the parallel arrangement (x += mixer(h) + ff(h), one norm in front) is two dense products and, between them,
// the attention:
//   in    one product of h over the stacked rows [q | dkv | g | gate, up interleaved]; its epilogue leaves q and dkv as f32,
//         sigmoid(g), and the gated feed-forward activation;
//   post  latent norm, rotations, cache append, queries into the latent space (rows of their own) or in prompt layout;
//   attention over the latent cache (single rows) or over keys and values formed for the portion (prompts);
//   out   one product over the concatenated columns [o | down] of [gated heads | feed-forward activation]: both sublayers
//         are summed by the product itself; its epilogue adds the residual and applies the next layer's Dynamic Tanh norm,
//         which needs no statistics of the row.
#include <algorithm>
#include <cmath>
#include <cstring>
#include <map>
#include <memory>

#include "checkpoint.cuh"
#include "mla.cuh"
#include "model.cuh"

// ------------------------------------------------------------------------------------------------ structures
namespace forge {

enum class Norm { DynamicTanh };
enum class Arrangement { Parallel };
enum class Mlp { ClampedGlu };
struct Architecture { const char* name; Norm norm; Arrangement arrangement; Mlp dense; };
static const Architecture kArchitectures[] = {
    {"Bolenex", Norm::DynamicTanh, Arrangement::Parallel, Mlp::ClampedGlu},
};

struct LayerSpec {
    LatentDims mix;
    double rot_base = 1.0;
    int ff = 0;            // 0: no feed-forward
    float limit = 0.f;
    int weights_of = -1;   // layer whose tensors are used
};
struct StackSpec {
    const Architecture* arch = nullptr;
    int width = 0, vocab = 0;
    float eps = 0.f;
    std::vector<LayerSpec> layers;
    int64_t parameters = 0;
};

struct DytNorm { float* w = nullptr; float* b = nullptr; float alpha = 0.f; };

struct LayerWeights {
    DytNorm norm;
    DenseWeight in, out, kv;      // kv: rows [uk | uv] over the latent
    int q_rows = 0, dkv_row = 0, g_row = 0, glu_row = 0, uv_row = 0;   // first rows of the segments of `in` / `kv`
    int heads_k = 0;              // columns of `out` in front of the feed-forward's
    float* kv_norm = nullptr;
    float* rope = nullptr;        // of this layer's base and dims
};

struct StackModel {
    StackSpec spec;
    int dtype = FORGE_BF16;
    int width_p = 0;
    void* embed = nullptr;
    std::vector<LayerWeights> w;                       // by layer; empty for a layer with weights_of
    DytNorm final_norm;
    DenseWeight head;
    std::map<std::pair<double, int>, std::pair<int, float*>> ropes;   // (base, dims) -> positions, table
    int rope_positions = 0;
    DenseScratch scratch;
    // step buffers, grown on demand (scratch_gen of the model counts the moves)
    struct Buf { void* p = nullptr; size_t cap = 0; };
    Buf x, h, proj, gate, mid, q, part, ml, ctx_c, ctx_r, ctx_k, ctx_v, sel, logits, meta;
    std::vector<Buf*> all() { return {&x, &h, &proj, &gate, &mid, &q, &part, &ml, &ctx_c, &ctx_r, &ctx_k, &ctx_v, &sel, &logits, &meta}; }
};

// Cache rows of every layer run: [pages][FORGE_KV_PAGE][row] of the model's type, one pool per run.
struct StackCache {
    struct Run { void* pool = nullptr; alignas(64) unsigned char map[128]; };
    std::vector<Run> runs;
    int splits = 1;     // of a captured decode step
};

namespace {

// ------------------------------------------------------------------------------------------------ configuration
int32_t need_int(const Json* o, const char* key, int* out, int lo = 1) {
    const Json* v = o ? o->get(key) : nullptr;
    if (!v || v->kind != Json::Number || v->num != std::floor(v->num) || v->num < lo || v->num > 1e9) { set_error("config.json: \"%s\" must be an integer of at least %d", key, lo); return FORGE_ERR_SHAPE; }
    *out = int(v->num);
    return FORGE_OK;
}
int32_t need_num(const Json* o, const char* key, double* out) {
    const Json* v = o ? o->get(key) : nullptr;
    if (!v || v->kind != Json::Number) { set_error("config.json: \"%s\" must be a number", key); return FORGE_ERR_SHAPE; }
    *out = v->num;
    return FORGE_OK;
}
int32_t need_string(const Json* o, const char* key, std::string* out) {
    const Json* v = o ? o->get(key) : nullptr;
    if (!v || v->kind != Json::String) { set_error("config.json: \"%s\" must be a string", key); return FORGE_ERR_SHAPE; }
    *out = v->str;
    return FORGE_OK;
}

int32_t parse_latent(const Json* m, float eps, LayerSpec* L) {
    LatentDims& d = L->mix;
    double scale;
    FORGE_TRY(need_int(m, "heads", &d.heads));
    FORGE_TRY(need_int(m, "dim", &d.dim));
    FORGE_TRY(need_int(m, "rot_dim", &d.rot, 0));
    FORGE_TRY(need_int(m, "vdim", &d.vdim));
    FORGE_TRY(need_int(m, "kv_rank", &d.rank));
    FORGE_TRY(need_num(m, "scale", &scale));
    if (d.rot > 0) {
        const Json* rot = m->get("rot");
        FORGE_TRY(need_int(rot, "dims", &d.rot_dims, 0));
        FORGE_TRY(need_num(rot, "base", &L->rot_base));
        if (d.rot_dims > d.rot || d.rot_dims % 2 || !(L->rot_base > 0)) { set_error("config.json: rot.dims %d does not fit rot_dim %d", d.rot_dims, d.rot); return FORGE_ERR_SHAPE; }
    }
    d.scale = float(scale); d.eps = eps;
    d.rank_p = pad_to(d.rank, 64); d.rot_p = pad_to(d.rot, 64); d.dim_p = pad_to(d.dim, 64); d.vdim_p = pad_to(d.vdim, 64);
    return FORGE_OK;
}

int32_t parse_spec(const Json& c, StackSpec* s) {
    std::string name;
    FORGE_TRY(need_string(&c, "architecture", &name));
    for (const Architecture& a : kArchitectures) if (name == a.name) s->arch = &a;
    if (!s->arch) { set_error("architecture \"%s\" is not registered", name.c_str()); return FORGE_ERR_UNSUPPORTED; }
    FORGE_TRY(need_int(&c, "width", &s->width));
    FORGE_TRY(need_int(&c, "vocab", &s->vocab));
    double eps;
    FORGE_TRY(need_num(c.get("norm"), "eps", &eps));
    s->eps = float(eps);
    const Json* layers = c.get("layers");
    if (!layers || layers->kind != Json::Array || layers->items.empty()) { set_error("config.json: \"layers\" must list at least one layer"); return FORGE_ERR_SHAPE; }
    for (size_t i = 0; i < layers->items.size(); ++i) {
        const Json& e = layers->items[i];
        LayerSpec L;
        std::string type;
        FORGE_TRY(need_string(&e, "type", &type));
        if (type != "latent_attention") { set_error("layer %zu: mixer \"%s\" is not supported", i, type.c_str()); return FORGE_ERR_UNSUPPORTED; }
        FORGE_TRY(parse_latent(e.get("mixer"), s->eps, &L));
        const Json* mlp = e.get("mlp");
        if (mlp && mlp->kind != Json::Null) {
            std::string kind;
            FORGE_TRY(need_string(mlp, "kind", &kind));
            if (kind != "dense") { set_error("layer %zu: feed-forward \"%s\" is not supported", i, kind.c_str()); return FORGE_ERR_UNSUPPORTED; }
            double limit;
            FORGE_TRY(need_int(mlp, "ff", &L.ff));
            FORGE_TRY(need_num(mlp, "limit", &limit));
            L.limit = float(limit);
        }
        const Json* of = e.get("weights_of");
        if (of && of->kind != Json::Null) {
            FORGE_TRY(need_int(&e, "weights_of", &L.weights_of, 0));
            if (L.weights_of >= int(layers->items.size()) || L.weights_of == int(i)) { set_error("layer %zu: weights_of %d is not another layer", i, L.weights_of); return FORGE_ERR_SHAPE; }
        }
        s->layers.push_back(L);
    }
    for (size_t i = 0; i < s->layers.size(); ++i) {
        const LayerSpec& L = s->layers[i];
        if (L.weights_of < 0) continue;
        const LayerSpec& O = s->layers[L.weights_of];
        const LatentDims &a = L.mix, &b = O.mix;
        if (O.weights_of >= 0 || a.heads != b.heads || a.dim != b.dim || a.rot != b.rot || a.vdim != b.vdim || a.rank != b.rank || L.ff != O.ff) {
            set_error("layer %zu: weights_of %d names a layer of other sizes or without tensors", i, L.weights_of);
            return FORGE_ERR_SHAPE;
        }
    }
    return FORGE_OK;
}

// every tensor of the design, with its shape
struct LayerTensors { const TensorView *norm, *norm_b, *norm_a, *q, *dkv, *kvn, *uk, *uv, *g, *o, *gate, *up, *down; };
struct StackTensors { const TensorView *embed, *head, *fn, *fb, *fa; std::vector<LayerTensors> layers; };

int32_t find_tensors(const Checkpoint& ck, const StackSpec& s, StackTensors* t) {
#define GET(dst, ...) do { dst = ck.tensor(__VA_ARGS__); if (!dst) return FORGE_ERR_SHAPE; } while (0)
    const int64_t W = s.width, V = s.vocab;
    GET(t->embed, "embed", {V, W});
    GET(t->head, "head", {V, W});
    GET(t->fn, "final.norm", {W}); GET(t->fb, "final.norm.b", {W}); GET(t->fa, "final.norm.alpha", {});
    for (size_t i = 0; i < s.layers.size(); ++i) {
        t->layers.push_back(LayerTensors{});
        const LayerSpec& L = s.layers[i];
        if (L.weights_of >= 0) continue;
        LayerTensors& o = t->layers.back();
        const LatentDims& d = L.mix;
        const std::string p = "l" + std::to_string(i) + ".", x = p + "mix.";
        const int64_t HV = int64_t(d.heads) * d.vdim;
        GET(o.norm, p + "norm1", {W}); GET(o.norm_b, p + "norm1.b", {W}); GET(o.norm_a, p + "norm1.alpha", {});
        GET(o.q, x + "q", {int64_t(d.heads) * (d.dim + d.rot), W});
        GET(o.dkv, x + "dkv", {d.rank + d.rot, W});
        GET(o.kvn, x + "dkv.norm", {d.rank});
        GET(o.uk, x + "uk", {int64_t(d.heads) * d.dim, d.rank});
        GET(o.uv, x + "uv", {HV, d.rank});
        GET(o.g, x + "g", {HV, W});
        GET(o.o, x + "o", {W, HV});
        if (L.ff) {
            GET(o.gate, p + "mlp.gate", {L.ff, W});
            GET(o.up, p + "mlp.up", {L.ff, W});
            GET(o.down, p + "mlp.down", {W, L.ff});
        }
    }
#undef GET
    return FORGE_OK;
}

void fill_info(const StackSpec& s, ForgeCheckpointInfo* out) {
    memset(out, 0, sizeof(*out));
    snprintf(out->architecture, sizeof out->architecture, "%s", s.arch->name);
    out->hidden_size = s.width; out->vocab_size = s.vocab; out->num_layers = int32_t(s.layers.size());
    out->parameters = s.parameters;
    for (const LayerSpec& L : s.layers) { out->num_weight_layers += L.weights_of < 0; out->cache_values_per_token += L.mix.row(); }
}

// ------------------------------------------------------------------------------------------------ loading
void store(void* dst, int dtype, size_t i, const TensorView& t, size_t j) {
    if (dtype == FORGE_F32) { static_cast<float*>(dst)[i] = t.at(j); return; }
    if (t.dtype == "BF16") { memcpy(static_cast<uint16_t*>(dst) + i, t.data + 2 * j, 2); return; }
    static_cast<__nv_bfloat16*>(dst)[i] = __float2bfloat16_rn(t.at(j));
}
// rows of `t` [n][k] into the host image of a matrix with rows of `ld`: row r -> row0 + r * step, columns from col0
void put_rows(std::vector<uint8_t>& img, int dtype, int ld, const TensorView& t, int row0, int step = 1, int col0 = 0) {
    const int64_t n = t.shape[0], k = t.shape[1];
    for (int64_t r = 0; r < n; ++r) {
        const size_t at = size_t(row0 + r * step) * ld + col0;
        if (dtype == FORGE_BF16 && t.dtype == "BF16") memcpy(img.data() + at * 2, t.data + size_t(r) * k * 2, size_t(k) * 2);
        else if (dtype == FORGE_F32 && t.dtype == "F32") memcpy(img.data() + at * 4, t.data + size_t(r) * k * 4, size_t(k) * 4);
        else for (int64_t c = 0; c < k; ++c) store(img.data(), dtype, at + c, t, size_t(r * k + c));
    }
}
int32_t upload(ForgeModel* m, void** dst, const std::vector<uint8_t>& img) {
    uint8_t* p = nullptr;
    FORGE_TRY(dev_alloc(m, &p, img.size()));
    FORGE_CUDA(cudaMemcpyAsync(p, img.data(), img.size(), cudaMemcpyHostToDevice, m->stream));
    FORGE_CUDA(cudaStreamSynchronize(m->stream));
    *dst = p;
    return FORGE_OK;
}
int32_t upload_f32(ForgeModel* m, float** dst, const TensorView& t) {
    std::vector<float> v(size_t(t.count()));
    for (size_t i = 0; i < v.size(); ++i) v[i] = t.at(i);
    FORGE_TRY(dev_alloc(m, dst, v.size()));
    FORGE_CUDA(cudaMemcpyAsync(*dst, v.data(), v.size() * 4, cudaMemcpyHostToDevice, m->stream));
    FORGE_CUDA(cudaStreamSynchronize(m->stream));
    return FORGE_OK;
}
int32_t load_dyt(ForgeModel* m, DytNorm* n, const TensorView& w, const TensorView& b, const TensorView& a) {
    n->alpha = a.at(0);
    FORGE_TRY(upload_f32(m, &n->w, w));
    return upload_f32(m, &n->b, b);
}
// row_reads: some kernel reads rows of the matrix, so it is kept in rows as well
int32_t load_dense(ForgeModel* m, DenseWeight* w, int N, int K, int dtype, const std::vector<uint8_t>& img, bool row_reads = false) {
    w->N = N; w->K = K; w->dtype = dtype;
    if (dtype == FORGE_F32 || row_reads) FORGE_TRY(upload(m, &w->w, img));
    if (dtype == FORGE_BF16) {
        std::vector<uint8_t> tiles(dense_tile_bytes(N, K));
        dense_tile_image(tiles.data(), img.data(), N, K);
        FORGE_TRY(upload(m, &w->tiles, tiles));
    }
    return FORGE_OK;
}

int32_t load_layer(ForgeModel* m, const LayerSpec& L, const LayerTensors& t, LayerWeights* w) {
    StackModel& S = *m->stack;
    const LatentDims& d = L.mix;
    const size_t es = dense_size(S.dtype);
    FORGE_TRY(load_dyt(m, &w->norm, *t.norm, *t.norm_b, *t.norm_a));
    FORGE_TRY(upload_f32(m, &w->kv_norm, *t.kvn));
    w->q_rows = d.heads * (d.dim + d.rot);
    w->dkv_row = pad_to(w->q_rows, kSegAlign);
    w->g_row = w->dkv_row + pad_to(d.rank + d.rot, kSegAlign);
    w->glu_row = w->g_row + pad_to(d.heads * d.vdim, kSegAlign);
    const int n_in = w->glu_row + 2 * L.ff;
    {
        std::vector<uint8_t> img(size_t(n_in) * S.width_p * es, 0);
        put_rows(img, S.dtype, S.width_p, *t.q, 0);
        put_rows(img, S.dtype, S.width_p, *t.dkv, w->dkv_row);
        put_rows(img, S.dtype, S.width_p, *t.g, w->g_row);
        if (L.ff) { put_rows(img, S.dtype, S.width_p, *t.gate, w->glu_row, 2); put_rows(img, S.dtype, S.width_p, *t.up, w->glu_row + 1, 2); }
        FORGE_TRY(load_dense(m, &w->in, n_in, S.width_p, S.dtype, img));
    }
    {
        w->uv_row = pad_to(d.heads * d.dim, kSegAlign);
        const int n = w->uv_row + d.heads * d.vdim;
        std::vector<uint8_t> img(size_t(n) * d.rank_p * es, 0);
        put_rows(img, S.dtype, d.rank_p, *t.uk, 0);
        put_rows(img, S.dtype, d.rank_p, *t.uv, w->uv_row);
        FORGE_TRY(load_dense(m, &w->kv, n, d.rank_p, S.dtype, img, true));
    }
    {
        w->heads_k = pad_to(d.heads * d.vdim, kDensePad);
        const int k = w->heads_k + pad_to(L.ff, kDensePad);
        std::vector<uint8_t> img(size_t(S.spec.width) * k * es, 0);
        put_rows(img, S.dtype, k, *t.o, 0);
        if (L.ff) put_rows(img, S.dtype, k, *t.down, 0, 1, w->heads_k);
        FORGE_TRY(load_dense(m, &w->out, S.spec.width, k, S.dtype, img));
    }
    return FORGE_OK;
}

// rotation tables of every (base, dims) for at least n positions
int32_t ensure_rope(ForgeModel* m, int n) {
    StackModel& S = *m->stack;
    if (n <= S.rope_positions) return FORGE_OK;
    n = pad_to(n, 1024);
    FORGE_CUDA(cudaStreamSynchronize(m->stream));
    for (const LayerSpec& L : S.spec.layers) {
        auto& e = S.ropes[{L.rot_base, L.mix.rot_dims}];
        if (e.first >= n) continue;
        std::vector<float> tab(std::max<size_t>(1, size_t(n) * L.mix.rot_dims));
        FORGE_TRY(rope_half_table(tab.data(), n, L.mix.rot_dims, L.rot_base));
        float* p = nullptr;
        FORGE_CUDA(cudaMalloc(&p, tab.size() * 4));
        if (e.second) cudaFree(e.second);
        e = {n, p};
        FORGE_CUDA(cudaMemcpyAsync(p, tab.data(), tab.size() * 4, cudaMemcpyHostToDevice, m->stream));
        FORGE_CUDA(cudaStreamSynchronize(m->stream));
    }
    S.rope_positions = n;
    ++m->scratch_gen;   // captured steps hold the old tables
    return FORGE_OK;
}

// ------------------------------------------------------------------------------------------------ step buffers
int32_t grow(ForgeModel* m, StackModel::Buf& b, size_t bytes) {
    if (bytes <= b.cap) return FORGE_OK;
    FORGE_CUDA(cudaStreamSynchronize(m->stream));   // nothing in flight reads the old one
    if (b.p) cudaFree(b.p);
    b.p = nullptr; b.cap = 0;
    bytes = (bytes + bytes / 4 + 255) & ~size_t(255);
    FORGE_CUDA(cudaMalloc(&b.p, bytes));
    b.cap = bytes;
    FORGE_CUDA(cudaMemsetAsync(b.p, 0, bytes, m->stream));   // padding columns meet zero weights: they must be finite
    ++m->scratch_gen;
    return FORGE_OK;
}

bool tensor_core_rows(const StackModel& S, const LatentDims& d) { return S.dtype == FORGE_BF16 && latent_decode_tc_supported(d); }

// splits of the row attention: at most one CTA per SM over all rows and head groups, no more than there are pages
int row_splits(const StackModel& S, int rows, int pages) {
    int groups = 1;
    for (const LayerSpec& L : S.spec.layers) groups = std::max(groups, tensor_core_rows(S, L.mix) ? latent_decode_head_groups(L.mix) : L.mix.heads);
    return std::max(1, std::min(pages, 148 / std::max(1, rows * groups)));
}

int32_t ensure_step(ForgeModel* m, int rows, int single, int splits, int prompt, int ctx_rows) {
    StackModel& S = *m->stack;
    const size_t es = dense_size(S.dtype), r = size_t(rows);
    size_t proj = 0, gate = 0, mid = 0, qa = 0, part = 0, heads = 0, qp = 0, cc = 0, cr = 0, ck = 0, cv = 0;
    for (size_t i = 0; i < S.spec.layers.size(); ++i) {
        const LayerSpec& L = S.spec.layers[i];
        const LayerWeights& w = S.w[L.weights_of >= 0 ? L.weights_of : int(i)];
        const LatentDims& d = L.mix;
        proj = std::max(proj, size_t(w.g_row));
        gate = std::max(gate, size_t(d.heads) * d.vdim);
        mid = std::max(mid, size_t(w.out.K));
        qa = std::max(qa, size_t(d.heads) * d.row());
        part = std::max(part, size_t(d.heads) * d.rank_p);
        heads = std::max(heads, size_t(d.heads));
        qp = std::max(qp, size_t(d.heads) * (d.dim_p + d.rot_p));
        cc = std::max(cc, size_t(d.rank_p)); cr = std::max(cr, size_t(std::max(d.rot_p, 64)));
        ck = std::max(ck, size_t(d.heads) * d.dim_p); cv = std::max(cv, size_t(d.heads) * d.vdim_p);
    }
    FORGE_TRY(grow(m, S.x, r * S.spec.width * 4));
    FORGE_TRY(grow(m, S.h, r * S.width_p * es));
    FORGE_TRY(grow(m, S.proj, r * proj * 4));
    FORGE_TRY(grow(m, S.gate, r * gate * es));
    FORGE_TRY(grow(m, S.mid, r * mid * es));
    FORGE_TRY(grow(m, S.q, std::max(size_t(single) * qa * es, size_t(prompt) * qp * es)));
    FORGE_TRY(grow(m, S.part, size_t(single) * part * splits * 4));
    FORGE_TRY(grow(m, S.ml, size_t(single) * heads * splits * sizeof(float2)));
    if (ctx_rows) {
        FORGE_TRY(grow(m, S.ctx_c, size_t(ctx_rows) * cc * es));
        FORGE_TRY(grow(m, S.ctx_r, size_t(ctx_rows) * cr * es));
        FORGE_TRY(grow(m, S.ctx_k, size_t(ctx_rows) * ck * es));
        FORGE_TRY(grow(m, S.ctx_v, size_t(ctx_rows) * cv * es));
    }
    // one ticket per output tile of the largest product (128 rows x at least 16 tokens)
    size_t n_max = size_t(S.head.N);
    for (const LayerWeights& w : S.w) n_max = std::max({n_max, size_t(w.in.N), size_t(w.out.N), size_t(w.kv.N)});
    const size_t tiles = ((n_max + 127) / 128) * std::max<size_t>(1, (size_t(std::max(rows, ctx_rows)) + 127) / 128);
    if (tiles > S.scratch.tickets_cap) {
        FORGE_TRY(dev_alloc(m, &S.scratch.tickets, tiles));
        FORGE_CUDA(cudaMemsetAsync(S.scratch.tickets, 0, tiles * sizeof(int), m->stream));
        S.scratch.tickets_cap = tiles;
        ++m->scratch_gen;
    }
    return FORGE_OK;
}

struct Step {
    const uint32_t* tokens = nullptr;        // device
    StepRows rows;
    int single = 0, splits = 1;              // rows [0, single): attention row by row; the rest are prompt rows
    const PromptTile* tiles = nullptr; int n_tiles = 0;
    const int32_t* ctx_pages = nullptr; int ctx_rows = 0;
    uint32_t* hist = nullptr; const int32_t* step = nullptr;
    float* trace = nullptr; size_t trace_stride = 0;
};

char* at(void* p, size_t elems, int dtype) { return static_cast<char*>(p) + elems * dense_size(dtype); }

// the whole stack for the rows of a step; leaves the final norm's rows in S.h
int32_t run_layers(ForgeModel* m, ForgeKV* kv, const Step& s) {
    StackModel& S = *m->stack;
    cudaStream_t st = m->stream;
    const int n = s.rows.n, W = S.spec.width, dt = S.dtype, nl = int(S.spec.layers.size());
    auto weights = [&](int l) -> const LayerWeights& { return S.w[S.spec.layers[l].weights_of >= 0 ? S.spec.layers[l].weights_of : l]; };
    auto norm_of = [&](int l) -> const DytNorm& { return l < nl ? weights(l).norm : S.final_norm; };
    FORGE_TRY(embed_dyt(static_cast<float*>(S.x.p), S.h.p, S.width_p, S.embed, dt, s.tokens, n, W, norm_of(0).alpha, norm_of(0).w, norm_of(0).b, s.hist, s.step, st));
    for (int l = 0; l < nl; ++l) {
        const LayerSpec& L = S.spec.layers[l];
        const LayerWeights& w = weights(l);
        const LatentDims& d = L.mix;
        const int ldp = w.g_row, gate_ld = d.heads * d.vdim, mid_ld = w.out.K;
        float* proj = static_cast<float*>(S.proj.p);
        const float* rope = S.ropes.at({L.rot_base, d.rot_dims}).second;
        StackCache::Run& run = kv->stack->runs[l];
        {
            DenseOut o;
            auto add = [&](int kind, int row0, int rows, void* dst, int ld) -> OutSeg& { OutSeg& g = o.seg[o.nseg++]; g.kind = kind; g.row0 = row0; g.rows = rows; g.dst = dst; g.ld = ld; return g; };
            add(SEG_F32, 0, w.q_rows, proj, ldp);
            add(SEG_F32, w.dkv_row, d.rank + d.rot, proj + w.dkv_row, ldp);
            add(SEG_SIGMOID, w.g_row, gate_ld, S.gate.p, gate_ld);
            if (L.ff) add(SEG_CLAMPED_GLU, w.glu_row, 2 * L.ff, at(S.mid.p, w.heads_k, dt), mid_ld).limit = L.limit;
            FORGE_TRY(dense_gemm(w.in, S.h.p, S.width_p, n, o, S.scratch, m->d_err, st));
        }
        StepRows single = s.rows;
        single.n = s.single;
        if (s.single > 0) {
            float* part = static_cast<float*>(S.part.p);
            float2* ml = static_cast<float2*>(S.ml.p);
            FORGE_TRY(latent_post(d, dt, proj, ldp, w.dkv_row, w.kv_norm, rope, w.kv.w, w.kv.K, S.q.p, run.pool, single, st));
            if (tensor_core_rows(S, d)) FORGE_TRY(latent_decode_tc(d, S.q.p, run.map, single, s.splits, part, ml, m->d_err, st));
            else FORGE_TRY(latent_attn_rows(d, dt, S.q.p, run.pool, single, s.splits, part, ml, st));
            FORGE_TRY(latent_value(d, dt, part, ml, s.splits, at(w.kv.w, size_t(w.uv_row) * w.kv.K, dt), w.kv.K, S.gate.p, gate_ld, S.mid.p, mid_ld, single, st));
        }
        const int np = n - s.single;
        if (np > 0) {
            StepRows pr = s.rows;
            pr.n = np; pr.pos += s.single; pr.seq += s.single;
            FORGE_TRY(latent_post_prompt(d, proj + size_t(s.single) * ldp, ldp, w.dkv_row, w.kv_norm, rope, S.q.p, run.pool, pr, st));
            FORGE_TRY(latent_gather_context(d, run.pool, s.ctx_pages, s.ctx_rows, S.ctx_c.p, S.ctx_r.p, st));
            DenseOut o;
            o.nseg = 2;
            o.seg[0].kind = o.seg[1].kind = SEG_CAST;
            o.seg[0].rows = d.heads * d.dim; o.seg[0].dst = S.ctx_k.p; o.seg[0].ld = d.heads * d.dim_p; o.seg[0].group = d.dim; o.seg[0].group_ld = d.dim_p;
            o.seg[1].row0 = w.uv_row; o.seg[1].rows = d.heads * d.vdim; o.seg[1].dst = S.ctx_v.p; o.seg[1].ld = d.heads * d.vdim_p; o.seg[1].group = d.vdim; o.seg[1].group_ld = d.vdim_p;
            FORGE_TRY(dense_gemm(w.kv, S.ctx_c.p, d.rank_p, s.ctx_rows, o, S.scratch, m->d_err, st));
            PromptAttnArgs a{S.q.p, S.ctx_k.p, S.ctx_r.p, S.ctx_v.p, at(S.gate.p, size_t(s.single) * gate_ld, dt), gate_ld, at(S.mid.p, size_t(s.single) * mid_ld, dt), mid_ld,
                             np, s.ctx_rows, s.tiles, s.n_tiles, m->d_err};
            FORGE_TRY(attn_prefill_kv(d, a, st));
        }
        {
            const DytNorm& nx = norm_of(l + 1);
            DenseOut o;
            o.nseg = 1;
            OutSeg& g = o.seg[0];
            g.kind = SEG_RESID; g.rows = W; g.dst = S.x.p; g.ld = W;
            g.alpha = nx.alpha; g.norm_w = nx.w; g.norm_b = nx.b; g.next = S.h.p; g.next_ld = S.width_p;
            FORGE_TRY(dense_gemm(w.out, S.mid.p, mid_ld, n, o, S.scratch, m->d_err, st));
        }
        if (s.trace) FORGE_CUDA(cudaMemcpyAsync(s.trace + size_t(l) * s.trace_stride, S.x.p, sizeof(float) * n * W, cudaMemcpyDeviceToDevice, st));
    }
    return FORGE_OK;
}

int32_t run_head(ForgeModel* m, const void* h, int n, float* logits) {
    StackModel& S = *m->stack;
    DenseOut o;
    o.nseg = 1;
    o.seg[0].rows = S.spec.vocab; o.seg[0].dst = logits; o.seg[0].ld = S.spec.vocab;
    return dense_gemm(S.head, h, S.width_p, n, o, S.scratch, m->d_err, m->stream);
}

// Entries of fewer tokens than this run row by row over the latent cache: forming the keys and values of the whole context
// does not pay for them.
constexpr int kPromptRows = 32;
constexpr int kPortion = 4096;      // rows of a prompt per pass

}  // namespace

void stack_destroy(ForgeModel* m) {
    if (!m->stack) return;
    for (StackModel::Buf* b : m->stack->all()) if (b->p) cudaFree(b->p);
    for (auto& e : m->stack->ropes) if (e.second.second) cudaFree(e.second.second);
    delete m->stack;
    m->stack = nullptr;
}

// ------------------------------------------------------------------------------------------------ cache
int32_t stack_cache_create(ForgeKV* kv) {
    ForgeModel* m = kv->model;
    StackModel& S = *m->stack;
    FORGE_TRY(ensure_rope(m, kv->max_seq));
    kv->stack = new StackCache();
    kv->stack->runs.resize(S.spec.layers.size());
    const size_t rows = size_t(kv->num_pages) * FORGE_KV_PAGE;
    for (size_t i = 0; i < S.spec.layers.size(); ++i) {
        const LatentDims& d = S.spec.layers[i].mix;
        StackCache::Run& r = kv->stack->runs[i];
        const size_t bytes = rows * d.row() * dense_size(S.dtype);
        FORGE_CUDA(cudaMalloc(&r.pool, bytes));
        FORGE_CUDA(cudaMemsetAsync(r.pool, 0, bytes, m->stream));
        if (tensor_core_rows(S, d)) FORGE_TRY(latent_cache_map(r.map, r.pool, d, rows));
    }
    kv->stack->splits = row_splits(S, kv->batch, kv->pages_per_seq);
    return FORGE_OK;
}

void stack_cache_destroy(ForgeKV* kv) {
    if (!kv->stack) return;
    for (StackCache::Run& r : kv->stack->runs) if (r.pool) cudaFree(r.pool);
    delete kv->stack;
    kv->stack = nullptr;
}

int32_t stack_kv_read(ForgeKV* kv, int seq, int layer, int which, float* out_host) {
    ForgeModel* m = kv->model;
    const StackModel& S = *m->stack;
    const LatentDims& d = S.spec.layers[layer].mix;
    const int len = kv->len[seq], n = which ? d.rot : d.rank, col = which ? d.rank_p : 0;
    const size_t es = dense_size(S.dtype), row = size_t(d.row()) * es;
    std::vector<uint8_t> page(row * FORGE_KV_PAGE);
    for (int t0 = 0; t0 < len; t0 += FORGE_KV_PAGE) {
        const int pg = kv->h_page_table[size_t(seq) * kv->pages_per_seq + t0 / FORGE_KV_PAGE];
        FORGE_CUDA(cudaMemcpyAsync(page.data(), static_cast<char*>(kv->stack->runs[layer].pool) + size_t(pg) * page.size(), page.size(), cudaMemcpyDeviceToHost, m->stream));
        FORGE_CUDA(cudaStreamSynchronize(m->stream));
        for (int t = t0; t < std::min(len, t0 + FORGE_KV_PAGE); ++t)
            for (int i = 0; i < n; ++i) {
                const uint8_t* p = page.data() + (t - t0) * row + (col + i) * es;
                float& v = out_host[size_t(t) * n + i];
                if (es == 4) memcpy(&v, p, 4);
                else { uint16_t h; memcpy(&h, p, 2); const uint32_t u = uint32_t(h) << 16; memcpy(&v, &u, 4); }
            }
    }
    return FORGE_OK;
}

size_t stack_kv_bytes_per_token(const ForgeKV* kv) {
    const StackModel& S = *kv->model->stack;
    size_t n = 0;
    for (const LayerSpec& L : S.spec.layers) n += L.mix.row();
    return n * dense_size(S.dtype);
}

int32_t stack_kv_copy(ForgeKV* kv, int seq, int len, char* host, bool to_host) {
    ForgeModel* m = kv->model;
    const StackModel& S = *m->stack;
    for (size_t l = 0; l < S.spec.layers.size(); ++l) {
        const size_t row = size_t(S.spec.layers[l].mix.row()) * dense_size(S.dtype);
        for (int t0 = 0; t0 < len; t0 += FORGE_KV_PAGE) {
            const int pg = kv->h_page_table[size_t(seq) * kv->pages_per_seq + t0 / FORGE_KV_PAGE];
            char* dev = static_cast<char*>(kv->stack->runs[l].pool) + size_t(pg) * FORGE_KV_PAGE * row;
            const size_t bytes = row * std::min(FORGE_KV_PAGE, len - t0);
            FORGE_CUDA(to_host ? cudaMemcpyAsync(host, dev, bytes, cudaMemcpyDeviceToHost, m->stream) : cudaMemcpyAsync(dev, host, bytes, cudaMemcpyHostToDevice, m->stream));
            host += bytes;
        }
    }
    FORGE_CUDA(cudaStreamSynchronize(m->stream));
    return FORGE_OK;
}

// ------------------------------------------------------------------------------------------------ steps
int32_t stack_step(ForgeModel* m, ForgeKV* kv, const ForgeStepEntry* entries, int n_entries, const uint32_t* tokens, const int32_t* want, float** d_logits,
                   int trace_rows, int trace_row0) {
    StackModel& S = *m->stack;
    bool prompt_ok = S.dtype == FORGE_BF16;
    for (const LayerSpec& L : S.spec.layers) prompt_ok = prompt_ok && attn_prefill_kv_supported(L.mix);
    // rows: the short entries first, then the prompt portions
    struct Place { int row, tok, want; };
    std::vector<Place> at_entry(n_entries);
    int tok = 0, wants = 0, rows = 0, single = 0, max_pages = 1;
    for (int i = 0; i < n_entries; ++i) { at_entry[i] = {0, tok, wants}; tok += entries[i].n_tokens; wants += entries[i].n_want; }
    auto is_prompt = [&](int i) { return prompt_ok && entries[i].n_tokens >= kPromptRows; };
    for (int pass = 0; pass < 2; ++pass)
        for (int i = 0; i < n_entries; ++i)
            if (is_prompt(i) == (pass == 1)) {
                at_entry[i].row = rows;
                rows += entries[i].n_tokens;
                if (pass == 0) { single = rows; max_pages = std::max(max_pages, (kv->len[entries[i].seq] + entries[i].n_tokens + FORGE_KV_PAGE - 1) / FORGE_KV_PAGE); }
            }
    // one upload: tokens | positions | sequences | wanted rows | context pages | prompt tiles
    std::vector<int32_t> meta(size_t(3) * rows + wants);
    std::vector<int32_t> pages;
    std::vector<PromptTile> tiles;
    for (int i = 0; i < n_entries; ++i) {
        const ForgeStepEntry& e = entries[i];
        const int base = kv->len[e.seq], r0 = at_entry[i].row;
        for (int k = 0; k < e.n_tokens; ++k) {
            meta[r0 + k] = int32_t(tokens[at_entry[i].tok + k]);
            meta[rows + r0 + k] = base + k;
            meta[2 * rows + r0 + k] = e.seq;
        }
        for (int k = 0; k < e.n_want; ++k) meta[3 * rows + at_entry[i].want + k] = r0 + want[at_entry[i].want + k];
        if (is_prompt(i)) {
            const int ctx0 = int(pages.size()) * FORGE_KV_PAGE, np = (base + e.n_tokens + FORGE_KV_PAGE - 1) / FORGE_KV_PAGE;
            for (int p = 0; p < np; ++p) pages.push_back(kv->h_page_table[size_t(e.seq) * kv->pages_per_seq + p]);
            for (int t = 0; t < e.n_tokens; t += 128) tiles.push_back({r0 - single + t, std::min(128, e.n_tokens - t), base + t, ctx0});
        }
    }
    std::stable_sort(tiles.begin(), tiles.end(), [](const PromptTile& a, const PromptTile& b) { return a.pos0 + a.rows > b.pos0 + b.rows; });   // the longest first
    const size_t o_pages = (meta.size() + 3) & ~size_t(3), o_tiles = (o_pages + pages.size() + 3) & ~size_t(3), total = o_tiles + tiles.size() * 4;
    meta.resize(total);
    std::copy(pages.begin(), pages.end(), meta.begin() + o_pages);
    if (!tiles.empty()) memcpy(meta.data() + o_tiles, tiles.data(), tiles.size() * sizeof(PromptTile));
    const int splits = row_splits(S, std::max(1, single), max_pages), ctx_rows = int(pages.size()) * FORGE_KV_PAGE;
    FORGE_TRY(ensure_step(m, std::max(rows, wants), single, splits, rows - single, ctx_rows));
    FORGE_TRY(grow(m, S.meta, total * 4));
    FORGE_TRY(grow(m, S.sel, size_t(wants) * S.width_p * dense_size(S.dtype)));
    FORGE_TRY(grow(m, S.logits, size_t(wants) * S.spec.vocab * 4));
    int32_t* dm = static_cast<int32_t*>(S.meta.p);
    FORGE_CUDA(cudaMemcpyAsync(dm, meta.data(), total * 4, cudaMemcpyHostToDevice, m->stream));
    Step s;
    s.tokens = reinterpret_cast<const uint32_t*>(dm);
    s.rows = StepRows{rows, dm + rows, dm + 2 * rows, kv->d_page_table, kv->pages_per_seq};
    for (int i = 0; i < n_entries; ++i) if (!is_prompt(i)) s.rows.fresh = std::max(s.rows.fresh, int(entries[i].n_tokens));
    s.single = single; s.splits = splits;
    s.ctx_pages = dm + o_pages; s.ctx_rows = ctx_rows;
    s.tiles = reinterpret_cast<const PromptTile*>(dm + o_tiles); s.n_tiles = int(tiles.size());
    if (trace_rows) { s.trace = m->trace + size_t(trace_row0) * S.spec.width; s.trace_stride = size_t(trace_rows) * S.spec.width; }
    FORGE_TRY(run_layers(m, kv, s));
    if (wants) {
        FORGE_TRY(gather_act_rows(S.sel.p, S.h.p, dm + 3 * rows, wants, S.width_p, S.dtype, m->stream));
        FORGE_TRY(run_head(m, S.sel.p, wants, static_cast<float*>(S.logits.p)));
    }
    if (d_logits) *d_logits = static_cast<float*>(S.logits.p);
    FORGE_CUDA(cudaStreamSynchronize(m->stream));   // the host's tables are read by the copy
    return FORGE_OK;
}

int32_t stack_prefill(ForgeModel* m, ForgeKV* kv, int seq, const uint32_t* tokens_host, int n) {
    FORGE_TRY(ensure_decode_scratch(m, 1));
    if (m->trace_on) FORGE_TRY(ensure_trace(m, n));
    const int len0 = kv->len[seq];
    int32_t rc = FORGE_OK;
    for (int t = 0; t < n && rc == FORGE_OK; t += kPortion) {
        const int k = std::min(kPortion, n - t), place = k - 1;
        const bool last = t + k == n;
        const ForgeStepEntry e{seq, k, last ? 1 : 0};
        float* lg = nullptr;
        rc = stack_step(m, kv, &e, 1, tokens_host + t, &place, &lg, m->trace_on ? n : 0, t);
        if (rc == FORGE_OK && last && cudaMemcpyAsync(m->d_logits, lg, sizeof(float) * m->V, cudaMemcpyDeviceToDevice, m->stream) != cudaSuccess) { set_error("logits copy failed"); rc = FORGE_ERR_CUDA; }
        if (rc == FORGE_OK) kv->len[seq] += k;
    }
    if (rc != FORGE_OK) kv->len[seq] = len0;
    return rc;
}

int32_t stack_ensure_decode(ForgeModel* m, ForgeKV* kv, int batch) { return ensure_step(m, batch, batch, kv->stack->splits, 0, 0); }

int32_t stack_decode_launches(ForgeModel* m, ForgeKV* kv, int batch, bool greedy, bool record) {
    StackModel& S = *m->stack;
    Step s;
    s.tokens = m->d_tok;
    s.rows = StepRows{batch, kv->d_seq_len, nullptr, kv->d_page_table, kv->pages_per_seq};
    s.single = batch; s.splits = kv->stack->splits;
    if (record) { s.hist = m->d_hist; s.step = m->d_step; }
    if (m->trace_on) { s.trace = m->trace; s.trace_stride = size_t(batch) * S.spec.width; }
    FORGE_TRY(run_layers(m, kv, s));
    FORGE_TRY(run_head(m, S.h.p, batch, m->d_logits));
    if (greedy) FORGE_TRY(argmax_slices(m->d_tok, m->d_logits, m->V, batch, m->d_amax_val, m->d_amax_idx, m->d_amax_ticket, m->stream));
    return step_advance(kv->d_seq_len, batch, m->d_step, m->stream);
}

}  // namespace forge

// ------------------------------------------------------------------------------------------------ C API
extern "C" {

int32_t forge_checkpoint_info(const char* dir, ForgeCheckpointInfo* out) {
    if (!dir || !out) { set_error("bad argument to forge_checkpoint_info"); return FORGE_ERR_INVALID_ARG; }
    Checkpoint ck;
    StackSpec s;
    StackTensors t;
    FORGE_TRY(ck.open(dir));
    FORGE_TRY(parse_spec(ck.config(), &s));
    FORGE_TRY(find_tensors(ck, s, &t));
    s.parameters = ck.parameters();
    fill_info(s, out);
    return FORGE_OK;
}

int32_t forge_model_info(const ForgeModel* m, ForgeCheckpointInfo* out) {
    if (!m || !out) { set_error("bad argument to forge_model_info"); return FORGE_ERR_INVALID_ARG; }
    if (!m->stack) { set_error("not a layer-list model"); return FORGE_ERR_UNSUPPORTED; }
    fill_info(m->stack->spec, out);
    return FORGE_OK;
}

int32_t forge_model_open(const char* dir, int32_t dtype, int32_t device, ForgeModel** out) {
    if (!dir || !out) { set_error("bad argument to forge_model_open"); return FORGE_ERR_INVALID_ARG; }
    *out = nullptr;
    if (dtype != FORGE_BF16 && dtype != FORGE_F32) { set_error("a layer-list model runs in FORGE_BF16 or FORGE_F32"); return FORGE_ERR_INVALID_ARG; }
    Checkpoint ck;
    StackSpec spec;
    StackTensors t;
    FORGE_TRY(ck.open(dir));
    FORGE_TRY(parse_spec(ck.config(), &spec));
    FORGE_TRY(find_tensors(ck, spec, &t));
    spec.parameters = ck.parameters();
    const int ndev = forge_device_count();
    if (ndev == 0) { set_error("no CUDA device: this backend has no CPU fallback"); return FORGE_ERR_CUDA; }
    if (device < 0 || device >= ndev) { set_error("device %d out of range (%d visible)", device, ndev); return FORGE_ERR_INVALID_ARG; }
    FORGE_CUDA(cudaSetDevice(device));
    ForgeModel* m = new ForgeModel();
    m->cfg = ForgeModelConfig{};
    m->cfg.hidden_size = spec.width; m->cfg.num_layers = int32_t(spec.layers.size()); m->cfg.vocab_size = spec.vocab;
    m->cfg.max_seq_len = 1 << 20; m->cfg.tp_world = 1; m->cfg.quant = dtype;
    m->device = device; m->h = spec.width; m->V = spec.vocab; m->max_seq = 1 << 20;
    m->uniform_basic = false;
    m->stack = new StackModel();
    StackModel& S = *m->stack;
    S.spec = spec; S.dtype = dtype; S.width_p = pad_to(spec.width, kDensePad);
    auto build = [&]() -> int32_t {
        FORGE_CUDA(cudaStreamCreateWithFlags(&m->stream, cudaStreamNonBlocking));
        for (auto& e : m->ev) FORGE_CUDA(cudaEventCreate(&e));
        FORGE_TRY(dev_alloc(m, &m->d_err, 1));
        FORGE_CUDA(cudaMemsetAsync(m->d_err, 0, sizeof(int), m->stream));
        FORGE_TRY(dev_alloc(m, &S.scratch.part, kDensePartFloats));
        const size_t es = dense_size(dtype);
        {
            std::vector<uint8_t> img(size_t(spec.vocab) * spec.width * es);
            put_rows(img, dtype, spec.width, *t.embed, 0);
            FORGE_TRY(upload(m, &S.embed, img));
        }
        {
            std::vector<uint8_t> img(size_t(spec.vocab) * S.width_p * es, 0);
            put_rows(img, dtype, S.width_p, *t.head, 0);
            FORGE_TRY(load_dense(m, &S.head, spec.vocab, S.width_p, dtype, img));
        }
        FORGE_TRY(load_dyt(m, &S.final_norm, *t.fn, *t.fb, *t.fa));
        S.w.resize(spec.layers.size());
        for (size_t i = 0; i < spec.layers.size(); ++i)
            if (spec.layers[i].weights_of < 0) FORGE_TRY(load_layer(m, spec.layers[i], t.layers[i], &S.w[i]));
        return FORGE_OK;
    };
    const int32_t rc = build();
    if (rc != FORGE_OK) { forge_model_destroy(m); return rc; }
    *out = m;
    return FORGE_OK;
}

}  // extern "C"
