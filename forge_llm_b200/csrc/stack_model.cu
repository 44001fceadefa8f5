// Layer-list models: loader, cache and state, launch sequences.  The session calls (model.cu) - cache, prompt, decode graph, greedy
// loop, sampling, mixed steps - take such a model like a quantised decoder.
//
// A sublayer is a dense product of its normed input (all projections of a mixer in one), the mechanism, and a dense product
// whose epilogue adds the residual and leaves what the next reader of the stream takes (After): its norm, or the stream itself where a
// pass of the loop begins with a product.
//   parallel arrangement   the `in` product also holds the feed-forward's rows, and `out` runs over the concatenated columns
//                          [o | down] of [gated heads | activation], so both sublayers are summed by the product itself;
//   delta rules            in [q k v | gate | beta | decay] (a second product for two-step gates and decays), recurrence, out;
//   two parallel norms     the input's columns are [x (1 + w1) | x (1 + w2)], the RMS of the stream is a factor of the product's epilogue; the mixer's rows
//                          read the first block, the feed-forward's the second; experts: see experts();
//   norms on outputs       the stream itself, in the model's type, is every product's input; the sublayer's sum is left as f32 rows, and one
//                          kernel norms it, adds it and leaves the stream's next form; experts beside a shared one: see mixture();
//   attention | scan       one `in` product for both, the convolution's projections, one `out` product over [heads | channels] whose
//                          columns carry the two factors already;
//   attention | time mix   the input's columns are [h | five shifted mixes] and every row of `in` reads the block it belongs to; keys
//                          and values go from the epilogue into the cache; one product with both outputs, then the sum of their norms.
#include <algorithm>
#include <cmath>
#include <cstring>
#include <map>
#include <memory>

#include "model.cuh"
#include "stack.cuh"

// ------------------------------------------------------------------------------------------------ structures
namespace forge {

struct StreamNorm { float* w = nullptr; float* b = nullptr; float alpha = 0.f; };   // RMS norm: w = one plus the weight, or alpha (and in w) the one for all columns

struct LayerWeights {
    StreamNorm norm1, norm2;
    DenseWeight in, out;
    DenseWeight ff_in, ff_out;    // sequential arrangement; norms on outputs: [router | shared], [shared | expert 0 | expert 1 ...]
    // latent attention
    DenseWeight kv;               // rows [uk | uv] over the latent
    int q_rows = 0, dkv_row = 0, g_row = 0, glu_row = 0, uv_row = 0;   // first rows of the segments of `in` / `kv`
    int heads_k = 0;              // columns of `out` in front of the feed-forward's
    float* kv_norm = nullptr;
    // recurrent mixers
    int gate_row = 0, beta_row = 0, decay_row = 0, low_gate_row = 0;   // first rows of the segments of `in`
    int decay_k = 0;              // columns of the decay's inner values in front of the gate's
    int low_row = 0;              // first row of the gate in `low`
    DenseWeight low;              // second step of decay [and gate]
    float *conv = nullptr, *decay_mul = nullptr, *decay_add = nullptr, *bonus = nullptr, *head_norm = nullptr;
    // attention beside time mixing
    int k_row = 0, v_row = 0, hg_row = 0, r_row = 0, rk_row = 0, rv_row = 0;
    int out_r_row = 0;            // first row of the second mixer in `out`; it reads the columns behind the first one's
    float *mu = nullptr, *norm_l = nullptr, *norm_r = nullptr;
    // attention with normed queries and keys (k_row, v_row as above)
    float *q_norm = nullptr, *k_norm = nullptr, *sink = nullptr, *q_bias = nullptr, *k_bias = nullptr, *v_bias = nullptr;
    float bias_bound = 0.f;       // largest bias by distance
    float *bias = nullptr, *talk = nullptr, *out_bias = nullptr, lambda = 0.f;   // biases by distance, mixing of heads, share of the blended values
    // selective scan (in_row, gate_row: first rows in `in`; conv, low as above): rows [step sizes' inner values | B C] over the channels
    DenseWeight scan_in;
    int in_row = 0, bc_row = 0;
    float *conv_add = nullptr, *scan_a = nullptr, *skip = nullptr, *minus = nullptr;
    // experts: their columns of `out` follow the heads', ff_k apart
    int router_row = 0, ff_k = 0;
    float* router_bias = nullptr;
    DenseWeight experts;          // gate and up rows, pairs interleaved, group by group expert_rows apart (norms on outputs: those of the shared expert's pieces first)
    void* router = nullptr;       // its rows
    int expert_rows = 0;
};

struct StackModel {
    StackSpec spec;
    int dtype = FORGE_BF16;
    int width_p = 0;
    void *embed = nullptr, *bigram = nullptr;
    std::vector<LayerWeights> w;                       // by layer; empty for a layer with weights_of
    StreamNorm final_norm;
    DenseWeight head, loop_in;
    float* loop_step = nullptr;                        // [times][width]
    std::map<Rotation, std::pair<int, float*>> ropes;   // -> positions, table
    int rope_positions = 0;
    DenseScratch scratch;
    // step buffers, grown on demand (scratch_gen of the model counts the moves)
    struct Buf { void* p = nullptr; size_t cap = 0; };
    Buf x, h, cat, proj, gate, mid, q, part, ml, ctx_c, ctx_r, ctx_k, ctx_v, hgate, decay, beta, low, conv, unit, o, pair, place, c_half, c_f32, sel, logits, meta, x0, sums, sum1, router, route, e_in, e_act, e_out, scores, joint, blocks, scan, bc;
    std::vector<Buf*> all() {
        return {&x, &h, &cat, &proj, &gate, &mid, &q, &part, &ml, &ctx_c, &ctx_r, &ctx_k, &ctx_v, &hgate, &decay, &beta, &low, &conv, &unit, &o, &pair, &place, &c_half, &c_f32, &sel, &logits, &meta,
                &x0, &sums, &sum1, &router, &route, &e_in, &e_act, &e_out, &scores, &joint, &blocks, &scan, &bc};
    }
    bool rms_stream() const { return spec.arch->norm == Norm::RmsPlusOne; }      // every reader of the stream takes an RMS norm of it
    bool rms_final() const { return spec.arch->norm != Norm::DynamicTanh; }
    const LayerWeights& weights(int layer) const { return w[spec.layers[layer].weights_of >= 0 ? spec.layers[layer].weights_of : layer]; }
};

// What a layer run keeps: cache rows in pages of the pool, [pages][FORGE_KV_PAGE][row] of the model's type, and per sequence a
// recurrent state (f32), the last inputs of its convolution and the last row of its token shift (the model's type).
struct StackCache {
    struct Run { void* pool = nullptr; alignas(64) unsigned char map[128]; float* state = nullptr; void* ring = nullptr; void* prev = nullptr; };
    std::vector<Run> runs;
    int splits = 1;     // of a captured decode step
    uint32_t* prev_token = nullptr;   // by sequence: its last token (bigram embeddings)
};

namespace {

// ------------------------------------------------------------------------------------------------ loading
void store(void* dst, int dtype, size_t i, const TensorView& t, size_t j) {
    if (dtype == FORGE_F32) { static_cast<float*>(dst)[i] = t.at(j); return; }
    if (t.dtype == "BF16") { memcpy(static_cast<uint16_t*>(dst) + i, t.data + 2 * j, 2); return; }
    static_cast<__nv_bfloat16*>(dst)[i] = __float2bfloat16_rn(t.at(j));
}
// rows [from, from + count) of `t` [n][k] (count < 0: all) into the host image of a matrix with rows of `ld`: row r -> row0 + (r - from) * step, columns from col0
void put_rows(std::vector<uint8_t>& img, int dtype, int ld, const TensorView& t, int row0, int step = 1, int col0 = 0, int from = 0, int count = -1) {
    const int64_t n = count < 0 ? t.shape[0] : from + count, k = t.shape[1];
    for (int64_t r = from; r < n; ++r) {
        const size_t at = size_t(row0 + (r - from) * step) * ld + col0;
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

int32_t upload_values(ForgeModel* m, float** dst, const std::vector<float>& v) {
    FORGE_TRY(dev_alloc(m, dst, v.size()));
    FORGE_CUDA(cudaMemcpyAsync(*dst, v.data(), v.size() * 4, cudaMemcpyHostToDevice, m->stream));
    FORGE_CUDA(cudaStreamSynchronize(m->stream));
    return FORGE_OK;
}

// the host image of a matrix of N rows and K (padded) columns, filled piece by piece
struct Image {
    std::vector<uint8_t> img;
    int N, K, dtype;
    Image(int n, int k, int dt) : img(size_t(n) * k * dense_size(dt), 0), N(n), K(k), dtype(dt) {}
    void put(const TensorView* t, int row0, int step = 1, int col0 = 0, int from = 0, int count = -1) { put_rows(img, dtype, K, *t, row0, step, col0, from, count); }
    // columns [from, from + count) of all rows of `t` to columns from col0
    void put_columns(const TensorView* t, int from, int count, int col0) {
        const int64_t k = t->shape[1];
        for (int64_t r = 0; r < t->shape[0]; ++r)
            for (int c = 0; c < count; ++c) store(img.data(), dtype, size_t(r) * K + col0 + c, *t, size_t(r * k + from + c));
    }
    int32_t load(ForgeModel* m, DenseWeight* w, bool row_reads = false) const { return load_dense(m, w, N, K, dtype, img, row_reads); }
};

int32_t load_norm(ForgeModel* m, StreamNorm* n, const TensorSet& t, const std::string& name) {
    if (m->stack->spec.arch->norm == Norm::RmsPlusOne) {
        std::vector<float> w(size_t(t.at(name)->count()));
        for (size_t i = 0; i < w.size(); ++i) w[i] = 1.f + t.at(name)->at(i);
        return upload_values(m, &n->w, w);
    }
    if (m->stack->spec.arch->norm == Norm::RmsScalar) {
        n->alpha = t.at(name)->at(0);
        return upload_values(m, &n->w, std::vector<float>(size_t(m->stack->spec.width), n->alpha));
    }
    n->alpha = t.at(name + ".alpha")->at(0);
    FORGE_TRY(upload_f32(m, &n->w, *t.at(name)));
    return upload_f32(m, &n->b, *t.at(name + ".b"));
}

int32_t load_latent(ForgeModel* m, const LayerSpec& L, const TensorSet& t, LayerWeights* w) {
    StackModel& S = *m->stack;
    const LatentDims& d = L.mix;
    const int ff = S.spec.arch->arrangement == Arrangement::Parallel ? L.ff : 0;
    FORGE_TRY(upload_f32(m, &w->kv_norm, *t.at("mix.dkv.norm")));
    w->q_rows = d.heads * (d.dim + d.rot);
    w->dkv_row = pad_to(w->q_rows, kSegAlign);
    w->g_row = w->dkv_row + pad_to(d.rank + d.rot, kSegAlign);
    w->glu_row = w->g_row + pad_to(d.heads * d.vdim, kSegAlign);
    Image in(w->glu_row + 2 * ff, S.width_p, S.dtype);
    in.put(t.at("mix.q"), 0);
    in.put(t.at("mix.dkv"), w->dkv_row);
    in.put(t.at("mix.g"), w->g_row);
    if (ff) { in.put(t.at("mlp.gate"), w->glu_row, 2); in.put(t.at("mlp.up"), w->glu_row + 1, 2); }
    FORGE_TRY(in.load(m, &w->in));
    w->uv_row = pad_to(d.heads * d.dim, kSegAlign);
    Image kv(w->uv_row + d.heads * d.vdim, d.rank_p, S.dtype);
    kv.put(t.at("mix.uk"), 0);
    kv.put(t.at("mix.uv"), w->uv_row);
    FORGE_TRY(kv.load(m, &w->kv, true));
    w->heads_k = pad_to(d.heads * d.vdim, kDensePad);
    Image out(S.spec.width, w->heads_k + pad_to(ff, kDensePad), S.dtype);
    out.put(t.at("mix.o"), 0);
    if (ff) out.put(t.at("mlp.down"), 0, 1, w->heads_k);
    return out.load(m, &w->out);
}

int32_t load_delta(ForgeModel* m, const LayerSpec& L, const TensorSet& t, LayerWeights* w) {
    StackModel& S = *m->stack;
    const RecurDims& d = L.rec;
    const int H = d.heads, HV = d.heads * d.vdim;
    {
        std::vector<float> conv;   // [taps][channels]
        for (int j = 0; j < d.taps; ++j)
            for (const char* n : {"mix.q.conv", "mix.k.conv", "mix.v.conv"})
                for (int64_t c = 0; c < t.at(n)->shape[0]; ++c) conv.push_back(t.at(n)->at(size_t(c * d.taps + j)));
        FORGE_TRY(upload_values(m, &w->conv, conv));
        // a decay's logarithm is -exp(A_log of the head) softplus(its row's value + dt_bias)
        const int per = d.channel ? d.dim : 1;
        std::vector<float> mul(size_t(H) * per);
        for (int h = 0; h < H; ++h) for (int i = 0; i < per; ++i) mul[size_t(h) * per + i] = float(std::exp(double(t.at("mix.A_log")->at(h))));
        FORGE_TRY(upload_values(m, &w->decay_mul, mul));
        FORGE_TRY(upload_f32(m, &w->decay_add, *t.at("mix.dt_bias")));
        FORGE_TRY(upload_f32(m, &w->head_norm, *t.at("mix.norm")));
    }
    int row = pad_to(d.channels(), kSegAlign);
    auto take = [&](int rows) { const int at = row; row += pad_to(rows, kSegAlign); return at; };
    if (d.channel) {
        w->beta_row = take(H); w->decay_row = take(L.decay_rank); w->low_gate_row = take(L.gate_rank);
    } else {
        w->gate_row = take(HV); w->beta_row = take(H); w->decay_row = take(H);
    }
    Image in(row, S.width_p, S.dtype);
    in.put(t.at("mix.q"), 0); in.put(t.at("mix.k"), d.qk()); in.put(t.at("mix.v"), 2 * d.qk());
    in.put(t.at("mix.b"), w->beta_row);
    if (d.channel) {
        in.put(t.at("mix.a1"), w->decay_row); in.put(t.at("mix.g1"), w->low_gate_row);
        // rows [a2 | g2]; each reads its own block of the inner values, K is the wider of the two
        w->decay_k = pad_to(L.decay_rank, kDensePad);
        w->low_row = pad_to(H * d.dim, 128);
        Image low(w->low_row + HV, std::max(w->decay_k, pad_to(L.gate_rank, kDensePad)), S.dtype);
        low.put(t.at("mix.a2"), 0);
        low.put(t.at("mix.g2"), w->low_row);
        FORGE_TRY(low.load(m, &w->low, true));
    } else {
        in.put(t.at("mix.g"), w->gate_row); in.put(t.at("mix.a"), w->decay_row);
    }
    FORGE_TRY(in.load(m, &w->in));
    Image out(S.spec.width, pad_to(HV, kDensePad), S.dtype);
    out.put(t.at("mix.o"), 0);
    return out.load(m, &w->out);
}

constexpr int kMixes = 5;   // r, k, v, g, w

int32_t load_pair(ForgeModel* m, const LayerSpec& L, const TensorSet& t, LayerWeights* w) {
    StackModel& S = *m->stack;
    const AttnDims& a = L.attn;
    const RecurDims& d = L.rec;
    const int D = d.heads * d.dim;
    int row = 0;
    auto take = [&](int rows, int align) { row = pad_to(row, align); const int at = row; row += rows; return at; };
    const int q_row = take(a.heads * a.dim, kSegAlign);
    w->k_row = take(a.groups * a.dim, kSegAlign); w->v_row = take(a.groups * a.vdim, kSegAlign); w->hg_row = take(a.heads, kSegAlign);
    // a tile of rows reads one block of the activations
    w->r_row = take(D, 128); w->rk_row = take(D, 128); w->rv_row = take(D, 128); w->gate_row = take(D, 128); w->decay_row = take(L.decay_rank, 128);
    Image in(row, S.width_p, S.dtype);
    in.put(t.at("mix.left.q"), q_row); in.put(t.at("mix.left.k"), w->k_row); in.put(t.at("mix.left.v"), w->v_row); in.put(t.at("mix.left.g"), w->hg_row);
    in.put(t.at("mix.right.r"), w->r_row); in.put(t.at("mix.right.k"), w->rk_row); in.put(t.at("mix.right.v"), w->rv_row);
    in.put(t.at("mix.right.g"), w->gate_row); in.put(t.at("mix.right.w1"), w->decay_row);
    FORGE_TRY(in.load(m, &w->in));
    Image low(D, pad_to(L.decay_rank, kDensePad), S.dtype);
    low.put(t.at("mix.right.w2"), 0);
    FORGE_TRY(low.load(m, &w->low, true));
    w->out_r_row = pad_to(S.spec.width, 128);
    Image out(w->out_r_row + S.spec.width, pad_to(std::max(a.heads * a.vdim, D), kDensePad), S.dtype);
    out.put(t.at("mix.left.o"), 0);
    out.put(t.at("mix.right.o"), w->out_r_row);
    FORGE_TRY(out.load(m, &w->out));
    std::vector<float> mu;
    for (const char* n : {"r", "k", "v", "g", "w"}) { const TensorView* v = t.at(std::string("mix.right.mu.") + n); for (int i = 0; i < S.spec.width; ++i) mu.push_back(v->at(size_t(i))); }
    FORGE_TRY(upload_values(m, &w->mu, mu));
    FORGE_TRY(upload_f32(m, &w->decay_add, *t.at("mix.right.w0")));
    FORGE_TRY(upload_f32(m, &w->bonus, *t.at("mix.right.u")));
    FORGE_TRY(upload_f32(m, &w->head_norm, *t.at("mix.right.norm")));
    FORGE_TRY(upload_f32(m, &w->norm_l, *t.at("mix.left.out")));
    return upload_f32(m, &w->norm_r, *t.at("mix.right.out"));
}

// Side by side behind two norms: the feed-forward's rows of `in` (or the router's) behind the mixer's `rows`, and `out` over [heads | feed-forward].
// fill_in puts the mixer's rows.
template <typename F>
int32_t load_two_norms(ForgeModel* m, const LayerSpec& L, const TensorSet& t, LayerWeights* w, int rows, int heads_cols, F fill_in) {
    StackModel& S = *m->stack;
    const int E = L.router.experts;
    w->glu_row = w->router_row = pad_to(rows, 128);   // a tile of rows reads one block of the activations
    Image in(E ? w->router_row + E : L.ff ? w->glu_row + 2 * L.ff : rows, S.width_p, S.dtype);
    fill_in(in);
    if (E) in.put(t.at("mlp.router"), w->router_row);
    else if (L.ff) { in.put(t.at("mlp.gate"), w->glu_row, 2); in.put(t.at("mlp.up"), w->glu_row + 1, 2); }
    FORGE_TRY(in.load(m, &w->in));
    w->heads_k = pad_to(heads_cols, kDensePad);
    w->ff_k = pad_to(L.ff, kDensePad);
    Image out(S.spec.width, w->heads_k + std::max(1, E) * w->ff_k, S.dtype);
    out.put(t.at("mix.o"), 0);
    if (E) {
        FORGE_TRY(upload_f32(m, &w->router_bias, *t.at("mlp.router.b")));
        w->expert_rows = pad_to(2 * L.ff, 128);
        Image ex(E * w->expert_rows, S.width_p, S.dtype);
        for (int e = 0; e < E; ++e) {
            const std::string x = "mlp.e" + std::to_string(e);
            ex.put(t.at(x + ".gate"), e * w->expert_rows, 2);
            ex.put(t.at(x + ".up"), e * w->expert_rows + 1, 2);
            out.put(t.at(x + ".down"), 0, 1, w->heads_k + e * w->ff_k);
        }
        FORGE_TRY(ex.load(m, &w->experts));
    } else if (L.ff) out.put(t.at("mlp.down"), 0, 1, w->heads_k);
    return out.load(m, &w->out);
}

int32_t load_softmax(ForgeModel* m, const LayerSpec& L, const TensorSet& t, LayerWeights* w) {
    const AttnDims& a = L.attn;
    w->k_row = pad_to(a.heads * a.dim, kSegAlign);
    w->v_row = w->k_row + pad_to(a.groups * a.dim, kSegAlign);
    FORGE_TRY(upload_f32(m, &w->q_norm, *t.at("mix.q.norm")));
    FORGE_TRY(upload_f32(m, &w->k_norm, *t.at("mix.k.norm")));
    if (L.soft.sink) FORGE_TRY(upload_f32(m, &w->sink, *t.at("mix.sink")));
    else FORGE_TRY(upload_values(m, &w->sink, std::vector<float>(size_t(a.heads), 0.f)));
    if (L.soft.bias) {
        FORGE_TRY(upload_f32(m, &w->q_bias, *t.at("mix.q.b")));
        FORGE_TRY(upload_f32(m, &w->k_bias, *t.at("mix.k.b")));
        FORGE_TRY(upload_f32(m, &w->v_bias, *t.at("mix.v.b")));
    }
    return load_two_norms(m, L, t, w, w->v_row + a.groups * a.vdim, a.heads * a.vdim, [&](Image& in) {
        in.put(t.at("mix.q"), 0); in.put(t.at("mix.k"), w->k_row); in.put(t.at("mix.v"), w->v_row);
    });
}

// What the mechanisms of an attention behind `at` need besides its matrices; norms of queries and keys without weights.
int32_t load_plain_attention(ForgeModel* m, const LayerSpec& L, const TensorSet& t, LayerWeights* w, const std::string& at, float factor) {
    const AttnDims& a = L.attn;
    const std::vector<float> ones(size_t(a.dim), 1.f);
    FORGE_TRY(upload_values(m, &w->q_norm, ones));
    w->k_norm = w->q_norm;
    FORGE_TRY(upload_f32(m, &w->q_bias, *t.at(at + "q.b")));
    FORGE_TRY(upload_f32(m, &w->k_bias, *t.at(at + "k.b")));
    FORGE_TRY(upload_f32(m, &w->v_bias, *t.at(at + "v.b")));
    std::vector<float> ob;
    for (int64_t i = 0; i < t.at(at + "o.b")->count(); ++i) ob.push_back(factor * t.at(at + "o.b")->at(size_t(i)));
    FORGE_TRY(upload_values(m, &w->out_bias, ob));
    if (L.soft.sink) FORGE_TRY(upload_f32(m, &w->sink, *t.at(at + "sink")));
    if (L.soft.talk) FORGE_TRY(upload_f32(m, &w->talk, *t.at(at + "talk")));
    if (L.soft.distance) {
        std::vector<float> by;   // [head][distance]
        for (int h = 0; h < a.heads; ++h)
            for (int n = 0; n < a.bias_n; ++n) by.push_back(t.at(at + "rel")->at(size_t(L.distance.of(n)) * a.heads + h));
        for (float b : by) w->bias_bound = std::max(w->bias_bound, std::fabs(b));
        FORGE_TRY(upload_values(m, &w->bias, by));
    }
    if (L.blend_layer >= 0) w->lambda = t.at(at + "vmix")->at(0);
    return FORGE_OK;
}

int32_t load_post_softmax(ForgeModel* m, const LayerSpec& L, const TensorSet& t, LayerWeights* w) {
    StackModel& S = *m->stack;
    const AttnDims& a = L.attn;
    FORGE_TRY(load_plain_attention(m, L, t, w, "mix.", 1.f));
    w->k_row = pad_to(a.heads * a.dim, kSegAlign);
    w->v_row = w->k_row + pad_to(a.groups * a.dim, kSegAlign);
    Image in(w->v_row + a.groups * a.vdim, S.width_p, S.dtype), out(S.spec.width, pad_to(a.heads * a.vdim, kDensePad), S.dtype);
    in.put(t.at("mix.q"), 0); in.put(t.at("mix.k"), w->k_row); in.put(t.at("mix.v"), w->v_row);
    out.put(t.at("mix.o"), 0);
    FORGE_TRY(in.load(m, &w->in));
    return out.load(m, &w->out);
}

int32_t load_attn_selective(ForgeModel* m, const LayerSpec& L, const TensorSet& t, LayerWeights* w) {
    StackModel& S = *m->stack;
    const AttnDims& a = L.attn;
    const SelectiveDims& d = L.sel;
    FORGE_TRY(load_plain_attention(m, L, t, w, "mix.left.", L.left_scale));
    w->k_row = pad_to(a.heads * a.dim, kSegAlign);
    w->v_row = w->k_row + pad_to(a.groups * a.dim, kSegAlign);
    w->in_row = w->v_row + pad_to(a.groups * a.vdim, kSegAlign);
    w->gate_row = w->in_row + pad_to(d.inner, kSegAlign);
    Image in(w->gate_row + d.inner, S.width_p, S.dtype);
    in.put(t.at("mix.left.q"), 0); in.put(t.at("mix.left.k"), w->k_row); in.put(t.at("mix.left.v"), w->v_row);
    in.put(t.at("mix.right.in"), w->in_row, 1, 0, 0, d.inner);
    in.put(t.at("mix.right.in"), w->gate_row, 1, 0, d.inner, d.inner);
    FORGE_TRY(in.load(m, &w->in));
    const int inner_p = pad_to(d.inner, kDensePad);
    w->bc_row = pad_to(d.rank, kSegAlign);
    Image x(w->bc_row + 2 * d.state, inner_p, S.dtype);
    x.put(t.at("mix.right.x"), 0, 1, 0, 0, d.rank);
    x.put(t.at("mix.right.x"), w->bc_row, 1, 0, d.rank, 2 * d.state);
    FORGE_TRY(x.load(m, &w->scan_in));
    Image low(d.inner, pad_to(d.rank, kDensePad), S.dtype);
    low.put(t.at("mix.right.dt"), 0);
    FORGE_TRY(low.load(m, &w->low, true));
    w->heads_k = pad_to(a.heads * a.vdim, kDensePad);
    Image out(S.spec.width, w->heads_k + inner_p, S.dtype);
    out.put(t.at("mix.left.o"), 0);
    out.put(t.at("mix.right.o"), 0, 1, w->heads_k);
    FORGE_TRY(out.load(m, &w->out));
    std::vector<float> conv, a2;   // [taps][channels]; decays are exp2(step size * a2)
    for (int j = 0; j < d.taps; ++j) for (int c = 0; c < d.inner; ++c) conv.push_back(t.at("mix.right.conv")->at(size_t(c) * d.taps + j));
    for (size_t i = 0; i < d.state_values(); ++i) a2.push_back(float(-std::exp(double(t.at("mix.right.A_log")->at(i))) / std::log(2.0)));
    FORGE_TRY(upload_values(m, &w->conv, conv));
    FORGE_TRY(upload_values(m, &w->scan_a, a2));
    FORGE_TRY(upload_values(m, &w->minus, std::vector<float>(size_t(d.inner), -1.f)));
    FORGE_TRY(upload_f32(m, &w->conv_add, *t.at("mix.right.conv.b")));
    FORGE_TRY(upload_f32(m, &w->decay_add, *t.at("mix.right.dt.b")));
    return upload_f32(m, &w->skip, *t.at("mix.right.D"));
}

// A mixture beside a shared expert: [router | shared gate, up | experts' gate, up] and, over [shared | expert 0 | expert 1 ...], the way back.
int32_t load_mixture(ForgeModel* m, const LayerSpec& L, const TensorSet& t, LayerWeights* w) {
    StackModel& S = *m->stack;
    const int E = L.router.experts, A = L.router.always;
    w->ff_k = pad_to(L.ff, kDensePad);
    w->expert_rows = pad_to(2 * L.ff, 128);
    w->glu_row = pad_to(L.router.choices(), 128);
    Image in(w->glu_row + (A + E) * w->expert_rows, S.width_p, S.dtype), out(S.spec.width, (A + E) * w->ff_k, S.dtype), router(L.router.choices(), S.width_p, S.dtype);
    in.put(t.at("mlp.router"), 0);
    router.put(t.at("mlp.router"), 0);
    FORGE_TRY(upload(m, &w->router, router.img));
    for (int a = 0; a < A; ++a) {   // a piece of the shared expert has as many rows as an expert
        const int from = a * L.ff, n = std::min(L.ff, L.shared_ff - from), row = w->glu_row + a * w->expert_rows;
        in.put(t.at("mlp.shared.gate"), row, 2, 0, from, n);
        in.put(t.at("mlp.shared.up"), row + 1, 2, 0, from, n);
        out.put_columns(t.at("mlp.shared.down"), from, n, a * w->ff_k);
    }
    for (int e = 0; e < E; ++e) {
        const std::string x = "mlp.e" + std::to_string(e);
        const int row = w->glu_row + (A + e) * w->expert_rows;
        in.put(t.at(x + ".gate"), row, 2);
        in.put(t.at(x + ".up"), row + 1, 2);
        out.put(t.at(x + ".down"), 0, 1, (A + e) * w->ff_k);
    }
    FORGE_TRY(in.load(m, &w->ff_in));
    w->experts = w->ff_in.rows(w->glu_row, (A + E) * w->expert_rows);
    w->ff_in = w->ff_in.rows(0, w->glu_row + A * w->expert_rows);
    FORGE_TRY(out.load(m, &w->ff_out));
    return upload_f32(m, &w->router_bias, *t.at("mlp.correction"));
}

int32_t load_linear(ForgeModel* m, const LayerSpec& L, const TensorSet& t, LayerWeights* w) {
    StackModel& S = *m->stack;
    const RecurDims& d = L.rec;
    const int D = d.qk(), HV = d.heads * d.vdim;
    // the logarithm of a decay, log(sigmoid(z)) / tau, is -softplus(-z) / tau: the second step and its bias are kept negated
    std::vector<float> bias(size_t(D), 0.f);
    for (int i = 0; i < D; ++i) bias[i] = -t.at("mix.a2.b")->at(size_t(i));
    FORGE_TRY(upload_values(m, &w->decay_add, bias));
    FORGE_TRY(upload_values(m, &w->decay_mul, std::vector<float>(size_t(D), float(1.0 / L.tau))));
    FORGE_TRY(upload_f32(m, &w->head_norm, *t.at("mix.norm")));
    Image low(D, pad_to(L.decay_rank, kDensePad), S.dtype);
    low.put(t.at("mix.a2"), 0);
    for (size_t i = dense_size(S.dtype) - 1; i < low.img.size(); i += dense_size(S.dtype)) low.img[i] ^= 0x80;   // sign bits
    FORGE_TRY(low.load(m, &w->low, true));
    w->gate_row = pad_to(d.channels(), kSegAlign);
    w->decay_row = w->gate_row + pad_to(HV, kSegAlign);
    return load_two_norms(m, L, t, w, w->decay_row + L.decay_rank, HV, [&](Image& in) {
        in.put(t.at("mix.q"), 0); in.put(t.at("mix.k"), D); in.put(t.at("mix.v"), 2 * D);
        in.put(t.at("mix.g"), w->gate_row); in.put(t.at("mix.a1"), w->decay_row);
    });
}

int32_t load_layer(ForgeModel* m, const LayerSpec& L, const TensorSet& t, LayerWeights* w) {
    StackModel& S = *m->stack;
    const bool post = S.spec.arch->arrangement == Arrangement::PostNorm;
    FORGE_TRY(load_norm(m, &w->norm1, t, "norm1"));
    switch (L.kind) {
        case Mixer::Latent: FORGE_TRY(load_latent(m, L, t, w)); break;
        case Mixer::Delta: case Mixer::ChannelDelta: FORGE_TRY(load_delta(m, L, t, w)); break;
        case Mixer::AttnTimeMix: FORGE_TRY(load_pair(m, L, t, w)); break;
        case Mixer::Softmax: FORGE_TRY(post ? load_post_softmax(m, L, t, w) : load_softmax(m, L, t, w)); break;
        case Mixer::GatedLinear: FORGE_TRY(load_linear(m, L, t, w)); break;
        case Mixer::AttnSelective: FORGE_TRY(load_attn_selective(m, L, t, w)); break;
    }
    if (L.ff && post) {
        FORGE_TRY(load_norm(m, &w->norm2, t, "norm2"));
        FORGE_TRY(load_mixture(m, L, t, w));
    }
    if (L.ff && S.spec.arch->arrangement == Arrangement::ParallelTwo) FORGE_TRY(load_norm(m, &w->norm2, t, "norm2"));
    if (L.ff && S.spec.arch->arrangement == Arrangement::Sequential) {
        FORGE_TRY(load_norm(m, &w->norm2, t, "norm2"));
        Image in(2 * L.ff, S.width_p, S.dtype), out(S.spec.width, pad_to(L.ff, kDensePad), S.dtype);
        in.put(t.at("mlp.gate"), 0, 2); in.put(t.at("mlp.up"), 1, 2);
        FORGE_TRY(in.load(m, &w->ff_in));
        out.put(t.at("mlp.down"), 0);
        FORGE_TRY(out.load(m, &w->ff_out));
    }
    return FORGE_OK;
}

// rotation tables for at least n positions
int32_t ensure_rope(ForgeModel* m, int n) {
    StackModel& S = *m->stack;
    if (n <= S.rope_positions) return FORGE_OK;
    n = pad_to(n, 1024);
    FORGE_CUDA(cudaStreamSynchronize(m->stream));
    for (const LayerSpec& L : S.spec.layers) {
        if (!L.has_rotation()) continue;
        auto& e = S.ropes[L.rot];
        if (e.first >= n) continue;
        std::vector<float> tab(std::max<size_t>(1, size_t(n) * L.rot.dims));
        FORGE_TRY(rope_table(tab.data(), n, L.rot.frequencies(), L.rot.magnitude()));
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

// A step of few tokens runs an expert over all of them and takes the experts' columns of `out` from a list; otherwise tokens are dealt to the experts.
bool few_tokens(const StackModel& S, const LayerWeights& w, int rows) { return dense_listed_supported(S.spec.arch->arrangement == Arrangement::PostNorm ? w.ff_out : w.out, rows); }
// values of a row in front of `out`
int mid_columns(const StackModel& S, const LayerSpec& L, const LayerWeights& w, int rows) {
    return L.router.experts && S.spec.arch->arrangement == Arrangement::ParallelTwo && !few_tokens(S, w, rows) ? w.heads_k : w.out.K;
}
// the same in front of a mixture's way back
int shared_columns(const LayerSpec& L, const LayerWeights& w) { return L.router.always * w.ff_k; }
constexpr size_t kScoreBytes = size_t(256) << 20;   // scores of rows with mixed heads, at most, if rows may go in turn

// splits of the row attention: at most one CTA per SM over all rows and head groups, no more than there are pages
int row_splits(const StackModel& S, int rows, int pages) {
    int groups = 1;
    for (const LayerSpec& L : S.spec.layers) if (L.has_latent()) groups = std::max(groups, tensor_core_rows(S, L.mix) ? latent_decode_head_groups(L.mix) : L.mix.heads);
    return std::max(1, std::min(pages, 148 / std::max(1, rows * groups)));
}

// block_rows: rows of gathered blocks; all_at_once: no row waits for its turn
int32_t ensure_step(ForgeModel* m, int rows, int single, int splits, int prompt, int ctx_rows, int seg_rows, int chunks, int max_keys, int block_rows, bool all_at_once) {
    StackModel& S = *m->stack;
    const size_t es = dense_size(S.dtype), r = size_t(rows), W = size_t(S.spec.width), WP = size_t(S.width_p);
    // bytes, rows times the widest layer
    size_t h = WP * es, proj = 0, gate = 0, mid = 0, q = 0, part = 0, heads = 0, cc = 0, cr = 0, ck = 0, cv = 0, hgate = 0, decay = 0, beta = 0, low = 0, conv = 0, unit = 0, o = 0, pair = 0, router = 0, route = 0, e_in = 0, e_act = 0, e_out = 0, scores = 0, joint = 0, blocks = 0, scan = 0, bc = 0;
    ChunkBytes cb{0, 0};
    auto most = [](size_t& a, size_t b) { a = std::max(a, b); };
    size_t n_max = size_t(S.head.N);
    for (size_t i = 0; i < S.spec.layers.size(); ++i) {
        const LayerSpec& L = S.spec.layers[i];
        const LayerWeights& w = S.weights(int(i));
        for (const DenseWeight* d : {&w.in, &w.out, &w.kv, &w.low, &w.scan_in, &w.ff_in, &w.ff_out}) most(n_max, size_t(d->N));
        most(mid, r * std::max(mid_columns(S, L, w, rows), S.spec.arch->arrangement == Arrangement::PostNorm ? shared_columns(L, w) : w.ff_out.K) * es);
        if (S.spec.arch->arrangement == Arrangement::PostNorm) most(pair, r * W * 4);
        if (S.spec.arch->arrangement == Arrangement::ParallelTwo) most(h, 2 * WP * es);
        if (L.router.experts) {
            const size_t pairs = r * L.router.top;
            most(mid, std::min<size_t>(r, kScaleRows) * std::max(w.out.K, w.ff_out.K) * es);
            most(router, r * L.router.choices() * 4);
            most(route, route_bytes(L.router, rows));
            if (!few_tokens(S, w, rows)) { most(e_in, pairs * WP * es); most(e_act, pairs * w.ff_k * es); most(e_out, pairs * W * 4); }
        }
        if (L.kind == Mixer::Softmax || L.kind == Mixer::AttnSelective) {
            const AttnDims& a = L.attn;
            most(proj, r * w.v_row * 4);
            most(q, r * a.heads * a.dim_p * es);
            if (L.soft.talk && single) {
                const size_t one = talk_rows_bytes(a, 1, a.most_keys(max_keys));
                most(scores, all_at_once ? one * single : std::max(one, std::min(one * single, kScoreBytes)));
            }
            if (L.soft.talk) most(joint, size_t(prompt) * a.heads * a.groups * a.vdim_p * es);
            if (a.pool) most(blocks, size_t(block_rows) * a.row() * es);
            if (L.kind == Mixer::AttnSelective) {
                const SelectiveDims& d = L.sel;
                most(scan, r * 2 * w.scan_in.K * es);
                most(gate, r * d.inner * es);
                most(bc, r * 2 * d.state * 4);
                most(low, r * w.low.K * es);
                most(decay, r * d.inner * 4);
            }
            continue;
        }
        if (L.has_latent()) {
            const LatentDims& d = L.mix;
            most(proj, r * w.g_row * 4);
            most(gate, r * d.heads * d.vdim * es);
            most(q, std::max(size_t(single) * d.heads * d.row(), size_t(prompt) * d.heads * (d.dim_p + d.rot_p)) * es);
            most(part, size_t(single) * d.heads * d.rank_p * splits * 4);
            most(heads, size_t(single) * d.heads * splits * sizeof(float2));
            most(cc, size_t(ctx_rows) * d.rank_p * es); most(cr, size_t(ctx_rows) * std::max(d.rot_p, 64) * es);
            most(ck, size_t(ctx_rows) * d.heads * d.dim_p * es); most(cv, size_t(ctx_rows) * d.heads * d.vdim_p * es);
            continue;
        }
        const RecurDims& d = L.rec;
        const size_t HV = size_t(d.heads) * d.vdim;
        most(proj, r * d.channels() * es);
        most(gate, r * HV * es);
        most(decay, r * (d.channel ? size_t(d.heads) * d.dim : d.heads) * 4);
        most(beta, r * d.heads * 4);
        most(low, r * (w.decay_k + w.low.K) * es);
        most(o, r * HV * 4);
        if (chunks && recur_chunked_supported(d)) {
            const ChunkBytes b = recur_chunk_bytes(d);
            most(cb.half, chunks * b.half); most(cb.f32, chunks * b.f32);
        }
        if (d.rule == Rule::Delta && seg_rows) { most(conv, r * d.channels() * es); most(unit, r * 2 * d.groups * 4); }
        if (L.kind == Mixer::AttnTimeMix) {
            most(h, (1 + kMixes) * WP * es);
            most(q, r * L.attn.heads * L.attn.dim_p * es);
            most(hgate, r * L.attn.heads * 4);
            most(mid, r * 2 * w.out.K * es);
            most(pair, r * 2 * W * 4);
        }
    }
    FORGE_TRY(grow(m, S.x, r * W * 4));
    FORGE_TRY(grow(m, S.h, r * h));
    if (S.loop_in.N) FORGE_TRY(grow(m, S.cat, r * 2 * WP * es));
    if (S.spec.adds_loop()) FORGE_TRY(grow(m, S.x0, r * W * 4));
    if (S.rms_final()) { FORGE_TRY(grow(m, S.sums, r * scale_parts(int(W)) * 4)); FORGE_TRY(grow(m, S.sum1, r * 4)); }
    FORGE_TRY(grow(m, S.place, r * sizeof(int32_t)));
    const std::pair<StackModel::Buf*, size_t> sizes[] = {{&S.proj, proj}, {&S.gate, gate}, {&S.mid, mid}, {&S.q, q}, {&S.part, part}, {&S.ml, heads}, {&S.hgate, hgate}, {&S.decay, decay},
        {&S.beta, beta}, {&S.low, low}, {&S.conv, conv}, {&S.unit, unit}, {&S.o, o}, {&S.pair, pair}, {&S.c_half, cb.half}, {&S.c_f32, cb.f32}, {&S.ctx_c, cc}, {&S.ctx_r, cr}, {&S.ctx_k, ck}, {&S.ctx_v, cv},
        {&S.router, router}, {&S.route, route}, {&S.e_in, e_in}, {&S.e_act, e_act}, {&S.e_out, e_out},
        {&S.scores, scores}, {&S.joint, joint}, {&S.blocks, blocks}, {&S.scan, scan}, {&S.bc, bc}};
    for (const auto& e : sizes) FORGE_TRY(grow(m, *e.first, e.second));
    // one ticket per output tile of the largest product (128 rows x at least 16 tokens)
    const size_t tiles = std::max<size_t>(256, ((n_max + 127) / 128) * std::max<size_t>(1, (size_t(std::max(rows, ctx_rows)) + 127) / 128));
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
    int ones = 0;                            // rows [0, ones): one token of its sequence each
    int single = 0, splits = 1;              // rows [0, single): attention row by row; the rest are prompt rows
    int max_keys = 1;                        // most keys a row of [0, single) has
    int scale_rows = 0;                      // most rows of a product that takes scales
    SegTable segs;                           // the rows [ones, n)
    const PromptTile* tiles = nullptr; int n_tiles = 0;
    const PromptTile* host_tiles = nullptr;
    const int32_t* ctx_pages = nullptr; int ctx_rows = 0;
    const PoolChunk* chunks = nullptr; int n_chunks = 0;   // of the prompts' blocks
    uint32_t* hist = nullptr; const int32_t* step = nullptr;
    float* trace = nullptr; size_t trace_stride = 0;
};

char* at(void* p, size_t elems, int dtype) { return static_cast<char*>(p) + elems * dense_size(dtype); }

// the scales of an RMS norm's tokens
RowScale stream_scale(const StackModel& S, int rows) {
    RowScale r;
    if (!S.rms_final()) return r;
    const bool summed = rows > kScaleRows;
    r.sums = static_cast<const float*>(summed ? S.sum1.p : S.sums.p);
    r.parts = summed ? 1 : scale_parts(S.spec.width);
    r.inv_n = 1.0f / float(S.spec.width); r.eps = S.spec.eps;
    return r;
}

// The launch sequence of one step.
struct Sequence {
    ForgeModel* m;
    ForgeKV* kv;
    const Step& s;
    StackModel& S;
    cudaStream_t st;
    const int n, W, WP, dt;
    const bool sequential, two_norms, post;
    Sequence(ForgeModel* m_, ForgeKV* kv_, const Step& s_)
        : m(m_), kv(kv_), s(s_), S(*m_->stack), st(m_->stream), n(s_.rows.n), W(S.spec.width), WP(S.width_p), dt(S.dtype), sequential(S.spec.arch->arrangement == Arrangement::Sequential),
          two_norms(S.spec.arch->arrangement == Arrangement::ParallelTwo), post(S.spec.arch->arrangement == Arrangement::PostNorm) {}

    int32_t gemm(const DenseWeight& w, const void* act, int ld, const DenseOut& o, int rows) { return dense_gemm(w, act, ld, rows, o, S.scratch, m->d_err, st); }
    int32_t gemm(const DenseWeight& w, const void* act, int ld, const DenseOut& o) { return gemm(w, act, ld, o, n); }

    After norm(const StreamNorm& d, int ld) {
        After a;
        a.dst = S.h.p; a.ld = ld; a.w = d.w;
        if (S.rms_final()) { a.kind = AFTER_RMS; a.sums = static_cast<float*>(S.sums.p); a.parts = scale_parts(W); }
        else { a.kind = AFTER_DYT; a.alpha = d.alpha; a.b = d.b; }
        return a;
    }
    int h_ld(int layer) const { return S.spec.layers[layer].kind == Mixer::AttnTimeMix ? (1 + kMixes) * WP : two_norms ? 2 * WP : WP; }
    After norm1(int layer) {
        if (post) return stream();
        After a = norm(S.weights(layer).norm1, h_ld(layer));
        if (two_norms && S.spec.layers[layer].ff) { a.w2 = S.weights(layer).norm2.w; a.col2 = WP; }
        return a;
    }
    // the stream itself
    After stream() {
        After a;
        a.kind = AFTER_CAST; a.dst = S.h.p; a.ld = WP;
        return a;
    }
    // what the first reader of the stream in front of run i takes
    After into(size_t i) {
        if (i == S.spec.runs.size()) return norm(S.final_norm, WP);
        const int pass = S.spec.runs[i].pass;
        if (pass < 0) return norm1(S.spec.runs[i].layer);
        After a;
        if (S.spec.adds_loop()) {
            a = norm1(S.spec.runs[i].layer);
            a.plus = S.loop_step + size_t(pass) * W;
            if (pass > 0) a.again = static_cast<float*>(S.x0.p);
            if (s.trace && i > 0) a.keep = s.trace + (i - 1) * s.trace_stride;
            return a;
        }
        a.kind = AFTER_CAST; a.dst = S.cat.p; a.ld = 2 * WP;
        return a;
    }
    static void resid(DenseOut* o, float* x, int W, const After& after) { o->add(SEG_RESID, 0, W, x, W).after = after; }
    float* x() { return static_cast<float*>(S.x.p); }
    // RMS norms: the tokens' scales from the sums that the stream's last writer left
    int32_t stats(bool last) { return (last ? S.rms_final() : S.rms_stream()) && s.scale_rows > kScaleRows ? row_sums(static_cast<float*>(S.sum1.p), static_cast<float*>(S.sums.p), n, scale_parts(W), st) : FORGE_OK; }
    RowScale scale() const { return S.rms_stream() ? stream_scale(S, s.scale_rows) : RowScale{}; }

    int32_t run() {
        EmbedArgs e;
        e.x = x(); e.table = S.embed; e.tokens = s.tokens; e.width = W; e.width_p = WP;
        e.after = into(0);
        if (S.loop_in.N) { e.x0 = at(S.cat.p, size_t(WP), dt); e.x0_ld = 2 * WP; }
        if (S.spec.adds_loop()) e.x0_f32 = static_cast<float*>(S.x0.p);
        e.scale = S.spec.embed_scale;
        if (S.spec.buckets) {
            e.bigram = S.bigram; e.buckets = uint32_t(S.spec.buckets); e.mul_prev = uint32_t(S.spec.mul_prev); e.mul_cur = uint32_t(S.spec.mul_cur);
            e.prev = kv->stack->prev_token;
        }
        e.place = static_cast<int32_t*>(S.place.p); e.rows = s.rows; e.hist = s.hist; e.step = s.step;
        FORGE_TRY(embed_rows(e, dt, st));
        if (S.spec.buckets) FORGE_TRY(keep_tokens(kv->stack->prev_token, s.tokens, s.rows, st));
        for (size_t i = 0; i < S.spec.runs.size(); ++i) {
            const LayerRun& r = S.spec.runs[i];
            const LayerSpec& L = S.spec.layers[r.layer];
            const LayerWeights& w = S.weights(r.layer);
            StackCache::Run& run = kv->stack->runs[i];
            if (r.pass >= 0 && !S.spec.adds_loop()) {
                DenseOut o;
                OutSeg& g = o.add(SEG_RESID, 0, W, x(), W);
                g.fresh = true; g.add = S.loop_step + size_t(r.pass) * W; g.after = norm1(r.layer);
                FORGE_TRY(gemm(S.loop_in, S.cat.p, 2 * WP, o));
            }
            const bool ff = sequential && L.ff;
            const After after = ff ? norm(w.norm2, WP) : post && L.ff ? stream() : into(i + 1);
            FORGE_TRY(stats(false));
            switch (L.kind) {
                case Mixer::Latent: FORGE_TRY(latent(L, w, run, after)); break;
                case Mixer::Delta: case Mixer::ChannelDelta: FORGE_TRY(delta(L, w, run, after)); break;
                case Mixer::AttnTimeMix: FORGE_TRY(pair(L, w, run, after)); break;
                case Mixer::Softmax: FORGE_TRY(softmax(L, w, run, after)); break;
                case Mixer::GatedLinear: FORGE_TRY(linear(L, w, run, after)); break;
                case Mixer::AttnSelective: FORGE_TRY(attn_selective(L, w, run, after)); break;
            }
            if (post && L.ff) FORGE_TRY(mixture(L, w, into(i + 1)));
            if (ff) {
                DenseOut in, out;
                in.add(S.spec.arch->dense == Mlp::ClampedGlu ? SEG_CLAMPED_GLU : SEG_SILU_GLU, 0, 2 * L.ff, S.mid.p, w.ff_out.K).limit = L.limit;
                FORGE_TRY(gemm(w.ff_in, S.h.p, WP, in));
                resid(&out, x(), W, into(i + 1));
                FORGE_TRY(gemm(w.ff_out, S.mid.p, w.ff_out.K, out));
            }
            if (s.trace && !after.keep) FORGE_CUDA(cudaMemcpyAsync(s.trace + i * s.trace_stride, S.x.p, sizeof(float) * n * W, cudaMemcpyDeviceToDevice, st));
        }
        return stats(true);
    }

    int32_t latent(const LayerSpec& L, const LayerWeights& w, StackCache::Run& run, const After& after) {
        const LatentDims& d = L.mix;
        const int ldp = w.g_row, gate_ld = d.heads * d.vdim, mid_ld = w.out.K, ff = sequential ? 0 : L.ff;
        float* proj = static_cast<float*>(S.proj.p);
        const float* rope = S.ropes.at(L.rot).second;
        {
            DenseOut o;
            o.add(SEG_F32, 0, w.q_rows, proj, ldp);
            o.add(SEG_F32, w.dkv_row, d.rank + d.rot, proj + w.dkv_row, ldp);
            o.add(SEG_SIGMOID, w.g_row, gate_ld, S.gate.p, gate_ld);
            if (ff) o.add(S.spec.arch->dense == Mlp::ClampedGlu ? SEG_CLAMPED_GLU : SEG_SILU_GLU, w.glu_row, 2 * ff, at(S.mid.p, w.heads_k, dt), mid_ld).limit = L.limit;
            FORGE_TRY(gemm(w.in, S.h.p, WP, o));
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
            OutSeg& k = o.add(SEG_CAST, 0, d.heads * d.dim, S.ctx_k.p, d.heads * d.dim_p);
            k.group = d.dim; k.group_ld = d.dim_p;
            OutSeg& v = o.add(SEG_CAST, w.uv_row, d.heads * d.vdim, S.ctx_v.p, d.heads * d.vdim_p);
            v.group = d.vdim; v.group_ld = d.vdim_p;
            FORGE_TRY(gemm(w.kv, S.ctx_c.p, d.rank_p, o, s.ctx_rows));
            PromptAttnArgs a;
            a.q = S.q.p; a.k = S.ctx_k.p; a.krot = S.ctx_r.p; a.v = S.ctx_v.p;
            a.gate = at(S.gate.p, size_t(s.single) * gate_ld, dt); a.gate_ld = gate_ld;
            a.out = at(S.mid.p, size_t(s.single) * mid_ld, dt); a.out_ld = mid_ld;
            a.q_rows = np; a.ctx_rows = s.ctx_rows; a.tiles = s.tiles; a.n_tiles = s.n_tiles; a.host_tiles = s.host_tiles; a.err = m->d_err;
            FORGE_TRY(attn_prefill_kv(PromptDims(d), a, st));
        }
        DenseOut o;
        resid(&o, x(), W, after);
        return gemm(w.out, S.mid.p, mid_ld, o);
    }

    // single tokens and segments of a recurrent mixer
    int32_t recur(const RecurDims& d, const RecurArgs& a) {
        StepRows ones = s.rows;
        ones.n = s.ones;
        FORGE_TRY(recur_decode(d, dt, a, ones, st));
        RecurScratch sc;
        sc.conv = S.conv.p; sc.unit = static_cast<float*>(S.unit.p); sc.o = static_cast<float*>(S.o.p);
        sc.chunk.half = static_cast<__nv_bfloat16*>(S.c_half.p); sc.chunk.f32 = static_cast<float*>(S.c_f32.p); sc.err = m->d_err;
        return recur_segments(d, dt, a, sc, s.segs, st);
    }
    RecurArgs recur_args(const RecurDims& d, const LayerWeights& w, StackCache::Run& run) {
        RecurArgs a;
        a.x = S.proj.p; a.x_ld = d.channels();
        a.decay = static_cast<float*>(S.decay.p); a.decay_ld = d.channel ? d.heads * d.dim : d.heads;
        a.beta = static_cast<float*>(S.beta.p); a.bonus = w.bonus; a.conv = w.conv; a.ring = run.ring; a.state = run.state;
        a.norm = w.head_norm;
        a.gate = S.gate.p; a.gate_ld = d.heads * d.vdim;
        return a;
    }

    // rows of `in` that the feed-forward of a layer with two norms takes, or its router
    void feed_forward_rows(DenseOut* o, const LayerSpec& L, const LayerWeights& w) {
        if (L.router.experts) {
            OutSeg& g = o->add(SEG_F32, w.router_row, L.router.experts, S.router.p, L.router.experts);
            g.add = w.router_bias; g.act_col = WP;
        } else if (L.ff) o->add(SEG_SILU_GLU, w.glu_row, 2 * L.ff, at(S.mid.p, w.heads_k, dt), w.out.K).act_col = WP;
    }
    // x += W_o (heads in front of `out`) + feed-forward
    int32_t two_norms_out(const LayerSpec& L, const LayerWeights& w, const After& after, bool routed = false) {
        if (L.router.experts) return experts(L, w, after, routed);
        DenseOut o;
        resid(&o, x(), W, after);
        return gemm(w.out, S.mid.p, w.out.K, o);
    }
    // Few tokens: every expert that is used runs over all of them (a token that does not use it gets zeros) into its columns in front of `out`, which
    // then is one product over the heads' columns and those of the experts that are used.  Otherwise the tokens are gathered expert by expert.
    // routed: a launch of the mixer has routed few tokens already.
    int32_t experts(const LayerSpec& L, const LayerWeights& w, const After& after, bool routed) {
        const RouteTables t = route_tables(S.route.p, L.router, n);
        const float* logits = static_cast<const float*>(S.router.p);
        GroupTable table;
        GroupShape shape;
        shape.rows = 2 * L.ff; shape.group_rows = w.expert_rows;
        DenseOut in;
        in.scale = scale();
        if (few_tokens(S, w, n)) {
            if (routed) table = few_table(L.router, n, t);
            else FORGE_TRY(route_few(L.router, logits, n, t, &table, st));
            shape.group_dst = size_t(w.ff_k);
            in.add(SEG_SILU_GLU, 0, 2 * L.ff, at(S.mid.p, w.heads_k, dt), w.out.K);
            FORGE_TRY(dense_gemm_groups(w.experts, shape, table, at(S.h.p, WP, dt), 2 * WP, n, in, m->d_err, st));
            DenseOut out;
            resid(&out, x(), W, after);
            return dense_gemm_listed(w.out, w.heads_k, w.ff_k, table, S.mid.p, w.out.K, n, out, m->d_err, st);
        }
        {
            DenseOut o;
            resid(&o, x(), W, After{});
            FORGE_TRY(gemm(w.out.columns(0, w.heads_k), S.mid.p, w.heads_k, o));
        }
        FORGE_TRY(route_slots(L.router, logits, n, t, &table, st));
        const int pairs = n * L.router.top;
        FORGE_TRY(gather_act_rows(S.e_in.p, at(S.h.p, WP, dt), 2 * WP, t.row, pairs, WP, dt, st));
        in.scale.row = t.row;
        in.add(SEG_SILU_GLU, 0, 2 * L.ff, S.e_act.p, w.ff_k);
        FORGE_TRY(dense_gemm_groups(w.experts, shape, table, S.e_in.p, WP, pairs, in, m->d_err, st));
        DenseOut down;
        down.add(SEG_F32, 0, W, S.e_out.p, W);
        GroupShape cols;
        cols.rows = W; cols.group_cols = w.ff_k;
        table.weight = nullptr;
        FORGE_TRY(dense_gemm_groups(w.out.columns(w.heads_k, w.ff_k), cols, table, S.e_act.p, w.ff_k, pairs, down, m->d_err, st));
        return add_experts(x(), static_cast<const float*>(S.e_out.p), L.router, t, n, W, after, dt, st);
    }

    // rows of `in` of queries, keys and values
    void qkv_rows(DenseOut* o, const LayerSpec& L, const LayerWeights& w, StackCache::Run& run) {
        const AttnDims& a = L.attn;
        float* proj = static_cast<float*>(S.proj.p);
        o->add(SEG_F32, 0, a.heads * a.dim, proj, w.v_row).add = w.q_bias;
        o->add(SEG_F32, w.k_row, a.groups * a.dim, proj + w.k_row, w.v_row).add = w.k_bias;
        OutSeg& v = o->add(SEG_CAST, w.v_row, a.groups * a.vdim, at(run.pool, size_t(a.groups) * a.dim_p, dt), a.row());
        v.group = a.vdim; v.group_ld = a.vdim_p; v.place = static_cast<const int32_t*>(S.place.p); v.add = w.v_bias;
        if (L.blend_layer >= 0) {   // the lender's values lie in its cache rows
            const AttnDims& b = S.spec.layers[L.blend_layer].attn;
            v.blend = at(lender(L.blend_layer).pool, size_t(b.groups) * b.dim_p, dt); v.blend_ld = b.row();
            v.own = 1.f - w.lambda; v.other = w.lambda;
        }
    }
    StackCache::Run& lender(int layer) {
        size_t i = 0;
        while (S.spec.runs[i].layer != layer) ++i;
        return kv->stack->runs[i];
    }
    // norms and rotation; then the attention of all rows of the step: factor * heads to the first columns of mid
    int32_t queries_and_keys(const LayerSpec& L, const LayerWeights& w, StackCache::Run& run, const RouteBeside* route, const ConvBeside* conv) {
        return qk_post(L.attn, L.soft.qk, dt, static_cast<const float*>(S.proj.p), w.v_row, w.k_row, w.q_norm, w.k_norm, S.ropes.at(L.rot).second, S.q.p, run.pool, static_cast<const int32_t*>(S.place.p),
                       s.rows, route, conv, st);
    }
    int32_t attend(const LayerSpec& L, const LayerWeights& w, StackCache::Run& run, int mid_ld, float factor) {
        AttnDims a = L.attn;
        a.pool_row0 = kv->num_pages * FORGE_KV_PAGE;
        const bool pools = a.pool && L.soft.talk && all_ones();
        if (a.pool && !pools) FORGE_TRY(pool_blocks(a, dt, run.pool, s.rows, st));
        StepRows single = s.rows;
        single.n = s.single;
        const int max_keys = a.most_keys(s.max_keys), np = n - s.single;
        if (L.soft.talk) FORGE_TRY(talk_rows(a, dt, S.q.p, run.pool, pools, w.talk, factor, S.scores.p, S.scores.cap, S.mid.p, mid_ld, single, max_keys, st));
        else FORGE_TRY(attn_rows(a, dt, S.q.p, run.pool, nullptr, w.sink, w.bias, S.mid.p, mid_ld, single, max_keys, st));
        if (np <= 0) return FORGE_OK;
        void* out = at(S.mid.p, size_t(s.single) * mid_ld, dt);
        PromptDims d(a);
        if (L.score_bound > 0.f) d.bound = L.score_bound + w.bias_bound;
        PromptAttnArgs p;
        p.q = at(S.q.p, size_t(s.single) * a.heads * a.dim_p, dt); p.k = run.pool; p.v = at(run.pool, size_t(a.groups) * a.dim_p, dt);
        p.sink = w.sink; p.bias = w.bias;
        p.out = out; p.out_ld = mid_ld;
        p.q_rows = np; p.ctx_rows = kv->num_pages * FORGE_KV_PAGE; p.tiles = s.tiles; p.n_tiles = s.n_tiles; p.host_tiles = s.host_tiles;
        p.pages = s.ctx_pages; p.page_row = a.row(); p.err = m->d_err;
        if (a.pool) {
            FORGE_TRY(gather_blocks(a, dt, S.blocks.p, run.pool, s.ctx_pages, s.chunks, s.n_chunks, st));
            p.blocks = S.blocks.p; p.block_rows = s.n_chunks * FORGE_KV_PAGE;
        }
        if (!L.soft.talk) return attn_prefill_kv(d, p, st);
        d.joint = true;
        p.out = S.joint.p; p.out_ld = a.heads * a.groups * a.vdim_p;
        FORGE_TRY(attn_prefill_kv(d, p, st));
        return talk_heads(a, S.joint.p, w.talk, factor, out, mid_ld, np, st);
    }

    int32_t softmax(const LayerSpec& L, const LayerWeights& w, StackCache::Run& run, const After& after) {
        DenseOut o;
        qkv_rows(&o, L, w, run);
        if (post) {
            FORGE_TRY(gemm(w.in, S.h.p, WP, o));
            FORGE_TRY(queries_and_keys(L, w, run, nullptr, nullptr));
            FORGE_TRY(attend(L, w, run, w.out.K, 1.f));
            return post_out(L, w, after);
        }
        o.scale = scale();
        feed_forward_rows(&o, L, w);
        FORGE_TRY(gemm(w.in, S.h.p, 2 * WP, o));
        const bool routed = L.router.experts && few_tokens(S, w, n);
        const RouteBeside route{L.router, static_cast<const float*>(S.router.p), route_tables(S.route.p, L.router, n)};
        FORGE_TRY(queries_and_keys(L, w, run, routed ? &route : nullptr, nullptr));
        FORGE_TRY(attend(L, w, run, mid_columns(S, L, w, n), 1.f));
        return two_norms_out(L, w, after, routed);
    }

    // x += norm1(W_o mid); few tokens are routed there, too
    RouterDims router_dims(const LayerSpec& L, const LayerWeights& w) {
        RouterDims r = L.router;
        r.correction = w.router_bias;
        return r;
    }
    bool routed_behind(const LayerSpec& L, const LayerWeights& w) { return L.router.experts && few_tokens(S, w, n) && route_behind_supported(L.router, W, n); }
    int32_t post_out(const LayerSpec& L, const LayerWeights& w, const After& after) {
        DenseOut o;
        o.add(SEG_F32, 0, W, S.pair.p, W).add = w.out_bias;
        FORGE_TRY(gemm(w.out, S.mid.p, w.out.K, o));
        const RouterDims r = router_dims(L, w);
        const RouteBehind route{r, w.router, WP, route_tables(S.route.p, r, n), S.scratch.tickets};
        return add_normed(x(), static_cast<const float*>(S.pair.p), n, W, S.spec.eps, w.norm1.alpha, MixtureSum{}, after, routed_behind(L, w) ? &route : nullptr, dt, st);
    }

    int32_t attn_selective(const LayerSpec& L, const LayerWeights& w, StackCache::Run& run, const After& after) {
        const SelectiveDims& d = L.sel;
        const int inner_p = w.scan_in.K;
        void *in = S.scan.p, *xc = at(S.scan.p, size_t(n) * pad_to(d.inner, kDensePad), dt);   // rows [inner], then padded ones
        {
            DenseOut o;
            qkv_rows(&o, L, w, run);
            o.add(SEG_CAST, w.in_row, d.inner, in, d.inner);
            o.add(SEG_SILU, w.gate_row, d.inner, S.gate.p, d.inner);
            FORGE_TRY(gemm(w.in, S.h.p, WP, o));
        }
        SelectiveArgs a;
        a.in = in; a.in_ld = d.inner; a.conv = w.conv; a.conv_add = w.conv_add; a.ring = run.ring;
        a.x = xc; a.x_ld = inner_p;
        a.bc = static_cast<const float*>(S.bc.p); a.bc_ld = 2 * d.state;
        a.a2 = w.scan_a; a.skip = w.skip; a.state = run.state;
        a.gate = S.gate.p; a.gate_ld = d.inner; a.factor = L.right_scale;
        a.out = at(S.mid.p, w.heads_k, dt); a.out_ld = w.out.K;
        StepRows ones = s.rows;
        ones.n = s.ones;
        if (all_ones()) {
            const ConvBeside conv{d, a};
            FORGE_TRY(queries_and_keys(L, w, run, nullptr, &conv));
        } else {
            FORGE_TRY(selective_conv(d, dt, a, ones, s.segs, st));
            FORGE_TRY(queries_and_keys(L, w, run, nullptr, nullptr));
        }
        {
            DenseOut o;
            o.add(SEG_CAST, 0, d.rank, S.low.p, w.low.K);
            o.add(SEG_F32, w.bc_row, 2 * d.state, S.bc.p, 2 * d.state);
            FORGE_TRY(gemm(w.scan_in, xc, inner_p, o));
        }
        // formed inside the recurrence, if every kernel of the step can
        if (all_ones() || selective_steps_inside(dt, w.low.K)) {
            a.dt_w = w.low.w; a.low = S.low.p; a.low_ld = a.low_k = w.low.K; a.dt_add = w.decay_add;
        } else {   // softplus: the epilogue of decays with a factor of minus one
            DenseOut o;
            OutSeg& g = o.add(SEG_DECAY, 0, d.inner, S.decay.p, d.inner);
            g.mul = w.minus; g.add = w.decay_add;
            FORGE_TRY(gemm(w.low, S.low.p, w.low.K, o));
            a.dt = static_cast<const float*>(S.decay.p); a.dt_ld = d.inner;
        }
        FORGE_TRY(selective_decode(d, dt, a, ones, st));
        FORGE_TRY(selective_segments(d, dt, a, s.segs, st));
        FORGE_TRY(attend(L, w, run, w.out.K, L.left_scale));
        return post_out(L, w, after);
    }

    // x += norm2(shared expert + experts + what is passed on); see experts() for few and many tokens
    int32_t mixture(const LayerSpec& L, const LayerWeights& w, const After& after) {
        const RouterDims r = router_dims(L, w);
        const bool few = few_tokens(S, w, n), routed = routed_behind(L, w);
        const int shared_k = shared_columns(L, w), mid_ld = few ? w.ff_out.K : shared_k;
        const RouteTables t = route_tables(S.route.p, r, n);
        const float* logits = static_cast<const float*>(S.router.p);
        float* y = static_cast<float*>(S.pair.p);
        MixtureSum sum;
        if (r.identity) sum.passed = t.passed;
        if (!few) {
            DenseOut o;
            o.add(SEG_F32, 0, r.choices(), S.router.p, r.choices());
            o.add(SEG_SILU_GLU, w.glu_row, r.always * w.expert_rows, S.mid.p, mid_ld);
            FORGE_TRY(gemm(w.ff_in, S.h.p, WP, o));
        } else if (!routed) {
            DenseOut o;
            o.add(SEG_F32, 0, r.choices(), S.router.p, r.choices());
            FORGE_TRY(gemm(w.ff_in.rows(0, w.glu_row), S.h.p, WP, o));
        }
        GroupTable table;
        GroupShape shape;
        shape.rows = 2 * L.ff; shape.group_rows = w.expert_rows;
        DenseOut in, out;
        out.add(SEG_F32, 0, W, y, W);
        if (few) {
            if (routed) table = few_table(r, n, t);
            else FORGE_TRY(route_few(r, logits, n, t, &table, st));
            shape.group_dst = size_t(w.ff_k);
            in.add(SEG_SILU_GLU, 0, 2 * L.ff, S.mid.p, mid_ld);
            FORGE_TRY(dense_gemm_groups(w.experts, shape, table, S.h.p, WP, n, in, m->d_err, st));
            FORGE_TRY(dense_gemm_listed(w.ff_out, shared_k, w.ff_k, listed_table(r, n, t), S.mid.p, mid_ld, n, out, m->d_err, st));
            return add_normed(x(), y, n, W, S.spec.eps, w.norm2.alpha, sum, after, nullptr, dt, st);
        }
        FORGE_TRY(gemm(w.ff_out.columns(0, shared_k), S.mid.p, mid_ld, out));
        FORGE_TRY(route_slots(r, logits, n, t, &table, st));
        const int pairs = n * r.top;
        FORGE_TRY(gather_act_rows(S.e_in.p, S.h.p, WP, t.row, pairs, WP, dt, st));
        in.add(SEG_SILU_GLU, 0, 2 * L.ff, S.e_act.p, w.ff_k);
        FORGE_TRY(dense_gemm_groups(w.experts, shape, table, S.e_in.p, WP, pairs, in, m->d_err, st));
        DenseOut down;
        down.add(SEG_F32, 0, W, S.e_out.p, W);
        GroupShape cols;
        cols.rows = W; cols.group_cols = w.ff_k;
        table.weight = nullptr;
        FORGE_TRY(dense_gemm_groups(w.ff_out.columns(0, w.ff_k), cols, table, S.e_act.p, w.ff_k, pairs, down, m->d_err, st));
        sum.e = static_cast<const float*>(S.e_out.p); sum.slot = t.slot; sum.top = r.top;
        return add_normed(x(), y, n, W, S.spec.eps, w.norm2.alpha, sum, after, nullptr, dt, st);
    }

    int32_t linear(const LayerSpec& L, const LayerWeights& w, StackCache::Run& run, const After& after) {
        const RecurDims& d = L.rec;
        const int D = d.qk(), HV = d.heads * d.vdim;
        RecurArgs a = recur_args(d, w, run);
        {
            DenseOut o;
            o.scale = scale();
            o.add(SEG_CAST, 0, d.channels(), S.proj.p, d.channels());
            o.add(SEG_SILU, w.gate_row, HV, S.gate.p, HV);
            o.add(SEG_CAST, w.decay_row, L.decay_rank, S.low.p, w.low.K);
            feed_forward_rows(&o, L, w);
            FORGE_TRY(gemm(w.in, S.h.p, 2 * WP, o));
        }
        if (all_ones()) two_step(&a, w, w.low.K);
        else {
            DenseOut lo;
            OutSeg& g = lo.add(SEG_DECAY, 0, D, S.decay.p, D);
            g.mul = w.decay_mul; g.add = w.decay_add;
            FORGE_TRY(gemm(w.low, S.low.p, w.low.K, lo));
        }
        a.out = S.mid.p; a.out_ld = mid_columns(S, L, w, n);
        FORGE_TRY(recur(d, a));
        return two_norms_out(L, w, after);
    }

    // a step of single tokens forms two-step decays and gates inside the recurrence
    bool all_ones() const { return s.ones == n; }
    void two_step(RecurArgs* a, const LayerWeights& w, int low_ld) {
        a->decay_w = w.low.w; a->low = S.low.p; a->low_ld = low_ld; a->low_k = w.low.K;
        a->decay_mul = w.decay_mul; a->decay_add = w.decay_add;
    }

    int32_t delta(const LayerSpec& L, const LayerWeights& w, StackCache::Run& run, const After& after) {
        const RecurDims& d = L.rec;
        const int H = d.heads, HV = H * d.vdim, low_ld = w.decay_k + w.low.K;
        RecurArgs a = recur_args(d, w, run);
        DenseOut o;
        o.add(SEG_CAST, 0, d.channels(), S.proj.p, d.channels());
        if (!d.channel) {
            o.add(SEG_SILU, w.gate_row, HV, S.gate.p, HV);
            o.add(SEG_SIGMOID_F32, w.beta_row, H, S.beta.p, H);
            OutSeg& g = o.add(SEG_DECAY, w.decay_row, H, S.decay.p, H);
            g.mul = w.decay_mul; g.add = w.decay_add;
            FORGE_TRY(gemm(w.in, S.h.p, WP, o));
        } else {
            o.add(SEG_SIGMOID_F32, w.beta_row, H, S.beta.p, H);
            o.add(SEG_CAST, w.decay_row, L.decay_rank, S.low.p, low_ld);
            o.add(SEG_CAST, w.low_gate_row, L.gate_rank, at(S.low.p, w.decay_k, dt), low_ld);
            FORGE_TRY(gemm(w.in, S.h.p, WP, o));
            if (all_ones()) {
                two_step(&a, w, low_ld);
                a.gate_w = at(w.low.w, size_t(w.low_row) * w.low.K, dt); a.gate_col = w.decay_k;
            } else {
                DenseOut lo;
                OutSeg& g = lo.add(SEG_DECAY, 0, H * d.dim, S.decay.p, H * d.dim);
                g.mul = w.decay_mul; g.add = w.decay_add;
                lo.add(SEG_SIGMOID, w.low_row, HV, S.gate.p, HV).act_col = w.decay_k;
                FORGE_TRY(gemm(w.low, S.low.p, low_ld, lo));
            }
        }
        a.out = S.mid.p; a.out_ld = w.out.K;
        FORGE_TRY(recur(d, a));
        DenseOut out;
        resid(&out, x(), W, after);
        return gemm(w.out, S.mid.p, w.out.K, out);
    }

    int32_t pair(const LayerSpec& L, const LayerWeights& w, StackCache::Run& run, const After& after) {
        const AttnDims& t = L.attn;
        const RecurDims& d = L.rec;
        const int D = d.heads * d.dim, ld = (1 + kMixes) * WP;
        float* hgate = static_cast<float*>(S.hgate.p);
        FORGE_TRY(token_shift(S.h.p, ld, W, WP, kMixes, w.mu, run.prev, dt, s.rows, s.ones, s.segs, st));
        DenseOut o;
        {
            const int32_t* place = static_cast<const int32_t*>(S.place.p);
            OutSeg& q = o.add(SEG_CAST, 0, t.heads * t.dim, S.q.p, t.heads * t.dim_p);
            q.group = t.dim; q.group_ld = t.dim_p;
            OutSeg& k = o.add(SEG_CAST, w.k_row, t.groups * t.dim, run.pool, t.row());
            k.group = t.dim; k.group_ld = t.dim_p; k.place = place;
            OutSeg& v = o.add(SEG_CAST, w.v_row, t.groups * t.vdim, at(run.pool, size_t(t.groups) * t.dim_p, dt), t.row());
            v.group = t.vdim; v.group_ld = t.vdim_p; v.place = place;
            o.add(SEG_SIGMOID_F32, w.hg_row, t.heads, hgate, t.heads);
            o.add(SEG_CAST, w.r_row, D, S.proj.p, 3 * D).act_col = WP;
            o.add(SEG_CAST, w.rk_row, D, at(S.proj.p, D, dt), 3 * D).act_col = 2 * WP;
            o.add(SEG_CAST, w.rv_row, D, at(S.proj.p, 2 * D, dt), 3 * D).act_col = 3 * WP;
            o.add(SEG_SILU, w.gate_row, D, S.gate.p, D).act_col = 4 * WP;
            o.add(SEG_TANH, w.decay_row, L.decay_rank, S.low.p, w.low.K).act_col = 5 * WP;
            FORGE_TRY(gemm(w.in, S.h.p, ld, o));
        }
        RecurArgs a = recur_args(d, w, run);
        const int mid_ld = 2 * w.out.K;
        if (all_ones()) two_step(&a, w, w.low.K);
        else {
            DenseOut lo;
            lo.add(SEG_EXP_DECAY, 0, D, S.decay.p, D).add = w.decay_add;
            FORGE_TRY(gemm(w.low, S.low.p, w.low.K, lo));
        }
        StepRows single = s.rows;
        single.n = s.single;
        FORGE_TRY(attn_rows(t, dt, S.q.p, run.pool, hgate, nullptr, nullptr, S.mid.p, mid_ld, single, t.most_keys(s.max_keys), st));
        const int np = n - s.single;
        if (np > 0) {
            PromptAttnArgs p;
            p.q = at(S.q.p, size_t(s.single) * t.heads * t.dim_p, dt); p.k = run.pool; p.v = at(run.pool, size_t(t.groups) * t.dim_p, dt);
            p.head_gate = hgate + size_t(s.single) * t.heads;
            p.out = at(S.mid.p, size_t(s.single) * mid_ld, dt); p.out_ld = mid_ld;
            p.q_rows = np; p.ctx_rows = kv->num_pages * FORGE_KV_PAGE; p.tiles = s.tiles; p.n_tiles = s.n_tiles; p.host_tiles = s.host_tiles;
            p.pages = s.ctx_pages; p.page_row = t.row(); p.err = m->d_err;
            FORGE_TRY(attn_prefill_kv(PromptDims(t), p, st));
        }
        a.norm_head = d.dim;
        a.out = at(S.mid.p, w.out.K, dt); a.out_ld = mid_ld;
        FORGE_TRY(recur(d, a));
        float* both = static_cast<float*>(S.pair.p);
        DenseOut out;
        out.add(SEG_F32, 0, W, both, 2 * W);
        out.add(SEG_F32, w.out_r_row, W, both + W, 2 * W).act_col = w.out.K;
        FORGE_TRY(gemm(w.out, S.mid.p, mid_ld, out));
        return add_normed_pair(x(), both, n, W, S.spec.eps, w.norm_l, w.norm_r, after, dt, st);
    }
};

// rows: of the stream that h's rows were taken from (null: the first n); step_rows: the step's scale_rows
int32_t run_head(ForgeModel* m, const void* h, const int32_t* rows, int n, int step_rows, float* logits) {
    StackModel& S = *m->stack;
    DenseOut o;
    o.scale = stream_scale(S, step_rows);
    o.scale.row = rows; o.scale.mul = S.spec.logit_scale;
    o.nseg = 1;
    o.seg[0].rows = S.spec.vocab; o.seg[0].dst = logits; o.seg[0].ld = S.spec.vocab;
    return dense_gemm(S.head, h, S.width_p, n, o, S.scratch, m->d_err, m->stream);
}

// The attention of entries of fewer tokens than this runs row by row over the cache: forming the keys and values of the whole
// context (latent attention), or filling a tile of 128 queries, does not pay for them.
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
static size_t state_bytes(const LayerSpec& L) { return L.state_values() * 4; }
static size_t ring_bytes(const StackModel& S, const LayerSpec& L) { return L.ring_values() * dense_size(S.dtype); }
static size_t prev_bytes(const StackModel& S, const LayerSpec& L) { return L.kind == Mixer::AttnTimeMix ? size_t(S.spec.width) * dense_size(S.dtype) : 0; }

int32_t stack_cache_create(ForgeKV* kv) {
    ForgeModel* m = kv->model;
    StackModel& S = *m->stack;
    FORGE_TRY(ensure_rope(m, kv->max_seq));
    kv->stack = new StackCache();
    kv->stack->runs.resize(S.spec.runs.size());
    const size_t slots = size_t(kv->batch);
    auto alloc = [&](auto** p, size_t bytes) -> int32_t {
        if (!bytes) return FORGE_OK;
        void* q = nullptr;
        FORGE_CUDA(cudaMalloc(&q, bytes));
        *p = static_cast<std::remove_reference_t<decltype(**p)>*>(q);
        FORGE_CUDA(cudaMemsetAsync(q, 0, bytes, m->stream));
        return FORGE_OK;
    };
    if (S.spec.buckets) FORGE_TRY(alloc(&kv->stack->prev_token, slots * sizeof(uint32_t)));
    for (size_t i = 0; i < S.spec.runs.size(); ++i) {
        const LayerSpec& L = S.spec.layers[S.spec.runs[i].layer];
        StackCache::Run& r = kv->stack->runs[i];
        char *pool = nullptr, *ring = nullptr, *prev = nullptr;
        const size_t rows = size_t(kv->num_pages) * L.page_rows();
        FORGE_TRY(alloc(&pool, rows * L.cache_row() * dense_size(S.dtype)));
        r.pool = pool;
        if (L.has_latent() && tensor_core_rows(S, L.mix)) FORGE_TRY(latent_cache_map(r.map, r.pool, L.mix, rows));
        FORGE_TRY(alloc(&r.state, slots * state_bytes(L)));
        FORGE_TRY(alloc(&ring, slots * ring_bytes(S, L)));
        r.ring = ring;
        FORGE_TRY(alloc(&prev, slots * prev_bytes(S, L)));
        r.prev = prev;
    }
    kv->stack->splits = row_splits(S, kv->batch, kv->pages_per_seq);
    return FORGE_OK;
}

void stack_cache_destroy(ForgeKV* kv) {
    if (!kv->stack) return;
    for (StackCache::Run& r : kv->stack->runs) for (void* p : {r.pool, static_cast<void*>(r.state), r.ring, r.prev}) if (p) cudaFree(p);
    if (kv->stack->prev_token) cudaFree(kv->stack->prev_token);
    delete kv->stack;
    kv->stack = nullptr;
}

bool stack_has_state(const ForgeModel* m) {
    if (m->stack->spec.buckets) return true;
    for (const LayerSpec& L : m->stack->spec.layers) if (L.has_state()) return true;
    return false;
}

int stack_kv_width(const ForgeKV* kv, int run, int which) {
    const StackModel& S = *kv->model->stack;
    const LayerSpec& L = S.spec.layers[S.spec.runs[run].layer];
    if (L.has_latent()) return which ? L.mix.rot : L.mix.rank;
    return L.has_attn() ? L.attn.groups * (which ? L.attn.vdim : L.attn.dim) : 0;
}

int32_t stack_kv_read(ForgeKV* kv, int seq, int run, int which, float* out_host) {
    ForgeModel* m = kv->model;
    const StackModel& S = *m->stack;
    const LayerSpec& L = S.spec.layers[S.spec.runs[run].layer];
    const int n = stack_kv_width(kv, run, which), len = kv->len[seq];
    if (n == 0) return FORGE_OK;
    auto column = [&](int i) {
        if (L.has_latent()) return (which ? L.mix.rank_p : 0) + i;
        const AttnDims& a = L.attn;
        return which ? a.groups * a.dim_p + i / a.vdim * a.vdim_p + i % a.vdim : i / a.dim * a.dim_p + i % a.dim;
    };
    const size_t es = dense_size(S.dtype), row = size_t(L.cache_row()) * es;
    std::vector<uint8_t> page(row * FORGE_KV_PAGE);
    for (int t0 = 0; t0 < len; t0 += FORGE_KV_PAGE) {
        const int pg = kv->h_page_table[size_t(seq) * kv->pages_per_seq + t0 / FORGE_KV_PAGE];
        FORGE_CUDA(cudaMemcpyAsync(page.data(), static_cast<char*>(kv->stack->runs[run].pool) + size_t(pg) * page.size(), page.size(), cudaMemcpyDeviceToHost, m->stream));
        FORGE_CUDA(cudaStreamSynchronize(m->stream));
        for (int t = t0; t < std::min(len, t0 + FORGE_KV_PAGE); ++t)
            for (int i = 0; i < n; ++i) {
                const uint8_t* p = page.data() + (t - t0) * row + column(i) * es;
                float& v = out_host[size_t(t) * n + i];
                if (es == 4) memcpy(&v, p, 4);
                else { uint16_t h; memcpy(&h, p, 2); const uint32_t u = uint32_t(h) << 16; memcpy(&v, &u, 4); }
            }
    }
    return FORGE_OK;
}

size_t stack_state_values(const ForgeKV* kv, int run) {
    const StackModel& S = *kv->model->stack;
    return state_bytes(S.spec.layers[S.spec.runs[run].layer]) / 4;
}
int32_t stack_state_read(ForgeKV* kv, int seq, int run, float* out_host) {
    const size_t n = stack_state_values(kv, run);
    if (n == 0) return FORGE_OK;
    if (kv->len[seq] == 0) { std::fill(out_host, out_host + n, 0.f); return FORGE_OK; }   // what a slot holds then counts as zero
    FORGE_CUDA(cudaMemcpyAsync(out_host, kv->stack->runs[run].state + size_t(seq) * n, n * 4, cudaMemcpyDeviceToHost, kv->model->stream));
    FORGE_CUDA(cudaStreamSynchronize(kv->model->stream));
    return FORGE_OK;
}

size_t stack_kv_bytes_per_token(const ForgeKV* kv) {
    const StackModel& S = *kv->model->stack;
    size_t n = 0;
    for (const LayerRun& r : S.spec.runs) {   // blocks: their rows of a page, rounded up per position
        const LayerSpec& L = S.spec.layers[r.layer];
        n += (size_t(L.cache_row()) * L.page_rows() + FORGE_KV_PAGE - 1) / FORGE_KV_PAGE;
    }
    return n * dense_size(S.dtype);
}
size_t stack_kv_bytes(const ForgeKV* kv, int len) {
    const StackModel& S = *kv->model->stack;
    size_t n = S.spec.buckets ? sizeof(uint32_t) : 0;
    const size_t pages = size_t(len + FORGE_KV_PAGE - 1) / FORGE_KV_PAGE;
    for (const LayerRun& r : S.spec.runs) {
        const LayerSpec& L = S.spec.layers[r.layer];
        n += (size_t(len) + pages * size_t(L.page_rows() - FORGE_KV_PAGE)) * L.cache_row() * dense_size(S.dtype) + state_bytes(L) + ring_bytes(S, L) + prev_bytes(S, L);
    }
    return n;
}

int32_t stack_kv_copy(ForgeKV* kv, int seq, int len, char* host, bool to_host) {
    ForgeModel* m = kv->model;
    const StackModel& S = *m->stack;
    auto copy = [&](char* dev, size_t bytes) -> int32_t {
        if (!bytes) return FORGE_OK;
        FORGE_CUDA(to_host ? cudaMemcpyAsync(host, dev, bytes, cudaMemcpyDeviceToHost, m->stream) : cudaMemcpyAsync(dev, host, bytes, cudaMemcpyHostToDevice, m->stream));
        host += bytes;
        return FORGE_OK;
    };
    for (size_t l = 0; l < S.spec.runs.size(); ++l) {
        const LayerSpec& L = S.spec.layers[S.spec.runs[l].layer];
        const StackCache::Run& r = kv->stack->runs[l];
        const size_t row = size_t(L.cache_row()) * dense_size(S.dtype);
        for (int t0 = 0; row && t0 < len; t0 += FORGE_KV_PAGE) {
            const int pg = kv->h_page_table[size_t(seq) * kv->pages_per_seq + t0 / FORGE_KV_PAGE];
            FORGE_TRY(copy(static_cast<char*>(r.pool) + size_t(pg) * FORGE_KV_PAGE * row, row * std::min(FORGE_KV_PAGE, len - t0)));
            const size_t blocks = size_t(L.page_rows() - FORGE_KV_PAGE);
            FORGE_TRY(copy(static_cast<char*>(r.pool) + (size_t(kv->num_pages) * FORGE_KV_PAGE + size_t(pg) * blocks) * row, row * blocks));
        }
        FORGE_TRY(copy(reinterpret_cast<char*>(r.state) + size_t(seq) * state_bytes(L), state_bytes(L)));
        FORGE_TRY(copy(static_cast<char*>(r.ring) + size_t(seq) * ring_bytes(S, L), ring_bytes(S, L)));
        FORGE_TRY(copy(static_cast<char*>(r.prev) + size_t(seq) * prev_bytes(S, L), prev_bytes(S, L)));
    }
    if (S.spec.buckets) FORGE_TRY(copy(reinterpret_cast<char*>(kv->stack->prev_token + seq), sizeof(uint32_t)));
    FORGE_CUDA(cudaStreamSynchronize(m->stream));
    return FORGE_OK;
}

// ------------------------------------------------------------------------------------------------ steps
int32_t stack_step(ForgeModel* m, ForgeKV* kv, const ForgeStepEntry* entries, int n_entries, const uint32_t* tokens, const int32_t* want, float** d_logits,
                   int trace_rows, int trace_row0) {
    StackModel& S = *m->stack;
    bool prompt_ok = S.dtype == FORGE_BF16;
    int least_pool = 0;   // of all layers
    for (const LayerSpec& L : S.spec.layers) {
        if (!L.has_latent() && !L.has_attn()) continue;
        PromptDims d = L.has_latent() ? PromptDims(L.mix) : PromptDims(L.attn);
        d.joint = L.soft.talk;
        prompt_ok = prompt_ok && attn_prefill_kv_supported(d);
        if (L.has_attn() && L.attn.pool) least_pool = least_pool ? std::min(least_pool, L.attn.pool) : L.attn.pool;
    }
    // rows: the single tokens first, then the short entries, then the prompt portions
    struct Place { int row, tok, want; };
    std::vector<Place> at_entry(n_entries);
    int tok = 0, wants = 0, rows = 0, ones = 0, single = 0, max_keys = 1;
    for (int i = 0; i < n_entries; ++i) { at_entry[i] = {0, tok, wants}; tok += entries[i].n_tokens; wants += entries[i].n_want; }
    auto is_prompt = [&](int i) { return prompt_ok && entries[i].n_tokens >= kPromptRows; };
    auto pass_of = [&](int i) { return is_prompt(i) ? 2 : entries[i].n_tokens > 1 ? 1 : 0; };
    for (int pass = 0; pass < 3; ++pass) {
        for (int i = 0; i < n_entries; ++i)
            if (pass_of(i) == pass) {
                at_entry[i].row = rows;
                rows += entries[i].n_tokens;
                if (pass < 2) max_keys = std::max(max_keys, kv->len[entries[i].seq] + entries[i].n_tokens);
            }
        if (pass == 0) ones = rows;
        if (pass < 2) single = rows;
    }
    // one upload: tokens | positions | sequences | wanted rows | context pages | prompt tiles | segments
    std::vector<int32_t> meta(size_t(3) * rows + wants);
    std::vector<int32_t> pages;
    std::vector<PromptTile> tiles;
    std::vector<PoolChunk> pools;
    std::vector<ScanSeg> segs;
    int max_seg = 0;
    for (int i = 0; i < n_entries; ++i) {
        const ForgeStepEntry& e = entries[i];
        const int base = kv->len[e.seq], r0 = at_entry[i].row;
        for (int k = 0; k < e.n_tokens; ++k) {
            meta[r0 + k] = int32_t(tokens[at_entry[i].tok + k]);
            meta[rows + r0 + k] = base + k;
            meta[2 * rows + r0 + k] = e.seq;
        }
        for (int k = 0; k < e.n_want; ++k) meta[3 * rows + at_entry[i].want + k] = r0 + want[at_entry[i].want + k];
        if (e.n_tokens > 1) { segs.push_back({r0, e.n_tokens, e.seq, base, 0, {}}); max_seg = std::max(max_seg, int(e.n_tokens)); }
        if (is_prompt(i)) {
            const int ctx0 = int(pages.size()) * FORGE_KV_PAGE, np = (base + e.n_tokens + FORGE_KV_PAGE - 1) / FORGE_KV_PAGE;
            for (int p = 0; p < np; ++p) pages.push_back(kv->h_page_table[size_t(e.seq) * kv->pages_per_seq + p]);
            const int len = base + e.n_tokens, pool0 = int(pools.size()) * FORGE_KV_PAGE;
            for (int b = 0; least_pool && b < len / least_pool; b += FORGE_KV_PAGE) pools.push_back({ctx0 / FORGE_KV_PAGE, b, len, 0});
            for (int t = 0; t < e.n_tokens; t += 128) tiles.push_back({r0 - single + t, std::min(128, e.n_tokens - t), base + t, ctx0, pool0, {}});
        }
    }
    std::stable_sort(tiles.begin(), tiles.end(), [](const PromptTile& a, const PromptTile& b) { return a.pos0 + a.rows > b.pos0 + b.rows; });   // the longest first
    const auto first_long = std::stable_partition(segs.begin(), segs.end(), [](const ScanSeg& g) { return g.n < kChunkedRows; });
    const int n_short = int(first_long - segs.begin());
    int chunks = 0;
    for (auto g = first_long; g != segs.end(); ++g) { g->chunk0 = chunks; chunks += (g->n + kRecurChunk - 1) / kRecurChunk; }
    static_assert(sizeof(ScanSeg) == 32 && sizeof(PromptTile) == 32 && sizeof(PoolChunk) == 16, "words");
    const size_t o_pages = (meta.size() + 3) & ~size_t(3), o_tiles = (o_pages + pages.size() + 3) & ~size_t(3), o_segs = o_tiles + tiles.size() * 8, o_pools = o_segs + segs.size() * 8,
                 total = o_pools + pools.size() * 4;
    meta.resize(total);
    std::copy(pages.begin(), pages.end(), meta.begin() + o_pages);
    if (!tiles.empty()) memcpy(meta.data() + o_tiles, tiles.data(), tiles.size() * sizeof(PromptTile));
    if (!segs.empty()) memcpy(meta.data() + o_segs, segs.data(), segs.size() * sizeof(ScanSeg));
    if (!pools.empty()) memcpy(meta.data() + o_pools, pools.data(), pools.size() * sizeof(PoolChunk));
    const int splits = row_splits(S, std::max(1, single), (max_keys + FORGE_KV_PAGE - 1) / FORGE_KV_PAGE), ctx_rows = int(pages.size()) * FORGE_KV_PAGE;
    FORGE_TRY(ensure_step(m, std::max(rows, wants), single, splits, rows - single, ctx_rows, rows - ones, chunks, max_keys, int(pools.size()) * FORGE_KV_PAGE, false));
    FORGE_TRY(grow(m, S.meta, total * 4));
    FORGE_TRY(grow(m, S.sel, size_t(wants) * S.width_p * dense_size(S.dtype)));
    FORGE_TRY(grow(m, S.logits, size_t(wants) * S.spec.vocab * 4));
    int32_t* dm = static_cast<int32_t*>(S.meta.p);
    FORGE_CUDA(cudaMemcpyAsync(dm, meta.data(), total * 4, cudaMemcpyHostToDevice, m->stream));
    Step s;
    s.tokens = reinterpret_cast<const uint32_t*>(dm);
    s.rows = StepRows{rows, dm + rows, dm + 2 * rows, kv->d_page_table, kv->pages_per_seq};
    for (int i = 0; i < n_entries; ++i) if (!is_prompt(i)) s.rows.fresh = std::max(s.rows.fresh, int(entries[i].n_tokens));
    s.ones = ones; s.single = single; s.splits = splits; s.max_keys = max_keys;
    s.segs = SegTable{reinterpret_cast<const ScanSeg*>(dm + o_segs), int(segs.size()), n_short, max_seg, chunks, ones, rows - ones};
    s.ctx_pages = dm + o_pages; s.ctx_rows = ctx_rows;
    s.chunks = reinterpret_cast<const PoolChunk*>(dm + o_pools); s.n_chunks = int(pools.size());
    s.tiles = reinterpret_cast<const PromptTile*>(dm + o_tiles); s.n_tiles = int(tiles.size()); s.host_tiles = tiles.data();
    s.scale_rows = std::max(rows, wants);
    if (trace_rows) { s.trace = m->trace + size_t(trace_row0) * S.spec.width; s.trace_stride = size_t(trace_rows) * S.spec.width; }
    FORGE_TRY(Sequence(m, kv, s).run());
    if (wants) {
        FORGE_TRY(gather_act_rows(S.sel.p, S.h.p, S.width_p, dm + 3 * rows, wants, S.width_p, S.dtype, m->stream));
        FORGE_TRY(run_head(m, S.sel.p, dm + 3 * rows, wants, s.scale_rows, static_cast<float*>(S.logits.p)));
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
    if (rc != FORGE_OK) { kv->len[seq] = len0; mark_lost(kv); }
    return rc;
}

int32_t stack_ensure_decode(ForgeModel* m, ForgeKV* kv, int batch) { return ensure_step(m, batch, batch, kv->stack->splits, 0, 0, 0, 0, kv->max_seq, 0, true); }

int32_t stack_decode_launches(ForgeModel* m, ForgeKV* kv, int batch, bool greedy, bool record) {
    StackModel& S = *m->stack;
    Step s;
    s.tokens = m->d_tok;
    s.rows = StepRows{batch, kv->d_seq_len, nullptr, kv->d_page_table, kv->pages_per_seq};
    s.rows.slot0 = kv->slot0;
    s.scale_rows = batch;
    s.ones = s.single = batch; s.splits = kv->stack->splits; s.max_keys = kv->max_seq;
    if (record) { s.hist = m->d_hist; s.step = m->d_step; }
    if (m->trace_on) { s.trace = m->trace; s.trace_stride = size_t(batch) * S.spec.width; }
    FORGE_TRY(Sequence(m, kv, s).run());
    FORGE_TRY(run_head(m, S.h.p, nullptr, batch, batch, m->d_logits));
    if (greedy) FORGE_TRY(argmax_slices(m->d_tok, m->d_logits, m->V, batch, m->d_amax_val, m->d_amax_idx, m->d_amax_ticket, m->stream));
    return step_advance(kv->d_seq_len, batch, m->d_step, m->stream);
}

}  // namespace forge

// ------------------------------------------------------------------------------------------------ C API
extern "C" {

int32_t forge_model_info(const ForgeModel* m, ForgeCheckpointInfo* out) {
    if (!m || !out) { set_error("bad argument to forge_model_info"); return FORGE_ERR_INVALID_ARG; }
    if (!m->stack) { set_error("not a layer-list model"); return FORGE_ERR_UNSUPPORTED; }
    stack_fill_info(m->stack->spec, out);
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
    FORGE_TRY(stack_parse(ck.config(), &spec));
    FORGE_TRY(stack_find_tensors(ck, &spec, &t));
    spec.parameters = ck.parameters();
    const int ndev = forge_device_count();
    if (ndev == 0) { set_error("no CUDA device: this backend has no CPU fallback"); return FORGE_ERR_CUDA; }
    if (device < 0 || device >= ndev) { set_error("device %d out of range (%d visible)", device, ndev); return FORGE_ERR_INVALID_ARG; }
    FORGE_CUDA(cudaSetDevice(device));
    ForgeModel* m = new ForgeModel();
    m->cfg = ForgeModelConfig{};
    m->cfg.hidden_size = spec.width; m->cfg.num_layers = int32_t(spec.runs.size()); m->cfg.vocab_size = spec.vocab;
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
            put_rows(img, dtype, spec.width, *t.top.at("embed"), 0);
            FORGE_TRY(upload(m, &S.embed, img));
        }
        if (spec.buckets) {
            std::vector<uint8_t> img((size_t(spec.buckets) + 1) * spec.width * es);
            put_rows(img, dtype, spec.width, *t.top.at("bigram"), 0);
            FORGE_TRY(upload(m, &S.bigram, img));
        }
        {
            Image head(spec.vocab, S.width_p, dtype);
            head.put(t.top.at("head"), 0);
            FORGE_TRY(head.load(m, &S.head));
        }
        if (spec.loop_times) FORGE_TRY(upload_f32(m, &S.loop_step, *t.top.at("loop.step")));
        if (spec.loop_times && !spec.adds_loop()) {   // columns [stream | embedding], each padded
            const TensorView& in = *t.top.at("loop.in");
            Image img(spec.width, 2 * S.width_p, dtype);
            for (int r = 0; r < spec.width; ++r)
                for (int c = 0; c < 2 * spec.width; ++c)
                    store(img.img.data(), dtype, size_t(r) * img.K + (c < spec.width ? c : S.width_p + c - spec.width), in, size_t(r) * 2 * spec.width + c);
            FORGE_TRY(img.load(m, &S.loop_in));
        }
        FORGE_TRY(load_norm(m, &S.final_norm, t.top, "final.norm"));
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
