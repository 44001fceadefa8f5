// Registry of architectures and the reader of a layer-list model's configuration and tensor names (host code).
#include <algorithm>
#include <cmath>
#include <cstdio>
#include <cstring>
#include <tuple>

#include "stack.cuh"

namespace forge {

static const Architecture kArchitectures[] = {
    {"Bolenex", Norm::DynamicTanh, Arrangement::Parallel, Mlp::ClampedGlu, LoopEntry::Project, false},
    {"Robazen", Norm::DynamicTanh, Arrangement::Sequential, Mlp::SiluGlu, LoopEntry::Project, false},
    {"Mokatar", Norm::RmsPlusOne, Arrangement::ParallelTwo, Mlp::SiluGlu, LoopEntry::Add, true},
    {"Tarulix", Norm::RmsScalar, Arrangement::PostNorm, Mlp::SiluGlu, LoopEntry::Project, false},
};
// mixers by architecture and the name a layer's "type" gives them
struct MixerName { const char* architecture; const char* name; Mixer kind; SoftmaxTraits soft; Rotation::Scaling scaling; };
static SoftmaxTraits traits(QkPost::Scope norm, bool interleaved, bool bias, bool sink) {
    SoftmaxTraits t;
    t.qk.norm = norm; t.qk.interleaved = interleaved; t.bias = bias; t.sink = sink;
    return t;
}
static SoftmaxTraits plain_traits(bool distance, bool sink, bool talk) {
    SoftmaxTraits t = traits(QkPost::PER_HEAD, false, true, sink);
    t.plain = true; t.distance = distance; t.talk = talk;
    return t;
}
static const MixerName kMixers[] = {
    {"Bolenex", "latent_attention", Mixer::Latent, {}, Rotation::None},
    {"Robazen", "latent_attention", Mixer::Latent, {}, Rotation::None},
    {"Robazen", "delta", Mixer::Delta, {}, Rotation::None},
    {"Robazen", "channel_delta", Mixer::ChannelDelta, {}, Rotation::None},
    {"Robazen", "parallel", Mixer::AttnTimeMix, {}, Rotation::None},
    {"Mokatar", "attention", Mixer::Softmax, traits(QkPost::PER_HEAD, true, false, true), Rotation::Yarn},
    {"Mokatar", "attention_2", Mixer::Softmax, traits(QkPost::WHOLE, false, true, false), Rotation::Linear},
    {"Mokatar", "gla", Mixer::GatedLinear, {}, Rotation::None},
    {"Tarulix", "attention", Mixer::Softmax, plain_traits(true, true, false), Rotation::None},
    {"Tarulix", "parallel", Mixer::AttnSelective, plain_traits(false, false, true), Rotation::None},
};

int DistanceBuckets::of(int n) const {
    const int half = count / 2;
    if (n < half) return n;
    if (half < 1 || longest <= half) return count - 1;
    // the quotient of logarithms is an integer where a bucket begins: there rounding must not decide
    const double x = std::log(double(n) / half) / std::log(double(longest) / half) * (count - half), near = std::round(x);
    const double b = half + (std::fabs(x - near) < 1e-9 ? near : std::floor(x));
    return b < count - 1 ? int(b) : count - 1;
}

bool Rotation::operator<(const Rotation& o) const {
    return std::tie(scaling, dims, base, factor, original, fast, slow) < std::tie(o.scaling, o.dims, o.base, o.factor, o.original, o.fast, o.slow);
}
// Yarn: pairs that turn more than `fast` times over the original length keep their frequency, those below `slow` are divided by the
// factor, with a ramp over the pairs between.
std::vector<double> Rotation::frequencies() const {
    std::vector<double> f;
    for (int i = 0; i < dims / 2; ++i) f.push_back(std::pow(base, -2.0 * i / dims));
    if (scaling == Linear) for (double& x : f) x /= factor;
    if (scaling == Yarn && dims > 0) {
        const double pi = 3.14159265358979323846;
        auto pair_of = [&](double turns) { return dims * std::log(original / (2 * pi * turns)) / (2 * std::log(base)); };
        const double lo = std::max(std::floor(pair_of(fast)), 0.0), hi = std::min(std::ceil(pair_of(slow)), double(dims - 1));
        for (int i = 0; i < dims / 2; ++i) {
            const double ramp = std::min(1.0, std::max(0.0, (i - lo) / std::max(hi - lo, 0.001)));
            f[i] = f[i] / factor * ramp + f[i] * (1 - ramp);
        }
    }
    return f;
}
double Rotation::magnitude() const { return scaling == Yarn ? 0.1 * std::log(factor) + 1.0 : 1.0; }

namespace {

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
        FORGE_TRY(need_num(rot, "base", &L->rot.base));
        L->rot.dims = d.rot_dims;
        if (d.rot_dims > d.rot || d.rot_dims % 2 || !(L->rot.base > 0)) { set_error("config.json: rot.dims %d does not fit rot_dim %d", d.rot_dims, d.rot); return FORGE_ERR_SHAPE; }
    }
    d.scale = float(scale); d.eps = eps;
    d.rank_p = pad_to(d.rank, 64); d.rot_p = pad_to(d.rot, 64); d.dim_p = pad_to(d.dim, 64); d.vdim_p = pad_to(d.vdim, 64);
    return FORGE_OK;
}

int32_t heads_fit(int heads, int groups) {
    if (heads % groups) { set_error("config.json: %d heads do not share %d kv_heads evenly", heads, groups); return FORGE_ERR_SHAPE; }
    return FORGE_OK;
}

int32_t check_recur(const RecurDims& d) {
    if (recur_supported(d)) return FORGE_OK;
    set_error("recurrent mixer: head sizes %d / %d with %d taps are not supported", d.dim, d.vdim, d.taps);
    return FORGE_ERR_UNSUPPORTED;
}

int32_t parse_delta(const Json* m, float eps, bool channel, LayerSpec* L) {
    RecurDims& d = L->rec;
    FORGE_TRY(need_int(m, "heads", &d.heads));
    FORGE_TRY(need_int(m, "kv_heads", &d.groups));
    FORGE_TRY(need_int(m, "dim", &d.dim));
    FORGE_TRY(need_int(m, "vdim", &d.vdim));
    FORGE_TRY(need_int(m, "conv", &d.taps));
    FORGE_TRY(heads_fit(d.heads, d.groups));
    d.rule = Rule::Delta; d.channel = channel; d.eps = eps;
    d.q_scale = float(1.0 / std::sqrt(double(d.dim)));
    return check_recur(d);
}

// mask: "size" is the length of chunks, or of a sliding window: beside "keep_first" kept tokens, alone, or behind blocks of "pool" tokens
enum class MaskKind { Chunks, Kept, Window, Pooled };
int32_t parse_attn(const Json* m, MaskKind kind, AttnDims* d) {
    double scale, cap = 0;
    FORGE_TRY(need_int(m, "heads", &d->heads));
    FORGE_TRY(need_int(m, "kv_heads", &d->groups));
    FORGE_TRY(need_int(m, "dim", &d->dim));
    FORGE_TRY(need_int(m, "vdim", &d->vdim));
    FORGE_TRY(need_num(m, "scale", &scale));
    const Json* c = m->get("softcap");
    if (c && c->kind != Json::Null) {
        FORGE_TRY(need_num(m, "softcap", &cap));
        if (!(cap > 0)) { set_error("config.json: \"softcap\" must be positive"); return FORGE_ERR_SHAPE; }
    }
    const Json* mask = m->get("mask");
    if (mask && mask->kind != Json::Null) {
        FORGE_TRY(need_int(mask, "size", kind == MaskKind::Chunks ? &d->chunk : &d->window));
        if (kind == MaskKind::Kept) FORGE_TRY(need_int(mask, "keep_first", &d->keep, 0));
        if (kind == MaskKind::Pooled) FORGE_TRY(need_int(mask, "pool", &d->pool));
    }
    FORGE_TRY(heads_fit(d->heads, d->groups));
    d->scale = float(scale); d->softcap = float(cap);
    d->dim_p = pad_to(d->dim, 64); d->vdim_p = pad_to(d->vdim, 64);
    if (attn_rows_supported(*d)) return FORGE_OK;
    set_error("attention: head sizes %d / %d are not supported", d->dim, d->vdim);
    return FORGE_ERR_UNSUPPORTED;
}

int32_t parse_pair(const Json* m, float eps, LayerSpec* L) {
    const Json* left = m ? m->get("left") : nullptr;
    const Json* right = m ? m->get("right") : nullptr;
    FORGE_TRY(parse_attn(left ? left : m, MaskKind::Chunks, &L->attn));
    RecurDims& d = L->rec;
    FORGE_TRY(need_int(right, "heads", &d.heads));
    FORGE_TRY(need_int(right, "dim", &d.dim));
    d.groups = d.heads; d.vdim = d.dim; d.channel = true; d.eps = eps;
    return check_recur(d);
}

int32_t parse_rotation(const Json* r, Rotation::Scaling kind, int dim, Rotation* rot) {
    FORGE_TRY(need_int(r, "dims", &rot->dims, 0));
    FORGE_TRY(need_num(r, "base", &rot->base));
    const Json* s = r->get("scaling");
    if (s && s->kind != Json::Null && kind != Rotation::None) {
        rot->scaling = kind;
        FORGE_TRY(need_num(s, "factor", &rot->factor));
        if (kind == Rotation::Yarn) {
            FORGE_TRY(need_num(s, "original", &rot->original));
            FORGE_TRY(need_num(s, "fast", &rot->fast));
            FORGE_TRY(need_num(s, "slow", &rot->slow));
        }
    }
    const bool yarn = rot->scaling == Rotation::Yarn;
    if (rot->dims > dim || rot->dims % 2 || !(rot->base > 0) || !(rot->factor > 0) || (yarn && (!(rot->original > 0) || !(rot->fast > 0) || !(rot->slow > 0) || rot->base == 1.0))) {
        set_error("config.json: \"rot\" does not fit heads of %d", dim);
        return FORGE_ERR_SHAPE;
    }
    return FORGE_OK;
}

int32_t parse_softmax(const Json* m, float eps, const MixerName& name, LayerSpec* L) {
    const SoftmaxTraits& soft = name.soft;
    AttnDims& a = L->attn;
    FORGE_TRY(parse_attn(m, !soft.plain ? MaskKind::Kept : soft.talk ? MaskKind::Pooled : MaskKind::Window, &a));
    if (a.dim > 512 || (soft.talk && !talk_rows_supported(a))) { set_error("attention: %d heads of %d / %d are not supported", a.heads, a.dim, a.vdim); return FORGE_ERR_UNSUPPORTED; }
    if (!soft.plain || m->get("rot")) FORGE_TRY(parse_rotation(m->get("rot"), name.scaling, a.dim, &L->rot));
    if (soft.distance) {
        FORGE_TRY(need_int(m, "bias_max", &L->distance.longest));
        const Json* v = m->get("v_mix");
        L->blends = v && v->kind == Json::Bool && v->flag;
        a.bias_n = a.window > 0 && a.window <= L->distance.longest ? a.window : L->distance.longest + 1;   // distances further on share the last bucket
    }
    L->soft = soft;
    L->soft.qk.eps = eps; L->soft.qk.rot_dims = L->rot.dims;
    if (soft.plain) {   // queries and keys are no longer than the root of their size (a little for rounding)
        L->score_bound = 1.01f * std::fabs(a.scale) * float(a.dim);
        if (a.softcap > 0.f) L->score_bound = std::min(L->score_bound, a.softcap);
    }
    return FORGE_OK;
}

int32_t parse_attn_selective(const Json* m, float eps, const MixerName& name, LayerSpec* L) {
    const Json *left = m->get("left"), *right = m->get("right");
    double l, r;
    if (!left || left->kind != Json::Object) { set_error("config.json: \"left\" must be an object"); return FORGE_ERR_SHAPE; }
    FORGE_TRY(need_num(m, "left_scale", &l));
    FORGE_TRY(need_num(m, "right_scale", &r));
    L->left_scale = float(l); L->right_scale = float(r);
    FORGE_TRY(parse_softmax(left, eps, name, L));
    SelectiveDims& d = L->sel;
    FORGE_TRY(need_int(right, "inner", &d.inner));
    FORGE_TRY(need_int(right, "state", &d.state));
    FORGE_TRY(need_int(right, "dt_rank", &d.rank));
    FORGE_TRY(need_int(right, "conv", &d.taps));
    if (selective_supported(d)) return FORGE_OK;
    set_error("selective scan: %d states with %d taps are not supported", d.state, d.taps);
    return FORGE_ERR_UNSUPPORTED;
}

int32_t parse_linear(const Json* m, float eps, LayerSpec* L) {
    RecurDims& d = L->rec;
    FORGE_TRY(need_int(m, "heads", &d.heads));
    FORGE_TRY(need_int(m, "dim", &d.dim));
    FORGE_TRY(need_int(m, "vdim", &d.vdim));
    FORGE_TRY(need_num(m, "tau", &L->tau));
    if (!(L->tau > 0)) { set_error("config.json: \"tau\" must be positive"); return FORGE_ERR_SHAPE; }
    d.groups = d.heads; d.rule = Rule::Linear; d.channel = true; d.eps = eps;
    d.q_scale = float(1.0 / std::sqrt(double(d.dim)));
    return check_recur(d);
}

int32_t parse_experts(const Json* mlp, int layer, bool shared, LayerSpec* L) {
    const Json* router = mlp->get("router");
    FORGE_TRY(need_int(mlp->get("expert"), "ff", &L->ff));
    FORGE_TRY(need_int(router, "experts", &L->router.experts));
    FORGE_TRY(need_int(router, "top", &L->router.top));
    if (shared) {
        FORGE_TRY(need_int(mlp->get("shared"), "ff", &L->shared_ff));
        FORGE_TRY(need_int(router, "identity", &L->router.identity, 0));
        L->router.always = (L->shared_ff + L->ff - 1) / L->ff;
    }
    if (L->router.top > L->router.choices()) { set_error("layer %d: top %d of %d experts", layer, L->router.top, L->router.choices()); return FORGE_ERR_SHAPE; }
    if (L->router.always > kMaxExperts) { set_error("layer %d: a shared expert of %d beside experts of %d is not supported", layer, L->shared_ff, L->ff); return FORGE_ERR_UNSUPPORTED; }
    if (L->router.choices() > kMaxExperts) { set_error("layer %d: %d experts are not supported", layer, L->router.choices()); return FORGE_ERR_UNSUPPORTED; }
    return FORGE_OK;
}

bool same_sizes(const LayerSpec& A, const LayerSpec& B) {
    const LatentDims &a = A.mix, &b = B.mix;
    return A.kind == Mixer::Latent && B.kind == Mixer::Latent && a.heads == b.heads && a.dim == b.dim && a.rot == b.rot && a.vdim == b.vdim && a.rank == b.rank && A.ff == B.ff;
}

}  // namespace

int32_t stack_parse(const Json& c, StackSpec* s) {
    std::string name;
    FORGE_TRY(need_string(&c, "architecture", &name));
    for (const Architecture& a : kArchitectures) if (name == a.name) s->arch = &a;
    if (!s->arch) { set_error("architecture \"%s\" is not registered", name.c_str()); return FORGE_ERR_UNSUPPORTED; }
    FORGE_TRY(need_int(&c, "width", &s->width));
    FORGE_TRY(need_int(&c, "vocab", &s->vocab));
    double eps;
    FORGE_TRY(need_num(c.get("norm"), "eps", &eps));
    s->eps = float(eps);
    if (s->arch->scaled) {
        double scale;
        const Json* e = c.get("embedding");
        FORGE_TRY(need_num(e, "scale", &scale));
        s->embed_scale = float(scale);
        const Json* b = e->get("bigram");
        if (b && b->kind != Json::Null) {
            FORGE_TRY(need_int(b, "buckets", &s->buckets));
            FORGE_TRY(need_int(b, "mul_prev", &s->mul_prev, 0));
            FORGE_TRY(need_int(b, "mul_cur", &s->mul_cur, 0));
        }
        FORGE_TRY(need_num(&c, "logit_scale", &scale));
        s->logit_scale = float(scale);
    }
    const Json* layers = c.get("layers");
    if (!layers || layers->kind != Json::Array || layers->items.empty()) { set_error("config.json: \"layers\" must list at least one layer"); return FORGE_ERR_SHAPE; }
    const int n = int(layers->items.size());
    for (int i = 0; i < n; ++i) {
        const Json& e = layers->items[i];
        LayerSpec L;
        std::string type;
        FORGE_TRY(need_string(&e, "type", &type));
        const MixerName* known = nullptr;
        for (const MixerName& m : kMixers) if (type == m.name && !strcmp(s->arch->name, m.architecture)) { L.kind = m.kind; known = &m; }
        if (!known) { set_error("layer %d: mixer \"%s\" is not supported", i, type.c_str()); return FORGE_ERR_UNSUPPORTED; }
        const Json* mx = e.get("mixer");
        if (!mx || mx->kind != Json::Object) { set_error("layer %d: \"mixer\" must be an object", i); return FORGE_ERR_SHAPE; }
        switch (L.kind) {
            case Mixer::Latent: FORGE_TRY(parse_latent(mx, s->eps, &L)); break;
            case Mixer::Delta: FORGE_TRY(parse_delta(mx, s->eps, false, &L)); break;
            case Mixer::ChannelDelta: FORGE_TRY(parse_delta(mx, s->eps, true, &L)); break;
            case Mixer::AttnTimeMix: FORGE_TRY(parse_pair(mx, s->eps, &L)); break;
            case Mixer::Softmax: FORGE_TRY(parse_softmax(mx, s->eps, *known, &L)); break;
            case Mixer::GatedLinear: FORGE_TRY(parse_linear(mx, s->eps, &L)); break;
            case Mixer::AttnSelective: FORGE_TRY(parse_attn_selective(mx, s->eps, *known, &L)); break;
        }
        const Json* mlp = e.get("mlp");
        if (mlp && mlp->kind != Json::Null) {
            std::string kind;
            FORGE_TRY(need_string(mlp, "kind", &kind));
            const bool post = s->arch->arrangement == Arrangement::PostNorm, experts = kind == "moe" && (post || s->arch->arrangement == Arrangement::ParallelTwo);
            if ((kind != "dense" || post) && !experts) { set_error("layer %d: feed-forward \"%s\" is not supported", i, kind.c_str()); return FORGE_ERR_UNSUPPORTED; }
            if (experts) FORGE_TRY(parse_experts(mlp, i, post, &L));
            else FORGE_TRY(need_int(mlp, "ff", &L.ff));
            if (s->arch->dense == Mlp::ClampedGlu) {
                double limit;
                FORGE_TRY(need_num(mlp, "limit", &limit));
                L.limit = float(limit);
            }
        }
        const Json* of = e.get("weights_of");
        if (of && of->kind != Json::Null) {
            FORGE_TRY(need_int(&e, "weights_of", &L.weights_of, 0));
            if (L.weights_of >= n || L.weights_of == i) { set_error("layer %d: weights_of %d is not another layer", i, L.weights_of); return FORGE_ERR_SHAPE; }
        }
        s->layers.push_back(L);
    }
    for (int i = 0; i < n; ++i) {
        const LayerSpec& L = s->layers[i];
        if (L.weights_of < 0) continue;
        const LayerSpec& O = s->layers[L.weights_of];
        if (O.weights_of >= 0 || !same_sizes(L, O)) {
            set_error("layer %d: weights_of %d names a layer of other sizes or without tensors", i, L.weights_of);
            return FORGE_ERR_SHAPE;
        }
    }
    int lender = -1;
    for (int i = 0; i < n; ++i) {
        LayerSpec& L = s->layers[i];
        if (!L.blends) continue;
        if (lender < 0) { lender = i; continue; }
        const AttnDims &a = L.attn, &b = s->layers[lender].attn;
        if (a.groups != b.groups || a.vdim != b.vdim) { set_error("layer %d: its values cannot be blended with those of layer %d", i, lender); return FORGE_ERR_SHAPE; }
        L.blend_layer = lender;
    }
    const Json* loop = c.get("loop");
    if (loop && loop->kind != Json::Null) {
        FORGE_TRY(need_int(loop, "start", &s->loop_start, 0));
        FORGE_TRY(need_int(loop, "stop", &s->loop_stop));
        FORGE_TRY(need_int(loop, "times", &s->loop_times));
        if (s->loop_start >= s->loop_stop || s->loop_stop > n || s->loop_times > 4096) { set_error("config.json: loop %d .. %d of %d layers", s->loop_start, s->loop_stop, n); return FORGE_ERR_SHAPE; }
    }
    for (int i = 0; i < n; ++i) {
        if (s->loop_times == 0 || i < s->loop_start || i >= s->loop_stop) { s->runs.push_back({i, -1}); continue; }
        for (int t = 0; t < s->loop_times; ++t)
            for (int l = s->loop_start; l < s->loop_stop; ++l) s->runs.push_back({l, l == s->loop_start ? t : -1});
        i = s->loop_stop - 1;
    }
    return FORGE_OK;
}

int32_t stack_find_tensors(const Checkpoint& ck, StackSpec* s, StackTensors* t) {
    const int64_t W = s->width, V = s->vocab;
    TensorSet* set = &t->top;
    std::string prefix;
    auto get = [&](const std::string& name, std::vector<int64_t> shape) -> int32_t {
        const TensorView* v = ck.tensor(prefix + name, shape);
        if (!v) return FORGE_ERR_SHAPE;
        (*set)[name] = v;
        return FORGE_OK;
    };
    auto norm = [&](const std::string& name) -> int32_t {
        if (s->arch->norm == Norm::RmsScalar) return get(name, {});
        FORGE_TRY(get(name, {W}));
        if (s->arch->norm != Norm::DynamicTanh) return FORGE_OK;
        FORGE_TRY(get(name + ".b", {W}));
        return get(name + ".alpha", {});
    };
    // queries, keys and values with their biases, the output's, behind `at`
    auto plain_attention = [&](const std::string& at, LayerSpec& L) -> int32_t {
        const AttnDims& a = L.attn;
        const int64_t q = int64_t(a.heads) * a.dim, k = int64_t(a.groups) * a.dim, v = int64_t(a.groups) * a.vdim;
        FORGE_TRY(get(at + "q", {q, W})); FORGE_TRY(get(at + "k", {k, W})); FORGE_TRY(get(at + "v", {v, W}));
        FORGE_TRY(get(at + "q.b", {q})); FORGE_TRY(get(at + "k.b", {k})); FORGE_TRY(get(at + "v.b", {v}));
        if (L.soft.distance) {
            const TensorView* rel = ck.find(prefix + at + "rel");
            if (!rel || rel->shape.size() != 2 || rel->shape[0] < 2 || rel->shape[0] > (1 << 20)) { set_error("tensor \"%srel\" is missing or no matrix", (prefix + at).c_str()); return FORGE_ERR_SHAPE; }
            L.distance.count = int(rel->shape[0]);
            FORGE_TRY(get(at + "rel", {rel->shape[0], a.heads}));
        }
        if (L.soft.sink) FORGE_TRY(get(at + "sink", {a.heads}));
        if (L.soft.talk) FORGE_TRY(get(at + "talk", {a.heads, a.heads}));
        if (L.blend_layer >= 0) FORGE_TRY(get(at + "vmix", {}));
        FORGE_TRY(get(at + "o", {W, int64_t(a.heads) * a.vdim}));
        return get(at + "o.b", {W});
    };
    // rows of a matrix [rank][cols] whose first size only its shape gives
    auto rank_of = [&](const std::string& name, int* rank) -> int32_t {
        const TensorView* v = ck.find(prefix + name);
        if (!v || v->shape.size() != 2 || v->shape[0] < 1 || v->shape[0] > (1 << 20)) { set_error("tensor \"%s\" is missing or no matrix", (prefix + name).c_str()); return FORGE_ERR_SHAPE; }
        *rank = int(v->shape[0]);
        return get(name, {v->shape[0], W});
    };
    FORGE_TRY(get("embed", {V, W}));
    FORGE_TRY(get("head", {V, W}));
    FORGE_TRY(norm("final.norm"));
    if (s->buckets) FORGE_TRY(get("bigram", {int64_t(s->buckets) + 1, W}));
    if (s->loop_times && s->arch->loop == LoopEntry::Project) FORGE_TRY(get("loop.in", {W, 2 * W}));
    if (s->loop_times) FORGE_TRY(get("loop.step", {s->loop_times, W}));
    for (size_t i = 0; i < s->layers.size(); ++i) {
        t->layers.push_back(TensorSet{});
        LayerSpec& L = s->layers[i];
        if (L.weights_of >= 0) continue;
        set = &t->layers.back();
        prefix = "l" + std::to_string(i) + ".";
        FORGE_TRY(norm("norm1"));
        const RecurDims& r = L.rec;
        const int64_t H = r.heads, D = int64_t(r.heads) * r.dim, HV = int64_t(r.heads) * r.vdim;
        switch (L.kind) {
            case Mixer::Latent: {
                const LatentDims& d = L.mix;
                const int64_t hv = int64_t(d.heads) * d.vdim;
                FORGE_TRY(get("mix.q", {int64_t(d.heads) * (d.dim + d.rot), W}));
                FORGE_TRY(get("mix.dkv", {d.rank + d.rot, W}));
                FORGE_TRY(get("mix.dkv.norm", {d.rank}));
                FORGE_TRY(get("mix.uk", {int64_t(d.heads) * d.dim, d.rank}));
                FORGE_TRY(get("mix.uv", {hv, d.rank}));
                FORGE_TRY(get("mix.g", {hv, W}));
                FORGE_TRY(get("mix.o", {W, hv}));
                break;
            }
            case Mixer::Delta:
            case Mixer::ChannelDelta: {
                FORGE_TRY(get("mix.q", {r.qk(), W})); FORGE_TRY(get("mix.q.conv", {r.qk(), r.taps}));
                FORGE_TRY(get("mix.k", {r.qk(), W})); FORGE_TRY(get("mix.k.conv", {r.qk(), r.taps}));
                FORGE_TRY(get("mix.v", {HV, W})); FORGE_TRY(get("mix.v.conv", {HV, r.taps}));
                FORGE_TRY(get("mix.b", {H, W}));
                FORGE_TRY(get("mix.A_log", {H}));
                FORGE_TRY(get("mix.norm", {r.vdim}));
                FORGE_TRY(get("mix.o", {W, HV}));
                if (L.kind == Mixer::Delta) {
                    FORGE_TRY(get("mix.a", {H, W})); FORGE_TRY(get("mix.dt_bias", {H}));
                    FORGE_TRY(get("mix.g", {HV, W}));
                } else {
                    FORGE_TRY(rank_of("mix.a1", &L.decay_rank)); FORGE_TRY(get("mix.a2", {D, L.decay_rank}));
                    FORGE_TRY(get("mix.dt_bias", {D}));
                    FORGE_TRY(rank_of("mix.g1", &L.gate_rank)); FORGE_TRY(get("mix.g2", {HV, L.gate_rank}));
                }
                break;
            }
            case Mixer::AttnTimeMix: {
                const AttnDims& a = L.attn;
                FORGE_TRY(get("mix.left.q", {int64_t(a.heads) * a.dim, W}));
                FORGE_TRY(get("mix.left.k", {int64_t(a.groups) * a.dim, W}));
                FORGE_TRY(get("mix.left.v", {int64_t(a.groups) * a.vdim, W}));
                FORGE_TRY(get("mix.left.g", {a.heads, W}));
                FORGE_TRY(get("mix.left.o", {W, int64_t(a.heads) * a.vdim}));
                FORGE_TRY(get("mix.left.out", {W}));
                for (const char* x : {"r", "k", "v", "g"}) FORGE_TRY(get(std::string("mix.right.") + x, {D, W}));
                for (const char* x : {"r", "k", "v", "g", "w"}) FORGE_TRY(get(std::string("mix.right.mu.") + x, {W}));
                FORGE_TRY(rank_of("mix.right.w1", &L.decay_rank)); FORGE_TRY(get("mix.right.w2", {D, L.decay_rank}));
                FORGE_TRY(get("mix.right.w0", {D}));
                FORGE_TRY(get("mix.right.u", {H, r.dim}));
                FORGE_TRY(get("mix.right.norm", {D}));
                FORGE_TRY(get("mix.right.o", {W, D}));
                FORGE_TRY(get("mix.right.out", {W}));
                break;
            }
            case Mixer::AttnSelective: {
                const SelectiveDims& d = L.sel;
                FORGE_TRY(plain_attention("mix.left.", L));
                FORGE_TRY(get("mix.right.in", {2 * int64_t(d.inner), W}));
                FORGE_TRY(get("mix.right.conv", {d.inner, d.taps})); FORGE_TRY(get("mix.right.conv.b", {d.inner}));
                FORGE_TRY(get("mix.right.x", {int64_t(d.rank) + 2 * d.state, d.inner}));
                FORGE_TRY(get("mix.right.dt", {d.inner, d.rank})); FORGE_TRY(get("mix.right.dt.b", {d.inner}));
                FORGE_TRY(get("mix.right.A_log", {d.inner, d.state})); FORGE_TRY(get("mix.right.D", {d.inner}));
                FORGE_TRY(get("mix.right.o", {W, d.inner}));
                break;
            }
            case Mixer::Softmax: {
                if (L.soft.plain) { FORGE_TRY(plain_attention("mix.", L)); break; }
                const AttnDims& a = L.attn;
                const int64_t q = int64_t(a.heads) * a.dim, k = int64_t(a.groups) * a.dim, v = int64_t(a.groups) * a.vdim;
                const bool whole = L.soft.qk.norm == QkPost::WHOLE;
                FORGE_TRY(get("mix.q", {q, W})); FORGE_TRY(get("mix.k", {k, W})); FORGE_TRY(get("mix.v", {v, W}));
                if (L.soft.bias) { FORGE_TRY(get("mix.q.b", {q})); FORGE_TRY(get("mix.k.b", {k})); FORGE_TRY(get("mix.v.b", {v})); }
                FORGE_TRY(get("mix.q.norm", {whole ? q : a.dim})); FORGE_TRY(get("mix.k.norm", {whole ? k : a.dim}));
                if (L.soft.sink) FORGE_TRY(get("mix.sink", {a.heads}));
                FORGE_TRY(get("mix.o", {W, int64_t(a.heads) * a.vdim}));
                break;
            }
            case Mixer::GatedLinear:
                FORGE_TRY(get("mix.q", {D, W})); FORGE_TRY(get("mix.k", {D, W})); FORGE_TRY(get("mix.v", {HV, W}));
                FORGE_TRY(rank_of("mix.a1", &L.decay_rank)); FORGE_TRY(get("mix.a2", {D, L.decay_rank})); FORGE_TRY(get("mix.a2.b", {D}));
                FORGE_TRY(get("mix.g", {HV, W}));
                FORGE_TRY(get("mix.norm", {r.vdim}));
                FORGE_TRY(get("mix.o", {W, HV}));
                break;
        }
        if (L.ff && s->arch->arrangement != Arrangement::Parallel) FORGE_TRY(norm("norm2"));
        for (int e = 0; e < L.router.experts; ++e) {
            const std::string x = "mlp.e" + std::to_string(e);
            FORGE_TRY(get(x + ".gate", {L.ff, W})); FORGE_TRY(get(x + ".up", {L.ff, W})); FORGE_TRY(get(x + ".down", {W, L.ff}));
        }
        if (L.router.experts) {
            FORGE_TRY(get("mlp.router", {L.router.choices(), W}));
            FORGE_TRY(get(L.shared_ff ? "mlp.correction" : "mlp.router.b", {L.router.choices()}));
        }
        if (L.shared_ff) { FORGE_TRY(get("mlp.shared.gate", {L.shared_ff, W})); FORGE_TRY(get("mlp.shared.up", {L.shared_ff, W})); FORGE_TRY(get("mlp.shared.down", {W, L.shared_ff})); }
        if (L.ff && !L.router.experts) {
            FORGE_TRY(get("mlp.gate", {L.ff, W}));
            FORGE_TRY(get("mlp.up", {L.ff, W}));
            FORGE_TRY(get("mlp.down", {W, L.ff}));
        }
    }
    return FORGE_OK;
}

void stack_fill_info(const StackSpec& s, ForgeCheckpointInfo* out) {
    memset(out, 0, sizeof(*out));
    snprintf(out->architecture, sizeof out->architecture, "%s", s.arch->name);
    out->hidden_size = s.width; out->vocab_size = s.vocab; out->num_layers = int32_t(s.runs.size());
    out->parameters = s.parameters;
    for (const LayerSpec& L : s.layers) out->num_weight_layers += L.weights_of < 0;
    for (const LayerRun& r : s.runs) {
        const LayerSpec& L = s.layers[r.layer];
        out->cache_values_per_token += L.cache_row();   // (rows of blocks: pool_slots() per page more)
        if (L.has_state()) out->state_values_per_sequence += int64_t(L.state_values() + L.ring_values()) + (L.kind == Mixer::AttnTimeMix ? s.width : 0);
    }
    if (s.buckets) out->state_values_per_sequence += 1;   // the last token
}

}  // namespace forge

// ------------------------------------------------------------------------------------------------ C API
using namespace forge;

extern "C" int32_t forge_checkpoint_info(const char* dir, ForgeCheckpointInfo* out) {
    if (!dir || !out) { set_error("bad argument to forge_checkpoint_info"); return FORGE_ERR_INVALID_ARG; }
    Checkpoint ck;
    StackSpec s;
    StackTensors t;
    FORGE_TRY(ck.open(dir));
    FORGE_TRY(stack_parse(ck.config(), &s));
    FORGE_TRY(stack_find_tensors(ck, &s, &t));
    s.parameters = ck.parameters();
    stack_fill_info(s, out);
    return FORGE_OK;
}
