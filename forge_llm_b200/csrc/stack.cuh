// Layer-list models: what a configuration describes (stack_config.cu) and what the loader makes of it (stack_model.cu).
#pragma once

#include <map>
#include <string>
#include <vector>

#include "attn_prompt.cuh"
#include "checkpoint.cuh"
#include "moe.cuh"
#include "recurrent.cuh"
#include "selective.cuh"

namespace forge {

enum class Norm { DynamicTanh, RmsPlusOne, RmsScalar };   // RmsPlusOne: the weight is stored around zero; RmsScalar: one weight for all columns
// Parallel: x += mixer(h) + ff(h) behind one norm.  Sequential: x += mixer(norm1(x)), then x += ff(norm2(x)).
// ParallelTwo: x += mixer(norm1(x)) + ff(norm2(x)).  PostNorm: x += norm1(mixer(x)), then x += norm2(ff(x)).
enum class Arrangement { Parallel, Sequential, ParallelTwo, PostNorm };
enum class Mlp { ClampedGlu, SiluGlu };
// What stands in front of a pass of the loop.  Project: a product over [stream | embedding] plus the pass's vector.  Add: the embedding
// (not in front of the first pass) and the pass's vector are added.
enum class LoopEntry { Project, Add };
struct Architecture {
    const char* name; Norm norm; Arrangement arrangement; Mlp dense; LoopEntry loop;
    bool scaled;      // embedding.scale, embedding.bigram and logit_scale of the configuration
};

enum class Mixer {
    Latent,        // latent attention
    Delta,         // gated delta rule, one decay per head
    ChannelDelta,  // gated delta rule, one decay per head and key channel
    AttnTimeMix,   // gated attention and time mixing side by side, half the sum of their normed outputs
    Softmax,       // attention with normed and rotated queries and keys
    GatedLinear,   // gated linear attention, one decay per head and key channel
    AttnSelective  // attention with mixed heads and a selective scan side by side, a weighted sum of their outputs
};
// Rotary positions: frequencies base^(-2 i / dims), scaled.
struct Rotation {
    enum Scaling { None, Linear, Yarn } scaling = None;
    int dims = 0;
    double base = 1.0, factor = 1.0, original = 0, fast = 0, slow = 0;
    bool operator<(const Rotation& o) const;
    std::vector<double> frequencies() const;
    double magnitude() const;          // of cos and sin
};
// sink: a learned score per head, else one of zero (not with mixed heads).  plain: norms of queries and keys have no weights, the output projection has a bias too, a
// mask is a plain window or one with blocks in front.  distance: a learned bias by distance.  talk: the heads' weights are mixed.
struct SoftmaxTraits { QkPost qk; bool bias = false, sink = false, plain = false, distance = false, talk = false; };
// learned biases by distance n: a bucket each up to half of them, then logarithmic ones up to the distance `longest`
struct DistanceBuckets {
    int count = 0, longest = 0;
    int of(int n) const;
};
struct LayerSpec {
    Mixer kind = Mixer::Latent;
    LatentDims mix;                          // Latent
    AttnDims attn;                           // AttnTimeMix, Softmax
    Rotation rot;                            // Latent, Softmax
    SoftmaxTraits soft;                      // Softmax, AttnSelective
    DistanceBuckets distance;
    float score_bound = 0.f;                 // plain: no score in front of the bias is larger or smaller than this
    int blend_layer = -1;                    // values are blended with those of this earlier layer
    bool blends = false;                     // takes part in it (the first such layer lends its values)
    SelectiveDims sel;                       // AttnSelective
    float left_scale = 1.f, right_scale = 1.f;
    RecurDims rec;                           // Delta, ChannelDelta, AttnTimeMix, GatedLinear
    int decay_rank = 0, gate_rank = 0;       // inner sizes of the two-step projections, from the tensors' shapes
    double tau = 1.0;                        // GatedLinear: a decay is sigmoid(z)^(1 / tau)
    int ff = 0;                              // 0: no feed-forward
    RouterDims router;                       // experts > 0: a mixture of experts of size ff
    int shared_ff = 0;                       // beside a shared expert
    float limit = 0.f;
    int weights_of = -1;                     // layer whose tensors are used
    bool has_attn() const { return kind == Mixer::AttnTimeMix || kind == Mixer::Softmax || kind == Mixer::AttnSelective; }
    bool has_latent() const { return kind == Mixer::Latent; }
    bool has_state() const { return kind != Mixer::Latent && kind != Mixer::Softmax; }
    bool has_rotation() const { return kind == Mixer::Latent || kind == Mixer::Softmax || kind == Mixer::AttnSelective; }
    // what a sequence keeps besides cache rows: f32 state values and values of the convolution's ring
    size_t state_values() const { return kind == Mixer::AttnSelective ? sel.state_values() : has_state() ? rec.state_values() : 0; }
    size_t ring_values() const { return kind == Mixer::AttnSelective ? sel.ring_values() : has_state() ? rec.ring_values() : 0; }
    int page_rows() const { return FORGE_KV_PAGE + (has_attn() ? attn.pool_slots() : 0); }   // cache rows of a page, those of blocks included
    int cache_row() const { return has_latent() ? mix.row() : has_attn() ? attn.row() : 0; }   // values per position, padding included
};
struct LayerRun { int layer, pass; };   // pass >= 0: this pass of the loop starts in front of the layer
struct StackSpec {
    const Architecture* arch = nullptr;
    int width = 0, vocab = 0;
    float eps = 0.f;
    float embed_scale = 1.f, logit_scale = 1.f;
    int buckets = 0, mul_prev = 0, mul_cur = 0;          // bigram embedding; buckets = 0: none
    std::vector<LayerSpec> layers;
    int loop_start = 0, loop_stop = 0, loop_times = 0;   // times = 0: no loop
    std::vector<LayerRun> runs;
    int64_t parameters = 0;
    bool adds_loop() const { return loop_times > 0 && arch->loop == LoopEntry::Add; }
};

typedef std::map<std::string, const TensorView*> TensorSet;   // by name, a layer's without its prefix
struct StackTensors { TensorSet top; std::vector<TensorSet> layers; };

// Reads and checks config.json; then every tensor it calls for, with its shape (also fills in the sizes that only shapes give).
int32_t stack_parse(const Json& config, StackSpec* s);
int32_t stack_find_tensors(const Checkpoint& ck, StackSpec* s, StackTensors* t);
void stack_fill_info(const StackSpec& s, ForgeCheckpointInfo* out);

}  // namespace forge
