// Layer-list models: what a configuration describes (stack_config.cu) and what the loader makes of it (stack_model.cu).
#pragma once

#include <map>
#include <string>
#include <vector>

#include "attn_prompt.cuh"
#include "checkpoint.cuh"
#include "moe.cuh"
#include "recurrent.cuh"

namespace forge {

enum class Norm { DynamicTanh, RmsPlusOne };   // RmsPlusOne: the weight is stored around zero
// Parallel: x += mixer(h) + ff(h) behind one norm.  Sequential: x += mixer(norm1(x)), then x += ff(norm2(x)).
// ParallelTwo: x += mixer(norm1(x)) + ff(norm2(x)).
enum class Arrangement { Parallel, Sequential, ParallelTwo };
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
    GatedLinear    // gated linear attention, one decay per head and key channel
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
struct SoftmaxTraits { QkPost qk; bool bias = false, sink = false; };   // sink: a learned score per head, else one of zero
struct LayerSpec {
    Mixer kind = Mixer::Latent;
    LatentDims mix;                          // Latent
    AttnDims attn;                           // AttnTimeMix, Softmax
    Rotation rot;                            // Latent, Softmax
    SoftmaxTraits soft;                      // Softmax
    RecurDims rec;                           // Delta, ChannelDelta, AttnTimeMix, GatedLinear
    int decay_rank = 0, gate_rank = 0;       // inner sizes of the two-step projections, from the tensors' shapes
    double tau = 1.0;                        // GatedLinear: a decay is sigmoid(z)^(1 / tau)
    int ff = 0;                              // 0: no feed-forward
    RouterDims router;                       // experts > 0: a mixture of experts of size ff
    float limit = 0.f;
    int weights_of = -1;                     // layer whose tensors are used
    bool has_attn() const { return kind == Mixer::AttnTimeMix || kind == Mixer::Softmax; }
    bool has_latent() const { return kind == Mixer::Latent; }
    bool has_state() const { return kind != Mixer::Latent && kind != Mixer::Softmax; }
    bool has_rotation() const { return kind == Mixer::Latent || kind == Mixer::Softmax; }
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
