// Layer-list models: what a configuration describes (stack_config.cu) and what the loader makes of it (stack_model.cu).
#pragma once

#include <map>
#include <string>
#include <vector>

#include "attn_prompt.cuh"
#include "checkpoint.cuh"
#include "recurrent.cuh"

namespace forge {

enum class Norm { DynamicTanh };
// Parallel: x += mixer(h) + ff(h) behind one norm.  Sequential: x += mixer(norm1(x)), then x += ff(norm2(x)).
enum class Arrangement { Parallel, Sequential };
enum class Mlp { ClampedGlu, SiluGlu };
struct Architecture { const char* name; Norm norm; Arrangement arrangement; Mlp dense; };

enum class Mixer {
    Latent,        // latent attention
    Delta,         // gated delta rule, one decay per head
    ChannelDelta,  // gated delta rule, one decay per head and key channel
    AttnTimeMix    // gated attention and time mixing side by side, half the sum of their normed outputs
};
struct LayerSpec {
    Mixer kind = Mixer::Latent;
    LatentDims mix; double rot_base = 1.0;   // Latent
    AttnDims attn;                           // AttnTimeMix
    RecurDims rec;                           // Delta, ChannelDelta, AttnTimeMix
    int decay_rank = 0, gate_rank = 0;       // inner sizes of the two-step projections, from the tensors' shapes
    int ff = 0;                              // 0: no feed-forward
    float limit = 0.f;
    int weights_of = -1;                     // layer whose tensors are used
    bool has_attn() const { return kind == Mixer::AttnTimeMix; }
    bool has_latent() const { return kind == Mixer::Latent; }
    bool has_state() const { return kind != Mixer::Latent; }
    int cache_row() const { return has_latent() ? mix.row() : has_attn() ? attn.row() : 0; }   // values per position, padding included
};
struct LayerRun { int layer, pass; };   // pass >= 0: this pass of the loop starts in front of the layer
struct StackSpec {
    const Architecture* arch = nullptr;
    int width = 0, vocab = 0;
    float eps = 0.f;
    std::vector<LayerSpec> layers;
    int loop_start = 0, loop_stop = 0, loop_times = 0;   // times = 0: no loop
    std::vector<LayerRun> runs;
    int64_t parameters = 0;
};

typedef std::map<std::string, const TensorView*> TensorSet;   // by name, a layer's without its prefix
struct StackTensors { TensorSet top; std::vector<TensorSet> layers; };

// Reads and checks config.json; then every tensor it calls for, with its shape (also fills in the sizes that only shapes give).
int32_t stack_parse(const Json& config, StackSpec* s);
int32_t stack_find_tensors(const Checkpoint& ck, StackSpec* s, StackTensors* t);
void stack_fill_info(const StackSpec& s, ForgeCheckpointInfo* out);

}  // namespace forge
