// Model registry and layer plans.
//
// The registry maps an architecture name (GGUF `general.architecture`, or `architecture` in a config.json) to the block
// the engine runs it with. Llama/Qwen and Phi-2 shaped decoders have one fixed block each (SpModelDesc says its sizes);
// every other design is a LAYER PLAN: a list of layers, each naming its mixer, its feed-forward, its norms and what
// happens to the residual stream between layers, with all sizes and constants as parameters. A plan-driven engine
// (engine_plan.cu) walks the list; a new design adds a plan reader here and, where it brings a new mechanism, a kernel
// beside the existing ones.
#pragma once
#include <stdint.h>

#include <memory>
#include <string>
#include <vector>

#include "json.h"

namespace sp {

enum ArchBlock : int { ARCH_LLAMA = 0, ARCH_PHI2 = 1, ARCH_PLAN = 2 };

// Rotary position embedding over `dims` coordinates, pairs (2 i, 2 i + 1), angle position * base^(-2 i / dims).
struct RotarySpec {
    double base = 10000.0;
    int dims = 0;
};

// Latent attention: per token only a normed latent of kv_rank values and one rotated key part of rot_dim values shared by
// all heads are cached; per-head keys and values are linear maps of the latent.
struct LatentAttentionSpec {
    int heads = 0, dim = 0, rot_dim = 0, vdim = 0, kv_rank = 0;
    int kv_from = -1;       // >= 0: reads the cache of that layer and has no down-projection of its own
    int window = 0x7FFFFFFF;  // keys j with 0 <= i - j < window are visible to query i
    float scale = 1.f;
    RotarySpec rot;
};

// Clamped gated expert: g = min(W_gate x, limit), u = clamp(W_up x, +-limit), y = W_down (g sigmoid(alpha g) (u + 1)).
struct ClampedExpertSpec {
    int ff = 0;
    float limit = 0.f;
    float alpha = 1.702f;
};

struct MoeSpec {
    int experts = 0, top = 0;
    ClampedExpertSpec expert;
    bool has_shared = false;  // a gated expert every token runs, times sigmoid of one projection
    ClampedExpertSpec shared;
};

struct LayerPlan {
    std::string prefix;  // tensor name prefix, with the dot
    LatentAttentionSpec mix;
    bool has_mlp = false;
    MoeSpec mlp;
};

struct ModelPlan {
    std::string name;
    int vocab = 0, width = 0;
    float eps = 1e-6f, embed_scale = 1.f;
    // Norms sit on a sublayer's output (x <- x + norm(f(x))) and have one gain for all coordinates.
    // depth_average: after each layer the stream becomes a learned combination of every layer result so far.
    bool depth_average = false;
    std::vector<LayerPlan> layers;
};

struct ArchEntry {
    const char* name;
    ArchBlock block;
    bool gguf;  // has a GGUF name map
    // Reads config.json into a plan (ARCH_PLAN entries): SP_OK or an error code with the message set.
    int (*read_plan)(const Json& cfg, ModelPlan* out);
};
// nullptr when the name is unknown.
const ArchEntry* find_arch(const std::string& name);

}  // namespace sp
