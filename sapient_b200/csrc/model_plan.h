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

// Rotary position embedding over `dims` coordinates, angle position * base^(-2 i / dims) for pair i. Pairs are neighbours
// (2 i, 2 i + 1) in latent attention and halves (i, i + dims / 2) in grouped attention.
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

// Grouped-query attention: `heads` query heads share kv_heads cached keys (dim) and values (vdim). The first rot.dims
// coordinates of queries and keys are rotated; with rotate_values all of a value's coordinates are rotated by its position
// before they are cached and every head's mixture is turned back by the query's.
struct GroupedAttentionSpec {
    int heads = 0, kv_heads = 0, dim = 0, vdim = 0;
    int window = 0x7FFFFFFF;  // as above
    float scale = 1.f;
    RotarySpec rot;
    bool rotate_values = false;
};

// A mixer whose memory is one matrix S [dim][vdim] per head and sequence, in f32, zero at the start; o = S^T q.
//   STATE_DECAY  S <- decay_h S + k v^T; q, k, v through silu; the heads' outputs are normed together.
//   STATE_DELTA  S <- diag(w) S - (a u)(u^T S) + k v^T with the unit key u = k / |k|, w = exp(-e^(-1/2) sigmoid(low-rank
//                logit)) and a = sigmoid(projection) per head and key channel; each head's output is normed by itself.
// Both then take a gain per coordinate and a sigmoid gate.
constexpr int STATE_MAX_DIM = 512;  // key channels the kernels cover
enum StateRule : int { STATE_DECAY = 0, STATE_DELTA = 1 };
struct StateMixerSpec {
    StateRule rule = STATE_DECAY;
    int heads = 0, dim = 0, vdim = 0;
    std::vector<float> decay;  // STATE_DECAY: per head
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

enum MixerKind : int { MIX_LATENT = 0, MIX_GROUPED = 1, MIX_STATE = 2 };
enum MlpKind : int { MLP_NONE = 0, MLP_MOE = 1, MLP_DENSE = 2 };

// W_down act(W_up h), act = the square of relu.
struct DenseSpec {
    int ff = 0;
};

struct LayerPlan {
    std::string prefix;  // tensor name prefix, with the dot
    MixerKind mixer = MIX_LATENT;
    LatentAttentionSpec latent;
    GroupedAttentionSpec grouped;
    StateMixerSpec state;
    MlpKind mlp = MLP_NONE;
    MoeSpec moe;
    DenseSpec dense;
};

// What happens to the residual stream x in a layer.
//   FORM_POST_NORM  x <- x + norm(mixer(x)), then x <- x + norm(ff(x)); norms have one gain for all coordinates.
//   FORM_PARALLEL   x <- x + mixer(h) + ff(h) with h = norm(x); norms have a gain per coordinate. Both sublayers are one
//                   product in and one product out.
enum LayerForm : int { FORM_POST_NORM = 0, FORM_PARALLEL = 1 };

struct ModelPlan {
    std::string name;
    int vocab = 0, width = 0;
    float eps = 1e-6f, embed_scale = 1.f;
    LayerForm form = FORM_POST_NORM;
    bool depth_average = false;  // after each layer the stream becomes a learned combination of every layer result so far
    bool tied_head = false;      // logits from the embedding table
    float logit_scale = 1.f, logit_softcap = 0.f;  // z <- z * scale, then cap * tanh(z / cap) (0: no cap)
    std::vector<LayerPlan> layers;
    bool recurrent() const {     // some layer keeps a state that cannot be rolled back
        for (const LayerPlan& l : layers)
            if (l.mixer == MIX_STATE) return true;
        return false;
    }
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
