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

#include <limits>
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

// Norm of each head's queries and keys by their root mean square.
//   QK_UNIT  without a weight     QK_WEIGHTED  a weight per coordinate, shared by the heads
enum QkNorm : int { QK_NONE = 0, QK_UNIT = 1, QK_WEIGHTED = 2 };

// Queries times 1 + coef * ln(floor((position + 1) / every) + 1).
struct TemperatureSpec {
    double coef = 0.0, every = 1.0;
};

// Grouped-query attention: `heads` query heads share kv_heads cached keys (dim) and values (vdim). Queries and keys go through
// the projection's bias, the norm, the temperature (queries) and the rotation of their first rot.dims coordinates, in this
// order; with rotate_values all of a value's coordinates are rotated by its position before they are cached and every head's
// mixture is turned back by the query's. A distance bias adds table[bucket(i - j)][head] to the scaled score: a bucket per
// distance up to half of the table's rows, then logarithmic ones up to bias_max. A sink is one more term exp(sink[head]) in
// the softmax's denominator. An output gate multiplies the mixtures, coordinate by coordinate, by sigmoid(W_g h).
struct GroupedAttentionSpec {
    int heads = 0, kv_heads = 0, dim = 0, vdim = 0;
    int window = 0x7FFFFFFF;  // as above
    float scale = 1.f;
    RotarySpec rot;
    bool rotate_values = false;
    bool shared_values = false;  // values are the keys as projected (no value projection; not with rotation)
    bool biases = false;         // of the q, k and v projections
    QkNorm qk_norm = QK_NONE;
    TemperatureSpec temperature;
    int bias_max = 0;            // 0: no distance bias
    bool sink = false, out_gate = false;
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

// Gated expert: g = min(W_gate x, limit), u = clamp(W_up x, +-limit), y = W_down (g sigmoid(alpha g) (u + shift)). As it
// stands here, y = W_down (silu(W_gate x) * W_up x).
struct GatedExpertSpec {
    int ff = 0;
    float limit = std::numeric_limits<float>::infinity();
    float alpha = 1.f, shift = 0.f;
};

// How the experts of a token are chosen and weighed, z being the router's logits.
//   ROUTE_CHOSEN  the `top` largest of z + bias; weights: the softmax over the chosen ones.
//   ROUTE_ALL     s = softmax(z) over all experts; the `top` largest of s + bias among the experts of the `keep` best of
//                 `groups` equal runs of experts (a group counts by its best expert); weights: s / (sum of the chosen s) * scale.
enum RouteRule : int { ROUTE_CHOSEN = 0, ROUTE_ALL = 1 };

struct MoeSpec {
    int experts = 0, top = 0;
    RouteRule rule = ROUTE_CHOSEN;
    int groups = 1, keep = 1;
    float scale = 1.f;
    const char* bias = "router.b";  // tensor name
    GatedExpertSpec expert;
    bool has_shared = false;   // an expert every token runs ...
    bool shared_gate = false;  // ... times sigmoid of one projection
    GatedExpertSpec shared;
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
//   FORM_POST_NORM  x <- x + m norm(mixer(x)), then x <- x + m norm(ff(x)), m = residual_mult.
//   FORM_PARALLEL   x <- x + mixer(h) + ff(h) with h = norm(x). Both sublayers are one product in and one product out.
enum LayerForm : int { FORM_POST_NORM = 0, FORM_PARALLEL = 1 };

// The gain of the stream's norms: one number, one per coordinate, or one per coordinate stored as its distance from one.
enum NormGain : int { GAIN_SCALAR = 0, GAIN_COORD = 1, GAIN_OFFSET = 2 };

struct ModelPlan {
    std::string name;
    int vocab = 0, width = 0;
    float eps = 1e-6f, embed_scale = 1.f;
    int max_positions = 0;       // rows of a table of learned position vectors, added to the embedding (0: none)
    float residual_mult = 1.f;
    LayerForm form = FORM_POST_NORM;
    NormGain norm_gain = GAIN_SCALAR;
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
