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
// (2 i, 2 i + 1) in latent attention and where `neighbours` is set, else halves (i, i + dims / 2). With factor > 0 frequencies are
// stretched for contexts beyond `original`: pairs that turn more than `fast` times within it keep theirs, pairs that turn less than
// `slow` times have it divided by factor, with a linear ramp over the pairs between; sines and cosines grow by 0.1 ln(factor) + 1.
struct RotarySpec {
    double base = 10000.0;
    int dims = 0;
    bool neighbours = false;
    double factor = 0.0, original = 0.0, fast = 0.0, slow = 0.0;
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
// A short convolution over time (conv taps per channel, the last one on the token itself) comes between bias and norm; the
// taps - 1 values before a token are state of its sequence. keep_first: the sequence's first keys stay visible behind the window.
// score_softcap: s <- cap tanh(s / cap) on the scaled score. talk: the heads' softmax weights are mixed, w_h <- sum_g T[h][g] w_g
// (without the sink's share), before they meet the values of h's cached head. Outputs are multiplied by out_scale.
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
    int conv = 0;                // 0: no convolution
    int keep_first = 0;
    float score_softcap = 0.f;   // 0: no cap
    bool talk = false;
    float out_scale = 1.f;
    std::string at = "mix.";     // tensor names behind the layer's prefix
};
constexpr int CONV_MAX_TAPS = 32;

// A mixer whose memory is one matrix S [dim][vdim] per head and sequence, in f32, zero at the start; o = S^T q.
//   STATE_DECAY   S <- decay_h S + k v^T.
//   STATE_DELTA   S <- diag(w) S - (a u)(u^T S) + k v^T with the unit key u = k / |k|, w = exp(-e^(-1/2) sigmoid(low-rank
//                 logit)) and a = sigmoid(projection) per head and key channel.
//   STATE_FORGET  S <- diag(f) S + (1 - f) v^T, f = l + (1 - l) sigmoid(projection + bias) per head and key channel, between the
//                 learned bound l and one. q through silu.
// The decaying sum may take q, k and v through silu, or rotate q and k by position, and scales its keys. Outputs are divided by
// their root mean square, head by head or all heads of a token together, then take a gain and a gate by a projection of h.
constexpr int STATE_MAX_DIM = 512;  // key channels the kernels cover
enum StateRule : int { STATE_DECAY = 0, STATE_DELTA = 1, STATE_FORGET = 2 };
enum StateGate : int { STATE_GATE_NONE = 0, STATE_GATE_SIGMOID = 1, STATE_GATE_SILU = 2 };
// The gain after the norm: none, one number per coordinate, or per coordinate of a head and the same for all heads.
enum StateGain : int { STATE_GAIN_NONE = 0, STATE_GAIN_COORD = 1, STATE_GAIN_HEAD = 2 };
struct StateMixerSpec {
    StateRule rule = STATE_DECAY;
    int heads = 0, dim = 0, vdim = 0;
    std::vector<float> decay;   // STATE_DECAY: per head
    bool silu_inputs = false;   // STATE_DECAY
    RotarySpec rot;             // STATE_DECAY
    float key_scale = 1.f;      // STATE_DECAY
    bool norm_all = false;      // STATE_DECAY
    StateGain gain = STATE_GAIN_COORD;
    StateGate gate = STATE_GATE_SIGMOID;
    float out_scale = 1.f;
    std::string at = "mix.";    // tensor names behind the layer's prefix
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

// MIX_BOTH: grouped attention and a state mixer side by side; both read the same input, their outputs are added.
enum MixerKind : int { MIX_LATENT = 0, MIX_GROUPED = 1, MIX_STATE = 2, MIX_BOTH = 3 };
enum MlpKind : int { MLP_NONE = 0, MLP_MOE = 1, MLP_DENSE = 2 };

// W_down act(W_up h).
//   DENSE_RELU2  the square of relu
//   DENSE_XIELU  z / 2 + softplus(p) z^2 right of zero, z / 2 + (1/2 + softplus(q)) (e^z - 1 - z) left of it, with learned p, q
enum DenseAct : int { DENSE_RELU2 = 0, DENSE_XIELU = 1 };
struct DenseSpec {
    int ff = 0;
    DenseAct act = DENSE_RELU2;
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
    bool has_grouped() const { return mixer == MIX_GROUPED || mixer == MIX_BOTH; }
    bool has_state() const { return mixer == MIX_STATE || mixer == MIX_BOTH; }
};

// What happens to the residual stream x in a layer.
//   FORM_POST_NORM  x <- x + m norm(mixer(x)), then x <- x + m norm(ff(x)), m = residual_mult.
//   FORM_PARALLEL   x <- x + mixer(h) + ff(h) with h = norm(x). Both sublayers are one product in and one product out.
//   FORM_PRE_NORM   x <- x + mixer(norm(x)), then x <- x + ff(norm(x)).
enum LayerForm : int { FORM_POST_NORM = 0, FORM_PARALLEL = 1, FORM_PRE_NORM = 2 };

// The stream's norm: by the root mean square, or tanh(alpha x) w + b with a learned number alpha and vectors w, b.
enum NormKind : int { NORM_RMS = 0, NORM_TANH = 1 };

// The gain of the stream's norms: one number, one per coordinate, or one per coordinate stored as its distance from one.
enum NormGain : int { GAIN_SCALAR = 0, GAIN_COORD = 1, GAIN_OFFSET = 2 };

struct ModelPlan {
    std::string name;
    int vocab = 0, width = 0;
    float eps = 1e-6f, embed_scale = 1.f;
    int max_positions = 0;       // rows of a table of learned position vectors, added to the embedding (0: none)
    float residual_mult = 1.f;
    LayerForm form = FORM_POST_NORM;
    NormKind norm = NORM_RMS;
    NormGain norm_gain = GAIN_SCALAR;
    bool depth_average = false;  // after each layer the stream becomes a learned combination of every layer result so far
    bool tied_head = false;      // logits from the embedding table
    float logit_scale = 1.f, logit_softcap = 0.f;  // z <- z * scale, then cap * tanh(z / cap) (0: no cap)
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
