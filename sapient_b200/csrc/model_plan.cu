// Registry of architectures and the readers of their configuration files (model_plan.h).
#include "model_plan.h"

#include <climits>
#include <cmath>

#include "engine.h"

namespace sp {

namespace {

// Typed access to a configuration object; the first problem is remembered with the path it was found at.
struct Cfg {
    const Json* j;
    std::string at;
    std::string* err;
    Cfg sub(const char* key) const {
        const Json* s = j ? j->get(key) : nullptr;
        if (!s || s->type != Json::OBJ) fail(std::string(key) + " is missing or not an object");
        return Cfg{s, at + key + ".", err};
    }
    bool has(const char* key) const { return j && j->get(key); }
    void fail(const std::string& what) const {
        if (err->empty()) *err = "config: " + at + what;
    }
    double num(const char* key) const {
        const Json* s = j ? j->get(key) : nullptr;
        if (!s || s->type != Json::NUM || !std::isfinite(s->num)) { fail(std::string(key) + " is missing or not a number"); return 0; }
        return s->num;
    }
    int size(const char* key, int least = 1) const {
        const double v = num(key);
        if (err->empty() && (v != std::floor(v) || v < least || v > INT_MAX)) fail(std::string(key) + " is out of range");
        return err->empty() ? (int)v : least;
    }
};

GatedExpertSpec read_clamped_expert(const Cfg& c) {
    GatedExpertSpec e;
    e.ff = c.size("ff");
    e.limit = (float)c.num("limit");
    e.alpha = 1.702f;
    e.shift = 1.f;
    return e;
}

GatedExpertSpec read_silu_expert(const Cfg& c) {
    GatedExpertSpec e;
    e.ff = c.size("ff");
    return e;
}

LatentAttentionSpec read_latent_attention(const Cfg& c, int layer, const ModelPlan& p) {
    LatentAttentionSpec m;
    m.heads = c.size("heads");
    m.dim = c.size("dim");
    m.rot_dim = c.size("rot_dim");
    m.vdim = c.size("vdim");
    m.kv_rank = c.size("kv_rank");
    m.scale = (float)c.num("scale");
    const Cfg rot = c.sub("rot");
    m.rot.base = rot.num("base");
    m.rot.dims = rot.has("dims") ? rot.size("dims") : m.rot_dim;
    if (m.rot.dims != m.rot_dim || (m.rot_dim & 1) || m.rot.base <= 0) c.fail("rot does not fit rot_dim");
    if (c.has("mask") && c.sub("mask").has("size")) m.window = c.sub("mask").size("size");
    if (c.has("kv_from")) {
        m.kv_from = c.size("kv_from", 0);
        if (!c.err->empty()) return m;
        if (m.kv_from >= layer) { c.fail("kv_from must name an earlier layer"); return m; }
        const LatentAttentionSpec& o = p.layers[(size_t)m.kv_from].latent;
        if (o.kv_from >= 0 || o.kv_rank != m.kv_rank || o.rot_dim != m.rot_dim || o.rot.base != m.rot.base)
            c.fail("kv_from names a layer whose latent does not fit");
    }
    return m;
}

// What every kind of grouped attention has.
GroupedAttentionSpec read_heads(const Cfg& c) {
    GroupedAttentionSpec m;
    m.heads = c.size("heads");
    m.kv_heads = c.size("kv_heads");
    m.dim = c.size("dim");
    m.vdim = c.size("vdim");
    m.scale = (float)c.num("scale");
    if (c.err->empty() && m.heads % m.kv_heads) c.fail("heads is no multiple of kv_heads");
    return m;
}

TemperatureSpec read_temperature(const Cfg& c) {
    TemperatureSpec t;
    t.coef = c.num("coef");
    t.every = c.num("every");
    if (c.err->empty() && t.every <= 0) c.fail("every must be positive");
    return t;
}

// The entry "rot" of a mixer whose heads have `dim` coordinates.
RotarySpec read_rotary(const Cfg& c, int dim) {
    RotarySpec r;
    const Cfg rot = c.sub("rot");
    r.base = rot.num("base");
    r.dims = rot.has("dims") ? rot.size("dims", 0) : dim;
    if (c.err->empty() && ((r.dims & 1) || r.dims > dim || r.base <= 0)) c.fail("rot does not fit dim");
    if (rot.has("scaling")) {
        const Cfg s = rot.sub("scaling");
        r.factor = s.num("factor");
        r.original = s.num("original");
        r.fast = s.num("fast");
        r.slow = s.num("slow");
        if (c.err->empty() && (r.factor <= 0 || r.original <= 0 || r.fast <= 0 || r.slow <= 0 || r.base == 1.0)) s.fail("its numbers must be positive, and rot.base not one");
    }
    return r;
}

GroupedAttentionSpec read_rotated_attention(const Cfg& c, bool rotate_values) {
    GroupedAttentionSpec m = read_heads(c);
    m.rot = read_rotary(c, m.dim);
    m.rotate_values = rotate_values;
    if (c.has("mask") && c.sub("mask").has("size")) m.window = c.sub("mask").size("size");
    if (!c.err->empty()) return m;
    if (rotate_values && (m.vdim & 1)) c.fail("vdim must be even");
    return m;
}

// The sizes of a mixer with a state, and its decays where the rule has them.
StateMixerSpec read_state_mixer(const Cfg& c, StateRule rule) {
    StateMixerSpec m;
    m.rule = rule;
    m.heads = c.size("heads");
    m.dim = c.size("dim");
    m.vdim = rule == STATE_DELTA ? m.dim : c.size("vdim");
    if (rule == STATE_DECAY) {
        const Json* d = c.j ? c.j->get("decay") : nullptr;
        if (!d || d->type != Json::ARR || (c.err->empty() && (int)d->arr.size() != m.heads)) { c.fail("decay must list a number per head"); return m; }
        for (const Json& v : d->arr) {
            if (v.type != Json::NUM || !std::isfinite(v.num)) { c.fail("decay must list a number per head"); return m; }
            m.decay.push_back((float)v.num);
        }
    }
    if (c.err->empty() && m.dim > STATE_MAX_DIM) c.fail("dim is above " + std::to_string(STATE_MAX_DIM));
    return m;
}

// A layer's entry is null or has no "mlp": no feed-forward.
void read_dense(const Cfg& lc, LayerPlan* l) {
    if (!lc.has("mlp")) return;
    const Cfg c = lc.sub("mlp");
    const Json* kind = c.j ? c.j->get("kind") : nullptr;
    if (!kind || kind->str != "dense") { c.fail("kind is not a feed-forward of this design"); return; }
    l->mlp = MLP_DENSE;
    l->dense.ff = c.size("ff");
}

int read_tedelix(const Json& cfg, ModelPlan* out) {
    std::string err;
    const Cfg c{&cfg, "", &err};
    ModelPlan p;
    p.name = "Tedelix";
    p.vocab = c.size("vocab");
    p.width = c.size("width");
    p.eps = (float)c.sub("norm").num("eps");
    p.form = FORM_PARALLEL;
    p.norm_gain = GAIN_COORD;
    p.tied_head = true;
    if (c.has("logit_scale")) p.logit_scale = (float)c.num("logit_scale");
    if (c.has("logit_softcap")) p.logit_softcap = (float)c.num("logit_softcap");
    const Json* layers = cfg.get("layers");
    if (!layers || layers->type != Json::ARR || layers->arr.empty()) c.fail("layers is missing or not a list");
    for (size_t i = 0; err.empty() && i < layers->arr.size(); ++i) {
        const std::string idx = std::to_string(i);
        const Cfg lc{&layers->arr[i], "layers[" + idx + "].", &err};
        LayerPlan l;
        l.prefix = "l" + idx + ".";
        const Json* type = lc.j->get("type");
        const std::string t = type ? type->str : "";
        if (t == "attention") {
            l.mixer = MIX_GROUPED;
            l.grouped = read_rotated_attention(lc.sub("mixer"), true);
        } else if (t == "lightning" || t == "general_delta") {
            l.mixer = MIX_STATE;
            l.state = read_state_mixer(lc.sub("mixer"), t == "lightning" ? STATE_DECAY : STATE_DELTA);
            l.state.silu_inputs = l.state.norm_all = t == "lightning";
        } else {
            lc.fail("type is not a mixer of this design");
            break;
        }
        read_dense(lc, &l);
        p.layers.push_back(l);
    }
    if (!err.empty()) { set_error(err); return SP_ERR_ARG; }
    *out = std::move(p);
    return SP_OK;
}

int read_lepalorn(const Json& cfg, ModelPlan* out) {
    std::string err;
    const Cfg c{&cfg, "", &err};
    ModelPlan p;
    p.name = "Lepalorn";
    p.vocab = c.size("vocab");
    p.width = c.size("width");
    p.eps = (float)c.sub("norm").num("eps");
    p.embed_scale = (float)c.sub("embedding").num("scale");
    p.depth_average = true;
    const Json* layers = cfg.get("layers");
    if (!layers || layers->type != Json::ARR || layers->arr.empty()) c.fail("layers is missing or not a list");
    for (size_t i = 0; err.empty() && i < layers->arr.size(); ++i) {
        const std::string idx = std::to_string(i);
        const Cfg lc{&layers->arr[i], "layers[" + idx + "].", &err};
        LayerPlan l;
        l.prefix = "l" + idx + ".";
        const Json* type = lc.j->get("type");
        if (!type || type->str != "latent_attention") { lc.fail("type is not a mixer of this design"); break; }
        l.latent = read_latent_attention(lc.sub("mixer"), (int)i, p);
        if (lc.has("mlp")) {
            const Cfg m = lc.sub("mlp");
            const Json* kind = m.j ? m.j->get("kind") : nullptr;
            if (!kind || kind->str != "moe") { m.fail("kind is not a feed-forward of this design"); break; }
            l.mlp = MLP_MOE;
            l.moe.experts = m.sub("router").size("experts");
            l.moe.top = m.sub("router").size("top");
            l.moe.expert = read_clamped_expert(m.sub("expert"));
            if (m.has("shared")) {
                l.moe.has_shared = l.moe.shared_gate = true;
                l.moe.shared = read_clamped_expert(m.sub("shared"));
            }
            if (l.moe.top > l.moe.experts) m.fail("router.top exceeds router.experts");
        }
        p.layers.push_back(l);
    }
    if (!err.empty()) { set_error(err); return SP_ERR_ARG; }
    *out = std::move(p);
    return SP_OK;
}

// Fatilix's two kinds of attention: without rotation, queries with a temperature, a sink and an output gate; `shared`:
// weighted norms and values that are the keys, else biases, unweighted norms and a distance bias.
GroupedAttentionSpec read_sink_attention(const Cfg& c, bool shared) {
    GroupedAttentionSpec m = read_heads(c);
    m.sink = m.out_gate = true;
    if (c.has("q_temp")) m.temperature = read_temperature(c.sub("q_temp"));
    if (shared) {
        m.shared_values = true;
        m.qk_norm = QK_WEIGHTED;
        if (c.err->empty() && m.vdim != m.dim) c.fail("vdim must be dim where the keys are the values");
    } else {
        m.biases = true;
        m.qk_norm = QK_UNIT;
        m.bias_max = c.size("bias_max");
    }
    return m;
}

MoeSpec read_grouped_choice(const Cfg& c) {
    MoeSpec m;
    const Cfg r = c.sub("router");
    m.rule = ROUTE_ALL;
    m.bias = "correction";
    m.experts = r.size("experts");
    m.top = r.size("top");
    if (r.has("scale")) m.scale = (float)r.num("scale");
    if (r.has("groups")) {
        m.groups = r.sub("groups").size("count");
        m.keep = r.sub("groups").size("keep");
    }
    m.expert = read_silu_expert(c.sub("expert"));
    if (c.has("shared")) {
        m.has_shared = true;
        m.shared = read_silu_expert(c.sub("shared"));
    }
    if (!c.err->empty()) return m;
    if (m.experts % m.groups) r.fail("groups.count does not divide experts");
    else if (m.keep > m.groups) r.fail("groups.keep exceeds groups.count");
    else if (m.top > m.experts / m.groups * m.keep) r.fail("top exceeds the experts of the groups kept");
    return m;
}

int read_fatilix(const Json& cfg, ModelPlan* out) {
    std::string err;
    const Cfg c{&cfg, "", &err};
    ModelPlan p;
    p.name = "Fatilix";
    p.vocab = c.size("vocab");
    p.width = c.size("width");
    p.max_positions = c.size("max_positions");
    p.eps = (float)c.sub("norm").num("eps");
    p.norm_gain = GAIN_OFFSET;
    p.embed_scale = (float)c.sub("embedding").num("scale");
    p.residual_mult = (float)c.num("residual_mult");
    const Json* layers = cfg.get("layers");
    if (!layers || layers->type != Json::ARR || layers->arr.empty()) c.fail("layers is missing or not a list");
    for (size_t i = 0; err.empty() && i < layers->arr.size(); ++i) {
        const std::string idx = std::to_string(i);
        const Cfg lc{&layers->arr[i], "layers[" + idx + "].", &err};
        LayerPlan l;
        l.prefix = "l" + idx + ".";
        const Json* type = lc.j->get("type");
        const std::string t = type ? type->str : "";
        if (t != "attention" && t != "attention_2") { lc.fail("type is not a mixer of this design"); break; }
        l.mixer = MIX_GROUPED;
        l.grouped = read_sink_attention(lc.sub("mixer"), t == "attention");
        const Json* kind = lc.has("mlp") ? lc.sub("mlp").j->get("kind") : nullptr;
        if (kind && kind->str == "moe") {
            l.mlp = MLP_MOE;
            l.moe = read_grouped_choice(lc.sub("mlp"));
        } else {
            read_dense(lc, &l);
        }
        p.layers.push_back(l);
    }
    if (!err.empty()) { set_error(err); return SP_ERR_ARG; }
    *out = std::move(p);
    return SP_OK;
}

// Decaying sum over rotated queries and scaled, rotated keys.
StateMixerSpec read_retention(const Cfg& c) {
    StateMixerSpec m = read_state_mixer(c, STATE_DECAY);
    m.rot = read_rotary(c, m.dim);
    m.key_scale = 1.f / std::sqrt((float)m.dim);
    m.gain = STATE_GAIN_NONE;
    m.gate = STATE_GATE_SILU;
    return m;
}

// Attention over convolved, biased projections whose heads' weights are mixed.
GroupedAttentionSpec read_talking_attention(const Cfg& c) {
    GroupedAttentionSpec m = read_heads(c);
    m.rot = read_rotary(c, m.dim);
    m.rot.neighbours = true;
    m.biases = m.sink = m.talk = true;
    if (c.has("conv")) m.conv = c.size("conv");
    if (c.has("softcap")) m.score_softcap = (float)c.num("softcap");
    if (c.has("mask")) {
        const Cfg mask = c.sub("mask");
        if (mask.has("size")) m.window = mask.size("size");
        if (mask.has("keep_first")) m.keep_first = mask.size("keep_first", 0);
    }
    if (c.err->empty() && m.conv > CONV_MAX_TAPS) c.fail("conv is above " + std::to_string(CONV_MAX_TAPS));
    if (c.err->empty() && c.has("softcap") && m.score_softcap <= 0) c.fail("softcap must be positive");
    return m;
}

int read_revelix(const Json& cfg, ModelPlan* out) {
    std::string err;
    const Cfg c{&cfg, "", &err};
    ModelPlan p;
    p.name = "Revelix";
    p.vocab = c.size("vocab");
    p.width = c.size("width");
    p.eps = (float)c.sub("norm").num("eps");
    p.form = FORM_PRE_NORM;
    p.norm = NORM_TANH;
    p.tied_head = true;
    if (c.has("logit_scale")) p.logit_scale = (float)c.num("logit_scale");
    const Json* layers = cfg.get("layers");
    if (!layers || layers->type != Json::ARR || layers->arr.empty()) c.fail("layers is missing or not a list");
    for (size_t i = 0; err.empty() && i < layers->arr.size(); ++i) {
        const std::string idx = std::to_string(i);
        const Cfg lc{&layers->arr[i], "layers[" + idx + "].", &err};
        LayerPlan l;
        l.prefix = "l" + idx + ".";
        const Json* type = lc.j->get("type");
        const std::string t = type ? type->str : "";
        if (t == "retention") {
            l.mixer = MIX_STATE;
            l.state = read_retention(lc.sub("mixer"));
        } else if (t == "parallel") {
            const Cfg m = lc.sub("mixer");
            l.mixer = MIX_BOTH;
            l.grouped = read_talking_attention(m.sub("left"));
            l.grouped.at = "mix.left.";
            if (m.has("left_scale")) l.grouped.out_scale = (float)m.num("left_scale");
            l.state = read_state_mixer(m.sub("right"), STATE_FORGET);
            l.state.gain = STATE_GAIN_HEAD;
            l.state.gate = STATE_GATE_NONE;
            l.state.at = "mix.right.";
            if (m.has("right_scale")) l.state.out_scale = (float)m.num("right_scale");
        } else {
            lc.fail("type is not a mixer of this design");
            break;
        }
        read_dense(lc, &l);
        l.dense.act = DENSE_XIELU;
        p.layers.push_back(l);
    }
    if (!err.empty()) { set_error(err); return SP_ERR_ARG; }
    *out = std::move(p);
    return SP_OK;
}

// GGUF names: crates/sapient-models/src/forward/mod.rs:223-316 (family dispatch of the reference's loader).
const ArchEntry ARCHS[] = {
    {"llama", ARCH_LLAMA, true, nullptr},   {"mistral", ARCH_LLAMA, true, nullptr}, {"qwen2", ARCH_LLAMA, true, nullptr},
    {"qwen3", ARCH_LLAMA, true, nullptr},   {"idefics3", ARCH_LLAMA, true, nullptr}, {"phi3", ARCH_LLAMA, true, nullptr},
    {"phi", ARCH_PHI2, true, nullptr},      {"phi2", ARCH_PHI2, true, nullptr},     {"Lepalorn", ARCH_PLAN, false, read_lepalorn},
    {"Tedelix", ARCH_PLAN, false, read_tedelix}, {"Fatilix", ARCH_PLAN, false, read_fatilix},
    {"Revelix", ARCH_PLAN, false, read_revelix},
};

}  // namespace

const ArchEntry* find_arch(const std::string& name) {
    for (const ArchEntry& a : ARCHS)
        if (name == a.name) return &a;
    return nullptr;
}

}  // namespace sp
