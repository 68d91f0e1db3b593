// State of a plan-driven engine: the packed weights of every layer, the cache and state pools and the buffers of a step.
// Owned by Engine, which keeps the sequence slots, the page tables, the step graphs and the host API. engine_plan.cu has
// what every plan shares, engine_plan_post_norm.cu (with experts), engine_plan_parallel.cu and engine_plan_pre_norm.cu the layer
// forms, engine_plan_latent.cu latent attention, engine_plan_grouped.cu grouped attention, engine_plan_state.cu state mixers.
#pragma once
#include <algorithm>
#include <map>
#include <string>
#include <utility>
#include <vector>

#include "engine.h"

#include "model_plan.h"
#include "plan_kernels.h"

namespace sp {

// Matrices in the compute type, rows padded to kp columns.
struct PlanMat {
    void* w = nullptr;
    int n = 0, kp = 0, groups = 1;
};

constexpr int PLAN_ROWS = MAT_GATHER_ROWS;  // rows of a decode-shaped step
static_assert(PLAN_ROWS <= STATE_STEP_ROWS, "a decode-shaped step runs the state mixers' step kernel");

#define SP_TRY(expr)                  \
    do {                              \
        int _s = (expr);              \
        if (_s != SP_OK) return _s;   \
    } while (0)

#define SP_LAUNCH(fam, expr)              \
    do {                                  \
        if (fam_mask & (1u << (fam))) {   \
            prof_begin(fam);              \
            SP_CUDA_TRY(expr);            \
            prof_end(fam);                \
        }                                 \
    } while (0)

struct PlanLayer {
    PlanMat proj;              // everything that reads the mixer's input. Latent: q | latent and rotated key part (own cache only) |
                               // output gate. Parallel form: the mixer's f32 rows | low-rank rows | feed-forward up
    int gate_col = 0;          // first gate column of the projection's output
    PlanMat uk_t;              // per head, transposed: query -> latent space
    PlanMat uv;                // per head: latent -> value
    PlanMat kv;                // per head key rows then value rows, each padded to 16: the expanded form
    PlanMat o;                 // output projection; parallel form: [W_o | W_down] over [mixer output | activation]
    RowGain norm1{}, norm2{};
    const float *dkv_norm = nullptr, *dwa = nullptr;
    PlanMat router;            // experts rows, then the shared expert's gate row where it has one
    const float* router_b = nullptr;
    PlanMat gu, down, shared_gu, shared_down;
    PlanMat up;                // dense feed-forward of the post-norm form (down as above)
    LatentShape shape{};
    LatentCache cache{};       // the layer's own, or the one it borrows
    bool own = true, expand = false;
    const float2* cos_sin = nullptr;
    GroupedShape grouped{};
    GroupedCache kv_cache{};
    GroupedInput grouped_in{};
    GroupedTerms grouped_terms{};  // without the step's gate
    int grouped_col = 0;       // of the projection's output: first column of grouped attention
    bool mixed = false;        // grouped attention whose heads are mixed (or whose scores have a cap, or its window kept keys)
    MixedTerms mixed_terms{};
    int mixed_rows = 0, mixed_span = 0;  // shape of the score scratch
    size_t tail_at = 0;        // convolution: of a slot's floats
    int mix_rows = 0;          // of proj: f32 rows (grouped attention, state mixers)
    // state mixers
    int silu_rows = 0, low_rows = 0;  // of the mix_rows those that come first; rows of proj behind them
    int state_col = 0;         // first column of the state mixer's output in o's input
    StateShape state_shape{};
    size_t state_at = 0;       // of a slot's floats
    PlanMat w2;
    const float *decay = nullptr, *a_bias = nullptr, *w0 = nullptr, *gain = nullptr, *lower = nullptr;
    // parallel form
    int ff = 0;                // rows of proj behind the low-rank ones
    int act_col = 0;           // first column of the activation in o's input
    // pre-norm form
    TanhNorm tanh1{}, tanh2{};
    float act_arg[2] = {};     // of the feed-forward's activation
};

// Elements per row that the step's buffers need: the largest of all layers.
struct PlanSizes {
    size_t proj = 0, qn = 0, qabs = 0, qf = 0, olat = 0, mixed = 0, act = 0, act_shared = 0, pairs = 0, kv = 0, lat = 0, part = 0, low = 0,
           wlogit = 0, state_rec = 0, q = 0, stat = 0, score = 0;
    int experts = 0;
    static void most(size_t& a, size_t b) { a = std::max(a, b); }
};

struct PlanState {
    ModelPlan plan;
    bool f32 = false;
    int elem() const { return f32 ? 4 : 2; }
    std::vector<PlanLayer> layers;
    PlanMat embed, head, pos;  // pos: learned position vectors
    RowGain final_norm{};
    TanhNorm final_tanh{};
    int wp = 0;                // padded width
    size_t page_bytes = 0;     // all layers' rows of one page
    std::vector<size_t> cache_run, cache_base;  // per layer: bytes of a page (0: none of its own), offset of its slice
    size_t cache_bytes = 0;
    void* cache = nullptr;
    // buffers of a step
    PlanSizes need;
    bool has_latent = false, has_grouped = false, has_state = false, has_mixed = false, has_conv = false;
    void *xb = nullptr, *qn = nullptr, *qabs = nullptr, *qf = nullptr, *olat = nullptr, *attn = nullptr, *act = nullptr, *act_shared = nullptr,
         *xs = nullptr, *kvx = nullptr, *lat = nullptr, *fin = nullptr, *q = nullptr, *low = nullptr;
    float *proj = nullptr, *y = nullptr, *y_expert = nullptr, *y_shared = nullptr, *logit = nullptr, *weight = nullptr, *part = nullptr, *history = nullptr, *wlogit = nullptr, *state_rec = nullptr,
          *score = nullptr;
    float2 *stat = nullptr, *score_part = nullptr;
    int32_t *pick = nullptr, *tables = nullptr, *host_tiles = nullptr, *dev_tiles = nullptr;
    // sections of host_tiles / dev_tiles, in ints
    size_t keys_at = 0, grouped_at = 0, narrow_at = 0, back_at = 0, ends_at = 0, seg_at = 0, groups_at = 0, table_ints = 0;
    MoeTables moe{};
    int keys_cap = 0;          // gathered keys a step may hold
    // the current step, when it is longer than PLAN_ROWS
    int n_tiles = 0, n_keys = 0;        // latent attention: tiles and gathered keys of the expanded form (0 tiles: absorbed)
    int n_grouped = 0, n_narrow = 0;    // grouped attention: tiles, and narrow ones of mixed heads
    int n_ends = 0;                     // convolutions: slots with rows in the step
    int n_seg = 0, n_groups = 0;        // state mixers: segments and groups of tokens
    // per slot and layer: states [heads][vdim][dim_pad], tails of convolutions [taps - 1][channels]; and what checkpoint() keeps of each slot
    float *states = nullptr, *checkpoints = nullptr;
    size_t slot_state = 0;              // floats per slot
    std::vector<int> checkpoint_len;    // per slot: tokens the kept state has seen, -1: none
    size_t groups_cap = 0;              // groups a step may have
    std::map<std::vector<double>, const float2*> angles;
    std::vector<void*> owned;
};

size_t plan_latent_part_rows();  // engine_plan_latent.cu

// A matrix that reads the mixer's input: tensor name behind the layer's prefix and rows.
struct MixPart {
    std::string name;
    int rows;
};

// Builds packed matrices out of the uploaded tensors.
struct PlanPacker {
    Engine& e;
    PlanState& p;
    int status = SP_OK;

    bool fail(int st, const std::string& msg);
    const DevTensor* need(const std::string& name, int64_t rows, int64_t cols);
    int64_t rows_of(const std::string& name);            // first dimension of a tensor whose size only its shape tells
    const float* vec(const std::string& name, int64_t n);
    RowGain gain(const std::string& name);               // of a norm of the stream (model_plan.h: NormGain)
    TanhNorm tanh_norm(const std::string& name);
    std::vector<float> host(const std::string& name, int64_t rows, int64_t cols);
    const float* upload(const std::vector<float>& v);
    bool alloc(PlanMat& m, int groups, int64_t rows, int k);
    // rows [r0, r0 + rows) of source tensor t to packed rows starting at `to` (counted over all groups), columns at c0
    bool put(PlanMat& m, int64_t to, const DevTensor* t, int64_t r0, int64_t rows, int k, bool transpose = false, int c0 = 0);
    // cos and sin by position and pair (model_plan.h: RotarySpec), for every position: computed in double, rounded once
    const float2* angles(const RotarySpec& r);
    const float2* angles(double base, int dims) {
        RotarySpec r;
        r.base = base;
        r.dims = dims;
        return angles(r);
    }
    void cache_slice(size_t page_bytes);                 // the next layer's share of the cache
    void latent_layer(int i);
    // Appends to parts the matrices that read the mixer's input, in the order of their output columns; returns what W_o reads.
    int grouped_mixer(int i, std::vector<MixPart>& parts);
    int state_mixer(int i, std::vector<MixPart>& parts);
    size_t slot_floats(size_t n);                        // the next n floats of a slot's states: where they begin
    // The layer's mixers, without a projection of their own yet; then their rows at the head of l.proj.
    int mixers(int i, std::vector<MixPart>& parts);
    void put_mixer_rows(int i, const std::vector<MixPart>& parts);
    void put_mixer_out(int i);                           // W_o (both: side by side) into l.o
    const float* distance_bias(const std::string& name, int heads, int far, int* n_rel);
    void experts(int i);
    void post_norm_layer(int i);
    void parallel_layer(int i);
    void pre_norm_layer(int i);
};

}  // namespace sp
