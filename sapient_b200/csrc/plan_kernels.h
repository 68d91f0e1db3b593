// Launch wrappers of the kernels that plan-driven engines (engine_plan.cu) add to kernels.h: matrix products on
// unquantised weights (dense, per head, per expert), latent attention over a paged latent cache, expert routing, and the
// residual / norm / depth-average steps between them.
//
// "Compute type": bf16 (weights, matrix operands, cache; f32 accumulation) or f32 (everything). Pointers of that type are
// void*, with `f32` telling which. Rows of a weight matrix are padded to a multiple of MAT_KPAD columns with zeros;
// activation rows have the same padded stride (whatever finite values the padding holds).
#pragma once
#include <cuda_runtime.h>
#include <stdint.h>

namespace sp {

constexpr int MAT_KPAD = 64;
inline int mat_kpad(int k) { return (k + MAT_KPAD - 1) / MAT_KPAD * MAT_KPAD; }

// A gated unit: g = min(., limit), u = clamp(., +-limit), y = g sigmoid(alpha g) (u + shift).
struct MatUnit {
    float limit, alpha, shift;
};

// A family of equally shaped matrices [groups][rows][kp]. `dual`: rows = 2 n, the first n are the gate and the last n the
// up-projection of a gated unit, whose n activations are the output.
struct MatSeg {
    const void* w;
    int n, kp, groups;
    MatUnit unit;              // dual
    const void* x;             // compute type
    int ldx;
    int64_t xgs;               // elements between the inputs of consecutive groups (per-head products)
    void* y;
    int ldy;
    int64_t ygs;
};

// Where a range of a matrix's rows goes: output elements [previous n_end, n_end) of every activation row to y (column 0 is
// the range's first), through an activation, as f32 or in the compute type; `add`: y (f32) += instead of =.
//   MAT_SOFTCAP  arg[1] * tanh(arg[0] * z / arg[1])
//   MAT_XIELU    z / 2 + arg[0] z^2 right of zero, z / 2 + arg[1] (e^z - 1 - z) left of it
enum MatAct : int { MAT_ID = 0, MAT_RELU2, MAT_TANH, MAT_SILU, MAT_SOFTCAP, MAT_XIELU };
struct MatOut {
    int n_end;
    void* y;
    int64_t ldy;
    MatAct act;
    bool f32, add;
};
constexpr int MAT_MAX_OUTS = 4;

// A norm without statistics: tanh(alpha x) w[c] + b[c] (null w: none).
struct TanhNorm {
    float alpha;
    const float *w, *b;
};
// What a product that adds into the stream leaves beside it: the norm of the sums in the compute type.
struct MatNorm {
    TanhNorm fn;
    void* y;
    int64_t ldy;
};

// Rows of a step sorted by expert, made on the device by launch_moe_route.
struct MoeRows {
    const int32_t* row_off;    // [experts + 1] first sorted row of each expert
    const int32_t* row_src;    // token of each sorted row
    const int32_t* active;     // experts with at least one row, ascending
    const int32_t* n_active;
    const int32_t* tile_group; // row tiles of MOE_TILE rows: which expert
    const int32_t* tile_row;   // ... and which sorted row they start at
    const int32_t* n_tiles;
};
constexpr int MOE_TILE = 128;

struct MatArgs {
    MatSeg seg[2];             // seg[0] grouped by expert when rows != null, else one product per group over all m rows;
    int nseg;                  // seg[1]: over all m rows
    int m;
    bool dual, f32, out_f32;   // out_f32: y is f32 whatever the compute type
    bool moe;                  // seg[0] is grouped by rows.*
    bool gather;               // its x rows are tokens (row_src), not sorted rows
    MoeRows rows;
    int slots;                 // moe: upper bound of active experts
    int x_rows;                // rows of seg[0].x when they are not the m rows (sorted rows)
    const float* gate;         // y *= sigmoid(gate[row * ldgate + group]) or null
    int ldgate;
    int n_outs;                // > 0: one plain product whose rows go where outs[] says (seg[0].y is not used)
    MatOut outs[MAT_MAX_OUTS];
    float arg[2];              // of the activation
    MatNorm norm;              // null w: none; else one range that adds
};

// The ranges cover the matrix, and the product is a plain one.
inline bool mat_outs_valid(const MatArgs& a) {
    if (a.n_outs == 0) return true;
    if (a.n_outs < 0 || a.n_outs > MAT_MAX_OUTS || a.nseg != 1 || a.seg[0].groups != 1 || a.moe || a.dual || a.gate) return false;
    int n = 0;
    for (int i = 0; i < a.n_outs; ++i) {
        if (a.outs[i].n_end <= n || !a.outs[i].y || (a.outs[i].add && !a.outs[i].f32 && !a.f32)) return false;
        n = a.outs[i].n_end;
    }
    return n == a.seg[0].n && (!a.norm.fn.w || (a.n_outs == 1 && a.outs[0].add && a.outs[0].act == MAT_ID));
}

// f32: plain fused multiply-adds on 32 x 32 tiles, any shape and row count.
cudaError_t launch_mat_f32(const MatArgs& a, cudaStream_t st);

// bf16: tcgen05 / TMEM, both operands staged by TMA, any shape and row count. Launches whose tiles leave SMs idle split K
// over several CTAs through `sc` (partial tiles, summed in order by the last to arrive). Grouped by expert: with `gather`
// (at most MAT_GATHER_ROWS rows) every expert multiplies all rows and keeps its own; otherwise the x rows are the sorted
// rows. max_tiles: upper bound of the row tiles of a grouped launch.
constexpr int MAT_GATHER_ROWS = 32;
cudaError_t launch_mat_tc5(const MatArgs& a, int max_tiles, cudaStream_t st);
int mat_tc5_take_timeout();    // as tc5_take_timeout (kernels.h)

// ── the stream between the products ──
// x0[t] = table[ids[t]] * scale (+ pos_table[tok_pos[t]], or null) (f32), xb (or null) = the same, or its norm (norm.w), in the
// compute type (row stride ldb, padding zeroed). Both tables have rows of ldt.
cudaError_t launch_embed_scaled(const void* table, const void* pos_table, int ldt, bool f32, const uint32_t* ids, const int32_t* tok_pos, int n_tok,
                                int width, float scale, const TanhNorm& norm, float* x0, void* xb, int ldb, cudaStream_t st);
// The gain of a norm: one number, or one per coordinate.
struct RowGain {
    const float* g;
    bool per_coord;
};
// x_out = x + mult * rms_norm(y) * gain, f32; xb as above.
cudaError_t launch_norm_residual(const float* y, int ldy, const RowGain& gain, float eps, float mult, const float* x, float* x_out, void* xb, int ldb,
                                 bool f32, int n_tok, int width, cudaStream_t st);
// x_out = x + mult * rms_norm(mixture of expert outputs) * gain, then (dwa) the depth average.
struct CombineArgs {
    const float* x;            // stream before the feed-forward
    float* history;            // [depth + 1][rows_cap][width]: layer results, the embedding output first (null: not kept)
    int64_t hist_stride;
    int depth;                 // this layer's result is history[depth]
    const float* dwa;          // [depth + 1] coefficients, null: no depth average
    float* x_out;
    void* xb;
    int ldb;
    bool f32;
    // feed-forward (null y: none): sum over k of weight[t][k] * y[slot_of[t][k]] (+ y_shared[t], times sigmoid(shared_gate)
    // where that is given)
    const float* y;
    int ldy;
    const int32_t* slot_of;
    const float* weight;
    int top;
    const float* y_shared;
    const float* shared_gate;
    int ld_gate;
    RowGain gain;
    float eps, mult;
};
cudaError_t launch_combine(const CombineArgs& a, int n_tok, int width, cudaStream_t st);
// out (compute type) = rms_norm(x[rows[i] or i]) * gain.
cudaError_t launch_row_norm(const float* x, const int32_t* rows, int n_rows, int width, const RowGain& gain, float eps, void* out, int ldo, bool f32,
                            cudaStream_t st);
// out (compute type) = tanh norm of x[rows[i] or i].
cudaError_t launch_tanh_norm(const float* x, const int32_t* rows, int n_rows, int width, const TanhNorm& norm, void* out, int ldo, bool f32, cudaStream_t st);

// ── experts ──
// How a token's experts follow from its logits (model_plan.h: RouteRule). Ties: the lower index.
struct RouteShape {
    int experts, top;
    bool all;                  // ROUTE_ALL
    int groups, keep;
    float scale;
};
// Per token the chosen experts with their weights weight[t][top], and the (token, choice) pairs sorted by expert: MoeRows
// tables and slot_of[t][k] = sorted row of a pair. pick[t][top] is scratch.
struct MoeTables {
    int32_t *row_off, *row_src, *active, *n_active, *tile_group, *tile_row, *n_tiles, *slot_of;
};
cudaError_t launch_moe_route(const float* logits, int ld, const float* bias, const RouteShape& r, int n_tok, int32_t* pick, float* weight,
                             const MoeTables& t, cudaStream_t st);
// dst[i] = src[row_src[i]] for n rows of ld elements of the compute type (ld * element size a multiple of 16).
cudaError_t launch_gather_act(const void* src, const int32_t* row_src, int n, int ld, bool f32, void* dst, cudaStream_t st);

// ── latent attention ──
// One layer's slice of the paged latent cache: [page][16 tokens][ld] rows of the compute type, a row being
// latent (rank16 = rank rounded to 16, zero-padded) then the rotated key part (rot16).
struct LatentCache {
    void* pool;
    const int32_t* page_table;
    int max_pages;
    int rank, rank16, rot, rot16, ld;
};
struct LatentShape {
    int heads, dim, rot, vdim;
    int window;
    float scale;
};
// proj[t] (f32, row stride ldp): q head by head [dim | rot], then (own cache only) latent | rotated key part.
// Rotates the q and key parts by cos_sin[pos][rot / 2], norms the latent (gain vector, eps), appends it to the cache.
// Absorbed form (qn != null): unrotated q parts to qn[t][heads][ldqn], rotated ones to qabs[t][heads][ld] at rank16.
// Expanded form (qf != null): qf[t][heads][dim16 + rot16].
cudaError_t launch_latent_append(const float* proj, int ldp, const LatentShape& s, const LatentCache& c, bool own, const float* norm_gain,
                                 float eps, const float2* cos_sin, const int32_t* tok_slot, const int32_t* tok_pos, void* qn, int ldqn,
                                 void* qabs, void* qf, bool f32, int n_tok, cudaStream_t st);
// Absorbed attention: scores and values straight from the latent rows. o[t][heads][ldo] (compute type) = normalised
// mixture of latents. n_splits > 1 splits the keys over blocks (latent_attention_splits of the longest range to visit, or
// fewer): bf16 over a cluster, f32 and ranks beyond the tensor-core kernel through `part`
// (latent_part_floats(n_tok, heads, splits, rank) floats).
int latent_attention_splits(int heads, int n_tok, int keys, bool f32);
size_t latent_part_floats(int n_tok, int heads, int n_splits, int rank);
cudaError_t launch_latent_attention(const void* qabs, const LatentShape& s, const LatentCache& c, const int32_t* tok_slot, const int32_t* tok_pos,
                                    void* o, int ldo, float* part, int n_splits, bool f32, int n_tok, cudaStream_t st);
// Expanded attention (bf16, many rows): keys and values of the step's key ranges have been rebuilt from gathered latents.
bool latent_expanded_supported(int dim, int rot, int vdim);
cudaError_t launch_latent_gather(const LatentCache& c, const int32_t* key_slot, const int32_t* key_pos, int n_keys, void* dst, cudaStream_t st);
// A tile of up to LATENT_Q_TILE consecutive tokens of one sequence.
struct LatentTile {
    int32_t row0, n;           // token rows
    int32_t pos0;              // position of the first
    int32_t key_row;           // gathered row of position key_pos0
    int32_t key_pos0;
};
constexpr int LATENT_Q_TILE = 64;
// kv[key][heads][dim16 + vdim16], lat[key][ld] the gathered latent rows (their rotated part is the keys'); out[t][ldo]
// head by head, times sigmoid(gate[t * ldgate + head]).
cudaError_t launch_latent_expanded(const void* qf, const void* kv, const void* lat, const LatentShape& s, const LatentCache& c,
                                   const LatentTile* tiles, int n_tiles, const float* gate, int ldgate, void* out, int ldo, cudaStream_t st);

// ── grouped attention ──
// One layer's slice of the paged cache: [page][kv head][16 tokens][ld] of the compute type. A row is dim16 | vdim16: the
// key and the value, rotated, padded with zeros to multiples of 16. Where the values are the keys (shared), a row is the key
// as projected, once, and GROUPED_TAIL elements whose first four bytes are the f32 reciprocal of its root mean square (one
// without a norm); scores take that factor, and the keys' norm weight is part of the queries.
constexpr int GROUPED_TAIL = 8;
struct GroupedCache {
    void* pool;
    const int32_t* page_table;
    int max_pages;
    int dim16, vdim16;
    int ld;                    // shared ? dim16 + GROUPED_TAIL : dim16 + vdim16
    bool shared;
};
struct GroupedShape {
    int heads, kv_heads, dim, vdim, rot;
    int window;
    float scale;
    bool neighbours;           // rotation of pairs (2 i, 2 i + 1), else (i, i + rot / 2)
    int keep;                  // attention with mixed heads: first keys that stay visible behind the window
    float softcap;             // attention with mixed heads: of the scaled scores (0: none)
};
// What happens to queries, keys and values between the projection and the cache; null: nothing.
struct GroupedInput {
    const float* bias;         // [heads * dim | kv_heads * dim | kv_heads * vdim]
    bool norm;                 // queries and keys over their root mean square ...
    const float *q_gain, *k_gain;  // ... times [dim]
    float eps;
    const float* temperature;  // factor of the queries, by position
    const float2 *cs_key, *cs_val;  // angles [pos][rot / 2] of queries and keys, [pos][vdim / 2] of values
    // Convolution over time behind the bias (launch_conv_append): [taps][channels], the last tap on the token itself. The taps - 1
    // values before a slot's next token are at tail + slot * tail_stride, [taps - 1][channels], the oldest first; what stands for
    // tokens before the sequence's start is not read. Rows of a slot may stand anywhere in a step.
    const float* conv;
    int taps;
    float* tail;
    int64_t tail_stride;
    const int32_t* back;       // many rows: row of the slot's token before this one, -1: in an earlier step
};
// proj[t] (f32, row stride ldp): queries head by head, keys, values (not when shared). q[t][heads][dim16] in the compute type,
// keys and values to the cache.
cudaError_t launch_grouped_append(const float* proj, int ldp, const GroupedShape& s, const GroupedCache& c, const GroupedInput& in,
                                  const int32_t* tok_slot, const int32_t* tok_pos, void* q, bool f32, int n_tok, cudaStream_t st);
// What else enters the scores, the softmax and the output; null: nothing.
struct GroupedTerms {
    const float* rel;          // [heads][n_rel], added to the scaled score: by distance, the last one from there on
    int n_rel;
    const float* sink;         // [heads]: logit of one more term of the denominator
    const float* gate;         // output times sigmoid(gate[t * ldgate + head * vdim + coordinate])
    int64_t ldgate;
    const float2* cs_val;      // mixtures are turned back by these angles
};
// out[t][ldo] (compute type), head by head vdim values: the mixtures. Any sizes up to GROUPED_MAX_VDIM. n_splits > 1 (bf16:
// grouped_attention_splits of the longest range to visit) splits the keys over the blocks of a cluster.
constexpr int GROUPED_MAX_VDIM = 1024;
bool grouped_mma_supported(const GroupedShape& s);
int grouped_attention_splits(const GroupedShape& s, int n_tok, int keys, bool f32);
cudaError_t launch_grouped_attention(const void* q, const GroupedShape& s, const GroupedCache& c, const GroupedTerms& x, const int32_t* tok_slot,
                                     const int32_t* tok_pos, void* out, int ldo, int n_splits, bool f32, int n_tok, cudaStream_t st);
// bf16, many rows: tiles of up to GROUPED_Q_TILE consecutive tokens of one sequence.
struct GroupedTile {
    int32_t row0, n;           // token rows
    int32_t pos0;              // position of the first
    int32_t slot;
};
constexpr int GROUPED_Q_TILE = 64;
cudaError_t launch_grouped_prefill(const void* q, const GroupedShape& s, const GroupedCache& c, const GroupedTerms& x, const GroupedTile* tiles,
                                   int n_tiles, void* out, int ldo, cudaStream_t st);

// launch_grouped_append with a convolution (without norms, temperature and rotated values). Up to 32 rows: tiles null; the tails
// are brought up to date. More: tiles of up to MIXED_Q_TILE tokens that cover the step, and launch_conv_tails behind it with every
// slot's last row in the step.
constexpr int MIXED_Q_TILE = 16;
cudaError_t launch_conv_append(const float* proj, int ldp, const GroupedShape& s, const GroupedCache& c, const GroupedInput& in, const GroupedTile* tiles,
                               int n_tiles, const int32_t* tok_slot, const int32_t* tok_pos, void* q, bool f32, int n_tok, cudaStream_t st);
cudaError_t launch_conv_tails(const float* proj, int ldp, const GroupedShape& s, const GroupedInput& in, const int32_t* tok_slot, const int32_t* ends,
                              int n_ends, cudaStream_t st);

// ── grouped attention whose heads' softmax weights are mixed ──
// w_h <- sum_g mix[h][g] w_g over all query heads, then head h takes the values of its own cached head. Needs every head's weights
// where one head's mixture is made, so there are two passes: scores and softmax denominators, then weights and values. Windows may
// keep a sequence's first keys, scores may be capped, denominators may have a sink. Kept pages and the window's pages are visited
// as one run: a row's i-th visited key is at score[row][head][i].
struct MixedTerms {
    const float* mix;          // [heads][heads]
    const float* sink;         // [heads] or null
};
struct MixedScratch {
    float* score;              // [rows][heads][span]
    int rows, span;            // span: mixed_span()
    float2* part;              // [rows][heads][MIXED_SPLITS]: maximum and sum of a split of the keys
    float2* stat;              // plain arithmetic: [tokens of a step][heads], maximum and reciprocal of the denominator
    float* norm;               // many rows: [tokens of a step][heads], what makes a log2 score a weight
};
constexpr int MIXED_SPLITS = 8;
int mixed_span(const GroupedShape& s, int max_ctx);       // most keys a token visits, whole pages
bool mixed_mma_supported(const GroupedShape& s, const GroupedCache& c);
int mixed_attention_splits(const GroupedShape& s, int n_tok, int keys);
// Few rows (bf16), or any sizes and rows in plain arithmetic (f32, and sizes the tensor-core kernels do not cover; n_splits 1).
cudaError_t launch_mixed_attention(const void* q, const GroupedShape& s, const GroupedCache& c, const MixedTerms& x, const MixedScratch& m,
                                   const int32_t* tok_slot, const int32_t* tok_pos, void* out, int ldo, int n_splits, bool f32, int n_tok, cudaStream_t st);
// bf16, many rows: the step's tokens as tiles of GROUPED_Q_TILE (first pass) and of MIXED_Q_TILE (second).
cudaError_t launch_mixed_prefill(const void* q, const GroupedShape& s, const GroupedCache& c, const MixedTerms& x, const MixedScratch& m,
                                 const GroupedTile* wide, int n_wide, const GroupedTile* narrow, int n_narrow, void* out, int ldo, cudaStream_t st);

// ── mixers with a state matrix (model_plan.h: StateMixerSpec) ──
// State of a slot: [heads][vdim][dim_pad] f32, slots slot_stride floats apart (a value column's keys are contiguous). A sequence's first token (position 0)
// starts from zeros, whatever the slot held.
struct StateShape {
    int heads, dim, vdim;
    int rule;                  // StateRule
    int dim_pad;               // state_dim_pad(dim)
    float eps;
    bool norm_all;             // STATE_DECAY: all heads of a token are normed together
    int gate;                  // StateGate
    int rot;                   // STATE_DECAY: coordinates of queries and keys that are rotated, in halves
    float key_scale;           // STATE_DECAY
};
int state_dim_pad(int dim);
struct StateArgs {
    StateShape s;
    float* state;
    int64_t slot_stride;
    const float* decay;        // STATE_DECAY: [heads]
    // STATE_DECAY: proj[t] = q | k | v (silu applied where the mixer has it) | gate logits. STATE_DELTA: r | k | v | removal logits |
    // gate logits. STATE_FORGET: q (silu applied) | forget logits | v. No gate: no logits.
    const float* proj;
    int ldp;
    const float* a_bias;       // STATE_DELTA: of the removal logits, STATE_FORGET: of the forget logits, [heads * dim]
    const float* lower;        // STATE_FORGET: [heads * dim]
    const float2* cs;          // STATE_DECAY: angles [pos][rot / 2]
    const float* w0;           // STATE_DELTA: decay logit = w0 + W2 low[t]
    const void* w2;            // compute type, [heads * dim][ldlow]
    const void* low;           // compute type, [t][ldlow]
    int ldlow;
    const float* wlogit;       // many rows: W2 low[t] (f32, [t][heads * dim])
    float* rec;                // many rows: scratch, state_record_floats per group
    const float* gain;         // [heads * vdim] or null
    const int32_t *tok_slot, *tok_pos;
    void* out;                 // compute type, [t][ldo]
    int ldo;
    bool f32;
};
// Up to STATE_STEP_ROWS rows: gates, recurrence, norm and output gate in one launch. Rows of one slot are taken in order.
constexpr int STATE_STEP_ROWS = 32;
cudaError_t launch_state_step(const StateArgs& a, int n_tok, cudaStream_t st);
// Any number of rows, in groups of up to state_group() tokens of one slot, in order: groups[i][] names their rows (-1 behind the
// last). A segment is a slot's run of groups.
constexpr int STATE_GROUP_F32 = 4, STATE_CHUNK = 16;
inline int state_group(bool f32) { return f32 ? STATE_GROUP_F32 : STATE_CHUNK; }
struct StateSegment {
    int32_t group0, n_groups, slot, fresh;  // fresh: starts at position 0
};
size_t state_record_floats(const StateShape& s, bool f32);  // of a group
cudaError_t launch_state_scan(const StateArgs& a, const StateSegment* seg, int n_seg, const int32_t* groups, int n_groups, cudaStream_t st);

}  // namespace sp
