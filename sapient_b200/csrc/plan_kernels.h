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

// A family of equally shaped matrices [groups][rows][kp]. `dual`: rows = 2 n, the first n are the gate and the last n the
// up-projection of a clamped gated unit, whose n activations are the output.
struct MatSeg {
    const void* w;
    int n, kp, groups;
    float limit, alpha;        // dual: g = min(., limit), u = clamp(., +-limit), y = g sigmoid(alpha g) (u + 1)
    const void* x;             // compute type
    int ldx;
    int64_t xgs;               // elements between the inputs of consecutive groups (per-head products)
    void* y;
    int ldy;
    int64_t ygs;
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
};

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
// x0[t] = table[ids[t]] * scale (f32), xb = the same in the compute type (row stride ldb, padding zeroed).
cudaError_t launch_embed_scaled(const void* table, int ldt, bool f32, const uint32_t* ids, int n_tok, int width, float scale, float* x0, void* xb,
                                int ldb, cudaStream_t st);
// x += rms_norm(y) * gain (one number), f32; xb as above.
cudaError_t launch_norm_residual(const float* y, int ldy, const float* gain, float eps, const float* x, float* x_out, void* xb, int ldb, bool f32,
                                 int n_tok, int width, cudaStream_t st);
struct CombineArgs {
    const float* x;            // stream before the feed-forward
    float* history;            // [depth + 1][rows_cap][width]: layer results, the embedding output first
    int64_t hist_stride;
    int depth;                 // this layer's result is history[depth]
    const float* dwa;          // [depth + 1] coefficients, null: no depth average
    float* x_out;
    void* xb;
    int ldb;
    bool f32;
    // feed-forward (null y: none): sum over k of weight[t][k] * y[slot_of[t][k]] (+ sigmoid(shared_gate) * y_shared[t])
    const float* y;
    int ldy;
    const int32_t* slot_of;
    const float* weight;
    int top;
    const float* y_shared;
    const float* shared_gate;
    int ld_gate;
    const float* gain;
    float eps;
};
cudaError_t launch_combine(const CombineArgs& a, int n_tok, int width, cudaStream_t st);
// out (compute type) = rms_norm(x[rows[i] or i]) * gain.
cudaError_t launch_final_norm(const float* x, const int32_t* rows, int n_rows, int width, const float* gain, float eps, void* out, int ldo, bool f32,
                              cudaStream_t st);

// ── experts ──
// Per token the `top` largest of logits[t][0..experts) + bias (ties: the lower index) with the softmax over the chosen ones
// as weight[t][top], and the (token, choice) pairs sorted by expert: MoeRows tables and slot_of[t][k] = sorted row of a
// pair. pick[t][top] is scratch.
struct MoeTables {
    int32_t *row_off, *row_src, *active, *n_active, *tile_group, *tile_row, *n_tiles, *slot_of;
};
cudaError_t launch_moe_route(const float* logits, int ld, const float* bias, int n_tok, int experts, int top, int32_t* pick, float* weight,
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

}  // namespace sp
