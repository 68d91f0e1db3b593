// What the kernels of state mixers (state_mixer.cu, state_chunk.cu) share.
#pragma once
#include "model_plan.h"
#include "plan_common.cuh"
#include "plan_kernels.h"

namespace sp {

// Columns of a projection row (plan_kernels.h: StateArgs::proj).
struct StateCols {
    int r, k, v, a, g;
};
__host__ __device__ __forceinline__ StateCols state_cols(const StateShape& s) {
    const int hd = s.heads * s.dim, hv = s.heads * s.vdim;
    if (s.rule == STATE_FORGET) return StateCols{0, 0, 2 * hd, hd, 2 * hd + hv};  // (its keys follow from the forget logits)
    return s.rule == STATE_DELTA ? StateCols{0, hd, 2 * hd, 3 * hd, 4 * hd} : StateCols{0, hd, 2 * hd, 0, 2 * hd + hv};
}

constexpr float EXP_MINUS_HALF = 0.60653065971263342f;
__device__ __forceinline__ float channel_decay(float logit) { return expf(-EXP_MINUS_HALF * sigmoid_f32(logit)); }

// STATE_FORGET: how much of a channel stays, and its key, one minus that.
__device__ __forceinline__ float2 forget_gate(float logit, float lower) {
    return make_float2(fmaf(1.f - lower, sigmoid_f32(logit), lower), (1.f - lower) * sigmoid_f32(-logit));
}
// Coordinate c of x, the first `rot` of which are turned in halves by cs.
__device__ __forceinline__ float rotated(const float* x, int c, int rot, const float2* cs) {
    if (c >= rot) return x[c];
    const int half = rot / 2;
    return c < half ? x[c] * cs[c].x - x[c + half] * cs[c].y : x[c] * cs[c - half].x + x[c - half] * cs[c - half].y;
}
// What is left to do with a normed output: coordinate i of the heads' outputs of a row whose gate logits are at g.
__device__ __forceinline__ float state_factor(const StateArgs& a, const float* g, int i) {
    float f = a.gain ? a.gain[i] : 1.f;
    if (a.s.gate == STATE_GATE_SIGMOID) f *= sigmoid_f32(g[i]);
    else if (a.s.gate == STATE_GATE_SILU) f *= silu_f32(g[i]);
    return f;
}

// Where a scan's record has the outputs: value t of column c at v + t * v_pad + c; records are `floats` apart.
struct StateRecordView {
    int v, v_pad, floats;
};
StateRecordView state_chunk_view(const StateShape& s);  // state_chunk.cu
cudaError_t launch_state_chunks(const StateArgs& a, const StateSegment* seg, int n_seg, const int32_t* groups, int n_groups, cudaStream_t st);

}  // namespace sp
