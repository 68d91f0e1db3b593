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
    return s.rule == STATE_DELTA ? StateCols{0, hd, 2 * hd, 3 * hd, 4 * hd} : StateCols{0, hd, 2 * hd, 0, 2 * hd + hv};
}

constexpr float EXP_MINUS_HALF = 0.60653065971263342f;
__device__ __forceinline__ float channel_decay(float logit) { return expf(-EXP_MINUS_HALF * sigmoid_f32(logit)); }

// Where a scan's record has the outputs: value t of column c at v + t * v_pad + c; records are `floats` apart.
struct StateRecordView {
    int v, v_pad, floats;
};
StateRecordView state_chunk_view(const StateShape& s);  // state_chunk.cu
cudaError_t launch_state_chunks(const StateArgs& a, const StateSegment* seg, int n_seg, const int32_t* groups, int n_groups, cudaStream_t st);

}  // namespace sp
