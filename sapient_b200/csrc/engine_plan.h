// State of a plan-driven engine (engine_plan.cu): the packed weights of every layer, the latent cache and the buffers of
// a step. Owned by Engine, which keeps the sequence slots, the page tables, the step graphs and the host API.
#pragma once
#include <vector>

#include "model_plan.h"
#include "plan_kernels.h"

namespace sp {

// Matrices in the compute type, rows padded to kp columns.
struct PlanMat {
    void* w = nullptr;
    int n = 0, kp = 0, groups = 1;
};

struct PlanLayer {
    PlanMat proj;              // q | latent and rotated key part (own cache only) | output gate
    int gate_col = 0;          // first gate column of the projection's output
    PlanMat uk_t;              // per head, transposed: query -> latent space
    PlanMat uv;                // per head: latent -> value
    PlanMat kv;                // per head key rows then value rows, each padded to 16: the expanded form
    PlanMat o;
    const float *norm1 = nullptr, *norm2 = nullptr, *dkv_norm = nullptr, *dwa = nullptr;
    PlanMat router;            // experts rows, then the shared expert's gate row
    const float* router_b = nullptr;
    PlanMat gu, down, shared_gu, shared_down;
    LatentShape shape{};
    LatentCache cache{};       // the layer's own, or the one it borrows
    bool own = true, expand = false;
    const float2* cos_sin = nullptr;
};

struct PlanState {
    ModelPlan plan;
    bool f32 = false;
    int elem() const { return f32 ? 4 : 2; }
    std::vector<PlanLayer> layers;
    PlanMat embed, head;
    const float* final_norm = nullptr;
    int wp = 0;                // padded width
    size_t page_bytes = 0;     // all layers' rows of one page
    std::vector<size_t> cache_run, cache_base;  // per owning layer: bytes of a page, offset of its slice
    void* cache = nullptr;
    // buffers of a step
    void *xb = nullptr, *qn = nullptr, *qabs = nullptr, *qf = nullptr, *olat = nullptr, *attn = nullptr, *act = nullptr, *act_shared = nullptr,
         *xs = nullptr, *kvx = nullptr, *lat = nullptr, *fin = nullptr;
    float *proj = nullptr, *y = nullptr, *y_expert = nullptr, *y_shared = nullptr, *logit = nullptr, *weight = nullptr, *part = nullptr, *history = nullptr;
    int32_t *pick = nullptr, *tables = nullptr, *host_tiles = nullptr, *dev_tiles = nullptr;
    MoeTables moe{};
    int keys_cap = 0;          // gathered keys a step may hold
    // the expanded form of the current step (0 tiles: absorbed)
    int n_tiles = 0, n_keys = 0;
    std::vector<void*> owned;
};

}  // namespace sp
