// Plan layers of the pre-norm form (model_plan.h: FORM_PRE_NORM): x <- x + mixer(norm(x)), then x <- x + ff(norm(x)). A norm without
// statistics costs no launch: the product that adds into the stream leaves the next sublayer's input beside it. A layer is then
// product in, the mixers' launches, product out, and two products for its feed-forward.
#include <cmath>

#include "engine_plan.h"
#include "sp_common.cuh"

namespace sp {

void PlanPacker::pre_norm_layer(int i) {
    const LayerPlan& lp = p.plan.layers[(size_t)i];
    PlanLayer& l = p.layers[(size_t)i];
    const int W = p.plan.width;
    const bool tanh = p.plan.norm == NORM_TANH;
    if (tanh) l.tanh1 = tanh_norm(lp.prefix + "norm1");
    else l.norm1 = gain(lp.prefix + "norm1");
    if (lp.mixer == MIX_LATENT || lp.mlp == MLP_MOE) { fail(SP_ERR_ARG, "latent attention and experts are not part of the pre-norm form"); return; }
    std::vector<MixPart> parts;
    const int out_cols = mixers(i, parts);
    if (status != SP_OK || !alloc(l.proj, 1, (int64_t)l.mix_rows + l.low_rows, W) || !alloc(l.o, 1, W, out_cols)) return;
    put_mixer_rows(i, parts);
    put_mixer_out(i);
    if (status != SP_OK || lp.mlp == MLP_NONE) return;
    if (tanh) l.tanh2 = tanh_norm(lp.prefix + "norm2");
    else l.norm2 = gain(lp.prefix + "norm2");
    const std::string ml = lp.prefix + "mlp.";
    const int F = lp.dense.ff;
    if (!alloc(l.up, 1, F, W) || !alloc(l.down, 1, W, F)) return;
    put(l.up, 0, need(ml + "up", F, W), 0, F, W);
    put(l.down, 0, need(ml + "down", W, F), 0, W, F);
    PlanSizes::most(p.need.act, (size_t)l.down.kp);
    if (lp.dense.act == DENSE_XIELU) {
        const std::vector<float> pq = host(ml + "act", 1, 2);
        if (status != SP_OK) return;
        auto softplus = [](double z) { return std::max(z, 0.0) + std::log1p(std::exp(-std::fabs(z))); };
        l.act_arg[0] = (float)softplus(pq[0]);
        l.act_arg[1] = (float)(0.5 + softplus(pq[1]));
    }
}

int Engine::plan_layer_pre_norm(int i, int T) {
    PlanState& p = *plan_;
    PlanLayer& l = p.layers[(size_t)i];
    const int W = p.plan.width;
    const bool tanh = p.plan.norm == NORM_TANH, ff = p.plan.layers[(size_t)i].mlp != MLP_NONE;
    const TanhNorm next = tanh && i + 1 < (int)p.layers.size() ? p.layers[(size_t)i + 1].tanh1 : TanhNorm{};
    MatArgs a{};
    if (!tanh) SP_LAUNCH(F_NORM, launch_row_norm(x_, nullptr, T, W, l.norm1, p.plan.eps, p.xb, p.wp, p.f32, stream));
    SP_TRY(plan_mixer_in(i, T, a));
    SP_TRY(plan_mixers(i, T));
    // x += W y, and the norm of the result for what reads it
    auto add = [&](const PlanMat& w, const void* y, const TanhNorm& norm) {
        a.n_outs = 1;
        a.seg[0] = MatSeg{w.w, W, w.kp, 1, MatUnit{}, y, w.kp, 0, nullptr, 0, 0};
        a.outs[0] = MatOut{W, x_, W, MAT_ID, true, true};
        a.norm = MatNorm{norm, p.xb, p.wp};
        return plan_product(a, 0);
    };
    SP_TRY(add(l.o, p.attn, ff ? l.tanh2 : next));
    if (!ff) return SP_OK;
    if (!tanh) SP_LAUNCH(F_NORM, launch_row_norm(x_, nullptr, T, W, l.norm2, p.plan.eps, p.xb, p.wp, p.f32, stream));
    a.norm = MatNorm{};
    a.arg[0] = l.act_arg[0];
    a.arg[1] = l.act_arg[1];
    a.seg[0] = MatSeg{l.up.w, l.up.n, l.up.kp, 1, MatUnit{}, p.xb, p.wp, 0, nullptr, 0, 0};
    a.outs[0] = MatOut{l.up.n, p.act, l.down.kp, p.plan.layers[(size_t)i].dense.act == DENSE_XIELU ? MAT_XIELU : MAT_RELU2, p.f32, false};
    SP_TRY(plan_product(a, 0));
    return add(l.down, p.act, next);
}

}  // namespace sp
