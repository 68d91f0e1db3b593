// Plan layers of the parallel form (model_plan.h: FORM_PARALLEL): h = norm(x), x <- x + mixer(h) + ff(h). Everything that
// reads h is one product — the mixer's projections in f32, low-rank rows and feed-forward activations in the compute type —
// and the two output projections are one product over [mixer output | activation] that adds into the stream. A layer is
// four launches with a state mixer and five with attention (decode-shaped steps): norm, product in, mixer, product out.
#include "engine_plan.h"

#include "sp_common.cuh"

namespace sp {

void PlanPacker::parallel_layer(int i) {
    const LayerPlan& lp = p.plan.layers[(size_t)i];
    PlanLayer& l = p.layers[(size_t)i];
    const std::string ml = lp.prefix + "mlp.";
    const int W = p.plan.width;
    l.norm1 = gain(lp.prefix + "norm1");
    l.ff = lp.mlp == MLP_DENSE ? lp.dense.ff : 0;
    std::vector<MixPart> parts;
    const int out_cols = mixers(i, parts);
    if (status != SP_OK || !alloc(l.proj, 1, (int64_t)l.mix_rows + l.low_rows + l.ff, W)) return;
    put_mixer_rows(i, parts);
    if (l.ff) put(l.proj, l.mix_rows + l.low_rows, need(ml + "up", l.ff, W), 0, l.ff, W);
    l.act_col = l.ff ? (out_cols + 7) & ~7 : out_cols;
    if (!alloc(l.o, 1, W, l.act_col + l.ff)) return;
    put_mixer_out(i);
    if (l.ff) put(l.o, 0, need(ml + "down", W, l.ff), 0, W, l.ff, false, l.act_col);
}

int Engine::plan_layer_parallel(int i, int T) {
    PlanState& p = *plan_;
    PlanLayer& l = p.layers[(size_t)i];
    const int W = p.plan.width;
    SP_LAUNCH(F_NORM, launch_row_norm(x_, nullptr, T, W, l.norm1, p.plan.eps, p.xb, p.wp, p.f32, stream));
    MatArgs a{};
    if (l.ff) {
        a.outs[0] = MatOut{l.proj.n, (uint8_t*)p.attn + (size_t)l.act_col * p.elem(), l.o.kp, MAT_RELU2, p.f32, false};
        a.n_outs = 1;
    }
    SP_TRY(plan_mixer_in(i, T, a));
    SP_TRY(plan_mixers(i, T));
    a.n_outs = 1;
    a.seg[0] = MatSeg{l.o.w, W, l.o.kp, 1, MatUnit{}, p.attn, l.o.kp, 0, nullptr, 0, 0};
    a.outs[0] = MatOut{W, x_, W, MAT_ID, true, true};
    return plan_product(a, 0);
}

}  // namespace sp
