// Plan layers of the post-norm form (model_plan.h: FORM_POST_NORM): x <- x + m norm(mixer(x)), then x <- x + m norm(ff(x)). Every
// sublayer reads the stream itself, which each kernel that changes it also leaves in the compute type. Mixers are latent or
// grouped attention. A dense feed-forward is two products; experts are router, choice and grouping, gate | up of the chosen
// and the shared expert, down, and one kernel for mixture, norm, residual and, where the design has it, depth average.
#include "engine_plan.h"

#include "sp_common.cuh"

namespace sp {

void PlanPacker::post_norm_layer(int i) {
    const LayerPlan& lp = p.plan.layers[(size_t)i];
    PlanLayer& l = p.layers[(size_t)i];
    const int W = p.plan.width;
    l.norm1 = gain(lp.prefix + "norm1");
    if (lp.mixer == MIX_LATENT) {
        latent_layer(i);
    } else {
        std::vector<MixPart> parts;
        const int out_cols = mixers(i, parts);
        if (status != SP_OK || !alloc(l.proj, 1, l.mix_rows, W) || !alloc(l.o, 1, W, out_cols)) return;
        put_mixer_rows(i, parts);
        put_mixer_out(i);
    }
    if (p.plan.depth_average) l.dwa = vec(lp.prefix + "dwa", i + 2);
    if (status != SP_OK || lp.mlp == MLP_NONE) return;
    l.norm2 = gain(lp.prefix + "norm2");
    if (lp.mlp == MLP_MOE) {
        experts(i);
    } else {
        const int F = lp.dense.ff;
        if (!alloc(l.up, 1, F, W) || !alloc(l.down, 1, W, F)) return;
        put(l.up, 0, need(lp.prefix + "mlp.up", F, W), 0, F, W);
        put(l.down, 0, need(lp.prefix + "mlp.down", W, F), 0, W, F);
        PlanSizes::most(p.need.act, (size_t)l.down.kp);
    }
}

void PlanPacker::experts(int i) {
    const LayerPlan& lp = p.plan.layers[(size_t)i];
    const MoeSpec& s = lp.moe;
    PlanLayer& l = p.layers[(size_t)i];
    const std::string ml = lp.prefix + "mlp.";
    const int W = p.plan.width, E = s.experts, F = s.expert.ff;
    if (!alloc(l.router, 1, E + (s.shared_gate ? 1 : 0), W)) return;
    put(l.router, 0, need(ml + "router", E, W), 0, E, W);
    l.router_b = vec(ml + s.bias, E);
    if (!alloc(l.gu, E, 2 * (int64_t)F, W) || !alloc(l.down, E, W, F)) return;
    for (int x = 0; x < E; ++x) {
        const std::string ex = ml + "e" + std::to_string(x) + ".";
        put(l.gu, (int64_t)x * 2 * F, need(ex + "gate", F, W), 0, F, W);
        put(l.gu, (int64_t)x * 2 * F + F, need(ex + "up", F, W), 0, F, W);
        put(l.down, (int64_t)x * W, need(ex + "down", W, F), 0, W, F);
    }
    if (s.has_shared) {
        const int S = s.shared.ff;
        if (!alloc(l.shared_gu, 1, 2 * (int64_t)S, W) || !alloc(l.shared_down, 1, W, S)) return;
        put(l.shared_gu, 0, need(ml + "shared.gate", S, W), 0, S, W);
        put(l.shared_gu, S, need(ml + "shared.up", S, W), 0, S, W);
        put(l.shared_down, 0, need(ml + "shared.down", W, S), 0, W, S);
        if (s.shared_gate) put(l.router, E, need(ml + "shared.sg", 1, W), 0, 1, W);
        PlanSizes::most(p.need.act_shared, (size_t)l.shared_down.kp);
    }
    PlanSizes::most(p.need.act, (size_t)s.top * l.down.kp);
    PlanSizes::most(p.need.pairs, (size_t)s.top);
    p.need.experts = std::max(p.need.experts, E);
}

static MatUnit unit_of(const GatedExpertSpec& s) { return MatUnit{s.limit, s.alpha, s.shift}; }

int Engine::plan_experts(int li, int T) {
    PlanState& p = *plan_;
    PlanLayer& l = p.layers[(size_t)li];
    const MoeSpec& s = p.plan.layers[(size_t)li].moe;
    const int W = p.plan.width, E = s.experts, pairs = T * s.top;
    SP_TRY(plan_mat(l.router, p.xb, p.wp, T, p.logit, l.router.n, true));
    SP_LAUNCH(F_ELEM, launch_moe_route(p.logit, l.router.n, l.router_b, RouteShape{E, s.top, s.rule == ROUTE_ALL, s.groups, s.keep, s.scale}, T, p.pick, p.weight, p.moe, stream));
    MatArgs a{};
    a.f32 = p.f32;
    a.m = T;
    a.dual = true;
    a.moe = true;
    a.rows = MoeRows{p.moe.row_off, p.moe.row_src, p.moe.active, p.moe.n_active, p.moe.tile_group, p.moe.tile_row, p.moe.n_tiles};
    a.slots = std::min(E, pairs);
    const MatSeg gu{l.gu.w, s.expert.ff, l.gu.kp, E, unit_of(s.expert), p.xb, p.wp, 0, p.act, l.down.kp, 0};
    const MatSeg sgu{l.shared_gu.w, s.shared.ff, l.shared_gu.kp, 1, unit_of(s.shared), p.xb, p.wp, 0, p.act_shared, l.shared_down.kp, 0};
    const MatSeg dn{l.down.w, W, l.down.kp, E, MatUnit{}, p.act, l.down.kp, 0, p.y_expert, W, 0};
    const MatSeg sdn{l.shared_down.w, W, l.shared_down.kp, 1, MatUnit{}, p.act_shared, l.shared_down.kp, 0, p.y_shared, W, 0};
    const int max_tiles = std::min(pairs / MOE_TILE + std::min(E, pairs), pairs);
    if (T <= PLAN_ROWS || p.f32) {
        a.gather = true;
        a.nseg = s.has_shared ? 2 : 1;
        a.seg[0] = gu;
        a.seg[1] = sgu;
        SP_TRY(plan_product(a, max_tiles));
        a.gather = a.dual = false;
        a.out_f32 = true;
        a.x_rows = pairs;
        a.seg[0] = dn;
        a.seg[1] = sdn;
        return plan_product(a, max_tiles);
    }
    SP_LAUNCH(F_ELEM, launch_gather_act(p.xb, p.moe.row_src, pairs, p.wp, p.f32, p.xs, stream));
    a.nseg = 1;
    a.x_rows = pairs;
    a.seg[0] = gu;
    a.seg[0].x = p.xs;
    SP_TRY(plan_product(a, max_tiles));
    a.seg[0] = dn;
    a.dual = false;
    a.out_f32 = true;
    SP_TRY(plan_product(a, max_tiles));
    if (s.has_shared) {
        a.moe = false;
        a.x_rows = 0;
        a.dual = true;
        a.out_f32 = false;
        a.seg[0] = sgu;
        SP_TRY(plan_product(a, 0));
        a.dual = false;
        a.out_f32 = true;
        a.seg[0] = sdn;
        SP_TRY(plan_product(a, 0));
    }
    return SP_OK;
}

// p.y = W_down act(W_up x)
int Engine::plan_dense(int li, int T) {
    PlanState& p = *plan_;
    PlanLayer& l = p.layers[(size_t)li];
    MatArgs a{};
    a.f32 = p.f32;
    a.nseg = a.n_outs = 1;
    a.m = T;
    a.seg[0] = MatSeg{l.up.w, l.up.n, l.up.kp, 1, MatUnit{}, p.xb, p.wp, 0, nullptr, 0, 0};
    a.outs[0] = MatOut{l.up.n, p.act, l.down.kp, MAT_RELU2, p.f32, false};
    SP_TRY(plan_product(a, 0));
    return plan_mat(l.down, p.act, l.down.kp, T, p.y, p.plan.width, true);
}

int Engine::plan_layer_post_norm(int i, int T) {
    PlanState& p = *plan_;
    const int W = p.plan.width;
    const float mult = p.plan.residual_mult, eps = p.plan.eps;
    PlanLayer& l = p.layers[(size_t)i];
    const LayerPlan& lp = p.plan.layers[(size_t)i];
    if (lp.mixer == MIX_LATENT) {
        SP_TRY(plan_latent(i, T));
    } else {
        SP_TRY(plan_mat(l.proj, p.xb, p.wp, T, p.proj, l.mix_rows, true));
        SP_TRY(plan_grouped(i, T));
    }
    SP_TRY(plan_mat(l.o, p.attn, l.o.kp, T, p.y, W, true));
    SP_LAUNCH(F_NORM, launch_norm_residual(p.y, W, l.norm1, eps, mult, i == 0 && p.history ? p.history : x_, x_, p.xb, p.wp, p.f32, T, W, stream));
    if (lp.mlp == MLP_DENSE) {
        SP_TRY(plan_dense(i, T));
        SP_LAUNCH(F_NORM, launch_norm_residual(p.y, W, l.norm2, eps, mult, x_, x_, p.xb, p.wp, p.f32, T, W, stream));
        if (!p.history) return SP_OK;
    }
    CombineArgs c{};
    if (lp.mlp == MLP_MOE) {
        SP_TRY(plan_experts(i, T));
        c.y = p.y_expert;
        c.ldy = W;
        c.slot_of = p.moe.slot_of;
        c.weight = p.weight;
        c.top = lp.moe.top;
        if (lp.moe.has_shared) c.y_shared = p.y_shared;
        if (lp.moe.shared_gate) {
            c.shared_gate = p.logit + lp.moe.experts;
            c.ld_gate = l.router.n;
        }
        c.gain = l.norm2;
        c.eps = eps;
        c.mult = mult;
    } else if (!p.history) {
        return SP_OK;
    }
    c.x = x_;
    c.history = p.history;
    c.hist_stride = (int64_t)d.max_tokens * W;
    c.depth = i + 1;
    c.dwa = l.dwa;
    c.x_out = x_;
    c.xb = p.xb;
    c.ldb = p.wp;
    c.f32 = p.f32;
    SP_LAUNCH(F_NORM, launch_combine(c, T, W, stream));
    return SP_OK;
}

}  // namespace sp
