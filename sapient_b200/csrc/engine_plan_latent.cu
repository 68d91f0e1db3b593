// Plan layers with latent attention and experts (model_plan.h: FORM_POST_NORM), ten to fifteen launches each: projections,
// rotation + cache append, then either queries to latent space, absorbed attention and value maps or gather, rebuilt keys
// and values and expanded attention; output projection, norm + residual, router, choice and grouping, gate|up of the chosen
// and the shared expert, down, mixture + norm + residual + depth average. Steps of up to PLAN_ROWS rows take the absorbed
// attention; longer ones, where rebuilding the keys pays, the expanded attention.
#include "engine_plan.h"

#include "sp_common.cuh"

namespace sp {

constexpr int PLAN_SPLIT_ROWS = 256;  // (rows x key splits) of the absorbed attention's partials

size_t plan_latent_part_rows() { return PLAN_SPLIT_ROWS; }

void PlanPacker::latent_layer(int i) {
    const ModelPlan& mp = p.plan;
    const LayerPlan& lp = mp.layers[(size_t)i];
    const LatentAttentionSpec& m = lp.latent;
    PlanLayer& l = p.layers[(size_t)i];
    const std::string mx = lp.prefix + "mix.";
    const int W = mp.width, H = m.heads, D = m.dim, R = m.rot_dim, V = m.vdim, K = m.kv_rank;
    p.has_latent = true;
    l.own = m.kv_from < 0;
    l.shape = LatentShape{H, D, R, V, m.window, m.scale};
    l.norm1 = vec(lp.prefix + "norm1", 1);
    // projections that read the mixer's input
    const int q_rows = H * (D + R), kv_rows = l.own ? K + R : 0;
    l.gate_col = q_rows + kv_rows;
    if (!alloc(l.proj, 1, q_rows + kv_rows + H, W)) return;
    put(l.proj, 0, need(mx + "q", q_rows, W), 0, q_rows, W);
    if (l.own) {
        put(l.proj, q_rows, need(mx + "dkv", kv_rows, W), 0, kv_rows, W);
        l.dkv_norm = vec(mx + "dkv.norm", K);
    }
    put(l.proj, l.gate_col, need(mx + "g", H, W), 0, H, W);
    const DevTensor *uk = need(mx + "uk", (int64_t)H * D, K), *uv = need(mx + "uv", (int64_t)H * V, K);
    if (!alloc(l.uk_t, H, K, D) || !alloc(l.uv, H, V, K)) return;
    for (int h = 0; h < H; ++h) {
        put(l.uk_t, (int64_t)h * K, uk, (int64_t)h * D, K, D, true);
        put(l.uv, (int64_t)h * V, uv, (int64_t)h * V, V, K);
    }
    const int D16 = (D + 15) & ~15, V16 = (V + 15) & ~15, R16 = (R + 15) & ~15, K16 = (K + 15) & ~15;
    l.expand = !p.f32 && latent_expanded_supported(D, R, V);
    if (l.expand) {
        if (!alloc(l.kv, 1, (int64_t)H * (D16 + V16), K)) return;
        for (int h = 0; h < H; ++h) {
            put(l.kv, (int64_t)h * (D16 + V16), uk, (int64_t)h * D, D, K);
            put(l.kv, (int64_t)h * (D16 + V16) + D16, uv, (int64_t)h * V, V, K);
        }
    }
    if (!alloc(l.o, 1, W, H * V)) return;
    put(l.o, 0, need(mx + "o", W, (int64_t)H * V), 0, W, H * V);
    // the latent cache
    l.cache.rank = K;
    l.cache.rank16 = K16;
    l.cache.rot = R;
    l.cache.rot16 = R16;
    l.cache.ld = mat_kpad(K16 + R16);
    l.cache.page_table = e.kv_.page_table;
    l.cache.max_pages = e.kv_.max_pages;
    cache_slice(l.own ? (size_t)KV_PAGE * l.cache.ld * p.elem() : 0);
    if (K > 1024) { fail(SP_ERR_ARG, "latent rank above 1024 is not supported"); return; }
    l.cos_sin = angles(m.rot.base, R);
    if (mp.depth_average) l.dwa = vec(lp.prefix + "dwa", i + 2);
    PlanSizes& n = p.need;
    PlanSizes::most(n.proj, (size_t)l.proj.n);
    PlanSizes::most(n.qn, (size_t)H * l.uk_t.kp);
    PlanSizes::most(n.qabs, (size_t)H * l.cache.ld);
    PlanSizes::most(n.qf, (size_t)H * (D16 + R16));
    PlanSizes::most(n.olat, (size_t)H * l.uv.kp);
    PlanSizes::most(n.mixed, (size_t)l.o.kp);
    PlanSizes::most(n.kv, (size_t)H * (D16 + V16));
    PlanSizes::most(n.lat, (size_t)l.cache.ld);
    PlanSizes::most(n.part, (size_t)H * (K + 2));
}

void PlanPacker::experts(int i) {
    const LayerPlan& lp = p.plan.layers[(size_t)i];
    const MoeSpec& s = lp.moe;
    PlanLayer& l = p.layers[(size_t)i];
    const std::string ml = lp.prefix + "mlp.";
    const int W = p.plan.width, E = s.experts, F = s.expert.ff;
    l.norm2 = vec(lp.prefix + "norm2", 1);
    if (!alloc(l.router, 1, E + (s.has_shared ? 1 : 0), W)) return;
    put(l.router, 0, need(ml + "router", E, W), 0, E, W);
    l.router_b = vec(ml + "router.b", E);
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
        put(l.router, E, need(ml + "shared.sg", 1, W), 0, 1, W);
        PlanSizes::most(p.need.act_shared, (size_t)l.shared_down.kp);
    }
    PlanSizes::most(p.need.act, (size_t)s.top * l.down.kp);
    PlanSizes::most(p.need.pairs, (size_t)s.top);
    p.need.experts = std::max(p.need.experts, E);
}

static int plan_splits(const PlanLayer& l, bool f32, int bucket, int T) {
    if (T > PLAN_ROWS) return 1;
    int s = latent_attention_splits(l.shape.heads, T, std::min(1 << bucket, l.shape.window), f32);
    while (s > 1 && T * s > PLAN_SPLIT_ROWS) s >>= 1;
    return s;
}

// Decides how the staged tokens attend and fills the tables of the expanded form.
void Engine::plan_stage_latent(int T) {
    PlanState& p = *plan_;
    int window = 0;
    for (const PlanLayer& l : p.layers) window = std::max(window, l.shape.window);
    LatentTile* tiles = reinterpret_cast<LatentTile*>(p.host_tiles);
    int32_t *slot = p.host_tiles + p.keys_at, *pos = slot + p.keys_cap;
    int keys = 0, nt = 0;
    for (int i = 0; i < T;) {
        int n = 1;
        while (i + n < T && p_slot_[i + n] == p_slot_[i] && p_pos_[i + n] == p_pos_[i] + n) ++n;
        const int first = window > p_pos_[i] ? 0 : p_pos_[i] - window + 1, cnt = p_pos_[i] + n - first;
        if (keys + cnt > p.keys_cap || keys + cnt > 3 * T) return;  // more keys to rebuild than it saves
        for (int t = 0; t < n; t += LATENT_Q_TILE) tiles[nt++] = LatentTile{i + t, std::min(LATENT_Q_TILE, n - t), p_pos_[i] + t, keys, first};
        for (int k = 0; k < cnt; ++k) { slot[keys + k] = p_slot_[i]; pos[keys + k] = first + k; }
        keys += cnt;
        i += n;
    }
    p.n_tiles = nt;
    p.n_keys = keys;
}

int Engine::plan_latent(int li, int T) {
    PlanState& p = *plan_;
    PlanLayer& l = p.layers[(size_t)li];
    const LatentShape& s = l.shape;
    const int H = s.heads, ldp = l.proj.n;
    SP_TRY(plan_mat(l.proj, p.xb, p.wp, T, p.proj, ldp, true));
    const bool expanded = p.n_tiles > 0 && T > PLAN_ROWS && l.expand && !graph_step_;
    const float* gate = p.proj + l.gate_col;
    SP_LAUNCH(F_ROPE, launch_latent_append(p.proj, ldp, s, l.cache, l.own, l.dkv_norm, p.plan.eps, l.cos_sin, d_tok_slot_, d_tok_pos_,
                                           expanded ? nullptr : p.qn, l.uk_t.kp, p.qabs, p.qf, p.f32, T, stream));
    if (expanded) {
        const int32_t* keys = p.dev_tiles + p.keys_at;
        SP_LAUNCH(F_ATTN, launch_latent_gather(l.cache, keys, keys + p.keys_cap, p.n_keys, p.lat, stream));
        SP_TRY(plan_mat(l.kv, p.lat, l.cache.ld, p.n_keys, p.kvx, l.kv.n, false));
        SP_LAUNCH(F_ATTN, launch_latent_expanded(p.qf, p.kvx, p.lat, s, l.cache, (const LatentTile*)p.dev_tiles, p.n_tiles, gate, ldp, p.attn, l.o.kp, stream));
    } else {
        MatArgs a{};
        a.f32 = p.f32;
        a.nseg = 1;
        a.m = T;
        a.seg[0] = MatSeg{l.uk_t.w, l.uk_t.n, l.uk_t.kp, H, 0.f, 0.f, p.qn, H * l.uk_t.kp, l.uk_t.kp, p.qabs, H * l.cache.ld, l.cache.ld};
        SP_TRY(plan_product(a, 0));
        SP_LAUNCH(F_ATTN, launch_latent_attention(p.qabs, s, l.cache, d_tok_slot_, d_tok_pos_, p.olat, l.uv.kp, p.part,
                                                  plan_splits(l, p.f32, plan_ctx_bucket(), T), p.f32, T, stream));
        a.seg[0] = MatSeg{l.uv.w, l.uv.n, l.uv.kp, H, 0.f, 0.f, p.olat, H * l.uv.kp, l.uv.kp, p.attn, l.o.kp, s.vdim};
        a.gate = gate;
        a.ldgate = ldp;
        SP_TRY(plan_product(a, 0));
    }
    return plan_mat(l.o, p.attn, l.o.kp, T, p.y, p.plan.width, true);
}

int Engine::plan_experts(int li, int T) {
    PlanState& p = *plan_;
    PlanLayer& l = p.layers[(size_t)li];
    const MoeSpec& s = p.plan.layers[(size_t)li].moe;
    const int W = p.plan.width, E = s.experts, pairs = T * s.top;
    SP_TRY(plan_mat(l.router, p.xb, p.wp, T, p.logit, l.router.n, true));
    SP_LAUNCH(F_ELEM, launch_moe_route(p.logit, l.router.n, l.router_b, T, E, s.top, p.pick, p.weight, p.moe, stream));
    MatArgs a{};
    a.f32 = p.f32;
    a.m = T;
    a.dual = true;
    a.moe = true;
    a.rows = MoeRows{p.moe.row_off, p.moe.row_src, p.moe.active, p.moe.n_active, p.moe.tile_group, p.moe.tile_row, p.moe.n_tiles};
    a.slots = std::min(E, pairs);
    const MatSeg gu{l.gu.w, s.expert.ff, l.gu.kp, E, s.expert.limit, s.expert.alpha, p.xb, p.wp, 0, p.act, l.down.kp, 0};
    const MatSeg sgu{l.shared_gu.w, s.shared.ff, l.shared_gu.kp, 1, s.shared.limit, s.shared.alpha, p.xb, p.wp, 0, p.act_shared, l.shared_down.kp, 0};
    const MatSeg dn{l.down.w, W, l.down.kp, E, 0.f, 0.f, p.act, l.down.kp, 0, p.y_expert, W, 0};
    const MatSeg sdn{l.shared_down.w, W, l.shared_down.kp, 1, 0.f, 0.f, p.act_shared, l.shared_down.kp, 0, p.y_shared, W, 0};
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

int Engine::plan_layer_post_norm(int i, int T) {
    PlanState& p = *plan_;
    const int W = p.plan.width;
    PlanLayer& l = p.layers[(size_t)i];
    const LayerPlan& lp = p.plan.layers[(size_t)i];
    SP_TRY(plan_latent(i, T));
    SP_LAUNCH(F_NORM, launch_norm_residual(p.y, W, l.norm1, p.plan.eps, i == 0 ? p.history : x_, x_, p.xb, p.wp, p.f32, T, W, stream));
    CombineArgs c{};
    if (lp.mlp == MLP_MOE) {
        SP_TRY(plan_experts(i, T));
        c.y = p.y_expert;
        c.ldy = W;
        c.slot_of = p.moe.slot_of;
        c.weight = p.weight;
        c.top = lp.moe.top;
        if (lp.moe.has_shared) {
            c.y_shared = p.y_shared;
            c.shared_gate = p.logit + lp.moe.experts;
            c.ld_gate = l.router.n;
        }
        c.gain = l.norm2;
        c.eps = p.plan.eps;
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
