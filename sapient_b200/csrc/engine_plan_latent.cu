// Latent attention of plan layers: projections, rotation + cache append, then either queries to latent space, absorbed
// attention and value maps or gather, rebuilt keys and values and expanded attention; output projection. Steps of up to
// PLAN_ROWS rows take the absorbed attention; longer ones, where rebuilding the keys pays, the expanded attention.
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
        a.seg[0] = MatSeg{l.uk_t.w, l.uk_t.n, l.uk_t.kp, H, MatUnit{}, p.qn, H * l.uk_t.kp, l.uk_t.kp, p.qabs, H * l.cache.ld, l.cache.ld};
        SP_TRY(plan_product(a, 0));
        SP_LAUNCH(F_ATTN, launch_latent_attention(p.qabs, s, l.cache, d_tok_slot_, d_tok_pos_, p.olat, l.uv.kp, p.part,
                                                  plan_splits(l, p.f32, plan_ctx_bucket(), T), p.f32, T, stream));
        a.seg[0] = MatSeg{l.uv.w, l.uv.n, l.uv.kp, H, MatUnit{}, p.olat, H * l.uv.kp, l.uv.kp, p.attn, l.o.kp, s.vdim};
        a.gate = gate;
        a.ldgate = ldp;
        SP_TRY(plan_product(a, 0));
    }
    return SP_OK;
}

}  // namespace sp
