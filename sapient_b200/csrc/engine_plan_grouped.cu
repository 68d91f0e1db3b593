// Grouped attention of plan layers, in either form: what its projections are, its share of the cache, its tables by position
// and by distance, and the two launches behind the projection — what happens to queries, keys and values on the way into the
// cache, and the attention itself.
#include <cmath>

#include "engine_plan.h"
#include "sp_common.cuh"

namespace sp {

// Row of the bias table for a distance: one per distance up to half of the rows, then logarithmic up to `far`.
static int distance_bucket(int distance, int rows, int far) {
    const int half = rows / 2;
    if (distance < half) return distance;
    const double step = std::log((double)distance / half) / std::log((double)far / half) * (rows - half);
    return step >= rows - half ? rows - 1 : std::min(rows - 1, half + (int)std::floor(step));
}

// The layer's bias table [rows][heads] by head and distance, up to the first distance of the last row.
const float* PlanPacker::distance_bias(const std::string& name, int heads, int far, int* n_rel) {
    const int rows = (int)rows_of(name);
    if (status != SP_OK) return nullptr;
    if (rows < 2 || far <= rows / 2) { fail(SP_ERR_SHAPE, "bias_max does not fit the rows of '" + name + "'"); return nullptr; }
    const std::vector<float> table = host(name, rows, heads);
    if (table.empty()) return nullptr;
    int n = 0;
    while (distance_bucket(n, rows, far) < rows - 1) ++n;
    *n_rel = ++n;
    std::vector<float> rel((size_t)heads * n);
    for (int i = 0; i < n; ++i)
        for (int h = 0; h < heads; ++h) rel[(size_t)h * n + i] = table[(size_t)distance_bucket(i, rows, far) * heads + h];
    return upload(rel);
}

int PlanPacker::grouped_mixer(int i, std::vector<MixPart>& all_parts) {
    const LayerPlan& lp = p.plan.layers[(size_t)i];
    const GroupedAttentionSpec& m = lp.grouped;
    PlanLayer& l = p.layers[(size_t)i];
    const std::string mx = lp.prefix + m.at;
    const int H = m.heads, G = m.kv_heads, out_cols = H * m.vdim;
    p.has_grouped = true;
    l.grouped = GroupedShape{H, G, m.dim, m.vdim, m.rot.dims, m.window, m.scale, m.rot.neighbours, m.keep_first, m.score_softcap};
    l.mixed = m.talk || m.keep_first > 0 || m.score_softcap > 0 || m.out_scale != 1.f;
    if (m.vdim > GROUPED_MAX_VDIM) { fail(SP_ERR_ARG, "attention values above " + std::to_string(GROUPED_MAX_VDIM) + " coordinates are not supported"); return 0; }
    if (m.shared_values && (m.rot.dims || m.rotate_values || m.vdim != m.dim || m.conv)) { fail(SP_ERR_ARG, "keys that are the values cannot be rotated or convolved"); return 0; }
    if (m.conv && (m.qk_norm != QK_NONE || m.temperature.coef != 0.0 || m.rotate_values)) {
        fail(SP_ERR_ARG, "convolutions do not go with norms or temperatures of queries and keys, or with rotated values");
        return 0;
    }
    if (l.mixed && (m.shared_values || m.rotate_values || m.bias_max > 0 || m.out_gate)) {
        fail(SP_ERR_ARG, "mixed heads, kept first keys and capped scores do not go with distance biases, output gates or values that are rotated or the keys");
        return 0;
    }
    std::vector<MixPart> parts = {{m.at + "q", H * m.dim}, {m.at + "k", G * m.dim}};
    if (!m.shared_values) parts.push_back({m.at + "v", G * m.vdim});
    for (const MixPart& part : all_parts) l.grouped_col += part.rows;
    const int dim16 = (m.dim + 15) & ~15, vdim16 = (m.vdim + 15) & ~15;
    l.kv_cache = GroupedCache{nullptr, e.kv_.page_table, e.kv_.max_pages, dim16, vdim16, m.shared_values ? dim16 + GROUPED_TAIL : dim16 + vdim16, m.shared_values};
    cache_slice((size_t)G * KV_PAGE * l.kv_cache.ld * p.elem());
    PlanSizes::most(p.need.q, (size_t)H * dim16);
    GroupedInput& in = l.grouped_in;
    GroupedTerms& x = l.grouped_terms;
    in.cs_key = angles(m.rot);
    if (m.rotate_values) in.cs_val = x.cs_val = angles(m.rot.base, m.vdim);
    if (m.biases) {
        std::vector<float> all;
        for (const MixPart& part : parts) {
            const std::vector<float> b = host(lp.prefix + part.name + ".b", 1, part.rows);
            all.insert(all.end(), b.begin(), b.end());
        }
        if (status != SP_OK) return 0;
        in.bias = upload(all);
    }
    if (m.conv > 0) {
        std::vector<float> all;
        size_t channels = 0;
        for (const MixPart& part : parts) {
            const std::vector<float> w = host(lp.prefix + part.name + ".conv", part.rows, m.conv);
            all.insert(all.end(), w.begin(), w.end());
            channels += (size_t)part.rows;
        }
        if (status != SP_OK) return 0;
        std::vector<float> by_tap(all.size());
        for (size_t ch = 0; ch < channels; ++ch)
            for (int j = 0; j < m.conv; ++j) by_tap[(size_t)j * channels + ch] = all[ch * (size_t)m.conv + j];
        in.conv = upload(by_tap);
        in.taps = m.conv;
        l.tail_at = slot_floats((size_t)(m.conv - 1) * channels);
        p.has_conv = true;
    }
    in.norm = m.qk_norm != QK_NONE;
    in.eps = p.plan.eps;
    if (m.qk_norm == QK_WEIGHTED) {
        std::vector<float> q = host(mx + "q.norm", 1, m.dim), k = host(mx + "k.norm", 1, m.dim);
        if (status != SP_OK) return 0;
        if (m.shared_values) {  // the cache keeps keys without the weight
            for (int c = 0; c < m.dim; ++c) q[(size_t)c] *= k[(size_t)c];
        } else {
            in.k_gain = upload(k);
        }
        in.q_gain = upload(q);
    }
    if (m.temperature.coef != 0.0) {
        std::vector<float> t((size_t)e.d.max_ctx);
        for (size_t pos = 0; pos < t.size(); ++pos)
            t[pos] = (float)(1.0 + m.temperature.coef * std::log(std::floor((double)(pos + 1) / m.temperature.every) + 1.0));
        in.temperature = upload(t);
    }
    if (m.bias_max > 0) x.rel = distance_bias(mx + "rel", H, m.bias_max, &x.n_rel);
    if (m.sink) x.sink = vec(mx + "sink", H);
    if (l.mixed) {
        std::vector<float> mix((size_t)H * H, 0.f);
        if (m.talk) mix = host(mx + "talk", H, H);
        else
            for (int h = 0; h < H; ++h) mix[(size_t)h * H + h] = 1.f;
        for (float& v : mix) v *= m.out_scale;
        l.mixed_terms = MixedTerms{upload(mix), x.sink};
        l.mixed_span = mixed_span(l.grouped, e.d.max_ctx);
        // scores of a decode-shaped step, or (plain arithmetic) of as many rows as a quarter of a gigabyte holds
        const size_t row = (size_t)H * l.mixed_span;
        const bool plain = p.f32 || !mixed_mma_supported(l.grouped, l.kv_cache);
        l.mixed_rows = plain ? (int)std::max<size_t>(1, std::min<size_t>((size_t)e.d.max_tokens, ((size_t)1 << 26) / row)) : std::min(PLAN_ROWS, e.d.max_tokens);
        PlanSizes::most(p.need.score, row * (size_t)l.mixed_rows);
        PlanSizes::most(p.need.stat, (size_t)H);
        p.has_mixed = true;
    }
    if (m.out_gate) {
        for (const MixPart& part : parts) l.gate_col += part.rows;
        l.gate_col += l.grouped_col;
        parts.push_back({m.at + "g", out_cols});
    }
    all_parts.insert(all_parts.end(), parts.begin(), parts.end());
    return out_cols;
}

// From p.proj (rows of mix_rows) to p.attn.
int Engine::plan_grouped(int li, int T) {
    PlanState& p = *plan_;
    PlanLayer& l = p.layers[(size_t)li];
    const GroupedShape& s = l.grouped;
    GroupedTerms x = l.grouped_terms;
    if (l.gate_col) {
        x.gate = p.proj + l.gate_col;
        x.ldgate = l.mix_rows;
    }
    const float* proj = p.proj + l.grouped_col;
    GroupedInput in = l.grouped_in;
    if (in.conv) {
        in.tail = p.states + l.tail_at;
        in.tail_stride = (int64_t)p.slot_state;
        in.back = T > PLAN_ROWS ? p.dev_tiles + p.back_at : nullptr;
    }
    if (in.conv) {
        const GroupedTile* tiles = in.back ? (const GroupedTile*)(p.dev_tiles + p.narrow_at) : nullptr;
        SP_LAUNCH(F_ROPE, launch_conv_append(proj, l.mix_rows, s, l.kv_cache, in, tiles, p.n_narrow, d_tok_slot_, d_tok_pos_, p.q, p.f32, T, stream));
        if (in.back) SP_LAUNCH(F_ROPE, launch_conv_tails(proj, l.mix_rows, s, in, d_tok_slot_, p.dev_tiles + p.ends_at, p.n_ends, stream));
    } else {
        SP_LAUNCH(F_ROPE, launch_grouped_append(proj, l.mix_rows, s, l.kv_cache, in, d_tok_slot_, d_tok_pos_, p.q, p.f32, T, stream));
    }
    if (l.mixed) {
        const MixedScratch m{p.score, l.mixed_rows, l.mixed_span, p.score_part, p.stat, (float*)p.stat};  // (a step uses one of the last two)
        if (p.n_grouped > 0 && T > PLAN_ROWS && !graph_step_ && mixed_mma_supported(s, l.kv_cache)) {
            SP_LAUNCH(F_ATTN, launch_mixed_prefill(p.q, s, l.kv_cache, l.mixed_terms, m, (const GroupedTile*)(p.dev_tiles + p.grouped_at), p.n_grouped,
                                                   (const GroupedTile*)(p.dev_tiles + p.narrow_at), p.n_narrow, p.attn, l.o.kp, stream));
            return SP_OK;
        }
        const int splits = T > PLAN_ROWS ? 1 : mixed_attention_splits(s, T, std::min(1 << plan_ctx_bucket(), l.mixed_span));
        SP_LAUNCH(F_ATTN, launch_mixed_attention(p.q, s, l.kv_cache, l.mixed_terms, m, d_tok_slot_, d_tok_pos_, p.attn, l.o.kp, splits, p.f32, T, stream));
        return SP_OK;
    }
    if (p.n_grouped > 0 && T > PLAN_ROWS && !graph_step_ && grouped_mma_supported(s)) {
        SP_LAUNCH(F_ATTN, launch_grouped_prefill(p.q, s, l.kv_cache, x, (const GroupedTile*)(p.dev_tiles + p.grouped_at), p.n_grouped, p.attn, l.o.kp, stream));
        return SP_OK;
    }
    const int splits = T > PLAN_ROWS ? 1 : grouped_attention_splits(s, T, std::min(1 << plan_ctx_bucket(), s.window), p.f32);
    SP_LAUNCH(F_ATTN, launch_grouped_attention(p.q, s, l.kv_cache, x, d_tok_slot_, d_tok_pos_, p.attn, l.o.kp, splits, p.f32, T, stream));
    return SP_OK;
}

}  // namespace sp
