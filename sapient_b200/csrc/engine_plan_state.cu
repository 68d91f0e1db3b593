// Mixers of plan layers, whatever the layer form: state mixers — their projections, their share of a slot's states and the launches
// behind the projection — and what grouped attention and state mixers have in common when a layer has either or both side by side.
#include "engine_plan.h"

#include "sp_common.cuh"

namespace sp {

size_t PlanPacker::slot_floats(size_t n) {
    const size_t at = p.slot_state;
    p.slot_state += (n + 3) / 4 * 4;  // vectors of four
    return at;
}

int PlanPacker::state_mixer(int i, std::vector<MixPart>& parts) {
    const LayerPlan& lp = p.plan.layers[(size_t)i];
    const StateMixerSpec& m = lp.state;
    PlanLayer& l = p.layers[(size_t)i];
    PlanSizes& n = p.need;
    const std::string mx = lp.prefix + m.at;
    const int H = m.heads, hd = H * m.dim, hv = H * m.vdim;
    p.has_state = true;
    l.state_shape = StateShape{H, m.dim, m.vdim, m.rule, state_dim_pad(m.dim), p.plan.eps, m.norm_all, m.gate, m.rot.dims, m.key_scale};
    l.state_at = slot_floats((size_t)hv * l.state_shape.dim_pad);
    auto part = [&](const char* name, int rows) { parts.push_back({m.at + name, rows}); };
    if (m.rule == STATE_DELTA) {
        l.low_rows = (int)rows_of(mx + "w1");
        if (status != SP_OK) return 0;
        part("r", hd);
        part("k", hd);
        part("v", hv);
        part("a", hd);
        l.a_bias = vec(mx + "a.b", hd);
        l.w0 = vec(mx + "w0", hd);
        if (!alloc(l.w2, 1, hd, l.low_rows)) return 0;
        put(l.w2, 0, need(mx + "w2", hd, l.low_rows), 0, hd, l.low_rows);
        PlanSizes::most(n.low, (size_t)l.w2.kp);
        PlanSizes::most(n.wlogit, (size_t)hd);
    } else if (m.rule == STATE_FORGET) {
        part("q", hd);
        part("f", hd);
        part("v", hv);
        l.silu_rows = hd;
        l.a_bias = vec(mx + "f.b", hd);
        l.lower = vec(mx + "lower", hd);
    } else {
        part("q", hd);
        part("k", hd);
        part("v", hv);
        if (m.silu_inputs) l.silu_rows = 2 * hd + hv;
        l.decay = upload(m.decay);
        l.cos_sin = angles(m.rot);
    }
    if (m.gate != STATE_GATE_NONE) part("g", hv);
    if (m.gain == STATE_GAIN_COORD && m.out_scale == 1.f) {
        l.gain = vec(mx + "norm", hv);
    } else if (m.gain != STATE_GAIN_NONE || m.out_scale != 1.f) {
        std::vector<float> g(1, 1.f);
        if (m.gain != STATE_GAIN_NONE) g = host(mx + "norm", 1, m.gain == STATE_GAIN_COORD ? hv : m.vdim);
        if (status != SP_OK) return 0;
        std::vector<float> all((size_t)hv);
        for (int c = 0; c < hv; ++c) all[(size_t)c] = g[(size_t)c % g.size()] * m.out_scale;
        l.gain = upload(all);
    }
    PlanSizes::most(n.state_rec, state_record_floats(l.state_shape, p.f32));
    return hv;
}

// State mixers come first: the rows of a projection that go through silu are its first ones.
int PlanPacker::mixers(int i, std::vector<MixPart>& parts) {
    const LayerPlan& lp = p.plan.layers[(size_t)i];
    PlanLayer& l = p.layers[(size_t)i];
    const int state_cols = lp.has_state() ? state_mixer(i, parts) : 0;
    if (lp.has_grouped()) l.state_col = grouped_mixer(i, parts);
    else cache_slice(0);
    if (status != SP_OK) return 0;
    for (const MixPart& part : parts) l.mix_rows += part.rows;
    PlanSizes::most(p.need.proj, (size_t)l.mix_rows);
    return l.state_col + state_cols;
}

void PlanPacker::put_mixer_rows(int i, const std::vector<MixPart>& parts) {
    const LayerPlan& lp = p.plan.layers[(size_t)i];
    PlanLayer& l = p.layers[(size_t)i];
    const int W = p.plan.width;
    int at = 0;
    for (const MixPart& part : parts) {
        put(l.proj, at, need(lp.prefix + part.name, part.rows, W), 0, part.rows, W);
        at += part.rows;
    }
    if (l.low_rows) put(l.proj, at, need(lp.prefix + lp.state.at + "w1", l.low_rows, W), 0, l.low_rows, W);
}

void PlanPacker::put_mixer_out(int i) {
    const LayerPlan& lp = p.plan.layers[(size_t)i];
    PlanLayer& l = p.layers[(size_t)i];
    const int W = p.plan.width;
    if (lp.has_grouped()) put(l.o, 0, need(lp.prefix + lp.grouped.at + "o", W, l.state_col), 0, W, l.state_col);
    if (lp.has_state()) {
        const int cols = lp.state.heads * lp.state.vdim;
        put(l.o, 0, need(lp.prefix + lp.state.at + "o", W, cols), 0, W, cols, false, l.state_col);
    }
    PlanSizes::most(p.need.mixed, (size_t)l.o.kp);
}

// The product that reads the mixer's input p.xb: f32 rows to p.proj, low-rank rows to p.low; a.outs may hold one more range.
int Engine::plan_mixer_in(int i, int T, MatArgs& a) {
    PlanState& p = *plan_;
    PlanLayer& l = p.layers[(size_t)i];
    const MatOut more = a.outs[0];
    const bool has_more = a.n_outs > 0;
    a.n_outs = 0;
    a.f32 = p.f32;
    a.nseg = 1;
    a.m = T;
    a.seg[0] = MatSeg{l.proj.w, l.proj.n, l.proj.kp, 1, MatUnit{}, p.xb, p.wp, 0, nullptr, 0, 0};
    int at = 0;
    auto rows_to = [&](int rows, void* y, int64_t ld, MatAct act, bool f32) {
        if (rows) a.outs[a.n_outs++] = MatOut{at += rows, y, ld, act, f32, false};
    };
    rows_to(l.silu_rows, p.proj, l.mix_rows, MAT_SILU, true);
    rows_to(l.mix_rows - l.silu_rows, p.proj + l.silu_rows, l.mix_rows, MAT_ID, true);
    rows_to(l.low_rows, p.low, l.w2.kp, MAT_TANH, p.f32);
    if (has_more) a.outs[a.n_outs++] = more;
    return plan_product(a, 0);
}

// From p.proj to p.attn.
int Engine::plan_mixers(int i, int T) {
    const LayerPlan& lp = plan_->plan.layers[(size_t)i];
    if (lp.has_grouped()) SP_TRY(plan_grouped(i, T));
    return lp.has_state() ? plan_state(i, T) : SP_OK;
}

int Engine::plan_state(int li, int T) {
    PlanState& p = *plan_;
    PlanLayer& l = p.layers[(size_t)li];
    StateArgs a{};
    a.s = l.state_shape;
    a.state = p.states + l.state_at;
    a.slot_stride = (int64_t)p.slot_state;
    a.decay = l.decay;
    a.proj = p.proj;
    a.ldp = l.mix_rows;
    a.a_bias = l.a_bias;
    a.lower = l.lower;
    a.cs = l.cos_sin;
    a.w0 = l.w0;
    a.w2 = l.w2.w;
    a.low = p.low;
    a.ldlow = l.w2.kp;
    a.wlogit = p.wlogit;
    a.rec = p.state_rec;
    a.gain = l.gain;
    a.tok_slot = d_tok_slot_;
    a.tok_pos = d_tok_pos_;
    a.out = (uint8_t*)p.attn + (size_t)l.state_col * p.elem();
    a.ldo = l.o.kp;
    a.f32 = p.f32;
    if (T <= PLAN_ROWS) {
        SP_LAUNCH(F_STATE, launch_state_step(a, T, stream));
        return SP_OK;
    }
    if (l.low_rows) SP_TRY(plan_mat(l.w2, p.low, l.w2.kp, T, p.wlogit, l.w2.n, true));
    SP_LAUNCH(F_STATE, launch_state_scan(a, (const StateSegment*)(p.dev_tiles + p.seg_at), p.n_seg, p.dev_tiles + p.groups_at, p.n_groups, stream));
    return SP_OK;
}

}  // namespace sp
