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
    PlanSizes& n = p.need;
    const std::string mx = lp.prefix + "mix.", ml = lp.prefix + "mlp.";
    const int W = p.plan.width;
    l.norm1 = gain(lp.prefix + "norm1");
    l.ff = lp.mlp == MLP_DENSE ? lp.dense.ff : 0;
    std::vector<MixPart> parts;
    int out_cols = 0;
    if (lp.mixer == MIX_GROUPED) {
        grouped_mixer(i, parts, &out_cols);
        if (status != SP_OK) return;
    } else {
        const StateMixerSpec& m = lp.state;
        const int H = m.heads, hd = H * m.dim, hv = H * m.vdim;
        p.has_state = true;
        l.state_shape = StateShape{H, m.dim, m.vdim, m.rule, state_dim_pad(m.dim), p.plan.eps};
        l.state_at = p.slot_state;
        p.slot_state += (size_t)hv * l.state_shape.dim_pad;
        out_cols = hv;
        l.gain = vec(mx + "norm", hv);
        if (m.rule == STATE_DELTA) {
            l.low_rows = (int)rows_of(mx + "w1");
            if (status != SP_OK) return;
            parts = {{"r", hd}, {"k", hd}, {"v", hv}, {"a", hd}, {"g", hv}};
            l.a_bias = vec(mx + "a.b", hd);
            l.w0 = vec(mx + "w0", hd);
            if (!alloc(l.w2, 1, hd, l.low_rows)) return;
            put(l.w2, 0, need(mx + "w2", hd, l.low_rows), 0, hd, l.low_rows);
            PlanSizes::most(n.low, (size_t)l.w2.kp);
            PlanSizes::most(n.wlogit, (size_t)hd);
        } else {
            parts = {{"q", hd}, {"k", hd}, {"v", hv}, {"g", hv}};
            l.silu_rows = 2 * hd + hv;
            void* q = nullptr;
            if (cudaMalloc(&q, (size_t)H * 4) != cudaSuccess) { fail(SP_ERR_OOM, "cannot allocate the decays"); return; }
            p.owned.push_back(q);
            if (cudaMemcpy(q, m.decay.data(), (size_t)H * 4, cudaMemcpyHostToDevice) != cudaSuccess) { fail(SP_ERR_CUDA, "cudaMemcpy failed"); return; }
            l.decay = (const float*)q;
        }
        PlanSizes::most(n.state_rec, state_record_floats(l.state_shape, p.f32));
        cache_slice(0);
    }
    for (const MixPart& part : parts) l.mix_rows += part.rows;
    if (!alloc(l.proj, 1, (int64_t)l.mix_rows + l.low_rows + l.ff, W)) return;
    int at = 0;
    for (const MixPart& part : parts) {
        put(l.proj, at, need(mx + part.name, part.rows, W), 0, part.rows, W);
        at += part.rows;
    }
    if (l.low_rows) put(l.proj, at, need(mx + "w1", l.low_rows, W), 0, l.low_rows, W);
    if (l.ff) put(l.proj, at + l.low_rows, need(ml + "up", l.ff, W), 0, l.ff, W);
    l.act_col = l.ff ? (out_cols + 7) & ~7 : out_cols;
    if (!alloc(l.o, 1, W, l.act_col + l.ff)) return;
    put(l.o, 0, need(mx + "o", W, out_cols), 0, W, out_cols);
    if (l.ff) put(l.o, 0, need(ml + "down", W, l.ff), 0, W, l.ff, false, l.act_col);
    PlanSizes::most(n.proj, (size_t)l.mix_rows);
    PlanSizes::most(n.mixed, (size_t)l.o.kp);
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
    a.w0 = l.w0;
    a.w2 = l.w2.w;
    a.low = p.low;
    a.ldlow = l.w2.kp;
    a.wlogit = p.wlogit;
    a.rec = p.state_rec;
    a.gain = l.gain;
    a.tok_slot = d_tok_slot_;
    a.tok_pos = d_tok_pos_;
    a.out = p.attn;
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

int Engine::plan_layer_parallel(int i, int T) {
    PlanState& p = *plan_;
    PlanLayer& l = p.layers[(size_t)i];
    const int W = p.plan.width;
    SP_LAUNCH(F_NORM, launch_row_norm(x_, nullptr, T, W, l.norm1, p.plan.eps, p.xb, p.wp, p.f32, stream));
    MatArgs a{};
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
    rows_to(l.ff, (uint8_t*)p.attn + (size_t)l.act_col * p.elem(), l.o.kp, MAT_RELU2, p.f32);
    SP_TRY(plan_product(a, 0));
    SP_TRY(p.plan.layers[(size_t)i].mixer == MIX_GROUPED ? plan_grouped(i, T) : plan_state(i, T));
    a.n_outs = 1;
    a.seg[0] = MatSeg{l.o.w, W, l.o.kp, 1, MatUnit{}, p.attn, l.o.kp, 0, nullptr, 0, 0};
    a.outs[0] = MatOut{W, x_, W, MAT_ID, true, true};
    return plan_product(a, 0);
}

}  // namespace sp
