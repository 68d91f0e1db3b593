// Plan-driven models (model_plan.h) on the resident engine: what every plan shares — weights packed once into the shapes
// the kernels read, a paged cache behind the same page pool, state pools, the buffers and tables of a step, the output head.
// The layers themselves are in engine_plan_post_norm.cu, engine_plan_parallel.cu and engine_plan_pre_norm.cu. bf16 products run on the tcgen05 kernel
// (mat_tc5.cu) at every row count, f32 ones on mat_f32.cu. Steps of up to PLAN_ROWS rows can be captured as a graph.
#include "engine_plan.h"

#include <cmath>
#include <cstring>

#include "plan_common.cuh"
#include "sp_common.cuh"

namespace sp {

namespace {

__device__ __forceinline__ float load_elem(int dtype, const uint8_t* p, int64_t i) {
    if (dtype == T_F32) return reinterpret_cast<const float*>(p)[i];
    if (dtype == T_BF16) return __bfloat162float(reinterpret_cast<const bf16*>(p)[i]);
    return __half2float(reinterpret_cast<const __half*>(p)[i]);
}

// dst[r][c0 .. c0 + k) = src[r][0 .. k) (or src[0 .. k)[r] transposed, source row stride lds); dst rows are kp long.
template <typename T>
__global__ void pack_rows_kernel(int dtype, const uint8_t* __restrict__ src, int64_t lds, bool transpose, int k, int kp, int c0, T* __restrict__ dst) {
    const int64_t r = blockIdx.x;
    for (int c = threadIdx.x; c < k; c += blockDim.x) dst[r * kp + c0 + c] = from_f32<T>(load_elem(dtype, src, transpose ? (int64_t)c * lds + r : r * lds + c));
}

size_t esize(int dtype) { return dtype == T_F32 ? 4 : 2; }

}  // namespace

bool PlanPacker::fail(int st, const std::string& msg) {
    if (status == SP_OK) { set_error(msg); status = st; }
    return false;
}

const DevTensor* PlanPacker::need(const std::string& name, int64_t rows, int64_t cols) {
    const DevTensor* t = e.find(name);
    if (!t) { fail(SP_ERR_STATE, "missing weight '" + name + "'"); return nullptr; }
    const int64_t r = t->dims.size() == 2 ? t->dims[0] : 1, c = t->dims.back();
    if (r * c != rows * cols || (cols > 1 && c != cols) || (t->dtype != T_F32 && t->dtype != T_BF16 && t->dtype != T_F16)) {
        fail(SP_ERR_SHAPE, "shape or dtype mismatch for '" + name + "'");
        return nullptr;
    }
    return t;
}

const float* PlanPacker::vec(const std::string& name, int64_t n) {
    if (!need(name, 1, n)) return nullptr;
    const float* f = e.find_f32(name, n);
    if (!f) fail(SP_ERR_OOM, "cannot convert '" + name + "'");
    return f;
}

RowGain PlanPacker::gain(const std::string& name) {
    const int W = p.plan.width;
    if (p.plan.norm_gain == GAIN_SCALAR) return RowGain{vec(name, 1), false};
    if (p.plan.norm_gain == GAIN_COORD) return RowGain{vec(name, W), true};
    std::vector<float> g = host(name, 1, W);
    for (float& v : g) v += 1.f;
    return RowGain{upload(g), true};
}

TanhNorm PlanPacker::tanh_norm(const std::string& name) {
    const std::vector<float> alpha = host(name + ".alpha", 1, 1);
    return TanhNorm{alpha.empty() ? 0.f : alpha[0], vec(name, p.plan.width), vec(name + ".b", p.plan.width)};
}

std::vector<float> PlanPacker::host(const std::string& name, int64_t rows, int64_t cols) {
    const DevTensor* t = need(name, rows, cols);
    const int64_t n = rows * cols;
    float* f = nullptr;
    std::vector<float> out;
    if (!t) return out;
    if (t->dtype != T_F32 && cudaMalloc((void**)&f, (size_t)n * 4) != cudaSuccess) { fail(SP_ERR_OOM, "cannot convert '" + name + "'"); return out; }
    out.resize((size_t)n);
    if ((f && launch_dequant(t->dtype, t->d, 1, n, f, 0) != cudaSuccess) ||
        cudaMemcpy(out.data(), f ? f : (const float*)t->d, (size_t)n * 4, cudaMemcpyDeviceToHost) != cudaSuccess) {
        fail(SP_ERR_CUDA, "cannot convert '" + name + "'");
        out.clear();
    }
    if (f) cudaFree(f);
    return out;
}

const float* PlanPacker::upload(const std::vector<float>& v) {
    void* q = nullptr;
    if (v.empty()) return nullptr;
    if (cudaMalloc(&q, v.size() * 4) != cudaSuccess) { fail(SP_ERR_OOM, "cannot allocate a table"); return nullptr; }
    p.owned.push_back(q);
    if (cudaMemcpy(q, v.data(), v.size() * 4, cudaMemcpyHostToDevice) != cudaSuccess) { fail(SP_ERR_CUDA, "cudaMemcpy failed"); return nullptr; }
    return (const float*)q;
}

bool PlanPacker::alloc(PlanMat& m, int groups, int64_t rows, int k) {
    m.groups = groups;
    m.n = (int)rows;
    m.kp = mat_kpad(k);
    const size_t bytes = (size_t)groups * rows * m.kp * p.elem();
    if (cudaMalloc(&m.w, bytes) != cudaSuccess) return fail(SP_ERR_OOM, "cannot allocate packed weights");
    p.owned.push_back(m.w);
    if (cudaMemset(m.w, 0, bytes) != cudaSuccess) return fail(SP_ERR_CUDA, "cudaMemset failed");
    e.weight_bytes += bytes;
    return true;
}

bool PlanPacker::put(PlanMat& m, int64_t to, const DevTensor* t, int64_t r0, int64_t rows, int k, bool transpose, int c0) {
    if (!t || !m.w) return false;
    const int64_t lds = t->dims.back();
    const uint8_t* src = t->d + (size_t)(r0 * lds) * esize(t->dtype);
    uint8_t* dst = (uint8_t*)m.w + (size_t)to * m.kp * p.elem();
    if (p.f32) pack_rows_kernel<float><<<(unsigned)rows, 128>>>(t->dtype, src, lds, transpose, k, m.kp, c0, (float*)dst);
    else pack_rows_kernel<bf16><<<(unsigned)rows, 128>>>(t->dtype, src, lds, transpose, k, m.kp, c0, (bf16*)dst);
    if (cudaGetLastError() != cudaSuccess) return fail(SP_ERR_CUDA, "pack_rows_kernel failed");
    return true;
}

int64_t PlanPacker::rows_of(const std::string& name) {
    const DevTensor* t = e.find(name);
    if (!t || t->dims.size() != 2) { fail(t ? SP_ERR_SHAPE : SP_ERR_STATE, (t ? "shape mismatch for '" : "missing weight '") + name + "'"); return 0; }
    return t->dims[0];
}

const float2* PlanPacker::angles(const RotarySpec& rot) {
    const int dims = rot.dims;
    if (dims == 0) return nullptr;
    const float2*& tab = p.angles[{rot.base, (double)dims, rot.factor, rot.original, rot.fast, rot.slow}];
    if (tab) return tab;
    const int half = dims / 2, ctx = e.d.max_ctx;
    const bool stretched = rot.factor > 0;
    double lo = 0, hi = 0, grow = 1;
    if (stretched) {
        // the pair that turns this often within the original length
        auto pair = [&](double turns) { return dims * std::log(rot.original / (2 * 3.14159265358979323846 * turns)) / (2 * std::log(rot.base)); };
        lo = std::max(std::floor(pair(rot.fast)), 0.0);
        hi = std::min(std::ceil(pair(rot.slow)), dims - 1.0);
        grow = 0.1 * std::log(rot.factor) + 1.0;
    }
    std::vector<float2> cs((size_t)ctx * half);
    for (int i = 0; i < half; ++i) {
        double f = std::pow(rot.base, -2.0 * i / dims);
        if (stretched) {
            const double ramp = std::min(std::max((i - lo) / std::max(hi - lo, 0.001), 0.0), 1.0);
            f = f / rot.factor * ramp + f * (1 - ramp);
        }
        for (int pos = 0; pos < ctx; ++pos) cs[(size_t)pos * half + i] = make_float2((float)(std::cos(pos * f) * grow), (float)(std::sin(pos * f) * grow));
    }
    void* q = nullptr;
    if (cudaMalloc(&q, cs.size() * sizeof(float2)) != cudaSuccess) { fail(SP_ERR_OOM, "cannot allocate the angle tables"); return nullptr; }
    p.owned.push_back(q);
    if (cudaMemcpy(q, cs.data(), cs.size() * sizeof(float2), cudaMemcpyHostToDevice) != cudaSuccess) { fail(SP_ERR_CUDA, "cudaMemcpy failed"); return nullptr; }
    return tab = (const float2*)q;
}

void PlanPacker::cache_slice(size_t page_bytes) {
    p.cache_base.push_back(p.cache_bytes);
    p.cache_run.push_back(page_bytes);
    p.cache_bytes += (page_bytes * (size_t)e.kv_.n_pages + 255) / 256 * 256;
}

void Engine::plan_release() {
    if (!plan_) return;
    for (void* q : plan_->owned) cudaFree(q);
    if (plan_->cache) cudaFree(plan_->cache);
    if (plan_->states) cudaFree(plan_->states);
    if (plan_->checkpoints) cudaFree(plan_->checkpoints);
    if (plan_->host_tiles) cudaFreeHost(plan_->host_tiles);
    plan_.reset();
}

int Engine::finalize_plan() {
    PlanState& p = *plan_;
    const ModelPlan& mp = p.plan;
    PlanPacker pk{*this, p};
    const int W = mp.width, L = (int)mp.layers.size();
    if (d.tp_size > 1) { set_error("tensor parallelism covers the Llama/Qwen block only"); return SP_ERR_ARG; }
    if (d.max_ctx <= 0) { set_error("finalize: max_ctx must be positive"); return SP_ERR_ARG; }
    p.wp = mat_kpad(W);
    p.layers.resize((size_t)L);
    if (pk.alloc(p.embed, 1, mp.vocab, W)) pk.put(p.embed, 0, pk.need("embed", mp.vocab, W), 0, mp.vocab, W);
    if (mp.tied_head) p.head = p.embed;
    else if (pk.alloc(p.head, 1, mp.vocab, W)) pk.put(p.head, 0, pk.need("head", mp.vocab, W), 0, mp.vocab, W);
    if (mp.max_positions > 0 && pk.alloc(p.pos, 1, mp.max_positions, W)) pk.put(p.pos, 0, pk.need("pos", mp.max_positions, W), 0, mp.max_positions, W);
    if (mp.norm == NORM_TANH) p.final_tanh = pk.tanh_norm("final.norm");
    else p.final_norm = pk.gain("final.norm");
    // pages first: the layers' cache slices are laid out one after another
    const int pages_per_seq = (d.max_ctx + KV_PAGE - 1) / KV_PAGE;
    const int64_t n_pages = d.kv_pages > 0 ? d.kv_pages : (int64_t)d.max_batch * pages_per_seq;
    SP_CUDA_TRY(cudaMalloc((void**)&d_page_table_, (size_t)d.max_batch * pages_per_seq * 4));
    SP_CUDA_TRY(cudaMemset(d_page_table_, 0, (size_t)d.max_batch * pages_per_seq * 4));
    pages.init(d.max_batch, pages_per_seq, (int)n_pages);
    kv_.n_pages = (int)n_pages;
    kv_.max_pages = pages_per_seq;
    kv_.page_table = d_page_table_;
    for (int i = 0; i < L && pk.status == SP_OK; ++i) {
        if (mp.form == FORM_PARALLEL) pk.parallel_layer(i);
        else if (mp.form == FORM_PRE_NORM) pk.pre_norm_layer(i);
        else pk.post_norm_layer(i);
    }
    if (pk.status != SP_OK) return pk.status;
    SP_CUDA_TRY(cudaDeviceSynchronize());
    // the uploaded matrices have been packed; vectors stay (find_f32 may hand out their bytes)
    for (auto& kv : tensors_) {
        DevTensor& t = kv.second;
        if (t.dims.size() == 2 && t.dims[0] > 1 && t.d) {
            cudaFree(t.d);
            t.d = nullptr;
            weight_bytes -= t.nbytes;
        }
    }
    SP_CUDA_TRY(cudaMalloc(&p.cache, p.cache_bytes + 1024));
    SP_CUDA_TRY(cudaMemset(p.cache, 0, p.cache_bytes + 1024));
    const size_t state_bytes = p.slot_state * (size_t)d.max_batch * 4;
    if (p.slot_state > 0) {
        SP_CUDA_TRY(cudaMalloc((void**)&p.states, state_bytes));
        SP_CUDA_TRY(cudaMemset(p.states, 0, state_bytes));
        p.checkpoint_len.assign((size_t)d.max_batch, -1);
    }
    kv_bytes = p.cache_bytes + state_bytes;
    for (int i = 0; i < L; ++i) {
        const LayerPlan& lp = mp.layers[(size_t)i];
        PlanLayer& l = p.layers[(size_t)i];
        const int from = lp.mixer == MIX_LATENT ? lp.latent.kv_from : -1;
        void* slice = (uint8_t*)p.cache + p.cache_base[(size_t)(from >= 0 ? from : i)];
        if (lp.mixer == MIX_LATENT) l.cache.pool = slice;
        else if (lp.has_grouped()) l.kv_cache.pool = slice;
    }
    // buffers of a step
    const size_t T = (size_t)d.max_tokens;
    const bool long_steps = d.max_tokens > PLAN_ROWS, many = long_steps && !p.f32;
    auto take = [&](size_t bytes) -> void* {
        void* q = nullptr;
        if (pk.status != SP_OK || bytes == 0) return nullptr;
        if (cudaMalloc(&q, bytes + 1024) != cudaSuccess || cudaMemset(q, 0, bytes + 1024) != cudaSuccess) {
            pk.fail(SP_ERR_OOM, "cannot allocate the step's buffers");
            return nullptr;
        }
        p.owned.push_back(q);
        return q;
    };
    const size_t el = (size_t)p.elem();
    const PlanSizes& n = p.need;
    p.xb = take(T * p.wp * el);
    p.proj = (float*)take(T * n.proj * 4);
    p.attn = take(T * n.mixed * el);
    p.fin = take((size_t)PLAN_ROWS * p.wp * el);
    if (p.has_latent) {
        p.qn = take(T * n.qn * el);
        p.qabs = take(T * n.qabs * el);
        p.olat = take(T * n.olat * el);
        p.part = (float*)take(plan_latent_part_rows() * n.part * 4);
    }
    p.q = take(T * n.q * el);
    p.stat = (float2*)take(T * n.stat * sizeof(float2));
    p.score = (float*)take(n.score * 4);
    p.score_part = (float2*)take(PLAN_ROWS * n.stat * MIXED_SPLITS * sizeof(float2));
    p.low = take(T * n.low * el);
    if (mp.form == FORM_POST_NORM) {
        p.y = (float*)take(T * W * 4);
        if (mp.depth_average) p.history = (float*)take((size_t)(L + 1) * T * W * 4);
    }
    p.act = take(T * n.act * el);
    if (long_steps) {
        p.wlogit = (float*)take(T * n.wlogit * 4);
        p.groups_cap = p.has_state ? T / state_group(p.f32) + std::min<size_t>(T, (size_t)d.max_batch) + 1 : 0;
        p.state_rec = (float*)take(p.groups_cap * n.state_rec * 4);
    }
    if (n.pairs) {
        p.act_shared = take(T * n.act_shared * el);
        p.y_expert = (float*)take(T * n.pairs * W * 4);
        p.y_shared = (float*)take(T * W * 4);
        p.logit = (float*)take(T * (size_t)(n.experts + 1) * 4);
        p.weight = (float*)take(T * n.pairs * 4);
        p.pick = (int32_t*)take(T * n.pairs * 4);
        const size_t pairs = T * n.pairs, tiles = pairs / MOE_TILE + n.experts + 1;
        p.tables = (int32_t*)take((2 * (size_t)n.experts + 3 + 2 * pairs + 2 * tiles) * 4);
        if (many) p.xs = take((pairs + MOE_TILE) * p.wp * el);
        int32_t* q = p.tables;
        p.moe.row_off = q; q += n.experts + 1;
        p.moe.active = q; q += n.experts;
        p.moe.n_active = q++;
        p.moe.n_tiles = q++;
        p.moe.row_src = q; q += pairs;
        p.moe.slot_of = q; q += pairs;
        p.moe.tile_group = q; q += tiles;
        p.moe.tile_row = q;
    }
    if (many && p.has_latent) {
        p.keys_cap = (int)(3 * T);
        p.qf = take(T * n.qf * el);
        p.kvx = take((size_t)p.keys_cap * n.kv * el);
        p.lat = take((size_t)p.keys_cap * n.lat * el);
    }
    if (long_steps) {
        p.keys_at = p.has_latent ? T * (sizeof(LatentTile) / 4) : 0;
        p.grouped_at = p.keys_at + 2 * (size_t)p.keys_cap;
        p.narrow_at = p.grouped_at + (p.has_grouped ? T * (sizeof(GroupedTile) / 4) : 0);
        p.back_at = p.narrow_at + (p.has_mixed || p.has_conv ? T * (sizeof(GroupedTile) / 4) : 0);
        p.ends_at = p.back_at + (p.has_conv ? T : 0);
        p.seg_at = p.ends_at + (p.has_conv ? (size_t)d.max_batch : 0);
        p.groups_at = (p.seg_at + (p.has_state ? (size_t)d.max_batch * (sizeof(StateSegment) / 4) : 0) + 3) / 4 * 4;
        p.table_ints = p.groups_at + p.groups_cap * state_group(p.f32);
        p.dev_tiles = (int32_t*)take(p.table_ints * 4);
        if (p.table_ints) SP_CUDA_TRY(cudaMallocHost((void**)&p.host_tiles, p.table_ints * 4));
    }
    return pk.status;
}

int Engine::plan_privatise_copy(int from, int to) {
    PlanState& p = *plan_;
    for (size_t i = 0; i < p.layers.size(); ++i) {
        const size_t run = p.cache_run[i];
        if (!run) continue;
        uint8_t* base = (uint8_t*)p.cache + p.cache_base[i];
        SP_CUDA_TRY(cudaMemcpyAsync(base + run * (size_t)to, base + run * (size_t)from, run, cudaMemcpyDeviceToDevice, stream));
    }
    return SP_OK;
}

// The step's longest context as a power of two (exponent): what the key splits of every layer follow from.
int Engine::plan_ctx_bucket() const {
    int b = 6;
    while (b < 30 && (1 << b) < step_ctx_) ++b;
    return b;
}

// Tables of the staged tokens, for steps longer than PLAN_ROWS. Host data only: called outside graphs.
int Engine::plan_stage(int T) {
    PlanState& p = *plan_;
    p.n_tiles = p.n_keys = p.n_grouped = p.n_narrow = p.n_ends = p.n_seg = p.n_groups = 0;
    if (T <= PLAN_ROWS) return SP_OK;
    if (p.has_latent && !p.f32) plan_stage_latent(T);
    // tiles of consecutive tokens of a sequence; the longest ranges of keys first: the blocks that start last are short
    auto tile_rows = [&](size_t at, int rows, int& count) {
        GroupedTile* tiles = reinterpret_cast<GroupedTile*>(p.host_tiles + at);
        for (int i = 0; i < T;) {
            int n = 1;
            while (i + n < T && p_slot_[i + n] == p_slot_[i] && p_pos_[i + n] == p_pos_[i] + n) ++n;
            for (int t = 0; t < n; t += rows) tiles[count++] = GroupedTile{i + t, std::min(rows, n - t), p_pos_[i] + t, p_slot_[i]};
            i += n;
        }
        std::stable_sort(tiles, tiles + count, [](const GroupedTile& a, const GroupedTile& b) { return a.pos0 > b.pos0; });
    };
    if (p.has_grouped && !p.f32) tile_rows(p.grouped_at, GROUPED_Q_TILE, p.n_grouped);
    if (p.has_conv || (p.has_mixed && !p.f32)) tile_rows(p.narrow_at, MIXED_Q_TILE, p.n_narrow);
    if (p.has_conv) {
        std::vector<int> last((size_t)d.max_batch, -1);
        for (int i = 0; i < T; ++i) {
            p.host_tiles[p.back_at + i] = last[p_slot_[i]];
            last[p_slot_[i]] = i;
        }
        for (int s = 0; s < d.max_batch; ++s)
            if (last[s] >= 0) p.host_tiles[p.ends_at + p.n_ends++] = last[s];
    }
    if (p.has_state) {
        StateSegment* seg = reinterpret_cast<StateSegment*>(p.host_tiles + p.seg_at);
        int32_t* groups = p.host_tiles + p.groups_at;
        const int group = state_group(p.f32);
        std::vector<int> count((size_t)d.max_batch, 0), next((size_t)d.max_batch, 0);
        for (int i = 0; i < T; ++i) ++count[p_slot_[i]];
        for (int s = 0; s < d.max_batch; ++s) {
            if (!count[s]) continue;
            const int n = (count[s] + group - 1) / group;
            next[s] = p.n_groups * group;
            std::fill(groups + next[s], groups + next[s] + n * group, -1);
            seg[p.n_seg++] = StateSegment{p.n_groups, n, s, seq_len[s] == count[s]};
            p.n_groups += n;
        }
        for (int i = 0; i < T; ++i) groups[next[p_slot_[i]]++] = i;
    }
    if (p.table_ints) SP_CUDA_TRY(cudaMemcpyAsync(p.dev_tiles, p.host_tiles, p.table_ints * 4, cudaMemcpyHostToDevice, stream));
    return SP_OK;
}

int Engine::plan_product(const MatArgs& a, int max_tiles) {
    SP_LAUNCH(F_GEMV, a.f32 ? launch_mat_f32(a, stream) : launch_mat_tc5(a, max_tiles, stream));
    return SP_OK;
}

int Engine::plan_mat(const PlanMat& w, const void* x, int ldx, int m, void* y, int ldy, bool out_f32) {
    MatArgs a{};
    a.f32 = plan_->f32;
    a.out_f32 = out_f32;
    a.nseg = 1;
    a.m = m;
    a.seg[0] = MatSeg{w.w, w.n, w.kp, 1, MatUnit{}, x, ldx, 0, y, ldy, 0};
    return plan_product(a, 0);
}

int Engine::plan_layers(int T) {
    PlanState& p = *plan_;
    const int W = p.plan.width, L = (int)p.layers.size();
    const LayerForm form = p.plan.form;
    const TanhNorm first = p.plan.norm == NORM_TANH ? p.layers[0].tanh1 : TanhNorm{};
    SP_LAUNCH(F_EMBED, launch_embed_scaled(p.embed.w, p.pos.w, p.embed.kp, p.f32, d_ids_, d_tok_pos_, T, W, p.plan.embed_scale, first, p.history ? p.history : x_,
                                           form == FORM_POST_NORM || first.w ? p.xb : nullptr, p.wp, stream));
    for (int i = 0; i < L; ++i) {
        SP_TRY(form == FORM_PARALLEL ? plan_layer_parallel(i, T) : form == FORM_PRE_NORM ? plan_layer_pre_norm(i, T) : plan_layer_post_norm(i, T));
        if (trace_on) SP_CUDA_TRY(cudaMemcpyAsync(trace_ + (size_t)i * d.max_tokens * W, x_, (size_t)T * W * 4, cudaMemcpyDeviceToDevice, stream));
    }
    trace_tokens_ = T;
    return SP_OK;
}

// Final norm, output head and arg-max of n rows of the stream (rows: device indices, null: 0 .. n - 1).
int Engine::plan_head(const int32_t* rows, int n) {
    PlanState& p = *plan_;
    const int V = p.plan.vocab;
    if (p.plan.norm == NORM_TANH) SP_LAUNCH(F_NORM, launch_tanh_norm(x_, rows, n, p.plan.width, p.final_tanh, p.fin, p.wp, p.f32, stream));
    else SP_LAUNCH(F_NORM, launch_row_norm(x_, rows, n, p.plan.width, p.final_norm, p.plan.eps, p.fin, p.wp, p.f32, stream));
    if (p.plan.logit_scale == 1.f && p.plan.logit_softcap <= 0.f) {
        SP_TRY(plan_mat(p.head, p.fin, p.wp, n, logits_, V, true));
    } else {
        MatArgs a{};
        a.f32 = p.f32;
        a.nseg = a.n_outs = 1;
        a.m = n;
        a.seg[0] = MatSeg{p.head.w, V, p.head.kp, 1, MatUnit{}, p.fin, p.wp, 0, nullptr, 0, 0};
        a.outs[0] = MatOut{V, logits_, V, MAT_SOFTCAP, true, false};
        a.arg[0] = p.plan.logit_scale;
        a.arg[1] = p.plan.logit_softcap;
        SP_TRY(plan_product(a, 0));
    }
    SP_LAUNCH(F_ARGMAX, launch_argmax(logits_, n, V, V, d_argmax_, stream, argmax_scratch_));
    return SP_OK;
}

// ── rollback of sequences with a state ──
bool Engine::keeps_state() const { return plan_ && plan_->slot_state > 0; }

int Engine::checkpoint(int slot) {
    if (slot < 0 || slot >= d.max_batch) { set_error("slot out of range"); return SP_ERR_ARG; }
    if (!keeps_state()) return SP_OK;
    SP_CUDA_TRY(cudaSetDevice(d.device));
    PlanState& p = *plan_;
    if (!p.checkpoints) SP_CUDA_TRY(cudaMalloc((void**)&p.checkpoints, p.slot_state * (size_t)d.max_batch * 4));
    SP_CUDA_TRY(cudaMemcpyAsync(p.checkpoints + p.slot_state * slot, p.states + p.slot_state * slot, p.slot_state * 4, cudaMemcpyDeviceToDevice, stream));
    p.checkpoint_len[(size_t)slot] = seq_len[slot];
    return SP_OK;
}

// The longest length of at most n whose state is at hand: the current one, the checkpoint's or 0.
int Engine::plan_rollback(int slot, int n, int* kept) {
    PlanState& p = *plan_;
    int& c = p.checkpoint_len[(size_t)slot];
    *kept = n == seq_len[slot] ? n : c >= 0 && c <= n ? c : 0;
    if (*kept < seq_len[slot] && *kept == c)
        SP_CUDA_TRY(cudaMemcpyAsync(p.states + p.slot_state * slot, p.checkpoints + p.slot_state * slot, p.slot_state * 4, cudaMemcpyDeviceToDevice, stream));
    if (*kept < c || *kept == 0) c = -1;
    return SP_OK;
}

}  // namespace sp
