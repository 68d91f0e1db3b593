// Plan-driven models (model_plan.h) on the resident engine: weights packed once into the shapes the kernels read, a paged
// latent cache behind the same page pool, and the launch sequence of a step.
//
// A layer is ten to fifteen launches: projections, rotation + cache append, then either queries to latent space, absorbed
// attention and value maps or gather, rebuilt keys and values and expanded attention; output projection, norm + residual,
// router, choice and grouping, gate|up of the chosen and the shared expert, down, mixture + norm + residual + depth
// average. bf16 products run on the tcgen05 kernel (mat_tc5.cu) at
// every row count, f32 ones on mat_f32.cu. Steps of up to PLAN_ROWS rows take the absorbed attention and can be captured as
// a graph; longer ones, where rebuilding the keys pays, the expanded attention.
#include "engine_plan.h"

#include <algorithm>
#include <cmath>
#include <cstring>
#include <map>

#include "engine.h"
#include "plan_common.cuh"
#include "sp_common.cuh"

namespace sp {

#define SP_TRY(expr)                  \
    do {                              \
        int _s = (expr);              \
        if (_s != SP_OK) return _s;   \
    } while (0)

#define SP_LAUNCH(fam, expr)              \
    do {                                  \
        if (fam_mask & (1u << (fam))) {   \
            prof_begin(fam);              \
            SP_CUDA_TRY(expr);            \
            prof_end(fam);                \
        }                                 \
    } while (0)

constexpr int PLAN_ROWS = MAT_GATHER_ROWS;  // rows of a decode-shaped step
constexpr int PLAN_SPLIT_ROWS = 256;  // (rows x key splits) of the absorbed attention's partials

namespace {

__device__ __forceinline__ float load_elem(int dtype, const uint8_t* p, int64_t i) {
    if (dtype == T_F32) return reinterpret_cast<const float*>(p)[i];
    if (dtype == T_BF16) return __bfloat162float(reinterpret_cast<const bf16*>(p)[i]);
    return __half2float(reinterpret_cast<const __half*>(p)[i]);
}

// dst[r][0 .. kp) = src[r][0 .. k) (or src[0 .. k)[r] transposed, source row stride lds), zero-padded.
template <typename T>
__global__ void pack_rows_kernel(int dtype, const uint8_t* __restrict__ src, int64_t lds, bool transpose, int k, int kp, T* __restrict__ dst) {
    const int64_t r = blockIdx.x;
    for (int c = threadIdx.x; c < kp; c += blockDim.x) {
        float v = 0.f;
        if (c < k) v = load_elem(dtype, src, transpose ? (int64_t)c * lds + r : r * lds + c);
        dst[r * kp + c] = from_f32<T>(v);
    }
}

size_t esize(int dtype) { return dtype == T_F32 ? 4 : 2; }

}  // namespace

// Builds packed matrices out of the uploaded tensors.
struct PlanPacker {
    Engine& e;
    PlanState& p;
    int status = SP_OK;

    bool fail(int st, const std::string& msg) {
        if (status == SP_OK) { set_error(msg); status = st; }
        return false;
    }
    const DevTensor* need(const std::string& name, int64_t rows, int64_t cols) {
        const DevTensor* t = e.find(name);
        if (!t) { fail(SP_ERR_STATE, "missing weight '" + name + "'"); return nullptr; }
        const int64_t r = t->dims.size() == 2 ? t->dims[0] : 1, c = t->dims.back();
        if (r * c != rows * cols || (cols > 1 && c != cols) || (t->dtype != T_F32 && t->dtype != T_BF16 && t->dtype != T_F16)) {
            fail(SP_ERR_SHAPE, "shape or dtype mismatch for '" + name + "'");
            return nullptr;
        }
        return t;
    }
    const float* vec(const std::string& name, int64_t n) {
        if (!need(name, 1, n)) return nullptr;
        const float* f = e.find_f32(name, n);
        if (!f) fail(SP_ERR_OOM, "cannot convert '" + name + "'");
        return f;
    }
    bool alloc(PlanMat& m, int groups, int64_t rows, int k) {
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
    // rows [r0, r0 + rows) of source tensor t to packed rows starting at `to` (counted over all groups)
    bool put(PlanMat& m, int64_t to, const DevTensor* t, int64_t r0, int64_t rows, int k, bool transpose = false) {
        if (!t || !m.w) return false;
        const int64_t lds = t->dims.back();
        const uint8_t* src = t->d + (size_t)(r0 * lds) * esize(t->dtype);
        uint8_t* dst = (uint8_t*)m.w + (size_t)to * m.kp * p.elem();
        if (p.f32) pack_rows_kernel<float><<<(unsigned)rows, 128>>>(t->dtype, src, lds, transpose, k, m.kp, (float*)dst);
        else pack_rows_kernel<bf16><<<(unsigned)rows, 128>>>(t->dtype, src, lds, transpose, k, m.kp, (bf16*)dst);
        if (cudaGetLastError() != cudaSuccess) return fail(SP_ERR_CUDA, "pack_rows_kernel failed");
        return true;
    }
};

void Engine::plan_release() {
    if (!plan_) return;
    for (void* q : plan_->owned) cudaFree(q);
    if (plan_->cache) cudaFree(plan_->cache);
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
    if (pk.alloc(p.head, 1, mp.vocab, W)) pk.put(p.head, 0, pk.need("head", mp.vocab, W), 0, mp.vocab, W);
    p.final_norm = pk.vec("final.norm", 1);
    // pages first: the layers' cache slices are laid out one after another, [layer][page][16 tokens][ld]
    const int pages_per_seq = (d.max_ctx + KV_PAGE - 1) / KV_PAGE;
    const int64_t n_pages = d.kv_pages > 0 ? d.kv_pages : (int64_t)d.max_batch * pages_per_seq;
    SP_CUDA_TRY(cudaMalloc((void**)&d_page_table_, (size_t)d.max_batch * pages_per_seq * 4));
    SP_CUDA_TRY(cudaMemset(d_page_table_, 0, (size_t)d.max_batch * pages_per_seq * 4));
    pages.init(d.max_batch, pages_per_seq, (int)n_pages);
    kv_.n_pages = (int)n_pages;
    kv_.max_pages = pages_per_seq;
    kv_.page_table = d_page_table_;

    std::map<std::pair<double, int>, const float2*> tables;
    size_t cache_bytes = 0;
    size_t n_proj = 0, n_qn = 0, n_qabs = 0, n_qf = 0, n_olat = 0, n_attn = 0, n_act = 0, n_act_s = 0, n_pairs = 0, n_kv = 0, n_lat = 0, n_part = 0;
    int max_experts = 0;
    for (int i = 0; i < L && pk.status == SP_OK; ++i) {
        const LayerPlan& lp = mp.layers[(size_t)i];
        const LatentAttentionSpec& m = lp.mix;
        PlanLayer& l = p.layers[(size_t)i];
        const std::string mx = lp.prefix + "mix.", ml = lp.prefix + "mlp.";
        const int H = m.heads, D = m.dim, R = m.rot_dim, V = m.vdim, K = m.kv_rank;
        l.own = m.kv_from < 0;
        l.shape = LatentShape{H, D, R, V, m.window, m.scale};
        l.norm1 = pk.vec(lp.prefix + "norm1", 1);
        // projections that read the mixer's input
        const int q_rows = H * (D + R), kv_rows = l.own ? K + R : 0;
        l.gate_col = q_rows + kv_rows;
        if (!pk.alloc(l.proj, 1, q_rows + kv_rows + H, W)) break;
        pk.put(l.proj, 0, pk.need(mx + "q", q_rows, W), 0, q_rows, W);
        if (l.own) {
            pk.put(l.proj, q_rows, pk.need(mx + "dkv", kv_rows, W), 0, kv_rows, W);
            l.dkv_norm = pk.vec(mx + "dkv.norm", K);
        }
        pk.put(l.proj, l.gate_col, pk.need(mx + "g", H, W), 0, H, W);
        const DevTensor *uk = pk.need(mx + "uk", (int64_t)H * D, K), *uv = pk.need(mx + "uv", (int64_t)H * V, K);
        if (!pk.alloc(l.uk_t, H, K, D) || !pk.alloc(l.uv, H, V, K)) break;
        for (int h = 0; h < H; ++h) {
            pk.put(l.uk_t, (int64_t)h * K, uk, (int64_t)h * D, K, D, true);
            pk.put(l.uv, (int64_t)h * V, uv, (int64_t)h * V, V, K);
        }
        const int D16 = (D + 15) & ~15, V16 = (V + 15) & ~15, R16 = (R + 15) & ~15, K16 = (K + 15) & ~15;
        l.expand = !p.f32 && latent_expanded_supported(D, R, V);
        if (l.expand) {
            if (!pk.alloc(l.kv, 1, (int64_t)H * (D16 + V16), K)) break;
            for (int h = 0; h < H; ++h) {
                pk.put(l.kv, (int64_t)h * (D16 + V16), uk, (int64_t)h * D, D, K);
                pk.put(l.kv, (int64_t)h * (D16 + V16) + D16, uv, (int64_t)h * V, V, K);
            }
        }
        if (!pk.alloc(l.o, 1, W, H * V)) break;
        pk.put(l.o, 0, pk.need(mx + "o", W, (int64_t)H * V), 0, W, H * V);
        // the latent cache
        l.cache.rank = K;
        l.cache.rank16 = K16;
        l.cache.rot = R;
        l.cache.rot16 = R16;
        l.cache.ld = mat_kpad(K16 + R16);
        l.cache.page_table = d_page_table_;
        l.cache.max_pages = pages_per_seq;
        p.cache_base.push_back(cache_bytes);
        p.cache_run.push_back(l.own ? (size_t)KV_PAGE * l.cache.ld * p.elem() : 0);
        cache_bytes += p.cache_run.back() * (size_t)n_pages;
        if (K > 1024) { set_error("latent rank above 1024 is not supported"); return SP_ERR_ARG; }
        // angles are computed in double and rounded once
        const float2*& tab = tables[{m.rot.base, R}];
        if (!tab) {
            std::vector<float2> cs((size_t)d.max_ctx * (R / 2));
            for (int i2 = 0; i2 < R / 2; ++i2) {
                const double f = std::pow(m.rot.base, -2.0 * i2 / R);
                for (int pos = 0; pos < d.max_ctx; ++pos) cs[(size_t)pos * (R / 2) + i2] = make_float2((float)std::cos(pos * f), (float)std::sin(pos * f));
            }
            void* q = nullptr;
            SP_CUDA_TRY(cudaMalloc(&q, cs.size() * sizeof(float2)));
            p.owned.push_back(q);
            SP_CUDA_TRY(cudaMemcpy(q, cs.data(), cs.size() * sizeof(float2), cudaMemcpyHostToDevice));
            tab = (const float2*)q;
        }
        l.cos_sin = tab;
        if (mp.depth_average) l.dwa = pk.vec(lp.prefix + "dwa", i + 2);
        // experts
        if (lp.has_mlp) {
            const MoeSpec& s = lp.mlp;
            const int E = s.experts, F = s.expert.ff;
            l.norm2 = pk.vec(lp.prefix + "norm2", 1);
            if (!pk.alloc(l.router, 1, E + (s.has_shared ? 1 : 0), W)) break;
            pk.put(l.router, 0, pk.need(ml + "router", E, W), 0, E, W);
            l.router_b = pk.vec(ml + "router.b", E);
            if (!pk.alloc(l.gu, E, 2 * (int64_t)F, W) || !pk.alloc(l.down, E, W, F)) break;
            for (int x = 0; x < E; ++x) {
                const std::string ex = ml + "e" + std::to_string(x) + ".";
                pk.put(l.gu, (int64_t)x * 2 * F, pk.need(ex + "gate", F, W), 0, F, W);
                pk.put(l.gu, (int64_t)x * 2 * F + F, pk.need(ex + "up", F, W), 0, F, W);
                pk.put(l.down, (int64_t)x * W, pk.need(ex + "down", W, F), 0, W, F);
            }
            if (s.has_shared) {
                const int S = s.shared.ff;
                if (!pk.alloc(l.shared_gu, 1, 2 * (int64_t)S, W) || !pk.alloc(l.shared_down, 1, W, S)) break;
                pk.put(l.shared_gu, 0, pk.need(ml + "shared.gate", S, W), 0, S, W);
                pk.put(l.shared_gu, S, pk.need(ml + "shared.up", S, W), 0, S, W);
                pk.put(l.shared_down, 0, pk.need(ml + "shared.down", W, S), 0, W, S);
                pk.put(l.router, E, pk.need(ml + "shared.sg", 1, W), 0, 1, W);
                n_act_s = std::max<size_t>(n_act_s, (size_t)l.shared_down.kp);
            }
            n_act = std::max<size_t>(n_act, (size_t)s.top * l.down.kp);
            n_pairs = std::max<size_t>(n_pairs, (size_t)s.top);
            max_experts = std::max(max_experts, E);
        }
        n_proj = std::max<size_t>(n_proj, (size_t)l.proj.n);
        n_qn = std::max<size_t>(n_qn, (size_t)H * l.uk_t.kp);
        n_qabs = std::max<size_t>(n_qabs, (size_t)H * l.cache.ld);
        n_qf = std::max<size_t>(n_qf, (size_t)H * (D16 + R16));
        n_olat = std::max<size_t>(n_olat, (size_t)H * l.uv.kp);
        n_attn = std::max<size_t>(n_attn, (size_t)l.o.kp);
        n_kv = std::max<size_t>(n_kv, (size_t)H * (D16 + V16));
        n_lat = std::max<size_t>(n_lat, (size_t)l.cache.ld);
        n_part = std::max<size_t>(n_part, (size_t)H * (K + 2));
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
    kv_bytes = cache_bytes;
    SP_CUDA_TRY(cudaMalloc(&p.cache, cache_bytes + 1024));
    SP_CUDA_TRY(cudaMemset(p.cache, 0, cache_bytes + 1024));
    for (int i = 0; i < L; ++i) {
        const int from = mp.layers[(size_t)i].mix.kv_from;
        p.layers[(size_t)i].cache.pool = (uint8_t*)p.cache + p.cache_base[(size_t)(from >= 0 ? from : i)];
    }
    // buffers of a step
    const size_t T = (size_t)d.max_tokens;
    const bool many = !p.f32 && d.max_tokens > PLAN_ROWS;
    auto take = [&](size_t bytes) -> void* {
        void* q = nullptr;
        if (pk.status != SP_OK) return nullptr;
        if (cudaMalloc(&q, bytes + 1024) != cudaSuccess || cudaMemset(q, 0, bytes + 1024) != cudaSuccess) {
            pk.fail(SP_ERR_OOM, "cannot allocate the step's buffers");
            return nullptr;
        }
        p.owned.push_back(q);
        return q;
    };
    const size_t el = (size_t)p.elem();
    p.xb = take(T * p.wp * el);
    p.proj = (float*)take(T * n_proj * 4);
    p.qn = take(T * n_qn * el);
    p.qabs = take(T * n_qabs * el);
    p.olat = take(T * n_olat * el);
    p.attn = take(T * n_attn * el);
    p.y = (float*)take(T * W * 4);
    p.part = (float*)take((size_t)PLAN_SPLIT_ROWS * n_part * 4);
    p.history = (float*)take((size_t)(L + 1) * T * W * 4);
    p.fin = take((size_t)PLAN_ROWS * p.wp * el);
    if (n_pairs) {
        p.act = take(T * n_act * el);
        p.act_shared = take(T * n_act_s * el);
        p.y_expert = (float*)take(T * n_pairs * W * 4);
        p.y_shared = (float*)take(T * W * 4);
        p.logit = (float*)take(T * (size_t)(max_experts + 1) * 4);
        p.weight = (float*)take(T * n_pairs * 4);
        p.pick = (int32_t*)take(T * n_pairs * 4);
        const size_t pairs = T * n_pairs, tiles = pairs / MOE_TILE + max_experts + 1;
        p.tables = (int32_t*)take((2 * (size_t)max_experts + 3 + 2 * pairs + 2 * tiles) * 4);
        if (many) p.xs = take((pairs + MOE_TILE) * p.wp * el);
        int32_t* q = p.tables;
        p.moe.row_off = q; q += max_experts + 1;
        p.moe.active = q; q += max_experts;
        p.moe.n_active = q++;
        p.moe.n_tiles = q++;
        p.moe.row_src = q; q += pairs;
        p.moe.slot_of = q; q += pairs;
        p.moe.tile_group = q; q += tiles;
        p.moe.tile_row = q;
    }
    if (many) {
        p.keys_cap = (int)(3 * T);
        p.qf = take(T * n_qf * el);
        p.kvx = take((size_t)p.keys_cap * n_kv * el);
        p.lat = take((size_t)p.keys_cap * n_lat * el);
        const size_t ints = T * (sizeof(LatentTile) / 4) + 2 * (size_t)p.keys_cap;
        p.dev_tiles = (int32_t*)take(ints * 4);
        SP_CUDA_TRY(cudaMallocHost((void**)&p.host_tiles, ints * 4));
    }
    if (pk.status != SP_OK) return pk.status;
    return SP_OK;
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

static int plan_splits(const PlanLayer& l, bool f32, int bucket, int T) {
    if (T > PLAN_ROWS) return 1;
    int s = latent_attention_splits(l.shape.heads, T, std::min(1 << bucket, l.shape.window), f32);
    while (s > 1 && T * s > PLAN_SPLIT_ROWS) s >>= 1;
    return s;
}

// Decides how the staged tokens attend and uploads the tables of the expanded form. Host data only: called outside graphs.
int Engine::plan_stage(int T) {
    PlanState& p = *plan_;
    p.n_tiles = p.n_keys = 0;
    if (p.f32 || T <= PLAN_ROWS) return SP_OK;
    int window = 0;
    for (const PlanLayer& l : p.layers) window = std::max(window, l.shape.window);
    LatentTile* tiles = reinterpret_cast<LatentTile*>(p.host_tiles);
    const size_t key_at = (size_t)d.max_tokens * (sizeof(LatentTile) / 4);
    int32_t *slot = p.host_tiles + key_at, *pos = slot + p.keys_cap;
    int keys = 0, nt = 0;
    for (int i = 0; i < T;) {
        int n = 1;
        while (i + n < T && p_slot_[i + n] == p_slot_[i] && p_pos_[i + n] == p_pos_[i] + n) ++n;
        const int first = window > p_pos_[i] ? 0 : p_pos_[i] - window + 1, cnt = p_pos_[i] + n - first;
        if (keys + cnt > p.keys_cap || keys + cnt > 3 * T) return SP_OK;  // more keys to rebuild than it saves
        for (int t = 0; t < n; t += LATENT_Q_TILE) tiles[nt++] = LatentTile{i + t, std::min(LATENT_Q_TILE, n - t), p_pos_[i] + t, keys, first};
        for (int k = 0; k < cnt; ++k) { slot[keys + k] = p_slot_[i]; pos[keys + k] = first + k; }
        keys += cnt;
        i += n;
    }
    const size_t ints = key_at + 2 * (size_t)p.keys_cap;
    SP_CUDA_TRY(cudaMemcpyAsync(p.dev_tiles, p.host_tiles, ints * 4, cudaMemcpyHostToDevice, stream));
    p.n_tiles = nt;
    p.n_keys = keys;
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
    a.seg[0] = MatSeg{w.w, w.n, w.kp, 1, 0.f, 0.f, x, ldx, 0, y, ldy, 0};
    return plan_product(a, 0);
}

int Engine::plan_mixer(int li, int T) {
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
        const int32_t* keys = p.dev_tiles + (size_t)d.max_tokens * (sizeof(LatentTile) / 4);
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
    const MoeSpec& s = p.plan.layers[(size_t)li].mlp;
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

int Engine::plan_layers(int T) {
    PlanState& p = *plan_;
    const int W = p.plan.width, L = (int)p.layers.size();
    const int64_t hs = (int64_t)d.max_tokens * W;
    SP_LAUNCH(F_EMBED, launch_embed_scaled(p.embed.w, p.embed.kp, p.f32, d_ids_, T, W, p.plan.embed_scale, p.history, p.xb, p.wp, stream));
    for (int i = 0; i < L; ++i) {
        PlanLayer& l = p.layers[(size_t)i];
        const LayerPlan& lp = p.plan.layers[(size_t)i];
        SP_TRY(plan_mixer(i, T));
        SP_LAUNCH(F_NORM, launch_norm_residual(p.y, W, l.norm1, p.plan.eps, i == 0 ? p.history : x_, x_, p.xb, p.wp, p.f32, T, W, stream));
        CombineArgs c{};
        if (lp.has_mlp) {
            SP_TRY(plan_experts(i, T));
            c.y = p.y_expert;
            c.ldy = W;
            c.slot_of = p.moe.slot_of;
            c.weight = p.weight;
            c.top = lp.mlp.top;
            if (lp.mlp.has_shared) {
                c.y_shared = p.y_shared;
                c.shared_gate = p.logit + lp.mlp.experts;
                c.ld_gate = l.router.n;
            }
            c.gain = l.norm2;
            c.eps = p.plan.eps;
        }
        c.x = x_;
        c.history = p.history;
        c.hist_stride = hs;
        c.depth = i + 1;
        c.dwa = l.dwa;
        c.x_out = x_;
        c.xb = p.xb;
        c.ldb = p.wp;
        c.f32 = p.f32;
        SP_LAUNCH(F_NORM, launch_combine(c, T, W, stream));
        if (trace_on) SP_CUDA_TRY(cudaMemcpyAsync(trace_ + (size_t)i * d.max_tokens * W, x_, (size_t)T * W * 4, cudaMemcpyDeviceToDevice, stream));
    }
    trace_tokens_ = T;
    return SP_OK;
}

// Final norm, output head and arg-max of n rows of the stream (rows: device indices, null: 0 .. n - 1).
int Engine::plan_head(const int32_t* rows, int n) {
    PlanState& p = *plan_;
    SP_LAUNCH(F_NORM, launch_final_norm(x_, rows, n, p.plan.width, p.final_norm, p.plan.eps, p.fin, p.wp, p.f32, stream));
    SP_TRY(plan_mat(p.head, p.fin, p.wp, n, logits_, p.plan.vocab, true));
    SP_LAUNCH(F_ARGMAX, launch_argmax(logits_, n, p.plan.vocab, p.plan.vocab, d_argmax_, stream, argmax_scratch_));
    return SP_OK;
}

}  // namespace sp
