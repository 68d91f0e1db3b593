// The residual stream of plan-driven models: scaled embedding, norms on a sublayer's output, the mixture of expert
// outputs, depth averages — all in f32, each kernel also leaving the stream in the compute type for the next product —
// and the routing of tokens to experts.
#include "kernels.h"
#include "pdl.cuh"
#include "plan_common.cuh"
#include "plan_kernels.h"

namespace sp {

cudaError_t count_launch_and_check();  // kernels.cu

constexpr int ST_WARPS = 16, ST_THREADS = 32 * ST_WARPS;

// V consecutive elements of a row (V = 4 where the width allows it).
template <int V> struct Row;
template <> struct Row<1> {
    static __device__ __forceinline__ void load(const float* p, float (&v)[1]) { v[0] = *p; }
    static __device__ __forceinline__ void store(float* p, const float (&v)[1]) { *p = v[0]; }
    static __device__ __forceinline__ void store(bf16* p, const float (&v)[1]) { *p = __float2bfloat16_rn(v[0]); }
};
template <> struct Row<4> {
    static __device__ __forceinline__ void load(const float* p, float (&v)[4]) {
        const float4 q = *reinterpret_cast<const float4*>(p);
        v[0] = q.x; v[1] = q.y; v[2] = q.z; v[3] = q.w;
    }
    static __device__ __forceinline__ void store(float* p, const float (&v)[4]) { *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]); }
    static __device__ __forceinline__ void store(bf16* p, const float (&v)[4]) {
        *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16(v[0], v[1]), pack_bf16(v[2], v[3]));
    }
};

template <typename T>
__global__ void __launch_bounds__(ST_THREADS) embed_scaled_kernel(const T* __restrict__ table, const T* __restrict__ pos_table, int ldt,
                                                                  const uint32_t* __restrict__ ids, const int32_t* __restrict__ tok_pos, int width, float scale,
                                                                  const TanhNorm norm, float* __restrict__ x0, T* __restrict__ xb, int ldb) {
    pdl_wait();
    pdl_trigger();
    const int t = blockIdx.x;
    const T* row = table + (int64_t)ids[t] * ldt;
    const T* prow = pos_table ? pos_table + (int64_t)tok_pos[t] * ldt : nullptr;
    for (int c = threadIdx.x; c < ldb; c += ST_THREADS) {
        float v = c < width ? to_f32(row[c]) * scale : 0.f;
        if (prow && c < width) v += to_f32(prow[c]);
        if (c < width) x0[(int64_t)t * width + c] = v;
        if (norm.w && c < width) v = tanh_norm(norm, v, c);
        if (xb) xb[(int64_t)t * ldb + c] = from_f32<T>(v);
    }
}

cudaError_t launch_embed_scaled(const void* table, const void* pos_table, int ldt, bool f32, const uint32_t* ids, const int32_t* tok_pos, int n_tok,
                                int width, float scale, const TanhNorm& norm, float* x0, void* xb, int ldb, cudaStream_t st) {
    if (n_tok == 0) return cudaSuccess;
    const dim3 grid(n_tok), block(ST_THREADS);
#define SP_EM(T) launch_pdl(embed_scaled_kernel<T>, grid, block, 0, st, (const T*)table, (const T*)pos_table, ldt, ids, tok_pos, width, scale, norm, x0, (T*)xb, ldb)
    const cudaError_t le = f32 ? SP_EM(float) : SP_EM(bf16);
#undef SP_EM
    if (le != cudaSuccess) return le;
    return count_launch_and_check();
}

template <typename T, int V>
__global__ void __launch_bounds__(ST_THREADS) norm_residual_kernel(const float* __restrict__ y, int ldy, const RowGain gain, float eps, float mult,
                                                                   const float* x, float* x_out, T* __restrict__ xb, int ldb, int width) {
    __shared__ float sh[ST_WARPS];
    pdl_wait();
    pdl_trigger();
    const int64_t t = blockIdx.x;
    const float* yr = y + t * ldy;
    const float g0 = gain.per_coord ? 1.f : *gain.g;
    float ss = 0.f, v[V], o[V], g[V];
    for (int c = V * threadIdx.x; c < width; c += V * ST_THREADS) {
        Row<V>::load(yr + c, v);
#pragma unroll
        for (int i = 0; i < V; ++i) ss = fmaf(v[i], v[i], ss);
    }
    const float r = rsqrtf(block_sum<ST_WARPS>(ss, sh) / (float)width + eps) * g0 * mult;
#pragma unroll
    for (int i = 0; i < V; ++i) g[i] = 1.f;
    for (int c = V * threadIdx.x; c < ldb; c += V * ST_THREADS) {
#pragma unroll
        for (int i = 0; i < V; ++i) o[i] = 0.f;
        if (c < width) {
            Row<V>::load(yr + c, v);
            Row<V>::load(x + t * width + c, o);
            if (gain.per_coord) Row<V>::load(gain.g + c, g);
#pragma unroll
            for (int i = 0; i < V; ++i) o[i] = fmaf(v[i] * g[i], r, o[i]);
            Row<V>::store(x_out + t * width + c, o);
        }
        Row<V>::store(xb + t * ldb + c, o);
    }
}

// Four coordinates at a time: rows and gains start on 16-byte boundaries.
static bool wide_rows(int width, int ld, const RowGain& gain) {
    return width % 4 == 0 && ld % 4 == 0 && (!gain.per_coord || (reinterpret_cast<uintptr_t>(gain.g) & 15) == 0);
}

cudaError_t launch_norm_residual(const float* y, int ldy, const RowGain& gain, float eps, float mult, const float* x, float* x_out, void* xb, int ldb,
                                 bool f32, int n_tok, int width, cudaStream_t st) {
    if (n_tok == 0) return cudaSuccess;
    const bool wide = wide_rows(width, ldy, gain);
#define SP_NR(T, V) launch_pdl(norm_residual_kernel<T, V>, dim3(n_tok), dim3(ST_THREADS), 0, st, y, ldy, gain, eps, mult, x, x_out, (T*)xb, ldb, width)
    const cudaError_t le = f32 ? (wide ? SP_NR(float, 4) : SP_NR(float, 1)) : (wide ? SP_NR(bf16, 4) : SP_NR(bf16, 1));
#undef SP_NR
    if (le != cudaSuccess) return le;
    return count_launch_and_check();
}

// One block per token. Shared memory: the feed-forward's sum between the two passes over the width, the weights and rows
// of the chosen experts, the depth coefficients.
template <typename T, int V>
__global__ void __launch_bounds__(ST_THREADS) combine_kernel(const CombineArgs a, int width) {
    extern __shared__ __align__(16) float ff[];
    __shared__ float sh[ST_WARPS];
    float* w_s = ff + (a.y ? (width + 3) / 4 * 4 : 0);
    int* row_s = reinterpret_cast<int*>(w_s + a.top);
    float* dwa_s = w_s + 2 * a.top;
    pdl_wait();
    pdl_trigger();
    const int64_t t = blockIdx.x;
    for (int k = threadIdx.x; k < a.top; k += ST_THREADS) {
        w_s[k] = a.weight[t * a.top + k];
        row_s[k] = a.slot_of[t * a.top + k];
    }
    if (a.dwa)
        for (int j = threadIdx.x; j <= a.depth; j += ST_THREADS) dwa_s[j] = a.dwa[j];
    const float sg = a.shared_gate ? sigmoid_f32(a.shared_gate[t * a.ld_gate]) : 1.f;
    __syncthreads();
    float r = 0.f;
    if (a.y) {
        const float gain = a.gain.per_coord ? 1.f : *a.gain.g;
        float ss = 0.f;
        for (int c = V * threadIdx.x; c < width; c += V * ST_THREADS) {
            float s[V], q[V];
#pragma unroll
            for (int i = 0; i < V; ++i) s[i] = 0.f;
#pragma unroll 4
            for (int k = 0; k < a.top; ++k) {
                Row<V>::load(a.y + (int64_t)row_s[k] * a.ldy + c, q);
#pragma unroll
                for (int i = 0; i < V; ++i) s[i] = fmaf(w_s[k], q[i], s[i]);
            }
            if (a.y_shared) {
                Row<V>::load(a.y_shared + t * a.ldy + c, q);
#pragma unroll
                for (int i = 0; i < V; ++i) s[i] = fmaf(sg, q[i], s[i]);
            }
            Row<V>::store(ff + c, s);
#pragma unroll
            for (int i = 0; i < V; ++i) ss = fmaf(s[i], s[i], ss);
        }
        r = rsqrtf(block_sum<ST_WARPS>(ss, sh) / (float)width + a.eps) * gain * a.mult;
    }
    float* mine = a.history ? a.history + (int64_t)a.depth * a.hist_stride + t * width : nullptr;
    for (int c = V * threadIdx.x; c < a.ldb; c += V * ST_THREADS) {
        float v[V], q[V];
#pragma unroll
        for (int i = 0; i < V; ++i) v[i] = 0.f;
        if (c < width) {
            Row<V>::load(a.x + t * width + c, v);
            if (a.y) {
                Row<V>::load(ff + c, q);  // written above by this same thread
                if (a.gain.per_coord) {
                    float g[V];
                    Row<V>::load(a.gain.g + c, g);
#pragma unroll
                    for (int i = 0; i < V; ++i) q[i] *= g[i];
                }
#pragma unroll
                for (int i = 0; i < V; ++i) v[i] = fmaf(q[i], r, v[i]);
            }
            if (mine) Row<V>::store(mine + c, v);
            if (a.dwa) {
                const float* h = a.history + t * width + c;
                float s[V];
#pragma unroll
                for (int i = 0; i < V; ++i) s[i] = 0.f;
#pragma unroll 8
                for (int j = 0; j < a.depth; ++j) {
                    Row<V>::load(h + (int64_t)j * a.hist_stride, q);
#pragma unroll
                    for (int i = 0; i < V; ++i) s[i] = fmaf(dwa_s[j], q[i], s[i]);
                }
#pragma unroll
                for (int i = 0; i < V; ++i) v[i] = fmaf(dwa_s[a.depth], v[i], s[i]);
            }
            Row<V>::store(a.x_out + t * width + c, v);
        }
        Row<V>::store(reinterpret_cast<T*>(a.xb) + t * a.ldb + c, v);
    }
}

cudaError_t launch_combine(const CombineArgs& a, int n_tok, int width, cudaStream_t st) {
    if (n_tok == 0) return cudaSuccess;
    const size_t smem = ((size_t)(a.y ? (width + 3) / 4 * 4 : 0) + 2 * (size_t)a.top + (a.dwa ? a.depth + 1 : 0)) * 4;
    constexpr int CAP = 200 * 1024;
    if (smem > CAP) return cudaErrorInvalidValue;
    static PerDeviceOnce once;
    cudaError_t le = once.run([] {
        const void* fns[] = {(const void*)combine_kernel<float, 1>, (const void*)combine_kernel<float, 4>, (const void*)combine_kernel<bf16, 1>,
                             (const void*)combine_kernel<bf16, 4>};
        for (const void* f : fns) {
            const cudaError_t e = cudaFuncSetAttribute(f, cudaFuncAttributeMaxDynamicSharedMemorySize, CAP);
            if (e != cudaSuccess) return e;
        }
        return cudaSuccess;
    });
    if (le != cudaSuccess) return le;
    const dim3 grid(n_tok), block(ST_THREADS);
    if (wide_rows(width, a.y ? a.ldy : width, a.gain)) le = a.f32 ? launch_pdl(combine_kernel<float, 4>, grid, block, smem, st, a, width) : launch_pdl(combine_kernel<bf16, 4>, grid, block, smem, st, a, width);
    else le = a.f32 ? launch_pdl(combine_kernel<float, 1>, grid, block, smem, st, a, width) : launch_pdl(combine_kernel<bf16, 1>, grid, block, smem, st, a, width);
    if (le != cudaSuccess) return le;
    return count_launch_and_check();
}

template <typename T, int V>
__global__ void __launch_bounds__(ST_THREADS) row_norm_kernel(const float* __restrict__ x, const int32_t* __restrict__ rows, int width,
                                                              const RowGain gain, float eps, T* __restrict__ out, int ldo) {
    __shared__ float sh[ST_WARPS];
    pdl_wait();
    pdl_trigger();
    const float* xr = x + (int64_t)(rows ? rows[blockIdx.x] : (int)blockIdx.x) * width;
    float ss = 0.f, v[V], g[V];
    for (int c = V * threadIdx.x; c < width; c += V * ST_THREADS) {
        Row<V>::load(xr + c, v);
#pragma unroll
        for (int i = 0; i < V; ++i) ss = fmaf(v[i], v[i], ss);
    }
    const float r = rsqrtf(block_sum<ST_WARPS>(ss, sh) / (float)width + eps);
    for (int c = V * threadIdx.x; c < ldo; c += V * ST_THREADS) {
#pragma unroll
        for (int i = 0; i < V; ++i) v[i] = 0.f;
        if (c < width) {
            Row<V>::load(xr + c, v);
            if (gain.per_coord) Row<V>::load(gain.g + c, g);
#pragma unroll
            for (int i = 0; i < V; ++i) v[i] = v[i] * r * (gain.per_coord ? g[i] : *gain.g);
        }
        Row<V>::store(out + (int64_t)blockIdx.x * ldo + c, v);
    }
}

cudaError_t launch_row_norm(const float* x, const int32_t* rows, int n_rows, int width, const RowGain& gain, float eps, void* out, int ldo, bool f32,
                            cudaStream_t st) {
    if (n_rows == 0) return cudaSuccess;
    const bool wide = wide_rows(width, ldo, gain);
    const dim3 grid(n_rows), block(ST_THREADS);
#define SP_RN(T, V) launch_pdl(row_norm_kernel<T, V>, grid, block, 0, st, x, rows, width, gain, eps, (T*)out, ldo)
    const cudaError_t le = f32 ? (wide ? SP_RN(float, 4) : SP_RN(float, 1)) : (wide ? SP_RN(bf16, 4) : SP_RN(bf16, 1));
#undef SP_RN
    if (le != cudaSuccess) return le;
    return count_launch_and_check();
}

template <typename T>
__global__ void __launch_bounds__(ST_THREADS) tanh_norm_kernel(const float* __restrict__ x, const int32_t* __restrict__ rows, int width, const TanhNorm norm,
                                                               T* __restrict__ out, int ldo) {
    pdl_wait();
    pdl_trigger();
    const float* xr = x + (int64_t)(rows ? rows[blockIdx.x] : (int)blockIdx.x) * width;
    for (int c = threadIdx.x; c < ldo; c += ST_THREADS) out[(int64_t)blockIdx.x * ldo + c] = from_f32<T>(c < width ? tanh_norm(norm, xr[c], c) : 0.f);
}

cudaError_t launch_tanh_norm(const float* x, const int32_t* rows, int n_rows, int width, const TanhNorm& norm, void* out, int ldo, bool f32, cudaStream_t st) {
    if (n_rows == 0) return cudaSuccess;
    const dim3 grid(n_rows), block(ST_THREADS);
    const cudaError_t le = f32 ? launch_pdl(tanh_norm_kernel<float>, grid, block, 0, st, x, rows, width, norm, (float*)out, ldo)
                               : launch_pdl(tanh_norm_kernel<bf16>, grid, block, 0, st, x, rows, width, norm, (bf16*)out, ldo);
    return le != cudaSuccess ? le : count_launch_and_check();
}

// ── experts ──
// Index of the largest of z[0 .. n) that is below `below`, the lower index first; *value is it. Past n: none (or only NaN).
__device__ __forceinline__ int warp_argmax(const float* z, int n, float below, float* value) {
    float v = -INFINITY;
    int at = 0x7FFFFFFF;
    for (int e = threadIdx.x & 31; e < n; e += 32)
        if (z[e] < below && (z[e] > v || (z[e] == v && e < at))) { v = z[e]; at = e; }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
        const float ov = __shfl_xor_sync(0xFFFFFFFFu, v, o);
        const int oa = __shfl_xor_sync(0xFFFFFFFFu, at, o);
        if (ov > v || (ov == v && oa < at)) { v = ov; at = oa; }
    }
    *value = v;
    return at;
}

__host__ __device__ __forceinline__ int route_floats(const RouteShape& r) { return r.experts + (r.keep < r.groups ? r.groups : 0); }

// One warp's choice for a token: its logits (ROUTE_ALL: probabilities) plus bias wait in shared memory (z, route_floats) and a
// chosen one is struck out.
__device__ __forceinline__ void choose_experts(const float* __restrict__ logits, const float* __restrict__ bias, const RouteShape& r, float* z,
                                               int32_t* pick, float* weight) {
    const int lane = threadIdx.x & 31, experts = r.experts, top = r.top;
    float best = -INFINITY, all = 0.f;
    if (r.all) {
        for (int e = lane; e < experts; e += 32) best = fmaxf(best, logits[e]);
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) best = fmaxf(best, __shfl_xor_sync(0xFFFFFFFFu, best, o));
        for (int e = lane; e < experts; e += 32) all += expf(logits[e] - best);
        all = warp_sum(all);
    }
    for (int e = lane; e < experts; e += 32) z[e] = (r.all ? expf(logits[e] - best) / all : logits[e]) + (bias ? bias[e] : 0.f);
    __syncwarp();
    float v;
    if (r.keep < r.groups) {  // a kept group is marked by an infinite score, the experts of the others are struck out
        const int run = experts / r.groups;
        float* gs = z + experts;
        for (int g = lane; g < r.groups; g += 32) {
            float m = -INFINITY;
            for (int e = g * run; e < (g + 1) * run; ++e) m = fmaxf(m, z[e]);
            gs[g] = m;
        }
        __syncwarp();
        for (int k = 0; k < r.keep; ++k) {
            const int at = warp_argmax(gs, r.groups, INFINITY, &v);
            __syncwarp();
            if (lane == 0 && at < r.groups) gs[at] = INFINITY;
            __syncwarp();
        }
        for (int e = lane; e < experts; e += 32)
            if (gs[e / run] != INFINITY) z[e] = -INFINITY;
        __syncwarp();
    }
    float best0 = 0.f, sum = 0.f;
    for (int k = 0; k < top; ++k) {
        int at = warp_argmax(z, experts, INFINITY, &v);
        if (at >= experts) at = k;  // logits that compare with nothing (NaN) still name a valid expert
        if (k == 0) best0 = v;
        const float ex = r.all ? expf(logits[at] - best) / all : expf(v - best0);
        sum += ex;
        __syncwarp();
        if (lane == 0) {
            pick[k] = at;
            weight[k] = ex;
            z[at] = -INFINITY;
        }
        __syncwarp();
    }
    const float norm = r.all ? r.scale / (sum + 1e-20f) : 1.f / sum;
    for (int k = lane; k < top; k += 32) weight[k] *= norm;
}

constexpr int TK_WARPS = 4;
__global__ void __launch_bounds__(TK_WARPS * 32) moe_topk_kernel(const float* __restrict__ logits, int ld, const float* __restrict__ bias, int n_tok,
                                                                 const RouteShape r, int32_t* __restrict__ pick, float* __restrict__ weight) {
    extern __shared__ float tk_smem[];
    pdl_wait();
    pdl_trigger();
    const int warp = threadIdx.x >> 5, t = blockIdx.x * TK_WARPS + warp;
    if (t >= n_tok) return;
    choose_experts(logits + (int64_t)t * ld, bias, r, tk_smem + warp * route_floats(r), pick + (int64_t)t * r.top, weight + (int64_t)t * r.top);
}

// One block: counts per expert, prefix sums, the tables. Within an expert the rows come in no particular order (every row
// is computed by itself and found again through slot_of).
__device__ __forceinline__ void group_rows(const int32_t* pick, int n_pairs, int experts, int top, const MoeTables& t, int* mg_smem) {
    int *cnt = mg_smem, *off = mg_smem + experts;
    for (int e = threadIdx.x; e < experts; e += blockDim.x) cnt[e] = 0;
    __syncthreads();
    for (int i = threadIdx.x; i < n_pairs; i += blockDim.x) atomicAdd(&cnt[pick[i]], 1);
    __syncthreads();
    if (threadIdx.x < 32) {
        // warp scan of (rows, active experts, row tiles), 32 experts at a time
        const int lane = threadIdx.x;
        int rows = 0, act = 0, tiles = 0;
        for (int e0 = 0; e0 < experts; e0 += 32) {
            const int e = e0 + lane, c = e < experts ? cnt[e] : 0;
            int a = c, b = c > 0, d = (c + MOE_TILE - 1) / MOE_TILE;
            const int nt = d;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const int pa = __shfl_up_sync(0xFFFFFFFFu, a, o), pb = __shfl_up_sync(0xFFFFFFFFu, b, o), pd = __shfl_up_sync(0xFFFFFFFFu, d, o);
                if (lane >= o) { a += pa; b += pb; d += pd; }
            }
            if (e < experts) {
                const int begin = rows + a - c;
                off[e] = begin;
                t.row_off[e] = begin;
                if (c > 0) t.active[act + b - 1] = e;
                for (int i = 0; i < nt; ++i) {
                    t.tile_group[tiles + d - nt + i] = e;
                    t.tile_row[tiles + d - nt + i] = begin + i * MOE_TILE;
                }
            }
            rows += __shfl_sync(0xFFFFFFFFu, a, 31);
            act += __shfl_sync(0xFFFFFFFFu, b, 31);
            tiles += __shfl_sync(0xFFFFFFFFu, d, 31);
        }
        if (lane == 0) {
            t.row_off[experts] = rows;
            *t.n_active = act;
            *t.n_tiles = tiles;
        }
    }
    __syncthreads();
    for (int i = threadIdx.x; i < n_pairs; i += blockDim.x) {
        const int at = atomicAdd(&off[pick[i]], 1);
        t.row_src[at] = i / top;
        t.slot_of[i] = at;
    }
}

__global__ void __launch_bounds__(1024) moe_group_kernel(const int32_t* __restrict__ pick, int n_pairs, int experts, int top, const MoeTables t) {
    extern __shared__ int mg_smem[];
    pdl_wait();
    pdl_trigger();
    group_rows(pick, n_pairs, experts, top, t, mg_smem);
}

// Choice and grouping of up to 8 tokens in one block, a warp per token.
__global__ void __launch_bounds__(256) moe_route_kernel(const float* __restrict__ logits, int ld, const float* __restrict__ bias, int n_tok,
                                                         const RouteShape r, float* __restrict__ weight, const MoeTables t) {
    extern __shared__ int mr_smem[];  // counts and offsets, the choices, a row of logits per warp
    pdl_wait();
    pdl_trigger();
    int* pick = mr_smem + 2 * r.experts;
    float* z = reinterpret_cast<float*>(pick + n_tok * r.top);
    const int warp = threadIdx.x >> 5;
    if (warp < n_tok) choose_experts(logits + (int64_t)warp * ld, bias, r, z + warp * route_floats(r), pick + warp * r.top, weight + (int64_t)warp * r.top);
    __syncthreads();
    group_rows(pick, n_tok * r.top, r.experts, r.top, t, mr_smem);
}

cudaError_t launch_moe_route(const float* logits, int ld, const float* bias, const RouteShape& r, int n_tok, int32_t* pick, float* weight,
                             const MoeTables& t, cudaStream_t st) {
    if (n_tok == 0) return cudaSuccess;
    if (r.groups < 1 || r.keep < 1 || r.keep > r.groups || r.experts % r.groups || r.top > r.experts / r.groups * r.keep) return cudaErrorInvalidValue;
    constexpr size_t CAP = 48 * 1024;
    const int experts = r.experts, top = r.top, z = route_floats(r);
    const size_t small = ((size_t)2 * experts + (size_t)n_tok * (z + top)) * 4;
    if (n_tok <= 8 && small <= CAP) {
        const cudaError_t le = launch_pdl(moe_route_kernel, dim3(1), dim3(256), small, st, logits, ld, bias, n_tok, r, weight, t);
        return le != cudaSuccess ? le : count_launch_and_check();
    }
    const size_t rows = (size_t)TK_WARPS * z * 4, counts = (size_t)experts * 8;
    if (rows > CAP || counts > CAP) return cudaErrorInvalidValue;
    cudaError_t le = launch_pdl(moe_topk_kernel, dim3((n_tok + TK_WARPS - 1) / TK_WARPS), dim3(TK_WARPS * 32), rows, st, logits, ld, bias, n_tok, r, pick,
                                weight);
    if (le == cudaSuccess) le = count_launch_and_check();
    if (le != cudaSuccess) return le;
    le = launch_pdl(moe_group_kernel, dim3(1), dim3(1024), counts, st, (const int32_t*)pick, n_tok * top, experts, top, t);
    return le != cudaSuccess ? le : count_launch_and_check();
}

__global__ void gather_act_kernel(const uint4* __restrict__ src, const int32_t* __restrict__ row_src, int ld16, uint4* __restrict__ dst) {
    pdl_wait();
    pdl_trigger();
    const int64_t from = (int64_t)row_src[blockIdx.x] * ld16, to = (int64_t)blockIdx.x * ld16;
    for (int c = threadIdx.x; c < ld16; c += blockDim.x) dst[to + c] = src[from + c];
}

cudaError_t launch_gather_act(const void* src, const int32_t* row_src, int n, int ld, bool f32, void* dst, cudaStream_t st) {
    if (n == 0) return cudaSuccess;
    const int64_t bytes = (int64_t)ld * (f32 ? 4 : 2);
    if (bytes % 16 != 0) return cudaErrorInvalidValue;
    cudaError_t le = launch_pdl(gather_act_kernel, dim3(n), dim3(128), 0, st, (const uint4*)src, row_src, (int)(bytes / 16), (uint4*)dst);
    if (le != cudaSuccess) return le;
    return count_launch_and_check();
}

}  // namespace sp
