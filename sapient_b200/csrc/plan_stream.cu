// The residual stream of plan-driven models: scaled embedding, norms on a sublayer's output, the mixture of expert
// outputs, depth averages — all in f32, each kernel also leaving the stream in the compute type for the next product —
// and the routing of tokens to experts.
#include "kernels.h"
#include "pdl.cuh"
#include "plan_common.cuh"
#include "plan_kernels.h"

namespace sp {

cudaError_t count_launch_and_check();  // kernels.cu

#define SP_BY_TYPE(f32, K, ...) ((f32) ? launch_pdl(K<float>, __VA_ARGS__) : launch_pdl(K<bf16>, __VA_ARGS__))

constexpr int ST_WARPS = 8, ST_THREADS = 32 * ST_WARPS;

template <typename T>
__global__ void __launch_bounds__(ST_THREADS) embed_scaled_kernel(const T* __restrict__ table, int ldt, const uint32_t* __restrict__ ids, int width,
                                                                  float scale, float* __restrict__ x0, T* __restrict__ xb, int ldb) {
    pdl_wait();
    pdl_trigger();
    const int t = blockIdx.x;
    const T* row = table + (int64_t)ids[t] * ldt;
    for (int c = threadIdx.x; c < ldb; c += ST_THREADS) {
        const float v = c < width ? to_f32(row[c]) * scale : 0.f;
        if (c < width) x0[(int64_t)t * width + c] = v;
        xb[(int64_t)t * ldb + c] = from_f32<T>(v);
    }
}

cudaError_t launch_embed_scaled(const void* table, int ldt, bool f32, const uint32_t* ids, int n_tok, int width, float scale, float* x0, void* xb,
                                int ldb, cudaStream_t st) {
    if (n_tok == 0) return cudaSuccess;
    cudaError_t le = f32 ? launch_pdl(embed_scaled_kernel<float>, dim3(n_tok), dim3(ST_THREADS), 0, st, (const float*)table, ldt, ids, width, scale, x0, (float*)xb, ldb)
                         : launch_pdl(embed_scaled_kernel<bf16>, dim3(n_tok), dim3(ST_THREADS), 0, st, (const bf16*)table, ldt, ids, width, scale, x0, (bf16*)xb, ldb);
    if (le != cudaSuccess) return le;
    return count_launch_and_check();
}

template <typename T>
__global__ void __launch_bounds__(ST_THREADS) norm_residual_kernel(const float* __restrict__ y, int ldy, const float* __restrict__ gain, float eps,
                                                                   const float* x, float* x_out, T* __restrict__ xb, int ldb, int width) {
    __shared__ float sh[ST_WARPS];
    pdl_wait();
    pdl_trigger();
    const int64_t t = blockIdx.x;
    const float* yr = y + t * ldy;
    float ss = 0.f;
    for (int c = threadIdx.x; c < width; c += ST_THREADS) ss = fmaf(yr[c], yr[c], ss);
    const float r = rsqrtf(block_sum<ST_WARPS>(ss, sh) / (float)width + eps) * *gain;
    for (int c = threadIdx.x; c < ldb; c += ST_THREADS) {
        float v = 0.f;
        if (c < width) {
            v = fmaf(yr[c], r, x[t * width + c]);
            x_out[t * width + c] = v;
        }
        xb[t * ldb + c] = from_f32<T>(v);
    }
}

cudaError_t launch_norm_residual(const float* y, int ldy, const float* gain, float eps, const float* x, float* x_out, void* xb, int ldb, bool f32,
                                 int n_tok, int width, cudaStream_t st) {
    if (n_tok == 0) return cudaSuccess;
    cudaError_t le = f32 ? launch_pdl(norm_residual_kernel<float>, dim3(n_tok), dim3(ST_THREADS), 0, st, y, ldy, gain, eps, x, x_out, (float*)xb, ldb, width)
                         : launch_pdl(norm_residual_kernel<bf16>, dim3(n_tok), dim3(ST_THREADS), 0, st, y, ldy, gain, eps, x, x_out, (bf16*)xb, ldb, width);
    if (le != cudaSuccess) return le;
    return count_launch_and_check();
}

// One block per token. The feed-forward's sum lives in shared memory between the two passes over the width.
template <typename T>
__global__ void __launch_bounds__(ST_THREADS) combine_kernel(const CombineArgs a, int width) {
    extern __shared__ float ff[];
    __shared__ float sh[ST_WARPS];
    pdl_wait();
    pdl_trigger();
    const int64_t t = blockIdx.x;
    float r = 0.f;
    if (a.y) {
        const float sg = a.shared_gate ? sigmoid_f32(a.shared_gate[t * a.ld_gate]) : 0.f;
        float ss = 0.f;
        for (int c = threadIdx.x; c < width; c += ST_THREADS) {
            float v = 0.f;
            for (int k = 0; k < a.top; ++k) v = fmaf(a.weight[t * a.top + k], a.y[(int64_t)a.slot_of[t * a.top + k] * a.ldy + c], v);
            if (a.y_shared) v = fmaf(sg, a.y_shared[t * a.ldy + c], v);
            ff[c] = v;
            ss = fmaf(v, v, ss);
        }
        r = rsqrtf(block_sum<ST_WARPS>(ss, sh) / (float)width + a.eps) * *a.gain;
    }
    float* mine = a.history + (int64_t)a.depth * a.hist_stride + t * width;
    for (int c = threadIdx.x; c < a.ldb; c += ST_THREADS) {
        float v = 0.f;
        if (c < width) {
            v = a.x[t * width + c];
            if (a.y) v = fmaf(ff[c], r, v);  // written above by this same thread
            mine[c] = v;
            if (a.dwa) {
                float s = 0.f;
                const float* h = a.history + t * width + c;
#pragma unroll 8
                for (int j = 0; j < a.depth; ++j) s = fmaf(a.dwa[j], h[(int64_t)j * a.hist_stride], s);
                v = fmaf(a.dwa[a.depth], v, s);
            }
            a.x_out[t * width + c] = v;
        }
        reinterpret_cast<T*>(a.xb)[t * a.ldb + c] = from_f32<T>(v);
    }
}

cudaError_t launch_combine(const CombineArgs& a, int n_tok, int width, cudaStream_t st) {
    if (n_tok == 0) return cudaSuccess;
    const size_t smem = a.y ? (size_t)width * 4 : 0;
    if (smem > 200 * 1024) return cudaErrorInvalidValue;
    static PerDeviceOnce once;
    cudaError_t le = once.run([] {
        cudaError_t e = cudaFuncSetAttribute(combine_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
        return e != cudaSuccess ? e : cudaFuncSetAttribute(combine_kernel<bf16>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
    });
    if (le != cudaSuccess) return le;
    le = SP_BY_TYPE(a.f32, combine_kernel, dim3(n_tok), dim3(ST_THREADS), smem, st, a, width);
    if (le != cudaSuccess) return le;
    return count_launch_and_check();
}

template <typename T>
__global__ void __launch_bounds__(ST_THREADS) final_norm_kernel(const float* __restrict__ x, const int32_t* __restrict__ rows, int width,
                                                                const float* __restrict__ gain, float eps, T* __restrict__ out, int ldo) {
    __shared__ float sh[ST_WARPS];
    pdl_wait();
    pdl_trigger();
    const float* xr = x + (int64_t)(rows ? rows[blockIdx.x] : (int)blockIdx.x) * width;
    float ss = 0.f;
    for (int c = threadIdx.x; c < width; c += ST_THREADS) ss = fmaf(xr[c], xr[c], ss);
    const float r = rsqrtf(block_sum<ST_WARPS>(ss, sh) / (float)width + eps) * *gain;
    for (int c = threadIdx.x; c < ldo; c += ST_THREADS) out[(int64_t)blockIdx.x * ldo + c] = from_f32<T>(c < width ? xr[c] * r : 0.f);
}

cudaError_t launch_final_norm(const float* x, const int32_t* rows, int n_rows, int width, const float* gain, float eps, void* out, int ldo, bool f32,
                              cudaStream_t st) {
    if (n_rows == 0) return cudaSuccess;
    cudaError_t le = f32 ? launch_pdl(final_norm_kernel<float>, dim3(n_rows), dim3(ST_THREADS), 0, st, x, rows, width, gain, eps, (float*)out, ldo)
                         : launch_pdl(final_norm_kernel<bf16>, dim3(n_rows), dim3(ST_THREADS), 0, st, x, rows, width, gain, eps, (bf16*)out, ldo);
    if (le != cudaSuccess) return le;
    return count_launch_and_check();
}

// ── experts ──
// One warp per token; the logits wait in shared memory and a chosen one is struck out.
constexpr int TK_WARPS = 4;
__global__ void __launch_bounds__(TK_WARPS * 32) moe_topk_kernel(const float* __restrict__ logits, int ld, const float* __restrict__ bias, int n_tok,
                                                                 int experts, int top, int32_t* __restrict__ pick, float* __restrict__ weight) {
    extern __shared__ float tk_smem[];
    pdl_wait();
    pdl_trigger();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, t = blockIdx.x * TK_WARPS + warp;
    if (t >= n_tok) return;
    float* z = tk_smem + warp * experts;
    for (int e = lane; e < experts; e += 32) z[e] = logits[(int64_t)t * ld + e] + (bias ? bias[e] : 0.f);
    __syncwarp();
    float best0 = 0.f, sum = 0.f;
    for (int k = 0; k < top; ++k) {
        float v = -INFINITY;
        int at = 0x7FFFFFFF;
        for (int e = lane; e < experts; e += 32)
            if (z[e] > v || (z[e] == v && e < at)) { v = z[e]; at = e; }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            const float ov = __shfl_xor_sync(0xFFFFFFFFu, v, o);
            const int oa = __shfl_xor_sync(0xFFFFFFFFu, at, o);
            if (ov > v || (ov == v && oa < at)) { v = ov; at = oa; }
        }
        if (at >= experts) at = k;  // logits that compare with nothing (NaN) still name a valid expert
        if (k == 0) best0 = v;
        const float ex = expf(v - best0);
        sum += ex;
        if (lane == 0) {
            pick[(int64_t)t * top + k] = at;
            weight[(int64_t)t * top + k] = ex;
            z[at] = -INFINITY;
        }
        __syncwarp();
    }
    for (int k = lane; k < top; k += 32) weight[(int64_t)t * top + k] /= sum;
}

cudaError_t launch_moe_topk(const float* logits, int ld, const float* bias, int n_tok, int experts, int top, int32_t* pick, float* weight,
                            cudaStream_t st) {
    if (n_tok == 0) return cudaSuccess;
    const size_t smem = (size_t)TK_WARPS * experts * 4;
    if (smem > 48 * 1024) return cudaErrorInvalidValue;
    cudaError_t le = launch_pdl(moe_topk_kernel, dim3((n_tok + TK_WARPS - 1) / TK_WARPS), dim3(TK_WARPS * 32), smem, st, logits, ld, bias, n_tok, experts,
                                top, pick, weight);
    if (le != cudaSuccess) return le;
    return count_launch_and_check();
}

// One block: counts per expert, prefix sums, the tables. Within an expert the rows come in no particular order (every row
// is computed by itself and found again through slot_of).
__global__ void __launch_bounds__(1024) moe_group_kernel(const int32_t* __restrict__ pick, int n_pairs, int experts, int top, const MoeTables t) {
    extern __shared__ int mg_smem[];
    int *cnt = mg_smem, *off = mg_smem + experts;
    pdl_wait();
    pdl_trigger();
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

cudaError_t launch_moe_group(const int32_t* pick, int n_tok, int experts, int top, const MoeTables& t, cudaStream_t st) {
    if (n_tok == 0) return cudaSuccess;
    const size_t smem = (size_t)experts * 8;
    if (smem > 48 * 1024) return cudaErrorInvalidValue;
    cudaError_t le = launch_pdl(moe_group_kernel, dim3(1), dim3(n_tok * top > 256 ? 1024 : 256), smem, st, pick, n_tok * top, experts, top, t);
    if (le != cudaSuccess) return le;
    return count_launch_and_check();
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
