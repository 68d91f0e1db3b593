// Matrix products on f32 weights (plan-driven models in f32): y[r, n] = sum_k x[r, k] W[n, k], dense, per head or grouped by
// expert, plain or as the gate / up pair of a gated unit. A block owns a 32 x 32 tile; plain fused multiply-adds.
#include "kernels.h"
#include "pdl.cuh"
#include "plan_common.cuh"
#include "plan_kernels.h"

namespace sp {

cudaError_t count_launch_and_check();  // kernels.cu

// Which matrix and rows a block works on. false: nothing to do.
struct MatWork {
    int si, g, r_begin, cnt;
    bool moe;
};
__device__ __forceinline__ bool mat_work(const MatArgs& a, int slot, MatWork& w) {
    const int slots0 = a.moe ? a.slots : a.seg[0].groups;
    if (slot < slots0) {
        w.si = 0;
        w.moe = a.moe;
        if (a.moe) {
            if (slot >= *a.rows.n_active) return false;
            w.g = a.rows.active[slot];
            w.r_begin = a.rows.row_off[w.g];
            w.cnt = a.rows.row_off[w.g + 1] - w.r_begin;
        } else {
            w.g = slot;
            w.r_begin = 0;
            w.cnt = a.m;
        }
    } else {
        w.si = 1;
        w.g = slot - slots0;
        w.moe = false;
        w.r_begin = 0;
        w.cnt = a.m;
    }
    return w.cnt > 0;
}

__device__ __forceinline__ void mat_store(const MatArgs& a, const MatSeg& s, const MatWork& w, int row, int n, float v) {
    if (a.n_outs) {
        int i = 0;
        while (n >= a.outs[i].n_end) ++i;
        float* y = reinterpret_cast<float*>(a.outs[i].y) + row * a.outs[i].ldy + n - (i ? a.outs[i - 1].n_end : 0);
        v = mat_act(a.outs[i].act, v, a.arg);
        if (a.outs[i].add) v += *y;
        *y = v;
        if (a.norm.fn.w) reinterpret_cast<float*>(a.norm.y)[row * a.norm.ldy + n] = tanh_norm(a.norm.fn, v, n);
        return;
    }
    if (a.gate) v *= sigmoid_f32(a.gate[(int64_t)row * a.ldgate + w.g]);
    reinterpret_cast<float*>(s.y)[(int64_t)row * s.ldy + (int64_t)w.g * s.ygs + n] = v;
}

// f32: 32 weight rows x 32 activation rows per block, K in steps of 32.
template <bool DUAL>
__global__ void __launch_bounds__(256) mat_f32_kernel(const MatArgs a) {
    __shared__ float ws[DUAL ? 2 : 1][32][33], xs[32][33];
    pdl_wait();
    pdl_trigger();
    MatWork w;
    if (!mat_work(a, blockIdx.y, w)) return;
    const MatSeg& s = a.seg[w.si];
    const int n0 = blockIdx.x * 32;
    if (n0 >= s.n) return;
    constexpr int D = DUAL ? 2 : 1;
    const float* base = reinterpret_cast<const float*>(s.w) + (int64_t)w.g * D * s.n * s.kp;
    const int tn = threadIdx.x & 31, tr = threadIdx.x >> 5;  // this thread: weight row tn, activation rows tr + 8 i
    for (int c0 = 32 * (int)blockIdx.z; c0 < w.cnt; c0 += 32 * (int)gridDim.z) {
        float acc[D][4] = {};
        for (int k0 = 0; k0 < s.kp; k0 += 32) {
            __syncthreads();
            for (int i = threadIdx.x; i < 32 * 32; i += 256) {
                const int r = i >> 5, k = i & 31;
#pragma unroll
                for (int d = 0; d < D; ++d) ws[d][r][k] = base[((int64_t)d * s.n + min(n0 + r, s.n - 1)) * s.kp + k0 + k];
                const int row = w.r_begin + min(c0 + r, w.cnt - 1);
                const int src = (w.moe && a.gather) ? a.rows.row_src[row] : row;
                xs[r][k] = reinterpret_cast<const float*>(s.x)[(int64_t)src * s.ldx + (int64_t)w.g * s.xgs + k0 + k];
            }
            __syncthreads();
#pragma unroll 8
            for (int k = 0; k < 32; ++k)
#pragma unroll
                for (int d = 0; d < D; ++d) {
                    const float wv = ws[d][tn][k];
#pragma unroll
                    for (int i = 0; i < 4; ++i) acc[d][i] = fmaf(wv, xs[tr + 8 * i][k], acc[d][i]);
                }
        }
        if (n0 + tn < s.n)
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const int c = c0 + tr + 8 * i;
                if (c < w.cnt) mat_store(a, s, w, w.r_begin + c, n0 + tn, DUAL ? gated_unit(acc[0][i], acc[D - 1][i], s.unit) : acc[0][i]);
            }
    }
}

cudaError_t launch_mat_f32(const MatArgs& a, cudaStream_t st) {
    if (a.m <= 0) return cudaSuccess;
    if (!a.f32 || a.nseg < 1 || a.nseg > 2) return cudaErrorInvalidValue;
    if (!mat_outs_valid(a)) return cudaErrorInvalidValue;
    int n_max = 0, slots = a.moe ? a.slots : a.seg[0].groups;
    for (int i = 0; i < a.nseg; ++i) {
        if (a.seg[i].kp % MAT_KPAD != 0 || a.seg[i].n <= 0) return cudaErrorInvalidValue;
        n_max = a.seg[i].n > n_max ? a.seg[i].n : n_max;
    }
    if (a.nseg == 2) slots += a.seg[1].groups;
    const int z = a.m > 32 ? (a.m + 31) / 32 < 64 ? (a.m + 31) / 32 : 64 : 1;
    const dim3 grid((n_max + 31) / 32, slots, z);
    const cudaError_t le = a.dual ? launch_pdl(mat_f32_kernel<true>, grid, dim3(256), 0, st, a) : launch_pdl(mat_f32_kernel<false>, grid, dim3(256), 0, st, a);
    if (le != cudaSuccess) return le;
    return count_launch_and_check();
}

}  // namespace sp
