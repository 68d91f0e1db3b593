// Matrix products of few rows on unquantised weights: y[r, n] = sum_k x[r, k] W[n, k].
//
// bf16: a block of 8 warps owns 16 weight rows of one matrix (dense, one head's, or one expert's) and splits K over its
// warps. The weights are the row operand of mma.sync.m16n8k16, straight from global memory: lane (g, t) of a warp reads
// the 16 bytes of row g (and g + 8) at columns 8 t of a 32-column group — a fixed permutation of the group's columns, the
// same for both operands, so nothing has to be rearranged — and the activations of up to 32 rows are the column operand
// (four 8-row tiles), read the same way through L1. Each weight byte is read once per 32 rows. The warps' partial tiles
// meet in shared memory in warp order.
// f32: a block owns a 32 x 32 tile, plain fused multiply-adds.
#include "kernels.h"
#include "pdl.cuh"
#include "plan_common.cuh"
#include "plan_kernels.h"

namespace sp {

cudaError_t count_launch_and_check();  // kernels.cu

constexpr int MR_WARPS = 8;

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

template <typename T>
__device__ __forceinline__ void mat_store(const MatArgs& a, const MatSeg& s, const MatWork& w, int row, int n, float v) {
    if (a.gate) v *= sigmoid_f32(a.gate[(int64_t)row * a.ldgate + w.g]);
    const int64_t at = (int64_t)row * s.ldy + (int64_t)w.g * s.ygs + n;
    if (a.out_f32) reinterpret_cast<float*>(s.y)[at] = v;
    else reinterpret_cast<T*>(s.y)[at] = from_f32<T>(v);
}

__device__ __forceinline__ uint4 ldg_stream(const bf16* p) {
    uint4 v;
    asm volatile("ld.global.nc.L1::no_allocate.v4.u32 {%0,%1,%2,%3}, [%4];\n" : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w) : "l"(p));
    return v;
}

// One pass over K for NT 8-row tiles of activations.
template <int NT, bool DUAL>
__device__ __forceinline__ void mr_pass(const MatArgs& a, const MatSeg& s, const MatWork& w, const bf16* wr0, const bf16* wr1, int64_t up_off,
                                        int c0, int n0, float* sh) {
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
    const bf16* xp[NT];
#pragma unroll
    for (int j = 0; j < NT; ++j) {
        const int i = w.r_begin + min(c0 + 8 * j + g, w.cnt - 1);
        const int src = (w.moe && a.gather) ? a.rows.row_src[i] : i;
        xp[j] = reinterpret_cast<const bf16*>(s.x) + (int64_t)src * s.ldx + (int64_t)w.g * s.xgs + 8 * t;
    }
    float acc[DUAL ? 2 : 1][NT][4];
#pragma unroll
    for (int d = 0; d < (DUAL ? 2 : 1); ++d)
#pragma unroll
        for (int j = 0; j < NT; ++j) acc[d][j][0] = acc[d][j][1] = acc[d][j][2] = acc[d][j][3] = 0.f;
    constexpr int D = DUAL ? 2 : 1;
    uint4 cur[D][4];
    auto fetch = [&](int k0, uint4 (&q)[D][4]) {
#pragma unroll
        for (int d = 0; d < D; ++d) {
            q[d][0] = ldg_stream(wr0 + d * up_off + k0 + 8 * t);
            q[d][1] = ldg_stream(wr1 + d * up_off + k0 + 8 * t);
            q[d][2] = ldg_stream(wr0 + d * up_off + k0 + 32 + 8 * t);
            q[d][3] = ldg_stream(wr1 + d * up_off + k0 + 32 + 8 * t);
        }
    };
    int k0 = warp * 64;
    if (k0 < s.kp) fetch(k0, cur);
    for (; k0 < s.kp; k0 += MR_WARPS * 64) {
        uint4 nxt[D][4];
        const bool more = k0 + MR_WARPS * 64 < s.kp;
        if (more) fetch(k0 + MR_WARPS * 64, nxt);
#pragma unroll
        for (int h = 0; h < 2; ++h) {
#pragma unroll
            for (int j = 0; j < NT; ++j) {
                const uint4 x = *reinterpret_cast<const uint4*>(xp[j] + k0 + 32 * h);
#pragma unroll
                for (int d = 0; d < D; ++d) {
                    const uint4 p = cur[d][2 * h], r = cur[d][2 * h + 1];
                    mma_bf16(acc[d][j], p.x, r.x, p.y, r.y, x.x, x.y);
                    mma_bf16(acc[d][j], p.z, r.z, p.w, r.w, x.z, x.w);
                }
            }
        }
        if (more) {
#pragma unroll
            for (int d = 0; d < D; ++d)
#pragma unroll
                for (int i = 0; i < 4; ++i) cur[d][i] = nxt[d][i];
        }
    }
    // sh[d][warp][column][16 rows + 1]
    constexpr int COLS = 8 * NT, LD = 17;
#pragma unroll
    for (int d = 0; d < D; ++d)
#pragma unroll
        for (int j = 0; j < NT; ++j) {
            float* p = sh + ((d * MR_WARPS + warp) * COLS + 8 * j + 2 * t) * LD + g;
            p[0] = acc[d][j][0];
            p[LD] = acc[d][j][1];
            p[8] = acc[d][j][2];
            p[LD + 8] = acc[d][j][3];
        }
    __syncthreads();
    for (int i = threadIdx.x; i < COLS * 16; i += MR_WARPS * 32) {
        const int c = i >> 4, r = i & 15;
        if (c0 + c < w.cnt && n0 + r < s.n) {
            float v[D];
#pragma unroll
            for (int d = 0; d < D; ++d) {
                v[d] = 0.f;
#pragma unroll
                for (int q = 0; q < MR_WARPS; ++q) v[d] += sh[((d * MR_WARPS + q) * COLS + c) * LD + r];
            }
            mat_store<bf16>(a, s, w, w.r_begin + c0 + c, n0 + r, DUAL ? clamped_unit(v[0], v[D - 1], s.limit, s.alpha) : v[0]);
        }
    }
    __syncthreads();
}

template <bool DUAL>
__global__ void __launch_bounds__(MR_WARPS * 32) mat_rows_kernel(const MatArgs a) {
    __shared__ float sh[(DUAL ? 2 : 1) * MR_WARPS * 32 * 17 / (DUAL ? 2 : 1)];
    pdl_wait();
    pdl_trigger();
    MatWork w;
    if (!mat_work(a, blockIdx.y, w)) return;
    const MatSeg& s = a.seg[w.si];
    const int n0 = blockIdx.x * 16;
    if (n0 >= s.n) return;
    const int g = (threadIdx.x & 31) >> 2;
    const bf16* base = reinterpret_cast<const bf16*>(s.w) + (int64_t)w.g * (DUAL ? 2 : 1) * s.n * s.kp;
    const bf16* wr0 = base + (int64_t)min(n0 + g, s.n - 1) * s.kp;  // rows past the matrix repeat its last one and are not stored
    const bf16* wr1 = base + (int64_t)min(n0 + g + 8, s.n - 1) * s.kp;
    const int64_t up = (int64_t)s.n * s.kp;
    for (int c0 = 0; c0 < w.cnt;) {
        const int left = w.cnt - c0;
        if (left <= 8) { mr_pass<1, DUAL>(a, s, w, wr0, wr1, up, c0, n0, sh); c0 += 8; }
        else if (left <= 16 || DUAL) { mr_pass<2, DUAL>(a, s, w, wr0, wr1, up, c0, n0, sh); c0 += 16; }
        else { mr_pass<4, DUAL>(a, s, w, wr0, wr1, up, c0, n0, sh); c0 += 32; }
    }
}

// f32: 32 weight rows x 32 activation rows per block, K in steps of 32.
template <bool DUAL>
__global__ void __launch_bounds__(256) mat_rows_f32_kernel(const MatArgs a) {
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
                if (c < w.cnt) mat_store<float>(a, s, w, w.r_begin + c, n0 + tn, DUAL ? clamped_unit(acc[0][i], acc[D - 1][i], s.limit, s.alpha) : acc[0][i]);
            }
    }
}

cudaError_t launch_mat_rows(const MatArgs& a, cudaStream_t st) {
    if (a.m <= 0) return cudaSuccess;
    if (a.nseg < 1 || a.nseg > 2) return cudaErrorInvalidValue;
    int n_max = 0, slots = a.moe ? a.slots : a.seg[0].groups;
    for (int i = 0; i < a.nseg; ++i) {
        if (a.seg[i].kp % MAT_KPAD != 0 || a.seg[i].n <= 0) return cudaErrorInvalidValue;
        n_max = a.seg[i].n > n_max ? a.seg[i].n : n_max;
    }
    if (a.nseg == 2) slots += a.seg[1].groups;
    cudaError_t le;
    if (a.f32) {
        const int z = a.m > 32 ? (a.m + 31) / 32 < 64 ? (a.m + 31) / 32 : 64 : 1;
        const dim3 grid((n_max + 31) / 32, slots, z);
        le = a.dual ? launch_pdl(mat_rows_f32_kernel<true>, grid, dim3(256), 0, st, a) : launch_pdl(mat_rows_f32_kernel<false>, grid, dim3(256), 0, st, a);
    } else {
        const dim3 grid((n_max + 15) / 16, slots);
        le = a.dual ? launch_pdl(mat_rows_kernel<true>, grid, dim3(MR_WARPS * 32), 0, st, a)
                    : launch_pdl(mat_rows_kernel<false>, grid, dim3(MR_WARPS * 32), 0, st, a);
    }
    if (le != cudaSuccess) return le;
    return count_launch_and_check();
}

}  // namespace sp
