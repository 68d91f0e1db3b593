// Many-row matrix products on bf16 weights with the 5th-generation tensor cores (tcgen05 + TMEM), dense or grouped by
// expert, plain or as the gate / up pair of a clamped gated unit.
//
// y[r, n] = sum_k x[r, k] W[n, k]. A CTA owns 128 weight rows (the MMA's M; for a gated unit 128 gate rows and the 128 up
// rows that belong to them, two accumulators) x up to BN activation rows (the MMA's N). Warp 1 lane 0 has TMA fetch, per
// 64 columns of K, the weight tile(s) and the activation tile into a ring of shared-memory stages (128-byte swizzle, both
// operands K-major; columns past a matrix arrive as zeros, rows past it as zeros or as rows nobody stores); warp 0 lane 0
// issues four tcgen05.mma per tile and stage and commits them to the stage's `empty` mbarrier; four epilogue warps read
// the accumulators back (one weight row per thread), apply the gated unit and store with n contiguous across the warp.
// Tiles are kept small enough for two CTAs per SM where that fits (256 TMEM columns and ~100 KB each), so that one CTA's
// epilogue runs under the other's MMAs. Every mbarrier wait is bounded; on expiry the kernel raises a flag, still frees
// its tensor memory and returns.
#include <algorithm>
#include <atomic>

#include "kernels.h"
#include "pdl.cuh"
#include "plan_common.cuh"
#include "plan_kernels.h"
#include "tc5_ptx.cuh"

namespace sp {

cudaError_t count_launch_and_check();  // kernels.cu

constexpr int MT_BM = 128, MT_BK = 64, MT_MAX_STAGES = 6;
constexpr int MT_THREADS = 192;            // MMA warp, TMA warp, four epilogue warps
constexpr int MT_A_BYTES = MT_BM * MT_BK * 2;
constexpr int MT_SMEM_HALF = 100 * 1024;   // two CTAs per SM
constexpr int MT_SMEM_FULL = 200 * 1024;

__device__ int g_mat_tc5_timeout = 0;

struct MatTc5Args {
    void* y;
    int ldy, n, kp, m;
    int bn;               // activation rows per tile (box height)
    int stages, stage_bytes, tmem_cols;
    bool dual, out_f32, moe;
    float limit, alpha;
    MoeRows rows;
};

__global__ void __launch_bounds__(MT_THREADS) mat_tc5_kernel(const MatTc5Args a, const __grid_constant__ CUtensorMap map_w,
                                                             const __grid_constant__ CUtensorMap map_x) {
    extern __shared__ uint8_t mt_smem_raw[];
    __shared__ __align__(8) uint64_t full[MT_MAX_STAGES], empty[MT_MAX_STAGES], done_bar;
    __shared__ uint32_t tmem_slot;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    uint8_t* smem = mt_smem_raw + ((1024u - (tc5_smem_u32(mt_smem_raw) & 1023u)) & 1023u);
    if (warp == 0) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;\n" ::"r"(tc5_smem_u32(&tmem_slot)), "r"(a.tmem_cols) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;\n" ::: "memory");
    }
    if (tid == 0) {
        for (int s = 0; s < a.stages; ++s) {
            asm volatile("mbarrier.init.shared::cta.b64 [%0], 1;\n" ::"r"(tc5_smem_u32(&full[s])) : "memory");
            asm volatile("mbarrier.init.shared::cta.b64 [%0], 1;\n" ::"r"(tc5_smem_u32(&empty[s])) : "memory");
        }
        asm volatile("mbarrier.init.shared::cta.b64 [%0], 1;\n" ::"r"(tc5_smem_u32(&done_bar)) : "memory");
        asm volatile("fence.mbarrier_init.release.cluster;\n" ::: "memory");
    }
    asm volatile("tcgen05.fence::before_thread_sync;\n" ::: "memory");
    __syncthreads();
    asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
    const uint32_t tmem = tmem_slot;
    pdl_wait();
    pdl_trigger();
    // this CTA's tile: weight rows n0.. of matrix g, activation rows r0 .. r0 + rows - 1
    const int n0 = blockIdx.x * MT_BM;
    int g = 0, r0 = blockIdx.y * a.bn, rows;
    bool live = true;
    if (a.moe) {
        live = (int)blockIdx.y < *a.rows.n_tiles;
        if (live) {
            g = a.rows.tile_group[blockIdx.y];
            r0 = a.rows.tile_row[blockIdx.y];
            rows = min(a.bn, a.rows.row_off[g + 1] - r0);
        } else {
            rows = 0;
        }
    } else {
        rows = min(a.bn, a.m - r0);
    }
    const int nb = (rows + 15) & ~15;
    const int n_chunks = live ? a.kp / MT_BK : 0;
    const int64_t wrow = (int64_t)g * (a.dual ? 2 : 1) * a.n + n0;
    bool ok = true;
    if (warp == 0) {
        if (lane == 0 && live) {
            const uint32_t idesc = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(nb >> 3) << 17) | ((uint32_t)(MT_BM >> 4) << 24);  // bf16 x bf16 -> f32
            for (int c = 0, s = 0, u = 0; c < n_chunks; ++c, ++s) {
                if (s == a.stages) { s = 0; ++u; }
                ok = ok && tc5_wait(&full[s], (uint32_t)(u & 1));
                if (!ok) break;
                asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
                const uint32_t st = tc5_smem_u32(smem + (size_t)s * a.stage_bytes);
                const uint64_t ad = tc5_desc(st), ad2 = tc5_desc(st + MT_A_BYTES), bd = tc5_desc(st + (a.dual ? 2 : 1) * MT_A_BYTES);
#pragma unroll
                for (int i = 0; i < MT_BK / 16; ++i) {  // 16 columns: 32 bytes inside the swizzle row
                    tc5_mma(tmem, ad + 2u * i, bd + 2u * i, idesc, (uint32_t)(c > 0 || i > 0));
                    if (a.dual) tc5_mma(tmem + (uint32_t)a.bn, ad2 + 2u * i, bd + 2u * i, idesc, (uint32_t)(c > 0 || i > 0));
                }
                tc5_commit(&empty[s]);
            }
            if (ok) tc5_commit(&done_bar);
        }
    } else if (warp == 1) {
        if (lane == 0 && live) {
            for (int c = 0, s = 0, u = 0; c < n_chunks; ++c, ++s) {
                if (s == a.stages) { s = 0; ++u; }
                if (u > 0) ok = ok && tc5_wait(&empty[s], (uint32_t)((u - 1) & 1));
                if (!ok) break;
                const uint32_t bar = tc5_smem_u32(&full[s]);
                uint32_t dst = tc5_smem_u32(smem + (size_t)s * a.stage_bytes);
                asm volatile("mbarrier.arrive.expect_tx.shared::cta.b64 _, [%0], %1;\n" ::"r"(bar), "r"(a.stage_bytes) : "memory");
                tc5_tma_2d(dst, &map_w, c * MT_BK, (int)wrow, bar);
                dst += MT_A_BYTES;
                if (a.dual) {
                    tc5_tma_2d(dst, &map_w, c * MT_BK, (int)wrow + a.n, bar);
                    dst += MT_A_BYTES;
                }
                tc5_tma_2d(dst, &map_x, c * MT_BK, r0, bar);
            }
        }
    } else if (live) {
        ok = tc5_wait(&done_bar, 0u);
        ok = __all_sync(0xFFFFFFFFu, ok);  // one verdict for the warp: the loads below are warp-collective
        asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
        if (ok) {
            const int q4 = warp & 3, n = n0 + 32 * q4 + lane;
            const uint32_t lanes = tmem + ((uint32_t)(32 * q4) << 16);
            for (int c = 0; c < nb; c += 16) {
                uint32_t v[16], up[16];
                tc5_ld16(lanes + (uint32_t)c, v);
                if (a.dual) tc5_ld16(lanes + (uint32_t)(a.bn + c), up);
                asm volatile("tcgen05.wait::ld.sync.aligned;\n" ::: "memory");
                if (n < a.n) {
#pragma unroll
                    for (int j = 0; j < 16; ++j) {
                        if (c + j < rows) {
                            float f = __uint_as_float(v[j]);
                            if (a.dual) f = clamped_unit(f, __uint_as_float(up[j]), a.limit, a.alpha);
                            const int64_t at = (int64_t)(r0 + c + j) * a.ldy + n;
                            if (a.out_f32) reinterpret_cast<float*>(a.y)[at] = f;
                            else reinterpret_cast<bf16*>(a.y)[at] = __float2bfloat16_rn(f);
                        }
                    }
                }
            }
        }
    }
    if (!ok) atomicExch(&g_mat_tc5_timeout, 1);
    asm volatile("tcgen05.fence::before_thread_sync;\n" ::: "memory");
    __syncthreads();
    if (warp == 0) asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;\n" ::"r"(tmem), "r"(a.tmem_cols) : "memory");
}

static std::atomic<int> g_mat_tc5_launched[SP_MAX_DEVICES];
int mat_tc5_take_timeout() {
    if (g_mat_tc5_launched[current_device_index()].exchange(0) == 0) return 0;
    int flag = 0;
    if (cudaMemcpyFromSymbol(&flag, g_mat_tc5_timeout, sizeof(int)) != cudaSuccess) { cudaGetLastError(); return -1; }
    if (flag) {
        const int zero = 0;
        cudaMemcpyToSymbol(g_mat_tc5_timeout, &zero, sizeof(int));
    }
    return flag ? 1 : 0;
}

bool mat_tc5_supported(const MatArgs& a) {
    const MatSeg& s = a.seg[0];
    return !a.f32 && a.nseg == 1 && !a.gate && !a.gather && (a.moe || s.groups == 1) && s.ldx % 8 == 0 &&
           (reinterpret_cast<uintptr_t>(s.x) & 15) == 0 && (reinterpret_cast<uintptr_t>(s.w) & 15) == 0 &&
           (int64_t)s.groups * s.n * (a.dual ? 2 : 1) < (1ll << 31);
}

cudaError_t launch_mat_tc5(const MatArgs& a, int x_rows, int max_tiles, cudaStream_t st) {
    if (a.m <= 0 || x_rows <= 0) return cudaSuccess;
    if (!mat_tc5_supported(a)) return cudaErrorInvalidValue;
    const MatSeg& s = a.seg[0];
    const int row_tiles = (s.n + MT_BM - 1) / MT_BM;
    MatTc5Args k{};
    // activation rows per tile: as many as keep the SMs busy
    int bn = a.moe ? MOE_TILE : (a.dual ? 128 : 256);
    if (!a.moe)
        while (bn > 32 && ((int64_t)row_tiles * ((a.m + bn - 1) / bn) < device_sm_count() || bn >= 2 * a.m)) bn >>= 1;
    k.y = s.y; k.ldy = s.ldy; k.n = s.n; k.kp = s.kp; k.m = a.m;
    k.bn = bn;
    k.dual = a.dual; k.out_f32 = a.out_f32; k.moe = a.moe; k.limit = s.limit; k.alpha = s.alpha; k.rows = a.rows;
    k.stage_bytes = (a.dual ? 2 : 1) * MT_A_BYTES + bn * MT_BK * 2;
    k.tmem_cols = std::max(32, (a.dual ? 2 : 1) * bn);
    k.stages = std::min(MT_MAX_STAGES, MT_SMEM_HALF / k.stage_bytes);
    const int smem = k.stages * k.stage_bytes + 1024;
    const PFN_encodeTiled encode = tensor_map_encoder();
    if (!encode) return cudaErrorNotSupported;
    CUtensorMap mw, mx;
    const cuuint32_t estr[2] = {1u, 1u};
    {
        const cuuint64_t dim[2] = {(cuuint64_t)s.kp, (cuuint64_t)s.groups * (cuuint64_t)s.n * (a.dual ? 2 : 1)}, stride[1] = {(cuuint64_t)s.kp * 2};
        const cuuint32_t box[2] = {MT_BK, MT_BM};
        if (encode(&mw, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(s.w), dim, stride, box, estr, CU_TENSOR_MAP_INTERLEAVE_NONE,
                   CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) != CUDA_SUCCESS)
            return cudaErrorInvalidValue;
    }
    {
        const cuuint64_t dim[2] = {(cuuint64_t)std::min(s.kp, s.ldx), (cuuint64_t)x_rows}, stride[1] = {(cuuint64_t)s.ldx * 2};
        const cuuint32_t box[2] = {MT_BK, (cuuint32_t)bn};
        if (encode(&mx, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(s.x), dim, stride, box, estr, CU_TENSOR_MAP_INTERLEAVE_NONE,
                   CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_128B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) != CUDA_SUCCESS)
            return cudaErrorInvalidValue;
    }
    static PerDeviceOnce once;
    cudaError_t le = once.run([] { return cudaFuncSetAttribute(mat_tc5_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, MT_SMEM_FULL + 1024); });
    if (le != cudaSuccess) return le;
    g_mat_tc5_launched[current_device_index()].store(1);
    const dim3 grid((unsigned)row_tiles, (unsigned)(a.moe ? max_tiles : (a.m + bn - 1) / bn));
    le = launch_pdl(mat_tc5_kernel, grid, dim3(MT_THREADS), (size_t)smem, st, k, mw, mx);
    if (le != cudaSuccess) return le;
    return count_launch_and_check();
}

}  // namespace sp
