// Matrix products on bf16 weights with the 5th-generation tensor cores (tcgen05 + TMEM), for one row or thousands: dense,
// per head or grouped by expert, plain or as the gate / up pair of a gated unit.
//
// y[r, n] = sum_k x[r, k] W[n, k]. A CTA owns 128 weight rows of one matrix (the MMA's M; for a gated unit 128 gate rows
// and the 128 up rows that belong to them, two accumulators) x up to bn activation rows (the MMA's N), over all of K or a
// part of it. Warp 1 lane 0 has TMA fetch, per 64 columns of K, the weight tile(s) and the activation tile into a ring of
// shared-memory stages (128-byte swizzle, both operands K-major; columns past a matrix arrive as zeros, rows past it as
// zeros or as rows nobody stores) — the weights of the first stages before the previous kernel is waited for, since no
// kernel writes weights; warp 0 lane 0 issues four tcgen05.mma per tile and stage and commits them to the stage's `empty`
// mbarrier; four epilogue warps read the accumulators back (one weight row per thread), apply the gated unit or the output
// gate and store with n contiguous across the warp. Two CTAs per SM (256 TMEM columns and 109 KB each), so that one
// CTA's epilogue runs under the other's loads and MMAs.
// Few rows: the same kernel with 16- or 32-row activation tiles is a weight stream (all of a stage's bytes are weights but
// an eighth); K is split over the CTAs of a cluster until the SMs are busy, and they add each other's partial tiles in a fixed
// order through distributed shared memory. Experts of a small step (`gather`) multiply every row of the step, which costs nothing at this
// tile size, and keep the rows that chose them: no gathered copy.
// Every mbarrier wait is bounded; on expiry the kernel raises a flag, still frees its tensor memory and returns.
#include <algorithm>
#include <atomic>
#include <type_traits>

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
constexpr int MT_SMEM = 108 * 1024;        // per CTA, two of which share an SM
constexpr int MT_MAX_PARTS = 8;

__device__ int g_mat_tc5_timeout = 0;

struct MatTc5Seg {
    void* y;
    int64_t ygs;
    int xgs;              // elements between the inputs of consecutive groups
    int ldy, n, kp;
    MatUnit unit;
};
struct MatTc5Args {
    MatTc5Seg seg[2];
    int slots0;           // blockIdx.y below this: seg[0]
    int row_tiles;        // row tiles of a dense or per-head product (blockIdx.y = group * row_tiles + tile)
    int m, bn;            // activation rows, rows per tile (box height)
    int stages, stage_bytes, tmem_cols;
    int parts;            // CTAs (blockIdx.z, one cluster) that share a tile's K range
    bool moe, gather;
    MoeRows rows;
    const float* gate;
    int ldgate;
    int n_outs;
    MatOut outs[MAT_MAX_OUTS];
    float arg[2];
    MatNorm norm;
};

// OUTS: a plain product whose weight rows go where a.outs says (OUT_F32 then has no meaning). NORM: it adds into the stream and
// leaves the norm of the sums, too.
template <bool DUAL, bool OUT_F32, bool OUTS = false, bool NORM = false>
__global__ void __launch_bounds__(MT_THREADS, 2) mat_tc5_kernel(const MatTc5Args a, const __grid_constant__ CUtensorMap map_w0,
                                                             const __grid_constant__ CUtensorMap map_x0, const __grid_constant__ CUtensorMap map_w1,
                                                             const __grid_constant__ CUtensorMap map_x1) {
    extern __shared__ uint8_t mt_smem_raw[];
    __shared__ __align__(8) uint64_t full[MT_MAX_STAGES], empty[MT_MAX_STAGES], done_bar;
    __shared__ uint32_t tmem_slot;
    __shared__ int dest[MAT_GATHER_ROWS];  // gather: output row of each of the step's rows, -1: not this expert's
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int si = (int)blockIdx.y >= a.slots0;
    const MatTc5Seg& s = a.seg[si];
    const int n0 = blockIdx.x * MT_BM;
    const bool grouped = a.moe && si == 0;
    const bool in_range = n0 < s.n;
    // whose tile: known at once unless the routing step decides it
    int g = 0, r0 = 0, rows = 0;
    if (!grouped) {
        const int slot = blockIdx.y - (si ? a.slots0 : 0);
        g = slot / a.row_tiles;
        r0 = (slot - g * a.row_tiles) * a.bn;
        rows = min(a.bn, a.m - r0);
    }
    uint8_t* smem = mt_smem_raw + ((1024u - (tc5_smem_u32(mt_smem_raw) & 1023u)) & 1023u);
    if (warp == 0) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;\n" ::"r"(tc5_smem_u32(&tmem_slot)), "r"(a.tmem_cols) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;\n" ::: "memory");
    }
    if (tid == 32) {
        tc5_prefetch_map(si ? &map_w1 : &map_w0);
        tc5_prefetch_map(si ? &map_x1 : &map_x0);
        for (int i = 0; i < a.stages; ++i) {
            asm volatile("mbarrier.init.shared::cta.b64 [%0], 1;\n" ::"r"(tc5_smem_u32(&full[i])) : "memory");
            asm volatile("mbarrier.init.shared::cta.b64 [%0], 1;\n" ::"r"(tc5_smem_u32(&empty[i])) : "memory");
        }
        asm volatile("mbarrier.init.shared::cta.b64 [%0], 1;\n" ::"r"(tc5_smem_u32(&done_bar)) : "memory");
        asm volatile("fence.mbarrier_init.release.cluster;\n" ::: "memory");
    }
    asm volatile("tcgen05.fence::before_thread_sync;\n" ::: "memory");
    __syncthreads();
    asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
    const uint32_t tmem = tmem_slot;
    const int all_chunks = s.kp / MT_BK, part = blockIdx.z;
    const int c_begin = part * all_chunks / a.parts, n_chunks_all = (part + 1) * all_chunks / a.parts - c_begin;
    const CUtensorMap* mw = si ? &map_w1 : &map_w0;
    const CUtensorMap* mx = si ? &map_x1 : &map_x0;
    constexpr int a_tiles = DUAL ? 2 : 1;
    auto load_w = [&](int c, int st) {  // expects the whole stage, fetches its weight part
        const uint32_t bar = tc5_smem_u32(&full[st]);
        const uint32_t dst = tc5_smem_u32(smem + (size_t)st * a.stage_bytes);
        const int wrow = g * a_tiles * s.n + n0;
        asm volatile("mbarrier.arrive.expect_tx.shared::cta.b64 _, [%0], %1;\n" ::"r"(bar), "r"(a.stage_bytes) : "memory");
        tc5_tma_2d(dst, mw, (c_begin + c) * MT_BK, wrow, bar);
        if (DUAL) tc5_tma_2d(dst + MT_A_BYTES, mw, (c_begin + c) * MT_BK, wrow + s.n, bar);
    };
    const int early = (grouped || !in_range) ? 0 : min(a.stages, n_chunks_all);
    if (warp == 1 && lane == 0)
        for (int c = 0; c < early; ++c) load_w(c, c);
    pdl_wait();
    pdl_trigger();
    bool live = in_range;
    if (grouped) {
        live = live && (int)blockIdx.y < *a.rows.n_tiles;
        if (live) {
            g = a.rows.tile_group[blockIdx.y];
            r0 = a.rows.tile_row[blockIdx.y];
            rows = min(a.bn, a.rows.row_off[g + 1] - r0);
        }
    }
    const bool by_index = grouped && a.gather;
    const int cols = by_index ? a.m : rows;       // activation rows in the tile
    const int nb = (cols + 15) & ~15;
    const int x0 = by_index ? 0 : r0;
    const int n_chunks = live ? n_chunks_all : 0;
    float* const partial = reinterpret_cast<float*>(smem);  // [accumulator][bn columns][128], once the ring has drained
    bool ok = true;
    if (warp == 0) {
        if (lane == 0 && live) {
            const uint32_t idesc = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(nb >> 3) << 17) | ((uint32_t)(MT_BM >> 4) << 24);  // bf16 x bf16 -> f32
            for (int c = 0, st = 0, u = 0; c < n_chunks; ++c, ++st) {
                if (st == a.stages) { st = 0; ++u; }
                ok = ok && tc5_wait(&full[st], (uint32_t)(u & 1));
                if (!ok) break;
                asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
                const uint32_t base = tc5_smem_u32(smem + (size_t)st * a.stage_bytes);
                const uint64_t ad = tc5_desc(base), ad2 = tc5_desc(base + MT_A_BYTES), bd = tc5_desc(base + a_tiles * MT_A_BYTES);
#pragma unroll
                for (int i = 0; i < MT_BK / 16; ++i) {  // 16 columns: 32 bytes inside the swizzle row
                    tc5_mma(tmem, ad + 2u * i, bd + 2u * i, idesc, (uint32_t)(c > 0 || i > 0));
                    if (DUAL) tc5_mma(tmem + (uint32_t)a.bn, ad2 + 2u * i, bd + 2u * i, idesc, (uint32_t)(c > 0 || i > 0));
                }
                tc5_commit(&empty[st]);
            }
            if (ok) tc5_commit(&done_bar);
        }
    } else if (warp == 1) {
        if (lane == 0 && live) {
            for (int c = 0, st = 0, u = 0; c < n_chunks; ++c, ++st) {
                if (st == a.stages) { st = 0; ++u; }
                if (u > 0) ok = ok && tc5_wait(&empty[st], (uint32_t)((u - 1) & 1));
                if (!ok) break;
                if (c >= early) load_w(c, st);
                tc5_tma_2d(tc5_smem_u32(smem + (size_t)st * a.stage_bytes) + a_tiles * MT_A_BYTES, mx, g * s.xgs + (c_begin + c) * MT_BK, x0,
                           tc5_smem_u32(&full[st]));
            }
        }
    } else if (live) {
        const int q4 = warp & 3, n = n0 + 32 * q4 + lane;
        if (by_index) {
            // the four epilogue warps agree on where each of the step's rows goes
            if (warp == 2) {
                dest[lane] = -1;
                __syncwarp();
                for (int j = lane; j < rows; j += 32) dest[a.rows.row_src[r0 + j]] = r0 + j;
            }
            asm volatile("bar.sync 1, 128;\n" ::: "memory");
        }
        ok = tc5_wait(&done_bar, 0u);
        ok = __all_sync(0xFFFFFFFFu, ok);  // one verdict for the warp: the loads below are warp-collective
        asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
        using Out = typename std::conditional<OUT_F32, float, bf16>::type;
        Out* const yn = reinterpret_cast<Out*>(s.y) + (int64_t)g * s.ygs + n;
        // gate: what the output gate's logit of (row, g) is; the callers load a batch of them before the first store
        auto gate_of = [&](int row) { return a.gate[(int64_t)row * a.ldgate + g]; };
        auto finish = [&](int row, float f, float up, float gate) {
            if (DUAL) f = gated_unit(f, up, s.unit);
            if (a.gate) f *= sigmoid_f32(gate);
            yn[(int64_t)row * s.ldy] = from_f32<Out>(f);
        };
        // OUTS: this thread's range
        int act = MAT_ID;
        int64_t oldd = 0;
        float* of = nullptr;   // f32 destination of row 0
        bf16* ob = nullptr;    // or bf16
        bool add = false;
        if (OUTS && n < s.n) {
            int i = 0;
            while (n >= a.outs[i].n_end) ++i;
            const int col = n - (i ? a.outs[i - 1].n_end : 0);
            act = a.outs[i].act;
            oldd = a.outs[i].ldy;
            add = a.outs[i].add;
            if (a.outs[i].f32) of = reinterpret_cast<float*>(a.outs[i].y) + col;
            else ob = reinterpret_cast<bf16*>(a.outs[i].y) + col;
        }
        float norm_w = 0.f, norm_b = 0.f;
        bf16* on = nullptr;
        if (NORM && n < s.n) {
            norm_w = a.norm.fn.w[n];
            norm_b = a.norm.fn.b[n];
            on = reinterpret_cast<bf16*>(a.norm.y) + n;
        }
        auto held = [&](int row) { return add ? of[row * oldd] : 0.f; };
        auto put = [&](int row, float f, float before) {  // (f has been through the activation)
            if (NORM) {
                f += before;
                of[row * oldd] = f;
                on[row * a.norm.ldy] = __float2bfloat16_rn(fmaf(tanh_by_exp(a.norm.fn.alpha * f), norm_w, norm_b));
                return;
            }
            if (of) of[row * oldd] = add ? before + f : f;
            else ob[row * oldd] = __float2bfloat16_rn(f);
        };
        if (ok) {
            const uint32_t lanes = tmem + ((uint32_t)(32 * q4) << 16);
            float* mine = partial + 32 * q4 + lane;
            for (int c = 0; c < nb; c += 16) {
                uint32_t v[16], up[16];
                tc5_ld16(lanes + (uint32_t)c, v);
                if (DUAL) tc5_ld16(lanes + (uint32_t)(a.bn + c), up);
                asm volatile("tcgen05.wait::ld.sync.aligned;\n" ::: "memory");
                if (a.parts > 1) {
#pragma unroll
                    for (int j = 0; j < 16; ++j) {
                        if (c + j >= cols) continue;
                        // (a short K may leave a part without chunks)
                        mine[(c + j) * MT_BM] = n_chunks ? __uint_as_float(v[j]) : 0.f;
                        if (DUAL) mine[(a.bn + c + j) * MT_BM] = n_chunks ? __uint_as_float(up[j]) : 0.f;
                    }
                } else if (OUTS) {
                    if (n < s.n) {
                        float before[16], f[16];
#pragma unroll
                        for (int j = 0; j < 16; ++j) {
                            before[j] = c + j < cols ? held(r0 + c + j) : 0.f;
                            f[j] = __uint_as_float(v[j]);
                        }
                        if (!NORM) mat_act_fast(act, f, a.arg);
#pragma unroll
                        for (int j = 0; j < 16; ++j)
                            if (c + j < cols) put(r0 + c + j, f[j], before[j]);
                    }
                } else if (n < s.n) {
                    if (by_index || a.gate || c + 16 > cols) {
                        int row[16];
                        float gt[16];
#pragma unroll
                        for (int j = 0; j < 16; ++j) {
                            row[j] = c + j < cols ? (by_index ? dest[c + j] : r0 + c + j) : -1;
                            gt[j] = a.gate && row[j] >= 0 ? gate_of(row[j]) : 0.f;
                        }
#pragma unroll
                        for (int j = 0; j < 16; ++j)
                            if (row[j] >= 0) finish(row[j], __uint_as_float(v[j]), DUAL ? __uint_as_float(up[j]) : 0.f, gt[j]);
                    } else {
                        Out* d = yn + (int64_t)(r0 + c) * s.ldy;
#pragma unroll
                        for (int j = 0; j < 16; ++j, d += s.ldy) {
                            float f = __uint_as_float(v[j]);
                            if (DUAL) f = gated_unit(f, __uint_as_float(up[j]), s.unit);
                            *d = from_f32<Out>(f);
                        }
                    }
                }
            }
        }
        if (a.parts > 1) {
            // the cluster's CTAs share out the columns; each adds its columns' partials in part order
            cluster_sync();
            if (n < s.n) {
                constexpr int NC = 4;
                const uint32_t my_row = tc5_smem_u32(partial + 32 * q4 + lane);
                for (int c0 = part; c0 < cols; c0 += NC * a.parts) {
                    int row[NC];
                    float f[NC], up[NC], gt[NC];
#pragma unroll
                    for (int j = 0; j < NC; ++j) {
                        const int c = c0 + j * a.parts;
                        row[j] = c < cols ? (by_index ? dest[c] : r0 + c) : -1;
                        gt[j] = row[j] < 0 ? 0.f : OUTS ? held(row[j]) : a.gate ? gate_of(row[j]) : 0.f;
                        f[j] = up[j] = 0.f;
                    }
#pragma unroll 4
                    for (int p = 0; p < a.parts; ++p) {
                        const uint32_t peer = peer_smem(my_row, p);
#pragma unroll
                        for (int j = 0; j < NC; ++j) {
                            if (row[j] < 0) continue;
                            const int c = c0 + j * a.parts;
                            f[j] += ld_peer(peer + (uint32_t)c * MT_BM * 4);
                            if (DUAL) up[j] += ld_peer(peer + (uint32_t)(a.bn + c) * MT_BM * 4);
                        }
                    }
                    if (OUTS && !NORM) mat_act_fast(act, f, a.arg);
#pragma unroll
                    for (int j = 0; j < NC; ++j)
                        if (row[j] >= 0) {
                            if (OUTS) put(row[j], f[j], gt[j]);
                            else finish(row[j], f[j], up[j], gt[j]);
                        }
                }
            }
        }
    }
    if (a.parts > 1 && live) {
        if (warp < 2) { __syncwarp(); cluster_sync(); }  // the service warps' share of the cluster's first barrier
        cluster_sync();                                  // nobody leaves while its partials are being read
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

// [rows][cols] bf16 with a row stride of ld elements, boxes of 64 columns x box_rows.
static bool mat_map(CUtensorMap* map, const void* p, int64_t cols, int64_t rows, int64_t ld, int box_rows) {
    const PFN_encodeTiled encode = tensor_map_encoder();
    const cuuint64_t dim[2] = {(cuuint64_t)cols, (cuuint64_t)rows}, stride[1] = {(cuuint64_t)ld * 2};
    const cuuint32_t box[2] = {MT_BK, (cuuint32_t)box_rows}, estr[2] = {1u, 1u};
    return encode && encode(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(p), dim, stride, box, estr, CU_TENSOR_MAP_INTERLEAVE_NONE,
                            CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}

cudaError_t launch_mat_tc5(const MatArgs& a, int max_tiles, cudaStream_t st) {
    if (a.m <= 0) return cudaSuccess;
    if (a.f32 || a.nseg < 1 || a.nseg > 2 || (a.nseg == 2 && a.seg[1].groups != 1) || (a.gather && (!a.moe || a.m > MAT_GATHER_ROWS))) return cudaErrorInvalidValue;
    if (!mat_outs_valid(a)) return cudaErrorInvalidValue;
    MatTc5Args k{};
    int n_max = 0, kp_max = 0;
    for (int i = 0; i < a.nseg; ++i) {
        const MatSeg& s = a.seg[i];
        if (s.kp % MAT_KPAD != 0 || s.n <= 0 || s.ldx % 8 != 0 || s.xgs % 8 != 0 || (int64_t)s.groups * s.n * 2 >= (1ll << 31)) return cudaErrorInvalidValue;
        k.seg[i] = MatTc5Seg{s.y, s.ygs, (int)s.xgs, s.ldy, s.n, s.kp, s.unit};
        n_max = std::max(n_max, s.n);
        kp_max = std::max(kp_max, s.kp);
    }
    const int row_blocks = (n_max + MT_BM - 1) / MT_BM, sms = device_sm_count();
    const int groups = a.moe ? 1 : a.seg[0].groups;
    // activation rows per tile: all of a small step, else as many as keep the SMs busy
    int bn = a.m <= 16 ? 16 : a.m <= 32 ? 32 : a.moe ? MOE_TILE : a.dual ? 128 : 256;
    if (!a.moe)
        while (bn > 32 && ((int64_t)row_blocks * groups * ((a.m + bn - 1) / bn) < sms || bn >= 2 * a.m)) bn >>= 1;
    k.bn = bn;
    k.m = a.m;
    k.row_tiles = (a.m + bn - 1) / bn;
    k.slots0 = a.moe ? max_tiles : groups * k.row_tiles;
    const int slots = k.slots0 + (a.nseg == 2 ? k.row_tiles : 0);
    k.moe = a.moe; k.gather = a.gather; k.rows = a.rows; k.gate = a.gate; k.ldgate = a.ldgate;
    k.n_outs = a.n_outs; k.norm = a.norm;
    std::copy(a.arg, a.arg + 2, k.arg);
    std::copy(a.outs, a.outs + MAT_MAX_OUTS, k.outs);
    const int acc = a.dual ? 2 : 1;
    k.stage_bytes = acc * MT_A_BYTES + bn * MT_BK * 2;
    k.tmem_cols = std::max(32, acc * bn);
    k.stages = std::min(MT_MAX_STAGES, MT_SMEM / k.stage_bytes);
    k.parts = 1;
    int64_t busy = 0;  // tiles that exist
    for (int i = 0; i < a.nseg; ++i) busy += (int64_t)((a.seg[i].n + MT_BM - 1) / MT_BM) * (i ? k.row_tiles : k.slots0);
    // a CTA per SM, but no part shorter than four chunks of K
    if (a.m <= 32)
        while (k.parts < MT_MAX_PARTS && busy * k.parts < sms && kp_max / MT_BK >= 8 * k.parts) k.parts *= 2;
    CUtensorMap mw[2], mx[2];
    for (int i = 0; i < a.nseg; ++i) {
        const MatSeg& s = a.seg[i];
        const int64_t x_rows = i == 0 && a.x_rows > 0 ? a.x_rows : a.m;
        if (!mat_map(&mw[i], s.w, s.kp, (int64_t)s.groups * s.n * acc, s.kp, MT_BM) || !mat_map(&mx[i], s.x, s.ldx, x_rows, s.ldx, bn)) return cudaErrorInvalidValue;
    }
    if (a.nseg == 1) { mw[1] = mw[0]; mx[1] = mx[0]; }
    static PerDeviceOnce once;
    cudaError_t le = once.run([] {
        const void* fns[] = {(const void*)mat_tc5_kernel<false, false>, (const void*)mat_tc5_kernel<false, true>, (const void*)mat_tc5_kernel<true, false>,
                             (const void*)mat_tc5_kernel<true, true>, (const void*)mat_tc5_kernel<false, true, true>, (const void*)mat_tc5_kernel<false, true, true, true>};
        for (const void* f : fns) {
            const cudaError_t e = cudaFuncSetAttribute(f, cudaFuncAttributeMaxDynamicSharedMemorySize, MT_SMEM + 1024);
            if (e != cudaSuccess) return e;
        }
        return cudaSuccess;
    });
    if (le != cudaSuccess) return le;
    g_mat_tc5_launched[current_device_index()].store(1);
    const dim3 grid((unsigned)row_blocks, (unsigned)slots, (unsigned)k.parts), block(MT_THREADS);
    const size_t smem = (size_t)(k.stages * k.stage_bytes + 1024);
#define SP_MT(DUAL, F32) le = launch_pdl_cluster(mat_tc5_kernel<DUAL, F32>, grid, block, smem, st, k.parts, k, mw[0], mx[0], mw[1], mx[1])
    if (a.n_outs && a.norm.fn.w) le = launch_pdl_cluster(mat_tc5_kernel<false, true, true, true>, grid, block, smem, st, k.parts, k, mw[0], mx[0], mw[1], mx[1]);
    else if (a.n_outs) le = launch_pdl_cluster(mat_tc5_kernel<false, true, true>, grid, block, smem, st, k.parts, k, mw[0], mx[0], mw[1], mx[1]);
    else if (a.dual) { if (a.out_f32) SP_MT(true, true); else SP_MT(true, false); }
    else { if (a.out_f32) SP_MT(false, true); else SP_MT(false, false); }
#undef SP_MT
    if (le != cudaSuccess) return le;
    return count_launch_and_check();
}

}  // namespace sp
