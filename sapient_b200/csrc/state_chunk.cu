// Scans of mixers with a state matrix (plan_kernels.h) over many rows on the tensor cores, for engines that compute in bf16:
// chunks of 16 tokens of one sequence, products in 3xTF32 — every f32 operand as a leading TF32 part plus the TF32 of the
// remainder, three products into f32 accumulators, ~2^-21 per product.
//
// Delta rule within a chunk, g_t = w_1 .. w_t (per key channel), S the state before it, rows of U~, R~, K~, B~ being
// g_{t-1} u_t, g_t r_t, k_t / g_t, a_t u_t / g_t (w > 0.54, so g_16 > 5e-5):
//   (I + L) D = U~ S + A V,  O = R~ S + Ark V - Arb D,  S <- g_16 (S + K~^T V - B~^T D)
// with D the values found under the unit keys and L, A, Arb, Ark the lower triangles of U~ B~^T, U~ K~^T (strict), R~ B~^T, R~ K~^T.
// A kernel that is parallel over chunks and heads solves for U = (I + L)^-1 U~, P = (I + L)^-1 A, R = R~ - Arb U, Q = Ark - Arb P,
// which leaves the scan D = U S + P V, O = R S + Q V and the update. The decaying sum has R, Q and K only.
#include <algorithm>

#include "kernels.h"
#include "model_plan.h"
#include "pdl.cuh"
#include "plan_common.cuh"
#include "plan_kernels.h"
#include "state_common.cuh"

namespace sp {

cudaError_t count_launch_and_check();  // kernels.cu

constexpr int CH = STATE_CHUNK;   // tokens
constexpr int TS = CH + 8;        // row stride of matrices with a token per column: pairs of four rows fall into different banks
constexpr int CV = 16, CVS = 20;  // value columns of a scan block, their row stride in shared memory

// A record per (chunk, head): U, R [CH][row] (delta; the decaying sum has R only), K, -B [dim_pad][TS], P, Q [CH][TS], g [dim_pad],
// values [CH][v_pad], where the scan leaves the outputs.
struct ChunkRecord {
    int row, r, k, b, p, q, g, v, v_pad, floats;
};
__host__ __device__ __forceinline__ ChunkRecord chunk_record(const StateShape& s) {
    ChunkRecord c;
    const bool delta = s.rule == STATE_DELTA;
    c.row = s.dim_pad + 8;
    c.r = delta ? CH * c.row : 0;
    c.k = c.r + CH * c.row;
    c.b = c.k + s.dim_pad * TS;
    c.p = delta ? c.b + s.dim_pad * TS : c.b;
    c.q = delta ? c.p + CH * TS : c.p;
    c.g = c.q + CH * TS;
    c.v = c.g + s.dim_pad;
    c.v_pad = (s.vdim + 3) & ~3;
    c.floats = c.v + CH * c.v_pad;
    return c;
}
StateRecordView state_chunk_view(const StateShape& s) {
    const ChunkRecord c = chunk_record(s);
    return StateRecordView{c.v, c.v_pad, c.floats};
}

// ── what a chunk owes to itself ──
constexpr int CP_THREADS = 128;
static size_t cp_smem(const StateShape& s) { return ((size_t)(s.rule == STATE_DELTA ? 4 : 2) * CH * (s.dim_pad + 4) + 4 * CH * CH) * 4; }

template <bool DELTA>
__global__ void __launch_bounds__(CP_THREADS) chunk_prepare_kernel(const StateArgs a, const int32_t* __restrict__ groups) {
    extern __shared__ __align__(16) float cp_sm[];
    __shared__ float inv_s[CH];
    __shared__ int row_s[CH];
    pdl_wait();
    pdl_trigger();
    const int h = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, D = a.s.dim, DP = a.s.dim_pad, V = a.s.vdim, H = a.s.heads, LD = DP + 4;
    const StateCols co = state_cols(a.s);
    const ChunkRecord rec = chunk_record(a.s);
    float* out = a.rec + ((int64_t)blockIdx.x * H + h) * rec.floats;
    float *rs = cp_sm, *ks = rs + CH * LD, *us = ks + CH * LD, *bs = us + CH * LD;
    float* tri = cp_sm + (DELTA ? 4 : 2) * CH * LD;  // Ark, Arb, A, L [CH][CH]
    if (tid < CH) row_s[tid] = groups[(int64_t)blockIdx.x * CH + tid];
    __syncthreads();
    int n = 0;  // tokens of the chunk
#pragma unroll
    for (int t = 0; t < CH; ++t) n += row_s[t] >= 0;
    if (DELTA) {
        for (int t = warp; t < n; t += CP_THREADS / 32) {
            const float* k = a.proj + (int64_t)row_s[t] * a.ldp + co.k + h * D;
            float ss = 0.f;
            for (int c = lane; c < D; c += 32) ss = fmaf(k[c], k[c], ss);
            ss = warp_sum(ss);
            if (lane == 0) inv_s[t] = 1.0f / sqrtf(ss + 1e-6f);
        }
        __syncthreads();
    }
    const float decay = DELTA ? 0.f : a.decay[h];
    for (int c = tid; c < DP; c += CP_THREADS) {
        const int hc = h * D + c;
        float k[CH], b[CH], g = 1.f;
#pragma unroll
        for (int t = 0; t < CH; ++t) {
            const bool live = c < D && t < n;
            const float* pr = a.proj + (int64_t)(live ? row_s[t] : 0) * a.ldp;
            k[t] = live ? pr[co.k + hc] : 0.f;
            const float r = live ? pr[co.r + hc] : 0.f;
            if (DELTA) {
                const float w = live ? channel_decay(a.wlogit[(int64_t)row_s[t] * H * D + hc] + a.w0[hc]) : 1.f;
                const float u = live ? k[t] * inv_s[t] : 0.f;
                us[t * LD + c] = u * g;
                g *= w;
                const float back = 1.0f / g;
                b[t] = live ? u * sigmoid_f32(pr[co.a + hc] + a.a_bias[hc]) * back : 0.f;
                k[t] *= back;
                bs[t * LD + c] = b[t];
                rs[t * LD + c] = r * g;
                ks[t * LD + c] = k[t];
            } else {
                rs[t * LD + c] = r;
                ks[t * LD + c] = k[t];
                if (t < n) g *= decay;
                out[rec.r + t * rec.row + c] = r * g;
            }
        }
        float f = 1.f;
        if (!DELTA) {  // k_s decay^(n - 1 - s)
#pragma unroll
            for (int t = CH - 1; t >= 0; --t) {
                k[t] *= f;
                if (t < n) f *= decay;
            }
        }
#pragma unroll
        for (int t = 0; t < CH; t += 4) {
            const float m = DELTA ? g : 1.f;
            *reinterpret_cast<float4*>(out + rec.k + c * TS + t) = make_float4(k[t] * m, k[t + 1] * m, k[t + 2] * m, k[t + 3] * m);
            if (DELTA) *reinterpret_cast<float4*>(out + rec.b + c * TS + t) = make_float4(-b[t] * m, -b[t + 1] * m, -b[t + 2] * m, -b[t + 3] * m);
        }
        out[rec.g + c] = g;
    }
    for (int i = tid; i < CH * rec.v_pad; i += CP_THREADS) {
        const int t = i / rec.v_pad, c = i - t * rec.v_pad;
        out[rec.v + i] = t < n && c < V ? a.proj[(int64_t)row_s[t] * a.ldp + co.v + h * V + c] : 0.f;
    }
    __syncthreads();
    // the triangles: thread (t, s and s + 8)
    {
        const int t = tid >> 3, s0 = tid & 7;
        float acc[2][4] = {};
        for (int c = 0; c < DP; c += 4) {
            const float4 r = *reinterpret_cast<const float4*>(rs + t * LD + c);
            float4 u = make_float4(0.f, 0.f, 0.f, 0.f);
            if (DELTA) u = *reinterpret_cast<const float4*>(us + t * LD + c);
#pragma unroll
            for (int j = 0; j < 2; ++j) {
                if (s0 + 8 * j > t) continue;
                const float4 k = *reinterpret_cast<const float4*>(ks + (s0 + 8 * j) * LD + c);
                acc[j][0] = fmaf(r.x, k.x, fmaf(r.y, k.y, fmaf(r.z, k.z, fmaf(r.w, k.w, acc[j][0]))));
                if (DELTA) {
                    const float4 b = *reinterpret_cast<const float4*>(bs + (s0 + 8 * j) * LD + c);
                    acc[j][1] = fmaf(r.x, b.x, fmaf(r.y, b.y, fmaf(r.z, b.z, fmaf(r.w, b.w, acc[j][1]))));
                    acc[j][2] = fmaf(u.x, k.x, fmaf(u.y, k.y, fmaf(u.z, k.z, fmaf(u.w, k.w, acc[j][2]))));
                    acc[j][3] = fmaf(u.x, b.x, fmaf(u.y, b.y, fmaf(u.z, b.z, fmaf(u.w, b.w, acc[j][3]))));
                }
            }
        }
#pragma unroll
        for (int j = 0; j < 2; ++j) {
            const int s = s0 + 8 * j;
            if (!DELTA) {
                float f = s <= t ? acc[j][0] : 0.f;
                for (int i = s; i < t; ++i) f *= decay;
                out[rec.q + t * TS + s] = f;
            } else {
#pragma unroll
                for (int m = 0; m < 4; ++m) tri[m * CH * CH + t * CH + s] = s < t || (m < 2 && s == t) ? acc[j][m] : 0.f;
            }
        }
    }
    if (!DELTA) return;
    __syncthreads();
    // a thread per column of (U | P), then of (R | Q)
    for (int j = tid; j < DP + CH; j += CP_THREADS) {
        const bool key = j < DP;
        const int p = j - DP;
        float x[CH];
#pragma unroll
        for (int t = 0; t < CH; ++t) {
            float v = key ? us[t * LD + j] : tri[2 * CH * CH + t * CH + p];
#pragma unroll
            for (int s = 0; s < t; ++s) v = fmaf(-tri[3 * CH * CH + t * CH + s], x[s], v);
            x[t] = v;
            out[key ? t * rec.row + j : rec.p + t * TS + p] = v;
        }
#pragma unroll
        for (int t = 0; t < CH; ++t) {
            float v = key ? rs[t * LD + j] : tri[t * CH + p];
#pragma unroll
            for (int s = 0; s <= t; ++s) v = fmaf(-tri[CH * CH + t * CH + s], x[s], v);
            out[key ? rec.r + t * rec.row + j : rec.q + t * TS + p] = v;
        }
    }
}

// ── the scan ──
struct Tf32 {
    uint32_t hi, lo;
};
__device__ __forceinline__ uint32_t to_tf32(float v) {
    uint32_t r;
    asm("cvt.rna.tf32.f32 %0, %1;\n" : "=r"(r) : "f"(v));
    return r;
}
__device__ __forceinline__ Tf32 split_tf32(float v) {
    Tf32 s;
    s.hi = to_tf32(v);
    s.lo = to_tf32(v - __uint_as_float(s.hi));
    return s;
}
__device__ __forceinline__ void mma_tf32(float (&c)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k8.row.col.f32.tf32.tf32.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}
// An operand of 16 rows x 8: the accumulator layout (row g: columns 2 tq, 2 tq + 1; row g + 8: the same) serves as the A
// operand when both operands number the columns that way.
struct FragA {
    Tf32 v[4];
};
__device__ __forceinline__ FragA frag_of(const float (&c)[4]) { return FragA{split_tf32(c[0]), split_tf32(c[2]), split_tf32(c[1]), split_tf32(c[3])}; }
__device__ __forceinline__ void mma3(float (&c)[4], const FragA& a, const float* b) {
    const float2 w = *reinterpret_cast<const float2*>(b);
    const Tf32 b0 = split_tf32(w.x), b1 = split_tf32(w.y);
    mma_tf32(c, a.v[0].lo, a.v[1].lo, a.v[2].lo, a.v[3].lo, b0.hi, b1.hi);
    mma_tf32(c, a.v[0].hi, a.v[1].hi, a.v[2].hi, a.v[3].hi, b0.lo, b1.lo);
    mma_tf32(c, a.v[0].hi, a.v[1].hi, a.v[2].hi, a.v[3].hi, b0.hi, b1.hi);
}

// Block (16 value columns, head, segment): S^T in the warps' accumulators, a warp having all 16 columns and 8 KT keys. The warps'
// shares of D and O meet in shared memory, once per chunk. Records arrive in a ring of NS stages.
template <int KT, int NS, bool DELTA>
__global__ void __launch_bounds__(256) chunk_scan_kernel(const StateArgs a, const StateSegment* __restrict__ segs) {
    extern __shared__ __align__(16) float cs_sm[];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, tq = lane & 3, warps = blockDim.x >> 5;
    const int H = a.s.heads, V = a.s.vdim, DP = a.s.dim_pad, h = blockIdx.y, col0 = blockIdx.x * CV, key0 = warp * 8 * KT;
    const ChunkRecord rec = chunk_record(a.s);
    const int stage = rec.v + CH * CVS;
    float4* const red = reinterpret_cast<float4*>(cs_sm + NS * stage);  // [parity][warp][D, O x two tiles][lane]
    pdl_wait();
    pdl_trigger();
    const StateSegment sg = segs[blockIdx.z];
    float* const first = a.rec + ((int64_t)sg.group0 * H + h) * rec.floats;
    const int64_t step = (int64_t)H * rec.floats;
    const int v_pieces = min(CV, rec.v_pad - col0) / 4;
    for (int i = tid; i < NS * CH * CVS; i += blockDim.x) cs_sm[(i / (CH * CVS)) * stage + rec.v + i % (CH * CVS)] = 0.f;  // columns past the last
    __syncthreads();
    auto fetch = [&](int c) {
        if (c < sg.n_groups) {
            const float* src = first + c * step;
            float* d = cs_sm + (c % NS) * stage;
            for (int i = 4 * tid; i < rec.v; i += 4 * blockDim.x) cp_async16(d + i, src + i, 16);
            for (int i = tid; i < CH * (CV / 4); i += blockDim.x) {
                const int t = i / (CV / 4), q = i % (CV / 4);
                if (q < v_pieces) cp_async16(d + rec.v + t * CVS + 4 * q, src + rec.v + t * rec.v_pad + col0 + 4 * q, 16);
            }
        }
        cp_async_commit();
    };
    float* const state = a.state + sg.slot * a.slot_stride + ((int64_t)h * V + col0 + g) * DP + key0 + 2 * tq;
    const bool on0 = col0 + g < V, on1 = col0 + g + 8 < V;
    float s[KT][4];
#pragma unroll
    for (int i = 0; i < KT; ++i) {
        const float2 z = make_float2(0.f, 0.f);
        const float2 x = on0 && !sg.fresh ? *reinterpret_cast<const float2*>(state + 8 * i) : z;
        const float2 y = on1 && !sg.fresh ? *reinterpret_cast<const float2*>(state + (int64_t)8 * DP + 8 * i) : z;
        s[i][0] = x.x; s[i][1] = x.y; s[i][2] = y.x; s[i][3] = y.y;
    }
#pragma unroll
    for (int i = 0; i < (NS > 2 ? NS - 1 : NS); ++i) fetch(i);
    cp_async_wait<(NS > 2 ? NS - 2 : NS - 1)>();
    __syncthreads();
    for (int c = 0; c < sg.n_groups; ++c) {
        const float* d = cs_sm + (c % NS) * stage;
        float4* const rd = red + (c & 1) * warps * 128;
        FragA v[2];  // values of tokens 0 .. 7 and 8 .. 15
#pragma unroll
        for (int j = 0; j < 2; ++j) {
            const float* p = d + rec.v + (8 * j + 2 * tq) * CVS + g;
            const float q[4] = {p[0], p[CVS], p[8], p[CVS + 8]};
            v[j] = frag_of(q);
        }
        float dd[2][4] = {}, oo[2][4] = {};
#pragma unroll
        for (int i = 0; i < KT; ++i) {
            const FragA sf = frag_of(s[i]);
#pragma unroll
            for (int n = 0; n < 2; ++n) {
                const int at = (8 * n + g) * rec.row + key0 + 8 * i + 2 * tq;
                if (DELTA) mma3(dd[n], sf, d + at);
                mma3(oo[n], sf, d + rec.r + at);
            }
        }
#pragma unroll
        for (int u = 0; u < 4; ++u)  // the values' own share: one warp has it
            if (u % warps == warp) {
                const int at = (8 * (u >> 1) + g) * TS + 8 * (u & 1) + 2 * tq;
                if (DELTA) mma3(dd[u >> 1], v[u & 1], d + rec.p + at);
                mma3(oo[u >> 1], v[u & 1], d + rec.q + at);
            }
#pragma unroll
        for (int n = 0; n < 2; ++n) {
            if (DELTA) rd[warp * 128 + n * 32 + lane] = make_float4(dd[n][0], dd[n][1], dd[n][2], dd[n][3]);
            rd[warp * 128 + (2 + n) * 32 + lane] = make_float4(oo[n][0], oo[n][1], oo[n][2], oo[n][3]);
        }
        if (NS > 2) cp_async_wait<(NS > 3 ? NS - 3 : 0)>();  // the next chunk is there
        __syncthreads();
        if (NS > 2) fetch(c + NS - 1);  // into the stage of the chunk before this one
        auto total = [&](int n) {
            float4 x = rd[n * 32 + lane];
            for (int w = 1; w < warps; ++w) {
                const float4 y = rd[w * 128 + n * 32 + lane];
                x.x += y.x; x.y += y.y; x.z += y.z; x.w += y.w;
            }
            return x;
        };
#pragma unroll
        for (int i = 0; i < KT; ++i) {
            const float2 w = *reinterpret_cast<const float2*>(d + rec.g + key0 + 8 * i + 2 * tq);
            s[i][0] *= w.x; s[i][1] *= w.y; s[i][2] *= w.x; s[i][3] *= w.y;
        }
#pragma unroll
        for (int j = 0; j < 2; ++j) {
            FragA df;
            if (DELTA) {
                const float4 x = total(j);
                const float q[4] = {x.x, x.y, x.z, x.w};
                df = frag_of(q);
            }
#pragma unroll
            for (int i = 0; i < KT; ++i) {
                const int at = (key0 + 8 * i + g) * TS + 8 * j + 2 * tq;
                mma3(s[i], v[j], d + rec.k + at);
                if (DELTA) mma3(s[i], df, d + rec.b + at);
            }
        }
        float* const out = first + c * step + rec.v + col0 + g;
        for (int n = warp; n < 2; n += warps) {
            const float4 o = total(2 + n);
            float* p = out + (8 * n + 2 * tq) * rec.v_pad;
            if (on0) { p[0] = o.x; p[rec.v_pad] = o.y; }
            if (on1) { p[8] = o.z; p[rec.v_pad + 8] = o.w; }
        }
        if (NS <= 2) {  // the stage is free once everyone is here
            __syncthreads();
            fetch(c + NS);
            cp_async_wait<NS - 1>();
            __syncthreads();
        }
    }
    cp_async_wait<0>();
#pragma unroll
    for (int i = 0; i < KT; ++i) {
        if (on0) *reinterpret_cast<float2*>(state + 8 * i) = make_float2(s[i][0], s[i][1]);
        if (on1) *reinterpret_cast<float2*>(state + (int64_t)8 * DP + 8 * i) = make_float2(s[i][2], s[i][3]);
    }
}

template <int KT, int NS, bool DELTA>
static cudaError_t chunk_scan_launch(const StateArgs& a, const StateSegment* seg, int n_seg, cudaStream_t st) {
    const int warps = a.s.dim_pad / (8 * KT);
    const size_t smem = ((size_t)NS * (chunk_record(a.s).v + CH * CVS) + 2 * (size_t)warps * 128 * 4) * 4;
    constexpr int CAP = 220 * 1024;
    if (warps < 1 || warps > 8 || smem > CAP) return cudaErrorInvalidValue;
    static PerDeviceOnce once;
    const cudaError_t le = once.run([] { return cudaFuncSetAttribute(chunk_scan_kernel<KT, NS, DELTA>, cudaFuncAttributeMaxDynamicSharedMemorySize, CAP); });
    if (le != cudaSuccess) return le;
    return launch_pdl(chunk_scan_kernel<KT, NS, DELTA>, dim3((a.s.vdim + CV - 1) / CV, a.s.heads, n_seg), dim3(32 * warps), smem, st, a, seg);
}

cudaError_t launch_state_chunks(const StateArgs& a, const StateSegment* seg, int n_seg, const int32_t* groups, int n_groups, cudaStream_t st) {
    const bool delta = a.s.rule == STATE_DELTA;
    constexpr int CAP = 160 * 1024;
    static PerDeviceOnce once;
    cudaError_t le = once.run([] {
        const cudaError_t e = cudaFuncSetAttribute(chunk_prepare_kernel<true>, cudaFuncAttributeMaxDynamicSharedMemorySize, CAP);
        return e != cudaSuccess ? e : cudaFuncSetAttribute(chunk_prepare_kernel<false>, cudaFuncAttributeMaxDynamicSharedMemorySize, CAP);
    });
    if (le != cudaSuccess) return le;
    const size_t smem = cp_smem(a.s);
    if (smem > CAP) return cudaErrorInvalidValue;
    const dim3 grid(n_groups, a.s.heads), block(CP_THREADS);
    le = delta ? launch_pdl(chunk_prepare_kernel<true>, grid, block, smem, st, a, groups) : launch_pdl(chunk_prepare_kernel<false>, grid, block, smem, st, a, groups);
    if (le == cudaSuccess) le = count_launch_and_check();
    if (le != cudaSuccess) return le;
    le = cudaErrorInvalidValue;
#define SP_CS(KT, NS) le = delta ? chunk_scan_launch<KT, NS, true>(a, seg, n_seg, st) : chunk_scan_launch<KT, NS, false>(a, seg, n_seg, st)
    switch (a.s.dim_pad) {
        case 16: case 32: case 64: SP_CS(2, 4); break;
        case 128: SP_CS(2, 3); break;
        case 256: SP_CS(4, 2); break;
        case 512: SP_CS(8, 1); break;
    }
#undef SP_CS
    return le != cudaSuccess ? le : count_launch_and_check();
}

}  // namespace sp
