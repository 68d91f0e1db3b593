// Scans of mixers with a state matrix (plan_kernels.h) over many rows on the tensor cores, for engines that compute in bf16:
// chunks of 16 tokens of one sequence, products in 3xTF32 — every f32 operand as a leading TF32 part plus the TF32 of the
// remainder, three products into f32 accumulators, ~2^-20 per product.
//
// Delta rule within a chunk, g_t = w_1 .. w_t (per key channel), S the state before it, rows of U~, R~, K~, B~ being
// g_{t-1} u_t, g_t r_t, k_t / g_t, a_t u_t / g_t (w > 0.54, so g_16 > 5e-5):
//   (I + L) D = U~ S + A V,  O = R~ S + Ark V - Arb D,  S <- g_16 (S + K~^T V - B~^T D)
// with D the values found under the unit keys and L, A, Arb, Ark the lower triangles of U~ B~^T, U~ K~^T (strict), R~ B~^T, R~ K~^T.
// A kernel that is parallel over chunks and heads solves for U = (I + L)^-1 U~, P = (I + L)^-1 A, R = R~ - Arb U, Q = Ark - Arb P,
// which leaves the scan D = U S + P V, O = R S + Q V and the update. The decaying sum and the forget gate have R, Q and K only; a
// gate may forget everything at once, so its products of decays are made without a division, one for each pair of tokens.
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
__host__ __device__ constexpr ChunkRecord chunk_record(bool delta, int dim_pad, int vdim) {
    ChunkRecord c{};
    c.row = dim_pad + 8;
    c.r = delta ? CH * c.row : 0;
    c.k = c.r + CH * c.row;
    c.b = c.k + dim_pad * TS;
    c.p = delta ? c.b + dim_pad * TS : c.b;
    c.q = delta ? c.p + CH * TS : c.p;
    c.g = c.q + CH * TS;
    c.v = c.g + dim_pad;
    c.v_pad = (vdim + 3) & ~3;
    c.floats = c.v + CH * c.v_pad;
    return c;
}
__host__ __device__ __forceinline__ ChunkRecord chunk_record(const StateShape& s) { return chunk_record(s.rule == STATE_DELTA, s.dim_pad, s.vdim); }
StateRecordView state_chunk_view(const StateShape& s) {
    const ChunkRecord c = chunk_record(s);
    return StateRecordView{c.v, c.v_pad, c.floats};
}

// ── what a chunk owes to itself ──
constexpr int CP_THREADS = 128;
__host__ __device__ constexpr int cp_rows(int rule) { return rule == STATE_DELTA ? 4 : rule == STATE_FORGET ? 3 : 2; }
static size_t cp_smem(const StateShape& s) { return ((size_t)cp_rows(s.rule) * CH * (s.dim_pad + 4) + 4 * CH * CH) * 4; }

template <int RULE>
__global__ void __launch_bounds__(CP_THREADS, 6) chunk_prepare_kernel(const StateArgs a, const int32_t* __restrict__ groups) {
    constexpr bool DELTA = RULE == STATE_DELTA, FORGET = RULE == STATE_FORGET;
    extern __shared__ __align__(16) float cp_sm[];
    __shared__ float inv_s[CH], pow_s[CH + 1];
    __shared__ int row_s[CH];
    pdl_wait();
    pdl_trigger();
    const int h = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, D = a.s.dim, DP = a.s.dim_pad, V = a.s.vdim, H = a.s.heads, LD = DP + 4;
    const StateCols co = state_cols(a.s);
    const ChunkRecord rec = chunk_record(a.s);
    float* out = a.rec + ((int64_t)blockIdx.x * H + h) * rec.floats;
    float *rs = cp_sm, *ks = rs + CH * LD, *us = ks + CH * LD, *bs = us + CH * LD;
    float* tri = cp_sm + cp_rows(RULE) * CH * LD;  // Ark, Arb, A, L [CH][CH]
    if (tid < CH) row_s[tid] = groups[(int64_t)blockIdx.x * CH + tid];
    __syncthreads();
    int n = 0;  // tokens of the chunk
#pragma unroll
    for (int t = 0; t < CH; ++t) n += row_s[t] >= 0;
    // r, k, decay and removal logits as they are; the channels and tokens that do not exist: zeros
    const bool wide = D % 4 == 0 && a.ldp % 4 == 0;
    for (int t = warp; t < CH; t += CP_THREADS / 32) {
        const int64_t row = max(row_s[t], 0);
        const float* pr = a.proj + row * a.ldp + h * D;
        const float* src[4] = {pr + co.r, pr + co.k, DELTA ? a.wlogit + (row * H + h) * D : pr + co.a, pr + co.a};
#pragma unroll
        for (int q = 0; q < cp_rows(RULE); ++q) {
            if (FORGET && q == 1) continue;  // the keys follow from the forget logits
            float* d = cp_sm + (q * CH + t) * LD;
            if (wide)
                for (int c = 4 * lane; c < DP; c += 128) cp_async16(d + c, src[q] + min(c, D - 4), t < n && c < D ? 16 : 0);
            else
                for (int c = lane; c < DP; c += 32) d[c] = t < n && c < D ? src[q][c] : 0.f;
        }
    }
    cp_async_commit();
    const bool wide_v = V % 4 == 0 && a.ldp % 4 == 0 && (co.v + h * V) % 4 == 0;
    if (wide_v) {
        for (int i = 4 * tid; i < CH * V; i += 4 * CP_THREADS) {
            const int t = i / V;
            *reinterpret_cast<float4*>(out + rec.v + i) = t < n ? *reinterpret_cast<const float4*>(a.proj + (int64_t)row_s[t] * a.ldp + co.v + h * V + i - t * V) : make_float4(0.f, 0.f, 0.f, 0.f);
        }
    } else {
        for (int i = tid; i < CH * rec.v_pad; i += CP_THREADS) {
            const int t = i / rec.v_pad, c = i - t * rec.v_pad;
            out[rec.v + i] = t < n && c < V ? a.proj[(int64_t)row_s[t] * a.ldp + co.v + h * V + c] : 0.f;
        }
    }
    const float decay = RULE == STATE_DECAY ? a.decay[h] : 0.f;
    if (RULE == STATE_DECAY && tid == 0) {
        pow_s[0] = 1.f;
        for (int i = 0; i < CH; ++i) pow_s[i + 1] = pow_s[i] * decay;
    }
    cp_async_wait<0>();
    __syncthreads();
    if (RULE == STATE_DECAY && (a.s.rot || a.s.key_scale != 1.f)) {
        const int half = a.s.rot / 2, parts = DP - half;  // pairs, then single coordinates
        for (int i = tid; i < CH * parts; i += CP_THREADS) {
            const int t = i / parts, c = i - t * parts;
            float *r = rs + t * LD, *k = ks + t * LD;
            if (t >= n) continue;
            if (c < half) {
                const float2 w = a.cs[(int64_t)a.tok_pos[row_s[t]] * half + c];
                const float ru = r[c], rv = r[c + half], ku = k[c], kv = k[c + half];
                r[c] = ru * w.x - rv * w.y;
                r[c + half] = rv * w.x + ru * w.y;
                k[c] = (ku * w.x - kv * w.y) * a.s.key_scale;
                k[c + half] = (kv * w.x + ku * w.y) * a.s.key_scale;
            } else {
                k[c + half] *= a.s.key_scale;
            }
        }
        __syncthreads();
    }
    if (FORGET) {
        for (int c = tid; c < DP; c += CP_THREADS) {
            const bool on = c < D;
            const int hc = h * D + min(c, D - 1);
            const float bias = a.a_bias[hc], lower = a.lower[hc];
            float g = 1.f;
#pragma unroll 4
            for (int t = 0; t < CH; ++t) {
                const float2 f = on && t < n ? forget_gate(us[t * LD + c] + bias, lower) : make_float2(1.f, 0.f);
                us[t * LD + c] = f.x;
                ks[t * LD + c] = f.y;
                g *= f.x;
                out[rec.r + t * rec.row + c] = rs[t * LD + c] * g;
            }
            out[rec.g + c] = g;
            float after = 1.f;
#pragma unroll
            for (int t = CH - 4; t >= 0; t -= 4) {
                float k[4];
#pragma unroll
                for (int i = 3; i >= 0; --i) {
                    k[i] = ks[(t + i) * LD + c] * after;
                    after *= us[(t + i) * LD + c];
                }
                *reinterpret_cast<float4*>(out + rec.k + c * TS + t) = make_float4(k[0], k[1], k[2], k[3]);
            }
        }
        __syncthreads();
        // thread (s, eighth of the channels): token s's key on its way through the later tokens
        const int s = tid >> 3, c8 = tid & 7;
        float acc[CH];
#pragma unroll
        for (int t = 0; t < CH; ++t) acc[t] = 0.f;
        for (int c = 4 * c8; c < DP; c += 32) {
            float4 p = *reinterpret_cast<const float4*>(ks + s * LD + c);
#pragma unroll
            for (int t = 0; t < CH; ++t) {
                if (t < s) continue;
                if (t > s) {
                    const float4 f = *reinterpret_cast<const float4*>(us + t * LD + c);
                    p.x *= f.x; p.y *= f.y; p.z *= f.z; p.w *= f.w;
                }
                const float4 r = *reinterpret_cast<const float4*>(rs + t * LD + c);
                acc[t] = fmaf(r.x, p.x, fmaf(r.y, p.y, fmaf(r.z, p.z, fmaf(r.w, p.w, acc[t]))));
            }
        }
        // the eight lanes share out the sixteen sums while they make them
#pragma unroll
        for (int m = 4; m > 0; m >>= 1) {
            const bool up = c8 & m;
#pragma unroll
            for (int i = 0; i < 2 * m; ++i) {
                const float send = up ? acc[i] : acc[i + 2 * m], keep = up ? acc[i + 2 * m] : acc[i];
                acc[i] = keep + __shfl_xor_sync(0xFFFFFFFFu, send, m);
            }
        }
#pragma unroll
        for (int i = 0; i < 2; ++i) out[rec.q + (2 * c8 + i) * TS + s] = acc[i];
        return;
    }
    if (DELTA) {
        for (int t = warp; t < CH; t += CP_THREADS / 32) {
            float ss = 0.f;
            for (int c = lane; c < D; c += 32) ss = fmaf(ks[t * LD + c], ks[t * LD + c], ss);
            ss = warp_sum(ss);
            if (lane == 0) inv_s[t] = 1.0f / sqrtf(ss + 1e-6f);
        }
        __syncthreads();
        for (int i = tid; i < CH * DP; i += CP_THREADS) {
            const int t = i / DP, c = i - t * DP, at = t * LD + c;
            const bool live = t < n && c < D;
            us[at] = live ? channel_decay(us[at] + a.w0[h * D + c]) : 1.f;
            bs[at] = live ? ks[at] * inv_s[t] * sigmoid_f32(bs[at] + a.a_bias[h * D + c]) : 0.f;
        }
        __syncthreads();
        for (int c = tid; c < DP; c += CP_THREADS) {
            float g = 1.f;
#pragma unroll 4
            for (int t = 0; t < CH; ++t) {
                const int at = t * LD + c;
                const float before = g, k = ks[at];
                g *= us[at];
                const float back = 1.0f / g;
                us[at] = k * inv_s[t] * before;
                rs[at] *= g;
                ks[at] = k * back;
                bs[at] *= back;
            }
#pragma unroll
            for (int t = 0; t < CH; t += 4) {
                const float *k = ks + t * LD + c, *b = bs + t * LD + c;
                *reinterpret_cast<float4*>(out + rec.k + c * TS + t) = make_float4(k[0] * g, k[LD] * g, k[2 * LD] * g, k[3 * LD] * g);
                *reinterpret_cast<float4*>(out + rec.b + c * TS + t) = make_float4(-b[0] * g, -b[LD] * g, -b[2 * LD] * g, -b[3 * LD] * g);
            }
            out[rec.g + c] = g;
        }
    } else {
        for (int c = tid; c < DP; c += CP_THREADS) {
#pragma unroll
            for (int t = 0; t < CH; t += 4) {
                float k[4];
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    out[rec.r + (t + i) * rec.row + c] = rs[(t + i) * LD + c] * pow_s[t + i + 1];
                    k[i] = ks[(t + i) * LD + c] * pow_s[max(n - 1 - t - i, 0)];
                }
                *reinterpret_cast<float4*>(out + rec.k + c * TS + t) = make_float4(k[0], k[1], k[2], k[3]);
            }
            out[rec.g + c] = pow_s[n];
        }
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
                out[rec.q + t * TS + s] = s <= t ? acc[j][0] * pow_s[t - s] : 0.f;
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
        auto minus = [&](const float* row, int n, float v) {  // v - row[0 .. n) . x
#pragma unroll
            for (int s = 0; s < CH; s += 4) {
                if (s >= n) continue;
                const float4 l = *reinterpret_cast<const float4*>(row + s);
                v = fmaf(-l.x, x[s], v);
                if (s + 1 < n) v = fmaf(-l.y, x[s + 1], v);
                if (s + 2 < n) v = fmaf(-l.z, x[s + 2], v);
                if (s + 3 < n) v = fmaf(-l.w, x[s + 3], v);
            }
            asm volatile("" ::: "memory");  // a row's coefficients at a time
            return v;
        };
#pragma unroll
        for (int t = 0; t < CH; ++t) {
            x[t] = minus(tri + 3 * CH * CH + t * CH, t, key ? us[t * LD + j] : tri[2 * CH * CH + t * CH + p]);
            out[key ? t * rec.row + j : rec.p + t * TS + p] = x[t];
        }
#pragma unroll
        for (int t = 0; t < CH; ++t)
            out[key ? rec.r + t * rec.row + j : rec.q + t * TS + p] = minus(tri + CH * CH + t * CH, t + 1, key ? rs[t * LD + j] : tri[t * CH + p]);
    }
}

// ── the scan ──
// x = hi + lo with hi of TF32's eleven bits; the tensor cores read the leading bits of lo. The A operand's hi is rounded to
// nearest (half a unit added to the bits, then cut), the B operand's just cut.
struct Tf32 {
    uint32_t hi, lo;
};
__device__ __forceinline__ Tf32 parts_of(float v, uint32_t half) {
    const uint32_t hi = (__float_as_uint(v) + half) & 0xFFFFE000u;
    return Tf32{hi, __float_as_uint(v - __uint_as_float(hi))};
}
__device__ __forceinline__ void mma_tf32(float (&c)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
    asm("mma.sync.aligned.m16n8k8.row.col.f32.tf32.tf32.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
        : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
        : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}
// An operand of 16 rows x 8: the accumulator layout (row g: columns 2 tq, 2 tq + 1; row g + 8: the same) serves as the A
// operand when both operands number the columns that way.
struct FragA {
    Tf32 v[4];
};
struct FragB {
    Tf32 v[2];
};
__device__ __forceinline__ FragA frag_of(const float (&c)[4]) {
    return FragA{parts_of(c[0], 0x1000u), parts_of(c[2], 0x1000u), parts_of(c[1], 0x1000u), parts_of(c[3], 0x1000u)};
}
__device__ __forceinline__ FragB frag_at(const float* b) {
    const float2 w = *reinterpret_cast<const float2*>(b);
    return FragB{parts_of(w.x, 0u), parts_of(w.y, 0u)};
}
// N products into accumulators of their own, part by part, so that no product waits for the one before it.
template <int N>
__device__ __forceinline__ void mma3(float (*(&c)[N])[4], const FragA* const (&a)[N], const FragB (&b)[N]) {
#pragma unroll
    for (int i = 0; i < N; ++i) mma_tf32(*c[i], a[i]->v[0].lo, a[i]->v[1].lo, a[i]->v[2].lo, a[i]->v[3].lo, b[i].v[0].hi, b[i].v[1].hi);
#pragma unroll
    for (int i = 0; i < N; ++i) mma_tf32(*c[i], a[i]->v[0].hi, a[i]->v[1].hi, a[i]->v[2].hi, a[i]->v[3].hi, b[i].v[0].lo, b[i].v[1].lo);
#pragma unroll
    for (int i = 0; i < N; ++i) mma_tf32(*c[i], a[i]->v[0].hi, a[i]->v[1].hi, a[i]->v[2].hi, a[i]->v[3].hi, b[i].v[0].hi, b[i].v[1].hi);
}

// Block (16 value columns, head, segment): S^T in the warps' accumulators, a warp having all 16 columns and 8 KT keys. The warps'
// shares of D and O meet in shared memory, once per chunk. Records arrive in a ring of NS stages.
__host__ __device__ constexpr int scan_key_tiles(int dp) { return dp >= 512 ? 8 : dp >= 256 ? 4 : 2; }
__host__ __device__ constexpr int scan_warps(int dp) { return dp / (8 * scan_key_tiles(dp)); }
template <int DP, int NS, bool DELTA>
__global__ void __launch_bounds__(32 * scan_warps(DP)) chunk_scan_kernel(const StateArgs a, const StateSegment* __restrict__ segs) {
    extern __shared__ __align__(16) float cs_sm[];
    constexpr int KT = scan_key_tiles(DP), warps = scan_warps(DP), THREADS = 32 * warps;
    constexpr ChunkRecord rec = chunk_record(DELTA, DP, 0);
    constexpr int stage = rec.v + CH * CVS;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, tq = lane & 3;
    const int H = a.s.heads, V = a.s.vdim, h = blockIdx.y, col0 = blockIdx.x * CV, key0 = warp * 8 * KT;
    const int v_pad = (V + 3) & ~3, floats = rec.v + CH * v_pad;
    float4* const red = reinterpret_cast<float4*>(cs_sm + NS * stage);  // [parity][warp][D, O x two tiles][lane]
    pdl_wait();
    pdl_trigger();
    const StateSegment sg = segs[blockIdx.z];
    float* const first = a.rec + ((int64_t)sg.group0 * H + h) * floats;
    const int64_t step = (int64_t)H * floats;
    const int v_pieces = min(CV, v_pad - col0) / 4;
    for (int i = tid; i < NS * CH * CVS; i += THREADS) cs_sm[(i / (CH * CVS)) * stage + rec.v + i % (CH * CVS)] = 0.f;  // columns past the last
    __syncthreads();
    const uint32_t ring = smem_addr(cs_sm);
    auto fetch = [&](int c, int slot) {
        if (c < sg.n_groups) {
            const float* src = first + c * step;
            const uint32_t d = ring + 4u * (uint32_t)(slot * stage);
#pragma unroll
            for (int i = 0; i < rec.v; i += 4 * THREADS)
                if (i + 4 * THREADS <= rec.v || i + 4 * tid < rec.v) cp_async16_at(d + 4u * (uint32_t)(i + 4 * tid), src + i + 4 * tid, 16);
#pragma unroll
            for (int i = 0; i < CH * (CV / 4); i += THREADS) {
                const int t = (i + tid) / (CV / 4), q = tid % (CV / 4);
                if (t < CH && q < v_pieces) cp_async16_at(d + 4u * (uint32_t)(rec.v + t * CVS + 4 * q), src + rec.v + t * v_pad + col0 + 4 * q, 16);
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
    for (int i = 0; i < (NS > 2 ? NS - 1 : NS); ++i) fetch(i, i);
    cp_async_wait<(NS > 2 ? NS - 2 : NS - 1)>();
    __syncthreads();
    for (int c = 0, slot = 0; c < sg.n_groups; ++c, slot = slot + 1 == NS ? 0 : slot + 1) {
        const float* d = cs_sm + slot * stage;
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
            const float* u = d + g * rec.row + key0 + 8 * i + 2 * tq;
            if (DELTA) {
                float(*c[4])[4] = {&dd[0], &dd[1], &oo[0], &oo[1]};
                const FragA* const x[4] = {&sf, &sf, &sf, &sf};
                const FragB y[4] = {frag_at(u), frag_at(u + 8 * rec.row), frag_at(u + rec.r), frag_at(u + rec.r + 8 * rec.row)};
                mma3(c, x, y);
            } else {
                float(*c[2])[4] = {&oo[0], &oo[1]};
                const FragA* const x[2] = {&sf, &sf};
                const FragB y[2] = {frag_at(u + rec.r), frag_at(u + rec.r + 8 * rec.row)};
                mma3(c, x, y);
            }
        }
#pragma unroll
        for (int w = 0; w < 4; ++w)  // the values' own share: one warp has it
            if (w % warps == warp) {
                const float* p = d + (8 * (w >> 1) + g) * TS + 8 * (w & 1) + 2 * tq;
                if (DELTA) {
                    float(*c[2])[4] = {&dd[w >> 1], &oo[w >> 1]};
                    const FragA* const x[2] = {&v[w & 1], &v[w & 1]};
                    const FragB y[2] = {frag_at(p + rec.p), frag_at(p + rec.q)};
                    mma3(c, x, y);
                } else {
                    float(*c[1])[4] = {&oo[w >> 1]};
                    const FragA* const x[1] = {&v[w & 1]};
                    const FragB y[1] = {frag_at(p + rec.q)};
                    mma3(c, x, y);
                }
            }
#pragma unroll
        for (int n = 0; n < 2; ++n) {
            if (DELTA) rd[warp * 128 + n * 32 + lane] = make_float4(dd[n][0], dd[n][1], dd[n][2], dd[n][3]);
            rd[warp * 128 + (2 + n) * 32 + lane] = make_float4(oo[n][0], oo[n][1], oo[n][2], oo[n][3]);
        }
        // the values' part of the update needs no D
#pragma unroll
        for (int i = 0; i < KT; ++i) {
            const float2 w = *reinterpret_cast<const float2*>(d + rec.g + key0 + 8 * i + 2 * tq);
            s[i][0] *= w.x; s[i][1] *= w.y; s[i][2] *= w.x; s[i][3] *= w.y;
            const float* p = d + rec.k + (key0 + 8 * i + g) * TS + 2 * tq;
            float more[4] = {};
            float(*e[2])[4] = {&s[i], &more};
            const FragA* const x[2] = {&v[0], &v[1]};
            const FragB y[2] = {frag_at(p), frag_at(p + 8)};
            mma3(e, x, y);
#pragma unroll
            for (int q = 0; q < 4; ++q) s[i][q] += more[q];
        }
        if (NS > 2) cp_async_wait<(NS > 3 ? NS - 3 : 0)>();  // the next chunk is there
        __syncthreads();
        if (NS > 2) fetch(c + NS - 1, slot == 0 ? NS - 1 : slot - 1);  // into the stage of the chunk before this one
        auto total = [&](int n) {
            float4 x = rd[n * 32 + lane];
#pragma unroll
            for (int w = 1; w < warps; ++w) {
                const float4 y = rd[w * 128 + n * 32 + lane];
                x.x += y.x; x.y += y.y; x.z += y.z; x.w += y.w;
            }
            return x;
        };
        if (DELTA) {
            FragA df[2];
#pragma unroll
            for (int j = 0; j < 2; ++j) {
                const float4 x = total(j);
                const float q[4] = {x.x, x.y, x.z, x.w};
                df[j] = frag_of(q);
            }
            float back[KT][4] = {};  // the second half of the tokens
#pragma unroll
            for (int i = 0; i < KT; ++i) {
                const float* p = d + rec.b + (key0 + 8 * i + g) * TS + 2 * tq;
                float(*e[2])[4] = {&s[i], &back[i]};
                const FragA* const x[2] = {&df[0], &df[1]};
                const FragB y[2] = {frag_at(p), frag_at(p + 8)};
                mma3(e, x, y);
            }
#pragma unroll
            for (int i = 0; i < KT; ++i)
#pragma unroll
                for (int e = 0; e < 4; ++e) s[i][e] += back[i][e];
        }
        float* const out = first + c * step + rec.v + col0 + g;
        for (int n = warp; n < 2; n += warps) {
            const float4 o = total(2 + n);
            float* p = out + (8 * n + 2 * tq) * v_pad;
            if (on0) { p[0] = o.x; p[v_pad] = o.y; }
            if (on1) { p[8] = o.z; p[v_pad + 8] = o.w; }
        }
        if (NS <= 2) {  // the stage is free once everyone is here
            __syncthreads();
            fetch(c + NS, slot);
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

template <int DP, int NS, bool DELTA>
static cudaError_t chunk_scan_launch(const StateArgs& a, const StateSegment* seg, int n_seg, cudaStream_t st) {
    constexpr int warps = scan_warps(DP), smem = (NS * (chunk_record(DELTA, DP, 0).v + CH * CVS) + 2 * warps * 128 * 4) * 4;
    static_assert(smem <= 220 * 1024, "the ring does not fit");
    static PerDeviceOnce once;
    const cudaError_t le = once.run([] { return cudaFuncSetAttribute(chunk_scan_kernel<DP, NS, DELTA>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem); });
    if (le != cudaSuccess) return le;
    return launch_pdl(chunk_scan_kernel<DP, NS, DELTA>, dim3((a.s.vdim + CV - 1) / CV, a.s.heads, n_seg), dim3(32 * warps), (size_t)smem, st, a, seg);
}

cudaError_t launch_state_chunks(const StateArgs& a, const StateSegment* seg, int n_seg, const int32_t* groups, int n_groups, cudaStream_t st) {
    const bool delta = a.s.rule == STATE_DELTA;
    constexpr int CAP = 160 * 1024;
    static PerDeviceOnce once;
    const auto prepare = a.s.rule == STATE_DELTA ? chunk_prepare_kernel<STATE_DELTA> : a.s.rule == STATE_FORGET ? chunk_prepare_kernel<STATE_FORGET> : chunk_prepare_kernel<STATE_DECAY>;
    cudaError_t le = once.run([] {
        for (const auto f : {chunk_prepare_kernel<STATE_DELTA>, chunk_prepare_kernel<STATE_FORGET>, chunk_prepare_kernel<STATE_DECAY>}) {
            const cudaError_t e = cudaFuncSetAttribute(f, cudaFuncAttributeMaxDynamicSharedMemorySize, CAP);
            if (e != cudaSuccess) return e;
        }
        return cudaSuccess;
    });
    if (le != cudaSuccess) return le;
    const size_t smem = cp_smem(a.s);
    if (smem > CAP) return cudaErrorInvalidValue;
    const dim3 grid(n_groups, a.s.heads), block(CP_THREADS);
    le = launch_pdl(prepare, grid, block, smem, st, a, groups);
    if (le == cudaSuccess) le = count_launch_and_check();
    if (le != cudaSuccess) return le;
    le = cudaErrorInvalidValue;
#define SP_CS(DP, NS) le = delta ? chunk_scan_launch<DP, NS, true>(a, seg, n_seg, st) : chunk_scan_launch<DP, NS, false>(a, seg, n_seg, st)
    switch (a.s.dim_pad) {
        case 16: SP_CS(16, 3); break;
        case 32: SP_CS(32, 3); break;
        case 64: SP_CS(64, 3); break;
        case 128: SP_CS(128, 3); break;
        case 256: SP_CS(256, 2); break;
        case 512: SP_CS(512, 1); break;
    }
#undef SP_CS
    return le != cudaSuccess ? le : count_launch_and_check();
}

}  // namespace sp
