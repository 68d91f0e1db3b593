// Mixers whose memory is a state matrix per head and sequence (plan_kernels.h, model_plan.h: StateMixerSpec).
//
// A value column j of S never meets another one: S[:, j] <- w . S[:, j] + k (v_j - a (u.S[:, j]) |k|^-1) in the delta rule,
// S[:, j] <- decay S[:, j] + k v_j in the decaying sum, o_j = r . S[:, j]. So L lanes share a column, 4 R keys each in
// registers, and columns spread over warps and blocks. Everything is f32.
//   Step (few rows): a block has a whole head, so gates, recurrence, norm and output gate are one launch; where the norm runs
//   over all heads the blocks of a row are a cluster and exchange their sums of squares. The state is requested before the
//   previous kernel is waited for: no kernel of the last two before this one writes it.
//   Scan (many rows): a block has a few columns of a head and walks the tokens, whose vectors arrive in tiles by cp.async; gates
//   come before and norms after it as kernels of their own.
#include <algorithm>

#include "kernels.h"
#include "model_plan.h"
#include "pdl.cuh"
#include "plan_common.cuh"
#include "plan_kernels.h"

namespace sp {

cudaError_t count_launch_and_check();  // kernels.cu

int state_dim_pad(int dim) {
    int p = 16;
    while (p < dim) p <<= 1;
    return p;
}

// Columns of a projection row.
struct StateCols {
    int r, k, v, a, g;
};
__host__ __device__ __forceinline__ StateCols state_cols(const StateShape& s) {
    const int hd = s.heads * s.dim, hv = s.heads * s.vdim;
    return s.rule == STATE_DELTA ? StateCols{0, hd, 2 * hd, 3 * hd, 4 * hd} : StateCols{0, hd, 2 * hd, 0, 2 * hd + hv};
}

constexpr float EXP_MINUS_HALF = 0.60653065971263342f;
__device__ __forceinline__ float channel_decay(float logit) { return expf(-EXP_MINUS_HALF * sigmoid_f32(logit)); }

template <int L> __device__ __forceinline__ float lanes_sum(float v) {
#pragma unroll
    for (int o = L / 2; o > 0; o >>= 1) v += __shfl_xor_sync(0xFFFFFFFFu, v, o);
    return v;
}
__device__ __forceinline__ void dot4(const float4& a, const float4& b, float4& acc) {
    acc.x = fmaf(a.x, b.x, acc.x);
    acc.y = fmaf(a.y, b.y, acc.y);
    acc.z = fmaf(a.z, b.z, acc.z);
    acc.w = fmaf(a.w, b.w, acc.w);
}

// One token of one column: updates the lane's keys and returns the column's output (the same in its L lanes). Vectors are in
// shared memory, dim_pad floats each.
template <int L, int R, bool DELTA>
__device__ __forceinline__ float state_token(float4 (&st)[R], const float* kv, const float* rv, const float* wv, const float* av, float decay, float v, int l) {
    float4 k[R];
#pragma unroll
    for (int i = 0; i < R; ++i) k[i] = *reinterpret_cast<const float4*>(kv + 4 * (l + L * i));
    if (DELTA) {
        float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int i = 0; i < R; ++i) dot4(k[i], st[i], acc);
        const float d = lanes_sum<L>((acc.x + acc.y) + (acc.z + acc.w));
#pragma unroll
        for (int i = 0; i < R; ++i) {
            const float4 w = *reinterpret_cast<const float4*>(wv + 4 * (l + L * i)), a = *reinterpret_cast<const float4*>(av + 4 * (l + L * i));
            st[i].x = fmaf(k[i].x, fmaf(-a.x, d, v), w.x * st[i].x);
            st[i].y = fmaf(k[i].y, fmaf(-a.y, d, v), w.y * st[i].y);
            st[i].z = fmaf(k[i].z, fmaf(-a.z, d, v), w.z * st[i].z);
            st[i].w = fmaf(k[i].w, fmaf(-a.w, d, v), w.w * st[i].w);
        }
    } else {
#pragma unroll
        for (int i = 0; i < R; ++i) {
            st[i].x = fmaf(k[i].x, v, decay * st[i].x);
            st[i].y = fmaf(k[i].y, v, decay * st[i].y);
            st[i].z = fmaf(k[i].z, v, decay * st[i].z);
            st[i].w = fmaf(k[i].w, v, decay * st[i].w);
        }
    }
    float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int i = 0; i < R; ++i) dot4(*reinterpret_cast<const float4*>(rv + 4 * (l + L * i)), st[i], acc);
    return lanes_sum<L>((acc.x + acc.y) + (acc.z + acc.w));
}

__device__ __forceinline__ float dot_low(const float* w, const float* x, int n, int q) {
    float s = 0.f;
    for (int i = 4 * q; i < n; i += 16) {
        const float4 a = *reinterpret_cast<const float4*>(w + i), b = *reinterpret_cast<const float4*>(x + i);
        s = fmaf(a.x, b.x, fmaf(a.y, b.y, fmaf(a.z, b.z, fmaf(a.w, b.w, s))));
    }
    return s;
}
__device__ __forceinline__ float dot_low(const bf16* w, const bf16* x, int n, int q) {
    float s = 0.f;
    for (int i = 8 * q; i < n; i += 32) {
        const uint4 a = *reinterpret_cast<const uint4*>(w + i), b = *reinterpret_cast<const uint4*>(x + i);
        const uint32_t aw[4] = {a.x, a.y, a.z, a.w}, bw[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const float2 u = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&aw[j])), v = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&bw[j]));
            s = fmaf(u.x, v.x, fmaf(u.y, v.y, s));
        }
    }
    return s;
}

// ── few rows ──
// Block (row, group of hp heads); the groups of a row form a cluster of `cl` where the norm runs over all heads.
template <typename T, int L, int R, bool DELTA>
__global__ void __launch_bounds__(1024) state_step_kernel(const StateArgs a, int n_tok, int hp, int cl) {
    extern __shared__ __align__(16) float ss_smem[];
    __shared__ float cl_sum;
    constexpr int DP = 4 * L * R;
    const int tid = threadIdx.x, lane = tid & 31, t = blockIdx.x, l = tid % L, H = a.s.heads, D = a.s.dim, V = a.s.vdim;
    float *kv = ss_smem, *rv = kv + DP, *wv = rv + DP, *av = wv + DP, *os = DELTA ? av + DP : wv;
    const int mine = lane < n_tok ? a.tok_slot[lane] : -1, slot = __shfl_sync(0xFFFFFFFFu, mine, t);
    uint32_t rows = __ballot_sync(0xFFFFFFFFu, mine == slot);
    if (rows & ((1u << t) - 1)) return;  // an earlier row of this slot has a block that takes this one too
    bool fresh = a.tok_pos[t] == 0;
    const int h0 = blockIdx.z * hp, nh = min(hp, H - h0), per_pass = blockDim.x / L;
    float4 st[R];
    auto at = [&](int h, int col) { return a.state + slot * a.slot_stride + ((int64_t)h * V + col) * DP + 4 * l; };
    auto load = [&](int h, int col) {
#pragma unroll
        for (int i = 0; i < R; ++i) st[i] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (col < V && !fresh) {
            const float* p = at(h, col);
#pragma unroll
            for (int i = 0; i < R; ++i) st[i] = *reinterpret_cast<const float4*>(p + 4 * L * i);
        }
    };
    if (nh > 0) load(h0, tid / L);
    bool ready = true;                               // the registers hold what the next pass needs
    const bool keep = nh == 1 && per_pass >= V;      // one pass: they go on holding it
    pdl_wait();
    pdl_trigger();
    const StateCols co = state_cols(a.s);
    for (; rows; rows &= rows - 1) {
        const int64_t row = __ffs(rows) - 1;
        const float* pr = a.proj + row * a.ldp;
        for (int hh = 0; hh < nh; ++hh) {
            const int h = h0 + hh;
            if (DELTA) {
                float ss = 0.f;
                for (int c = lane; c < D; c += 32) {
                    const float k = pr[co.k + h * D + c];
                    ss = fmaf(k, k, ss);
                }
                const float inv = 1.0f / (warp_sum(ss) + 1e-6f);
                // four lanes to a channel's decay logit
                for (int c0 = 0; c0 < DP; c0 += blockDim.x / 4) {
                    const int c = c0 + tid / 4;
                    float z = 0.f;
                    if (c < D) z = dot_low(reinterpret_cast<const T*>(a.w2) + ((int64_t)h * D + c) * a.ldlow, reinterpret_cast<const T*>(a.low) + row * a.ldlow, a.ldlow, tid & 3);
                    z = lanes_sum<4>(z);
                    if ((tid & 3) == 0 && c < DP) {
                        const bool on = c < D;
                        const int hc = h * D + c;
                        kv[c] = on ? pr[co.k + hc] : 0.f;
                        rv[c] = on ? pr[co.r + hc] : 0.f;
                        wv[c] = on ? channel_decay(z + a.w0[hc]) : 0.f;
                        av[c] = on ? sigmoid_f32(pr[co.a + hc] + a.a_bias[hc]) * inv : 0.f;
                    }
                }
            } else {
                for (int c = tid; c < DP; c += blockDim.x) {
                    kv[c] = c < D ? pr[co.k + h * D + c] : 0.f;
                    rv[c] = c < D ? pr[co.r + h * D + c] : 0.f;
                }
            }
            __syncthreads();
            const float decay = DELTA ? 0.f : a.decay[h];
            for (int c0 = 0; c0 < V; c0 += per_pass) {
                const int col = c0 + tid / L;
                if (!ready) load(h, col);
                ready = keep;
                const float o = state_token<L, R, DELTA>(st, kv, rv, wv, av, decay, col < V ? pr[co.v + h * V + col] : 0.f, l);
                if (col < V) {
                    float* p = at(h, col);
#pragma unroll
                    for (int i = 0; i < R; ++i) *reinterpret_cast<float4*>(p + 4 * L * i) = st[i];
                    if (l == 0) os[hh * V + col] = o;
                }
            }
            __syncthreads();
        }
        // every warp sums the squares for itself
        const int n = max(nh, 0) * V;
        float ss = 0.f;
        for (int i = lane; i < n; i += 32) ss = fmaf(os[i], os[i], ss);
        ss = warp_sum(ss);
        int count = n;
        if (!DELTA) {
            count = H * V;
            if (cl > 1) {
                if (tid == 0) cl_sum = ss;
                cluster_sync();
                ss = 0.f;
                for (int p = 0; p < cl; ++p) ss += ld_peer(peer_smem(smem_addr(&cl_sum), p));
                cluster_sync();
            }
        }
        const float r = rsqrtf(ss / (float)count + a.s.eps);
        T* out = reinterpret_cast<T*>(a.out) + row * a.ldo + (int64_t)h0 * V;
        for (int i = tid; i < n; i += blockDim.x) out[i] = from_f32<T>(os[i] * r * a.gain[h0 * V + i] * sigmoid_f32(pr[co.g + h0 * V + i]));
        __syncthreads();
        fresh = false;
    }
}

constexpr int SS_MAX_CLUSTER = 8;

template <typename T, int L, int R, bool DELTA>
static cudaError_t state_step_launch(const StateArgs& a, int n_tok, cudaStream_t st) {
    int hp = 1, cl = 1;
    if (!DELTA) {
        hp = (a.s.heads + SS_MAX_CLUSTER - 1) / SS_MAX_CLUSTER;
        while (cl < SS_MAX_CLUSTER && cl * hp < a.s.heads) cl <<= 1;
    }
    const int all = L * a.s.vdim, threads = all <= 1024 ? (all + 31) / 32 * 32 : 512;
    const size_t smem = ((size_t)(DELTA ? 4 : 2) * 4 * L * R + (size_t)hp * a.s.vdim) * 4;
    constexpr int CAP = 200 * 1024;
    if (smem > CAP) return cudaErrorInvalidValue;
    static PerDeviceOnce once;
    const cudaError_t le = once.run([] { return cudaFuncSetAttribute(state_step_kernel<T, L, R, DELTA>, cudaFuncAttributeMaxDynamicSharedMemorySize, CAP); });
    if (le != cudaSuccess) return le;
    return launch_pdl_cluster(state_step_kernel<T, L, R, DELTA>, dim3(n_tok, 1, DELTA ? a.s.heads : cl), dim3(threads), smem, st, cl, a, n_tok, hp, cl);
}

cudaError_t launch_state_step(const StateArgs& a, int n_tok, cudaStream_t st) {
    if (n_tok == 0) return cudaSuccess;
    if (n_tok > STATE_STEP_ROWS || a.s.dim > STATE_MAX_DIM || a.s.dim_pad != state_dim_pad(a.s.dim)) return cudaErrorInvalidValue;
    const bool delta = a.s.rule == STATE_DELTA;
    cudaError_t le = cudaErrorInvalidValue;
#define SP_SS(L, R)                                                                                                                    \
    le = a.f32 ? (delta ? state_step_launch<float, L, R, true>(a, n_tok, st) : state_step_launch<float, L, R, false>(a, n_tok, st))       \
               : (delta ? state_step_launch<bf16, L, R, true>(a, n_tok, st) : state_step_launch<bf16, L, R, false>(a, n_tok, st))
    switch (a.s.dim_pad) {
        case 16: SP_SS(4, 1); break;
        case 32: SP_SS(4, 2); break;
        case 64: SP_SS(4, 4); break;
        case 128: SP_SS(8, 4); break;
        case 256: SP_SS(16, 4); break;
        case 512: SP_SS(32, 4); break;
    }
#undef SP_SS
    return le != cudaSuccess ? le : count_launch_and_check();
}

// ── many rows ──
// A warp per (token, head): decays from their logits (in place), removal rates times the key's inverse square length.
constexpr int SG_WARPS = 4;
__global__ void __launch_bounds__(SG_WARPS * 32) state_gates_kernel(const StateArgs a) {
    pdl_wait();
    pdl_trigger();
    const int64_t t = blockIdx.x;
    const int h = blockIdx.y * SG_WARPS + (threadIdx.x >> 5), lane = threadIdx.x & 31, D = a.s.dim;
    if (h >= a.s.heads) return;
    const StateCols co = state_cols(a.s);
    float* pr = a.proj + t * a.ldp + h * D;
    float* wl = a.wlogit + (t * a.s.heads + h) * D;
    float ss = 0.f;
    for (int c = lane; c < D; c += 32) ss = fmaf(pr[co.k + c], pr[co.k + c], ss);
    const float inv = 1.0f / (warp_sum(ss) + 1e-6f);
    for (int c = lane; c < D; c += 32) {
        wl[c] = channel_decay(wl[c] + a.w0[h * D + c]);
        pr[co.a + c] = sigmoid_f32(pr[co.a + c] + a.a_bias[h * D + c]) * inv;
    }
}

// A block per token: norms of the heads (delta) or of all of them together, gain, gate.
constexpr int SN_WARPS = 8;
template <typename T>
__global__ void __launch_bounds__(SN_WARPS * 32) state_norm_kernel(const StateArgs a) {
    __shared__ float sh[SN_WARPS];
    pdl_wait();
    pdl_trigger();
    const int64_t t = blockIdx.x;
    const int H = a.s.heads, V = a.s.vdim, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const float *o = a.o + t * H * V, *g = a.proj + t * a.ldp + state_cols(a.s).g;
    T* out = reinterpret_cast<T*>(a.out) + t * a.ldo;
    auto finish = [&](int i, float r) { out[i] = from_f32<T>(o[i] * r * a.gain[i] * sigmoid_f32(g[i])); };
    if (a.s.rule == STATE_DELTA) {
        for (int h = warp; h < H; h += SN_WARPS) {
            float ss = 0.f;
            for (int i = lane; i < V; i += 32) ss = fmaf(o[h * V + i], o[h * V + i], ss);
            const float r = rsqrtf(warp_sum(ss) / (float)V + a.s.eps);
            for (int i = lane; i < V; i += 32) finish(h * V + i, r);
        }
        return;
    }
    float ss = 0.f;
    for (int i = threadIdx.x; i < H * V; i += SN_WARPS * 32) ss = fmaf(o[i], o[i], ss);
    const float r = rsqrtf(block_sum<SN_WARPS>(ss, sh) / (float)(H * V) + a.s.eps);
    for (int i = threadIdx.x; i < H * V; i += SN_WARPS * 32) finish(i, r);
}

__device__ __forceinline__ void cp_async4(float* dst, const float* src) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;\n" ::"r"(smem_addr(dst)), "l"(src) : "memory");
}

// Block (columns, head, segment). Tiles of tb tokens in two stages: per token the vectors k, r (, w, a) of dim_pad floats and
// the block's values.
constexpr int SC_WARPS = 4, SC_THREADS = SC_WARPS * 32;
template <int L, int R, bool DELTA>
__global__ void __launch_bounds__(SC_THREADS) state_scan_kernel(const StateArgs a, const StateSegment* __restrict__ segs, const int32_t* __restrict__ order, int tb) {
    extern __shared__ __align__(16) float sc_smem[];
    constexpr int DP = 4 * L * R, NV = DELTA ? 4 : 2, COLS = SC_THREADS / L, TOK = NV * DP + COLS;  // floats per token
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, l = tid % L, H = a.s.heads, D = a.s.dim, V = a.s.vdim;
    const int h = blockIdx.y, col0 = blockIdx.x * COLS, col = col0 + tid / L;
    for (int i = tid; i < 2 * tb * TOK; i += SC_THREADS) sc_smem[i] = 0.f;  // the padding stays zero
    pdl_wait();
    pdl_trigger();
    const StateSegment sg = segs[blockIdx.z];
    const StateCols co = state_cols(a.s);
    float* state = a.state + sg.slot * a.slot_stride + ((int64_t)h * V + col) * DP + 4 * l;
    float4 st[R];
#pragma unroll
    for (int i = 0; i < R; ++i) st[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (col < V && !sg.fresh)
#pragma unroll
        for (int i = 0; i < R; ++i) st[i] = *reinterpret_cast<const float4*>(state + 4 * L * i);
    const float decay = DELTA ? 0.f : a.decay[h];
    const bool wide = D % 4 == 0 && a.ldp % 4 == 0, wide_v = wide && V % 4 == 0;
    auto row_of = [&](int i) { return (int64_t)(sg.row0 >= 0 ? sg.row0 + i : order[sg.begin + i]); };
    const int nv = min(COLS, V - col0);
    auto fetch = [&](int i0, int buf) {
        for (int k = warp; k < tb && i0 + k < sg.n; k += SC_WARPS) {
            const int64_t row = row_of(i0 + k);
            const float* pr = a.proj + row * a.ldp;
            float* d = sc_smem + (buf * tb + k) * TOK;
            const float* src[4] = {pr + co.k + h * D, pr + co.r + h * D, DELTA ? a.wlogit + (row * H + h) * D : nullptr, DELTA ? pr + co.a + h * D : nullptr};
            const float* v = pr + co.v + h * V + col0;
#pragma unroll
            for (int q = 0; q < NV; ++q) {
                if (wide)
                    for (int c = 4 * lane; c < D; c += 128) cp_async16(d + q * DP + c, src[q] + c, 16);
                else
                    for (int c = lane; c < D; c += 32) cp_async4(d + q * DP + c, src[q] + c);
            }
            if (wide_v)
                for (int c = 4 * lane; c < nv; c += 128) cp_async16(d + NV * DP + c, v + c, 16);
            else
                for (int c = lane; c < nv; c += 32) cp_async4(d + NV * DP + c, v + c);
        }
    };
    __syncthreads();
    fetch(0, 0);
    cp_async_commit();
    for (int i0 = 0, buf = 0; i0 < sg.n; i0 += tb, buf ^= 1) {
        if (i0 + tb < sg.n) fetch(i0 + tb, buf ^ 1);
        cp_async_commit();
        cp_async_wait<1>();
        __syncthreads();
        const float* d = sc_smem + buf * tb * TOK;
        const int n = min(tb, sg.n - i0);
        for (int k = 0; k < n; ++k, d += TOK) {
            const float o = state_token<L, R, DELTA>(st, d, d + DP, d + 2 * DP, d + 3 * DP, decay, d[NV * DP + tid / L], l);
            if (l == 0 && col < V) a.o[(row_of(i0 + k) * H + h) * V + col] = o;
        }
        __syncthreads();
    }
    cp_async_wait<0>();
    if (col < V)
#pragma unroll
        for (int i = 0; i < R; ++i) *reinterpret_cast<float4*>(state + 4 * L * i) = st[i];
}

template <int L, int R, bool DELTA>
static cudaError_t state_scan_launch(const StateArgs& a, const StateSegment* seg, int n_seg, const int32_t* order, cudaStream_t st) {
    constexpr int COLS = SC_THREADS / L, TOK = (DELTA ? 4 : 2) * 4 * L * R + COLS, CAP = 96 * 1024;
    int tb = 16;
    while (tb > 2 && 2 * tb * TOK * 4 > CAP) tb >>= 1;
    static PerDeviceOnce once;
    const cudaError_t le = once.run([] { return cudaFuncSetAttribute(state_scan_kernel<L, R, DELTA>, cudaFuncAttributeMaxDynamicSharedMemorySize, CAP); });
    if (le != cudaSuccess) return le;
    return launch_pdl(state_scan_kernel<L, R, DELTA>, dim3((a.s.vdim + COLS - 1) / COLS, a.s.heads, n_seg), dim3(SC_THREADS), (size_t)2 * tb * TOK * 4, st, a, seg,
                      order, tb);
}

cudaError_t launch_state_scan(const StateArgs& a, const StateSegment* seg, int n_seg, const int32_t* order, int n_tok, cudaStream_t st) {
    if (n_tok == 0 || n_seg == 0) return cudaSuccess;
    if (a.s.dim > STATE_MAX_DIM || a.s.dim_pad != state_dim_pad(a.s.dim)) return cudaErrorInvalidValue;
    const bool delta = a.s.rule == STATE_DELTA;
    cudaError_t le = cudaSuccess;
    if (delta) {
        le = launch_pdl(state_gates_kernel, dim3(n_tok, (a.s.heads + SG_WARPS - 1) / SG_WARPS), dim3(SG_WARPS * 32), 0, st, a);
        if (le == cudaSuccess) le = count_launch_and_check();
        if (le != cudaSuccess) return le;
    }
    le = cudaErrorInvalidValue;
#define SP_SC(L, R) le = delta ? state_scan_launch<L, R, true>(a, seg, n_seg, order, st) : state_scan_launch<L, R, false>(a, seg, n_seg, order, st)
    switch (a.s.dim_pad) {
        case 16: SP_SC(4, 1); break;
        case 32: SP_SC(4, 2); break;
        case 64: SP_SC(8, 2); break;
        case 128: SP_SC(8, 4); break;
        case 256: SP_SC(16, 4); break;
        case 512: SP_SC(32, 4); break;
    }
#undef SP_SC
    if (le == cudaSuccess) le = count_launch_and_check();
    if (le != cudaSuccess) return le;
    le = a.f32 ? launch_pdl(state_norm_kernel<float>, dim3(n_tok), dim3(SN_WARPS * 32), 0, st, a) : launch_pdl(state_norm_kernel<bf16>, dim3(n_tok), dim3(SN_WARPS * 32), 0, st, a);
    return le != cudaSuccess ? le : count_launch_and_check();
}

}  // namespace sp
