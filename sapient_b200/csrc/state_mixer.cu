// Mixers whose memory is a state matrix per head and sequence (plan_kernels.h, model_plan.h: StateMixerSpec).
//
// A value column j of S never meets another one: S[:, j] <- w . S[:, j] + k (v_j - a (u.S[:, j]) |k|^-1) in the delta rule,
// S[:, j] <- decay S[:, j] + k v_j in the decaying sum, S[:, j] <- f . S[:, j] + (1 - f) v_j with a forget gate, o_j = r . S[:, j]. So L lanes share a column, 4 R keys each in
// registers, and columns spread over warps and blocks. Everything is f32.
//   Step (few rows): a block has a whole head, so gates, recurrence, norm and output gate are one launch; where the norm runs
//   over all heads the blocks of a row are a cluster and exchange their sums of squares. The state is requested before the
//   previous kernel is waited for: no kernel of the last two before this one writes it.
//   Scan (many rows): gates and what a group of four tokens owes to itself are made in parallel, then a block with a few columns
//   of a head walks the groups, then come norm and output gate.
#include <algorithm>

#include "kernels.h"
#include "model_plan.h"
#include "pdl.cuh"
#include "plan_common.cuh"
#include "plan_kernels.h"
#include "state_common.cuh"

namespace sp {

cudaError_t count_launch_and_check();  // kernels.cu

int state_dim_pad(int dim) {
    int p = 16;
    while (p < dim) p <<= 1;
    return p;
}

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
template <int L, int R, int RULE>
__device__ __forceinline__ float state_token(float4 (&st)[R], const float* kv, const float* rv, const float* wv, const float* av, float decay, float v, int l) {
    float4 k[R];
#pragma unroll
    for (int i = 0; i < R; ++i) k[i] = *reinterpret_cast<const float4*>(kv + 4 * (l + L * i));
    if (RULE == STATE_DELTA) {
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
            float4 w = make_float4(decay, decay, decay, decay);
            if (RULE == STATE_FORGET) w = *reinterpret_cast<const float4*>(wv + 4 * (l + L * i));
            st[i].x = fmaf(k[i].x, v, w.x * st[i].x);
            st[i].y = fmaf(k[i].y, v, w.y * st[i].y);
            st[i].z = fmaf(k[i].z, v, w.z * st[i].z);
            st[i].w = fmaf(k[i].w, v, w.w * st[i].w);
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
// Block (row, group of hp heads); the groups of a row form a cluster of `cl` where the norm runs over all heads, else hp is one.
__host__ __device__ constexpr int step_vectors(int rule) { return rule == STATE_DELTA ? 4 : rule == STATE_FORGET ? 3 : 2; }
template <typename T, int L, int R, int RULE>
__global__ void __launch_bounds__(1024) state_step_kernel(const StateArgs a, int n_tok, int hp, int cl) {
    extern __shared__ __align__(16) float ss_smem[];
    __shared__ float cl_sum;
    constexpr int DP = 4 * L * R;
    constexpr bool DELTA = RULE == STATE_DELTA;
    const int tid = threadIdx.x, lane = tid & 31, t = blockIdx.x, l = tid % L, H = a.s.heads, D = a.s.dim, V = a.s.vdim;
    float *kv = ss_smem, *rv = kv + DP, *wv = rv + DP, *av = wv + DP, *os = ss_smem + step_vectors(RULE) * DP;
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
        // what the outputs are multiplied by after the norm, as far as there is a thread for each: ahead of the recurrence
        const int n = max(nh, 0) * V;
        const float factor = tid < n ? state_factor(a, pr + co.g, h0 * V + tid) : 0.f;
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
            } else if (RULE == STATE_FORGET) {
                for (int c = tid; c < DP; c += blockDim.x) {
                    const int hc = h * D + c;
                    const float2 f = c < D ? forget_gate(pr[co.a + hc] + a.a_bias[hc], a.lower[hc]) : make_float2(0.f, 0.f);
                    wv[c] = f.x;
                    kv[c] = f.y;
                    rv[c] = c < D ? pr[co.r + hc] : 0.f;
                }
            } else {
                const float2* cs = a.s.rot ? a.cs + (int64_t)a.tok_pos[row] * (a.s.rot / 2) : nullptr;
                for (int c = tid; c < DP; c += blockDim.x) {
                    kv[c] = c < D ? rotated(pr + co.k + h * D, c, a.s.rot, cs) * a.s.key_scale : 0.f;
                    rv[c] = c < D ? rotated(pr + co.r + h * D, c, a.s.rot, cs) : 0.f;
                }
            }
            __syncthreads();
            const float decay = RULE == STATE_DECAY ? a.decay[h] : 0.f;
            for (int c0 = 0; c0 < V; c0 += per_pass) {
                const int col = c0 + tid / L;
                if (!ready) load(h, col);
                ready = keep;
                const float o = state_token<L, R, RULE>(st, kv, rv, wv, av, decay, col < V ? pr[co.v + h * V + col] : 0.f, l);
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
        float ss = 0.f;
        for (int i = lane; i < n; i += 32) ss = fmaf(os[i], os[i], ss);
        ss = warp_sum(ss);
        int count = n;
        if (RULE == STATE_DECAY && a.s.norm_all) {
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
        for (int i = tid; i < n; i += blockDim.x) out[i] = from_f32<T>(os[i] * r * (i == tid ? factor : state_factor(a, pr + co.g, h0 * V + i)));
        __syncthreads();
        fresh = false;
    }
}

constexpr int SS_MAX_CLUSTER = 8;

template <typename T, int L, int R, int RULE>
static cudaError_t state_step_launch(const StateArgs& a, int n_tok, cudaStream_t st) {
    int hp = 1, cl = 1;
    const bool all_heads = RULE == STATE_DECAY && a.s.norm_all;
    if (all_heads) {
        hp = (a.s.heads + SS_MAX_CLUSTER - 1) / SS_MAX_CLUSTER;
        while (cl < SS_MAX_CLUSTER && cl * hp < a.s.heads) cl <<= 1;
    }
    const int all = L * a.s.vdim, threads = all <= 1024 ? (all + 31) / 32 * 32 : 512;
    const size_t smem = ((size_t)step_vectors(RULE) * 4 * L * R + (size_t)hp * a.s.vdim) * 4;
    constexpr int CAP = 200 * 1024;
    if (smem > CAP) return cudaErrorInvalidValue;
    static PerDeviceOnce once;
    const cudaError_t le = once.run([] { return cudaFuncSetAttribute(state_step_kernel<T, L, R, RULE>, cudaFuncAttributeMaxDynamicSharedMemorySize, CAP); });
    if (le != cudaSuccess) return le;
    return launch_pdl_cluster(state_step_kernel<T, L, R, RULE>, dim3(n_tok, 1, all_heads ? cl : a.s.heads), dim3(threads), smem, st, cl, a, n_tok, hp, cl);
}

cudaError_t launch_state_step(const StateArgs& a, int n_tok, cudaStream_t st) {
    if (n_tok == 0) return cudaSuccess;
    if (n_tok > STATE_STEP_ROWS || a.s.dim > STATE_MAX_DIM || a.s.dim_pad != state_dim_pad(a.s.dim)) return cudaErrorInvalidValue;
    const int rule = a.s.rule;
    cudaError_t le = cudaErrorInvalidValue;
#define SP_SR(T, L, R)                                                                                                                     \
    (rule == STATE_DELTA ? state_step_launch<T, L, R, STATE_DELTA>(a, n_tok, st) : rule == STATE_FORGET ? state_step_launch<T, L, R, STATE_FORGET>(a, n_tok, st) \
                                                                                                : state_step_launch<T, L, R, STATE_DECAY>(a, n_tok, st))
#define SP_SS(L, R) le = a.f32 ? SP_SR(float, L, R) : SP_SR(bf16, L, R)
    switch (a.s.dim_pad) {
        case 16: SP_SS(4, 1); break;
        case 32: SP_SS(4, 2); break;
        case 64: SP_SS(4, 4); break;
        case 128: SP_SS(8, 4); break;
        case 256: SP_SS(16, 4); break;
        case 512: SP_SS(32, 4); break;
    }
#undef SP_SS
#undef SP_SR
    return le != cudaSuccess ? le : count_launch_and_check();
}

// ── many rows, f32 engines (bf16 ones: state_chunk.cu) ──
// Plain fused multiply-adds. Tokens go in groups of four of one sequence. With c(s, t) the product of the decays of tokens s + 1 .. t (per key channel)
// and S the state before the group,
//   d_t = U_t . S + sum_{s < t} Auk[t][s] v_s - Aub[t][s] d_s      what the unit key u_t finds (delta rule)
//   o_t = R_t . S + sum_{s <= t} Ark[t][s] v_s - Arb[t][s] d_s
//   S  <- c(0, 4) S + sum_s K_s v_s - B_s d_s
// where U_t = c(0, t - 1) u_t, R_t = c(0, t) r_t, K_s = c(s, 4) k_s, B_s = c(s, 4) a_s u_s and, summed over the channels,
// Auk = u_t c(s, t - 1) k_s, Aub = u_t c(s, t - 1) a_s u_s, Ark = r_t c(s, t) k_s, Arb = r_t c(s, t) a_s u_s. So the scan's
// chain of reductions has a link per group, not per token. Everything but d, o and S is made by a kernel that is parallel
// over groups and heads; a sequence's last group is filled up with tokens that change nothing (k = r = a = 0, decay 1).
// Per (group, head) a record: U | R | K | B as [4][dim_pad] each (R | K without the delta rule), c(0, 4) by channel (not in the
// decaying sum), the coefficients, and the values [4][v_pad], where the scan leaves the outputs.
constexpr int SGRP = STATE_GROUP_F32, A_UB = 8, A_RK = 16, A_RB = 32, A_FLOATS = 48;  // Auk at 0: (t, s < t) in order of t
struct StateRecord {
    int k, b, c, a, v, v_pad, floats;  // offsets of U (or R) = 0, ...
    int r;
};
__host__ __device__ __forceinline__ StateRecord state_record(const StateShape& s) {
    StateRecord r;
    const int m = SGRP * s.dim_pad;
    const bool delta = s.rule == STATE_DELTA;
    r.r = delta ? m : 0;
    r.k = r.r + m;
    r.b = r.k + m;
    r.c = delta ? r.b + m : r.b;
    r.a = s.rule == STATE_DECAY ? r.c : r.c + s.dim_pad;
    r.v = r.a + A_FLOATS;
    r.v_pad = (s.vdim + 3) & ~3;
    r.floats = r.v + SGRP * r.v_pad;
    return r;
}
static StateRecordView state_view(const StateShape& s, bool f32) {
    const StateRecord r = state_record(s);
    return f32 ? StateRecordView{r.v, r.v_pad, r.floats} : state_chunk_view(s);
}
size_t state_record_floats(const StateShape& s, bool f32) { return (size_t)s.heads * state_view(s, f32).floats; }

// Sums p[i] over the warp for all i at once: lane i receives the sum of p[i].
__device__ __forceinline__ float warp_sums(float (&p)[32]) {
    const int lane = threadIdx.x & 31;
#pragma unroll
    for (int m = 16; m > 0; m >>= 1) {
        const bool up = lane & m;
#pragma unroll
        for (int i = 0; i < m; ++i) {
            const float send = up ? p[i] : p[i + m], keep = up ? p[i + m] : p[i];
            p[i] = keep + __shfl_xor_sync(0xFFFFFFFFu, send, m);
        }
    }
    return p[0];
}

// A warp per (group, head).
constexpr int SG_WARPS = 4;
template <int RULE>
__global__ void __launch_bounds__(SG_WARPS * 32) state_prepare_kernel(const StateArgs a, const int4* __restrict__ groups) {
    constexpr bool DELTA = RULE == STATE_DELTA;
    pdl_wait();
    pdl_trigger();
    const int h = blockIdx.y * SG_WARPS + (threadIdx.x >> 5), lane = threadIdx.x & 31, D = a.s.dim, DP = a.s.dim_pad, V = a.s.vdim, H = a.s.heads;
    if (h >= H) return;
    const StateCols co = state_cols(a.s);
    const StateRecord rec = state_record(a.s);
    float* out = a.rec + ((int64_t)blockIdx.x * H + h) * rec.floats;
    const int4 g4 = groups[blockIdx.x];
    const int row[SGRP] = {g4.x, g4.y, g4.z, g4.w};
    const float* pr[SGRP];
#pragma unroll
    for (int t = 0; t < SGRP; ++t) pr[t] = a.proj + (int64_t)max(row[t], 0) * a.ldp;
    float inv[SGRP] = {};  // 1 / |k|
    if (DELTA) {
        for (int c = lane; c < D; c += 32)
#pragma unroll
            for (int t = 0; t < SGRP; ++t) {
                const float k = pr[t][co.k + h * D + c];
                inv[t] = fmaf(k, k, inv[t]);
            }
#pragma unroll
        for (int t = 0; t < SGRP; ++t) inv[t] = 1.0f / sqrtf(warp_sum(inv[t]) + 1e-6f);
    }
    const float decay = RULE == STATE_DECAY ? a.decay[h] : 1.f;
    float p[32];  // Auk, Aub (t, s < t), then Ark, Arb (t, s <= t); the decaying sum: Ark alone
#pragma unroll
    for (int i = 0; i < 32; ++i) p[i] = 0.f;
    float whole = 1.f;
    for (int c = lane; c < DP; c += 32) {
        const bool on = c < D;
        const int hc = h * D + min(c, D - 1);
        float k[SGRP], r[SGRP], w[SGRP], u[SGRP], b[SGRP];
#pragma unroll
        for (int t = 0; t < SGRP; ++t) {
            const bool live = on && row[t] >= 0;
            w[t] = row[t] < 0 ? 1.f : decay;
            if (RULE == STATE_DECAY) {
                const float2* cs = live && a.s.rot ? a.cs + (int64_t)a.tok_pos[row[t]] * (a.s.rot / 2) : nullptr;
                k[t] = live ? rotated(pr[t] + co.k + h * D, c, a.s.rot, cs) * a.s.key_scale : 0.f;
                r[t] = live ? rotated(pr[t] + co.r + h * D, c, a.s.rot, cs) : 0.f;
            } else {
                k[t] = live ? pr[t][co.k + hc] : 0.f;
                r[t] = live ? pr[t][co.r + hc] : 0.f;
            }
            if (RULE == STATE_FORGET) {
                const float2 f = live ? forget_gate(pr[t][co.a + hc] + a.a_bias[hc], a.lower[hc]) : make_float2(1.f, 0.f);
                w[t] = f.x;
                k[t] = f.y;
            }
            if (DELTA) {
                w[t] = live ? channel_decay(a.wlogit[(int64_t)row[t] * H * D + hc] + a.w0[hc]) : 1.f;
                u[t] = k[t] * inv[t];
                b[t] = live ? u[t] * sigmoid_f32(pr[t][co.a + hc] + a.a_bias[hc]) : 0.f;
            }
        }
        int i = 0;
        if (DELTA) {
#pragma unroll
            for (int t = 1; t < SGRP; ++t)
#pragma unroll
                for (int s = 0; s < t; ++s, ++i) {
                    float q = u[t];
#pragma unroll
                    for (int j = s + 1; j < t; ++j) q *= w[j];
                    p[i] = fmaf(q, k[s], p[i]);
                    p[6 + i] = fmaf(q, b[s], p[6 + i]);
                }
            i = 12;
        }
#pragma unroll
        for (int t = 0; t < SGRP; ++t)
#pragma unroll
            for (int s = 0; s <= t; ++s, ++i) {
                float q = r[t];
#pragma unroll
                for (int j = s + 1; j <= t; ++j) q *= w[j];
                p[i] = fmaf(q, k[s], p[i]);
                if (DELTA) p[10 + i] = fmaf(q, b[s], p[10 + i]);
            }
        float before = 1.f, after = 1.f;
#pragma unroll
        for (int t = 0; t < SGRP; ++t) {
            if (DELTA) out[t * DP + c] = before * u[t];
            before *= w[t];
            out[rec.r + t * DP + c] = before * r[t];
        }
#pragma unroll
        for (int t = SGRP - 1; t >= 0; --t) {
            out[rec.k + t * DP + c] = after * k[t];
            if (DELTA) out[rec.b + t * DP + c] = after * b[t];
            after *= w[t];
        }
        if (RULE != STATE_DECAY) out[rec.c + c] = before;
        whole = before;
    }
    const float sum = warp_sums(p);
    // lane -> (t, s) of its coefficient; the upper triangles stay zero
    float* A = out + rec.a;
    for (int i = lane; i < A_FLOATS; i += 32) A[i] = 0.f;
    __syncwarp();
    const int first = DELTA ? 12 : 0;
    if (DELTA && lane < 12) A[lane < 6 ? lane : A_UB + lane - 6] = sum;
    else if (lane >= first && lane < first + (DELTA ? 20 : 10)) {
        const int i = lane - first, q = i % 10, t = q >= 6 ? 3 : q >= 3 ? 2 : q >= 1 ? 1 : 0;
        A[(i >= 10 ? A_RB : A_RK) + 4 * t + q - t * (t + 1) / 2] = sum;
    }
    if (RULE == STATE_DECAY && lane == 0) A[0] = whole;
    for (int c = lane; c < rec.v_pad; c += 32)
#pragma unroll
        for (int t = 0; t < SGRP; ++t) out[rec.v + t * rec.v_pad + c] = c < V && row[t] >= 0 ? pr[t][co.v + h * V + c] : 0.f;
}

// Block (SC_COLS columns, head, segment); records arrive in tiles of tg groups, two stages of cp.async.
constexpr int SC_COLS = 16;
template <int L, int R, int RULE>
__global__ void __launch_bounds__(SC_COLS * L) state_scan_kernel(const StateArgs a, const StateSegment* __restrict__ segs, int tg) {
    extern __shared__ __align__(16) float sc_smem[];
    constexpr int DP = 4 * L * R, THREADS = SC_COLS * L;
    constexpr bool DELTA = RULE == STATE_DELTA;
    const int tid = threadIdx.x, l = tid % L, cl = tid / L, H = a.s.heads, V = a.s.vdim, h = blockIdx.y, col0 = blockIdx.x * SC_COLS, col = col0 + cl;
    const StateRecord rec = state_record(a.s);
    const int stage = rec.v + SGRP * SC_COLS;  // floats of a group in shared memory: the record with this block's values only
    pdl_wait();
    pdl_trigger();
    const StateSegment sg = segs[blockIdx.z];
    float* state = a.state + sg.slot * a.slot_stride + ((int64_t)h * V + col) * DP + 4 * l;
    float4 st[R];
#pragma unroll
    for (int i = 0; i < R; ++i) st[i] = col < V && !sg.fresh ? *reinterpret_cast<const float4*>(state + 4 * L * i) : make_float4(0.f, 0.f, 0.f, 0.f);
    float* const first = a.rec + ((int64_t)sg.group0 * H + h) * rec.floats;
    const int64_t step = (int64_t)H * rec.floats;
    const int v_pieces = min(SC_COLS, rec.v_pad - col0) / 4;
    auto fetch = [&](int g0, int buf) {
        for (int k = 0; k < tg && g0 + k < sg.n_groups; ++k) {
            const float* src = first + (g0 + k) * step;
            float* d = sc_smem + (buf * tg + k) * stage;
            for (int i = 4 * tid; i < rec.v; i += 4 * THREADS) cp_async16(d + i, src + i, 16);
            const int t = tid / (SC_COLS / 4), q = tid % (SC_COLS / 4);
            if (t < SGRP && q < v_pieces) cp_async16(d + rec.v + t * SC_COLS + 4 * q, src + rec.v + t * rec.v_pad + col0 + 4 * q, 16);
        }
    };
    fetch(0, 0);
    cp_async_commit();
    // the token whose output this lane finishes, after the exchange below
    const int mine = 2 * (l & 1) + ((l >> 1) & 1);
    for (int g0 = 0, buf = 0; g0 < sg.n_groups; g0 += tg, buf ^= 1) {
        if (g0 + tg < sg.n_groups) fetch(g0 + tg, buf ^ 1);
        cp_async_commit();
        cp_async_wait<1>();
        __syncthreads();
        const int n = min(tg, sg.n_groups - g0);
        for (int k = 0; k < n; ++k) {
            const float* d = sc_smem + (buf * tg + k) * stage;
            const float* A = d + rec.a;
            float v[SGRP], e[SGRP] = {}, f[SGRP] = {};
#pragma unroll
            for (int t = 0; t < SGRP; ++t) v[t] = d[rec.v + t * SC_COLS + cl];
#pragma unroll
            for (int i = 0; i < R; ++i) {
                const int at = 4 * (l + L * i);
#pragma unroll
                for (int t = 0; t < SGRP; ++t) {
                    if (DELTA) {
                        const float4 u = *reinterpret_cast<const float4*>(d + t * DP + at);
                        e[t] = fmaf(u.x, st[i].x, fmaf(u.y, st[i].y, fmaf(u.z, st[i].z, fmaf(u.w, st[i].w, e[t]))));
                    }
                    const float4 r = *reinterpret_cast<const float4*>(d + rec.r + t * DP + at);
                    f[t] = fmaf(r.x, st[i].x, fmaf(r.y, st[i].y, fmaf(r.z, st[i].z, fmaf(r.w, st[i].w, f[t]))));
                }
            }
            if (DELTA) {
#pragma unroll
                for (int t = 0; t < SGRP; ++t) e[t] = lanes_sum<L>(e[t]);
                const float4 k0 = *reinterpret_cast<const float4*>(A), b0 = *reinterpret_cast<const float4*>(A + A_UB);
                const float2 k1 = *reinterpret_cast<const float2*>(A + 4), b1 = *reinterpret_cast<const float2*>(A + A_UB + 4);
                e[1] = fmaf(k0.x, v[0], fmaf(-b0.x, e[0], e[1]));
                e[2] = fmaf(k0.y, v[0], fmaf(k0.z, v[1], fmaf(-b0.y, e[0], fmaf(-b0.z, e[1], e[2]))));
                e[3] = fmaf(k0.w, v[0], fmaf(k1.x, v[1], fmaf(k1.y, v[2], fmaf(-b0.w, e[0], fmaf(-b1.x, e[1], fmaf(-b1.y, e[2], e[3]))))));
            }
            const float whole = RULE == STATE_DECAY ? A[0] : 0.f;
#pragma unroll
            for (int i = 0; i < R; ++i) {
                const int at = 4 * (l + L * i);
                float4 c = make_float4(whole, whole, whole, whole);
                if (RULE != STATE_DECAY) c = *reinterpret_cast<const float4*>(d + rec.c + at);
                st[i].x *= c.x; st[i].y *= c.y; st[i].z *= c.z; st[i].w *= c.w;
#pragma unroll
                for (int t = 0; t < SGRP; ++t) {
                    const float4 q = *reinterpret_cast<const float4*>(d + rec.k + t * DP + at);
                    st[i].x = fmaf(q.x, v[t], st[i].x);
                    st[i].y = fmaf(q.y, v[t], st[i].y);
                    st[i].z = fmaf(q.z, v[t], st[i].z);
                    st[i].w = fmaf(q.w, v[t], st[i].w);
                    if (DELTA) {
                        const float4 b = *reinterpret_cast<const float4*>(d + rec.b + t * DP + at);
                        st[i].x = fmaf(-b.x, e[t], st[i].x);
                        st[i].y = fmaf(-b.y, e[t], st[i].y);
                        st[i].z = fmaf(-b.z, e[t], st[i].z);
                        st[i].w = fmaf(-b.w, e[t], st[i].w);
                    }
                }
            }
            // the lanes of a column share out the four outputs while they sum them
            {
                const bool up = l & 1, up2 = l & 2;
                const float x = (up ? f[2] : f[0]) + __shfl_xor_sync(0xFFFFFFFFu, up ? f[0] : f[2], 1);
                const float y = (up ? f[3] : f[1]) + __shfl_xor_sync(0xFFFFFFFFu, up ? f[1] : f[3], 1);
                float o = (up2 ? y : x) + __shfl_xor_sync(0xFFFFFFFFu, up2 ? x : y, 2);
#pragma unroll
                for (int m = 4; m < L; m <<= 1) o += __shfl_xor_sync(0xFFFFFFFFu, o, m);
                const float4 q = *reinterpret_cast<const float4*>(A + A_RK + 4 * mine);
                o = fmaf(q.x, v[0], fmaf(q.y, v[1], fmaf(q.z, v[2], fmaf(q.w, v[3], o))));
                if (DELTA) {
                    const float4 b = *reinterpret_cast<const float4*>(A + A_RB + 4 * mine);
                    o = fmaf(-b.x, e[0], fmaf(-b.y, e[1], fmaf(-b.z, e[2], fmaf(-b.w, e[3], o))));
                }
                if (l < 4 && col < V) first[(g0 + k) * step + rec.v + mine * rec.v_pad + col] = o;
            }
        }
        __syncthreads();
    }
    cp_async_wait<0>();
    if (col < V)
#pragma unroll
        for (int i = 0; i < R; ++i) *reinterpret_cast<float4*>(state + 4 * L * i) = st[i];
}

// Norms of the scan's outputs, gain, gate. EACH: a warp per (token, head); else a block per token, for the norm is over all heads.
constexpr int SN_WARPS = 8, SN_KEEP = 4;  // values a lane keeps in registers
template <typename T, bool EACH>
__global__ void __launch_bounds__(SN_WARPS * 32) state_norm_kernel(const StateArgs a, const StateRecordView rec, const int32_t* __restrict__ groups, int group) {
    __shared__ float sh[SN_WARPS];
    pdl_wait();
    pdl_trigger();
    const int H = a.s.heads, V = a.s.vdim, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, t = blockIdx.x % group;
    const int64_t row = groups[blockIdx.x];
    if (row < 0) return;
    const float *o = a.rec + (int64_t)(blockIdx.x / group) * H * rec.floats + rec.v + t * rec.v_pad, *g = a.proj + row * a.ldp + state_cols(a.s).g;
    T* out = reinterpret_cast<T*>(a.out) + row * a.ldo;
    auto finish = [&](int h, int i, float v, float r) { out[h * V + i] = from_f32<T>(v * r * state_factor(a, g, h * V + i)); };
    if (EACH) {
        const int h = blockIdx.y * SN_WARPS + warp;
        if (h >= H) return;
        const float* oh = o + (int64_t)h * rec.floats;
        float v[SN_KEEP], f[SN_KEEP], ss = 0.f;  // outputs, gain and gate
#pragma unroll
        for (int j = 0; j < SN_KEEP; ++j) {
            const int i = lane + 32 * j;
            v[j] = i < V ? oh[i] : 0.f;
            f[j] = i < V ? state_factor(a, g, h * V + i) : 0.f;
            ss = fmaf(v[j], v[j], ss);
        }
        for (int i = lane + 32 * SN_KEEP; i < V; i += 32) ss = fmaf(oh[i], oh[i], ss);
        const float r = rsqrtf(warp_sum(ss) / (float)V + a.s.eps);
#pragma unroll
        for (int j = 0; j < SN_KEEP; ++j)
            if (lane + 32 * j < V) out[h * V + lane + 32 * j] = from_f32<T>(v[j] * r * f[j]);
        for (int i = lane + 32 * SN_KEEP; i < V; i += 32) finish(h, i, oh[i], r);
        return;
    }
    float ss = 0.f;
    for (int i = threadIdx.x; i < H * V; i += SN_WARPS * 32) {
        const float v = o[(int64_t)(i / V) * rec.floats + i % V];
        ss = fmaf(v, v, ss);
    }
    const float r = rsqrtf(block_sum<SN_WARPS>(ss, sh) / (float)(H * V) + a.s.eps);
    for (int i = threadIdx.x; i < H * V; i += SN_WARPS * 32) finish(i / V, i % V, o[(int64_t)(i / V) * rec.floats + i % V], r);
}

template <int L, int R, int RULE>
static cudaError_t state_scan_launch(const StateArgs& a, const StateSegment* seg, int n_seg, cudaStream_t st) {
    constexpr int CAP = 96 * 1024;
    const size_t group = (size_t)(state_record(a.s).v + SGRP * SC_COLS) * 4;
    int tg = 4;
    while (tg > 1 && 2 * tg * group > CAP) tg >>= 1;
    static PerDeviceOnce once;
    const cudaError_t le = once.run([] { return cudaFuncSetAttribute(state_scan_kernel<L, R, RULE>, cudaFuncAttributeMaxDynamicSharedMemorySize, CAP); });
    if (le != cudaSuccess) return le;
    return launch_pdl(state_scan_kernel<L, R, RULE>, dim3((a.s.vdim + SC_COLS - 1) / SC_COLS, a.s.heads, n_seg), dim3(SC_COLS * L), 2 * tg * group, st, a, seg, tg);
}

static cudaError_t launch_state_groups(const StateArgs& a, const StateSegment* seg, int n_seg, const int4* groups, int n_groups, cudaStream_t st) {
    const int rule = a.s.rule;
    const dim3 pg(n_groups, (a.s.heads + SG_WARPS - 1) / SG_WARPS);
    const auto prepare = rule == STATE_DELTA ? state_prepare_kernel<STATE_DELTA> : rule == STATE_FORGET ? state_prepare_kernel<STATE_FORGET> : state_prepare_kernel<STATE_DECAY>;
    cudaError_t le = launch_pdl(prepare, pg, dim3(SG_WARPS * 32), 0, st, a, groups);
    if (le == cudaSuccess) le = count_launch_and_check();
    if (le != cudaSuccess) return le;
    le = cudaErrorInvalidValue;
#define SP_SC(L, R)                                                                                                                            \
    le = rule == STATE_DELTA ? state_scan_launch<L, R, STATE_DELTA>(a, seg, n_seg, st) : rule == STATE_FORGET ? state_scan_launch<L, R, STATE_FORGET>(a, seg, n_seg, st) \
                                                                                                      : state_scan_launch<L, R, STATE_DECAY>(a, seg, n_seg, st)
    switch (a.s.dim_pad) {
        case 16: SP_SC(4, 1); break;
        case 32: SP_SC(8, 1); break;
        case 64: SP_SC(8, 2); break;
        case 128: SP_SC(16, 2); break;
        case 256: SP_SC(16, 4); break;
        case 512: SP_SC(32, 4); break;
    }
#undef SP_SC
    return le != cudaSuccess ? le : count_launch_and_check();
}

cudaError_t launch_state_scan(const StateArgs& a, const StateSegment* seg, int n_seg, const int32_t* groups, int n_groups, cudaStream_t st) {
    if (n_groups == 0 || n_seg == 0) return cudaSuccess;
    if (a.s.dim > STATE_MAX_DIM || a.s.dim_pad != state_dim_pad(a.s.dim)) return cudaErrorInvalidValue;
    cudaError_t le = a.f32 ? launch_state_groups(a, seg, n_seg, reinterpret_cast<const int4*>(groups), n_groups, st) : launch_state_chunks(a, seg, n_seg, groups, n_groups, st);
    if (le != cudaSuccess) return le;
    const bool each = !a.s.norm_all;
    const int group = state_group(a.f32);
    const dim3 grid(n_groups * group, each ? (a.s.heads + SN_WARPS - 1) / SN_WARPS : 1), block(SN_WARPS * 32);
    const StateRecordView rec = state_view(a.s, a.f32);
#define SP_SN(T, D) launch_pdl(state_norm_kernel<T, D>, grid, block, 0, st, a, rec, groups, group)
    le = a.f32 ? (each ? SP_SN(float, true) : SP_SN(float, false)) : (each ? SP_SN(bf16, true) : SP_SN(bf16, false));
#undef SP_SN
    return le != cudaSuccess ? le : count_launch_and_check();
}

}  // namespace sp
