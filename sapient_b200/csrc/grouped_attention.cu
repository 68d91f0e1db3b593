// Grouped-query attention over a paged cache of keys and values, or of keys that are the values (plan_kernels.h). Keys and
// values may differ in size; scores, softmax and accumulation are f32, the softmax weights enter the tensor cores as a leading
// bf16 part plus its remainder. A sliding window bounds the pages a block visits. Distance biases, sinks and output gates are
// uniform branches of the same kernels: a bias is read from a table by distance, in prompts through shared memory (a tile's
// distances are one run of it), and is one constant for tiles that are far enough.
#include <algorithm>

#include "kernels.h"
#include "pdl.cuh"
#include "plan_common.cuh"
#include "plan_kernels.h"
#include "sp_common.cuh"

namespace sp {

cudaError_t count_launch_and_check();  // kernels.cu

// ── rotation and cache append ──
constexpr int GA_WARPS = 4;

// dst[0 .. pad) = src(0 .. n) with coordinates i and i + dims / 2 (neighbours: 2 i and 2 i + 1) turned by cs[i] for i < dims / 2;
// zeros past n.
template <typename T, typename Src>
__device__ __forceinline__ void rotate_pairs(const Src& src, T* dst, const float2* cs, int dims, bool neighbours, int n, int pad) {
    const int half = dims / 2, lane = threadIdx.x & 31;
    for (int i = lane; i < half; i += 32) {
        const int a = neighbours ? 2 * i : i, b = neighbours ? a + 1 : i + half;
        const float u = src(a), v = src(b);
        const float2 r = cs[i];
        dst[a] = from_f32<T>(u * r.x - v * r.y);
        dst[b] = from_f32<T>(v * r.x + u * r.y);
    }
    for (int i = dims + lane; i < pad; i += 32) dst[i] = from_f32<T>(i < n ? src(i) : 0.f);
}

// A warp per (token, part): the heads' queries, then the cached heads' keys and values (shared: the keys alone).
template <typename T>
__global__ void __launch_bounds__(GA_WARPS * 32) grouped_append_kernel(const float* __restrict__ proj, int ldp, const GroupedShape s, const GroupedCache c,
                                                                    const GroupedInput in, const int32_t* __restrict__ tok_slot,
                                                                    const int32_t* __restrict__ tok_pos, T* __restrict__ q) {
    pdl_wait();
    pdl_trigger();
    const int t = blockIdx.x, part = blockIdx.y * GA_WARPS + (threadIdx.x >> 5), pos = tok_pos[t], lane = threadIdx.x & 31;
    const bool query = part < s.heads;
    const int per = c.shared ? 1 : 2, g = query ? 0 : (part - s.heads) / per;
    if (g >= s.kv_heads) return;
    const bool value = !query && (part - s.heads) % per == 1;
    const int n = value ? s.vdim : s.dim;
    const int64_t at = query ? (int64_t)part * s.dim : value ? (int64_t)(s.heads + s.kv_heads) * s.dim + (int64_t)g * s.vdim : (int64_t)(s.heads + g) * s.dim;
    const float* pr = proj + (int64_t)t * ldp + at;
    const float* bias = in.bias ? in.bias + at : nullptr;
    auto projected = [&](int i) { return bias ? pr[i] + bias[i] : pr[i]; };
    float r = 1.f;
    if (in.norm && !value) {
        float ss = 0.f;
        for (int i = lane; i < n; i += 32) {
            const float v = projected(i);
            ss = fmaf(v, v, ss);
        }
        r = rsqrtf(warp_sum(ss) / (float)n + in.eps);
    }
    const float2* ck = in.cs_key ? in.cs_key + (int64_t)pos * (s.rot / 2) : nullptr;
    auto normed = [&](const float* gain, float mult) {
        return [=](int i) { return gain ? projected(i) * mult * gain[i] : projected(i) * mult; };
    };
    if (query) {
        if (in.temperature) r *= in.temperature[pos];
        rotate_pairs<T>(normed(in.q_gain, r), q + ((int64_t)t * s.heads + part) * c.dim16, ck, s.rot, s.neighbours, s.dim, c.dim16);
        return;
    }
    const int page = c.page_table[(int64_t)tok_slot[t] * c.max_pages + pos / KV_PAGE];
    T* row = reinterpret_cast<T*>(c.pool) + (((int64_t)page * s.kv_heads + g) * KV_PAGE + pos % KV_PAGE) * c.ld;
    if (c.shared) {
        rotate_pairs<T>(projected, row, nullptr, 0, false, n, c.dim16);
        if (lane == 0) *reinterpret_cast<float*>(row + c.dim16) = r;
    } else if (value) {
        rotate_pairs<T>(projected, row + c.dim16, in.cs_val ? in.cs_val + (int64_t)pos * (s.vdim / 2) : nullptr, in.cs_val ? s.vdim : 0, false, n, c.vdim16);
    } else {
        rotate_pairs<T>(normed(in.k_gain, r), row, ck, s.rot, s.neighbours, n, c.dim16);
    }
}

cudaError_t launch_grouped_append(const float* proj, int ldp, const GroupedShape& s, const GroupedCache& c, const GroupedInput& in,
                                  const int32_t* tok_slot, const int32_t* tok_pos, void* q, bool f32, int n_tok, cudaStream_t st) {
    if (n_tok == 0) return cudaSuccess;
    if (c.shared && (s.rot || in.cs_val || in.k_gain || s.dim != s.vdim)) return cudaErrorInvalidValue;
    const dim3 grid(n_tok, (s.heads + (c.shared ? 1 : 2) * s.kv_heads + GA_WARPS - 1) / GA_WARPS), block(GA_WARPS * 32);
    if (in.conv) return cudaErrorInvalidValue;
    const cudaError_t le = f32 ? launch_pdl(grouped_append_kernel<float>, grid, block, 0, st, proj, ldp, s, c, in, tok_slot, tok_pos, (float*)q)
                               : launch_pdl(grouped_append_kernel<bf16>, grid, block, 0, st, proj, ldp, s, c, in, tok_slot, tok_pos, (bf16*)q);
    return le != cudaSuccess ? le : count_launch_and_check();
}

// The f32 factor behind a shared row's key.
template <typename T>
__device__ __forceinline__ float row_factor(const T* row, int dim16) { return *reinterpret_cast<const float*>(row + dim16); }

// Writes coordinates m and m + half of a head's mixture, turned back by the angles cs and gated (null: as they are).
template <typename T>
__device__ __forceinline__ void store_mixed(T* dst, int m, int half, float u, float v, const float2* cs, const float* gate) {
    if (cs) {
        const float2 r = cs[m];
        const float x = u * r.x + v * r.y;
        v = v * r.x - u * r.y;
        u = x;
    }
    if (gate) {
        u *= sigmoid_f32(gate[m]);
        v *= sigmoid_f32(gate[m + half]);
    }
    dst[m] = from_f32<T>(u);
    dst[m + half] = from_f32<T>(v);
}

template <typename T>
__device__ __forceinline__ void store_one(T* dst, int m, float u, const float* gate) { dst[m] = from_f32<T>(gate ? u * sigmoid_f32(gate[m]) : u); }

__device__ __forceinline__ const float* gate_row(const GroupedTerms& x, int64_t t, int h, int vdim) {
    return x.gate ? x.gate + t * x.ldgate + (int64_t)h * vdim : nullptr;
}

// ── any compute type and sizes ──
constexpr int GS_WARPS = 4, GS_PER_LANE = GROUPED_MAX_VDIM / 32;
template <typename T>
__global__ void __launch_bounds__(GS_WARPS * 32) grouped_simple_kernel(const T* __restrict__ q, const GroupedShape s, const GroupedCache c,
                                                                    const GroupedTerms x, const int32_t* __restrict__ tok_slot,
                                                                    const int32_t* __restrict__ tok_pos, T* __restrict__ out, int ldo) {
    extern __shared__ float gs_smem[];  // query, then one output row per warp
    __shared__ float sm[GS_WARPS], sl[GS_WARPS];
    pdl_wait();
    pdl_trigger();
    const int h = blockIdx.x, t = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = h / (s.heads / s.kv_heads);
    const int pos = tok_pos[t], lo = s.window > pos ? 0 : pos - s.window + 1, val = c.shared ? 0 : c.dim16;
    const float* rel = x.rel ? x.rel + (int64_t)h * x.n_rel : nullptr;
    float *qs = gs_smem, *os = gs_smem + c.dim16;
    for (int i = threadIdx.x; i < c.dim16; i += GS_WARPS * 32) qs[i] = to_f32(q[((int64_t)t * s.heads + h) * c.dim16 + i]);
    __syncthreads();
    const int32_t* pt = c.page_table + (int64_t)tok_slot[t] * c.max_pages;
    float o[GS_PER_LANE];
#pragma unroll
    for (int i = 0; i < GS_PER_LANE; ++i) o[i] = 0.f;
    float m = -INFINITY, l = 0.f;
    for (int key = lo + warp; key <= pos; key += GS_WARPS) {
        const T* row = reinterpret_cast<const T*>(c.pool) + (((int64_t)pt[key / KV_PAGE] * s.kv_heads + g) * KV_PAGE + key % KV_PAGE) * c.ld;
        float dot = 0.f;
        for (int i = lane; i < s.dim; i += 32) dot = fmaf(qs[i], to_f32(row[i]), dot);
        float sc = warp_sum(dot) * s.scale;
        if (c.shared) sc *= row_factor(row, c.dim16);
        if (rel) sc += rel[min(pos - key, x.n_rel - 1)];
        const float mn = fmaxf(m, sc), corr = expf(m - mn), p = expf(sc - mn);
#pragma unroll
        for (int i = 0; i < GS_PER_LANE; ++i)
            if (lane + 32 * i < s.vdim) o[i] = fmaf(p, to_f32(row[val + lane + 32 * i]), o[i] * corr);
        l = fmaf(l, corr, p);
        m = mn;
    }
    if (lane == 0) { sm[warp] = m; sl[warp] = l; }
#pragma unroll
    for (int i = 0; i < GS_PER_LANE; ++i)
        if (lane + 32 * i < s.vdim) os[warp * s.vdim + lane + 32 * i] = o[i];
    __syncthreads();
    float M = -INFINITY, sum = 0.f, cw[GS_WARPS];
#pragma unroll
    for (int w = 0; w < GS_WARPS; ++w) M = fmaxf(M, sm[w]);
    if (x.sink) {
        M = fmaxf(M, x.sink[h]);
        sum = expf(x.sink[h] - M);
    }
#pragma unroll
    for (int w = 0; w < GS_WARPS; ++w) {
        cw[w] = sm[w] == -INFINITY ? 0.f : expf(sm[w] - M);
        sum = fmaf(cw[w], sl[w], sum);
    }
    const float inv = 1.0f / sum;
    auto mixed = [&](int e) {
        float v = 0.f;
#pragma unroll
        for (int w = 0; w < GS_WARPS; ++w) v = fmaf(cw[w], os[w * s.vdim + e], v);
        return v * inv;
    };
    T* d = out + (int64_t)t * ldo + (int64_t)h * s.vdim;
    const int half = s.vdim / 2;
    const float* gate = gate_row(x, t, h, s.vdim);
    for (int e = threadIdx.x; e < half; e += GS_WARPS * 32)
        store_mixed<T>(d, e, half, mixed(e), mixed(e + half), x.cs_val ? x.cs_val + (int64_t)pos * half : nullptr, gate);
    if ((s.vdim & 1) && threadIdx.x == 0) store_one<T>(d, s.vdim - 1, mixed(s.vdim - 1), gate);
}

// ── few rows, bf16 ──
// Block per (cached head, 16 of its query heads; token; split of the keys), the splits being the blocks of a cluster. Each of
// the four warps walks pages of 16 keys of its own with three stages of cp.async; with up to eight query heads the remainders
// of the softmax weights fill the other eight rows of the tile, else they are a second product.
constexpr int GD_WARPS = 4, GD_STAGES = 3, GD_MAX_SPLITS = 8;
// Row stride of a page in shared memory: an odd number of 16-byte pieces where the sizes are multiples of 16.
__host__ __device__ __forceinline__ int gd_row(const GroupedCache& c) { return c.shared ? c.ld : c.ld + 8; }
static size_t gd_smem(const GroupedCache& c) {
    const size_t ring = (size_t)(GD_WARPS * GD_STAGES * KV_PAGE * gd_row(c) + 16 * (c.dim16 + 8)) * 2, mixtures = (size_t)GD_WARPS * 16 * (c.vdim16 + 4) * 4;
    return std::max(ring, mixtures);
}

// REL: a distance bias, SHARED: keys that are the values.
template <int VT, bool PACKED, bool REL, bool SHARED>
__global__ void __launch_bounds__(GD_WARPS * 32) grouped_decode_kernel(const bf16* __restrict__ q, const GroupedShape s, const GroupedCache c,
                                                                    const GroupedTerms x, const int32_t* __restrict__ tok_slot,
                                                                    const int32_t* __restrict__ tok_pos, bf16* __restrict__ out, int ldo, int n_splits) {
    extern __shared__ __align__(16) bf16 gd_sm[];
    __shared__ float m_s[GD_WARPS][16], l_s[GD_WARPS][16], bm_s[16], bl_s[16], share_s[16][GD_MAX_SPLITS];
    const int ld = c.ld, LD = gd_row(c), LQ = c.dim16 + 8, val = SHARED ? 0 : c.dim16;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, tq = lane & 3;
    const int group = s.heads / s.kv_heads, tiles = (group + 15) / 16, kvh = blockIdx.x / tiles, h0 = kvh * group + (blockIdx.x % tiles) * 16;
    const int nq = min(16, (kvh + 1) * group - h0), t = blockIdx.y;
    bf16 *qs = gd_sm, *ring = gd_sm + 16 * LQ + warp * GD_STAGES * KV_PAGE * LD;
    pdl_wait();
    pdl_trigger();
    const int pos = tok_pos[t], lo = s.window > pos ? 0 : pos - s.window + 1;
    const int32_t* pt = c.page_table + (int64_t)tok_slot[t] * c.max_pages;
    for (int i = tid; i < 16 * (c.dim16 / 8); i += GD_WARPS * 32) {
        const int r = i / (c.dim16 / 8), p = i - r * (c.dim16 / 8);
        *reinterpret_cast<uint4*>(qs + r * LQ + p * 8) =
            r < nq ? *reinterpret_cast<const uint4*>(q + ((int64_t)t * s.heads + h0 + r) * c.dim16 + p * 8) : make_uint4(0u, 0u, 0u, 0u);
    }
    const int page_end = pos / KV_PAGE, stride = GD_WARPS * n_splits, page0 = lo / KV_PAGE + blockIdx.z * GD_WARPS + warp;
    const int pieces = ld / 8;
    auto fetch = [&](int page, int st) {
        if (page <= page_end) {
            const bf16* src = reinterpret_cast<const bf16*>(c.pool) + ((int64_t)pt[page] * s.kv_heads + kvh) * KV_PAGE * ld;
            const uint32_t d = smem_addr(ring + st * KV_PAGE * LD);
            int r = lane / pieces, p = lane - r * pieces;  // the page is one run of 16 rows
            for (int i = lane; i < KV_PAGE * pieces; i += 32) {
                cp_async16_at(d + (uint32_t)(r * LD + p * 8) * 2, src + (int64_t)i * 8, page * KV_PAGE + r <= pos ? 16 : 0);
                p += 32;
                while (p >= pieces) { p -= pieces; ++r; }
            }
        }
        cp_async_commit();
    };
#pragma unroll
    for (int i = 0; i < GD_STAGES; ++i) fetch(page0 + i * stride, i);
    __syncthreads();
    float o[VT][4];
#pragma unroll
    for (int i = 0; i < VT; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
    float m0 = -INFINITY, m1 = -INFINITY, l0 = 0.f, l1 = 0.f;
    const uint32_t qa = smem_addr(qs + (lane & 15) * LQ + (lane >> 4) * 8);
    // this thread's heads' biases by distance (PACKED: one head), and the one for every key that is far
    const float* rel0 = REL ? x.rel + (int64_t)(h0 + min(g, nq - 1)) * x.n_rel : nullptr;
    const float* rel1 = REL && !PACKED ? x.rel + (int64_t)(h0 + min(g + 8, nq - 1)) * x.n_rel : nullptr;
    const float far0 = REL ? rel0[x.n_rel - 1] : 0.f, far1 = REL && !PACKED ? rel1[x.n_rel - 1] : 0.f;
    for (int page = page0, st = 0; page <= page_end; page += stride, st = st + 1 == GD_STAGES ? 0 : st + 1) {
        float b0[2][2], b1[2][2];
        if (REL) {
            const bool near = pos - (page * KV_PAGE + KV_PAGE - 1) < x.n_rel - 1;
#pragma unroll
            for (int j = 0; j < 2; ++j)
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    const int dist = max(0, min(pos - (page * KV_PAGE + 8 * j + 2 * tq + e), x.n_rel - 1));
                    b0[j][e] = near ? rel0[dist] : far0;
                    b1[j][e] = PACKED ? 0.f : near ? rel1[dist] : far1;
                }
        }
        cp_async_wait<GD_STAGES - 1>();
        __syncwarp();
        const bf16* kt = ring + st * KV_PAGE * LD;
        float sc[2][4] = {};
        const uint32_t ka = smem_addr(kt + ((lane & 7) + (lane >> 4) * 8) * LD + ((lane >> 3) & 1) * 8);
#pragma unroll 4
        for (int k = 0; k < c.dim16; k += 16) {
            uint32_t a[4], b[4];
            ldsm_x4(a, qa + 2 * k);
            ldsm_x4(b, ka + 2 * k);
            mma_bf16(sc[0], a[0], a[1], a[2], a[3], b[0], b[1]);
            mma_bf16(sc[1], a[0], a[1], a[2], a[3], b[2], b[3]);
        }
        float x0 = m0, x1 = m1;
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const int key = page * KV_PAGE + 8 * j + 2 * tq + e;
                const bool on = key >= lo && key <= pos;
                float f = s.scale;
                if (SHARED) f *= row_factor(kt + (8 * j + 2 * tq + e) * LD, c.dim16);
                sc[j][e] = on ? (REL ? fmaf(sc[j][e], f, b0[j][e]) : sc[j][e] * f) : -INFINITY;
                sc[j][2 + e] = on ? (REL ? fmaf(sc[j][2 + e], f, b1[j][e]) : sc[j][2 + e] * f) : -INFINITY;
                x0 = fmaxf(x0, sc[j][e]);
                x1 = fmaxf(x1, sc[j][2 + e]);
            }
#pragma unroll
        for (int off = 1; off < 4; off <<= 1) {
            x0 = fmaxf(x0, __shfl_xor_sync(0xFFFFFFFFu, x0, off));
            if (!PACKED) x1 = fmaxf(x1, __shfl_xor_sync(0xFFFFFFFFu, x1, off));
        }
        // every page visited has a visible key, so the maxima are finite
        const float c0 = expf(m0 - x0), c1 = PACKED ? c0 : expf(m1 - x1);
        m0 = x0;
        m1 = x1;
        uint32_t hi[4], lw[4];
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
            for (int r2 = 0; r2 < (PACKED ? 1 : 2); ++r2) {
                const float a = expf(sc[j][2 * r2] - (r2 ? m1 : m0)), b = expf(sc[j][2 * r2 + 1] - (r2 ? m1 : m0));
                const uint32_t w = pack_bf16(a, b);
                const float2 back = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&w));
                hi[2 * j + r2] = w;
                lw[2 * j + r2] = pack_bf16(a - back.x, b - back.y);
                if (r2) l1 = (j ? l1 : l1 * c1) + a + b;
                else l0 = (j ? l0 : l0 * c0) + a + b;
            }
        if (PACKED) {  // row g + 8: the remainders of row g
            hi[1] = lw[0];
            hi[3] = lw[2];
        }
#pragma unroll
        for (int i = 0; i < VT; ++i) { o[i][0] *= c0; o[i][1] *= c0; o[i][2] *= c1; o[i][3] *= c1; }
        const uint32_t va = smem_addr(kt + (lane & 15) * LD + val + (lane >> 4) * 8);
#pragma unroll
        for (int i = 0; i < VT; i += 2) {
            if (i * 8 < c.vdim16) {
                uint32_t b[4];
                ldsm_x4_t(b, va + 2 * (i * 8));
                mma_bf16(o[i], hi[0], hi[1], hi[2], hi[3], b[0], b[1]);
                mma_bf16(o[i + 1], hi[0], hi[1], hi[2], hi[3], b[2], b[3]);
                if (!PACKED) {
                    mma_bf16(o[i], lw[0], lw[1], lw[2], lw[3], b[0], b[1]);
                    mma_bf16(o[i + 1], lw[0], lw[1], lw[2], lw[3], b[2], b[3]);
                }
            }
        }
        __syncwarp();  // the stage has been read
        fetch(page + GD_STAGES * stride, st);
    }
    cp_async_wait<0>();
#pragma unroll
    for (int off = 1; off < 4; off <<= 1) {
        l0 += __shfl_xor_sync(0xFFFFFFFFu, l0, off);
        if (!PACKED) l1 += __shfl_xor_sync(0xFFFFFFFFu, l1, off);
    }
    if (tq == 0) {
        m_s[warp][g] = m0;
        l_s[warp][g] = l0;
        m_s[warp][g + 8] = PACKED ? -INFINITY : m1;
        l_s[warp][g + 8] = PACKED ? 0.f : l1;
    }
    __syncthreads();
    // the warps' mixtures, each relative to its own maxima, where the ring was
    const int LO = c.vdim16 + 4, rows = PACKED ? 8 : 16;
    float* os = reinterpret_cast<float*>(gd_sm);
#pragma unroll
    for (int i = 0; i < VT; ++i) {
        if (i * 8 < c.vdim16) {
            float* d = os + (warp * rows + g) * LO + i * 8 + 2 * tq;
            if (PACKED) *reinterpret_cast<float2*>(d) = make_float2(o[i][0] + o[i][2], o[i][1] + o[i][3]);
            else {
                *reinterpret_cast<float2*>(d) = make_float2(o[i][0], o[i][1]);
                *reinterpret_cast<float2*>(d + 8 * LO) = make_float2(o[i][2], o[i][3]);
            }
        }
    }
    if (tid < 16) {
        float M = -INFINITY, L = 0.f;
#pragma unroll
        for (int w = 0; w < GD_WARPS; ++w) M = fmaxf(M, m_s[w][tid]);
#pragma unroll
        for (int w = 0; w < GD_WARPS; ++w) {
            const float f = m_s[w][tid] == -INFINITY ? 0.f : expf(m_s[w][tid] - M);
            L = fmaf(f, l_s[w][tid], L);
            m_s[w][tid] = f;
        }
        bm_s[tid] = M;
        bl_s[tid] = L;
    }
    __syncthreads();
    for (int i = tid; i < nq * s.vdim; i += GD_WARPS * 32) {  // the block's mixture, in the first warp's place
        const int r = i / s.vdim, e = i - r * s.vdim;
        float v = 0.f;
#pragma unroll
        for (int w = 0; w < GD_WARPS; ++w) v = fmaf(m_s[w][r], os[(w * rows + r) * LO + e], v);
        os[r * LO + e] = v;
    }
    if (n_splits > 1) cluster_sync();
    else __syncthreads();
    // a thread per (head, split): its share of the sum
    if (tid < 16 * GD_MAX_SPLITS) {
        const int r = tid / GD_MAX_SPLITS, p = tid % GD_MAX_SPLITS;
        const bool on = p < n_splits;
        const float mp = !on ? -INFINITY : n_splits == 1 ? bm_s[r] : ld_peer(peer_smem(smem_addr(bm_s + r), p));
        const float lp = !on ? 0.f : n_splits == 1 ? bl_s[r] : ld_peer(peer_smem(smem_addr(bl_s + r), p));
        float M = mp;
#pragma unroll
        for (int off = GD_MAX_SPLITS / 2; off > 0; off >>= 1) M = fmaxf(M, __shfl_xor_sync(0xFFFFFFFFu, M, off));
        const float sink = x.sink && r < nq ? x.sink[h0 + r] : -INFINITY;
        M = fmaxf(M, sink);
        const float f = mp == -INFINITY ? 0.f : expf(mp - M);
        float L = f * lp;
#pragma unroll
        for (int off = GD_MAX_SPLITS / 2; off > 0; off >>= 1) L += __shfl_xor_sync(0xFFFFFFFFu, L, off);
        if (sink != -INFINITY) L += expf(sink - M);
        share_s[r][p] = f / L;
    }
    __syncthreads();
    const int half = (s.vdim + 1) / 2;
    const float2* cs = x.cs_val ? x.cs_val + (int64_t)pos * half : nullptr;
    for (int i = blockIdx.z * GD_WARPS * 32 + tid; i < nq * half; i += n_splits * GD_WARPS * 32) {
        const int r = i / half, e = i - r * half;
        const bool two = e + half < s.vdim;
        float u = 0.f, v = 0.f;
        if (n_splits == 1) {
            u = share_s[r][0] * os[r * LO + e];
            if (two) v = share_s[r][0] * os[r * LO + e + half];
        } else {
            const uint32_t a = smem_addr(os + r * LO + e);
            for (int p = 0; p < n_splits; ++p) {
                if (share_s[r][p] == 0.f) continue;
                const uint32_t pa = peer_smem(a, p);
                u = fmaf(share_s[r][p], ld_peer(pa), u);
                if (two) v = fmaf(share_s[r][p], ld_peer(pa + 4 * half), v);
            }
        }
        bf16* d = out + (int64_t)t * ldo + (int64_t)(h0 + r) * s.vdim;
        const float* gate = gate_row(x, t, h0 + r, s.vdim);
        if (two) store_mixed<bf16>(d, e, half, u, v, cs, gate);
        else store_one<bf16>(d, e, u, gate);
    }
    if (n_splits > 1) cluster_sync();  // nobody leaves while its mixture is being read
}

bool grouped_mma_supported(const GroupedShape& s) { return s.dim <= 256 && s.vdim <= 256; }

int grouped_attention_splits(const GroupedShape& s, int n_tok, int keys, bool f32) {
    if (f32 || !grouped_mma_supported(s)) return 1;
    const int group = s.heads / s.kv_heads, blocks = s.kv_heads * ((group + 15) / 16) * n_tok, slots = 2 * device_sm_count();
    int n = 1;
    while (n < GD_MAX_SPLITS && blocks * 2 * n <= slots && keys >= 128 * 2 * n) n <<= 1;
    return n;
}

using GroupedDecodeFn = void (*)(const bf16*, GroupedShape, GroupedCache, GroupedTerms, const int32_t*, const int32_t*, bf16*, int, int);
template <int VT>
static GroupedDecodeFn gd_kernel(bool packed, bool rel, bool shared) {
    if (packed) return rel ? (shared ? grouped_decode_kernel<VT, true, true, true> : grouped_decode_kernel<VT, true, true, false>)
                           : (shared ? grouped_decode_kernel<VT, true, false, true> : grouped_decode_kernel<VT, true, false, false>);
    return rel ? (shared ? grouped_decode_kernel<VT, false, true, true> : grouped_decode_kernel<VT, false, true, false>)
               : (shared ? grouped_decode_kernel<VT, false, false, true> : grouped_decode_kernel<VT, false, false, false>);
}
static GroupedDecodeFn gd_kernel(int vdim16, bool packed, bool rel, bool shared) {
    return vdim16 <= 32 ? gd_kernel<4>(packed, rel, shared) : vdim16 <= 64 ? gd_kernel<8>(packed, rel, shared)
                      : vdim16 <= 128 ? gd_kernel<16>(packed, rel, shared) : gd_kernel<32>(packed, rel, shared);
}

cudaError_t launch_grouped_attention(const void* q, const GroupedShape& s, const GroupedCache& c, const GroupedTerms& x, const int32_t* tok_slot,
                                     const int32_t* tok_pos, void* out, int ldo, int n_splits, bool f32, int n_tok, cudaStream_t st) {
    if (n_tok == 0) return cudaSuccess;
    if (n_splits < 1 || n_splits > GD_MAX_SPLITS || (n_splits & (n_splits - 1)) || s.vdim > GROUPED_MAX_VDIM) return cudaErrorInvalidValue;
    cudaError_t le;
    if (!f32 && grouped_mma_supported(s)) {
        constexpr int CAP = 220 * 1024;
        static PerDeviceOnce once;
        le = once.run([] {
            for (int i = 0; i < 32; ++i) {
                const cudaError_t e = cudaFuncSetAttribute((const void*)gd_kernel(32 << (i >> 3), i & 1, i & 2, i & 4), cudaFuncAttributeMaxDynamicSharedMemorySize, CAP);
                if (e != cudaSuccess) return e;
            }
            return cudaSuccess;
        });
        if (le != cudaSuccess) return le;
        const int group = s.heads / s.kv_heads;
        const size_t smem = gd_smem(c);
        if (smem > CAP) return cudaErrorInvalidValue;
        const dim3 grid(s.kv_heads * ((group + 15) / 16), n_tok, n_splits), block(GD_WARPS * 32);
        le = launch_pdl_cluster(gd_kernel(c.vdim16, group <= 8, x.rel, c.shared), grid, block, smem, st, n_splits, (const bf16*)q, s, c, x, tok_slot, tok_pos,
                                (bf16*)out, ldo, n_splits);
        return le != cudaSuccess ? le : count_launch_and_check();
    }
    const dim3 grid(s.heads, n_tok), block(GS_WARPS * 32);
    const size_t smem = (size_t)(c.dim16 + GS_WARPS * s.vdim) * 4;
    if (n_splits != 1 || smem > 48 * 1024) return cudaErrorInvalidValue;
    le = f32 ? launch_pdl(grouped_simple_kernel<float>, grid, block, smem, st, (const float*)q, s, c, x, tok_slot, tok_pos, (float*)out, ldo)
             : launch_pdl(grouped_simple_kernel<bf16>, grid, block, smem, st, (const bf16*)q, s, c, x, tok_slot, tok_pos, (bf16*)out, ldo);
    return le != cudaSuccess ? le : count_launch_and_check();
}

// ── many rows, bf16 ──
// Block per (head, tile of 64 tokens), 4 warps x 16 query rows, key tiles of four pages double-buffered with cp.async.
constexpr int GP_KEYS = 64, GP_WARPS = 4;
static_assert(GROUPED_TAIL == 8, "a shared row's tail is the padding of its row in shared memory");
static size_t gp_smem(const GroupedCache& c) { return (size_t)(3 * 64 * (c.dim16 + 8) + (c.shared ? 0 : 2 * GP_KEYS * (c.vdim16 + 8))) * 2; }

template <int VT, bool REL, bool SHARED>
__global__ void __launch_bounds__(GP_WARPS * 32) grouped_prefill_kernel(const bf16* __restrict__ q, const GroupedShape s, const GroupedCache c,
                                                                     const GroupedTerms x, const GroupedTile* __restrict__ tiles,
                                                                     bf16* __restrict__ out, int ldo) {
    extern __shared__ __align__(16) bf16 gp_sm[];
    __shared__ float rel_s[2][REL ? GP_KEYS + 64 : 1];  // biases of a key tile: by 63 - (query row) + (key in the tile)
    pdl_wait();
    pdl_trigger();
    const int LQ = c.dim16 + 8, LV = c.vdim16 + 8, ld = c.ld;  // (shared: LV == LQ)
    bf16 *qs = gp_sm, *ks = qs + 64 * LQ, *vs = SHARED ? ks : ks + 2 * GP_KEYS * LQ;
    const int k_pieces = (SHARED ? c.ld : c.dim16) / 8, v_pieces = SHARED ? 0 : c.vdim16 / 8;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, tq = lane & 3;
    const int h = blockIdx.x, kvh = h / (s.heads / s.kv_heads);
    const GroupedTile tl = tiles[blockIdx.y];
    const int32_t* pt = c.page_table + (int64_t)tl.slot * c.max_pages;
    const int l8 = lane & 7, lr = warp * 16 + (lane >> 3);  // copies: eight lanes per row, a page per warp
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int r = lr + 4 * i;
        const bf16* src = q + ((int64_t)(tl.row0 + min(r, tl.n - 1)) * s.heads + h) * c.dim16;
        for (int p = l8; p < c.dim16 / 8; p += 8) cp_async16(qs + r * LQ + p * 8, src + p * 8, 16);
    }
    const float* rel = REL ? x.rel + (int64_t)h * x.n_rel : nullptr;
    const float far = REL ? rel[x.n_rel - 1] : 0.f;
    const int hi = tl.pos0 + tl.n - 1, lo = (s.window > tl.pos0 ? 0 : tl.pos0 - s.window + 1) / KV_PAGE * KV_PAGE;
    auto fetch = [&](int k0, int buf) {
        const int page = k0 / KV_PAGE + warp;
        const bool live = page * KV_PAGE <= hi;
        const bf16* base = reinterpret_cast<const bf16*>(c.pool) + ((int64_t)(live ? pt[page] : 0) * s.kv_heads + kvh) * KV_PAGE * ld;
        bf16 *kd = ks + buf * GP_KEYS * LQ, *vd = vs + buf * GP_KEYS * LV;
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int r = lr + 4 * i, bytes = k0 + r <= hi ? 16 : 0;  // keys past the newest: zeros
            const bf16* src = base + (r - warp * 16) * ld;
            for (int p = l8; p < k_pieces; p += 8) cp_async16(kd + r * LQ + p * 8, src + p * 8, bytes);
            for (int p = l8; p < v_pieces; p += 8) cp_async16(vd + r * LV + p * 8, src + c.dim16 + p * 8, bytes);
        }
        if (REL && tid < GP_KEYS + 63) {  // (distances below zero are of keys that are not seen)
            const int dist = max(0, min(tl.pos0 + 63 - k0 - tid, x.n_rel - 1));
            cp_async4(&rel_s[buf][tid], rel + dist);
        }
    };
    fetch(lo, 0);
    cp_async_commit();
    float o[VT][4];
#pragma unroll
    for (int i = 0; i < VT; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
    float m0 = -INFINITY, m1 = -INFINITY, l0 = 0.f, l1 = 0.f;
    const int r0 = warp * 16 + g, r1 = r0 + 8;
    const int p0 = tl.pos0 + min(r0, tl.n - 1), p1 = tl.pos0 + min(r1, tl.n - 1);
    for (int k0 = lo, buf = 0; k0 <= hi; k0 += GP_KEYS, buf ^= 1) {
        cp_async_wait<0>();
        __syncthreads();
        if (k0 + GP_KEYS <= hi) fetch(k0 + GP_KEYS, buf ^ 1);
        cp_async_commit();
        const bf16 *kt = ks + buf * GP_KEYS * LQ, *vt = vs + buf * GP_KEYS * LV;
        float sc[8][4];
#pragma unroll
        for (int j = 0; j < 8; ++j) sc[j][0] = sc[j][1] = sc[j][2] = sc[j][3] = 0.f;
        const uint32_t qa = smem_addr(qs + (warp * 16 + (lane & 15)) * LQ + (lane >> 4) * 8);
        const uint32_t ka = smem_addr(kt + ((lane & 7) + (lane >> 4) * 8) * LQ + ((lane >> 3) & 1) * 8);
        for (int k = 0; k < c.dim16; k += 16) {
            uint32_t a[4];
            ldsm_x4(a, qa + 2 * k);
#pragma unroll
            for (int j = 0; j < 8; j += 2) {
                uint32_t b[4];
                ldsm_x4(b, ka + 2 * (8 * j * LQ + k));
                mma_bf16(sc[j], a[0], a[1], a[2], a[3], b[0], b[1]);
                mma_bf16(sc[j + 1], a[0], a[1], a[2], a[3], b[2], b[3]);
            }
        }
        float x0 = m0, x1 = m1;
        const bool near = REL && tl.pos0 - (k0 + GP_KEYS - 1) < x.n_rel - 1;
        const float* rs = REL ? &rel_s[buf][63 - r0 + 2 * tq] : nullptr;  // of key 2 tq; the other row's stand eight before
        const bool edge = k0 + GP_KEYS - 1 > tl.pos0 || (int64_t)hi - k0 >= s.window;  // only the window's ends need the mask
#pragma unroll
        for (int j = 0; j < 8; ++j) {
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const int key = k0 + 8 * j + 2 * tq + e;
                float f = s.scale, b0 = far, b1 = far;
                if (SHARED) f *= row_factor(kt + (8 * j + 2 * tq + e) * LQ, c.dim16);
                if (near) {
                    b0 = rs[8 * j + e];
                    b1 = rs[8 * j + e - 8];
                }
                sc[j][e] = (!edge || (key <= p0 && p0 - key < s.window)) ? (REL ? fmaf(sc[j][e], f, b0) : sc[j][e] * f) : -INFINITY;
                sc[j][2 + e] = (!edge || (key <= p1 && p1 - key < s.window)) ? (REL ? fmaf(sc[j][2 + e], f, b1) : sc[j][2 + e] * f) : -INFINITY;
                x0 = fmaxf(x0, sc[j][e]);
                x1 = fmaxf(x1, sc[j][2 + e]);
            }
        }
#pragma unroll
        for (int off = 1; off < 4; off <<= 1) {
            x0 = fmaxf(x0, __shfl_xor_sync(0xFFFFFFFFu, x0, off));
            x1 = fmaxf(x1, __shfl_xor_sync(0xFFFFFFFFu, x1, off));
        }
        // a row that has seen no visible key yet keeps everything at zero
        const float b0 = x0 == -INFINITY ? 0.f : x0, b1 = x1 == -INFINITY ? 0.f : x1;
        const float c0 = expf(m0 - b0), c1 = expf(m1 - b1);
        float s0 = 0.f, s1 = 0.f;
#pragma unroll
        for (int j = 0; j < 8; ++j) {
            sc[j][0] = __expf(sc[j][0] - b0); sc[j][1] = __expf(sc[j][1] - b0);
            sc[j][2] = __expf(sc[j][2] - b1); sc[j][3] = __expf(sc[j][3] - b1);
            s0 += sc[j][0] + sc[j][1];
            s1 += sc[j][2] + sc[j][3];
        }
        l0 = fmaf(l0, c0, s0);
        l1 = fmaf(l1, c1, s1);
        m0 = x0;
        m1 = x1;
#pragma unroll
        for (int i = 0; i < VT; ++i) { o[i][0] *= c0; o[i][1] *= c0; o[i][2] *= c1; o[i][3] *= c1; }
#pragma unroll
        for (int kk = 0; kk < 4; ++kk) {
            uint32_t a[4], r[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const float u = sc[2 * kk + (i >> 1)][2 * (i & 1)], v = sc[2 * kk + (i >> 1)][2 * (i & 1) + 1];
                a[i] = pack_bf16(u, v);
                const float2 back = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&a[i]));
                r[i] = pack_bf16(u - back.x, v - back.y);
            }
            const uint32_t va = smem_addr(vt + (kk * 16 + (lane & 15)) * LV + (lane >> 4) * 8);
#pragma unroll
            for (int i = 0; i < VT; i += 2) {
                if (i * 8 < c.vdim16) {
                    uint32_t b[4];
                    ldsm_x4_t(b, va + 2 * (i * 8));
                    mma_bf16(o[i], a[0], a[1], a[2], a[3], b[0], b[1]);
                    mma_bf16(o[i + 1], a[0], a[1], a[2], a[3], b[2], b[3]);
                    mma_bf16(o[i], r[0], r[1], r[2], r[3], b[0], b[1]);
                    mma_bf16(o[i + 1], r[0], r[1], r[2], r[3], b[2], b[3]);
                }
            }
        }
    }
    cp_async_wait<0>();
#pragma unroll
    for (int off = 1; off < 4; off <<= 1) {
        l0 += __shfl_xor_sync(0xFFFFFFFFu, l0, off);
        l1 += __shfl_xor_sync(0xFFFFFFFFu, l1, off);
    }
    float f0 = 1.f / l0, f1 = 1.f / l1;
    if (x.sink) {
        const float sink = x.sink[h], M0 = fmaxf(m0, sink), M1 = fmaxf(m1, sink), e0 = expf(m0 - M0), e1 = expf(m1 - M1);
        f0 = e0 / fmaf(l0, e0, expf(sink - M0));
        f1 = e1 / fmaf(l1, e1, expf(sink - M1));
    }
    // a coordinate's partner is half a head away: the warp's rows meet in shared memory, a column range at a time
    __syncthreads();
    const int LO = c.vdim16 + 4;
    float* os = reinterpret_cast<float*>(gp_sm) + warp * 16 * LO;
#pragma unroll
    for (int i = 0; i < VT; ++i) {
        if (i * 8 < c.vdim16) {
            float* d = os + g * LO + i * 8 + 2 * tq;
            *reinterpret_cast<float2*>(d) = make_float2(o[i][0] * f0, o[i][1] * f0);
            *reinterpret_cast<float2*>(d + 8 * LO) = make_float2(o[i][2] * f1, o[i][3] * f1);
        }
    }
    __syncwarp();
    const int half = s.vdim / 2;
    for (int r = 0; r < 16 && warp * 16 + r < tl.n; ++r) {
        const int row = warp * 16 + r;
        bf16* d = out + (int64_t)(tl.row0 + row) * ldo + (int64_t)h * s.vdim;
        const float2* cs = x.cs_val ? x.cs_val + (int64_t)(tl.pos0 + row) * half : nullptr;
        const float* gate = gate_row(x, tl.row0 + row, h, s.vdim);
        for (int e = lane; e < half; e += 32) store_mixed<bf16>(d, e, half, os[r * LO + e], os[r * LO + e + half], cs, gate);
        if ((s.vdim & 1) && lane == 0) store_one<bf16>(d, s.vdim - 1, os[r * LO + s.vdim - 1], gate);
    }
}

using GroupedPrefillFn = void (*)(const bf16*, GroupedShape, GroupedCache, GroupedTerms, const GroupedTile*, bf16*, int);
template <int VT>
static GroupedPrefillFn gp_kernel(bool rel, bool shared) {
    return rel ? (shared ? grouped_prefill_kernel<VT, true, true> : grouped_prefill_kernel<VT, true, false>)
               : (shared ? grouped_prefill_kernel<VT, false, true> : grouped_prefill_kernel<VT, false, false>);
}
static GroupedPrefillFn gp_kernel(int vdim16, bool rel, bool shared) {
    return vdim16 <= 32 ? gp_kernel<4>(rel, shared) : vdim16 <= 64 ? gp_kernel<8>(rel, shared)
                      : vdim16 <= 128 ? gp_kernel<16>(rel, shared) : gp_kernel<32>(rel, shared);
}

cudaError_t launch_grouped_prefill(const void* q, const GroupedShape& s, const GroupedCache& c, const GroupedTerms& x, const GroupedTile* tiles,
                                   int n_tiles, void* out, int ldo, cudaStream_t st) {
    if (n_tiles == 0) return cudaSuccess;
    const size_t smem = std::max(gp_smem(c), (size_t)GP_WARPS * 16 * (c.vdim16 + 4) * 4);
    constexpr int CAP = 200 * 1024;
    if (!grouped_mma_supported(s) || smem > CAP) return cudaErrorInvalidValue;
    static PerDeviceOnce once;
    cudaError_t le = once.run([] {
        for (int i = 0; i < 16; ++i) {
            const cudaError_t e = cudaFuncSetAttribute((const void*)gp_kernel(32 << (i >> 2), i & 1, i & 2), cudaFuncAttributeMaxDynamicSharedMemorySize, CAP);
            if (e != cudaSuccess) return e;
        }
        return cudaSuccess;
    });
    if (le != cudaSuccess) return le;
    const dim3 grid(s.heads, n_tiles), block(GP_WARPS * 32);
    le = launch_pdl(gp_kernel(c.vdim16, x.rel, c.shared), grid, block, smem, st, (const bf16*)q, s, c, x, tiles, (bf16*)out, ldo);
    return le != cudaSuccess ? le : count_launch_and_check();
}

}  // namespace sp
