// Grouped attention whose heads' softmax weights are mixed before they meet the values (plan_kernels.h). A head's mixture needs the
// normalised weights of all heads, so scores and denominators come first, weights and values second:
//   few rows    mixed_scores_kernel leaves scores (in powers of two, below their cap) and, per split of the keys, maximum and sum;
//               mixed_mix_kernel makes the weights of all heads where it needs them, mixes them as a small product (16 output heads x
//               heads x keys) whose accumulators are the A operand of the product with the values, and adds the splits' shares
//               over a cluster.
//   many rows   mixed_stats_kernel walks the keys of 64 query rows per head; mixed_prefill_kernel has 16 query rows of all heads (a
//               cluster where one block cannot hold them): every warp makes its heads' weights for a page of keys, all read all of
//               them. mixed_prefill_halves_kernel does that for common sizes with half of its warps a page ahead of the others.
//   any sizes   simple_scores_kernel, simple_mix_kernel: plain arithmetic, rows in batches that the scratch holds.
// The products' bf16 operands that stand for weights are a leading part plus its remainder; everything else is f32. Pages that hold
// kept first keys and pages of the window are one run of visited pages.
#include <algorithm>
#include <atomic>
#include <climits>

#include "kernels.h"
#include "pdl.cuh"
#include "plan_common.cuh"
#include "plan_kernels.h"
#include "sp_common.cuh"

namespace sp {

cudaError_t count_launch_and_check();  // kernels.cu

// Pages visited by queries at positions p0 .. p1: `kept` pages from the first, then those from page `first` to the one of p1.
struct Visit {
    int kept, first, pages;
    __device__ __forceinline__ Visit(const GroupedShape& s, int p0, int p1) {
        first = (s.window > p0 ? 0 : p0 - s.window + 1) / KV_PAGE;
        kept = min((s.keep + KV_PAGE - 1) / KV_PAGE, first);
        pages = kept + p1 / KV_PAGE - first + 1;
    }
    __device__ __forceinline__ int page(int v) const { return v < kept ? v : first + v - kept; }
};
__device__ __forceinline__ bool visible(const GroupedShape& s, int key, int pos) { return key <= pos && (pos - key < s.window || key < s.keep); }

int mixed_span(const GroupedShape& s, int max_ctx) {
    const int64_t window = (int64_t)s.window + 2 * KV_PAGE + (s.keep + KV_PAGE - 1) / KV_PAGE * KV_PAGE;
    return (int)((std::min<int64_t>(window, max_ctx) + KV_PAGE - 1) / KV_PAGE * KV_PAGE);
}

// The scaled and capped score of a dot product.
__device__ __forceinline__ float score_of(const GroupedShape& s, float dot) {
    const float z = dot * s.scale;
    return s.softcap > 0.f ? s.softcap * tanhf(z / s.softcap) : z;
}
// The tensor-core kernels' version, in powers of two: log2 e^(score - top), where top is the cap (no cap: 0). tanh z = 1 - 2 / (e^(2 z) + 1)
// has an absolute error, as softmax needs it.
constexpr float LOG2E = 1.4426950408889634f;
__device__ __forceinline__ float exp2_fast(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;\n" : "=f"(y) : "f"(x));
    return y;
}
__device__ __forceinline__ float rcp_fast(float x) {
    float y;
    asm("rcp.approx.ftz.f32 %0, %1;\n" : "=f"(y) : "f"(x));
    return y;
}
struct Log2Score {
    float a, b, top;
    bool cap;
    __device__ __forceinline__ explicit Log2Score(const GroupedShape& s) : cap(s.softcap > 0.f) {
        a = cap ? 2.f * s.scale / s.softcap * LOG2E : s.scale * LOG2E;
        b = -2.f * s.softcap * LOG2E;
        top = cap ? s.softcap : 0.f;
    }
    __device__ __forceinline__ float operator()(float dot, float more) const {  // ... plus `more`
        return cap ? fmaf(b, rcp_fast(exp2_fast(dot * a) + 1.f), more) : fmaf(dot, a, more);
    }
};
// What to add to a log2 score for its normalised weight: maximum and sum of the keys, and the sink.
__device__ __forceinline__ float log2_norm(float m, float l, float sink) {
    const float M = fmaxf(m, sink);
    return -M - log2f(l * exp2f(m - M) + exp2f(sink - M));
}

__device__ __forceinline__ float2 stat_of(float m, float l, const float* sink, int h) {  // maximum, 1 / denominator
    if (sink) {
        const float M = fmaxf(m, sink[h]);
        l = l * expf(m - M) + expf(sink[h] - M);
        m = M;
    }
    return make_float2(m, 1.f / l);
}

// ── any sizes ──
constexpr int MS_WARPS = 4, MS_PER_LANE = GROUPED_MAX_VDIM / 32;
template <typename T>
__global__ void __launch_bounds__(MS_WARPS * 32) simple_scores_kernel(const T* __restrict__ q, const GroupedShape s, const GroupedCache c, const MixedTerms x,
                                                                   const MixedScratch m, const int32_t* __restrict__ tok_slot,
                                                                   const int32_t* __restrict__ tok_pos, int t0) {
    extern __shared__ float ms_q[];
    __shared__ float sm[MS_WARPS], sl[MS_WARPS];
    pdl_wait();
    pdl_trigger();
    const int h = blockIdx.x, t = t0 + blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = h / (s.heads / s.kv_heads), pos = tok_pos[t];
    for (int i = threadIdx.x; i < s.dim; i += MS_WARPS * 32) ms_q[i] = to_f32(q[((int64_t)t * s.heads + h) * c.dim16 + i]);
    __syncthreads();
    const int32_t* pt = c.page_table + (int64_t)tok_slot[t] * c.max_pages;
    const Visit vis(s, pos, pos);
    float* out = m.score + ((int64_t)blockIdx.y * s.heads + h) * m.span;
    float mx = -INFINITY, l = 0.f;
    for (int i = warp; i < vis.pages * KV_PAGE; i += MS_WARPS) {
        const int page = vis.page(i / KV_PAGE), key = page * KV_PAGE + i % KV_PAGE;
        float sc = -INFINITY;
        if (visible(s, key, pos)) {
            const T* row = reinterpret_cast<const T*>(c.pool) + (((int64_t)pt[page] * s.kv_heads + g) * KV_PAGE + i % KV_PAGE) * c.ld;
            float dot = 0.f;
            for (int e = lane; e < s.dim; e += 32) dot = fmaf(ms_q[e], to_f32(row[e]), dot);
            sc = score_of(s, warp_sum(dot));
            const float mn = fmaxf(mx, sc);
            l = fmaf(l, expf(mx - mn), expf(sc - mn));
            mx = mn;
        }
        if (lane == 0) out[i] = sc;
    }
    if (lane == 0) { sm[warp] = mx; sl[warp] = l; }
    __syncthreads();
    if (threadIdx.x == 0) {
        float M = -INFINITY, L = 0.f;
        for (int w = 0; w < MS_WARPS; ++w) M = fmaxf(M, sm[w]);
        for (int w = 0; w < MS_WARPS; ++w) L += sm[w] == -INFINITY ? 0.f : sl[w] * expf(sm[w] - M);
        m.stat[(int64_t)t * s.heads + h] = stat_of(M, L, x.sink, h);
    }
}

template <typename T>
__global__ void __launch_bounds__(MS_WARPS * 32) simple_mix_kernel(const GroupedShape s, const GroupedCache c, const MixedTerms x, const MixedScratch m,
                                                                const int32_t* __restrict__ tok_slot, const int32_t* __restrict__ tok_pos, int t0,
                                                                T* __restrict__ out, int ldo) {
    extern __shared__ float ms_o[];  // an output row per warp
    pdl_wait();
    pdl_trigger();
    const int h = blockIdx.x, t = t0 + blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = h / (s.heads / s.kv_heads), pos = tok_pos[t];
    const int32_t* pt = c.page_table + (int64_t)tok_slot[t] * c.max_pages;
    const Visit vis(s, pos, pos);
    const float* score = m.score + (int64_t)blockIdx.y * s.heads * m.span;
    const float2* stat = m.stat + (int64_t)t * s.heads;
    float o[MS_PER_LANE];
#pragma unroll
    for (int i = 0; i < MS_PER_LANE; ++i) o[i] = 0.f;
    for (int i = warp; i < vis.pages * KV_PAGE; i += MS_WARPS) {
        const int page = vis.page(i / KV_PAGE);
        if (!visible(s, page * KV_PAGE + i % KV_PAGE, pos)) continue;
        float p = 0.f;
        for (int e = lane; e < s.heads; e += 32) p = fmaf(x.mix[(int64_t)h * s.heads + e], expf(score[(int64_t)e * m.span + i] - stat[e].x) * stat[e].y, p);
        p = warp_sum(p);
        const T* row = reinterpret_cast<const T*>(c.pool) + (((int64_t)pt[page] * s.kv_heads + g) * KV_PAGE + i % KV_PAGE) * c.ld + c.dim16;
#pragma unroll
        for (int j = 0; j < MS_PER_LANE; ++j)
            if (lane + 32 * j < s.vdim) o[j] = fmaf(p, to_f32(row[lane + 32 * j]), o[j]);
    }
#pragma unroll
    for (int j = 0; j < MS_PER_LANE; ++j)
        if (lane + 32 * j < s.vdim) ms_o[warp * s.vdim + lane + 32 * j] = o[j];
    __syncthreads();
    for (int e = threadIdx.x; e < s.vdim; e += MS_WARPS * 32) {
        float v = 0.f;
#pragma unroll
        for (int w = 0; w < MS_WARPS; ++w) v += ms_o[w * s.vdim + e];
        out[(int64_t)t * ldo + (int64_t)h * s.vdim + e] = from_f32<T>(v);
    }
}

template <typename T>
static cudaError_t simple_launch(const T* q, const GroupedShape& s, const GroupedCache& c, const MixedTerms& x, const MixedScratch& m, const int32_t* tok_slot,
                                 const int32_t* tok_pos, T* out, int ldo, int n_tok, cudaStream_t st) {
    for (int t0 = 0; t0 < n_tok; t0 += m.rows) {
        const dim3 grid(s.heads, std::min(m.rows, n_tok - t0)), block(MS_WARPS * 32);
        cudaError_t le = launch_pdl(simple_scores_kernel<T>, grid, block, (size_t)s.dim * 4, st, q, s, c, x, m, tok_slot, tok_pos, t0);
        if (le == cudaSuccess) le = count_launch_and_check();
        if (le == cudaSuccess) le = launch_pdl(simple_mix_kernel<T>, grid, block, (size_t)MS_WARPS * s.vdim * 4, st, s, c, x, m, tok_slot, tok_pos, t0, out, ldo);
        if (le == cudaSuccess) le = count_launch_and_check();
        if (le != cudaSuccess) return le;
    }
    return cudaSuccess;
}

// ── few rows ──
// Blocks as in grouped_attention.cu: (cached head, 16 of its query heads; token; split of the keys), four warps that walk pages of
// their own with three stages of cp.async.
constexpr int MD_WARPS = 4, MD_STAGES = 3;

// `width` elements (a multiple of 8) of each row of a page, at column `col`, to rows of ld_s elements.
__device__ __forceinline__ void fetch_page(const GroupedCache& c, int kv_heads, int kvh, int page_id, int live, int col, int width, uint32_t dst, int ld_s, int lane, int lanes) {
    const bf16* src = reinterpret_cast<const bf16*>(c.pool) + ((int64_t)page_id * kv_heads + kvh) * KV_PAGE * c.ld + col;
    const int pieces = width / 8;
    int r = lane / pieces, p = lane - r * pieces;
    for (int i = lane; i < KV_PAGE * pieces; i += lanes) {
        cp_async16_at(dst + (uint32_t)(r * ld_s + p * 8) * 2, src + (int64_t)r * c.ld + p * 8, r < live ? 16 : 0);
        p += lanes;
        while (p >= pieces) { p -= pieces; ++r; }
    }
}

__global__ void __launch_bounds__(MD_WARPS * 32) mixed_scores_kernel(const bf16* __restrict__ q, const GroupedShape s, const GroupedCache c, const MixedScratch m,
                                                                  const int32_t* __restrict__ tok_slot, const int32_t* __restrict__ tok_pos, int n_splits) {
    extern __shared__ __align__(16) bf16 md_sm[];
    __shared__ float m_s[MD_WARPS][16], l_s[MD_WARPS][16];
    const int LD = c.dim16 + 8, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, tq = lane & 3;
    const int group = s.heads / s.kv_heads, tiles = (group + 15) / 16, kvh = blockIdx.x / tiles, h0 = kvh * group + (blockIdx.x % tiles) * 16;
    const int nq = min(16, (kvh + 1) * group - h0), t = blockIdx.y;
    bf16 *qs = md_sm, *ring = md_sm + 16 * LD + warp * MD_STAGES * KV_PAGE * LD;
    pdl_wait();
    pdl_trigger();
    const int pos = tok_pos[t], stride = MD_WARPS * n_splits;
    const Visit vis(s, pos, pos);
    const int32_t* pt = c.page_table + (int64_t)tok_slot[t] * c.max_pages;
    for (int i = tid; i < 16 * (c.dim16 / 8); i += MD_WARPS * 32) {
        const int r = i / (c.dim16 / 8), p = i - r * (c.dim16 / 8);
        *reinterpret_cast<uint4*>(qs + r * LD + p * 8) =
            r < nq ? *reinterpret_cast<const uint4*>(q + ((int64_t)t * s.heads + h0 + r) * c.dim16 + p * 8) : make_uint4(0u, 0u, 0u, 0u);
    }
    auto fetch = [&](int v, int st) {
        if (v < vis.pages) {
            const int page = vis.page(v);
            fetch_page(c, s.kv_heads, kvh, pt[page], pos - page * KV_PAGE + 1, 0, c.dim16, smem_addr(ring + st * KV_PAGE * LD), LD, lane, 32);
        }
        cp_async_commit();
    };
    const int v0 = blockIdx.z * MD_WARPS + warp;
#pragma unroll
    for (int i = 0; i < MD_STAGES; ++i) fetch(v0 + i * stride, i);
    __syncthreads();
    const Log2Score score(s);
    float m0 = -INFINITY, m1 = -INFINITY, l0 = 0.f, l1 = 0.f;  // maxima in powers of two, from the top
    const uint32_t qa = smem_addr(qs + (lane & 15) * LD + (lane >> 4) * 8);
    float* const out = m.score + ((int64_t)t * s.heads + h0) * m.span;
    for (int v = v0, st = 0; v < vis.pages; v += stride, st = st + 1 == MD_STAGES ? 0 : st + 1) {
        cp_async_wait<MD_STAGES - 1>();
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
        const int key0 = vis.page(v) * KV_PAGE;
        float x0 = m0, x1 = m1;
#pragma unroll
        for (int j = 0; j < 2; ++j) {
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const bool on = visible(s, key0 + 8 * j + 2 * tq + e, pos);
                sc[j][e] = on ? score(sc[j][e], 0.f) : -INFINITY;
                sc[j][2 + e] = on ? score(sc[j][2 + e], 0.f) : -INFINITY;
                x0 = fmaxf(x0, sc[j][e]);
                x1 = fmaxf(x1, sc[j][2 + e]);
            }
            float* d = out + v * KV_PAGE + 8 * j + 2 * tq;
            if (g < nq) *reinterpret_cast<float2*>(d + (int64_t)g * m.span) = make_float2(sc[j][0], sc[j][1]);
            if (g + 8 < nq) *reinterpret_cast<float2*>(d + (int64_t)(g + 8) * m.span) = make_float2(sc[j][2], sc[j][3]);
        }
        // (a thread's own maxima: its quad meets at the end; kept pages may show a thread nothing)
        const float b0 = x0 == -INFINITY ? 0.f : x0, b1 = x1 == -INFINITY ? 0.f : x1;
        l0 = l0 * exp2_fast(m0 - b0) + exp2_fast(sc[0][0] - b0) + exp2_fast(sc[0][1] - b0) + exp2_fast(sc[1][0] - b0) + exp2_fast(sc[1][1] - b0);
        l1 = l1 * exp2_fast(m1 - b1) + exp2_fast(sc[0][2] - b1) + exp2_fast(sc[0][3] - b1) + exp2_fast(sc[1][2] - b1) + exp2_fast(sc[1][3] - b1);
        m0 = x0;
        m1 = x1;
        __syncwarp();  // the stage has been read
        fetch(v + MD_STAGES * stride, st);
    }
    cp_async_wait<0>();
    auto meet = [](float& a, float& b, float om, float ol) {  // (maximum, sum) of two parts
        const float M = fmaxf(a, om), base = M == -INFINITY ? 0.f : M;
        b = b * exp2_fast(a - base) + ol * exp2_fast(om - base);
        a = M;
    };
#pragma unroll
    for (int off = 1; off < 4; off <<= 1) {
        meet(m0, l0, __shfl_xor_sync(0xFFFFFFFFu, m0, off), __shfl_xor_sync(0xFFFFFFFFu, l0, off));
        meet(m1, l1, __shfl_xor_sync(0xFFFFFFFFu, m1, off), __shfl_xor_sync(0xFFFFFFFFu, l1, off));
    }
    if (tq == 0) {
        m_s[warp][g] = m0;
        l_s[warp][g] = l0;
        m_s[warp][g + 8] = m1;
        l_s[warp][g + 8] = l1;
    }
    __syncthreads();
    if (tid < nq) {
        float M = m_s[0][tid], L = l_s[0][tid];
#pragma unroll
        for (int w = 1; w < MD_WARPS; ++w) meet(M, L, m_s[w][tid], l_s[w][tid]);
        m.part[((int64_t)t * s.heads + h0 + tid) * MIXED_SPLITS + blockIdx.z] = make_float2(M, L);
    }
}

// The splits of a token and cached head are a cluster. Shared memory: maxima and reciprocal denominators of all heads, the block's
// rows of the mixing matrix (leading part, remainder), the ring of values, where the shares meet at the end.
__host__ __device__ __forceinline__ int md_heads16(const GroupedShape& s) { return (s.heads + 15) & ~15; }
static size_t md_mix_smem(const GroupedShape& s, const GroupedCache& c) {
    const size_t head = (size_t)md_heads16(s) * 4 + (size_t)2 * 16 * (md_heads16(s) + 8) * 2;
    return head + std::max((size_t)MD_WARPS * MD_STAGES * KV_PAGE * (c.vdim16 + 8) * 2, (size_t)MD_WARPS * 16 * (c.vdim16 + 4) * 4);
}

template <int VT, bool PACKED>
__global__ void __launch_bounds__(MD_WARPS * 32) mixed_mix_kernel(const GroupedShape s, const GroupedCache c, const MixedTerms x, const MixedScratch m,
                                                               const int32_t* __restrict__ tok_slot, const int32_t* __restrict__ tok_pos,
                                                               bf16* __restrict__ out, int ldo, int n_splits) {
    extern __shared__ __align__(16) uint8_t mm_sm[];
    const int H16 = md_heads16(s), LT = H16 + 8, LV = c.vdim16 + 8, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, tq = lane & 3;
    const int group = s.heads / s.kv_heads, tiles = (group + 15) / 16, kvh = blockIdx.x / tiles, h0 = kvh * group + (blockIdx.x % tiles) * 16;
    const int nq = min(16, (kvh + 1) * group - h0), t = blockIdx.y;
    float* const norm = reinterpret_cast<float*>(mm_sm);  // what makes a head's score its weight, in powers of two
    bf16 *t_hi = reinterpret_cast<bf16*>(norm + H16), *t_lo = t_hi + 16 * LT, *rings = t_lo + 16 * LT, *ring = rings + warp * MD_STAGES * KV_PAGE * LV;
    for (int i = tid; i < 16 * H16; i += MD_WARPS * 32) {  // (no kernel writes the mixing matrix)
        const int r = i / H16, e = i - r * H16;
        const float v = r < nq && e < s.heads ? x.mix[(int64_t)(h0 + r) * s.heads + e] : 0.f;
        const bf16 hi = __float2bfloat16_rn(v);
        t_hi[r * LT + e] = hi;
        t_lo[r * LT + e] = __float2bfloat16_rn(v - __bfloat162float(hi));
    }
    pdl_wait();
    pdl_trigger();
    const int pos = tok_pos[t], stride = MD_WARPS * n_splits;
    const Visit vis(s, pos, pos);
    const int32_t* pt = c.page_table + (int64_t)tok_slot[t] * c.max_pages;
    auto fetch = [&](int v, int st) {
        if (v < vis.pages) {
            const int page = vis.page(v);
            fetch_page(c, s.kv_heads, kvh, pt[page], pos - page * KV_PAGE + 1, c.dim16, c.vdim16, smem_addr(ring + st * KV_PAGE * LV), LV, lane, 32);
        }
        cp_async_commit();
    };
    const int v0 = blockIdx.z * MD_WARPS + warp;
#pragma unroll
    for (int i = 0; i < MD_STAGES; ++i) fetch(v0 + i * stride, i);
    for (int h = tid; h < H16; h += MD_WARPS * 32) {
        float r = -INFINITY;  // heads that do not exist weigh nothing
        if (h < s.heads) {
            const float2* p = m.part + ((int64_t)t * s.heads + h) * MIXED_SPLITS;
            float M = -INFINITY, L = 0.f;
            for (int i = 0; i < n_splits; ++i) M = fmaxf(M, p[i].x);
            for (int i = 0; i < n_splits; ++i) L += p[i].x == -INFINITY ? 0.f : p[i].y * exp2f(p[i].x - M);
            r = log2_norm(M, L, x.sink ? (x.sink[h] - Log2Score(s).top) * LOG2E : -INFINITY);
        }
        norm[h] = r;
    }
    __syncthreads();
    float o[VT][4];
#pragma unroll
    for (int i = 0; i < VT; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
    const uint32_t ta = smem_addr(t_hi + (lane & 15) * LT + (lane >> 4) * 8), lo_off = 2u * 16 * LT;
    const float* const score = m.score + (int64_t)t * s.heads * m.span;
    for (int v = v0, st = 0; v < vis.pages; v += stride, st = st + 1 == MD_STAGES ? 0 : st + 1) {
        float p[2][4] = {};  // mixed weights: rows g and g + 8 (heads), keys 8 j + 2 tq and the next
        for (int k = 0; k < H16; k += 16) {
            uint32_t hi[2][2], lw[2][2], a[4], r[4];
#pragma unroll
            for (int j = 0; j < 2; ++j)
#pragma unroll
                for (int i = 0; i < 2; ++i) {
                    const int e0 = k + 8 * i + 2 * tq;
                    const float* d = score + v * KV_PAGE + 8 * j + g;
                    const float w0 = exp2_fast(d[(int64_t)min(e0, s.heads - 1) * m.span] + norm[e0]);
                    const float w1 = exp2_fast(d[(int64_t)min(e0 + 1, s.heads - 1) * m.span] + norm[e0 + 1]);
                    hi[j][i] = pack_bf16(w0, w1);
                    const float2 back = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&hi[j][i]));
                    lw[j][i] = pack_bf16(w0 - back.x, w1 - back.y);
                }
            ldsm_x4(a, ta + 2 * k);
            ldsm_x4(r, ta + lo_off + 2 * k);
#pragma unroll
            for (int j = 0; j < 2; ++j) {
                mma_bf16(p[j], a[0], a[1], a[2], a[3], hi[j][0], hi[j][1]);
                mma_bf16(p[j], a[0], a[1], a[2], a[3], lw[j][0], lw[j][1]);
                mma_bf16(p[j], r[0], r[1], r[2], r[3], hi[j][0], hi[j][1]);
            }
        }
        uint32_t hi[4], lw[4];
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
            for (int r2 = 0; r2 < 2; ++r2) {
                hi[2 * j + r2] = pack_bf16(p[j][2 * r2], p[j][2 * r2 + 1]);
                const float2 back = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&hi[2 * j + r2]));
                lw[2 * j + r2] = pack_bf16(p[j][2 * r2] - back.x, p[j][2 * r2 + 1] - back.y);
            }
        if (PACKED) {  // row g + 8: the remainders of row g
            hi[1] = lw[0];
            hi[3] = lw[2];
        }
        cp_async_wait<MD_STAGES - 1>();
        __syncwarp();
        const uint32_t va = smem_addr(ring + st * KV_PAGE * LV + (lane & 15) * LV + (lane >> 4) * 8);
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
        fetch(v + MD_STAGES * stride, st);
    }
    cp_async_wait<0>();
    __syncthreads();
    const int LO = c.vdim16 + 4, rows = PACKED ? 8 : 16;
    float* const os = reinterpret_cast<float*>(rings);
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
    __syncthreads();
    bf16* const d = out + (int64_t)t * ldo + (int64_t)h0 * s.vdim;
    auto share = [&](int r, int e) {
        float v = 0.f;
#pragma unroll
        for (int w = 0; w < MD_WARPS; ++w) v += os[(w * rows + r) * LO + e];
        return v;
    };
    if (n_splits == 1) {
        for (int i = tid; i < nq * s.vdim; i += MD_WARPS * 32) d[i] = __float2bfloat16_rn(share(i / s.vdim, i % s.vdim));
        return;
    }
    for (int i = tid; i < nq * s.vdim; i += MD_WARPS * 32) os[(i / s.vdim) * LO + i % s.vdim] = share(i / s.vdim, i % s.vdim);  // in the first warp's place
    cluster_sync();
    for (int i = blockIdx.z * MD_WARPS * 32 + tid; i < nq * s.vdim; i += n_splits * MD_WARPS * 32) {
        const uint32_t a = smem_addr(os + (i / s.vdim) * LO + i % s.vdim);
        float v = 0.f;
        for (int p = 0; p < n_splits; ++p) v += ld_peer(peer_smem(a, p));
        d[i] = __float2bfloat16_rn(v);
    }
    cluster_sync();  // nobody leaves while its share is being read
}

int mixed_attention_splits(const GroupedShape& s, int n_tok, int keys) {
    const int group = s.heads / s.kv_heads, blocks = s.kv_heads * ((group + 15) / 16) * n_tok, slots = 2 * device_sm_count();
    int n = 1;
    while (n < MIXED_SPLITS && blocks * 2 * n <= slots && keys >= 128 * 2 * n) n <<= 1;
    return n;
}

using MixedMixFn = void (*)(GroupedShape, GroupedCache, MixedTerms, MixedScratch, const int32_t*, const int32_t*, bf16*, int, int);
static MixedMixFn mm_kernel(int vdim16, bool packed) {
    if (vdim16 <= 32) return packed ? mixed_mix_kernel<4, true> : mixed_mix_kernel<4, false>;
    if (vdim16 <= 64) return packed ? mixed_mix_kernel<8, true> : mixed_mix_kernel<8, false>;
    if (vdim16 <= 128) return packed ? mixed_mix_kernel<16, true> : mixed_mix_kernel<16, false>;
    return packed ? mixed_mix_kernel<32, true> : mixed_mix_kernel<32, false>;
}
constexpr int MD_CAP = 220 * 1024;

cudaError_t launch_mixed_attention(const void* q, const GroupedShape& s, const GroupedCache& c, const MixedTerms& x, const MixedScratch& m,
                                   const int32_t* tok_slot, const int32_t* tok_pos, void* out, int ldo, int n_splits, bool f32, int n_tok, cudaStream_t st) {
    if (n_tok == 0) return cudaSuccess;
    if (s.vdim > GROUPED_MAX_VDIM || c.shared || m.rows < 1) return cudaErrorInvalidValue;
    if (f32) return simple_launch<float>((const float*)q, s, c, x, m, tok_slot, tok_pos, (float*)out, ldo, n_tok, st);
    if (!mixed_mma_supported(s, c) || n_tok > m.rows) return simple_launch<bf16>((const bf16*)q, s, c, x, m, tok_slot, tok_pos, (bf16*)out, ldo, n_tok, st);
    if (n_splits < 1 || n_splits > MIXED_SPLITS || (n_splits & (n_splits - 1))) return cudaErrorInvalidValue;
    static PerDeviceOnce once;
    cudaError_t le = once.run([] {
        for (int i = 0; i < 8; ++i) {
            const cudaError_t e = cudaFuncSetAttribute((const void*)mm_kernel(32 << (i >> 1), i & 1), cudaFuncAttributeMaxDynamicSharedMemorySize, MD_CAP);
            if (e != cudaSuccess) return e;
        }
        return cudaFuncSetAttribute(mixed_scores_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, MD_CAP);
    });
    if (le != cudaSuccess) return le;
    const int group = s.heads / s.kv_heads;
    const dim3 grid(s.kv_heads * ((group + 15) / 16), n_tok, n_splits), block(MD_WARPS * 32);
    const size_t smem = (size_t)(16 + MD_WARPS * MD_STAGES * KV_PAGE) * (c.dim16 + 8) * 2;
    le = launch_pdl(mixed_scores_kernel, grid, block, smem, st, (const bf16*)q, s, c, m, tok_slot, tok_pos, n_splits);
    if (le == cudaSuccess) le = count_launch_and_check();
    if (le != cudaSuccess) return le;
    le = launch_pdl_cluster(mm_kernel(c.vdim16, group <= 8), grid, block, md_mix_smem(s, c), st, n_splits, s, c, x, m, tok_slot, tok_pos, (bf16*)out, ldo, n_splits);
    return le != cudaSuccess ? le : count_launch_and_check();
}

// ── many rows: denominators ──
// Block per (head, tile of 64 tokens), 4 warps x 16 query rows, key tiles of four visited pages, double-buffered.
// CAPPED: the cap is low enough for sums of e^score as they are.
constexpr int MT_KEYS = 64, MT_WARPS = 4;
constexpr float MT_CAP = 70.f;
template <bool CAPPED, int DIM>  // DIM: of the keys, padded (0: any)
__global__ void __launch_bounds__(MT_WARPS * 32) mixed_stats_kernel(const bf16* __restrict__ q, const GroupedShape s, const GroupedCache c, const MixedTerms x,
                                                                 const MixedScratch m, const GroupedTile* __restrict__ tiles) {
    extern __shared__ __align__(16) bf16 mt_sm[];
    pdl_wait();
    pdl_trigger();
    const int D16 = DIM ? DIM : c.dim16, LQ = D16 + 8, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, tq = lane & 3;
    bf16 *qs = mt_sm, *ks = qs + 64 * LQ;
    const int h = blockIdx.x, kvh = h / (s.heads / s.kv_heads);
    const GroupedTile tl = tiles[blockIdx.y];
    const int hi = tl.pos0 + tl.n - 1;
    const Visit vis(s, tl.pos0, hi);
    const int32_t* pt = c.page_table + (int64_t)tl.slot * c.max_pages;
    const int l8 = lane & 7, lr = warp * 16 + (lane >> 3);  // copies: eight lanes per row, a page per warp
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int r = lr + 4 * i;
        const bf16* src = q + ((int64_t)(tl.row0 + min(r, tl.n - 1)) * s.heads + h) * D16;
        for (int p = l8; p < D16 / 8; p += 8) cp_async16(qs + r * LQ + p * 8, src + p * 8, 16);
    }
    auto fetch = [&](int v0, int buf) {
        const int v = v0 + warp, page = vis.page(min(v, vis.pages - 1));
        const bf16* base = reinterpret_cast<const bf16*>(c.pool) + ((int64_t)pt[page] * s.kv_heads + kvh) * KV_PAGE * c.ld;
        bf16* kd = ks + buf * MT_KEYS * LQ;
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int r = lr + 4 * i, in = r - warp * 16, bytes = v < vis.pages && page * KV_PAGE + in <= hi ? 16 : 0;
            for (int p = l8; p < D16 / 8; p += 8) cp_async16(kd + r * LQ + p * 8, base + in * c.ld + p * 8, bytes);
        }
    };
    fetch(0, 0);
    cp_async_commit();
    const Log2Score score(s);
    const float mid = CAPPED ? score.top * LOG2E : 0.f;
    float m0 = CAPPED ? -mid : -INFINITY, m1 = m0, l0 = 0.f, l1 = 0.f;
    const int r0 = warp * 16 + g, r1 = r0 + 8, p0 = tl.pos0 + min(r0, tl.n - 1), p1 = tl.pos0 + min(r1, tl.n - 1);
    for (int v0 = 0, buf = 0; v0 < vis.pages; v0 += MT_KEYS / KV_PAGE, buf ^= 1) {
        cp_async_wait<0>();
        __syncthreads();
        if (v0 + MT_KEYS / KV_PAGE < vis.pages) fetch(v0 + MT_KEYS / KV_PAGE, buf ^ 1);
        cp_async_commit();
        const bf16* kt = ks + buf * MT_KEYS * LQ;
        float sc[8][4];
#pragma unroll
        for (int j = 0; j < 8; ++j) sc[j][0] = sc[j][1] = sc[j][2] = sc[j][3] = 0.f;
        const uint32_t qa = smem_addr(qs + (warp * 16 + (lane & 15)) * LQ + (lane >> 4) * 8);
        const uint32_t ka = smem_addr(kt + ((lane & 7) + (lane >> 4) * 8) * LQ + ((lane >> 3) & 1) * 8);
#pragma unroll(DIM ? DIM / 16 : 1)
        for (int k = 0; k < D16; k += 16) {
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
        // a run of pages that all rows see whole needs no mask
        const int first = vis.page(v0) * KV_PAGE, last = vis.page(min(v0 + MT_KEYS / KV_PAGE, vis.pages) - 1) * KV_PAGE + KV_PAGE - 1;
        const bool whole = v0 + MT_KEYS / KV_PAGE <= vis.pages && last <= tl.pos0 && (hi - first < s.window || last < s.keep);
#pragma unroll
        for (int j = 0; j < 8; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) sc[j][e] = score(sc[j][e], mid);
        if (!whole) {
#pragma unroll
            for (int j = 0; j < 8; ++j) {
                const int v = v0 + j / 2, key0 = vis.page(min(v, vis.pages - 1)) * KV_PAGE + 8 * (j & 1) + 2 * tq;
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    if (v >= vis.pages || !visible(s, key0 + e, p0)) sc[j][e] = -INFINITY;
                    if (v >= vis.pages || !visible(s, key0 + e, p1)) sc[j][2 + e] = -INFINITY;
                }
            }
        }
        float b0 = 0.f, b1 = 0.f;
        if (!CAPPED) {
            float x0 = m0, x1 = m1;
#pragma unroll
            for (int j = 0; j < 8; ++j) {
                x0 = fmaxf(x0, fmaxf(sc[j][0], sc[j][1]));
                x1 = fmaxf(x1, fmaxf(sc[j][2], sc[j][3]));
            }
#pragma unroll
            for (int off = 1; off < 4; off <<= 1) {
                x0 = fmaxf(x0, __shfl_xor_sync(0xFFFFFFFFu, x0, off));
                x1 = fmaxf(x1, __shfl_xor_sync(0xFFFFFFFFu, x1, off));
            }
            b0 = x0 == -INFINITY ? 0.f : x0;
            b1 = x1 == -INFINITY ? 0.f : x1;
            l0 *= exp2_fast(m0 - b0);
            l1 *= exp2_fast(m1 - b1);
            m0 = x0;
            m1 = x1;
        }
        float s0 = 0.f, s1 = 0.f;
#pragma unroll
        for (int j = 0; j < 8; ++j) {
            s0 += exp2_fast(sc[j][0] - b0) + exp2_fast(sc[j][1] - b0);
            s1 += exp2_fast(sc[j][2] - b1) + exp2_fast(sc[j][3] - b1);
        }
        l0 += s0;
        l1 += s1;
    }
    cp_async_wait<0>();
#pragma unroll
    for (int off = 1; off < 4; off <<= 1) {
        l0 += __shfl_xor_sync(0xFFFFFFFFu, l0, off);
        l1 += __shfl_xor_sync(0xFFFFFFFFu, l1, off);
    }
    if (tq == 0) {
        const float sink = x.sink ? (x.sink[h] - score.top) * LOG2E : -INFINITY;
        if (r0 < tl.n) m.norm[(int64_t)(tl.row0 + r0) * s.heads + h] = log2_norm(m0, l0, sink);
        if (r1 < tl.n) m.norm[(int64_t)(tl.row0 + r1) * s.heads + h] = log2_norm(m1, l1, sink);
    }
}

// ── many rows: weights and values ──
// Block (cluster rank: a run of 8 HPW heads, tile of 16 tokens), a warp per HPW heads. Per page of keys: weights of the block's
// heads into every block's shared memory, one barrier, then each warp mixes for its heads and multiplies with the values. Keys are
// two stages ahead of the barrier, values one; weights alternate between two buffers. A thread's four keys of the A operand are
// neighbours, so that it reads a head's weights as one vector; the values' rows are numbered the same way.
constexpr int MP_WARPS = 8, MP_MAX_CLUSTER = 8, MP_CAP = 224 * 1024;
struct MixedTiling {
    int heads, kv, cluster;    // heads of a block, cached heads they touch at most, blocks
    int q, k, v, w, mix;       // offsets in shared memory (bytes)
    size_t smem;
};
__host__ __device__ __forceinline__ MixedTiling mp_tiling(const GroupedShape& s, const GroupedCache& c, int hpw) {
    MixedTiling t;
    const int group = s.heads / s.kv_heads;
    t.heads = MP_WARPS * hpw < s.heads ? MP_WARPS * hpw : s.heads;
    t.cluster = 1;
    while (t.cluster * t.heads < s.heads) t.cluster <<= 1;
    const int touched = (t.heads + group - 2) / group + 1;  // a run may begin inside a group
    t.kv = t.heads % group == 0 || group % t.heads == 0 ? (t.heads + group - 1) / group : touched < s.kv_heads ? touched : s.kv_heads;
    t.q = 0;
    t.k = t.q + MP_WARPS * hpw * 16 * (c.dim16 + 8) * 2;
    t.v = t.k + 2 * t.kv * KV_PAGE * (c.dim16 + 8) * 2;
    t.w = t.v + 2 * t.kv * KV_PAGE * (c.vdim16 + 8) * 2;
    t.mix = t.w + 2 * s.heads * 16 * KV_PAGE * 4;
    t.smem = (size_t)t.mix + (size_t)MP_WARPS * hpw * s.heads * 8;
    return t;
}
static int mp_heads_per_warp(const GroupedShape& s, const GroupedCache& c) {  // 0: not covered
    if (s.dim > 256 || s.vdim > 256) return 0;
    for (int hpw = c.vdim16 <= 128 && s.heads > MP_WARPS ? 2 : 1; hpw > 0; --hpw) {
        const MixedTiling t = mp_tiling(s, c, hpw);
        if (t.cluster <= MP_MAX_CLUSTER && t.smem <= MP_CAP) return hpw;
    }
    return 0;
}

__device__ __forceinline__ void st_peer(uint32_t addr, float a, float b) {
    asm volatile("st.shared::cluster.v2.f32 [%0], {%1, %2};\n" ::"r"(addr), "f"(a), "f"(b) : "memory");
}
// Two floats in a register pair: d += a * b.
__device__ __forceinline__ void fma_pair(unsigned long long& d, unsigned long long a, unsigned long long b) {
    asm("fma.rn.f32x2 %0, %1, %2, %0;\n" : "+l"(d) : "l"(a), "l"(b));
}
__device__ __forceinline__ unsigned long long both(float v) { return (unsigned long long)__float_as_uint(v) << 32 | __float_as_uint(v); }
__device__ __forceinline__ float2 pair_of(unsigned long long v) { return make_float2(__uint_as_float((uint32_t)v), __uint_as_float((uint32_t)(v >> 32))); }

template <int VT, int HPW>
__global__ void __launch_bounds__(MP_WARPS * 32, HPW == 1 && VT <= 16 ? 2 : 1)
    mixed_prefill_kernel(const bf16* __restrict__ q, const GroupedShape s, const GroupedCache c, const MixedTerms x, const MixedScratch m,
                         const GroupedTile* __restrict__ tiles, bf16* __restrict__ out, int ldo) {
    extern __shared__ __align__(16) uint8_t mp_sm[];
    const MixedTiling tg = mp_tiling(s, c, HPW);
    const int LQ = c.dim16 + 8, LV = c.vdim16 + 8, H = s.heads, group = H / s.kv_heads;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, tq = lane & 3;
    const int h0 = blockIdx.z * tg.heads, nh = min(tg.heads, H - h0);  // (a cluster's last blocks may have none)
    const int kv0 = h0 / group, nkv = nh > 0 ? (h0 + nh - 1) / group - kv0 + 1 : 0;
    const uint32_t sm = smem_addr(mp_sm);
    float2* const mix = reinterpret_cast<float2*>(mp_sm + tg.mix);  // [warp][head][HPW], twice side by side
    for (int i = tid; i < MP_WARPS * HPW * H; i += MP_WARPS * 32) {
        const int hh = i % HPW, e = i / HPW % H, h = i / HPW / H * HPW + hh;
        const float f = h < nh ? x.mix[(int64_t)(h0 + h) * H + e] : 0.f;
        mix[i] = make_float2(f, f);
    }
    pdl_wait();
    pdl_trigger();
    const GroupedTile tl = tiles[blockIdx.y];
    const int hi = tl.pos0 + tl.n - 1;
    const Visit vis(s, tl.pos0, hi);
    const int32_t* pt = c.page_table + (int64_t)tl.slot * c.max_pages;
    auto id = [&](int v) { return v < vis.pages ? pt[vis.page(v)] : 0; };
    // page v, whose place in the pool is `page`: half a warp per row, the rows of all cached heads spread over the block
    auto fetch = [&](int v, int page, int col, int width, int base, int ld) {
        if (v >= vis.pages) return;
        const int live = hi - vis.page(v) * KV_PAGE + 1, half = tid >> 4, l16 = tid & 15;
        const bf16* src = reinterpret_cast<const bf16*>(c.pool) + ((int64_t)page * s.kv_heads + kv0) * KV_PAGE * c.ld + col;
        const uint32_t dst = sm + (uint32_t)(base + (v & 1) * tg.kv * KV_PAGE * ld * 2);
        for (int row = half; row < nkv * KV_PAGE; row += MP_WARPS * 2)
            for (int p = l16; p < width / 8; p += 16)
                cp_async16_at(dst + (uint32_t)(row * ld + p * 8) * 2, src + (int64_t)row * c.ld + p * 8, row % KV_PAGE < live ? 16 : 0);
    };
    auto fetch_k = [&](int v, int page) { fetch(v, page, 0, c.dim16, tg.k, LQ); };
    auto fetch_v = [&](int v, int page) { fetch(v, page, c.dim16, c.vdim16, tg.v, LV); };
    int next = id(1), after = id(2);  // places of pages v + 1 and v + 2
    for (int i = warp; i < nh * 16; i += MP_WARPS) {
        const int h = i / 16, r = i % 16;
        const bf16* src = q + ((int64_t)(tl.row0 + min(r, tl.n - 1)) * H + h0 + h) * c.dim16;
        for (int p = lane; p < c.dim16 / 8; p += 32) cp_async16_at(sm + (uint32_t)(tg.q + (i * LQ + p * 8) * 2), src + p * 8, 16);
    }
    const int page0 = id(0);
    fetch_k(0, page0);
    cp_async_commit();
    const int ra = min(g, tl.n - 1), rb = min(g + 8, tl.n - 1), pa = tl.pos0 + ra, pb = tl.pos0 + rb;
    float na[HPW], nb[HPW];  // of the two rows: what makes a score a weight
#pragma unroll
    for (int j = 0; j < HPW; ++j) {
        const int h = min(h0 + warp * HPW + j, H - 1);
        na[j] = m.norm[(int64_t)(tl.row0 + ra) * H + h];
        nb[j] = m.norm[(int64_t)(tl.row0 + rb) * H + h];
    }
    cp_async_wait<0>();
    if (tg.cluster == 1) __syncthreads();
    else cluster_sync();  // (also: every peer has started)
    fetch_k(1, next);
    fetch_v(0, page0);
    cp_async_commit();
    const Log2Score score(s);
    float o[HPW][VT][4];
#pragma unroll
    for (int j = 0; j < HPW; ++j)
#pragma unroll
        for (int i = 0; i < VT; ++i) o[j][i][0] = o[j][i][1] = o[j][i][2] = o[j][i][3] = 0.f;
    // this thread's places in shared memory, stage 0 of each
    uint32_t qa[HPW], ka[HPW], va[HPW], wd[HPW];
    const int v_key = 4 * ((lane & 7) >> 1) + (lane & 1) + 2 * ((lane >> 3) & 1);  // the key of the operand's row lane & 15
#pragma unroll
    for (int j = 0; j < HPW; ++j) {
        const int h = min(warp * HPW + j, max(nh - 1, 0)), kv = (h0 + h) / group - kv0;
        qa[j] = sm + (uint32_t)(tg.q + ((h * 16 + (lane & 15)) * LQ + (lane >> 4) * 8) * 2);
        ka[j] = sm + (uint32_t)(tg.k + ((kv * KV_PAGE + (lane & 7) + (lane >> 4) * 8) * LQ + ((lane >> 3) & 1) * 8) * 2);
        va[j] = sm + (uint32_t)(tg.v + ((kv * KV_PAGE + v_key) * LV + (lane >> 4) * 8) * 2);
        wd[j] = sm + (uint32_t)(tg.w + (((h0 + h) * 16 + g) * KV_PAGE + 2 * tq) * 4);
    }
    const uint32_t k_stage = (uint32_t)(tg.kv * KV_PAGE * LQ * 2), v_stage = (uint32_t)(tg.kv * KV_PAGE * LV * 2), w_stage = (uint32_t)(H * 16 * KV_PAGE * 4);
    const uint8_t* const wr0 = mp_sm + tg.w + (g * KV_PAGE + 4 * tq) * 4;
    const float2* const mr = mix + warp * H * HPW;
    for (int v = 0; v < vis.pages; ++v) {
        const int key0 = vis.page(v) * KV_PAGE;
        const uint32_t odd = v & 1;
        const bool whole = key0 + KV_PAGE - 1 <= tl.pos0 && (hi - key0 < s.window || key0 + KV_PAGE <= s.keep);  // every row sees the page
        float sc[HPW][2][4];
#pragma unroll
        for (int j = 0; j < HPW; ++j)
#pragma unroll
            for (int e = 0; e < 8; ++e) sc[j][e >> 2][e & 3] = 0.f;
#pragma unroll
        for (int j = 0; j < HPW; ++j) {
            if (warp * HPW + j >= nh) continue;
            const uint32_t kp = ka[j] + odd * k_stage;
#pragma unroll 4
            for (int k = 0; k < c.dim16; k += 16) {
                uint32_t a[4], b[4];
                ldsm_x4(a, qa[j] + 2 * k);
                ldsm_x4(b, kp + 2 * k);
                mma_bf16(sc[j][0], a[0], a[1], a[2], a[3], b[0], b[1]);
                mma_bf16(sc[j][1], a[0], a[1], a[2], a[3], b[2], b[3]);
            }
        }
#pragma unroll
        for (int j = 0; j < HPW; ++j) {
            if (warp * HPW + j >= nh) continue;
            const uint32_t wp = wd[j] + odd * w_stage;
#pragma unroll
            for (int n = 0; n < 2; ++n) {
                float w[4];
#pragma unroll
                for (int e = 0; e < 4; ++e) w[e] = exp2_fast(score(sc[j][n][e], e < 2 ? na[j] : nb[j]));
                if (!whole) {
                    const int key = key0 + 8 * n + 2 * tq;
#pragma unroll
                    for (int e = 0; e < 4; ++e) w[e] = visible(s, key + (e & 1), e < 2 ? pa : pb) ? w[e] : 0.f;
                }
                if (tg.cluster == 1) {
                    float* d = reinterpret_cast<float*>(mp_sm + (wp - sm)) + 8 * n;
                    *reinterpret_cast<float2*>(d) = make_float2(w[0], w[1]);
                    *reinterpret_cast<float2*>(d + 8 * KV_PAGE) = make_float2(w[2], w[3]);
                } else {
                    for (int p = 0; p < tg.cluster; ++p) {
                        const uint32_t a = peer_smem(wp + 32u * n, p);
                        st_peer(a, w[0], w[1]);
                        st_peer(a + 8 * KV_PAGE * 4, w[2], w[3]);
                    }
                }
            }
        }
        cp_async_wait<0>();
        if (tg.cluster == 1) __syncthreads();
        else cluster_sync();
        fetch_k(v + 2, after);
        fetch_v(v + 1, next);
        cp_async_commit();
        next = after;
        after = id(v + 3);
        if (warp * HPW >= nh) continue;
        unsigned long long p[HPW][4];  // row g: keys 4 tq .. 4 tq + 3, then row g + 8, in pairs
#pragma unroll
        for (int j = 0; j < HPW; ++j)
#pragma unroll
            for (int i = 0; i < 4; ++i) p[j][i] = 0ull;
        const uint8_t* wr = wr0 + odd * w_stage;
#pragma unroll 4
        for (int e = 0; e < H; ++e) {
            const ulonglong2 a = *reinterpret_cast<const ulonglong2*>(wr + e * 16 * KV_PAGE * 4), b = *reinterpret_cast<const ulonglong2*>(wr + (e * 16 + 8) * KV_PAGE * 4);
            const unsigned long long w[4] = {a.x, a.y, b.x, b.y};
            unsigned long long f[HPW];
            if (HPW == 2) {
                const ulonglong2 t = *reinterpret_cast<const ulonglong2*>(mr + e * 2);
                f[0] = t.x;
                f[HPW - 1] = t.y;
            } else {
                f[0] = *reinterpret_cast<const unsigned long long*>(mr + e);
            }
#pragma unroll
            for (int j = 0; j < HPW; ++j)
#pragma unroll
                for (int i = 0; i < 4; ++i) fma_pair(p[j][i], f[j], w[i]);
        }
        uint32_t a[HPW][4], r[HPW][4];
#pragma unroll
        for (int j = 0; j < HPW; ++j)
#pragma unroll
            for (int i = 0; i < 4; ++i) {  // operand registers: (row g, keys 0 1), (row g + 8, keys 0 1), (row g, keys 2 3), (row g + 8, keys 2 3)
                const float2 u = pair_of(p[j][2 * (i & 1) + (i >> 1)]);
                a[j][i] = pack_bf16(u.x, u.y);
                const float2 back = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&a[j][i]));
                r[j][i] = pack_bf16(u.x - back.x, u.y - back.y);
            }
#pragma unroll
        for (int j = 0; j < HPW; ++j) {
            if (warp * HPW + j >= nh) continue;
            const uint32_t vp = va[j] + odd * v_stage;
#pragma unroll
            for (int i = 0; i < VT; i += 2) {
                if (i * 8 < c.vdim16) {
                    uint32_t b[4];
                    ldsm_x4_t(b, vp + 2 * (i * 8));
                    mma_bf16(o[j][i], a[j][0], a[j][1], a[j][2], a[j][3], b[0], b[1]);
                    mma_bf16(o[j][i + 1], a[j][0], a[j][1], a[j][2], a[j][3], b[2], b[3]);
                    mma_bf16(o[j][i], r[j][0], r[j][1], r[j][2], r[j][3], b[0], b[1]);
                    mma_bf16(o[j][i + 1], r[j][0], r[j][1], r[j][2], r[j][3], b[2], b[3]);
                }
            }
        }
    }
    cp_async_wait<0>();
#pragma unroll
    for (int j = 0; j < HPW; ++j) {
        const int h = warp * HPW + j;
        if (h >= nh) continue;
        bf16* d = out + (int64_t)tl.row0 * ldo + (int64_t)(h0 + h) * s.vdim;
#pragma unroll
        for (int i = 0; i < VT; ++i) {
            const int col = i * 8 + 2 * tq;
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                if (col + e >= s.vdim) continue;
                if (g < tl.n) d[(int64_t)g * ldo + col + e] = __float2bfloat16_rn(o[j][i][e]);
                if (g + 8 < tl.n) d[(int64_t)(g + 8) * ldo + col + e] = __float2bfloat16_rn(o[j][i][2 + e]);
            }
        }
    }
    if (tg.cluster > 1) cluster_sync();  // nobody leaves while a peer may still write here
}

// The same for keys and values of 8 VT coordinates (64 or 128), an even number of query heads per cached head and more than
// eight of them: half of the warps make the weights of a page while the other half mixes and multiplies those of the page before.
// The second half mixes together — a thread has two neighbouring keys of a row and eight output heads, so that a weight is read
// twice and not once per warp — and passes the mixed weights on through shared memory, leading parts and remainders. Either half
// has two heads per warp that share the fragments of their cached head. At 128 coordinates the second half needs registers that
// the first one gives up.
constexpr int MX_THREADS = 2 * MP_WARPS * 32, MX_FEW = 72, MX_MANY = 184;
static_assert(MX_FEW + MX_MANY == 2 * 128, "what the halves have together is what the block was launched with");
constexpr int MX_HEADS = 2 * MP_WARPS, MX_PART = MX_HEADS * 16 * KV_PAGE * 2;  // heads of a block; bytes of its mixed weights' leading parts
// Shared memory behind mp_tiling's weights: the mixing matrix [head][output head], mixed weights [part][output head][16 rows][16 keys].
static size_t mx_smem(const GroupedShape& s, const MixedTiling& t) { return (size_t)t.mix + (size_t)s.heads * MX_HEADS * 4 + 2 * MX_PART; }

template <int VT>
__global__ void __launch_bounds__(MX_THREADS, 1)
    mixed_prefill_halves_kernel(const bf16* __restrict__ q, const GroupedShape s, const GroupedCache c, const MixedTerms x, const MixedScratch m,
                                const GroupedTile* __restrict__ tiles, bf16* __restrict__ out, int ldo) {
    extern __shared__ __align__(16) uint8_t mp_sm[];
    constexpr int D = 8 * VT, LD = D + 8;
    const MixedTiling tg = mp_tiling(s, c, 2);
    const int H = s.heads, group = H / s.kv_heads, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, tq = lane & 3;
    const int h0 = blockIdx.z * tg.heads, nh = min(tg.heads, H - h0);  // (a cluster's last blocks may have none)
    const int kv0 = h0 / group, nkv = nh > 0 ? (h0 + nh - 1) / group - kv0 + 1 : 0;
    const uint32_t sm = smem_addr(mp_sm);
    float* const mix = reinterpret_cast<float*>(mp_sm + tg.mix);
    for (int i = tid; i < H * MX_HEADS; i += MX_THREADS) {
        const int e = i / MX_HEADS, h = i % MX_HEADS;
        mix[i] = h < nh ? x.mix[(int64_t)(h0 + h) * H + e] : 0.f;
    }
    pdl_wait();
    pdl_trigger();
    const GroupedTile tl = tiles[blockIdx.y];
    const int hi = tl.pos0 + tl.n - 1;
    const Visit vis(s, tl.pos0, hi);
    const int32_t* pt = c.page_table + (int64_t)tl.slot * c.max_pages;
    auto id = [&](int v) { return v < vis.pages ? pt[vis.page(v)] : 0; };
    const int row0 = tid / VT, piece = tid % VT;  // a row's pieces are neighbouring threads
    auto fetch = [&](int v, int page, int col, int base) {
        if (v >= vis.pages) return;
        const int live = hi - vis.page(v) * KV_PAGE + 1;
        const bf16* src = reinterpret_cast<const bf16*>(c.pool) + (((int64_t)page * s.kv_heads + kv0) * KV_PAGE + row0) * c.ld + col + piece * 8;
        uint32_t dst = sm + (uint32_t)(base + (((v & 1) * tg.kv * KV_PAGE + row0) * LD + piece * 8) * 2);
        for (int row = row0; row < nkv * KV_PAGE; row += MX_THREADS / VT) {
            cp_async16_at(dst, src, row % KV_PAGE < live ? 16 : 0);
            src += (int64_t)(MX_THREADS / VT) * c.ld;
            dst += (MX_THREADS / VT) * LD * 2;
        }
    };
    auto fetch_k = [&](int v, int page) { fetch(v, page, 0, tg.k); };
    auto fetch_v = [&](int v, int page) { fetch(v, page, D, tg.v); };
    auto meet = [&] {
        if (tg.cluster == 1) asm volatile("bar.sync 1, %0;\n" ::"n"(MX_THREADS) : "memory");
        else cluster_sync();
    };
    int next = id(1), after = id(2);  // places of pages v + 1 and v + 2
    const int page0 = id(0);
    // what stands between two steps of the loop: everyone is done with keys v and values v - 1, keys v + 1 and values v are there
    auto turn = [&](int v) {
        cp_async_wait<0>();
        meet();
        fetch_k(v + 2, after);
        fetch_v(v + 1, next);
        cp_async_commit();
        next = after;
        after = id(v + 3);
    };
    for (int i = row0; i < nh * 16; i += MX_THREADS / VT) {
        const int h = i / 16, r = i % 16;
        cp_async16_at(sm + (uint32_t)(tg.q + (i * LD + piece * 8) * 2), q + ((int64_t)(tl.row0 + min(r, tl.n - 1)) * H + h0 + h) * D + piece * 8, 16);
    }
    fetch_k(0, page0);
    cp_async_commit();
    cp_async_wait<0>();
    meet();  // (also: every peer has started)
    fetch_k(1, next);
    fetch_v(0, page0);
    cp_async_commit();
    const int pair = (warp % MP_WARPS) * 2, hp = min(pair, max(nh - 2, 0)), kv = (h0 + hp) / group - kv0;  // this warp's first head
    const bool busy = pair < nh;
    const uint32_t stage = (uint32_t)(tg.kv * KV_PAGE * LD * 2), w_stage = (uint32_t)(H * 16 * KV_PAGE * 4);
    if (warp < MP_WARPS) {
        if (VT > 8) asm volatile("setmaxnreg.dec.sync.aligned.u32 %0;\n" ::"n"(MX_FEW));
        const int ra = min(g, tl.n - 1), rb = min(g + 8, tl.n - 1), pa = tl.pos0 + ra, pb = tl.pos0 + rb;
        float na[2], nb[2];  // of the two rows: what makes a score a weight
#pragma unroll
        for (int j = 0; j < 2; ++j) {
            const int h = min(h0 + hp + j, H - 1);
            na[j] = m.norm[(int64_t)(tl.row0 + ra) * H + h];
            nb[j] = m.norm[(int64_t)(tl.row0 + rb) * H + h];
        }
        const Log2Score score(s);
        const uint32_t qa = sm + (uint32_t)(tg.q + ((hp * 16 + (lane & 15)) * LD + (lane >> 4) * 8) * 2);
        const uint32_t ka = sm + (uint32_t)(tg.k + ((kv * KV_PAGE + (lane & 7) + (lane >> 4) * 8) * LD + ((lane >> 3) & 1) * 8) * 2);
        const uint32_t wd = sm + (uint32_t)(tg.w + (((h0 + hp) * 16 + g) * KV_PAGE + 2 * tq) * 4);
        for (int v = 0; v <= vis.pages; ++v) {
            if (busy && v < vis.pages) {
                const int key0 = vis.page(v) * KV_PAGE;
                const bool whole = key0 + KV_PAGE - 1 <= tl.pos0 && (hi - key0 < s.window || key0 + KV_PAGE <= s.keep);  // every row sees the page
                const uint32_t kp = ka + (v & 1) * stage, wp = wd + (v & 1) * w_stage;
                float sc[2][2][4] = {};
#pragma unroll
                for (int k = 0; k < D; k += 16) {
                    uint32_t b[4];
                    ldsm_x4(b, kp + 2 * k);
#pragma unroll
                    for (int j = 0; j < 2; ++j) {
                        uint32_t a[4];
                        ldsm_x4(a, qa + (uint32_t)(j * 16 * LD + k) * 2);
                        mma_bf16(sc[j][0], a[0], a[1], a[2], a[3], b[0], b[1]);
                        mma_bf16(sc[j][1], a[0], a[1], a[2], a[3], b[2], b[3]);
                    }
                }
#pragma unroll
                for (int j = 0; j < 2; ++j)
#pragma unroll
                    for (int n = 0; n < 2; ++n) {
                        float w[4];
#pragma unroll
                        for (int e = 0; e < 4; ++e) w[e] = exp2_fast(score(sc[j][n][e], e < 2 ? na[j] : nb[j]));
                        if (!whole) {
                            const int key = key0 + 8 * n + 2 * tq;
#pragma unroll
                            for (int e = 0; e < 4; ++e) w[e] = visible(s, key + (e & 1), e < 2 ? pa : pb) ? w[e] : 0.f;
                        }
                        const uint32_t d = wp + (uint32_t)(j * 16 * KV_PAGE + 8 * n) * 4;
                        if (tg.cluster == 1) {
                            *reinterpret_cast<float2*>(mp_sm + (d - sm)) = make_float2(w[0], w[1]);
                            *reinterpret_cast<float2*>(mp_sm + (d - sm) + 8 * KV_PAGE * 4) = make_float2(w[2], w[3]);
                        } else {
                            for (int p = 0; p < tg.cluster; ++p) {
                                const uint32_t a = peer_smem(d, p);
                                st_peer(a, w[0], w[1]);
                                st_peer(a + 8 * KV_PAGE * 4, w[2], w[3]);
                            }
                        }
                    }
            }
            turn(v);
        }
    } else {
        if (VT > 8) asm volatile("setmaxnreg.inc.sync.aligned.u32 %0;\n" ::"n"(MX_MANY));
        float o[2][VT][4];
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
            for (int i = 0; i < VT; ++i) o[j][i][0] = o[j][i][1] = o[j][i][2] = o[j][i][3] = 0.f;
        const uint32_t va = sm + (uint32_t)(tg.v + ((kv * KV_PAGE + (lane & 15)) * LD + (lane >> 4) * 8) * 2);
        // mixing: eight output heads from m0, row mq, keys 2 mk and the next; a row's two runs of eight keys change places every
        // four rows, so that reads of eight rows meet every bank once
        const int m0 = (warp & 4) * 2, mq = (warp & 3) * 4 + (lane >> 3), mk = lane & 7;
        const uint8_t* const wr0 = mp_sm + tg.w + (mq * KV_PAGE + 2 * mk) * 4;
        uint8_t* const parts = mp_sm + tg.mix + H * MX_HEADS * 4;
        uint8_t* const put = parts + m0 * 16 * KV_PAGE * 2 + mq * 32 + (((mk >> 2) ^ ((mq >> 2) & 1)) * 16) + (mk & 3) * 4;
        const uint32_t pa = smem_addr(parts) + (uint32_t)(hp * 16 * KV_PAGE * 2 + (lane & 15) * 32 + (((lane >> 4) ^ ((lane >> 2) & 1)) * 16));
        turn(0);
        for (int v = 0; v < vis.pages; ++v) {
            if (m0 < nh) {
                unsigned long long p[2][4];  // two keys, pairs of heads
#pragma unroll
                for (int j = 0; j < 2; ++j)
#pragma unroll
                    for (int i = 0; i < 4; ++i) p[j][i] = 0ull;
                const uint8_t* wr = wr0 + (v & 1) * w_stage;
                const float* mr = mix + m0;
#pragma unroll 4
                for (int e = 0; e < H; ++e) {
                    const float2 w = *reinterpret_cast<const float2*>(wr + e * 16 * KV_PAGE * 4);
                    const ulonglong2 f = *reinterpret_cast<const ulonglong2*>(mr + e * MX_HEADS), f2 = *reinterpret_cast<const ulonglong2*>(mr + e * MX_HEADS + 4);
                    const unsigned long long wx = both(w.x), wy = both(w.y);
                    fma_pair(p[0][0], f.x, wx); fma_pair(p[0][1], f.y, wx); fma_pair(p[0][2], f2.x, wx); fma_pair(p[0][3], f2.y, wx);
                    fma_pair(p[1][0], f.x, wy); fma_pair(p[1][1], f.y, wy); fma_pair(p[1][2], f2.x, wy); fma_pair(p[1][3], f2.y, wy);
                }
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    const float2 x0 = pair_of(p[0][i]), x1 = pair_of(p[1][i]);
#pragma unroll
                    for (int k = 0; k < 2; ++k) {
                        const float u = k ? x0.y : x0.x, w = k ? x1.y : x1.x;
                        const uint32_t top = pack_bf16(u, w);
                        const float2 back = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&top));
                        uint8_t* d = put + (2 * i + k) * 16 * KV_PAGE * 2;
                        *reinterpret_cast<uint32_t*>(d) = top;
                        *reinterpret_cast<uint32_t*>(d + MX_PART) = pack_bf16(u - back.x, w - back.y);
                    }
                }
            }
            asm volatile("bar.sync 2, %0;\n" ::"n"(MX_THREADS / 2) : "memory");  // this half alone
            if (busy) {
                uint32_t a[2][4], r[2][4];
#pragma unroll
                for (int j = 0; j < 2; ++j) {
                    ldsm_x4(a[j], pa + j * 16 * KV_PAGE * 2);
                    ldsm_x4(r[j], pa + j * 16 * KV_PAGE * 2 + MX_PART);
                }
                const uint32_t vp = va + (v & 1) * stage;
#pragma unroll
                for (int i = 0; i < VT; i += 2) {
                    uint32_t b[4];
                    ldsm_x4_t(b, vp + 2 * (i * 8));
#pragma unroll
                    for (int j = 0; j < 2; ++j) {
                        mma_bf16(o[j][i], a[j][0], a[j][1], a[j][2], a[j][3], b[0], b[1]);
                        mma_bf16(o[j][i + 1], a[j][0], a[j][1], a[j][2], a[j][3], b[2], b[3]);
                    }
#pragma unroll
                    for (int j = 0; j < 2; ++j) {
                        mma_bf16(o[j][i], r[j][0], r[j][1], r[j][2], r[j][3], b[0], b[1]);
                        mma_bf16(o[j][i + 1], r[j][0], r[j][1], r[j][2], r[j][3], b[2], b[3]);
                    }
                }
            }
            turn(v + 1);
        }
        if (busy) {
#pragma unroll
            for (int j = 0; j < 2; ++j) {
                bf16* d = out + (int64_t)tl.row0 * ldo + (int64_t)(h0 + pair + j) * D;
#pragma unroll
                for (int i = 0; i < VT; ++i) {
                    const int col = i * 8 + 2 * tq;
                    if (g < tl.n) *reinterpret_cast<uint32_t*>(d + (int64_t)g * ldo + col) = pack_bf16(o[j][i][0], o[j][i][1]);
                    if (g + 8 < tl.n) *reinterpret_cast<uint32_t*>(d + (int64_t)(g + 8) * ldo + col) = pack_bf16(o[j][i][2], o[j][i][3]);
                }
            }
        }
    }
    cp_async_wait<0>();
    if (tg.cluster > 1) cluster_sync();  // nobody leaves while a peer may still write here
}

bool mixed_mma_supported(const GroupedShape& s, const GroupedCache& c) {
    return mp_heads_per_warp(s, c) > 0 && md_mix_smem(s, c) <= MD_CAP && (size_t)(16 + MD_WARPS * MD_STAGES * KV_PAGE) * (c.dim16 + 8) * 2 <= MD_CAP;
}

using MixedPrefillFn = void (*)(const bf16*, GroupedShape, GroupedCache, MixedTerms, MixedScratch, const GroupedTile*, bf16*, int);
static MixedPrefillFn mp_kernel(int vdim16, int hpw) {
    if (vdim16 <= 32) return hpw == 2 ? mixed_prefill_kernel<4, 2> : mixed_prefill_kernel<4, 1>;
    if (vdim16 <= 64) return hpw == 2 ? mixed_prefill_kernel<8, 2> : mixed_prefill_kernel<8, 1>;
    if (vdim16 <= 128) return hpw == 2 ? mixed_prefill_kernel<16, 2> : mixed_prefill_kernel<16, 1>;
    return mixed_prefill_kernel<32, 1>;
}
using MixedStatsFn = void (*)(const bf16*, GroupedShape, GroupedCache, MixedTerms, MixedScratch, const GroupedTile*);
static MixedStatsFn mt_kernel(bool capped, int dim16) {
    if (dim16 == 64) return capped ? mixed_stats_kernel<true, 64> : mixed_stats_kernel<false, 64>;
    if (dim16 == 128) return capped ? mixed_stats_kernel<true, 128> : mixed_stats_kernel<false, 128>;
    return capped ? mixed_stats_kernel<true, 0> : mixed_stats_kernel<false, 0>;
}
// The kernel in halves: null where it does not fit, or was not compiled to start with the registers that the halves share out.
static MixedPrefillFn mx_kernel(const GroupedShape& s, const GroupedCache& c, int hpw) {
    if (hpw != 2 || (s.heads / s.kv_heads) % 2 || s.dim != s.vdim || (s.dim != 64 && s.dim != 128) || mx_smem(s, mp_tiling(s, c, hpw)) > MP_CAP) return nullptr;
    const MixedPrefillFn f = s.dim == 64 ? mixed_prefill_halves_kernel<8> : mixed_prefill_halves_kernel<16>;
    static std::atomic<int> regs[2];
    int n = regs[s.dim == 128].load(std::memory_order_relaxed);
    if (n == 0) {
        cudaFuncAttributes a{};
        n = cudaFuncGetAttributes(&a, (const void*)f) == cudaSuccess ? a.numRegs : -1;
        regs[s.dim == 128].store(n, std::memory_order_relaxed);
    }
    return s.dim == 64 || n == (MX_FEW + MX_MANY) / 2 ? f : nullptr;
}

cudaError_t launch_mixed_prefill(const void* q, const GroupedShape& s, const GroupedCache& c, const MixedTerms& x, const MixedScratch& m,
                                 const GroupedTile* wide, int n_wide, const GroupedTile* narrow, int n_narrow, void* out, int ldo, cudaStream_t st) {
    if (n_wide == 0 || n_narrow == 0) return cudaSuccess;
    const int hpw = mp_heads_per_warp(s, c);
    if (!hpw) return cudaErrorInvalidValue;
    static PerDeviceOnce once;
    cudaError_t le = once.run([] {
        for (int i = 0; i < 9; ++i) {
            const MixedPrefillFn f = i < 7 ? mp_kernel(32 << (i >> 1), 2 - (i & 1)) : i < 8 ? mixed_prefill_halves_kernel<8> : mixed_prefill_halves_kernel<16>;
            const cudaError_t e = cudaFuncSetAttribute((const void*)f, cudaFuncAttributeMaxDynamicSharedMemorySize, MP_CAP);
            if (e != cudaSuccess) return e;
        }
        for (int i = 0; i < 6; ++i) {
            const cudaError_t e = cudaFuncSetAttribute((const void*)mt_kernel(i & 1, 64 * (i >> 1)), cudaFuncAttributeMaxDynamicSharedMemorySize, MP_CAP);
            if (e != cudaSuccess) return e;
        }
        return cudaSuccess;
    });
    if (le != cudaSuccess) return le;
    le = launch_pdl(mt_kernel(s.softcap > 0.f && s.softcap <= MT_CAP, c.dim16), dim3(s.heads, n_wide), dim3(MT_WARPS * 32), (size_t)3 * 64 * (c.dim16 + 8) * 2, st, (const bf16*)q, s, c, x, m, wide);
    if (le == cudaSuccess) le = count_launch_and_check();
    if (le != cudaSuccess) return le;
    const MixedTiling t = mp_tiling(s, c, hpw);
    const MixedPrefillFn halves = mx_kernel(s, c, hpw);
    le = launch_pdl_cluster(halves ? halves : mp_kernel(c.vdim16, hpw), dim3(1, n_narrow, t.cluster), dim3(halves ? MX_THREADS : MP_WARPS * 32),
                            halves ? mx_smem(s, t) : t.smem, st, t.cluster, (const bf16*)q, s, c, x, m, narrow, (bf16*)out, ldo);
    return le != cudaSuccess ? le : count_launch_and_check();
}

}  // namespace sp
