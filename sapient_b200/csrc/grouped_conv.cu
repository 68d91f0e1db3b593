// Short convolutions over time on the way from the projection to queries and cache (plan_kernels.h: GroupedInput): bias, convolution,
// rotation and append in one launch. A thread owns two coordinates of a head that are turned together (or pass together) and
// walks tokens of a sequence in order with the values before them in registers, so that every projected value is read once.
//   Few rows: the blocks of a slot's first row take all of its rows and then write its tail. Everything but the projection is
//   requested before the previous kernel is waited for: no kernel of the last two before this one writes it.
//   Many rows: a tile of up to MIXED_Q_TILE consecutive tokens per block; the tails follow in a launch of their own, since other
//   blocks may still read them.
#include "kernels.h"
#include "model_plan.h"
#include "pdl.cuh"
#include "plan_common.cuh"
#include "plan_kernels.h"
#include "sp_common.cuh"

namespace sp {

cudaError_t count_launch_and_check();  // kernels.cu

__host__ __device__ __forceinline__ int conv_channels(const GroupedShape& s) { return (s.heads + s.kv_heads) * s.dim + s.kv_heads * s.vdim; }

__device__ __forceinline__ void store_two(float* d, int a, int b, float u, float v) {
    d[a] = u;
    d[b] = v;
}
__device__ __forceinline__ void store_two(bf16* d, int a, int b, float u, float v) {
    if (b == a + 1 && !(a & 1)) {  // (rows start on even elements)
        *reinterpret_cast<uint32_t*>(d + a) = pack_bf16(u, v);
    } else {
        d[a] = __float2bfloat16_rn(u);
        d[b] = __float2bfloat16_rn(v);
    }
}

constexpr int CA_THREADS = 128;
static_assert(MIXED_Q_TILE <= KV_PAGE, "a tile touches two pages at most");
// CAP: taps at most; missing older ones weigh nothing.
template <typename T, int CAP>
__global__ void __launch_bounds__(CA_THREADS) conv_append_kernel(const float* __restrict__ proj, int ldp, const GroupedShape s, const GroupedCache c,
                                                                 const GroupedInput in, const GroupedTile* __restrict__ tiles, const int32_t* __restrict__ tok_slot,
                                                                 const int32_t* __restrict__ tok_pos, T* __restrict__ q) {
    const int unit = blockIdx.x * CA_THREADS + threadIdx.x, per_key = c.dim16 / 2, per_value = c.vdim16 / 2, keys = (s.heads + s.kv_heads) * per_key;
    const bool on = unit < keys + s.kv_heads * per_value, value = unit >= keys, query = unit < s.heads * per_key;
    const int head = !on ? 0 : value ? (unit - keys) / per_value : unit / per_key, u = !on ? 0 : value ? (unit - keys) % per_value : unit % per_key;
    const int n = value ? s.vdim : s.dim, at = value ? (s.heads + s.kv_heads) * s.dim + head * s.vdim : head * s.dim, channels = conv_channels(s);
    const bool turn = !value && 2 * u < s.rot;
    const int a = turn && !s.neighbours ? u : 2 * u, b = turn && !s.neighbours ? u + s.rot / 2 : 2 * u + 1;
    const bool on_a = on && a < n, on_b = on && b < n;
    const int ca = on_a ? at + a : 0, cb = on_b ? at + b : 0, keep = in.taps - 1;
    float wa[CAP], wb[CAP], ha[CAP], hb[CAP];  // h[1 .. CAP - 1]: the values before, h[0] is not used
#pragma unroll
    for (int j = 0; j < CAP; ++j) {
        const int tap = j - (CAP - in.taps);
        wa[j] = tap >= 0 && on_a ? __ldg(in.conv + (int64_t)tap * channels + ca) : 0.f;
        wb[j] = tap >= 0 && on_b ? __ldg(in.conv + (int64_t)tap * channels + cb) : 0.f;
        ha[j] = hb[j] = 0.f;
    }
    const float bias_a = in.bias && on_a ? __ldg(in.bias + ca) : 0.f, bias_b = in.bias && on_b ? __ldg(in.bias + cb) : 0.f;
    // one token: its projected values come in, everything goes out to d
    auto token = [&](T* d, const float2& r, float x, float y) {
        float va = wa[CAP - 1] * x, vb = wb[CAP - 1] * y;
#pragma unroll
        for (int j = 1; j < CAP; ++j) {
            va = fmaf(wa[j - 1], ha[j], va);
            vb = fmaf(wb[j - 1], hb[j], vb);
        }
#pragma unroll
        for (int j = 1; j < CAP - 1; ++j) { ha[j] = ha[j + 1]; hb[j] = hb[j + 1]; }
        if (CAP > 1) { ha[CAP - 1] = x; hb[CAP - 1] = y; }
        if (turn) {
            const float z = va * r.x - vb * r.y;
            vb = vb * r.x + va * r.y;
            va = z;
        }
        if (on) store_two(d, a, b, va, vb);
    };
    const int turn_ld = s.rot / 2, g = value ? head : head - s.heads;
    auto query_row = [&](int t) { return q + ((int64_t)t * s.heads + head) * c.dim16; };
    auto cache_page = [&](int page) { return reinterpret_cast<T*>(c.pool) + ((int64_t)page * s.kv_heads + g) * KV_PAGE * c.ld + (value ? c.dim16 : 0); };
    auto angle = [&](int pos) { return __ldg(in.cs_key + (int64_t)pos * turn_ld + u); };
    // Projected values as they are, and with the bias. Two neighbours are one load where rows and heads start on even elements.
    const bool pairs = b == a + 1 && on_b && ((ldp | at) & 1) == 0 && (reinterpret_cast<uintptr_t>(proj) & 7) == 0;
    auto two_of = [&](int t) { return *reinterpret_cast<const float2*>(proj + (int64_t)t * ldp + ca); };
    auto each_of = [&](int t) { return make_float2(proj[(int64_t)t * ldp + ca], proj[(int64_t)t * ldp + cb]); };
    auto projected = [&](int t, float& x, float& y) {
        const float2 v = pairs ? two_of(t) : each_of(t);
        x = on_a ? v.x + bias_a : 0.f;
        y = on_b ? v.y + bias_b : 0.f;
    };
    if (tiles) {
        pdl_wait();
        pdl_trigger();
        const GroupedTile tl = tiles[blockIdx.y];
        const float* tail = in.tail + tl.slot * in.tail_stride;
        const int32_t* pt = c.page_table + (int64_t)tl.slot * c.max_pages + tl.pos0 / KV_PAGE;
        const int in0 = tl.pos0 % KV_PAGE, page0 = pt[0], page1 = in0 + tl.n > KV_PAGE ? pt[1] : 0;  // (a tile is no longer than a page)
        // everything the tile needs is requested at once, before anything is used
        float2 x[MIXED_Q_TILE], r[MIXED_Q_TILE];
        if (pairs) {
#pragma unroll
            for (int i = 0; i < MIXED_Q_TILE; ++i) x[i] = two_of(tl.row0 + min(i, tl.n - 1));
        } else {
#pragma unroll
            for (int i = 0; i < MIXED_Q_TILE; ++i) x[i] = each_of(tl.row0 + min(i, tl.n - 1));
        }
        if (turn) {
#pragma unroll
            for (int i = 0; i < MIXED_Q_TILE; ++i) r[i] = angle(tl.pos0 + min(i, tl.n - 1));
        }
        int near[CAP];  // mostly the row before a row is the one above it: requested at once
#pragma unroll
        for (int d = 0; d < CAP - 1; ++d) near[d] = d < keep ? __ldg(in.back + max(tl.row0 - d, 0)) : -1;
        int row = near[0], k = 0;  // rows of the slot before the tile, as far as they have been counted
#pragma unroll
        for (int d = 1; d < CAP; ++d) {
            if (d > keep || tl.pos0 < d) continue;
            if (row >= 0) {
                projected(row, ha[CAP - d], hb[CAP - d]);
                row = d < CAP - 1 && row == tl.row0 - d ? near[d] : in.back[row];
                ++k;
            } else {
                const int64_t place = (int64_t)(keep + k - d) * channels;
                if (on_a) ha[CAP - d] = tail[place + ca];
                if (on_b) hb[CAP - d] = tail[place + cb];
            }
        }
        const int64_t step = query ? (int64_t)s.heads * c.dim16 : c.ld;
        T *d = query ? query_row(tl.row0) : cache_page(page0) + (int64_t)in0 * c.ld, *const d1 = query ? nullptr : cache_page(page1);
#pragma unroll
        for (int i = 0; i < MIXED_Q_TILE; ++i)
            if (i < tl.n) {
                if (!query && in0 + i == KV_PAGE) d = d1;
                token(d, r[i], on_a ? x[i].x + bias_a : 0.f, on_b ? x[i].y + bias_b : 0.f);
                d += step;
            }
        return;
    }
    const int t0 = blockIdx.y, lane = threadIdx.x & 31, rows_all = gridDim.y, mine = lane < rows_all ? tok_slot[lane] : -1, slot = tok_slot[t0], pos0 = tok_pos[t0];
    uint32_t rows = __ballot_sync(0xFFFFFFFFu, mine == slot);
    if (rows & ((1u << t0) - 1)) return;
    float* const tail = in.tail + slot * in.tail_stride;
#pragma unroll
    for (int d = 1; d < CAP; ++d) {
        if (d > keep || pos0 < d) continue;
        if (on_a) ha[CAP - d] = tail[(int64_t)(keep - d) * channels + ca];
        if (on_b) hb[CAP - d] = tail[(int64_t)(keep - d) * channels + cb];
    }
    const int32_t* pt = c.page_table + (int64_t)slot * c.max_pages;
    pdl_wait();
    pdl_trigger();
    for (int i = 0; rows; rows &= rows - 1, ++i) {
        const int t = __ffs(rows) - 1;
        float x, y;
        projected(t, x, y);
        const int pos = pos0 + i;
        token(query ? query_row(t) : cache_page(pt[pos / KV_PAGE]) + (int64_t)(pos % KV_PAGE) * c.ld, turn ? angle(pos) : make_float2(1.f, 0.f), x, y);
    }
#pragma unroll
    for (int d = 1; d < CAP; ++d) {
        if (d > keep) continue;
        if (on_a) tail[(int64_t)(keep - d) * channels + ca] = ha[CAP - d];
        if (on_b) tail[(int64_t)(keep - d) * channels + cb] = hb[CAP - d];
    }
}

cudaError_t launch_conv_append(const float* proj, int ldp, const GroupedShape& s, const GroupedCache& c, const GroupedInput& in, const GroupedTile* tiles,
                               int n_tiles, const int32_t* tok_slot, const int32_t* tok_pos, void* q, bool f32, int n_tok, cudaStream_t st) {
    if (n_tok == 0) return cudaSuccess;
    if (!in.conv || in.taps < 1 || in.taps > CONV_MAX_TAPS || c.shared || in.norm || in.temperature || in.cs_val || (tiles ? !in.back : n_tok > 32)) return cudaErrorInvalidValue;
    const int units = (s.heads + s.kv_heads) * (c.dim16 / 2) + s.kv_heads * (c.vdim16 / 2);
    const dim3 grid((units + CA_THREADS - 1) / CA_THREADS, tiles ? n_tiles : n_tok), block(CA_THREADS);
#define SP_CA(T, CAP) launch_pdl(conv_append_kernel<T, CAP>, grid, block, 0, st, proj, ldp, s, c, in, tiles, tok_slot, tok_pos, (T*)q)
#define SP_CT(T) (in.taps <= 4 ? SP_CA(T, 4) : in.taps <= 8 ? SP_CA(T, 8) : SP_CA(T, CONV_MAX_TAPS))
    const cudaError_t le = f32 ? SP_CT(float) : SP_CT(bf16);
#undef SP_CT
#undef SP_CA
    return le != cudaSuccess ? le : count_launch_and_check();
}

// A thread per channel of a slot whose last row in the step is ends[blockIdx.y].
constexpr int CT_THREADS = 128;
__global__ void __launch_bounds__(CT_THREADS) conv_tails_kernel(const float* __restrict__ proj, int ldp, int channels, const GroupedInput in,
                                                             const int32_t* __restrict__ tok_slot, const int32_t* __restrict__ ends) {
    __shared__ int rows[CONV_MAX_TAPS];  // the slot's last rows, the newest first
    pdl_wait();
    pdl_trigger();
    const int end = ends[blockIdx.y], i = blockIdx.x * CT_THREADS + threadIdx.x, keep = in.taps - 1;
    if (threadIdx.x == 0)
        for (int d = 0, r = end; d < keep; ++d) {
            rows[d] = r;
            if (r >= 0) r = in.back[r];
        }
    __syncthreads();
    if (i >= channels) return;
    int n = 0;
    while (n < keep && rows[n] >= 0) ++n;
    float* const tail = in.tail + tok_slot[end] * in.tail_stride + i;
    for (int j = 0; j < keep; ++j) {  // the oldest first: what is read stands behind what has been written
        const int d = keep - 1 - j;
        float v;
        if (d < n) {
            v = proj[(int64_t)rows[d] * ldp + i];
            if (in.bias) v += in.bias[i];
        } else {
            v = tail[(int64_t)(j + n) * channels];
        }
        tail[(int64_t)j * channels] = v;
    }
}

cudaError_t launch_conv_tails(const float* proj, int ldp, const GroupedShape& s, const GroupedInput& in, const int32_t* tok_slot, const int32_t* ends,
                              int n_ends, cudaStream_t st) {
    if (n_ends == 0 || in.taps <= 1) return cudaSuccess;
    if (!in.conv || in.taps > CONV_MAX_TAPS || !in.back) return cudaErrorInvalidValue;
    const int channels = conv_channels(s);
    const cudaError_t le = launch_pdl(conv_tails_kernel, dim3((channels + CT_THREADS - 1) / CT_THREADS, n_ends), dim3(CT_THREADS), 0, st, proj, ldp, channels, in, tok_slot, ends);
    return le != cudaSuccess ? le : count_launch_and_check();
}

}  // namespace sp
