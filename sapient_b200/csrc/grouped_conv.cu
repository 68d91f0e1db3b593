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
        wa[j] = tap >= 0 && on_a ? in.conv[(int64_t)tap * channels + ca] : 0.f;
        wb[j] = tap >= 0 && on_b ? in.conv[(int64_t)tap * channels + cb] : 0.f;
        ha[j] = hb[j] = 0.f;
    }
    const float bias_a = in.bias && on_a ? in.bias[ca] : 0.f, bias_b = in.bias && on_b ? in.bias[cb] : 0.f;
    // one token: its projected values come in, everything goes out
    auto token = [&](int t, int slot, int pos, float x, float y) {
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
            const float2 r = in.cs_key[(int64_t)pos * (s.rot / 2) + u];
            const float z = va * r.x - vb * r.y;
            vb = vb * r.x + va * r.y;
            va = z;
        }
        if (!on) return;
        T* d;
        if (query) {
            d = q + ((int64_t)t * s.heads + head) * c.dim16;
        } else {
            const int page = c.page_table[(int64_t)slot * c.max_pages + pos / KV_PAGE], g = value ? head : head - s.heads;
            d = reinterpret_cast<T*>(c.pool) + (((int64_t)page * s.kv_heads + g) * KV_PAGE + pos % KV_PAGE) * c.ld + (value ? c.dim16 : 0);
        }
        store_two(d, a, b, va, vb);
    };
    auto projected = [&](int t, float& x, float& y) {
        x = on_a ? proj[(int64_t)t * ldp + ca] + bias_a : 0.f;
        y = on_b ? proj[(int64_t)t * ldp + cb] + bias_b : 0.f;
    };
    if (tiles) {
        pdl_wait();
        pdl_trigger();
        const GroupedTile tl = tiles[blockIdx.y];
        const float* tail = in.tail + tl.slot * in.tail_stride;
        float x[MIXED_Q_TILE], y[MIXED_Q_TILE];
#pragma unroll
        for (int i = 0; i < MIXED_Q_TILE; ++i)
            if (i < tl.n) projected(tl.row0 + i, x[i], y[i]);
        int r = in.back[tl.row0], k = 0;  // rows of the slot before the tile, as far as they have been counted
#pragma unroll
        for (int d = 1; d < CAP; ++d) {
            if (d > keep || tl.pos0 < d) continue;
            if (r >= 0) {
                projected(r, ha[CAP - d], hb[CAP - d]);
                r = in.back[r];
                ++k;
            } else {
                const int64_t place = (int64_t)(keep + k - d) * channels;
                if (on_a) ha[CAP - d] = tail[place + ca];
                if (on_b) hb[CAP - d] = tail[place + cb];
            }
        }
#pragma unroll
        for (int i = 0; i < MIXED_Q_TILE; ++i)
            if (i < tl.n) token(tl.row0 + i, tl.slot, tl.pos0 + i, x[i], y[i]);
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
    pdl_wait();
    pdl_trigger();
    for (int i = 0; rows; rows &= rows - 1, ++i) {
        const int t = __ffs(rows) - 1;
        float x, y;
        projected(t, x, y);
        token(t, slot, pos0 + i, x, y);
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
