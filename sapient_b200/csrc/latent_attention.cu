// Latent attention over a paged latent cache (plan_kernels.h).
//
// The cache keeps, per token and owning layer, a normed latent c and one rotated key part kr shared by the heads. With
// k_h = W_uk,h c and v_h = W_uv,h c, a head's score is q_h . W_uk,h c + qr_h . kr = [W_uk,h^T q_h | qr_h] . [c | kr]: in
// the ABSORBED form every head of a token attends to the same cached rows with a query of rank + rot coordinates, the
// softmax mixes the latents, and W_uv,h is applied to the mixture. It reads each cached byte once per token (16 heads are
// the rows of one mma tile) and rebuilds nothing: decode steps and short portions. The EXPANDED form rebuilds k_h and v_h
// of a key range with one matrix product and attends with dim + rot and vdim coordinates, a third of the work per
// (query, key) pair: prompts.
// Scores, softmax and accumulation are f32 in both; a sliding window bounds the keys a block visits.
#include "kernels.h"
#include "pdl.cuh"
#include "plan_common.cuh"
#include "plan_kernels.h"
#include "sp_common.cuh"

namespace sp {

cudaError_t count_launch_and_check();  // kernels.cu

// ── rotation, latent norm, cache append ──
constexpr int LA_WARPS = 4;

template <typename T>
__device__ __forceinline__ void rotate_pairs(const float* src, T* dst, const float2* cs, int rot, int rot16) {
    for (int i = threadIdx.x & 31; i < rot16 / 2; i += 32) {
        float u = 0.f, v = 0.f;
        if (2 * i < rot) {
            const float a = src[2 * i], b = src[2 * i + 1];
            const float2 r = cs[i];
            u = a * r.x - b * r.y;
            v = b * r.x + a * r.y;
        }
        dst[2 * i] = from_f32<T>(u);
        dst[2 * i + 1] = from_f32<T>(v);
    }
}

// A warp per (token, part): parts 0 .. heads - 1 are the heads' queries, part `heads` the cache row.
template <typename T>
__global__ void __launch_bounds__(LA_WARPS * 32) latent_append_kernel(const float* __restrict__ proj, int ldp, const LatentShape s, const LatentCache c,
                                                                   const float* __restrict__ norm_gain, float eps, const float2* __restrict__ cos_sin,
                                                                   const int32_t* __restrict__ tok_slot, const int32_t* __restrict__ tok_pos,
                                                                   T* __restrict__ qn, int ldqn, T* __restrict__ qabs, T* __restrict__ qf, int parts) {
    pdl_wait();
    pdl_trigger();
    const int t = blockIdx.x, h = blockIdx.y * LA_WARPS + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (h >= parts) return;
    const int pos = tok_pos[t];
    const float2* cs = cos_sin + (int64_t)pos * (s.rot / 2);
    if (h < s.heads) {
        const float* q = proj + (int64_t)t * ldp + (int64_t)h * (s.dim + s.rot);
        if (qn) {
            T* d = qn + ((int64_t)t * s.heads + h) * ldqn;
            for (int i = lane; i < ldqn; i += 32) d[i] = from_f32<T>(i < s.dim ? q[i] : 0.f);
            T* r = qabs + ((int64_t)t * s.heads + h) * c.ld;
            for (int i = c.rank + lane; i < c.rank16; i += 32) r[i] = from_f32<T>(0.f);
            rotate_pairs<T>(q + s.dim, r + c.rank16, cs, s.rot, c.rot16);
        } else {
            const int dim16 = (s.dim + 15) & ~15;
            T* d = qf + ((int64_t)t * s.heads + h) * (dim16 + c.rot16);
            for (int i = lane; i < dim16; i += 32) d[i] = from_f32<T>(i < s.dim ? q[i] : 0.f);
            rotate_pairs<T>(q + s.dim, d + dim16, cs, s.rot, c.rot16);
        }
        return;
    }
    const float* kv = proj + (int64_t)t * ldp + (int64_t)s.heads * (s.dim + s.rot);
    float ss = 0.f;
    for (int i = lane; i < c.rank; i += 32) ss = fmaf(kv[i], kv[i], ss);
    const float r = rsqrtf(warp_sum(ss) / (float)c.rank + eps);
    const int page = c.page_table[(int64_t)tok_slot[t] * c.max_pages + pos / KV_PAGE];
    T* row = reinterpret_cast<T*>(c.pool) + ((int64_t)page * KV_PAGE + pos % KV_PAGE) * c.ld;
    for (int i = lane; i < c.rank16; i += 32) row[i] = from_f32<T>(i < c.rank ? kv[i] * r * norm_gain[i] : 0.f);
    rotate_pairs<T>(kv + c.rank, row + c.rank16, cs, s.rot, c.rot16);
}

cudaError_t launch_latent_append(const float* proj, int ldp, const LatentShape& s, const LatentCache& c, bool own, const float* norm_gain,
                                 float eps, const float2* cos_sin, const int32_t* tok_slot, const int32_t* tok_pos, void* qn, int ldqn,
                                 void* qabs, void* qf, bool f32, int n_tok, cudaStream_t st) {
    if (n_tok == 0) return cudaSuccess;
    const int parts = s.heads + (own ? 1 : 0);
    const dim3 grid(n_tok, (parts + LA_WARPS - 1) / LA_WARPS);
    cudaError_t le = f32 ? launch_pdl(latent_append_kernel<float>, grid, dim3(LA_WARPS * 32), 0, st, proj, ldp, s, c, norm_gain, eps, cos_sin, tok_slot,
                                      tok_pos, (float*)qn, ldqn, (float*)qabs, (float*)qf, parts)
                         : launch_pdl(latent_append_kernel<bf16>, grid, dim3(LA_WARPS * 32), 0, st, proj, ldp, s, c, norm_gain, eps, cos_sin, tok_slot,
                                      tok_pos, (bf16*)qn, ldqn, (bf16*)qabs, (bf16*)qf, parts);
    if (le != cudaSuccess) return le;
    return count_launch_and_check();
}

// ── absorbed attention ──
// Key range of split sp of n_splits for a token at `pos`.
__device__ __forceinline__ void key_range(int pos, int window, int sp, int n_splits, int& begin, int& end) {
    const int lo = window > pos ? 0 : pos - window + 1, n = pos + 1 - lo;
    const int per = (n + n_splits - 1) / n_splits;
    begin = lo + sp * per;
    end = min(pos + 1, begin + per);
}

// Any compute type and sizes up to rank 1024: block per (head, token, split), a warp per key.
constexpr int LS_WARPS = 4, LS_MAX_PER_LANE = 32;
template <typename T>
__global__ void __launch_bounds__(LS_WARPS * 32) latent_attention_simple_kernel(const T* __restrict__ qabs, const LatentShape s, const LatentCache c,
                                                                                const int32_t* __restrict__ tok_slot, const int32_t* __restrict__ tok_pos,
                                                                                T* __restrict__ out, int ldo, float* __restrict__ part, int n_splits) {
    extern __shared__ float ls_smem[];  // query, then one output row per warp
    __shared__ float sm[LS_WARPS], sl[LS_WARPS];
    pdl_wait();
    pdl_trigger();
    const int h = blockIdx.x, t = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int width = c.rank16 + c.rot16;
    float *q = ls_smem, *os = ls_smem + width;
    const T* qr = qabs + ((int64_t)t * s.heads + h) * c.ld;
    for (int i = threadIdx.x; i < width; i += LS_WARPS * 32) q[i] = to_f32(qr[i]);
    __syncthreads();
    int begin, end;
    key_range(tok_pos[t], s.window, blockIdx.z, n_splits, begin, end);
    const int32_t* pt = c.page_table + (int64_t)tok_slot[t] * c.max_pages;
    float o[LS_MAX_PER_LANE];
#pragma unroll
    for (int i = 0; i < LS_MAX_PER_LANE; ++i) o[i] = 0.f;
    float m = -INFINITY, l = 0.f;
    for (int key = begin + warp; key < end; key += LS_WARPS) {
        const T* row = reinterpret_cast<const T*>(c.pool) + ((int64_t)pt[key / KV_PAGE] * KV_PAGE + key % KV_PAGE) * c.ld;
        float dot = 0.f;
        for (int i = lane; i < width; i += 32) dot = fmaf(q[i], to_f32(row[i]), dot);
        const float sc = warp_sum(dot) * s.scale;
        const float mn = fmaxf(m, sc), corr = expf(m - mn), p = expf(sc - mn);
#pragma unroll
        for (int i = 0; i < LS_MAX_PER_LANE; ++i)
            if (lane + 32 * i < c.rank) o[i] = fmaf(p, to_f32(row[lane + 32 * i]), o[i] * corr);
        l = fmaf(l, corr, p);
        m = mn;
    }
    if (lane == 0) { sm[warp] = m; sl[warp] = l; }
#pragma unroll
    for (int i = 0; i < LS_MAX_PER_LANE; ++i)
        if (lane + 32 * i < c.rank) os[warp * c.rank + lane + 32 * i] = o[i];
    __syncthreads();
    float M = -INFINITY, L = 0.f, cw[LS_WARPS];
#pragma unroll
    for (int w = 0; w < LS_WARPS; ++w) M = fmaxf(M, sm[w]);
#pragma unroll
    for (int w = 0; w < LS_WARPS; ++w) {
        cw[w] = sm[w] == -INFINITY ? 0.f : expf(sm[w] - M);
        L = fmaf(cw[w], sl[w], L);
    }
    float* pd = part + (((int64_t)t * s.heads + h) * n_splits + blockIdx.z) * (c.rank + 2);
    const float inv = n_splits == 1 ? 1.0f / L : 1.f;
    for (int e = threadIdx.x; e < c.rank; e += LS_WARPS * 32) {
        float v = 0.f;
#pragma unroll
        for (int w = 0; w < LS_WARPS; ++w) v = fmaf(cw[w], os[w * c.rank + e], v);
        if (n_splits == 1) out[((int64_t)t * s.heads + h) * ldo + e] = from_f32<T>(v * inv);
        else pd[2 + e] = v;
    }
    if (n_splits > 1 && threadIdx.x == 0) { pd[0] = M; pd[1] = L; }
}

// bf16: block per (HG groups of 16 heads, token, split), 8 warps per group, a ring of ST tiles of KEYS keys filled by
// cp.async and shared by the groups. Scores: a warp owns an eighth of the coordinates (its query fragments stay in registers) for all
// keys of the tile, the partial sums meet in shared memory; mixture: a warp owns NT 8-column tiles of the latent.
constexpr int LM_WARPS = 8, LM_PAGES = 256, LM_MAX_SPLITS = 16;  // splits are blocks of a cluster
constexpr int LM_ROW_THREADS = LM_WARPS * 2;  // of the softmax: threads per query
constexpr int LM_COPY = 3;       // 16-byte pieces of a row per lane: rank + rot up to 640, as
constexpr int LM_MAX_STEPS = 5;   // 16-coordinate steps per warp: rank + rot up to 640
static size_t lm_smem(int width, int hg, int keys, int st) { return (size_t)st * keys * (width + 8) * 2 + (size_t)hg * LM_WARPS * 16 * (keys + 8) * 4; }
__device__ __forceinline__ void group_sync(int grp) { asm volatile("bar.sync %0, %1;\n" ::"r"(grp + 1), "n"(LM_WARPS * 32) : "memory"); }

template <int NT, int HG, int KEYS, int ST>
__global__ void __launch_bounds__(LM_WARPS * 32 * HG) latent_attention_mma_kernel(const bf16* __restrict__ qabs, const LatentShape s, const LatentCache c,
                                                                                  const int32_t* __restrict__ tok_slot, const int32_t* __restrict__ tok_pos,
                                                                                  bf16* __restrict__ out, int ldo, int n_splits) {
    constexpr int PLD = KEYS + 8, SLD = KEYS + 8;
    static_assert(KEYS == 2 * LM_ROW_THREADS, "the softmax gives every thread two keys");
    extern __shared__ __align__(16) bf16 lm_smem_raw[];
    __shared__ int pages_s[LM_PAGES];
    __shared__ float corr_s[HG][16], l_s[HG][16], m_s[HG][16], share_s[HG * 16][LM_MAX_SPLITS];
    __shared__ __align__(16) bf16 ps_all[HG][16][PLD];
    const int width = c.rank16 + c.rot16, LD = width + 8;
    const int wid = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, tq = lane & 3;
    const int grp = HG > 1 ? wid / LM_WARPS : 0, warp = wid % LM_WARPS, tid = threadIdx.x % (LM_WARPS * 32);
    bf16* ks = lm_smem_raw;
    float* ss = reinterpret_cast<float*>(ks + ST * KEYS * LD) + grp * LM_WARPS * 16 * SLD;
    bf16(*ps)[PLD] = ps_all[grp];
    const int h0 = (blockIdx.x * HG + grp) * 16, t = blockIdx.y;
    pdl_wait();
    pdl_trigger();
    int begin, end;
    key_range(tok_pos[t], s.window, blockIdx.z, n_splits, begin, end);
    const int32_t* pt = c.page_table + (int64_t)tok_slot[t] * c.max_pages;
    const int pieces = width / 8, page0 = begin / KV_PAGE;
    // the range's page numbers, so that a copy does not wait for its own
    const bool listed = (end - 1) / KV_PAGE - page0 < LM_PAGES;
    if (listed)
        for (int i = threadIdx.x; begin < end && i <= (end - 1) / KV_PAGE - page0; i += LM_WARPS * 32 * HG) pages_s[i] = pt[page0 + i];
    __syncthreads();
    auto fetch = [&](int k0, int buf) {  // a warp copies every (8 HG)-th key: a row's address is found once
        constexpr int PER = KEYS / (LM_WARPS * HG);
        const uint32_t d0 = smem_addr(ks + (buf * KEYS + wid) * LD + lane * 8);
#pragma unroll
        for (int i = 0; i < PER; ++i) {
            const int key = k0 + wid + LM_WARPS * HG * i, at = min(key, end - 1), bytes = key < end ? 16 : 0;
            const int page = listed ? pages_s[at / KV_PAGE - page0] : pt[at / KV_PAGE];
            const bf16* src = reinterpret_cast<const bf16*>(c.pool) + ((int64_t)page * KV_PAGE + at % KV_PAGE) * c.ld + lane * 8;
            const uint32_t d = d0 + (uint32_t)(2 * LM_WARPS * HG * i * LD);
#pragma unroll
            for (int p = 0; p < LM_COPY; ++p)
                if (lane + 32 * p < pieces) cp_async16_at(d + 512 * p, src + 256 * p, bytes);
        }
    };
    // the ring is full from the start; a stage is refilled as soon as everyone is done with it
#pragma unroll
    for (int i = 0; i < ST; ++i) {
        if (begin + i * KEYS < end) fetch(begin + i * KEYS, i);
        cp_async_commit();
    }
    // this warp's coordinates of the 16 queries
    const int steps = width / 16, per = (steps + LM_WARPS - 1) / LM_WARPS, s0 = warp * per, my = max(0, min(per, steps - s0));
    uint32_t qf[LM_MAX_STEPS][4];
    {
        const int ha = h0 + g, hb = h0 + g + 8;
        const uint32_t* qa = reinterpret_cast<const uint32_t*>(qabs + ((int64_t)t * s.heads + min(ha, s.heads - 1)) * c.ld);
        const uint32_t* qb = reinterpret_cast<const uint32_t*>(qabs + ((int64_t)t * s.heads + min(hb, s.heads - 1)) * c.ld);
#pragma unroll
        for (int i = 0; i < LM_MAX_STEPS; ++i) {
            const int k = (s0 + i) * 8 + tq;  // in pairs
            const bool on = i < my;
            qf[i][0] = on && ha < s.heads ? qa[k] : 0u;
            qf[i][1] = on && hb < s.heads ? qb[k] : 0u;
            qf[i][2] = on && ha < s.heads ? qa[k + 4] : 0u;
            qf[i][3] = on && hb < s.heads ? qb[k + 4] : 0u;
        }
    }
    float o[NT][4];
#pragma unroll
    for (int i = 0; i < NT; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
    float m = -INFINITY, l = 0.f;  // of row tid / LM_ROW_THREADS, the same in all its threads
    const int col0 = warp * NT * 8;
    for (int k0 = begin, buf = 0; k0 < end; k0 += KEYS, buf = buf + 1 == ST ? 0 : buf + 1) {
        cp_async_wait<ST - 1>();
        __syncthreads();  // this tile has landed for everyone
        const bf16* kt = ks + buf * KEYS * LD;
        {
            float a[KEYS / 8][4];
#pragma unroll
            for (int j = 0; j < KEYS / 8; ++j) a[j][0] = a[j][1] = a[j][2] = a[j][3] = 0.f;
            const uint32_t ka = smem_addr(kt + ((lane & 7) + (lane >> 4) * 8) * LD + ((lane >> 3) & 1) * 8 + s0 * 16);
#pragma unroll
            for (int i = 0; i < LM_MAX_STEPS; ++i) {
                if (i < my) {
#pragma unroll
                    for (int j = 0; j < KEYS / 8; j += 2) {
                        uint32_t b[4];
                        ldsm_x4(b, ka + 2 * (8 * j * LD + 16 * i));
                        mma_bf16(a[j], qf[i][0], qf[i][1], qf[i][2], qf[i][3], b[0], b[1]);
                        mma_bf16(a[j + 1], qf[i][0], qf[i][1], qf[i][2], qf[i][3], b[2], b[3]);
                    }
                }
            }
            float* d = ss + (warp * 16 + g) * SLD + 2 * tq;
#pragma unroll
            for (int j = 0; j < KEYS / 8; ++j) {
                *reinterpret_cast<float2*>(d + 8 * j) = make_float2(a[j][0], a[j][1]);  // rows 40 floats apart: no bank conflicts in pairs
                *reinterpret_cast<float2*>(d + 8 * SLD + 8 * j) = make_float2(a[j][2], a[j][3]);
            }
        }
        group_sync(grp);
        {
            const int r = tid / LM_ROW_THREADS, key = tid % LM_ROW_THREADS * 2;
            float v[2] = {0.f, 0.f}, mx = m;
#pragma unroll
            for (int w = 0; w < LM_WARPS; ++w) {
                const float2 z = *reinterpret_cast<const float2*>(ss + (w * 16 + r) * SLD + key);
                v[0] += z.x;
                v[1] += z.y;
            }
#pragma unroll
            for (int i = 0; i < 2; ++i) {
                v[i] = k0 + key + i < end ? v[i] * s.scale : -INFINITY;
                mx = fmaxf(mx, v[i]);
            }
#pragma unroll
            for (int off = LM_ROW_THREADS / 2; off > 0; off >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xFFFFFFFFu, mx, off));
            // the tile's first key is live, so mx is finite
            const float cr = expf(m - mx);
            float sum = 0.f;
#pragma unroll
            for (int i = 0; i < 2; ++i) { v[i] = expf(v[i] - mx); sum += v[i]; }
#pragma unroll
            for (int off = LM_ROW_THREADS / 2; off > 0; off >>= 1) sum += __shfl_xor_sync(0xFFFFFFFFu, sum, off);
            *reinterpret_cast<uint32_t*>(&ps[r][key]) = pack_bf16(v[0], v[1]);
            l = fmaf(l, cr, sum);
            m = mx;
            if (tid % LM_ROW_THREADS == 0) corr_s[grp][r] = cr;
        }
        group_sync(grp);
        const float c0 = corr_s[grp][g], c1 = corr_s[grp][g + 8];
#pragma unroll
        for (int i = 0; i < NT; ++i) { o[i][0] *= c0; o[i][1] *= c0; o[i][2] *= c1; o[i][3] *= c1; }
#pragma unroll
        for (int kk = 0; kk < KEYS / 16; ++kk) {
            uint32_t p[4];
            ldsm_x4(p, smem_addr(&ps[lane & 15][kk * 16 + (lane >> 4) * 8]));
            const uint32_t va = smem_addr(kt + (kk * 16 + (lane & 15)) * LD + (lane >> 4) * 8);
#pragma unroll
            for (int i = 0; i < NT; i += 2) {
                if (col0 + i * 8 < c.rank16) {
                    uint32_t b[4];
                    ldsm_x4_t(b, va + 2 * (col0 + i * 8));
                    mma_bf16(o[i], p[0], p[1], p[2], p[3], b[0], b[1]);
                    mma_bf16(o[i + 1], p[0], p[1], p[2], p[3], b[2], b[3]);
                }
            }
        }
        __syncthreads();
        if (k0 + ST * KEYS < end) fetch(k0 + ST * KEYS, buf);
        cp_async_commit();
    }
    cp_async_wait<0>();
    if (tid % LM_ROW_THREADS == 0) { l_s[grp][tid / LM_ROW_THREADS] = l; m_s[grp][tid / LM_ROW_THREADS] = m; }
    if (n_splits == 1) {
        group_sync(grp);
#pragma unroll
        for (int r2 = 0; r2 < 2; ++r2) {
            const int r = g + 8 * r2, h = h0 + r;
            if (h >= s.heads) continue;
            const float inv = 1.0f / l_s[grp][r];
            bf16* d = out + ((int64_t)t * s.heads + h) * ldo + col0 + 2 * tq;
#pragma unroll
            for (int i = 0; i < NT; ++i) {
                const int e = col0 + i * 8 + 2 * tq;
                if (e + 1 < c.rank) *reinterpret_cast<uint32_t*>(d + 8 * i) = pack_bf16(o[i][2 * r2] * inv, o[i][2 * r2 + 1] * inv);
                else if (e < c.rank) d[8 * i] = __float2bfloat16_rn(o[i][2 * r2] * inv);
            }
        }
        return;
    }
    // The splits are the blocks of a cluster: each leaves its mixtures (relative to its own maxima) where the key ring was
    // and adds up a share of the columns of all of them, in split order.
    __syncthreads();
    const int LDO = c.rank16 + 8;
    float* mix = reinterpret_cast<float*>(lm_smem_raw);  // [HG * 16][LDO]
#pragma unroll
    for (int i = 0; i < NT; ++i) {
        if (col0 + i * 8 < c.rank16) {
            float* d = mix + (grp * 16 + g) * LDO + col0 + i * 8 + 2 * tq;
            *reinterpret_cast<float2*>(d) = make_float2(o[i][0], o[i][1]);
            *reinterpret_cast<float2*>(d + 8 * LDO) = make_float2(o[i][2], o[i][3]);
        }
    }
    cluster_sync();
    {
        // a thread per (head, split)
        static_assert(LM_WARPS * 32 == 16 * LM_MAX_SPLITS, "16 heads x 16 splits per group");
        const int hh = threadIdx.x / LM_MAX_SPLITS, p = threadIdx.x % LM_MAX_SPLITS;
        const bool on = p < n_splits;
        const float mp = on ? ld_peer(peer_smem(smem_addr(&m_s[0][0] + hh), p)) : -INFINITY, lp = on ? ld_peer(peer_smem(smem_addr(&l_s[0][0] + hh), p)) : 0.f;
        float M = mp;
#pragma unroll
        for (int off = LM_MAX_SPLITS / 2; off > 0; off >>= 1) M = fmaxf(M, __shfl_xor_sync(0xFFFFFFFFu, M, off));
        const float f = mp == -INFINITY ? 0.f : expf(mp - M);
        float L = f * lp;
#pragma unroll
        for (int off = LM_MAX_SPLITS / 2; off > 0; off >>= 1) L += __shfl_xor_sync(0xFFFFFFFFu, L, off);
        share_s[hh][p] = f / L;
    }
    __syncthreads();
    const int pairs = (c.rank + 1) / 2, rows = min(HG * 16, s.heads - (int)blockIdx.x * HG * 16);
    for (int idx = blockIdx.z * blockDim.x + threadIdx.x; idx < rows * pairs; idx += n_splits * blockDim.x) {
        const int r = idx / pairs, e = 2 * (idx - r * pairs);
        const uint32_t at = smem_addr(mix + r * LDO + e);
        float x = 0.f, y = 0.f;
        for (int p0 = 0; p0 < n_splits; p0 += 4) {  // n_splits is a power of two
            float2 v[4];
#pragma unroll
            for (int p = 0; p < 4; ++p) v[p] = p0 + p < n_splits ? ld_peer2(peer_smem(at, p0 + p)) : make_float2(0.f, 0.f);
#pragma unroll
            for (int p = 0; p < 4; ++p) {
                x = fmaf(share_s[r][p0 + p], v[p].x, x);
                y = fmaf(share_s[r][p0 + p], v[p].y, y);
            }
        }
        bf16* d = out + ((int64_t)t * s.heads + blockIdx.x * HG * 16 + r) * ldo + e;
        if (e + 1 < c.rank) *reinterpret_cast<uint32_t*>(d) = pack_bf16(x, y);
        else d[0] = __float2bfloat16_rn(x);
    }
    cluster_sync();  // nobody leaves while its mixtures are being read
}

// Block (head, token, 128 columns).
constexpr int LATENT_MAX_SPLITS = 16;
template <typename T>
__global__ void __launch_bounds__(128) latent_merge_kernel(const float* __restrict__ part, int heads, int n_splits, int rank, T* __restrict__ out, int ldo) {
    __shared__ float w_s[LATENT_MAX_SPLITS];
    pdl_wait();
    pdl_trigger();
    const int64_t th = (int64_t)blockIdx.y * heads + blockIdx.x;
    const float* src = part + th * n_splits * (rank + 2);
    const int e = blockIdx.z * 128 + threadIdx.x;
    float v[LATENT_MAX_SPLITS];
#pragma unroll
    for (int i = 0; i < LATENT_MAX_SPLITS; ++i) v[i] = i < n_splits && e < rank ? src[(int64_t)i * (rank + 2) + 2 + e] : 0.f;
    if (threadIdx.x < 32) {
        const int i = threadIdx.x;
        const float m = i < n_splits ? src[(int64_t)i * (rank + 2)] : -INFINITY, l = i < n_splits ? src[(int64_t)i * (rank + 2) + 1] : 0.f;
        const float M = warp_max(m);
        const float f = m == -INFINITY ? 0.f : expf(m - M);
        const float L = warp_sum(f * l);
        if (i < LATENT_MAX_SPLITS) w_s[i] = f / L;
    }
    __syncthreads();
    float o = 0.f;
#pragma unroll
    for (int i = 0; i < LATENT_MAX_SPLITS; ++i) o = fmaf(w_s[i], v[i], o);
    if (e < rank) out[th * ldo + e] = from_f32<T>(o);
}

// Two head groups share a block's keys once there are tokens enough to fill the device without splitting the heads up.
static int latent_head_groups(int heads, int n_tok) { return heads > 16 && n_tok >= 8 ? 2 : 1; }

int latent_attention_splits(int heads, int n_tok, int keys, bool f32) {
    const int hg = f32 ? 1 : latent_head_groups(heads, n_tok);
    const int blocks = (f32 ? heads : (heads + 16 * hg - 1) / (16 * hg)) * n_tok;
    const int slots = (hg == 1 ? 2 : 1) * device_sm_count();  // blocks the device holds at once
    const int most = hg == 1 ? LM_MAX_SPLITS : 8;             // (a cluster of 16 needs the small blocks)
    int n = 1;
    while (n < most && blocks * 2 * n <= slots && keys >= 64 * 2 * n) n <<= 1;
    return n;
}

size_t latent_part_floats(int n_tok, int heads, int n_splits, int rank) { return n_splits > 1 ? (size_t)n_tok * heads * n_splits * (rank + 2) : 0; }

cudaError_t launch_latent_attention(const void* qabs, const LatentShape& s, const LatentCache& c, const int32_t* tok_slot, const int32_t* tok_pos,
                                    void* o, int ldo, float* part, int n_splits, bool f32, int n_tok, cudaStream_t st) {
    if (n_tok == 0) return cudaSuccess;
    if (n_splits < 1 || n_splits > LATENT_MAX_SPLITS || (n_splits > 1 && !part) || c.rank > 32 * LS_MAX_PER_LANE) return cudaErrorInvalidValue;
    constexpr int CAP = 200 * 1024;
    static PerDeviceOnce once;
    cudaError_t le = once.run([] {
        const void* fns[] = {(const void*)latent_attention_mma_kernel<2, 1, 32, 2>, (const void*)latent_attention_mma_kernel<4, 1, 32, 2>,
                             (const void*)latent_attention_mma_kernel<8, 1, 32, 2>, (const void*)latent_attention_mma_kernel<2, 2, 32, 4>,
                             (const void*)latent_attention_mma_kernel<4, 2, 32, 4>, (const void*)latent_attention_mma_kernel<8, 2, 32, 4>,
                             (const void*)latent_attention_simple_kernel<float>, (const void*)latent_attention_simple_kernel<bf16>};
        for (const void* f : fns) {
            const cudaError_t e = cudaFuncSetAttribute(f, cudaFuncAttributeMaxDynamicSharedMemorySize, CAP);
            if (e != cudaSuccess) return e;
        }
        const void* wide[] = {(const void*)latent_attention_mma_kernel<2, 1, 32, 2>, (const void*)latent_attention_mma_kernel<4, 1, 32, 2>,
                              (const void*)latent_attention_mma_kernel<8, 1, 32, 2>};
        for (const void* f : wide) {
            const cudaError_t e = cudaFuncSetAttribute(f, cudaFuncAttributeNonPortableClusterSizeAllowed, 1);
            if (e != cudaSuccess) return e;
        }
        return cudaSuccess;
    });
    if (le != cudaSuccess) return le;
    const int width = c.rank16 + c.rot16;
    const int per_warp = (c.rank16 + 8 * LM_WARPS - 1) / (8 * LM_WARPS);  // 8-column tiles each warp has to cover
    const int hg = latent_head_groups(s.heads, n_tok);
    // one head group: two blocks per SM; two groups: one block of 16 warps and a deeper ring
    const size_t smem = lm_smem(width, hg, 32, hg == 1 ? 2 : 4);
    if (!f32 && per_warp <= 8 && width <= 16 * LM_WARPS * LM_MAX_STEPS && smem <= CAP && n_splits <= (hg == 1 ? LM_MAX_SPLITS : 8)) {
        const dim3 grid((s.heads + 16 * hg - 1) / (16 * hg), n_tok, n_splits), block(LM_WARPS * 32 * hg);
#define SP_LM(NT)                                                                                                                                  \
    le = hg == 1 ? launch_pdl_cluster(latent_attention_mma_kernel<NT, 1, 32, 2>, grid, block, smem, st, n_splits, (const bf16*)qabs, s, c, tok_slot, tok_pos, (bf16*)o, ldo, n_splits) \
                 : launch_pdl_cluster(latent_attention_mma_kernel<NT, 2, 32, 4>, grid, block, smem, st, n_splits, (const bf16*)qabs, s, c, tok_slot, tok_pos, (bf16*)o, ldo, n_splits)
        if (per_warp <= 2) SP_LM(2);
        else if (per_warp <= 4) SP_LM(4);
        else SP_LM(8);
#undef SP_LM
        return le != cudaSuccess ? le : count_launch_and_check();
    } else {
        const dim3 grid(s.heads, n_tok, n_splits), block(LS_WARPS * 32);
        const size_t smem = (size_t)(width + LS_WARPS * c.rank) * 4;
        if (smem > CAP) return cudaErrorInvalidValue;
        le = f32 ? launch_pdl(latent_attention_simple_kernel<float>, grid, block, smem, st, (const float*)qabs, s, c, tok_slot, tok_pos, (float*)o, ldo, part, n_splits)
                 : launch_pdl(latent_attention_simple_kernel<bf16>, grid, block, smem, st, (const bf16*)qabs, s, c, tok_slot, tok_pos, (bf16*)o, ldo, part, n_splits);
    }
    if (le != cudaSuccess) return le;
    le = count_launch_and_check();
    if (le != cudaSuccess || n_splits == 1) return le;
    le = f32 ? launch_pdl(latent_merge_kernel<float>, dim3(s.heads, n_tok, (c.rank + 127) / 128), dim3(128), 0, st, (const float*)part, s.heads, n_splits, c.rank, (float*)o, ldo)
             : launch_pdl(latent_merge_kernel<bf16>, dim3(s.heads, n_tok, (c.rank + 127) / 128), dim3(128), 0, st, (const float*)part, s.heads, n_splits, c.rank, (bf16*)o, ldo);
    if (le != cudaSuccess) return le;
    return count_launch_and_check();
}

// ── expanded attention ──
__global__ void latent_gather_kernel(const LatentCache c, const int32_t* __restrict__ key_slot, const int32_t* __restrict__ key_pos, uint4* __restrict__ dst) {
    pdl_wait();
    pdl_trigger();
    const int pos = key_pos[blockIdx.x], page = c.page_table[(int64_t)key_slot[blockIdx.x] * c.max_pages + pos / KV_PAGE];
    const int ld16 = c.ld / 8;
    const uint4* src = reinterpret_cast<const uint4*>(c.pool) + ((int64_t)page * KV_PAGE + pos % KV_PAGE) * ld16;
    for (int i = threadIdx.x; i < ld16; i += blockDim.x) dst[(int64_t)blockIdx.x * ld16 + i] = src[i];
}

cudaError_t launch_latent_gather(const LatentCache& c, const int32_t* key_slot, const int32_t* key_pos, int n_keys, void* dst, cudaStream_t st) {
    if (n_keys == 0) return cudaSuccess;
    cudaError_t le = launch_pdl(latent_gather_kernel, dim3(n_keys), dim3(64), 0, st, c, key_slot, key_pos, (uint4*)dst);
    if (le != cudaSuccess) return le;
    return count_launch_and_check();
}

// Block per (head, tile of 64 tokens), 4 warps x 16 query rows, key tiles of 64 double-buffered with cp.async.
constexpr int LE_KEYS = 64, LE_WARPS = 4;
static int le_smem(int dim16, int rot16, int vdim16) { return (3 * 64 * (dim16 + rot16 + 8) + 2 * LE_KEYS * (vdim16 + 8)) * 2; }
bool latent_expanded_supported(int dim, int rot, int vdim) {
    const int d = (dim + 15) & ~15, r = (rot + 15) & ~15, v = (vdim + 15) & ~15;
    return v <= 256 && le_smem(d, r, v) <= 200 * 1024;
}

template <int VT>
__global__ void __launch_bounds__(LE_WARPS * 32) latent_expanded_kernel(const bf16* __restrict__ qf, const bf16* __restrict__ kv, const bf16* __restrict__ lat,
                                                                        const LatentShape s, int rank16, int rot16, int ldl, const LatentTile* __restrict__ tiles,
                                                                        const float* __restrict__ gate, int ldgate, bf16* __restrict__ out, int ldo) {
    extern __shared__ __align__(16) bf16 le_sm[];
    pdl_wait();
    pdl_trigger();
    const int dim16 = (s.dim + 15) & ~15, vdim16 = (s.vdim + 15) & ~15, qw = dim16 + rot16, LQ = qw + 8, LV = vdim16 + 8, kvw = dim16 + vdim16;
    bf16 *qs = le_sm, *ks = qs + 64 * LQ, *vs = ks + 2 * LE_KEYS * LQ;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, tq = lane & 3;
    const int h = blockIdx.x;
    const LatentTile tl = tiles[blockIdx.y];
    // copies: eight lanes per row, four rows per warp and instruction
    const int l8 = lane & 7, lr = warp * 16 + (lane >> 3);
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int r = lr + 4 * i;
        const bf16* src = qf + ((int64_t)(tl.row0 + min(r, tl.n - 1)) * s.heads + h) * qw;
        for (int p = l8; p < qw / 8; p += 8) cp_async16(qs + r * LQ + p * 8, src + p * 8, 16);
    }
    const int hi = tl.pos0 + tl.n - 1, lo = s.window > tl.pos0 ? 0 : tl.pos0 - s.window + 1;
    auto fetch = [&](int k0, int buf) {
        bf16 *kd = ks + buf * LE_KEYS * LQ, *vd = vs + buf * LE_KEYS * LV;
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int r = lr + 4 * i, key = min(k0 + r, hi), bytes = k0 + r <= hi ? 16 : 0;
            const int64_t row = tl.key_row + (key - tl.key_pos0);
            const bf16 *kvr = kv + (row * s.heads + h) * kvw, *rr = lat + row * ldl + rank16;
            for (int p = l8; p < dim16 / 8; p += 8) cp_async16(kd + r * LQ + p * 8, kvr + p * 8, bytes);
            for (int p = l8; p < rot16 / 8; p += 8) cp_async16(kd + r * LQ + dim16 + p * 8, rr + p * 8, bytes);
            for (int p = l8; p < vdim16 / 8; p += 8) cp_async16(vd + r * LV + p * 8, kvr + dim16 + p * 8, bytes);
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
    for (int k0 = lo, buf = 0; k0 <= hi; k0 += LE_KEYS, buf ^= 1) {
        cp_async_wait<0>();
        __syncthreads();
        if (k0 + LE_KEYS <= hi) fetch(k0 + LE_KEYS, buf ^ 1);
        cp_async_commit();
        const bf16 *kt = ks + buf * LE_KEYS * LQ, *vt = vs + buf * LE_KEYS * LV;
        float sc[8][4];
#pragma unroll
        for (int j = 0; j < 8; ++j) sc[j][0] = sc[j][1] = sc[j][2] = sc[j][3] = 0.f;
        const uint32_t qa = smem_addr(qs + (warp * 16 + (lane & 15)) * LQ + (lane >> 4) * 8);
        const uint32_t ka = smem_addr(kt + ((lane & 7) + (lane >> 4) * 8) * LQ + ((lane >> 3) & 1) * 8);
        for (int k = 0; k < qw; k += 16) {
            uint32_t q[4];
            ldsm_x4(q, qa + 2 * k);
#pragma unroll
            for (int j = 0; j < 8; j += 2) {
                uint32_t b[4];
                ldsm_x4(b, ka + 2 * (8 * j * LQ + k));
                mma_bf16(sc[j], q[0], q[1], q[2], q[3], b[0], b[1]);
                mma_bf16(sc[j + 1], q[0], q[1], q[2], q[3], b[2], b[3]);
            }
        }
        float x0 = m0, x1 = m1;
        // only the window's two ends need the mask
        const bool edge = k0 + LE_KEYS - 1 > tl.pos0 || (int64_t)hi - k0 >= s.window;
#pragma unroll
        for (int j = 0; j < 8; ++j) {
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const int key = k0 + 8 * j + 2 * tq + e;
                sc[j][e] = (!edge || (key <= p0 && p0 - key < s.window)) ? sc[j][e] * s.scale : -INFINITY;
                sc[j][2 + e] = (!edge || (key <= p1 && p1 - key < s.window)) ? sc[j][2 + e] * s.scale : -INFINITY;
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
            const uint32_t a0 = pack_bf16(sc[2 * kk][0], sc[2 * kk][1]), a1 = pack_bf16(sc[2 * kk][2], sc[2 * kk][3]);
            const uint32_t a2 = pack_bf16(sc[2 * kk + 1][0], sc[2 * kk + 1][1]), a3 = pack_bf16(sc[2 * kk + 1][2], sc[2 * kk + 1][3]);
            const uint32_t va = smem_addr(vt + (kk * 16 + (lane & 15)) * LV + (lane >> 4) * 8);
#pragma unroll
            for (int i = 0; i < VT; i += 2) {
                if (i * 8 < vdim16) {
                    uint32_t b[4];
                    ldsm_x4_t(b, va + 2 * (i * 8));
                    mma_bf16(o[i], a0, a1, a2, a3, b[0], b[1]);
                    mma_bf16(o[i + 1], a0, a1, a2, a3, b[2], b[3]);
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
#pragma unroll
    for (int r2 = 0; r2 < 2; ++r2) {
        const int r = r2 ? r1 : r0;
        if (r >= tl.n) continue;
        const int64_t row = tl.row0 + r;
        const float f = (gate ? sigmoid_f32(gate[row * ldgate + h]) : 1.f) / (r2 ? l1 : l0);
        bf16* d = out + row * ldo + (int64_t)h * s.vdim;
#pragma unroll
        for (int i = 0; i < VT; ++i) {
            const int e = i * 8 + 2 * tq;
            if (e < s.vdim) d[e] = __float2bfloat16_rn(o[i][2 * r2] * f);
            if (e + 1 < s.vdim) d[e + 1] = __float2bfloat16_rn(o[i][2 * r2 + 1] * f);
        }
    }
}

cudaError_t launch_latent_expanded(const void* qf, const void* kv, const void* lat, const LatentShape& s, const LatentCache& c,
                                   const LatentTile* tiles, int n_tiles, const float* gate, int ldgate, void* out, int ldo, cudaStream_t st) {
    if (n_tiles == 0) return cudaSuccess;
    if (!latent_expanded_supported(s.dim, s.rot, s.vdim)) return cudaErrorInvalidValue;
    constexpr int CAP = 200 * 1024;
    static PerDeviceOnce once;
    cudaError_t le = once.run([] {
        const void* fns[] = {(const void*)latent_expanded_kernel<4>, (const void*)latent_expanded_kernel<8>, (const void*)latent_expanded_kernel<16>,
                             (const void*)latent_expanded_kernel<32>};
        for (const void* f : fns) {
            const cudaError_t e = cudaFuncSetAttribute(f, cudaFuncAttributeMaxDynamicSharedMemorySize, CAP);
            if (e != cudaSuccess) return e;
        }
        return cudaSuccess;
    });
    if (le != cudaSuccess) return le;
    const int vdim16 = (s.vdim + 15) & ~15;
    const size_t smem = (size_t)le_smem((s.dim + 15) & ~15, c.rot16, vdim16);
    const dim3 grid(s.heads, n_tiles), block(LE_WARPS * 32);
#define SP_LE(VT) le = launch_pdl(latent_expanded_kernel<VT>, grid, block, smem, st, (const bf16*)qf, (const bf16*)kv, (const bf16*)lat, s, c.rank16, c.rot16, c.ld, tiles, gate, ldgate, (bf16*)out, ldo)
    if (vdim16 <= 32) SP_LE(4);
    else if (vdim16 <= 64) SP_LE(8);
    else if (vdim16 <= 128) SP_LE(16);
    else SP_LE(32);
#undef SP_LE
    if (le != cudaSuccess) return le;
    return count_launch_and_check();
}

}  // namespace sp
