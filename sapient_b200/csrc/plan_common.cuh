// Shared device helpers of the plan kernels: the compute type's loads and stores, warp mma, reductions.
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include "plan_kernels.h"
#include "sp_common.cuh"

namespace sp {

using bf16 = __nv_bfloat16;

__device__ __forceinline__ float to_f32(float v) { return v; }
__device__ __forceinline__ float to_f32(bf16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T from_f32(float v);
template <> __device__ __forceinline__ float from_f32<float>(float v) { return v; }
template <> __device__ __forceinline__ bf16 from_f32<bf16>(float v) { return __float2bfloat16_rn(v); }

__device__ __forceinline__ float sigmoid_f32(float z) { return 1.0f / (1.0f + expf(-z)); }

// The gated unit of plan_kernels.h: MatUnit.
__device__ __forceinline__ float gated_unit(float g, float u, const MatUnit& p) {
    g = fminf(g, p.limit);
    u = fminf(fmaxf(u, -p.limit), p.limit);
    return g * sigmoid_f32(p.alpha * g) * (u + p.shift);
}

__device__ __forceinline__ float silu_f32(float z) { return z * sigmoid_f32(z); }

// The activation of a product's output range (plan_kernels.h: MatOut).
__device__ __forceinline__ float mat_act(int act, float z, const float (&arg)[2]) {
    switch (act) {
        case MAT_RELU2: z = fmaxf(z, 0.f); return z * z;
        case MAT_TANH: return tanhf(z);
        case MAT_SILU: return silu_f32(z);
        case MAT_SOFTCAP: return arg[1] > 0.f ? arg[1] * tanhf(z * arg[0] / arg[1]) : z * arg[0];
        case MAT_XIELU: return fmaf(0.5f, z, z > 0.f ? arg[0] * z * z : arg[1] * (expm1f(z) - z));
        default: return z;
    }
}

// tanh z = 1 - 2 / (e^(2 z) + 1): no branches, an absolute error of a few 2^-24.
__device__ __forceinline__ float tanh_by_exp(float z) { return fmaf(-2.f, __fdividef(1.f, __expf(2.f * z) + 1.f), 1.f); }
// The same for several values at once in a product on bf16 operands: one decision for all, fast exponentials and divisions
// (errors of a few 2^-22). Short, since a decoded token's product is mostly the fetching of its weights and its code.
template <int N>
__device__ __forceinline__ void mat_act_fast(int act, float (&z)[N], const float (&arg)[2]) {
    switch (act) {
        case MAT_ID: return;
        case MAT_RELU2:
#pragma unroll
            for (int i = 0; i < N; ++i) {
                z[i] = fmaxf(z[i], 0.f);
                z[i] *= z[i];
            }
            return;
        case MAT_SILU:
#pragma unroll
            for (int i = 0; i < N; ++i) z[i] = __fdividef(z[i], 1.f + __expf(-fmaxf(z[i], -80.f)));
            return;
        case MAT_XIELU:
#pragma unroll
            for (int i = 0; i < N; ++i) {
                const float left = fminf(z[i], 0.f), right = fmaxf(z[i], 0.f);  // one of the two is zero, and so is its term
                z[i] = fmaf(arg[0] * right, right, fmaf(arg[1], __expf(left) - 1.f - left, 0.5f * z[i]));
            }
            return;
        case MAT_TANH:
#pragma unroll
            for (int i = 0; i < N; ++i) z[i] = tanh_by_exp(z[i]);
            return;
        case MAT_SOFTCAP: {
            const bool cap = arg[1] > 0.f;
            const float scale = cap ? arg[0] / arg[1] : arg[0];
#pragma unroll
            for (int i = 0; i < N; ++i) z[i] = cap ? arg[1] * tanh_by_exp(z[i] * scale) : z[i] * scale;
        }
    }
}

__device__ __forceinline__ float tanh_norm(const TanhNorm& n, float x, int c) { return fmaf(tanhf(n.alpha * x), n.w[c], n.b[c]); }

// Sum over the block, the same value in every thread. sh: one float per warp.
template <int WARPS>
__device__ __forceinline__ float block_sum(float v, float* sh) {
    v = warp_sum(v);
    if ((threadIdx.x & 31) == 0) sh[threadIdx.x >> 5] = v;
    __syncthreads();
    float s = 0.f;
#pragma unroll
    for (int w = 0; w < WARPS; ++w) s += sh[w];
    return s;
}

__device__ __forceinline__ void mma_bf16(float (&c)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint32_t smem_addr(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void ldsm_x4(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ldsm_x4_t(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ldsm_x2(uint32_t (&r)[2], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0,%1}, [%2];\n" : "=r"(r[0]), "=r"(r[1]) : "r"(addr) : "memory");
}
// 16 bytes to shared memory; bytes = 0 reads nothing and writes zeros.
__device__ __forceinline__ void cp_async16(void* dst, const void* src, int bytes) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(smem_addr(dst)), "l"(src), "r"(bytes) : "memory");
}
__device__ __forceinline__ void cp_async16_at(uint32_t dst, const void* src, int bytes) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(dst), "l"(src), "r"(bytes) : "memory");
}
__device__ __forceinline__ void cp_async4(void* dst, const void* src) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;\n" ::"r"(smem_addr(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;\n" ::: "memory"); }
template <int N> __device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;\n" ::"n"(N) : "memory"); }

__device__ __forceinline__ uint32_t pack_bf16(float a, float b) {
    const __nv_bfloat162 v = __floats2bfloat162_rn(a, b);
    return *reinterpret_cast<const uint32_t*>(&v);
}

// A barrier of all threads of the cluster; shared-memory writes before it are visible to the peers after it.
__device__ __forceinline__ void cluster_sync() {
    asm volatile("barrier.cluster.arrive.release;\nbarrier.cluster.wait.acquire;\n" ::: "memory");
}
__device__ __forceinline__ uint32_t peer_smem(uint32_t addr, int rank) {
    uint32_t r;
    asm volatile("mapa.shared::cluster.u32 %0, %1, %2;\n" : "=r"(r) : "r"(addr), "r"(rank));
    return r;
}
__device__ __forceinline__ float ld_peer(uint32_t addr) {
    float v;
    asm volatile("ld.shared::cluster.f32 %0, [%1];\n" : "=f"(v) : "r"(addr) : "memory");
    return v;
}

__device__ __forceinline__ float2 ld_peer2(uint32_t addr) {
    float2 v;
    asm volatile("ld.shared::cluster.v2.f32 {%0, %1}, [%2];\n" : "=f"(v.x), "=f"(v.y) : "r"(addr) : "memory");
    return v;
}

}  // namespace sp
