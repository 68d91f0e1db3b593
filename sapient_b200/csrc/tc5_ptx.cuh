// Inline PTX of the 5th-generation tensor cores and the TMA / mbarrier plumbing around them, shared by the GEMMs that use
// them (gemm_tc5.cu: quantised weights rebuilt into tensor memory; mat_tc5.cu: bf16 operands from shared memory).
#pragma once
#include <cuda.h>
#include <cuda_runtime.h>
#include <stdint.h>

namespace sp {

constexpr int TC5_SPIN_LIMIT = 1 << 22;

__device__ __forceinline__ uint32_t tc5_smem_u32(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }

// Shared-memory matrix descriptor: K-major operand, 128-byte swizzle, rows of 128 B, 8-row groups 1024 B apart.
__device__ __forceinline__ uint64_t tc5_desc(uint32_t saddr) {
    uint64_t d = 0;
    d |= (uint64_t)((saddr & 0x3FFFFu) >> 4);  // start address / 16
    d |= (uint64_t)1 << 16;                    // leading-dimension byte offset / 16 (not used by swizzled K-major)
    d |= (uint64_t)(1024 >> 4) << 32;          // stride-dimension byte offset / 16: next 8-row group
    d |= (uint64_t)1 << 46;                    // descriptor version of this architecture
    d |= (uint64_t)2 << 61;                    // 128-byte swizzle
    return d;
}

__device__ __forceinline__ void tc5_mma(uint32_t d_tmem, uint64_t adesc, uint64_t bdesc, uint32_t idesc, uint32_t accumulate) {
    asm volatile(
        "{\n"
        ".reg .pred p;\n"
        "setp.ne.b32 p, %4, 0;\n"
        "tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, p;\n"
        "}\n" ::"r"(d_tmem), "l"(adesc), "l"(bdesc), "r"(idesc), "r"(accumulate)
        : "memory");
}

__device__ __forceinline__ void tc5_commit(uint64_t* bar) {
    asm volatile("tcgen05.commit.cta_group::1.mbarrier::arrive::one.shared::cluster.b64 [%0];\n" ::"r"(tc5_smem_u32(bar)) : "memory");
}

__device__ __forceinline__ void tc5_arrive(uint64_t* bar) {
    asm volatile("mbarrier.arrive.shared::cta.b64 _, [%0];\n" ::"r"(tc5_smem_u32(bar)) : "memory");
}

__device__ __forceinline__ bool tc5_wait(uint64_t* bar, uint32_t parity) {
    const uint32_t a = tc5_smem_u32(bar);
    for (int i = 0; i < TC5_SPIN_LIMIT; ++i) {
        uint32_t done;
        asm volatile(
            "{\n"
            ".reg .pred p;\n"
            "mbarrier.try_wait.parity.shared::cta.b64 p, [%1], %2;\n"
            "selp.u32 %0, 1, 0, p;\n"
            "}\n"
            : "=r"(done)
            : "r"(a), "r"(parity)
            : "memory");
        if (done) return true;
    }
    return false;
}

// A box of a 2-D tensor map into shared memory, counted in bytes on `bar`. x (elements) must start on 16 bytes.
__device__ __forceinline__ void tc5_tma_2d(uint32_t dst, const CUtensorMap* map, int x, int y, uint32_t bar) {
    asm volatile(
        "cp.async.bulk.tensor.2d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3}], [%4];\n" ::"r"(dst), "l"(map),
        "r"(x), "r"(y), "r"(bar)
        : "memory");
}

// Brings a tensor map (a kernel parameter) into the descriptor cache ahead of its first copy.
__device__ __forceinline__ void tc5_prefetch_map(const CUtensorMap* map) {
    asm volatile("prefetch.tensormap [%0];\n" ::"l"(map) : "memory");
}

// 16 consecutive tensor-memory columns of the warp's 32 lanes, one lane per thread.
__device__ __forceinline__ void tc5_ld16(uint32_t taddr, uint32_t (&r)[16]) {
    asm volatile(
        "tcgen05.ld.sync.aligned.32x32b.x16.b32 {%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15}, [%16];\n"
        : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]), "=r"(r[8]), "=r"(r[9]),
          "=r"(r[10]), "=r"(r[11]), "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15])
        : "r"(taddr)
        : "memory");
}

typedef CUresult (*PFN_encodeTiled)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*,
                                    const cuuint32_t*, const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle,
                                    CUtensorMapL2promotion, CUtensorMapFloatOOBfill);

// The driver's tensor map encoder, resolved once (thread-safe); null where the driver lacks it.
inline PFN_encodeTiled tensor_map_encoder() {
    static const PFN_encodeTiled encode = [] {
        void* fn = nullptr;
        cudaDriverEntryPointQueryResult qres;
        if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &fn, cudaEnableDefault, &qres) != cudaSuccess) fn = nullptr;
        return reinterpret_cast<PFN_encodeTiled>(fn);
    }();
    return encode;
}

}  // namespace sp
