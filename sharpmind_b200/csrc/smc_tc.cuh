// tcgen05 / TMEM / tiled-TMA primitives of the dense tensor-core kernel: bounded mbarrier waits with a CTA-wide abort
// flag, 128-byte-swizzled shared-memory matrix descriptors, MMA issue and accumulator reads.
#pragma once

#include <cuda.h>  // CUtensorMap (types only: the encoder is looked up through the runtime)

#include "smc_async.cuh"

#ifdef __CUDACC__
// Bounded wait of one thread; raises the abort flag and the context's status word when the limit runs out and returns,
// so that the kernel ends in bounded time whatever went wrong.
__device__ __forceinline__ void smc_tc_wait(uint32_t bar, uint32_t parity, volatile uint32_t *abort_flag, int *status)
{
    for (unsigned i = 0; i < SMC_WAIT_LIMIT; ++i) {
        if (smc_mbar_try_wait(bar, parity)) return;
        if ((i & 255u) == 255u && *abort_flag) return;
    }
    *abort_flag = 1;
    atomicExch(status, 4);
}
__device__ __forceinline__ void smc_tc_fence_before() { asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory"); }
__device__ __forceinline__ void smc_tc_fence_after() { asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory"); }
__device__ __forceinline__ void smc_tc_commit(uint32_t bar)
{
    asm volatile("tcgen05.commit.cta_group::1.mbarrier::arrive::one.shared::cluster.b64 [%0];" ::"r"(bar) : "memory");
}
__device__ __forceinline__ void smc_tc_alloc(uint32_t smem_dst, uint32_t cols)
{
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_dst), "r"(cols) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
}
__device__ __forceinline__ void smc_tc_dealloc(uint32_t tmem, uint32_t cols)
{
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(cols) : "memory");
}
// D[tmem] (+)= A[smem] * B[smem]^T, 16-bit operands of one type, fp32 accumulate; issued by one thread.
__device__ __forceinline__ void smc_tc_mma(uint32_t tmem_d, uint64_t adesc, uint64_t bdesc, uint32_t idesc, uint32_t accumulate)
{
    asm volatile(
        "{\n\t.reg .pred p;\n\tsetp.ne.b32 p, %4, 0;\n\t"
        "tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, p;\n\t}"
        :
        : "r"(tmem_d), "l"(adesc), "l"(bdesc), "r"(idesc), "r"(accumulate)
        : "memory");
}
// 16 consecutive fp32 columns of this thread's TMEM lane (complete after smc_tc_wait_ld).
__device__ __forceinline__ void smc_tc_ld16(uint32_t taddr, uint32_t (&r)[16])
{
    asm volatile(
        "tcgen05.ld.sync.aligned.32x32b.x16.b32 {%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15}, [%16];"
        : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]), "=r"(r[8]),
          "=r"(r[9]), "=r"(r[10]), "=r"(r[11]), "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15])
        : "r"(taddr)
        : "memory");
}
__device__ __forceinline__ void smc_tc_wait_ld() { asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory"); }
// K-major operand tile of 64 16-bit elements per row (128 bytes), rows in groups of eight of 1024 bytes, stored with the
// 128-byte swizzle a tiled TMA load applies.  The tile starts on a 1024-byte boundary; k advances by 32 bytes per MMA.
__device__ __forceinline__ uint64_t smc_tc_desc_sw128(uint32_t addr)
{
    return (uint64_t)((addr >> 4) & 0x3FFFu) | (1ull << 16) | ((uint64_t)(1024u >> 4) << 32) | (1ull << 46) | (2ull << 61);
}
// Instruction descriptor: fp32 accumulator, bfloat16 A and B, both K-major.
__host__ __device__ constexpr uint32_t smc_tc_idesc_bf16(int m, int n)
{
    return (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(n >> 3) << 17) | ((uint32_t)(m >> 4) << 24);
}
// Box of a 2-D tensor map -> shared memory; x (innermost, elements) must start on a 16-byte boundary.
__device__ __forceinline__ void smc_tma_2d(uint32_t dst, const CUtensorMap *map, int x, int y, uint32_t bar)
{
    asm volatile("cp.async.bulk.tensor.2d.shared::cluster.global.tile.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3}], [%4];" ::"r"(dst),
                 "l"(map), "r"(x), "r"(y), "r"(bar)
                 : "memory");
}
#endif
