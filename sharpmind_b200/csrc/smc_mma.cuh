// Device helpers shared by the layered decoders' kernels: element conversion, bfloat16 mma.sync fragments, 16-byte copies.
#pragma once
#include <cuda_bf16.h>

#include "smc_common.cuh"

#ifdef __CUDACC__
namespace {

typedef __nv_bfloat16 bf16;

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(bf16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T from_f(float v);
template <> __device__ __forceinline__ float from_f<float>(float v) { return v; }
template <> __device__ __forceinline__ bf16 from_f<bf16>(float v) { return __float2bfloat16_rn(v); }
__device__ __forceinline__ float silu(float z) { return __fdiv_rn(z, 1.0f + expf(-z)); }
// in front of a bfloat16 rounding the approximate exponential and quotient are enough
template <typename T> __device__ __forceinline__ float silu_for(float z) { return silu(z); }
template <> __device__ __forceinline__ float silu_for<bf16>(float z) { return __fdividef(z, 1.0f + __expf(-z)); }

// slot and position of row r of a batch
__device__ __forceinline__ void row_place(const smc_rows &rw, int r, int &slot, int &p)
{
    slot = rw.seq0 >= 0 ? rw.seq0 : r;
    p = rw.pos[slot] + (rw.seq0 >= 0 ? r : 0);
}

// V neighbouring elements as one access
template <typename T, int V> struct Pack;
template <> struct Pack<float, 1> { using type = float; };
template <> struct Pack<bf16, 1> { using type = bf16; };
template <> struct Pack<bf16, 4> { using type = uint2; };
template <> struct Pack<float, 4> { using type = float4; };
template <typename T, int V>
__device__ __forceinline__ void load_v(const T *p, float (&v)[V])
{
    typename Pack<T, V>::type raw = *reinterpret_cast<const typename Pack<T, V>::type *>(p);
    const T *e = reinterpret_cast<const T *>(&raw);
#pragma unroll
    for (int i = 0; i < V; ++i) v[i] = to_f(e[i]);
}
template <typename T, int V>
__device__ __forceinline__ void store_v(T *p, const float (&v)[V])
{
    typename Pack<T, V>::type raw;
    T *e = reinterpret_cast<T *>(&raw);
#pragma unroll
    for (int i = 0; i < V; ++i) e[i] = from_f<T>(v[i]);
    *reinterpret_cast<typename Pack<T, V>::type *>(p) = raw;
}

__device__ __forceinline__ void mma_bf16(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1)
{
    asm("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
        : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
        : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ldsm4(uint32_t addr, uint32_t (&r)[4])
{
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldsm4t(uint32_t addr, uint32_t (&r)[4])
{
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
// 16 bytes global -> shared, zeros when `in` is false (the address must be valid either way)
__device__ __forceinline__ void cp16(uint32_t dst, const void *src, bool in)
{
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(in ? 16 : 0) : "memory");
}
// 2^x for x <= 0
__device__ __forceinline__ float ex2(float x)
{
    float v;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(v) : "f"(x));
    return v;
}
__device__ __forceinline__ uint32_t pack2(float a, float b)
{
    const __nv_bfloat162 v = __floats2bfloat162_rn(a, b);
    return *reinterpret_cast<const uint32_t *>(&v);
}
// {a, b} as bfloat16 pairs: hi, and lo = what hi leaves
__device__ __forceinline__ void split2(float a, float b, uint32_t &hi, uint32_t &lo)
{
    const bf16 ah = __float2bfloat16_rn(a), bh = __float2bfloat16_rn(b);
    const __nv_bfloat162 h = __halves2bfloat162(ah, bh), l = __floats2bfloat162_rn(a - __bfloat162float(ah), b - __bfloat162float(bh));
    hi = *reinterpret_cast<const uint32_t *>(&h), lo = *reinterpret_cast<const uint32_t *>(&l);
}

}  // namespace
#endif
