// Pieces of kernels that multiply on the tensor cores with mma.sync.m16n8k16 (bf16 operands, fp32 sums): the instruction, the
// loads of its operands from shared memory, and fp32 numbers as two bf16 numbers each (head and remainder), which keeps an operand
// 32-bit in effect.
#pragma once
#include "common.cuh"

typedef __nv_bfloat16 bf16;

namespace {

__device__ __forceinline__ void mma_16816(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ldsm4(uint32_t (&r)[4], const bf16* p) {
    const uint32_t a = (uint32_t)__cvta_generic_to_shared(p);
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a) : "memory");
}
__device__ __forceinline__ void ldsm4t(uint32_t (&r)[4], const bf16* p) {
    const uint32_t a = (uint32_t)__cvta_generic_to_shared(p);
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a) : "memory");
}
__device__ __forceinline__ uint32_t pack2(float x, float y) {
    const __nv_bfloat162 v = __floats2bfloat162_rn(x, y);
    return *(const uint32_t*)&v;
}
// head and remainder of two fp32 numbers as packed bf16 pairs
__device__ __forceinline__ void split2(float x, float y, uint32_t& hi, uint32_t& lo) {
    const bf16 hx = __float2bfloat16_rn(x), hy = __float2bfloat16_rn(y);
    const __nv_bfloat162 h = __halves2bfloat162(hx, hy);
    hi = *(const uint32_t*)&h;
    lo = pack2(x - __bfloat162float(hx), y - __bfloat162float(hy));
}
// channels c .. c + 7 of a row of n channels (zero beyond) as stored
__device__ __forceinline__ uint4 raw8(const bf16* src, int c, int n) {
    if (c + 8 <= n && (((uintptr_t)(src + c)) & 15) == 0) return *(const uint4*)(src + c);
    uint4 v = make_uint4(0, 0, 0, 0);
    bf16* e = (bf16*)&v;
#pragma unroll
    for (int i = 0; i < 8; ++i) e[i] = c + i < n ? src[c + i] : __float2bfloat16_rn(0.f);
    return v;
}

}  // namespace
