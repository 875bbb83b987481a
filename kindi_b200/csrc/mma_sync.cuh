// Warp-level tensor-core pieces shared by kernels whose tiles are too small for a tcgen05 accumulator: ldmatrix, the
// bf16 m16n8k16 product with 32-bit accumulation, and the splitting of 32-bit operands into sums of bf16 numbers.
#pragma once
#include "common.cuh"

__device__ __forceinline__ void ldsm_x4(uint32_t addr, uint32_t& r0, uint32_t& r1, uint32_t& r2, uint32_t& r3) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
                 : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(addr));
}
__device__ __forceinline__ void ldsm_x4_t(uint32_t addr, uint32_t& r0, uint32_t& r1, uint32_t& r2, uint32_t& r3) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
                 : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(addr));
}
__device__ __forceinline__ void mma_bf16(float* c, const uint32_t* a, uint32_t b0, uint32_t b1) {
    asm volatile(
        "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, "
        "{%0, %1, %2, %3};"
        : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
        : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint32_t pack_bf16(float lo, float hi) {
    __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
    return *(uint32_t*)&v;
}

// 16 bytes from global to shared memory without a register in between; ok == false: zeros
__device__ __forceinline__ void cp_async16(uint32_t dst, const void* src, bool ok) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(ok ? 16 : 0) : "memory");
}
__device__ __forceinline__ void cp_async_wait_all() { asm volatile("cp.async.wait_all;" ::: "memory"); }

// x = s[0] + s[1] + s[2] up to 2^-24 of x: a product with a 32-bit operand is the sum of three bf16 products
#define KB_SPLIT 3
__device__ __forceinline__ void split_bf16(float x, bf16 (&s)[KB_SPLIT]) {
#pragma unroll
    for (int i = 0; i < KB_SPLIT; i++) {
        s[i] = __float2bfloat16_rn(x);
        x -= __bfloat162float(s[i]);
    }
}
// the same for a pair of neighbours in one 32-bit register (the lower one in the lower half)
__device__ __forceinline__ void split_pack_bf16(float x, float y, uint32_t (&s)[KB_SPLIT]) {
#pragma unroll
    for (int i = 0; i < KB_SPLIT; i++) {
        const __nv_bfloat162 v = __floats2bfloat162_rn(x, y);
        s[i] = *(const uint32_t*)&v;
        x -= __low2float(v);
        y -= __high2float(v);
    }
}
