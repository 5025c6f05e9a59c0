// Products of a float32 operand with a bfloat16 one on the tensor cores: the float32 operand goes as the sum of three bfloat16
// terms (8 + 8 + 8 of its 24 mantissa bits), each of which multiplies exactly, sums in float32.
#pragma once
#include "common.cuh"

namespace edgelm {

__device__ __forceinline__ uint32_t sp_smem(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }

__device__ __forceinline__ void sp_mma(float* c, uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void sp_ldmatrix_x4(uint32_t addr, uint32_t& r0, uint32_t& r1, uint32_t& r2, uint32_t& r3) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(addr));
}
__device__ __forceinline__ void sp_ldmatrix_x2(uint32_t addr, uint32_t& r0, uint32_t& r1) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0, %1}, [%2];" : "=r"(r0), "=r"(r1) : "r"(addr));
}
__device__ __forceinline__ void sp_ldmatrix_x4_trans(uint32_t addr, uint32_t& r0, uint32_t& r1, uint32_t& r2, uint32_t& r3) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(addr));
}
__device__ __forceinline__ void sp_cp16(uint32_t dst, const void* src, int src_bytes) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(src_bytes) : "memory");
}

// Two float32 values as three packed pairs of bfloat16 terms: x = t1 + t2 + t3 up to float32 rounding (each term the
// rounding of what the terms before left over; the remainders are exact in float32).
__device__ __forceinline__ void sp_split(float x, float y, uint32_t& t1, uint32_t& t2, uint32_t& t3) {
  const __nv_bfloat16 x1 = __float2bfloat16_rn(x), y1 = __float2bfloat16_rn(y);
  const float xr = x - __bfloat162float(x1), yr = y - __bfloat162float(y1);
  const __nv_bfloat16 x2 = __float2bfloat16_rn(xr), y2 = __float2bfloat16_rn(yr);
  const __nv_bfloat16 x3 = __float2bfloat16_rn(xr - __bfloat162float(x2)), y3 = __float2bfloat16_rn(yr - __bfloat162float(y2));
  const __nv_bfloat162 p1 = __halves2bfloat162(x1, y1), p2 = __halves2bfloat162(x2, y2), p3 = __halves2bfloat162(x3, y3);
  t1 = *reinterpret_cast<const uint32_t*>(&p1);
  t2 = *reinterpret_cast<const uint32_t*>(&p2);
  t3 = *reinterpret_cast<const uint32_t*>(&p3);
}

}  // namespace edgelm
