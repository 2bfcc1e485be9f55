// Building blocks of the decoding attention kernels (one query row per sequence, bf16): asynchronous 16-byte copies, the
// register-operand MMA, and packing of two fp32 values into one bf16 pair and back.
#pragma once
#include "common.cuh"

namespace {

__device__ __forceinline__ void dd_cp16(void* dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}
// on false: the destination is zero-filled and nothing is read
__device__ __forceinline__ void dd_cp16_zfill(void* dst, const void* src, bool on) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src),
               "r"(on ? 16 : 0)
               : "memory");
}
__device__ __forceinline__ void dd_mma(float (&c)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint32_t dd_pack(float lo, float hi) {
  uint32_t r;
  asm("cvt.rn.bf16x2.f32 %0, %1, %2;" : "=r"(r) : "f"(hi), "f"(lo));
  return r;
}
__device__ __forceinline__ float dd_lo(uint32_t v) { return __uint_as_float(v << 16); }
__device__ __forceinline__ float dd_hi(uint32_t v) { return __uint_as_float(v & 0xffff0000u); }

}  // namespace
