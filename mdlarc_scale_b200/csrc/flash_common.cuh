// Device helpers shared by the tcgen05 prefill kernels.
#pragma once
#include "common.cuh"
#include "ptx_sm100.cuh"

namespace {

// MN-major operand tile [K rows of 128 bytes][64 elements], 128-byte swizzle: 8-row groups are
// 1024 bytes apart along K (stride byte offset); a single 64-element group along MN.
__device__ __forceinline__ uint64_t umma_desc_mn_sw128(uint32_t smem_addr) {
  uint64_t d = 0;
  d |= (uint64_t)((smem_addr & 0x3FFFFu) >> 4);
  d |= (uint64_t)(1024 >> 4) << 16;  // leading byte offset (next 64-element MN group; unused for N = 64)
  d |= (uint64_t)(1024 >> 4) << 32;  // stride byte offset (next group of 8 K rows)
  d |= (uint64_t)1 << 46;
  d |= (uint64_t)2 << 61;
  return d;
}

__device__ __forceinline__ uint32_t pack2_prob(float a, float b, int f16) {
  if (f16) {
    __half2 h = __floats2half2_rn(a, b);
    return *reinterpret_cast<uint32_t*>(&h);
  }
  __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
  return *reinterpret_cast<uint32_t*>(&h);
}

// 2^x on the special-function unit, one instruction (flushes denormals; inputs here are <= 0 or
// masked afterwards)
__device__ __forceinline__ float ex2_fast(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

__device__ __forceinline__ uint32_t h2_bits(__half2 v) { return *reinterpret_cast<uint32_t*>(&v); }
__device__ __forceinline__ __half2 h2_from_bits(uint32_t b) { return *reinterpret_cast<__half2*>(&b); }

// Re-division of the CTA's registers between warpgroups (all four warps of a warpgroup execute it)
__device__ __forceinline__ void reg_dealloc_24() { asm volatile("setmaxnreg.dec.sync.aligned.u32 24;"); }
__device__ __forceinline__ void reg_alloc_112() { asm volatile("setmaxnreg.inc.sync.aligned.u32 112;"); }

__device__ __forceinline__ float max3_f32(float a, float b, float c) {
  float d;
  asm("max.f32 %0, %1, %2, %3;" : "=f"(d) : "f"(a), "f"(b), "f"(c));
  return d;
}
__device__ __forceinline__ uint64_t pack_f32x2(float lo, float hi) {
  uint64_t d;
  asm("mov.b64 %0, {%1, %2};" : "=l"(d) : "f"(lo), "f"(hi));
  return d;
}
// (t0, t1) = (s0 * c + m, s1 * c + m) with one two-wide fp32 fused multiply-add
__device__ __forceinline__ void shift2_f32(uint32_t s0, uint32_t s1, uint64_t c2, uint64_t m2, float& t0, float& t1) {
  uint64_t sp, tp;
  asm("mov.b64 %0, {%1, %2};" : "=l"(sp) : "r"(s0), "r"(s1));
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(tp) : "l"(sp), "l"(c2), "l"(m2));
  asm("mov.b64 {%0, %1}, %2;" : "=f"(t0), "=f"(t1) : "l"(tp));
}

}  // namespace
