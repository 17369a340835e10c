// Shared device helpers: 16-bit activation packing, error word, launch counter.
#pragma once
#include <cuda_runtime.h>
#include <cuda_bf16.h>
#include <cuda_fp16.h>
#include <stdint.h>

#define ARCB_HEAD_DIM 64
#define ARCB_VOCAB 14
#define ARCB_ROPE_PX 10  // rotary pairs driven by x   (src/transformer.py:87-90 with head_dim 64)
#define ARCB_ROPE_PY 10  // rotary pairs driven by y
#define ARCB_ROPE_PZ 12  // rotary pairs driven by z

enum : int { TOK_START = 10, TOK_NEWLINE = 11, TOK_IOSEP = 12, TOK_END = 13 };

// Device error codes written (atomicCAS, first writer wins) to the engine's error word.
enum : int {
  ARCB_DEV_OK = 0,
  ARCB_DEV_WAIT_TIMEOUT_TMA = 1,   // a consumer gave up waiting for a TMA stage
  ARCB_DEV_WAIT_TIMEOUT_MMA = 2,   // the producer gave up waiting for a free stage
  ARCB_DEV_WAIT_TIMEOUT_ACC = 3,   // the epilogue gave up waiting for the accumulator
  ARCB_DEV_BAD_INDEX = 4,          // a cache slot / length was out of range and skipped
};

__device__ __forceinline__ void arcb_set_error(int* err, int code) {
  if (err) atomicCAS(err, 0, code);
}

// Word 1 of the error block counts 16-bit saturations: values the half format cannot hold that were
// clamped to +-65504 on their way into a GEMM operand (or a score that overflowed to infinity).
// It is a warning, not an error: the run continues, the host reads and clears the count.
__device__ __forceinline__ void arcb_count_saturation(int* err) {
  if (err) atomicAdd(err + 1, 1);
}

// ---- programmatic dependent launch (see launch.cuh for the protocol) ----
// Both are no-ops for a kernel that was launched without the attribute.
__device__ __forceinline__ void pdl_launch_dependents() { asm volatile("griddepcontrol.launch_dependents;" ::: "memory"); }
__device__ __forceinline__ void pdl_wait() { asm volatile("griddepcontrol.wait;" ::: "memory"); }

// ---- 16-bit activation formats -------------------------------------------
// act_f16 != 0: IEEE half (values clamped to the finite half range), else bfloat16.

__device__ __forceinline__ uint32_t pack2_act(float a, float b, int act_f16) {
  if (act_f16) {
    a = fminf(fmaxf(a, -65504.f), 65504.f);
    b = fminf(fmaxf(b, -65504.f), 65504.f);
    __half2 h = __floats2half2_rn(a, b);
    return *reinterpret_cast<uint32_t*>(&h);
  }
  __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
  return *reinterpret_cast<uint32_t*>(&h);
}

// pack2_act that also reports a clamp (half format only) in the saturation counter
__device__ __forceinline__ uint32_t pack2_act_chk(float a, float b, int act_f16, int* err) {
  if (act_f16 && fmaxf(fabsf(a), fabsf(b)) > 65504.f) arcb_count_saturation(err);
  return pack2_act(a, b, act_f16);
}

// pack2_act in one conversion (which clamps to the finite range); `amax` collects the largest magnitude for a
// saturation check by the caller
__device__ __forceinline__ uint32_t pack2_act_max(float a, float b, int act_f16, float& amax) {
  if (act_f16) {
    uint32_t d;
    asm("cvt.rn.satfinite.f16x2.f32 %0, %1, %2;" : "=r"(d) : "f"(b), "f"(a));
    amax = fmaxf(fmaxf(amax, fabsf(a)), fabsf(b));
    return d;
  }
  __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
  return *reinterpret_cast<uint32_t*>(&h);
}

__device__ __forceinline__ float2 unpack2_act(uint32_t v, int act_f16) {
  if (act_f16) {
    __half2 h = *reinterpret_cast<__half2*>(&v);
    return __half22float2(h);
  }
  float2 r;
  r.x = __uint_as_float(v << 16);
  r.y = __uint_as_float(v & 0xffff0000u);
  return r;
}

__device__ __forceinline__ float2 unpack2_bf16(uint32_t v) {
  float2 r;
  r.x = __uint_as_float(v << 16);
  r.y = __uint_as_float(v & 0xffff0000u);
  return r;
}

__device__ __forceinline__ uint32_t pack2_bf16(float a, float b) {
  __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
  return *reinterpret_cast<uint32_t*>(&h);
}

// ---- activation elements in any of the three formats (0 = bfloat16, 1 = IEEE half, 2 = fp32) ----
__host__ __device__ __forceinline__ int act_bytes(int fmt) { return fmt == 2 ? 4 : 2; }

__device__ __forceinline__ float4 ld_act4(const void* base, size_t idx, int fmt) {
  if (fmt == 2) return *reinterpret_cast<const float4*>(reinterpret_cast<const float*>(base) + idx);
  const uint2 r = *reinterpret_cast<const uint2*>(reinterpret_cast<const uint16_t*>(base) + idx);
  const float2 a = unpack2_act(r.x, fmt), b = unpack2_act(r.y, fmt);
  return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void st_act4(void* base, size_t idx, float4 v, int fmt) {
  if (fmt == 2) {
    *reinterpret_cast<float4*>(reinterpret_cast<float*>(base) + idx) = v;
  } else {
    uint2 r;
    r.x = pack2_act(v.x, v.y, fmt);
    r.y = pack2_act(v.z, v.w, fmt);
    *reinterpret_cast<uint2*>(reinterpret_cast<uint16_t*>(base) + idx) = r;
  }
}
__device__ __forceinline__ float ld_act(const void* base, size_t idx, int fmt) {
  if (fmt == 2) return reinterpret_cast<const float*>(base)[idx];
  if (fmt == 1) return __half2float(reinterpret_cast<const __half*>(base)[idx]);
  return __bfloat162float(reinterpret_cast<const __nv_bfloat16*>(base)[idx]);
}
__device__ __forceinline__ void st_act(void* base, size_t idx, float v, int fmt) {
  if (fmt == 2) reinterpret_cast<float*>(base)[idx] = v;
  else if (fmt == 1) reinterpret_cast<__half*>(base)[idx] = __float2half_rn(fminf(fmaxf(v, -65504.f), 65504.f));
  else reinterpret_cast<__nv_bfloat16*>(base)[idx] = __float2bfloat16_rn(v);
}

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}

// Streaming 16-byte load that does not allocate in L1 (data is read once).
__device__ __forceinline__ uint4 ldg_stream16(const void* p) {
  uint4 r;
  asm volatile("ld.global.nc.L1::no_allocate.v4.u32 {%0,%1,%2,%3}, [%4];"
               : "=r"(r.x), "=r"(r.y), "=r"(r.z), "=r"(r.w)
               : "l"(p));
  return r;
}
