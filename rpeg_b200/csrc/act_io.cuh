// Vector loads and stores of activations that are stored either as bf16 or as fp32, always handed to the kernels as fp32.
#pragma once
#include "common.cuh"

namespace rpeg {

__device__ __forceinline__ float4 load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 load4(const __nv_bfloat16* p) {
  const uint2 v = *reinterpret_cast<const uint2*>(p);
  const float2 a = unpack_bf16x2(v.x), b = unpack_bf16x2(v.y);
  return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void store4(__nv_bfloat16* p, float4 v) {
  *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(v.x, v.y), pack_bf16x2(v.z, v.w));
}
__device__ __forceinline__ float2 load2(const float* p) { return *reinterpret_cast<const float2*>(p); }
__device__ __forceinline__ float2 load2(const __nv_bfloat16* p) { return unpack_bf16x2(*reinterpret_cast<const uint32_t*>(p)); }
__device__ __forceinline__ void store2(float* p, float a, float b) { *reinterpret_cast<float2*>(p) = make_float2(a, b); }
__device__ __forceinline__ void store2(__nv_bfloat16* p, float a, float b) { *reinterpret_cast<uint32_t*>(p) = pack_bf16x2(a, b); }
__device__ __forceinline__ float load1(const float* p) { return *p; }
__device__ __forceinline__ float load1(const __nv_bfloat16* p) { return __bfloat162float(*p); }

__device__ __forceinline__ float4 add4(float4 a, float4 b) { return make_float4(a.x + b.x, a.y + b.y, a.z + b.z, a.w + b.w); }

// Two fp32 numbers in one register pair, for the packed fp32 instructions.
__device__ __forceinline__ uint64_t pack2(float a, float b) {
  uint64_t r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
  return r;
}
__device__ __forceinline__ float2 unpack2(uint64_t v) {
  float2 r;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(r.x), "=f"(r.y) : "l"(v));
  return r;
}
__device__ __forceinline__ uint64_t fma2(uint64_t a, uint64_t b, uint64_t c) {
  uint64_t d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
  return d;
}
__device__ __forceinline__ uint64_t mul2(uint64_t a, uint64_t b) {
  uint64_t d;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}
__device__ __forceinline__ uint64_t add2(uint64_t a, uint64_t b) {
  uint64_t d;
  asm("add.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}

// Exact (erf) gelu.
__device__ __forceinline__ float gelu_erf(float z) { return 0.5f * z * (1.f + erff(z * 0.70710678118654752f)); }
__device__ __forceinline__ float sigmoidf(float z) { return 1.f / (1.f + __expf(-z)); }
// tanh to a few units in the last place (the compiler's fast-math tanhf is a 2^-11 approximation): Lambert's continued fraction
// z / (1 + z^2 / (3 + z^2 / (5 + z^2 / (7 + z^2 / 9)))) near zero, 1 - 2 / (e^2z + 1) where nothing cancels.
__device__ __forceinline__ float tanh_f32(float z) {
  const float a = fabsf(z), q = z * z;
  if (a < 0.55f) return z * (945.f + q * (105.f + q)) / (945.f + q * (420.f + 15.f * q));
  return copysignf(1.f - 2.f / (1.f + __expf(2.f * a)), z);
}

// What a feed-forward's first product is followed by. Gated: the product has twice the columns (gate rows of the weight, then up
// rows) and the result is silu(gate) * up.
enum { FF_NONE = 0, FF_GELU = 1, FF_SWIGLU = 2, FF_RELU2 = 3 };

template <int ACT>
__device__ __forceinline__ float ff_act(float z) {
  if constexpr (ACT == FF_GELU) return gelu_erf(z);
  if constexpr (ACT == FF_RELU2) { const float r = fmaxf(z, 0.f); return r * r; }
  return z;
}
__device__ __forceinline__ float silu_mul(float gate, float up) { return gate * sigmoidf(gate) * up; }

}  // namespace rpeg
