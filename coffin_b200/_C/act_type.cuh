// Storage types of activations: the same kernel source serves the bf16 serving mode and the fp32 mode.
#pragma once
#include "common.cuh"

template <typename T> __device__ __forceinline__ float act_load(const T* p);
template <> __device__ __forceinline__ float act_load<float>(const float* p) { return *p; }
template <> __device__ __forceinline__ float act_load<bf16>(const bf16* p) { return __bfloat162float(*p); }
template <typename T> __device__ __forceinline__ void act_store(T* p, float v);
template <> __device__ __forceinline__ void act_store<float>(float* p, float v) { *p = v; }
template <> __device__ __forceinline__ void act_store<bf16>(bf16* p, float v) { *p = __float2bfloat16(v); }
// the value as the storage type holds it
template <typename T> __device__ __forceinline__ float act_round(float v);
template <> __device__ __forceinline__ float act_round<float>(float v) { return v; }
template <> __device__ __forceinline__ float act_round<bf16>(float v) { return __bfloat162float(__float2bfloat16(v)); }
// four consecutive values (16-byte / 8-byte aligned)
__device__ __forceinline__ float4 act_load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 act_load4(const bf16* p) {
  const uint2 v = *reinterpret_cast<const uint2*>(p);
  return make_float4(__uint_as_float(v.x << 16), __uint_as_float(v.x & 0xffff0000u), __uint_as_float(v.y << 16),
                     __uint_as_float(v.y & 0xffff0000u));
}
__device__ __forceinline__ void act_store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void act_store4(bf16* p, float4 v) {
  *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf162(v.x, v.y), pack_bf162(v.z, v.w));
}
// full-precision forms (the ones in common.cuh use the fast intrinsics)
__device__ __forceinline__ float sigmoid_x(float x) { return 1.f / (1.f + expf(-x)); }
__device__ __forceinline__ float silu_x(float x) { return x * sigmoid_x(x); }
__device__ __forceinline__ float softplus_x(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }

// log(1 + exp(x)) to fp32 relative accuracy everywhere (decays near one need small values right, not just absolutely):
// log1p(e) = 2 atanh(e / (2 + e)) by the series of the inverse hyperbolic tangent, argument at most 1/3.
__device__ __forceinline__ float softplus_s(float x) {
  const float e = __expf(-fabsf(x)), s = __fdividef(e, 2.f + e), q = s * s;
  float p = 1.f / 13.f;
  p = fmaf(p, q, 1.f / 11.f); p = fmaf(p, q, 1.f / 9.f); p = fmaf(p, q, 1.f / 7.f);
  p = fmaf(p, q, 0.2f); p = fmaf(p, q, 1.f / 3.f); p = fmaf(p, q, 1.f);
  return fmaxf(x, 0.f) + 2.f * s * p;
}
// xIELU: a z^2 + z / 2 for z > 0, b (exp(z) - 1 - z) + z / 2 otherwise (_x: full precision)
__device__ __forceinline__ float xielu_s(float z, float a, float b) {
  return fmaf(0.5f, z, z > 0.f ? a * z * z : b * (__expf(fminf(z, 0.f)) - 1.f - z));
}
__device__ __forceinline__ float xielu_x(float z, float a, float b) {
  return fmaf(0.5f, z, z > 0.f ? a * z * z : b * (expm1f(fminf(z, 0.f)) - z));
}
__device__ __forceinline__ float relu2(float z) { z = fmaxf(z, 0.f); return z * z; }
// epilogue activations of the products: 1 xIELU with its coefficients, 2 squared relu
__device__ __forceinline__ float epi_act(int act, float z, float a, float b) { return act == 2 ? relu2(z) : xielu_s(z, a, b); }
__device__ __forceinline__ float sigmoid_s(float x) { return __fdividef(1.f, 1.f + __expf(-x)); }
__device__ __forceinline__ float silu_s(float x) { return x * sigmoid_s(x); }
