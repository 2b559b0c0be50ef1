// Element access shared by the kernels that exist for bf16 and for fp32 activations.
#pragma once
#include "decode.cuh"

namespace spark {

__device__ __forceinline__ float ldf(const float* p) { return *p; }
__device__ __forceinline__ float ldf(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void stf(float* p, float v) { *p = v; }
__device__ __forceinline__ void stf(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }

// four consecutive elements (16-byte / 8-byte aligned)
__device__ __forceinline__ float4 ldf4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 ldf4(const __nv_bfloat16* p) {
  const uint2 u = *reinterpret_cast<const uint2*>(p);
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.x));
  const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.y));
  return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void stf4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void stf4(__nv_bfloat16* p, float4 v) {
  const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
  *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
}

__device__ __forceinline__ float sigmoid_f(float x) { return 1.f / (1.f + expf(-x)); }
__device__ __forceinline__ float silu_f(float x) { return x / (1.f + expf(-x)); }
// Activations that are rounded to bf16 next: hardware exponential and reciprocal (relative error of a few 2^-22).
template <typename T> __device__ __forceinline__ float sigmoid_t(float x) {
  return sizeof(T) == 2 ? __fdividef(1.f, 1.f + __expf(-x)) : sigmoid_f(x);
}
template <typename T> __device__ __forceinline__ float silu_t(float x) {
  return sizeof(T) == 2 ? __fdividef(x, 1.f + __expf(-x)) : silu_f(x);
}
__device__ __forceinline__ float gelu_tanh_f(float z) {
  return 0.5f * z * (1.f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
}

// gelu_tanh(z) = z * sigmoid(2 sqrt(2/pi) (z + 0.044715 z^3))
template <typename T> __device__ __forceinline__ float gelu_tanh_t(float z) {
  return sizeof(T) == 2 ? __fdividef(z, 1.f + __expf(-1.5957691216057308f * (z + 0.044715f * z * z * z))) : gelu_tanh_f(z);
}

// ln(sigmoid(x)) / tau, bounded where the decay sigmoid(x)^(1 / tau) is 0 in fp32
__device__ __forceinline__ float log_sigmoid_decay(float x, float inv_tau) {
  return fmaxf((fminf(x, 0.f) - log1pf(expf(-fabsf(x)))) * inv_tau, -105.f);
}

// Sum over the block in a fixed order; every thread gets the same bits.  sh: >= 32 floats.
__device__ __forceinline__ float block_sum_all(float v, float* sh) {
  v = warp_sum(v);
  const int w = threadIdx.x >> 5, nw = blockDim.x >> 5;
  if ((threadIdx.x & 31) == 0) sh[w] = v;
  __syncthreads();
  float t = 0.f;
  for (int i = 0; i < nw; ++i) t += sh[i];
  __syncthreads();
  return t;
}

}  // namespace spark
