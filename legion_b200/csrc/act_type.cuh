// Activation element types of the kernels that run in bf16 and in fp32: scalar and four-wide loads and stores.
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>

namespace lb {

__device__ __forceinline__ float ld_f(const float* p) { return *p; }
__device__ __forceinline__ float ld_f(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void st_f(float* p, float v) { *p = v; }
__device__ __forceinline__ void st_f(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }

__device__ __forceinline__ void ld_f4(const float* p, float (&v)[4]) {
  const float4 f = *reinterpret_cast<const float4*>(p);
  v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w;
}
__device__ __forceinline__ void ld_f4(const __nv_bfloat16* p, float (&v)[4]) {
  const uint2 u = *reinterpret_cast<const uint2*>(p);
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.x));
  const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.y));
  v[0] = a.x; v[1] = a.y; v[2] = b.x; v[3] = b.y;
}
__device__ __forceinline__ void st_f4(float* p, const float (&v)[4]) {
  *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
}
__device__ __forceinline__ void st_f4(__nv_bfloat16* p, const float (&v)[4]) {
  const __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
  uint2 u;
  u.x = *reinterpret_cast<const unsigned int*>(&a);
  u.y = *reinterpret_cast<const unsigned int*>(&b);
  *reinterpret_cast<uint2*>(p) = u;
}
// VEC = 4 or 1 elements at p
template <int VEC, typename T>
__device__ __forceinline__ void ld_vec(const T* p, float (&v)[VEC]) {
  if constexpr (VEC == 4) ld_f4(p, v);
  else v[0] = ld_f(p);
}
template <int VEC, typename T>
__device__ __forceinline__ void st_vec(T* p, const float (&v)[VEC]) {
  if constexpr (VEC == 4) st_f4(p, v);
  else st_f(p, v[0]);
}

__device__ __forceinline__ float silu_f(float z) { return z / (1.f + expf(-z)); }
__device__ __forceinline__ float sigmoid_f(float z) { return 1.f / (1.f + expf(-z)); }
__device__ __forceinline__ float softplus_f(float z) { return z > 20.f ? z : log1pf(expf(z)); }
__device__ __forceinline__ float gelu_tanh_f(float z) {
  return 0.5f * z * (1.f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
}
// a z^2 + z / 2 for z > 0, b (exp(z) - 1 - z) + z / 2 otherwise
__device__ __forceinline__ float xielu_f(float z, float a, float b) {
  return z > 0.f ? z * fmaf(a, z, 0.5f) : fmaf(b, expm1f(z) - z, 0.5f * z);
}
// The same for results that are rounded to bf16: exp(z) - 1 - z by its series where the difference would cancel
// (|error| < 2e-6 of it for z > -0.5), by the hardware exponential elsewhere.
__device__ __forceinline__ float xielu_fast(float z, float a, float b) {
  const float n = fminf(z, 0.f);
  const float series = n * n * fmaf(n, fmaf(n, fmaf(n, fmaf(n, fmaf(n, 1.f / 5040.f, 1.f / 720.f), 1.f / 120.f), 1.f / 24.f), 1.f / 6.f), 0.5f);
  const float e = n > -0.5f ? series : __expf(n) - 1.f - n;
  const float p = fmaxf(z, 0.f);
  return fmaf(a * p, p, fmaf(b, e, 0.5f * z));
}
__device__ __forceinline__ float warp_sum_f(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}

}  // namespace lb
