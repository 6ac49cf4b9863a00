// Scale and soft cap of logits in place: cap * tanh(x * scale / cap), fp32 (compiled without fast math).
#include "common.cuh"
#include "layers.h"

namespace lb {
namespace {

__global__ void __launch_bounds__(256) softcap_kernel(float* __restrict__ x, float scale, float cap, long n) {
  griddep_wait();
  griddep_launch();
  const long i = (long(blockIdx.x) * 256 + threadIdx.x) * 4;
  const float k = scale / cap;
  if (i + 4 <= n) {
    float4 v = *reinterpret_cast<float4*>(x + i);
    v.x = cap * tanhf(v.x * k); v.y = cap * tanhf(v.y * k); v.z = cap * tanhf(v.z * k); v.w = cap * tanhf(v.w * k);
    *reinterpret_cast<float4*>(x + i) = v;
  } else {
    for (long j = i; j < n; ++j) x[j] = cap * tanhf(x[j] * k);
  }
}

}  // namespace

int softcap_launch(float* x, float scale, float cap, long n, cudaStream_t s) {
  if (n <= 0) return 0;
  if (!(cap > 0.f) || reinterpret_cast<uintptr_t>(x) % 16) return 1;
  return launch_pdl(softcap_kernel, dim3(unsigned((n + 1023) / 1024)), dim3(256), 0, s, x, scale, cap, n) != cudaSuccess;
}

}  // namespace lb
