// Pieces of latent attention for any sizes, bf16 and fp32, around the attention over the cached rows (attn_mla_sm100.cu;
// attn_general.cu for fp32): cache rows and rotated query parts, the output gate, and the two fused launches of a decode
// step - queries into the latent space with the cache append, and split merge with value projection and gate.
#include "act_type.cuh"
#include "common.cuh"
#include "layers.h"

namespace lb {
namespace {

// Column i of a vector whose first `rot` columns turn in neighbouring pairs; cs: cos | sin of the token's position.
template <typename T>
__device__ __forceinline__ float rotated(const T* v, int i, const float* cs, int rot) {
  const float x = ld_f(v + i);
  if (i >= rot) return x;
  const float c = cs[i >> 1], s = cs[(rot >> 1) + (i >> 1)];
  return (i & 1) ? x * c + ld_f(v + i - 1) * s : x * c - ld_f(v + i + 1) * s;
}

// Norm of the latent and rotation of the shared key part of one token, to its cache cell (one CTA of 128 threads).
template <typename T>
__device__ __forceinline__ void append_row(const LatentPrepArgs& a, int t, float* red) {
  const T* row = static_cast<const T*>(a.kv) + t * a.ldkv;
  float ss = 0.f;
  for (int i = threadIdx.x; i < a.L; i += blockDim.x) {
    const float v = ld_f(row + i);
    ss = fmaf(v, v, ss);
  }
  ss = warp_sum_f(ss);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
  __syncthreads();
  const long slot = a.slots[t];
  if (slot < 0) return;
  float tot = 0.f;
  for (int i = 0; i < int(blockDim.x) / 32; ++i) tot += red[i];
  const float inv = 1.f / sqrtf(tot / float(a.L) + a.eps);
  T* dst = static_cast<T*>(a.cache) + slot * a.cell;
  for (int i = threadIdx.x; i < a.L; i += blockDim.x) st_f(dst + i, ld_f(row + i) * inv * a.norm_w[i]);
  const float* cs = a.cos_sin + long(a.positions[t]) * a.rot;
  for (int i = threadIdx.x; i < a.R; i += blockDim.x) st_f(dst + a.L + i, rotated(row + a.L, i, cs, a.rot));
}

template <typename T>
__global__ void __launch_bounds__(128) latent_prep_kernel(const LatentPrepArgs a) {
  __shared__ float red[4];
  griddep_wait();
  griddep_launch();
  const int t = blockIdx.x;
  append_row<T>(a, t, red);
  const float* cs = a.cos_sin + long(a.positions[t]) * a.rot;
  for (int i = threadIdx.x; i < a.heads * a.R; i += blockDim.x) {
    const int h = i / a.R, j = i % a.R;
    const T* q = static_cast<const T*>(a.q) + t * a.ldq + long(h) * (a.dim + a.R) + a.dim;
    st_f(static_cast<T*>(a.q_abs) + (long(t) * a.heads + h) * a.q_row + a.L + j, rotated(q, j, cs, a.rot));
  }
}

template <typename T, int VEC>
__global__ void __launch_bounds__(256) latent_gate_kernel(T* __restrict__ x, const T* __restrict__ gate, long ldg,
                                                          int per_head, int vdim, int N, long n) {
  griddep_wait();
  griddep_launch();
  const long i = (long(blockIdx.x) * 256 + threadIdx.x) * VEC;
  if (i >= n) return;
  const long t = i / N;
  const int c = int(i % N);
  float v[VEC], g[VEC];
  ld_vec<VEC>(x + i, v);
  if (per_head) {
    const float s = sigmoid_f(ld_f(gate + t * ldg + c / vdim));
#pragma unroll
    for (int j = 0; j < VEC; ++j) v[j] *= s;
  } else {
    ld_vec<VEC>(gate + t * ldg + c, g);
#pragma unroll
    for (int j = 0; j < VEC; ++j) v[j] *= sigmoid_f(g[j]);
  }
  st_vec<VEC>(x + i, v);
}

template <typename T>
int gate_t(void* x, const void* gate, long ldg, int per_head, int vdim, int N, int T_, cudaStream_t s) {
  const long n = long(T_) * N;
  const bool v = vdim % 4 == 0 && reinterpret_cast<uintptr_t>(x) % (4 * sizeof(T)) == 0 &&
                 (per_head || (ldg % 4 == 0 && reinterpret_cast<uintptr_t>(gate) % (4 * sizeof(T)) == 0));
  const int vec = v ? 4 : 1;
  const dim3 grid(unsigned((n / vec + 255) / 256));
  return (v ? launch_pdl(latent_gate_kernel<T, 4>, grid, dim3(256), 0, s, static_cast<T*>(x), static_cast<const T*>(gate), ldg,
                         per_head, vdim, N, n)
            : launch_pdl(latent_gate_kernel<T, 1>, grid, dim3(256), 0, s, static_cast<T*>(x), static_cast<const T*>(gate), ldg,
                         per_head, vdim, N, n)) != cudaSuccess;
}

}  // namespace

int latent_prep_launch(const LatentPrepArgs& a, bool f32, cudaStream_t s) {
  if (a.T <= 0) return 0;
  if (a.rot % 2 || a.rot > a.R) return 1;
  return (f32 ? launch_pdl(latent_prep_kernel<float>, dim3(a.T), dim3(128), 0, s, a)
              : launch_pdl(latent_prep_kernel<__nv_bfloat16>, dim3(a.T), dim3(128), 0, s, a)) != cudaSuccess;
}

int latent_gate_launch(void* x, const void* gate, long ldg, int per_head, int vdim, int N, int T, bool f32, cudaStream_t s) {
  if (T <= 0 || N <= 0) return 0;
  return f32 ? gate_t<float>(x, gate, ldg, per_head, vdim, N, T, s)
             : gate_t<__nv_bfloat16>(x, gate, ldg, per_head, vdim, N, T, s);
}

}  // namespace lb
