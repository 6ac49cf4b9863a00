// Behind a layer whose two sublayers read one norm of the fp32 residual side by side, in one launch:
//   X_(i+1) = x + sigmoid(g1 + b1) y1 + sigmoid(g2 + b2) (sum of y2's rows + y2_b)
//   x'      = sum_{j <= i + 1} coef[j] X_j                 (X_0: the embedding output, X_(j+1): the result of layer j)
//   h       = x' / sqrt(mean(x'^2) + eps) * (w_offset + w)
// Gates, the second sublayer and the depth average are optional (without the average x' = X_(i+1)). X_0 .. X_i and x come from
// launches further back, so their weighted sum is formed ahead of the wait for the sublayer in front of this launch: of a
// decode step only the last term is left behind it. One CTA per token; x' waits in shared memory for the norm.
#include "act_type.cuh"
#include "common.cuh"
#include "layers.h"

namespace lb {
namespace {

template <typename T>
__device__ __forceinline__ float open_of(float z) {
  if constexpr (sizeof(T) == 2) return __fdividef(1.f, 1.f + __expf(-z));
  else return sigmoid_f(z);
}

template <typename T, int VEC>
__global__ void __launch_bounds__(512) depth_step_kernel(const DepthStepArgs a) {
  extern __shared__ __align__(16) float sm[];      // x' [H] | x [H]
  __shared__ float red[16];
  const int H = a.H, nt = blockDim.x;
  float* u_s = sm;
  float* x_s = sm + H;
  const long t = a.rows ? a.rows[blockIdx.x] : long(blockIdx.x);
  const float* xr = a.x + t * H;
  const float* hist = a.hist ? a.hist + t * H : nullptr;
  for (int d = threadIdx.x * VEC; d < H; d += nt * VEC) {
    float xv[VEC], acc[VEC];
    ld_vec<VEC>(xr + d, xv);
#pragma unroll
    for (int j = 0; j < VEC; ++j) acc[j] = 0.f;
    if (hist) {
      int k = 0;
      for (; k + 4 <= a.n_hist; k += 4) {
        float v[4][VEC];
#pragma unroll
        for (int i = 0; i < 4; ++i) ld_vec<VEC>(hist + (k + i) * a.hist_stride + d, v[i]);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const float c = a.coef[k + i];
#pragma unroll
          for (int j = 0; j < VEC; ++j) acc[j] = fmaf(c, v[i][j], acc[j]);
        }
      }
      for (; k < a.n_hist; ++k) {
        float v[VEC];
        ld_vec<VEC>(hist + k * a.hist_stride + d, v);
        const float c = a.coef[k];
#pragma unroll
        for (int j = 0; j < VEC; ++j) acc[j] = fmaf(c, v[j], acc[j]);
      }
    }
    st_vec<VEC>(x_s + d, xv);
    st_vec<VEC>(u_s + d, acc);
  }
  const float last = hist ? a.coef[a.n_hist] : 1.f;
  griddep_wait();
  griddep_launch();
  const T* y1 = static_cast<const T*>(a.y1) + t * a.ldy1;
  const T* y2 = a.y2 ? static_cast<const T*>(a.y2) + t * a.y2_rows * a.ldy2 : nullptr;
  const T* g1 = a.g1 ? static_cast<const T*>(a.g1) + t * a.ldg : nullptr;
  const T* g2 = a.g2 ? static_cast<const T*>(a.g2) + t * a.ldg : nullptr;
  float ss = 0.f;
  for (int d = threadIdx.x * VEC; d < H; d += nt * VEC) {       // (a thread's own columns in both loops)
    float v[VEC], y[VEC], f[VEC], g[VEC];
    ld_vec<VEC>(y1 + d, y);
    if (y2) {
      ld_vec<VEC>(y2 + d, f);
      for (int r = 1; r < a.y2_rows; ++r) {
        float fr[VEC];
        ld_vec<VEC>(y2 + r * a.ldy2 + d, fr);
#pragma unroll
        for (int j = 0; j < VEC; ++j) f[j] += fr[j];
      }
      if (a.y2_b) {
#pragma unroll
        for (int j = 0; j < VEC; ++j) f[j] += a.y2_b[d + j];
      }
    }
    if (g1) {
      ld_vec<VEC>(g1 + d, g);
#pragma unroll
      for (int j = 0; j < VEC; ++j) y[j] *= open_of<T>(g[j] + a.b1[d + j]);
    }
    if (g2) {
      ld_vec<VEC>(g2 + d, g);
#pragma unroll
      for (int j = 0; j < VEC; ++j) f[j] *= open_of<T>(g[j] + a.b2[d + j]);
    }
#pragma unroll
    for (int j = 0; j < VEC; ++j) {
      v[j] = x_s[d + j] + y[j];
      if (y2) v[j] += f[j];
    }
    if (a.hist_out) st_vec<VEC>(a.hist_out + t * H + d, v);
    float u[VEC];
#pragma unroll
    for (int j = 0; j < VEC; ++j) {
      u[j] = fmaf(last, v[j], u_s[d + j]);
      ss = fmaf(u[j], u[j], ss);
    }
    st_vec<VEC>(u_s + d, u);
    st_vec<VEC>(a.x_out + long(blockIdx.x) * H + d, u);
  }
  ss = warp_sum_f(ss);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
  __syncthreads();
  float tot = 0.f;
  for (int i = 0; i < nt / 32; ++i) tot += red[i];
  const float inv = 1.f / sqrtf(tot / float(H) + a.eps);
  T* hr = static_cast<T*>(a.h) + long(blockIdx.x) * a.ldh;
  for (int d = threadIdx.x * VEC; d < H; d += nt * VEC) {
    float v[VEC];
#pragma unroll
    for (int j = 0; j < VEC; ++j) v[j] = u_s[d + j] * inv * (a.w_offset + a.norm_w[d + j]);
    st_vec<VEC>(hr + d, v);
  }
}

template <typename T>
int launch_t(const DepthStepArgs& a, cudaStream_t s) {
  auto al = [](const void* p, size_t n) { return reinterpret_cast<uintptr_t>(p) % n == 0; };
  const size_t e = 4 * sizeof(T);
  const bool v4 = a.H % 4 == 0 && al(a.x, 16) && al(a.x_out, 16) && al(a.hist, 16) && al(a.hist_out, 16) && al(a.y1, e) &&
                  al(a.y2, e) && al(a.g1, e) && al(a.g2, e) && al(a.h, e) && a.ldy1 % 4 == 0 && a.ldy2 % 4 == 0 && a.ldg % 4 == 0 &&
                  a.ldh % 4 == 0;
  const int vec = v4 ? 4 : 1, top = a.n_rows <= 296 ? 512 : 256, smem = 2 * a.H * 4;
  int nt = 32;
  while (nt < top && nt * vec < a.H) nt *= 2;
  auto kfn = v4 ? depth_step_kernel<T, 4> : depth_step_kernel<T, 1>;
  if (smem > 200 * 1024) return 1;
  if (smem > 40 * 1024 && cudaFuncSetAttribute(kfn, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess) return 1;
  return launch_pdl(kfn, dim3(a.n_rows), dim3(nt), smem, s, a) != cudaSuccess;
}

}  // namespace

int depth_step_launch(const DepthStepArgs& a, bool f32, cudaStream_t s) {
  if (a.n_rows <= 0) return 0;
  if (a.H < 1 || a.y2_rows < 1 || (a.g1 && !a.b1) || (a.g2 && !a.b2) || (a.hist && (!a.coef || a.n_hist < 1))) return 1;
  return f32 ? launch_t<float>(a, s) : launch_t<__nv_bfloat16>(a, s);
}

}  // namespace lb
