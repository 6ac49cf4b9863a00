// Behind a layer whose two sublayers read one norm of the fp32 residual side by side, in one launch:
//   X_(i+1) = x + sigmoid(g1 + b1) y1 + sigmoid(g2 + b2) (sum of y2's rows + y2_b)
//   x'      = sum_{j <= i + 1} coef[j] X_j                 (X_0: the embedding output, X_(j+1): the result of layer j)
//   h       = x' / sqrt(mean(x'^2) + eps) * (w_offset + w)
// Gates, the second sublayer and the depth average are optional (without the average x' = X_(i+1)).
//
// The average would read every earlier result behind every layer. Instead one layer in four does, and on the same pass sums up,
// for the three layers behind it, what they need of X_0 .. X_(i+1); those add the one or two results since. (Rows read and
// written behind 24 layers: 192 instead of 372.) One CTA per token; x' waits in shared memory for the norm. In decode steps
// (EARLY) everything older than the sublayers in front of this launch, which comes from launches further back, is summed up
// ahead of the wait for them.
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

// sums over the earlier results: the next input's and, AHEAD > 0, those of the layers behind it
template <int VEC, int AHEAD>
__device__ __forceinline__ void earlier(const DepthStepArgs& a, const float* c_s, long off, float (&acc)[1 + AHEAD][VEC]) {
#pragma unroll
  for (int s = 0; s <= AHEAD; ++s)
#pragma unroll
    for (int j = 0; j < VEC; ++j) acc[s][j] = 0.f;
  if (a.part) ld_vec<VEC>(a.part + off, acc[0]);
  auto add = [&](int k, const float (&v)[VEC]) {
    float c[1 + AHEAD];
    ld_vec<1 + AHEAD>(c_s + k * (1 + AHEAD), c);
#pragma unroll
    for (int s = 0; s <= AHEAD; ++s)
#pragma unroll
      for (int j = 0; j < VEC; ++j) acc[s][j] = fmaf(c[s], v[j], acc[s][j]);
  };
  int k = 0;
  for (; k + 4 <= a.n_hist; k += 4) {
    float v[4][VEC];
#pragma unroll
    for (int i = 0; i < 4; ++i) ld_vec<VEC>(a.hist + (k + i) * a.hist_stride + off, v[i]);
#pragma unroll
    for (int i = 0; i < 4; ++i) add(k + i, v[i]);
  }
  for (; k < a.n_hist; ++k) {
    float v[VEC];
    ld_vec<VEC>(a.hist + k * a.hist_stride + off, v);
    add(k, v);
  }
}

template <typename T, int VEC, int AHEAD, bool EARLY>
__global__ void __launch_bounds__(512) depth_step_kernel(const DepthStepArgs a) {
  extern __shared__ __align__(16) float c_s[];     // coefficients [n_hist + 1][1 + AHEAD] | x' [H]; EARLY: and x, sums for the
                                                   // layers behind [H each]
  __shared__ float red[16];
  const int H = a.H, nt = blockDim.x;
  const long t = a.rows ? a.rows[blockIdx.x] : long(blockIdx.x);
  const bool average = a.coef != nullptr;
  float* sm = c_s + (a.n_hist + 4) / 4 * 4 * (1 + AHEAD);
  if (average) {
    for (int i = threadIdx.x; i < (a.n_hist + 1) * (1 + AHEAD); i += nt) {
      const int k = i / (1 + AHEAD), s = i % (1 + AHEAD);
      c_s[i] = s == 0 ? a.coef[k] : s <= a.n_ahead ? a.ahead_coef[s - 1][k] : 0.f;
    }
    __syncthreads();
  }
  if constexpr (EARLY) {
    for (int d = threadIdx.x * VEC; d < H; d += nt * VEC) {
      float xv[VEC], acc[1 + AHEAD][VEC];
      ld_vec<VEC>(a.x + t * H + d, xv);
      earlier<VEC, AHEAD>(a, c_s, t * H + d, acc);
      st_vec<VEC>(sm + H + d, xv);
      st_vec<VEC>(sm + d, acc[0]);
#pragma unroll
      for (int s = 1; s <= AHEAD; ++s) st_vec<VEC>(sm + (1 + s) * H + d, acc[s]);
    }
  }
  griddep_wait();
  griddep_launch();
  const T* y1 = static_cast<const T*>(a.y1) + t * a.ldy1;
  const T* y2 = a.y2 ? static_cast<const T*>(a.y2) + t * a.y2_rows * a.ldy2 : nullptr;
  const T* g1 = a.g1 ? static_cast<const T*>(a.g1) + t * a.ldg : nullptr;
  const T* g2 = a.g2 ? static_cast<const T*>(a.g2) + t * a.ldg : nullptr;
  const float* own = c_s + a.n_hist * (1 + AHEAD);
  const float last = average ? own[0] : 1.f;
  float ss = 0.f;
  for (int d = threadIdx.x * VEC; d < H; d += nt * VEC) {       // (a thread's own columns in both loops)
    float v[VEC], y[VEC], f[VEC], g[VEC], acc[1 + AHEAD][VEC];
    if constexpr (EARLY) {
      ld_vec<VEC>(sm + H + d, v);
      ld_vec<VEC>(sm + d, acc[0]);
#pragma unroll
      for (int s = 1; s <= AHEAD; ++s) ld_vec<VEC>(sm + (1 + s) * H + d, acc[s]);
    } else {
      ld_vec<VEC>(a.x + t * H + d, v);
      earlier<VEC, AHEAD>(a, c_s, t * H + d, acc);
    }
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
      v[j] += y[j];
      if (y2) v[j] += f[j];
    }
    if (a.hist_out) st_vec<VEC>(a.hist_out + t * H + d, v);
#pragma unroll
    for (int s = 1; s <= AHEAD; ++s) {
      if (s > a.n_ahead) break;
      const float c = own[s];
#pragma unroll
      for (int j = 0; j < VEC; ++j) acc[s][j] = fmaf(c, v[j], acc[s][j]);
      st_vec<VEC>(a.ahead_out + (s - 1) * a.hist_stride + t * H + d, acc[s]);
    }
#pragma unroll
    for (int j = 0; j < VEC; ++j) {
      v[j] = fmaf(last, v[j], acc[0][j]);
      ss = fmaf(v[j], v[j], ss);
    }
    st_vec<VEC>(sm + d, v);
    st_vec<VEC>(a.x_out + long(blockIdx.x) * H + d, v);
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
    ld_vec<VEC>(sm + d, v);
#pragma unroll
    for (int j = 0; j < VEC; ++j) v[j] = v[j] * inv * (a.w_offset + a.norm_w[d + j]);
    st_vec<VEC>(hr + d, v);
  }
}

template <typename T, int VEC, int AHEAD>
int launch_a(const DepthStepArgs& a, cudaStream_t s) {
  const bool few = a.n_rows <= 296, early = few && (3 + AHEAD) * a.H * 4 <= 200 * 1024;
  const int smem = ((early ? 2 + AHEAD : 1) * a.H + (a.n_hist + 4) / 4 * 4 * (1 + AHEAD)) * 4;
  int nt = 32;
  while (nt < (few ? 512 : 256) && nt * VEC < a.H) nt *= 2;
  auto kfn = early ? depth_step_kernel<T, VEC, AHEAD, true> : depth_step_kernel<T, VEC, AHEAD, false>;
  if (smem > 200 * 1024) return 1;
  if (smem > 40 * 1024 && cudaFuncSetAttribute(kfn, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess) return 1;
  return launch_pdl(kfn, dim3(a.n_rows), dim3(nt), smem, s, a) != cudaSuccess;
}

template <typename T>
int launch_t(const DepthStepArgs& a, cudaStream_t s) {
  auto al = [](const void* p, size_t n) { return reinterpret_cast<uintptr_t>(p) % n == 0; };
  const size_t e = 4 * sizeof(T);
  const bool v4 = a.H % 4 == 0 && al(a.x, 16) && al(a.x_out, 16) && al(a.hist, 16) && al(a.hist_out, 16) && al(a.part, 16) &&
                  al(a.ahead_out, 16) && al(a.y1, e) && al(a.y2, e) && al(a.g1, e) && al(a.g2, e) && al(a.h, e) &&
                  a.ldy1 % 4 == 0 && a.ldy2 % 4 == 0 && a.ldg % 4 == 0 && a.ldh % 4 == 0;
  if (a.n_ahead > 0) return v4 ? launch_a<T, 4, DEPTH_AHEAD>(a, s) : launch_a<T, 1, DEPTH_AHEAD>(a, s);
  return v4 ? launch_a<T, 4, 0>(a, s) : launch_a<T, 1, 0>(a, s);
}

}  // namespace

int depth_step_launch(const DepthStepArgs& a, bool f32, cudaStream_t s) {
  if (a.n_rows <= 0) return 0;
  if (a.H < 1 || a.y2_rows < 1 || (a.g1 && !a.b1) || (a.g2 && !a.b2) || a.n_hist < 0 || (a.n_hist > 0 && !a.hist) || a.n_ahead < 0 ||
      a.n_ahead > DEPTH_AHEAD || (a.n_ahead > 0 && !a.ahead_out) || (!a.coef && (a.n_hist || a.n_ahead || a.part)))
    return 1;
  return f32 ? launch_t<float>(a, s) : launch_t<__nv_bfloat16>(a, s);
}

}  // namespace lb
