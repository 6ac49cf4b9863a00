// Hyper-connections with static weights: the residual is S fp32 streams per token. One launch per sublayer does
//   y    = c0 * sum_j y0[t * y_rows + j] + c1 * y1[t]            (the sublayer's output, up to two terms; several rows
//                                                                 of y0 per token: the weighted expert rows of a MoE)
//   X'_t = sum_s mix[s, t] X_s + out[t] * y                      (all streams at once from the old ones)
//   u    = sum_t in[t] X'_t,   h = u / sqrt(mean(u^2) + eps) * (w_offset + w)
// so the stream update, the next sublayer's input mix and its norm read and write the streams once. The first launch of
// a step starts from the embedding rows instead (X_s = embedding for every s), normed first where a model has that. One CTA
// per token; u is kept in shared memory between the sum of squares and the write of h. With one stream, no mix weights and
// y scaled, this is the pre-norm residual step x + m y; without y only the norm.
#include "act_type.cuh"
#include "common.cuh"
#include "layers.h"

namespace lb {
namespace {

template <typename T, int S, int VEC, bool START>
__global__ void __launch_bounds__(256) hyper_kernel(const HyperArgs a) {
  extern __shared__ float u_s[];
  __shared__ float red[8];
  __shared__ float mix_s[S * S], out_s[S], in_s[S];
  griddep_wait();
  griddep_launch();
  const int t = blockIdx.x;
  const int H = a.H, Sr = a.S, nt = blockDim.x;
  for (int i = threadIdx.x; i < S * S; i += nt) {
    const int f = i / S, to = i % S;
    mix_s[i] = (!START && f < Sr && to < Sr) ? (a.mix ? a.mix[f * Sr + to] : float(f == to)) : 0.f;
  }
  if (threadIdx.x < S) {
    out_s[threadIdx.x] = (!START && threadIdx.x < Sr) ? (a.out_w ? a.out_w[threadIdx.x] : 1.f) : 0.f;
    in_s[threadIdx.x] = threadIdx.x < Sr ? (a.in_w ? a.in_w[threadIdx.x] : 1.f) : 0.f;
  }
  __syncthreads();
  const T* er = nullptr;
  if (START) {
    long row = t;
    if (a.ids) {
      const int id = a.ids[t];
      row = (id < 0 || id >= a.vocab) ? 0 : id;
    }
    er = static_cast<const T*>(a.emb) + row * a.ld_emb;
  }
  const float* xi = START ? nullptr : a.x_in + long(t) * Sr * H;
  float* xo = a.x_out + long(t) * Sr * H;
  float ss = 0.f;
  float pre_inv = 1.f;
  if (START && a.pre_w) {
    float es = 0.f;
    for (int d = threadIdx.x * VEC; d < H; d += nt * VEC) {
      float e[VEC];
      ld_vec<VEC>(er + d, e);
#pragma unroll
      for (int j = 0; j < VEC; ++j) es = fmaf(e[j], e[j], es);
    }
    es = warp_sum_f(es);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = es;
    __syncthreads();
    es = 0.f;
    for (int i = 0; i < nt / 32; ++i) es += red[i];
    pre_inv = 1.f / sqrtf(es / float(H) + a.eps);
    __syncthreads();
  }
  for (int d = threadIdx.x * VEC; d < H; d += nt * VEC) {
    float xn[S][VEC];
    if constexpr (START) {
      float e[VEC];
      ld_vec<VEC>(er + d, e);
      if (a.pre_w) {
#pragma unroll
        for (int j = 0; j < VEC; ++j) e[j] = e[j] * pre_inv * (a.w_offset + a.pre_w[d + j]);
      }
#pragma unroll
      for (int s = 0; s < S; ++s)
#pragma unroll
        for (int j = 0; j < VEC; ++j) xn[s][j] = e[j];
    } else {
      float xv[S][VEC], y[VEC], y1[VEC];
#pragma unroll
      for (int s = 0; s < S; ++s)
        if (s < Sr) ld_vec<VEC>(xi + long(s) * H + d, xv[s]);
#pragma unroll
      for (int j = 0; j < VEC; ++j) y[j] = 0.f;
      if (a.y0) {
        const T* y0 = static_cast<const T*>(a.y0) + long(t) * a.y_rows * a.ldy0 + d;
        ld_vec<VEC>(y0, y);
        for (int r = 1; r < a.y_rows; ++r) {
          float yr[VEC];
          ld_vec<VEC>(y0 + r * a.ldy0, yr);
#pragma unroll
          for (int j = 0; j < VEC; ++j) y[j] += yr[j];
        }
#pragma unroll
        for (int j = 0; j < VEC; ++j) y[j] *= a.c0;
      }
      if (a.y1) {
        ld_vec<VEC>(static_cast<const T*>(a.y1) + long(t) * a.ldy1 + d, y1);
#pragma unroll
        for (int j = 0; j < VEC; ++j) y[j] = fmaf(a.c1, y1[j], y[j]);
      }
#pragma unroll
      for (int to = 0; to < S; ++to) {
#pragma unroll
        for (int j = 0; j < VEC; ++j) {
          float v = out_s[to] * y[j];
#pragma unroll
          for (int s = 0; s < S; ++s)
            if (s < Sr) v = fmaf(mix_s[s * S + to], xv[s][j], v);
          xn[to][j] = v;
        }
      }
    }
    float u[VEC];
#pragma unroll
    for (int j = 0; j < VEC; ++j) u[j] = 0.f;
#pragma unroll
    for (int s = 0; s < S; ++s) {
      if (s < Sr) {
        st_vec<VEC>(xo + long(s) * H + d, xn[s]);
#pragma unroll
        for (int j = 0; j < VEC; ++j) u[j] = fmaf(in_s[s], xn[s][j], u[j]);
      }
    }
#pragma unroll
    for (int j = 0; j < VEC; ++j) {
      ss = fmaf(u[j], u[j], ss);
      u_s[d + j] = u[j];
    }
    if (a.raw) st_vec<VEC>(static_cast<T*>(a.raw) + long(t) * a.ldraw + d, u);
  }
  if (!a.h) return;
  ss = warp_sum_f(ss);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
  __syncthreads();
  float tot = 0.f;
  for (int i = 0; i < nt / 32; ++i) tot += red[i];
  const float inv = 1.f / sqrtf(tot / float(H) + a.eps);
  T* hr = static_cast<T*>(a.h) + long(t) * a.ldh;
  for (int d = threadIdx.x * VEC; d < H; d += nt * VEC) {
    float v[VEC];
#pragma unroll
    for (int j = 0; j < VEC; ++j) v[j] = u_s[d + j] * inv * (a.w_offset + a.norm_w[d + j]);
    st_vec<VEC>(hr + d, v);
  }
}

template <typename T, int S, int VEC>
int launch_s(const HyperArgs& a, cudaStream_t s) {
  int nt = 256;
  while (nt > 32 && (nt / 2) * VEC >= a.H) nt /= 2;
  const int smem = a.H * 4;
  auto k0 = hyper_kernel<T, S, VEC, true>;
  auto k1 = hyper_kernel<T, S, VEC, false>;
  auto kfn = a.x_in ? k1 : k0;
  if (smem > 40 * 1024) {
    if (smem > 200 * 1024) return 1;
    if (cudaFuncSetAttribute(kfn, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess) return 1;
  }
  return launch_pdl(kfn, dim3(a.rows), dim3(nt), smem, s, a) != cudaSuccess;
}

bool vec4_ok(const HyperArgs& a, size_t es) {
  auto al = [&](const void* p, size_t n) { return p == nullptr || reinterpret_cast<uintptr_t>(p) % n == 0; };
  return a.H % 4 == 0 && al(a.x_in, 16) && al(a.x_out, 16) && al(a.emb, 4 * es) && al(a.y0, 4 * es) &&
         al(a.y1, 4 * es) && al(a.h, 4 * es) && al(a.raw, 4 * es) && a.ldraw % 4 == 0 && a.ld_emb % 4 == 0 && a.ldy0 % 4 == 0 && a.ldy1 % 4 == 0 && a.ldh % 4 == 0;
}

template <typename T>
int dispatch(const HyperArgs& a, cudaStream_t s) {
  const bool v = vec4_ok(a, sizeof(T));
#define LB_S(N)                                                             \
  if (a.S <= N) return v ? launch_s<T, N, 4>(a, s) : launch_s<T, N, 1>(a, s);
  LB_S(1) LB_S(2) LB_S(3) LB_S(4) LB_S(6) LB_S(8) LB_S(16)
#undef LB_S
  return 1;
}

}  // namespace

int hyper_launch(const HyperArgs& a, bool f32, cudaStream_t s) {
  if (a.rows <= 0) return 0;
  if (a.S < 1 || a.H < 1 || a.y_rows < 1) return 1;
  return f32 ? dispatch<float>(a, s) : dispatch<__nv_bfloat16>(a, s);
}

}  // namespace lb
