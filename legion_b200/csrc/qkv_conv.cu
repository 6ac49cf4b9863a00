// Between a q | k | v projection and the attention scores, in one launch: bias, short causal convolution per channel with
// carried history, RMS norm of q and k (each head by itself, or the whole of q and of k at once), rotation, append of k and
// v to the paged cache. A CTA takes a few consecutive tokens of one sequence, so taps are read once for all of them and a
// norm over all heads stays inside it; q and k wait in shared memory in fp32 for their norms, v goes straight to its cell.
// Decode steps update the history here (each sequence is one CTA); prompts leave that to a second small launch, since
// other CTAs may still read the old one.
#include "act_type.cuh"
#include "common.cuh"
#include "layers.h"

namespace lb {
namespace {

constexpr int MAXTOK = 8;

template <typename T, int KC>
__global__ void __launch_bounds__(256) qkv_conv_kernel(const QkvConvArgs a) {
  extern __shared__ float y_s[];                   // [tok][nq + nk]
  __shared__ float red[2][MAXTOK][8];
  griddep_wait();
  griddep_launch();
  const int tok = a.tok;
  int seq = 0, s0, s1, t0;
  if (a.one) {                                     // a token per sequence
    seq = blockIdx.x;
    t0 = s0 = a.cu[seq];
    s1 = a.cu[seq + 1];
  } else {                                         // sequence i begins at tile cu[i] / tok + i
    int z = a.n_seqs;
    while (z - seq > 1) {
      const int m = (seq + z) >> 1;
      if (a.cu[m] / tok + m <= int(blockIdx.x)) seq = m; else z = m;
    }
    s0 = a.cu[seq];
    s1 = a.cu[seq + 1];
    t0 = s0 + (int(blockIdx.x) - (s0 / tok + seq)) * tok;
  }
  if (t0 >= s1) return;
  const int nt = min(tok, s1 - t0);
  const int nq = a.Hq * a.DK, nk = a.Hkv * a.DK, nv = a.Hkv * a.DV, C = nq + nk + nv, N = nq + nk;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int taps = a.conv_w ? a.KC : 1, K1 = taps - 1;
  const bool update = a.write_state && a.max_len <= 1 && K1 > 0;
  const T* x = static_cast<const T*>(a.x);
  float sq[MAXTOK], sk[MAXTOK];
#pragma unroll
  for (int t = 0; t < MAXTOK; ++t) sq[t] = sk[t] = 0.f;
  for (int c = threadIdx.x; c < C; c += 256) {
    const float b = a.in_b ? a.in_b[c] : 0.f;
    float* st = K1 > 0 ? a.conv_state + (long(a.state_slots[seq]) * C + c) * K1 : nullptr;
    float y[MAXTOK];
    if constexpr (KC > 0) {
      float u[KC - 1 + MAXTOK];
#pragma unroll
      for (int i = 0; i < KC - 1 + MAXTOK; ++i) {
        const int s = t0 - (KC - 1) + i;
        u[i] = i - (KC - 1) >= nt ? 0.f : s >= s0 ? ld_f(x + long(s) * a.ld + c) + b : st[K1 + (s - s0)];
      }
      float w[KC];
#pragma unroll
      for (int j = 0; j < KC; ++j) w[j] = KC == 1 && !a.conv_w ? 1.f : a.conv_w[long(c) * KC + j];
#pragma unroll
      for (int t = 0; t < MAXTOK; ++t) {
        float v = 0.f;
#pragma unroll
        for (int j = 0; j < KC; ++j) v = fmaf(w[j], u[t + j], v);
        y[t] = v;
      }
      if (update) {
#pragma unroll
        for (int j = 0; j < KC - 1; ++j) st[j] = u[j + 1];     // one token: what is behind moves up
      }
    } else {
#pragma unroll
      for (int t = 0; t < MAXTOK; ++t) {
        float v = 0.f;
        for (int j = 0; j < taps && t < nt; ++j) {
          const int s = t0 + t - K1 + j;
          v = fmaf(a.conv_w[long(c) * taps + j], s >= s0 ? ld_f(x + long(s) * a.ld + c) + b : st[K1 + (s - s0)], v);
        }
        y[t] = v;
      }
      if (update) {
        for (int j = 0; j + 1 < K1; ++j) st[j] = st[j + 1];
        st[K1 - 1] = ld_f(x + long(t0) * a.ld + c) + b;
      }
    }
    if (c < N) {
#pragma unroll
      for (int t = 0; t < MAXTOK; ++t)
        if (t < nt) {
          y_s[t * N + c] = y[t];
          if (c < nq) sq[t] = fmaf(y[t], y[t], sq[t]);
          else sk[t] = fmaf(y[t], y[t], sk[t]);
        }
    } else {
#pragma unroll
      for (int t = 0; t < MAXTOK; ++t)
        if (t < nt) {
          const long cell = a.slots[t0 + t];
          if (cell >= 0) st_f(static_cast<T*>(a.v_cache) + cell * a.v_cell + (c - N), y[t]);
        }
    }
  }
  if (a.qw && a.norm_all) {
#pragma unroll
    for (int t = 0; t < MAXTOK; ++t)
      if (t < nt) {
        const float q = warp_sum_f(sq[t]), k = warp_sum_f(sk[t]);
        if (lane == 0) { red[0][t][warp] = q; red[1][t][warp] = k; }
      }
  }
  __syncthreads();
  // a warp per (token, head)
  const int heads = a.Hq + a.Hkv, half = a.rot / 2;
  for (int i = warp; i < nt * heads; i += 8) {
    const int t = i / heads, h = i % heads;
    const bool is_q = h < a.Hq;
    const float* v = y_s + t * N + h * a.DK;
    const float* nw = is_q ? a.qw : a.kw;
    float inv = 1.f;
    if (nw) {
      float ss = 0.f;
      int n = a.DK;
      if (a.norm_all) {
        n = is_q ? nq : nk;
#pragma unroll
        for (int w = 0; w < 8; ++w) ss += red[is_q ? 0 : 1][t][w];
        nw += (is_q ? h : h - a.Hq) * a.DK;
      } else {
        for (int d = lane; d < a.DK; d += 32) ss = fmaf(v[d], v[d], ss);
        ss = warp_sum_f(ss);
      }
      inv = 1.f / sqrtf(ss / float(n) + a.eps);
    }
    T* dst;
    if (is_q) {
      dst = static_cast<T*>(a.q_out) + (long(t0 + t) * a.Hq + h) * a.DK;
    } else {
      const long cell = a.slots[t0 + t];
      if (cell < 0) continue;
      dst = static_cast<T*>(a.k_cache) + cell * a.k_cell + long(h - a.Hq) * a.DK;
    }
    const float* cs = a.cos_sin ? a.cos_sin + long(a.positions[t0 + t]) * a.rot : nullptr;
    for (int p = lane; p < half; p += 32) {
      const int i0 = a.rot_half ? p : 2 * p, i1 = a.rot_half ? p + half : 2 * p + 1;
      const float f = v[i0] * inv * (nw ? nw[i0] : 1.f), g = v[i1] * inv * (nw ? nw[i1] : 1.f);
      const float c = cs[p], s = cs[half + p];
      st_f(dst + i0, f * c - g * s);
      st_f(dst + i1, g * c + f * s);
    }
    for (int d = 2 * half + lane; d < a.DK; d += 32) st_f(dst + d, v[d] * inv * (nw ? nw[d] : 1.f));
  }
}

template <typename T>
__global__ void __launch_bounds__(128) qkv_history_kernel(const QkvConvArgs a) {
  griddep_wait();
  griddep_launch();
  const int C = (a.Hq + a.Hkv) * a.DK + a.Hkv * a.DV, c = blockIdx.x * 128 + threadIdx.x, seq = blockIdx.y, K1 = a.KC - 1;
  if (c >= C) return;
  const int t0 = a.cu[seq], t1 = a.cu[seq + 1];
  if (t1 <= t0) return;
  float* st = a.conv_state + (long(a.state_slots[seq]) * C + c) * K1;
  const float b = a.in_b ? a.in_b[c] : 0.f;
  for (int j = 0; j < K1; ++j) {           // position j takes what was behind it: never read after written
    const int s = t1 - K1 + j;
    st[j] = s >= t0 ? ld_f(static_cast<const T*>(a.x) + long(s) * a.ld + c) + b : st[K1 + (s - t0)];
  }
}

template <typename T>
int launch_t(const QkvConvArgs& a, cudaStream_t s) {
  const int taps = a.conv_w ? a.KC : 1;
  const long row = long(a.Hq + a.Hkv) * a.DK * 4;
  const int smem = int(row * a.tok);
  const dim3 grid(a.one ? a.n_seqs : a.T / a.tok + a.n_seqs);
  int rc = 1;
#define LB_KC(K_)                                                                                                            \
  {                                                                                                                          \
    auto kfn = qkv_conv_kernel<T, K_>;                                                                                       \
    if (smem > 40 * 1024 && cudaFuncSetAttribute(kfn, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess) return 1; \
    rc = launch_pdl(kfn, grid, dim3(256), smem, s, a) != cudaSuccess;                                                        \
  }
  if (taps == 1) LB_KC(1)
  else if (taps == 2) LB_KC(2)
  else if (taps == 3) LB_KC(3)
  else if (taps == 4) LB_KC(4)
  else LB_KC(0)
#undef LB_KC
  if (rc) return rc;
  if (a.write_state && taps > 1 && a.max_len > 1) {
    const int C = (a.Hq + a.Hkv) * a.DK + a.Hkv * a.DV;
    return launch_pdl(qkv_history_kernel<T>, dim3((C + 127) / 128, a.n_seqs), dim3(128), 0, s, a) != cudaSuccess;
  }
  return 0;
}

}  // namespace

int qkv_conv_append_launch(QkvConvArgs a, bool f32, cudaStream_t s) {
  if (a.T <= 0 || a.n_seqs <= 0) return 0;
  if (a.Hkv <= 0 || a.Hq % a.Hkv || a.rot % 2 || a.rot > a.DK || a.rot < 0 || (a.conv_w && a.KC < 1) || a.n_seqs > 65535) return 1;
  const long row = long(a.Hq + a.Hkv) * a.DK * 4;
  if (row > 200 * 1024) return 1;
  a.tok = a.max_len <= 1 ? 1 : MAXTOK;
  a.one = a.max_len <= 1 && a.T == a.n_seqs;
  while (a.tok > 1 && row * a.tok > 96 * 1024) a.tok /= 2;
  return f32 ? launch_t<float>(a, s) : launch_t<__nv_bfloat16>(a, s);
}

}  // namespace lb
