// Between a q | k | v projection and the attention scores, in one launch: bias, short causal convolution per channel with
// carried history, RMS norm of q and k (each head by itself, or the whole of q and of k at once), rotation, append of k and
// v to the paged cache. A CTA takes a few consecutive tokens of one sequence, so taps are read once for all of them and a
// norm over all heads stays inside it; q and k wait in shared memory in fp32 for their norms, v goes straight to its cell.
// Decode steps have a CTA per token with a thread per four columns and update the history here; prompts leave that to a
// second small launch, since other CTAs may still read the old one.
#include "act_type.cuh"
#include "common.cuh"
#include "layers.h"

namespace lb {
namespace {

constexpr int PROMPT_TOK = 8;

// TOK: most tokens of a CTA; VEC: columns per thread and turn; KC 0: any number of taps
template <typename T, int KC, int TOK, int VEC>
__global__ void __launch_bounds__(TOK == 1 ? 1024 : 256) qkv_conv_kernel(const QkvConvArgs a) {
  extern __shared__ float y_s[];                   // [tok][nq + nk]
  __shared__ float red[2][TOK][32];
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
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, n_warps = blockDim.x >> 5;
  const int taps = a.conv_w ? a.KC : 1, K1 = taps - 1;
  const bool update = a.write_state && a.max_len <= 1 && K1 > 0;
  const T* x = static_cast<const T*>(a.x);
  float* hist = K1 > 0 ? a.conv_state + long(a.state_slots[seq]) * K1 * C : nullptr;
  float sq[TOK], sk[TOK];
#pragma unroll
  for (int t = 0; t < TOK; ++t) sq[t] = sk[t] = 0.f;
  for (int c = threadIdx.x * VEC; c < C; c += blockDim.x * VEC) {
    float b[VEC], y[TOK][VEC];
#pragma unroll
    for (int j = 0; j < VEC; ++j) b[j] = 0.f;
    if (a.in_b) ld_vec<VEC>(a.in_b + c, b);
    if constexpr (KC > 0) {
      float u[KC - 1 + TOK][VEC], w[KC][VEC];
#pragma unroll
      for (int i = 0; i < KC - 1 + TOK; ++i) {
        const int s = t0 - (KC - 1) + i;
        if (i - (KC - 1) >= nt) {
#pragma unroll
          for (int j = 0; j < VEC; ++j) u[i][j] = 0.f;
        } else if (s >= s0) {
          ld_vec<VEC>(x + long(s) * a.ld + c, u[i]);
#pragma unroll
          for (int j = 0; j < VEC; ++j) u[i][j] += b[j];
        } else {
          ld_vec<VEC>(hist + long(K1 + (s - s0)) * C + c, u[i]);
        }
      }
#pragma unroll
      for (int k = 0; k < KC; ++k) {
        if (KC == 1 && !a.conv_w) {
#pragma unroll
          for (int j = 0; j < VEC; ++j) w[k][j] = 1.f;
        } else {
          ld_vec<VEC>(a.conv_w + long(k) * C + c, w[k]);
        }
      }
#pragma unroll
      for (int t = 0; t < TOK; ++t)
#pragma unroll
        for (int j = 0; j < VEC; ++j) {
          float v = 0.f;
#pragma unroll
          for (int k = 0; k < KC; ++k) v = fmaf(w[k][j], u[t + k][j], v);
          y[t][j] = v;
        }
      if (update) {
#pragma unroll
        for (int k = 0; k < KC - 1; ++k) st_vec<VEC>(hist + long(k) * C + c, u[k + 1]);     // one token: what is behind moves up
      }
    } else {
#pragma unroll
      for (int t = 0; t < TOK; ++t)
#pragma unroll
        for (int j = 0; j < VEC; ++j) {
          float v = 0.f;
          for (int k = 0; k < taps && t < nt; ++k) {
            const int s = t0 + t - K1 + k;
            v = fmaf(a.conv_w[long(k) * C + c + j],
                     s >= s0 ? ld_f(x + long(s) * a.ld + c + j) + b[j] : hist[long(K1 + (s - s0)) * C + c + j], v);
          }
          y[t][j] = v;
        }
      if (update) {
#pragma unroll
        for (int j = 0; j < VEC; ++j) {
          for (int k = 0; k + 1 < K1; ++k) hist[long(k) * C + c + j] = hist[long(k + 1) * C + c + j];
          hist[long(K1 - 1) * C + c + j] = ld_f(x + long(t0) * a.ld + c + j) + b[j];
        }
      }
    }
    // (q, k and v begin at multiples of VEC)
    if (c < N) {
#pragma unroll
      for (int t = 0; t < TOK; ++t)
        if (t < nt) {
          st_vec<VEC>(y_s + t * N + c, y[t]);
          float ss = 0.f;
#pragma unroll
          for (int j = 0; j < VEC; ++j) ss = fmaf(y[t][j], y[t][j], ss);
          if (c < nq) sq[t] += ss;
          else sk[t] += ss;
        }
    } else {
#pragma unroll
      for (int t = 0; t < TOK; ++t)
        if (t < nt) {
          const long cell = a.slots[t0 + t];
          if (cell >= 0) st_vec<VEC>(static_cast<T*>(a.v_cache) + cell * a.v_cell + (c - N), y[t]);
        }
    }
  }
  if (a.qw && a.norm_all) {
#pragma unroll
    for (int t = 0; t < TOK; ++t)
      if (t < nt) {
        const float q = warp_sum_f(sq[t]), k = warp_sum_f(sk[t]);
        if (lane == 0) { red[0][t][warp] = q; red[1][t][warp] = k; }
      }
  }
  __syncthreads();
  // a warp per (token, head); a lane takes PV neighbouring pairs
  constexpr int PV = VEC == 1 ? 1 : 2;
  const int heads = a.Hq + a.Hkv, half = a.rot / 2;
  for (int i = warp; i < nt * heads; i += n_warps) {
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
        ss = warp_sum_f(lane < n_warps ? red[is_q ? 0 : 1][t][lane] : 0.f);
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
    if (PV == 2 && a.rot_half && half % 2 == 0) {
      auto two = [&](int d, float (&o)[2]) {
        const float2 f = *reinterpret_cast<const float2*>(v + d);
        o[0] = f.x * inv;
        o[1] = f.y * inv;
        if (nw) {
          o[0] *= nw[d];
          o[1] *= nw[d + 1];
        }
      };
      auto put = [&](int d, float p, float q) {
        if constexpr (sizeof(T) == 2) *reinterpret_cast<uint32_t*>(dst + d) = pack_bf16x2(p, q);
        else *reinterpret_cast<float2*>(dst + d) = make_float2(p, q);
      };
      for (int p = 2 * lane; p < half; p += 64) {
        float f[2], g[2];
        two(p, f);
        two(p + half, g);
        const float2 c = *reinterpret_cast<const float2*>(cs + p), s = *reinterpret_cast<const float2*>(cs + half + p);
        put(p, f[0] * c.x - g[0] * s.x, f[1] * c.y - g[1] * s.y);
        put(p + half, g[0] * c.x + f[0] * s.x, g[1] * c.y + f[1] * s.y);
      }
      for (int d = 2 * half + 2 * lane; d < a.DK; d += 64) {
        float f[2];
        two(d, f);
        put(d, f[0], f[1]);
      }
      continue;
    }
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
  float* st = a.conv_state + long(a.state_slots[seq]) * K1 * C + c;
  const float b = a.in_b ? a.in_b[c] : 0.f;
  for (int j = 0; j < K1; ++j) {           // position j takes what was behind it: never read after written
    const int s = t1 - K1 + j;
    st[long(j) * C] = s >= t0 ? ld_f(static_cast<const T*>(a.x) + long(s) * a.ld + c) + b : st[long(K1 + (s - t0)) * C];
  }
}

template <typename T, int TOK, int VEC>
int launch_v(const QkvConvArgs& a, cudaStream_t s) {
  const int taps = a.conv_w ? a.KC : 1, C = (a.Hq + a.Hkv) * a.DK + a.Hkv * a.DV;
  const int smem = (a.Hq + a.Hkv) * a.DK * 4 * a.tok;
  const dim3 grid(a.one ? a.n_seqs : a.T / a.tok + a.n_seqs);
  const int nt = TOK == 1 ? min(1024, max(64, (C / VEC + 31) / 32 * 32)) : 256;
#define LB_KC(K_)                                                                                                            \
  {                                                                                                                          \
    auto kfn = qkv_conv_kernel<T, K_, TOK, VEC>;                                                                             \
    if (smem > 40 * 1024 && cudaFuncSetAttribute(kfn, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess) return 1; \
    return launch_pdl(kfn, grid, dim3(nt), smem, s, a) != cudaSuccess;                                                       \
  }
  if (taps == 1) LB_KC(1)
  if (taps == 2) LB_KC(2)
  if (taps == 3) LB_KC(3)
  if (taps == 4) LB_KC(4)
  LB_KC(0)
#undef LB_KC
}

template <typename T>
int launch_t(const QkvConvArgs& a, cudaStream_t s) {
  auto al = [](const void* p, size_t n) { return reinterpret_cast<uintptr_t>(p) % n == 0; };
  const bool vec = a.DK % 4 == 0 && a.DV % 4 == 0 && a.ld % 4 == 0 && al(a.x, 4 * sizeof(T)) && al(a.in_b, 16) && al(a.conv_w, 16) &&
                   al(a.conv_state, 16) && al(a.v_cache, 4 * sizeof(T)) && al(a.k_cache, 8) && al(a.q_out, 8) && al(a.cos_sin, 8);
  const int rc = a.tok == 1 ? (vec ? launch_v<T, 1, 4>(a, s) : launch_v<T, 1, 1>(a, s))
                            : (vec ? launch_v<T, PROMPT_TOK, 4>(a, s) : launch_v<T, PROMPT_TOK, 1>(a, s));
  if (rc) return rc;
  if (a.write_state && a.conv_w && a.KC > 1 && a.max_len > 1) {
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
  a.tok = a.max_len <= 1 ? 1 : PROMPT_TOK;
  a.one = a.max_len <= 1 && a.T == a.n_seqs;
  while (a.tok > 1 && row * a.tok > 96 * 1024) a.tok /= 2;
  return f32 ? launch_t<float>(a, s) : launch_t<__nv_bfloat16>(a, s);
}

}  // namespace lb
