// Between a q | k | v projection and the attention scores, in one launch: bias, short causal convolution per channel with
// carried history, RMS norm of q and k (each head by itself, or the whole of q and of k at once), rotation, append of k and
// v to the paged cache. A CTA takes a few consecutive tokens of one sequence, so taps are read once for all of them and a
// norm over all heads stays inside it; q and k wait in shared memory in fp32 for their norms, v goes straight to its cell.
// Decode steps have a CTA per token with a thread per four columns and update the history here; prompts leave that to a
// second small launch, since other CTAs may still read the old one. Rows that are only rotated (neighbouring columns) and
// appended have a form of their own: nothing passes between threads, so each takes eight columns of a token.
#include "act_type.cuh"
#include "common.cuh"
#include "layers.h"

namespace lb {
namespace {

constexpr int PROMPT_TOK = 4;

// TOK: most tokens of a CTA; VEC: columns per thread and turn; KC 0: any number of taps
template <typename T, int KC, int TOK, int VEC>
__global__ void __launch_bounds__(TOK == 1 ? 1024 : 256, TOK == 1 ? 1 : 4) qkv_conv_kernel(const QkvConvArgs a) {
  extern __shared__ __align__(16) float y_s[];     // [tok][nq + nk], then [tok][heads]
  __shared__ float red[2][TOK][32];
  const int nq = a.Hq * a.DK, nk = a.Hkv * a.DK, nv = a.Hkv * a.DV, C = nq + nk + nv, N = nq + nk;
  const int taps = a.conv_w ? a.KC : 1, K1 = taps - 1;
  // A step with one token per sequence: what the projection in front of this launch does not write is on its way before the
  // wait (bias, taps and history of the thread's first columns, the token's position and cell).
  constexpr bool EARLY = TOK == 1 && KC > 1;
  constexpr int EK = EARLY ? KC : 1;
  const bool early = EARLY && a.one;
  float eb[VEC], ew[EK][VEC], eh[EK][VEC];
  int pos1 = 0;
  long cell1 = -1;
  if constexpr (EARLY) {
    const int c = threadIdx.x * VEC;
    if (early && c < C) {
      const float* h = a.conv_state + long(a.state_slots[blockIdx.x]) * K1 * C + c;
#pragma unroll
      for (int j = 0; j < VEC; ++j) eb[j] = 0.f;
      if (a.in_b) ld_vec<VEC>(a.in_b + c, eb);
#pragma unroll
      for (int k = 0; k < KC; ++k) ld_vec<VEC>(a.conv_w + long(k) * C + c, ew[k]);
#pragma unroll
      for (int k = 0; k < KC - 1; ++k) ld_vec<VEC>(h + long(k) * C, eh[k]);
    }
    if (early) {
      const int t = a.cu[blockIdx.x];
      pos1 = a.positions[t];
      cell1 = a.slots[t];
    }
  }
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
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, n_warps = blockDim.x >> 5;
  if (TOK == 1 && !early) { pos1 = a.positions[t0]; cell1 = a.slots[t0]; }
  const bool update = a.write_state && a.max_len <= 1 && K1 > 0;
  const T* x = static_cast<const T*>(a.x);
  float* hist = K1 > 0 ? a.conv_state + long(a.state_slots[seq]) * K1 * C : nullptr;
  float sq[TOK], sk[TOK];
#pragma unroll
  for (int t = 0; t < TOK; ++t) sq[t] = sk[t] = 0.f;
  for (int c = threadIdx.x * VEC; c < C; c += blockDim.x * VEC) {
    const bool have = early && c == int(threadIdx.x) * VEC;
    float b[VEC], y[TOK][VEC];
#pragma unroll
    for (int j = 0; j < VEC; ++j) b[j] = have ? eb[j] : 0.f;
    if (a.in_b && !have) ld_vec<VEC>(a.in_b + c, b);
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
        } else if (have) {
#pragma unroll
          for (int j = 0; j < VEC; ++j) u[i][j] = eh[i < EK ? i : 0][j];
        } else {
          ld_vec<VEC>(hist + long(K1 + (s - s0)) * C + c, u[i]);
        }
      }
#pragma unroll
      for (int k = 0; k < KC; ++k) {
        if (KC == 1 && !a.conv_w) {
#pragma unroll
          for (int j = 0; j < VEC; ++j) w[k][j] = 1.f;
        } else if (have) {
#pragma unroll
          for (int j = 0; j < VEC; ++j) w[k][j] = ew[k < EK ? k : 0][j];
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
          const long cell = TOK == 1 ? cell1 : long(a.slots[t0 + t]);
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
  // 1 / root mean square per (token, head)
  const int heads = a.Hq + a.Hkv, half = a.rot / 2;
  float* inv_s = y_s + tok * N;                    // [tok][heads]
  float inv_q = 1.f, inv_k = 1.f;
  if (TOK == 1 && a.qw && a.norm_all) {            // every warp adds up for itself
    inv_q = 1.f / sqrtf(warp_sum_f(lane < n_warps ? red[0][0][lane] : 0.f) / float(nq) + a.eps);
    inv_k = 1.f / sqrtf(warp_sum_f(lane < n_warps ? red[1][0][lane] : 0.f) / float(nk) + a.eps);
  } else if (a.qw && a.norm_all) {
    for (int i = warp; i < 2 * nt; i += n_warps) {
      const int t = i >> 1, k = i & 1;
      const float ss = warp_sum_f(lane < n_warps ? red[k][t][lane] : 0.f);
      const float inv = 1.f / sqrtf(ss / float(k ? nk : nq) + a.eps);
      for (int h = (k ? a.Hq : 0) + lane; h < (k ? heads : a.Hq); h += 32) inv_s[t * heads + h] = inv;
    }
    __syncthreads();
  } else if (a.qw) {
    for (int i = warp; i < nt * heads; i += n_warps) {
      const float* v = y_s + (i / heads) * N + (i % heads) * a.DK;
      float ss = 0.f;
      for (int d = lane; d < a.DK; d += 32) ss = fmaf(v[d], v[d], ss);
      ss = warp_sum_f(ss);
      if (lane == 0) inv_s[i] = 1.f / sqrtf(ss / float(a.DK) + a.eps);
    }
    __syncthreads();
  }
  // norm and rotation: PV neighbouring pairs of columns per thread and turn (columns past the rotated ones pass in pairs too)
  constexpr int PV = VEC == 1 ? 1 : 2;
  const bool wide = PV == 2 && a.rot_half && half % 2 == 0;
  const int step = wide ? 2 : 1, odd = a.DK & 1;
  const int per = ((a.DK + odd) / 2) / step;       // turns per head
  auto item = [&](int i) {
    const int th = i / per, e = (i - th * per) * step, t = th / heads, h = th - t * heads;
    const bool is_q = h < a.Hq;
    T* dst;
    if (is_q) {
      dst = static_cast<T*>(a.q_out) + (long(t0 + t) * a.Hq + h) * a.DK;
    } else {
      const long cell = TOK == 1 ? cell1 : long(a.slots[t0 + t]);
      if (cell < 0) return;
      dst = static_cast<T*>(a.k_cache) + cell * a.k_cell + long(h - a.Hq) * a.DK;
    }
    const float* v = y_s + t * N + h * a.DK;
    const float* nw = is_q ? a.qw : a.kw;
    const float inv = !nw ? 1.f : TOK == 1 && a.norm_all ? (is_q ? inv_q : inv_k) : inv_s[t * heads + h];
    if (nw && a.norm_all) nw += (is_q ? h : h - a.Hq) * a.DK;
    const bool turn = e < half;
    // columns of the pair(s): rotated ones half a rotation (or one column) apart, the others side by side
    const int i0 = turn ? (a.rot_half ? e : 2 * e) : 2 * e, i1 = turn ? (a.rot_half ? e + half : 2 * e + 1) : 2 * e + step;
    if (wide) {
      float2 f = *reinterpret_cast<const float2*>(v + i0), g = *reinterpret_cast<const float2*>(v + i1);
      f.x *= inv; f.y *= inv; g.x *= inv; g.y *= inv;
      if (nw) {
        const float2 wf = *reinterpret_cast<const float2*>(nw + i0), wg = *reinterpret_cast<const float2*>(nw + i1);
        f.x *= wf.x; f.y *= wf.y; g.x *= wg.x; g.y *= wg.y;
      }
      if (turn) {
        const float* cs = a.cos_sin + long(TOK == 1 ? pos1 : a.positions[t0 + t]) * a.rot;
        const float2 c = *reinterpret_cast<const float2*>(cs + e), s = *reinterpret_cast<const float2*>(cs + half + e);
        const float2 p = make_float2(f.x * c.x - g.x * s.x, f.y * c.y - g.y * s.y);
        g = make_float2(g.x * c.x + f.x * s.x, g.y * c.y + f.y * s.y);
        f = p;
      }
      if constexpr (sizeof(T) == 2) {
        *reinterpret_cast<uint32_t*>(dst + i0) = pack_bf16x2(f.x, f.y);
        *reinterpret_cast<uint32_t*>(dst + i1) = pack_bf16x2(g.x, g.y);
      } else {
        *reinterpret_cast<float2*>(dst + i0) = f;
        *reinterpret_cast<float2*>(dst + i1) = g;
      }
      return;
    }
    float f = v[i0] * inv * (nw ? nw[i0] : 1.f), g = i1 < a.DK ? v[i1] * inv * (nw ? nw[i1] : 1.f) : 0.f;
    if (turn) {
      const float* cs = a.cos_sin + long(TOK == 1 ? pos1 : a.positions[t0 + t]) * a.rot;
      const float c = cs[e], s = cs[half + e], p = f * c - g * s;
      g = g * c + f * s;
      f = p;
    }
    st_f(dst + i0, f);
    if (i1 < a.DK) st_f(dst + i1, g);
  };
  const int total = nt * heads * per;
  int i = threadIdx.x;
  if constexpr (TOK > 1)
    for (; i + 3 * int(blockDim.x) < total; i += 4 * blockDim.x) {
#pragma unroll
      for (int u = 0; u < 4; ++u) item(i + u * blockDim.x);
    }
  for (; i < total; i += blockDim.x) item(i);
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

template <typename T>
__device__ __forceinline__ void ld8(const T* p, float (&v)[8]) {
  float a[4], b[4];
  if constexpr (sizeof(T) == 2) {
    const uint4 u = *reinterpret_cast<const uint4*>(p);
    const uint32_t w[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      v[2 * j] = __uint_as_float(w[j] << 16);
      v[2 * j + 1] = __uint_as_float(w[j] & 0xffff0000u);
    }
  } else {
    ld_f4(p, a);
    ld_f4(p + 4, b);
#pragma unroll
    for (int j = 0; j < 4; ++j) { v[j] = a[j]; v[4 + j] = b[j]; }
  }
}
template <typename T>
__device__ __forceinline__ void st8(T* p, const float (&v)[8]) {
  if constexpr (sizeof(T) == 2) {
    *reinterpret_cast<uint4*>(p) = make_uint4(pack_bf16x2(v[0], v[1]), pack_bf16x2(v[2], v[3]), pack_bf16x2(v[4], v[5]),
                                              pack_bf16x2(v[6], v[7]));
  } else {
    st_f4(p, {v[0], v[1], v[2], v[3]});
    st_f4(p + 4, {v[4], v[5], v[6], v[7]});
  }
}

template <typename T>
__global__ void __launch_bounds__(256) qkv_rotate_kernel(const QkvConvArgs a) {
  const int nq = a.Hq * a.DK, nk = a.Hkv * a.DK, per = (nq + nk + a.Hkv * a.DV) / 8;
  const long i = long(blockIdx.x) * 256 + threadIdx.x;
  if (i >= long(a.T) * per) return;
  const int t = int(i / per), c = int(i % per) * 8, d = c < nq + nk ? c % a.DK : a.rot;
  // positions, cells and the table are not written by the projection in front of this launch
  const long cell = c < nq ? 0 : a.slots[t];
  float cs[4], sn[4];
  const bool turn = d < a.rot;
  if (turn) {
    const float* row = a.cos_sin + long(a.positions[t]) * a.rot + d / 2;
    ld_f4(row, cs);
    ld_f4(row + a.rot / 2, sn);
  }
  griddep_wait();
  griddep_launch();
  if (cell < 0) return;
  float v[8];
  ld8(static_cast<const T*>(a.x) + t * a.ld + c, v);
  if (turn) {
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const float f = v[2 * j], g = v[2 * j + 1];
      v[2 * j] = f * cs[j] - g * sn[j];
      v[2 * j + 1] = g * cs[j] + f * sn[j];
    }
  }
  if (c < nq) st8(static_cast<T*>(a.q_out) + long(t) * nq + c, v);
  else if (c < nq + nk) st8(static_cast<T*>(a.k_cache) + cell * a.k_cell + (c - nq), v);
  else st8(static_cast<T*>(a.v_cache) + cell * a.v_cell + (c - nq - nk), v);
}

template <typename T, int TOK, int VEC>
int launch_v(const QkvConvArgs& a, cudaStream_t s) {
  const int taps = a.conv_w ? a.KC : 1, C = (a.Hq + a.Hkv) * a.DK + a.Hkv * a.DV;
  const int smem = (a.Hq + a.Hkv) * (a.DK + 1) * 4 * a.tok;
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
  if (!a.in_b && !a.conv_w && !a.qw && (a.rot == 0 || (!a.rot_half && al(a.cos_sin, 16))) && a.rot % 8 == 0 && a.DK % 8 == 0 &&
      a.DV % 8 == 0 && a.ld % 8 == 0 && al(a.x, 16) && al(a.q_out, 16) && al(a.k_cache, 16) && al(a.v_cache, 16)) {
    const long n = long(a.T) * (((a.Hq + a.Hkv) * a.DK + a.Hkv * a.DV) / 8);
    return launch_pdl(qkv_rotate_kernel<T>, dim3(unsigned((n + 255) / 256)), dim3(256), 0, s, a) != cudaSuccess;
  }
  const bool vec = a.DK % 4 == 0 && a.DV % 4 == 0 && a.ld % 4 == 0 && al(a.x, 4 * sizeof(T)) && al(a.in_b, 16) && al(a.conv_w, 16) &&
                   al(a.conv_state, 16) && al(a.v_cache, 4 * sizeof(T)) && al(a.k_cache, 8) && al(a.q_out, 8) && al(a.cos_sin, 8) && al(a.qw, 8) && al(a.kw, 8);
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
  const long row = long(a.Hq + a.Hkv) * (a.DK + 1) * 4;
  if (row > 200 * 1024) return 1;
  a.tok = a.max_len <= 1 ? 1 : PROMPT_TOK;
  a.one = a.max_len <= 1 && a.T == a.n_seqs;
  while (a.tok > 1 && row * a.tok > 96 * 1024) a.tok /= 2;
  return f32 ? launch_t<float>(a, s) : launch_t<__nv_bfloat16>(a, s);
}

}  // namespace lb
