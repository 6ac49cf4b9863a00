// Linear-attention state with a scalar decay per head, token by token:
//   S_t = a_t S_(t-1) + k_t v_t^T,   o_t = S_t^T q_t        (S: N x P, fp32, kept transposed as [P, N])
// Two forms share the kernels: a constant decay per head with silu on q, k and v (Lightning attention), and the
// selective form a_t = exp(dt_t A), v scaled by dt_t = softplus(raw + bias), skip D v and gate silu(z) (Mamba-2).
// Beside it: the one-launch decode step of a Mamba-2 mixer and the norms that follow the state (whole row or equal parts,
// optional sigmoid gate).
//
// The scan kernel owns 32 state rows (value columns) of one head per CTA: a warp holds four rows across its lanes, so
// a decode step streams the state once with 128-byte accesses, and a portion of several tokens keeps it in registers.
// Long portions run on the chunked tensor-core form (linear_scan_sm100.cu).
#include "act_type.cuh"
#include "common.cuh"
#include "layers.h"

namespace lb {
namespace {

constexpr int RPW = 4;                 // state rows per warp
constexpr int WARPS = 8;
constexpr int RPC = RPW * WARPS;       // rows per CTA

template <typename T, int NJ>
__global__ void __launch_bounds__(256) linear_scan_kernel(const LinScanArgs a) {
  griddep_wait();
  griddep_launch();
  const int pb = (a.P + RPC - 1) / RPC;
  const int h = blockIdx.x / pb, p0 = (blockIdx.x % pb) * RPC + (threadIdx.x >> 5) * RPW;
  const int seq = blockIdx.y, lane = threadIdx.x & 31;
  const int t0 = a.cu[seq], t1 = a.cu[seq + 1], slot = a.slots[seq];
  if (t1 <= t0 || slot < 0 || p0 >= a.P || (a.max_tokens > 0 && t1 - t0 > a.max_tokens)) return;
  const int N = a.N, g = h / (a.H / a.G);
  float* st = a.state + ((long(slot) * a.H + h) * a.P + p0) * N;
  float s[RPW][NJ];
#pragma unroll
  for (int r = 0; r < RPW; ++r)
#pragma unroll
    for (int j = 0; j < NJ; ++j) {
      const int n = lane + 32 * j;
      s[r][j] = (p0 + r < a.P && n < N) ? st[long(r) * N + n] : 0.f;
    }
  const T* qp = static_cast<const T*>(a.q) + long(g) * N;
  const T* kp = static_cast<const T*>(a.k) + long(g) * N;
  const T* vp = static_cast<const T*>(a.v) + long(h) * a.P + p0;
  const T* zp = a.z ? static_cast<const T*>(a.z) + long(h) * a.P + p0 : nullptr;
  const float dec_c = a.decay ? a.decay[h] : 0.f;
  const float Ah = a.decay ? 0.f : a.A[h], db = a.decay ? 0.f : a.dt_bias[h];
  const float Dh = a.D ? a.D[h] : 0.f;
  for (int t = t0; t < t1; ++t) {
    float dec = dec_c, dt = 1.f;
    if (!a.decay) {
      dt = softplus_f(ld_f(static_cast<const T*>(a.dt) + long(t) * a.lddt + h) + db);
      dec = expf(dt * Ah);
    }
    float q[NJ], k[NJ];
#pragma unroll
    for (int j = 0; j < NJ; ++j) {
      const int n = lane + 32 * j;
      q[j] = n < N ? ld_f(qp + long(t) * a.ldq + n) : 0.f;
      k[j] = n < N ? ld_f(kp + long(t) * a.ldk + n) : 0.f;
      if (a.silu_in) { q[j] = silu_f(q[j]); k[j] = silu_f(k[j]); }
    }
    float mine = 0.f, vmine = 0.f;
#pragma unroll
    for (int r = 0; r < RPW; ++r) {
      float v = p0 + r < a.P ? ld_f(vp + long(t) * a.ldv + r) : 0.f;
      if (a.silu_in) v = silu_f(v);
      const float vd = v * dt;
      float o = 0.f;
#pragma unroll
      for (int j = 0; j < NJ; ++j) {
        s[r][j] = fmaf(dec, s[r][j], vd * k[j]);
        o = fmaf(s[r][j], q[j], o);
      }
      o = warp_sum_f(o);
      if (lane == r) { mine = o; vmine = v; }
    }
    if (lane < RPW && p0 + lane < a.P) {
      float y = fmaf(Dh, vmine, mine);
      if (zp) y *= silu_f(ld_f(zp + long(t) * a.ldz + lane));
      st_f(static_cast<T*>(a.out) + long(t) * a.ldo + long(h) * a.P + p0 + lane, y);
    }
  }
  if (a.write_state) {
#pragma unroll
    for (int r = 0; r < RPW; ++r)
#pragma unroll
      for (int j = 0; j < NJ; ++j) {
        const int n = lane + 32 * j;
        if (p0 + r < a.P && n < N) st[long(r) * N + n] = s[r][j];
      }
  }
}

template <typename T>
int scan_t(const LinScanArgs& a, cudaStream_t s) {
  const dim3 grid(unsigned(a.H * ((a.P + RPC - 1) / RPC)), unsigned(a.n_seqs));
#define LB_NJ(NJ_) \
  if (a.N <= 32 * NJ_) return launch_pdl(linear_scan_kernel<T, NJ_>, grid, dim3(256), 0, s, a) != cudaSuccess;
  LB_NJ(1) LB_NJ(2) LB_NJ(4) LB_NJ(8) LB_NJ(16)
#undef LB_NJ
  return 1;
}

// ---------------------------------------------------------------------------------------------------------------
// Mamba-2 decode: one CTA per (head, sequence), one token per sequence. Phase 1: convolution + silu of the head's x
// channels and of its group's B and C channels into shared memory. Phase 2: the state rows. The head writes the new
// convolution history of its own x channels; B and C channels are shared by the heads of a group, so the last of them
// to have read the old history (an arrival counter per sequence and group) replaces it.
// ---------------------------------------------------------------------------------------------------------------
template <typename T, int NJ>
__global__ void __launch_bounds__(256) ssd_decode_kernel(const SsdDecodeArgs a) {
  extern __shared__ float sm[];                       // x [P] | B [N] | C [N]
  __shared__ int s_last;
  griddep_wait();
  griddep_launch();
  const LinScanArgs& L = a.s;
  const int h = blockIdx.x, n = blockIdx.y;
  const int P = L.P, N = L.N, G = L.G, H = L.H, hpg = H / G, g = h / hpg;
  const int slot = L.slots[n];
  if (slot < 0) return;
  const int inner = H * P, C = inner + 2 * G * N, K1 = a.KC - 1;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const T* x = static_cast<const T*>(a.xbc) + long(n) * a.ldx;
  float* hist = a.conv_state + long(slot) * C * K1;
  auto channel = [&](int i) { return i < P ? h * P + i : inner + (i < P + N ? g * N + (i - P) : G * N + g * N + (i - P - N)); };
  for (int i = threadIdx.x; i < P + 2 * N; i += 256) {
    const int c = channel(i);
    const float xv = ld_f(x + c);
    float* hc = hist + long(c) * K1;
    const float* wc = a.conv_w + long(c) * a.KC;
    float acc = a.conv_b ? a.conv_b[c] : 0.f;
    acc = fmaf(wc[K1], xv, acc);
    for (int j = 0; j < K1; ++j) {
      const float hv = hc[j];
      acc = fmaf(wc[j], hv, acc);
      if (i < P && j > 0) hc[j - 1] = hv;              // x channels belong to this head alone
    }
    if (i < P && K1 > 0) hc[K1 - 1] = xv;
    sm[i] = silu_f(acc);
  }
  __threadfence();
  __syncthreads();
  if (threadIdx.x == 0) {
    s_last = 0;
    if (K1 > 0) {
      const unsigned int old = atomicAdd(&a.ctr[long(n) * G + g], 1u);
      s_last = old == unsigned(hpg) - 1u;
      if (s_last) a.ctr[long(n) * G + g] = 0u;
    }
  }
  __syncthreads();
  if (s_last) {
    __threadfence();
    for (int i = P + threadIdx.x; i < P + 2 * N; i += 256) {
      const int c = channel(i);
      float* hc = hist + long(c) * K1;
      for (int j = 0; j + 1 < K1; ++j) hc[j] = __ldcg(&hc[j + 1]);
      hc[K1 - 1] = ld_f(x + c);
    }
  }
  const float dt = softplus_f(ld_f(static_cast<const T*>(L.dt) + long(n) * L.lddt + h) + L.dt_bias[h]);
  const float dec = expf(dt * L.A[h]);
  const float Dh = L.D ? L.D[h] : 0.f;
  float k[NJ], q[NJ];
#pragma unroll
  for (int j = 0; j < NJ; ++j) {
    const int i = lane + 32 * j;
    k[j] = i < N ? sm[P + i] : 0.f;
    q[j] = i < N ? sm[P + N + i] : 0.f;
  }
  for (int p0 = warp * RPW; p0 < P; p0 += WARPS * RPW) {
    float* st = L.state + ((long(slot) * H + h) * P + p0) * N;
    float s[RPW][NJ];
#pragma unroll
    for (int r = 0; r < RPW; ++r)
#pragma unroll
      for (int j = 0; j < NJ; ++j) {
        const int i = lane + 32 * j;
        s[r][j] = (p0 + r < P && i < N) ? st[long(r) * N + i] : 0.f;
      }
    float mine = 0.f;
#pragma unroll
    for (int r = 0; r < RPW; ++r) {
      const float vd = p0 + r < P ? sm[p0 + r] * dt : 0.f;
      float o = 0.f;
#pragma unroll
      for (int j = 0; j < NJ; ++j) {
        s[r][j] = fmaf(dec, s[r][j], vd * k[j]);
        o = fmaf(s[r][j], q[j], o);
        const int i = lane + 32 * j;
        if (p0 + r < P && i < N) st[long(r) * N + i] = s[r][j];
      }
      o = warp_sum_f(o);
      if (lane == r) mine = o;
    }
    if (lane < RPW && p0 + lane < P) {
      float y = fmaf(Dh, sm[p0 + lane], mine);
      if (L.z) y *= silu_f(ld_f(static_cast<const T*>(L.z) + long(n) * L.ldz + long(h) * P + p0 + lane));
      st_f(static_cast<T*>(L.out) + long(n) * L.ldo + long(h) * P + p0 + lane, y);
    }
  }
}

template <typename T>
int ssd_decode_t(const SsdDecodeArgs& a, cudaStream_t s) {
  const dim3 grid(a.s.H, a.s.n_seqs);
  const size_t smem = size_t(a.s.P + 2 * a.s.N) * 4;
  if (smem > 40 * 1024) return 1;
#define LB_NJ(NJ_) \
  if (a.s.N <= 32 * NJ_) return launch_pdl(ssd_decode_kernel<T, NJ_>, grid, dim3(256), smem, s, a) != cudaSuccess;
  LB_NJ(1) LB_NJ(2) LB_NJ(4) LB_NJ(8) LB_NJ(16)
#undef LB_NJ
  return 1;
}

// ---------------------------------------------------------------------------------------------------------------
template <typename T, int VEC>
__global__ void __launch_bounds__(256) group_norm_gate_kernel(const T* __restrict__ y, long ldy, const T* __restrict__ gate,
                                                              long ldg, const float* __restrict__ w, float eps, int part,
                                                              T* __restrict__ out, long ldo) {
  __shared__ float red[8];
  griddep_wait();
  griddep_launch();
  const long row = blockIdx.x;
  const int c0 = blockIdx.y * part;
  const T* yr = y + row * ldy + c0;
  float ss = 0.f;
  for (int c = threadIdx.x * VEC; c < part; c += blockDim.x * VEC) {
    float v[VEC];
    ld_vec<VEC>(yr + c, v);
#pragma unroll
    for (int j = 0; j < VEC; ++j) ss = fmaf(v[j], v[j], ss);
  }
  ss = warp_sum_f(ss);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
  __syncthreads();
  float tot = 0.f;
  for (int i = 0; i < int(blockDim.x) / 32; ++i) tot += red[i];
  const float inv = 1.f / sqrtf(tot / float(part) + eps);
  for (int c = threadIdx.x * VEC; c < part; c += blockDim.x * VEC) {
    float v[VEC], gv[VEC];
    ld_vec<VEC>(yr + c, v);
    if (gate) ld_vec<VEC>(gate + row * ldg + c0 + c, gv);
#pragma unroll
    for (int j = 0; j < VEC; ++j) {
      v[j] = v[j] * inv * w[c0 + c + j];
      if (gate) v[j] *= sigmoid_f(gv[j]);
    }
    st_vec<VEC>(out + row * ldo + c0 + c, v);
  }
}

template <typename T>
int group_norm_t(const void* y, long ldy, const void* gate, long ldg, const float* w, float eps, int groups, int C,
                 int rows, void* out, long ldo, cudaStream_t s) {
  const int part = C / groups;
  const size_t al = 4 * sizeof(T);
  const bool v4 = part % 4 == 0 && ldy % 4 == 0 && ldo % 4 == 0 && (!gate || ldg % 4 == 0) &&
                  ((reinterpret_cast<uintptr_t>(y) | reinterpret_cast<uintptr_t>(out) |
                    reinterpret_cast<uintptr_t>(gate)) % al) == 0;
  int nt = 256;
  while (nt > 32 && (nt / 2) * (v4 ? 4 : 1) >= part) nt /= 2;
  return launch_pdl(v4 ? group_norm_gate_kernel<T, 4> : group_norm_gate_kernel<T, 1>, dim3(rows, groups), dim3(nt), 0, s,
                    static_cast<const T*>(y), ldy, static_cast<const T*>(gate), ldg, w, eps, part, static_cast<T*>(out),
                    ldo) != cudaSuccess;
}

}  // namespace

int linear_scan_launch(const LinScanArgs& a, bool f32, cudaStream_t s) {
  if (a.n_seqs <= 0 || a.T <= 0) return 0;
  if (a.G <= 0 || a.H % a.G) return 1;
  return f32 ? scan_t<float>(a, s) : scan_t<__nv_bfloat16>(a, s);
}

int ssd_decode_launch(const SsdDecodeArgs& a, bool f32, cudaStream_t s) {
  if (a.s.n_seqs <= 0) return 0;
  if (a.s.G <= 0 || a.s.H % a.s.G || a.KC < 1) return 1;
  return f32 ? ssd_decode_t<float>(a, s) : ssd_decode_t<__nv_bfloat16>(a, s);
}

int group_norm_gate_launch(const void* y, long ldy, const void* gate, long ldg, const float* w, float eps, int groups,
                           int C, int rows, void* out, long ldo, bool f32, cudaStream_t s) {
  if (rows <= 0) return 0;
  if (groups <= 0 || C % groups) return 1;
  return f32 ? group_norm_t<float>(y, ldy, gate, ldg, w, eps, groups, C, rows, out, ldo, s)
             : group_norm_t<__nv_bfloat16>(y, ldy, gate, ldg, w, eps, groups, C, rows, out, ldo, s);
}

}  // namespace lb
