// HGRN2: a matrix state per head whose forget gate also decides what is written,
//   F_t = lower + (1 - lower) sigmoid(f_t + b),   S_t = diag(F_t) S_(t-1) + (1 - F_t) v_t^T,   o_t = S_t^T silu(q_t),
// followed by an RMS norm of each head's o (plain weight, times a constant). Token by token, fp32 state kept as
// [value column][key channel]; decode steps, short portions and fp32. Long bf16 portions run on the chunked tensor-core form
// (forget_scan_sm100.cu). 1 - F is formed as (1 - lower) sigmoid(-z), which keeps its relative accuracy where F is close to 1.
//
// A CTA owns a head of a sequence, so the norm stays inside it. Eight lanes share a state column, each with four neighbouring
// channels of every 32; up to 32 IT columns stay in registers from token to token, and a decode step asks for them ahead of the
// wait for the projection. Wider heads go through memory once per token.
#include "act_type.cuh"
#include "common.cuh"
#include "layers.h"
#include "state_cols.cuh"

namespace lb {
namespace {

template <typename T>
__device__ __forceinline__ float sigmoid_of(float z) {
  if constexpr (sizeof(T) == 2) return __fdividef(1.f, 1.f + __expf(-z));
  else return sigmoid_f(z);
}

template <typename T, int NI, int IT>
__global__ void __launch_bounds__(256) forget_scan_kernel(const ForgetScanArgs a) {
  constexpr int DKP = 32 * NI;
  extern __shared__ __align__(16) float sm[];          // F | 1 - F | q [DKP each] | v | o [P each]
  __shared__ float red[8];
  const int N = a.N, P = a.P, h = blockIdx.x, seq = blockIdx.y;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, r = lane & 7;
  float* ks = sm, *ws = sm + DKP, *qs = sm + 2 * DKP, *vs = sm + 3 * DKP, *os = vs + P;
  const int t0 = a.cu[seq], t1 = a.cu[seq + 1], slot = a.slots[seq];
  if (t1 <= t0 || slot < 0 || (a.max_tokens > 0 && t1 - t0 > a.max_tokens)) return;
  float* state = a.state + (long(slot) * a.H + h) * P * N;
  const int n_it = (P + 31) / 32;                      // groups of 32 columns
  const bool held = n_it <= IT;
  auto column = [&](int it) { return it * 32 + warp * 4 + (lane >> 3); };
  uint64_t S[IT][2 * NI];
  auto load = [&](int it0) {
#pragma unroll
    for (int it = 0; it < IT; ++it)
      if (it0 + it < n_it) load_state<NI>(state + long(min(column(it0 + it), P - 1)) * N, r, N, column(it0 + it) < P, S[it]);
  };
  auto store = [&](int it0) {
#pragma unroll
    for (int it = 0; it < IT; ++it)
      if (column(it0 + it) < P) store_state<NI>(state + long(column(it0 + it)) * N, r, N, S[it]);
  };
  // nothing in front of this launch writes state or weights of this step
  load(0);
  const float fb0 = tid < N ? a.f_b[h * N + tid] : 0.f, lo0 = tid < N ? a.lower[h * N + tid] : 0.f;
  const float nw0 = tid < P ? a.norm_w[tid] * a.scale : 0.f;
  griddep_wait();
  griddep_launch();
  const T* qp = static_cast<const T*>(a.q) + long(h) * N;
  const T* fp = static_cast<const T*>(a.f) + long(h) * N;
  const T* vp = static_cast<const T*>(a.v) + long(h) * P;
  for (int c = N + tid; c < DKP; c += 256) ks[c] = ws[c] = qs[c] = 0.f;
  for (int t = t0; t < t1; ++t) {
    for (int c = tid; c < N; c += 256) {
      const float z = ld_f(fp + t * a.ldf + c) + (c == tid ? fb0 : a.f_b[h * N + c]), lo = c == tid ? lo0 : a.lower[h * N + c];
      const float q = ld_f(qp + t * a.ldq + c);
      ks[c] = fmaf(1.f - lo, sigmoid_of<T>(z), lo);
      ws[c] = (1.f - lo) * sigmoid_of<T>(-z);
      qs[c] = q * sigmoid_of<T>(q);
    }
    for (int c = tid; c < P; c += 256) vs[c] = ld_f(vp + t * a.ldv + c);
    __syncthreads();
    float oo = 0.f;
    for (int it0 = 0; it0 < n_it; it0 += IT) {
      if (!held && (t > t0 || it0 > 0)) load(it0);
#pragma unroll
      for (int it = 0; it < IT; ++it) {
        if (it0 + it >= n_it) break;
        const int col = column(it0 + it);
        const float v = col < P ? vs[col] : 0.f;
        const uint64_t V = p2(v, v);
        uint64_t o2 = 0ull;
#pragma unroll
        for (int i = 0; i < NI; ++i) {
          uint64_t k0, k1, w0, w1, q0, q1;
          ld4(ks + 32 * i + 4 * r, k0, k1);
          ld4(ws + 32 * i + 4 * r, w0, w1);
          ld4(qs + 32 * i + 4 * r, q0, q1);
          S[it][2 * i] = fma2(S[it][2 * i], k0, mul2(w0, V));
          S[it][2 * i + 1] = fma2(S[it][2 * i + 1], k1, mul2(w1, V));
          o2 = fma2(S[it][2 * i], q0, o2);
          o2 = fma2(S[it][2 * i + 1], q1, o2);
        }
        float o, o_hi;
        u2(o2, o, o_hi);
        o += o_hi;
#pragma unroll
        for (int d = 4; d > 0; d >>= 1) o += __shfl_xor_sync(0xffffffffu, o, d);
        if (r == 0 && col < P) {
          os[col] = o;
          oo = fmaf(o, o, oo);
        }
      }
      if (a.write_state && (!held || t + 1 == t1)) store(it0);
    }
    oo = warp_sum_f(oo);
    if (lane == 0) red[warp] = oo;
    __syncthreads();
    oo = 0.f;
#pragma unroll
    for (int w = 0; w < 8; ++w) oo += red[w];
    const float inv = 1.f / sqrtf(oo / float(P) + a.eps);
    T* out = static_cast<T*>(a.out) + t * a.ldo + long(h) * P;
    for (int c = tid; c < P; c += 256) st_f(out + c, os[c] * inv * (c == tid ? nw0 : a.norm_w[c] * a.scale));
  }
}

template <typename T>
int launch_t(const ForgetScanArgs& a, cudaStream_t s) {
#define LB_NI(NI_, IT_)                                                                                                \
  if (a.N <= 32 * NI_) {                                                                                               \
    const size_t smem = size_t(3 * 32 * NI_ + 2 * a.P) * 4;                                                            \
    if (!a.write_state && (a.P + 31) / 32 > IT_ && a.T > a.n_seqs) return 1;   /* the state passes through the pool */ \
    return launch_pdl(forget_scan_kernel<T, NI_, IT_>, dim3(a.H, a.n_seqs), dim3(256), smem, s, a) != cudaSuccess;     \
  }
  LB_NI(1, 4) LB_NI(2, 4) LB_NI(4, 4) LB_NI(8, 2) LB_NI(16, 1)
#undef LB_NI
  return 1;
}

}  // namespace

int forget_scan_launch(const ForgetScanArgs& a, bool f32, cudaStream_t s) {
  if (a.n_seqs <= 0 || a.T <= 0) return 0;
  if (a.N < 1 || a.P < 1 || a.P > 4096 || a.n_seqs > 65535 || (reinterpret_cast<uintptr_t>(a.state) & 15)) return 1;
  return f32 ? launch_t<float>(a, s) : launch_t<__nv_bfloat16>(a, s);
}

}  // namespace lb
