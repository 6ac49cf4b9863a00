// Causal depth-wise convolution with carried history for any number of taps, bf16 and fp32 activations, SiLU and a bias of
// the input optional (conv1d.cu has the bf16 kernels of 2 to 8 taps). One thread per (token, channel).
#include "act_type.cuh"
#include "common.cuh"
#include "layers.h"

namespace lb {
namespace {

template <typename T>
__global__ void __launch_bounds__(128) conv_silu_any_kernel(const T* __restrict__ x, long ldx, const float* __restrict__ w,
                                                            const float* __restrict__ bias,
                                                            const float* __restrict__ conv_state,
                                                            const int* __restrict__ cu, const int* __restrict__ slots,
                                                            int n_seqs, int C, int KC, T* __restrict__ out, long ldo,
                                                            const float* __restrict__ in_bias, int silu) {
  griddep_wait();
  griddep_launch();
  const int c = blockIdx.x * 128 + threadIdx.x, t = blockIdx.y;
  if (c >= C) return;
  int lo = 0, hi = n_seqs;
  while (hi - lo > 1) {
    const int m = (lo + hi) >> 1;
    if (cu[m] <= t) lo = m; else hi = m;
  }
  const int t0 = cu[lo];
  const float* st = conv_state + (long(slots[lo]) * C + c) * (KC - 1);
  float acc = bias ? bias[c] : 0.f;
  const float ib = in_bias ? in_bias[c] : 0.f;
  for (int j = 0; j < KC; ++j) {
    const int s = t - (KC - 1) + j;
    const float v = s >= t0 ? ld_f(x + long(s) * ldx + c) + ib : st[(KC - 1) + (s - t0)];
    acc = fmaf(w[long(c) * KC + j], v, acc);
  }
  st_f(out + long(t) * ldo + c, silu ? silu_f(acc) : acc);
}

// history update: reads of the old history happen in the kernel before (stream order)
template <typename T>
__global__ void __launch_bounds__(128) conv_history_kernel(const T* __restrict__ x, long ldx, float* conv_state,
                                                           const int* __restrict__ cu, const int* __restrict__ slots,
                                                           int C, int KC, const float* __restrict__ in_bias) {
  griddep_wait();
  griddep_launch();
  const int c = blockIdx.x * 128 + threadIdx.x, seq = blockIdx.y;
  if (c >= C) return;
  const int t0 = cu[seq], t1 = cu[seq + 1];
  if (t1 <= t0) return;
  float* st = conv_state + (long(slots[seq]) * C + c) * (KC - 1);
  for (int j = 0; j < KC - 1; ++j) {           // position j takes what was j + n places later: never read after written
    const int s = t1 - (KC - 1) + j;
    st[j] = s >= t0 ? ld_f(x + long(s) * ldx + c) + (in_bias ? in_bias[c] : 0.f) : st[(KC - 1) + (s - t0)];
  }
}

template <typename T>
int conv_t(const void* x, long ldx, const float* w, const float* bias, float* conv_state, const int* cu, const int* slots,
           int n_seqs, int T_, int C, int KC, void* out, long ldo, int write_state, const float* in_bias, int silu,
           cudaStream_t s) {
  if (T_ > 65535) return 1;
  const int cb = (C + 127) / 128;
  if (launch_pdl(conv_silu_any_kernel<T>, dim3(cb, T_), dim3(128), 0, s, static_cast<const T*>(x), ldx, w, bias,
                 static_cast<const float*>(conv_state), cu, slots, n_seqs, C, KC, static_cast<T*>(out), ldo, in_bias,
                 silu) != cudaSuccess)
    return 1;
  if (write_state && KC > 1)
    return launch_pdl(conv_history_kernel<T>, dim3(cb, n_seqs), dim3(128), 0, s, static_cast<const T*>(x), ldx, conv_state,
                      cu, slots, C, KC, in_bias) != cudaSuccess;
  return 0;
}

}  // namespace

int conv_silu_any_launch(const void* x, long ldx, const float* w, const float* bias, float* conv_state,
                         const int* cu_seq, const int* slots, int n_seqs, int T, int C, int KC, void* out, long ldo,
                         int write_state, const float* in_bias, int silu, bool f32, cudaStream_t s) {
  if (n_seqs <= 0 || T <= 0) return 0;
  if (KC < 1) return 1;
  return f32 ? conv_t<float>(x, ldx, w, bias, conv_state, cu_seq, slots, n_seqs, T, C, KC, out, ldo, write_state, in_bias,
                             silu, s)
             : conv_t<__nv_bfloat16>(x, ldx, w, bias, conv_state, cu_seq, slots, n_seqs, T, C, KC, out, ldo, write_state,
                                     in_bias, silu, s);
}

}  // namespace lb
