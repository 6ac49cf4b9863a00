// Plain FMA matrix product with fp32 accumulation, for fp32 models (no reduced-precision matrix mode) and for bf16
// shapes the TMA-fed tcgen05 GEMM does not take (row pitches that are not multiples of 16 bytes). 64 features x 32
// tokens per CTA, 16-wide k steps through shared memory, 2 x 4 outputs per thread; the next k step's operands are
// fetched into registers while the current one is multiplied. The grouped form walks the same tile tables as
// gemm_sm100.cu (tile -> expert, first row, rows), so routed experts run on the same routing plan. A third grid dimension
// serves per-head products (each head's own slice of x, weights and output).
#include "act_type.cuh"
#include "common.cuh"
#include "layers.h"

namespace lb {
namespace {

constexpr int TM = 64, TN = SGEMM_BN, TK = 16;

template <typename T>
__device__ __forceinline__ float act_of(float g, int act) {
  return act == 0 ? silu_f(g) : gelu_tanh_f(g);
}

template <typename T, bool DUAL>
__global__ void __launch_bounds__(256) sgemm_kernel(const SgemmArgs a) {
  __shared__ float ws[DUAL ? 2 : 1][TK][TM + 4];
  __shared__ float xs[TK][TN + 4];
  griddep_wait();
  griddep_launch();
  int group = 0, tok0 = blockIdx.y * TN, ntok = min(TN, a.T - tok0);
  if (a.tile_group) {
    if (int(blockIdx.y) >= *a.n_tiles) return;
    group = a.tile_group[blockIdx.y];
    tok0 = a.tile_tok0[blockIdx.y];
    ntok = min(TN, a.tile_ntok[blockIdx.y]);
  }
  const int n0 = blockIdx.x * TM;
  const T* w = static_cast<const T*>(a.w) + long(group + blockIdx.z) * a.rows_per_group * a.ldw;
  const T* x = static_cast<const T*>(a.x) + blockIdx.z * a.x_head_col;
  const long out_col = blockIdx.z * a.out_head_col;
  const int tid = threadIdx.x;
  const int lk = tid % TK, lr = tid / TK;          // loader: k within the step, row 0..15
  float wr[DUAL ? 2 : 1][4], xr[2];
  auto fetch = [&](int k0) {
    const int k = k0 + lk;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int n = n0 + lr + 16 * i;
#pragma unroll
      for (int d = 0; d < (DUAL ? 2 : 1); ++d)
        wr[d][i] = (n < a.N && k < a.K) ? ld_f(w + (n + d * a.dual_offset) * a.ldw + k) : 0.f;
    }
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int r = lr + 16 * i;
      xr[i] = (r < ntok && k < a.K) ? ld_f(x + long(tok0 + r) * a.ldx + k) : 0.f;
    }
  };
  float acc[DUAL ? 2 : 1][2][4];
#pragma unroll
  for (int d = 0; d < (DUAL ? 2 : 1); ++d)
#pragma unroll
    for (int i = 0; i < 2; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) acc[d][i][j] = 0.f;
  const int fm = (tid % 16) * 4, fn = (tid / 16) * 2;
  fetch(0);
  for (int k0 = 0; k0 < a.K; k0 += TK) {
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int d = 0; d < (DUAL ? 2 : 1); ++d) ws[d][lk][lr + 16 * i] = wr[d][i];
#pragma unroll
    for (int i = 0; i < 2; ++i) xs[lk][lr + 16 * i] = xr[i];
    __syncthreads();
    if (k0 + TK < a.K) fetch(k0 + TK);
#pragma unroll
    for (int k = 0; k < TK; ++k) {
      const float x0 = xs[k][fn], x1 = xs[k][fn + 1];
#pragma unroll
      for (int d = 0; d < (DUAL ? 2 : 1); ++d)
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const float wv = ws[d][k][fm + j];
          acc[d][0][j] = fmaf(x0, wv, acc[d][0][j]);
          acc[d][1][j] = fmaf(x1, wv, acc[d][1][j]);
        }
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    if (fn + i >= ntok) continue;
    const long row = tok0 + fn + i;
    const long orow = a.out_rows ? a.out_rows[row] : row;
    if (orow < 0) continue;
    const float sc = a.tok_scale ? a.tok_scale[row] : 1.f;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + fm + j;
      if (n >= a.N) continue;
      float v = acc[0][i][j];
      if constexpr (DUAL) v = a.bias ? act_of<T>(v + a.bias[n], a.act) * (acc[1][i][j] + a.bias[a.N + n])
                                     : act_of<T>(v, a.act) * acc[1][i][j];
      else if (a.act == 2) { v = fmaxf(v, 0.f); v *= v; }
      else if (a.act == 3) v = xielu_f(v, a.act_ab[0], a.act_ab[1]);
      v *= sc;
      if (a.residual) v += ld_f(static_cast<const T*>(a.residual) + orow * a.ldr + n);
      if (a.out_f32) static_cast<float*>(a.out)[orow * a.ldo + out_col + n] = v;
      else st_f(static_cast<T*>(a.out) + orow * a.ldo + out_col + n, v);
    }
  }
}

template <typename T>
int launch_t(const SgemmArgs& a, cudaStream_t s) {
  const int tiles = a.tile_group ? a.max_tiles : (a.T + TN - 1) / TN;
  const dim3 grid((a.N + TM - 1) / TM, tiles, a.heads > 1 ? a.heads : 1);
  if (tiles <= 0) return 0;
  if (tiles > 65535) return 1;
  return (a.dual ? launch_pdl(sgemm_kernel<T, true>, grid, dim3(256), 0, s, a)
                 : launch_pdl(sgemm_kernel<T, false>, grid, dim3(256), 0, s, a)) != cudaSuccess;
}

}  // namespace

int sgemm_launch(const SgemmArgs& a, bool f32, cudaStream_t s) {
  if (a.N <= 0 || a.K <= 0) return 1;
  return f32 ? launch_t<float>(a, s) : launch_t<__nv_bfloat16>(a, s);
}

}  // namespace lb
