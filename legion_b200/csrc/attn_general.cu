// Attention pieces for any head sizes and for fp32: head norms + paged append, and paged causal attention on FMA
// units. The tcgen05 kernels (attn_prefill_sm100.cu, attn_decode_sm100.cu) take the bf16 shapes; this file serves fp32
// models and head widths those do not cover.
#include "act_type.cuh"
#include "attn_extra.h"
#include "common.cuh"
#include "layers.h"

namespace lb {
namespace {

// One warp per (token, head): Hq query heads, Hkv key heads, Hkv value heads. Keys and values go to the token's cell of
// the paged cache, queries to q_out. The head norm (weights qw / kw, none when null) is a plain RMS norm.
template <typename T>
__global__ void __launch_bounds__(128) qkv_norm_append_kernel(const T* __restrict__ q, const T* __restrict__ k,
                                                              const T* __restrict__ v, long ld,
                                                              const float* __restrict__ qw, const float* __restrict__ kw,
                                                              float eps, const long* __restrict__ slots,
                                                              T* __restrict__ q_out, T* __restrict__ k_cache,
                                                              T* __restrict__ v_cache, long k_cell, long v_cell, int nT,
                                                              int Hq, int Hkv, int DK, int DV) {
  griddep_wait();
  griddep_launch();
  const int lane = threadIdx.x & 31;
  const long gw = (long(blockIdx.x) * blockDim.x + threadIdx.x) >> 5;
  const int heads = Hq + 2 * Hkv;
  if (gw >= long(nT) * heads) return;
  const int t = int(gw / heads), h = int(gw % heads);
  const T* src;
  T* dst;
  const float* nw = nullptr;
  int D = DK;
  if (h < Hq) {
    src = q + t * ld + long(h) * DK;
    dst = q_out + (long(t) * Hq + h) * DK;
    nw = qw;
  } else {
    const long cell = slots[t];
    if (cell < 0) return;
    if (h < Hq + Hkv) {
      src = k + t * ld + long(h - Hq) * DK;
      dst = k_cache + cell * k_cell + long(h - Hq) * DK;
      nw = kw;
    } else {
      D = DV;
      src = v + t * ld + long(h - Hq - Hkv) * DV;
      dst = v_cache + cell * v_cell + long(h - Hq - Hkv) * DV;
    }
  }
  float inv = 1.f;
  if (nw) {
    float ss = 0.f;
    for (int d = lane; d < D; d += 32) {
      const float x = ld_f(src + d);
      ss = fmaf(x, x, ss);
    }
    inv = 1.f / sqrtf(warp_sum_f(ss) / float(D) + eps);
  }
  for (int d = lane; d < D; d += 32) {
    const float x = ld_f(src + d);
    st_f(dst + d, nw ? x * inv * nw[d] : x);
  }
}

// One warp per (token, query head). 32 keys at a time: lane = key for the scores, then lane = value columns.
template <typename T, int NV>
__global__ void __launch_bounds__(128) paged_attn_general_kernel(
    const T* __restrict__ q, long q_row, const T* __restrict__ k_cache, const T* __restrict__ v_cache, long k_cell, long v_cell,
    const int* __restrict__ cu_q, const int* __restrict__ ctx_lens, const int* __restrict__ block_table, int table_width,
    int page, int n_seqs, int nT, int Hq, int Hkv, int DK, int DV, float scale, float cap, int window, T* __restrict__ out, const AttnExtra x) {
  extern __shared__ float q_sm[];
  griddep_wait();
  griddep_launch();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const long gw = long(blockIdx.x) * 4 + warp;
  if (gw >= long(nT) * Hq) return;
  const int t = int(gw / Hq), h = int(gw % Hq);
  int lo_s = 0, hi_s = n_seqs;                       // the sequence whose rows hold t: last i with cu_q[i] <= t
  while (hi_s - lo_s > 1) {
    const int m = (lo_s + hi_s) >> 1;
    if (cu_q[m] <= t) lo_s = m; else hi_s = m;
  }
  const int seq = lo_s;
  const int pos = ctx_lens[seq] - (cu_q[seq + 1] - t);
  const int kvh = h / (Hq / Hkv);
  float* qs = q_sm + warp * DK;
  for (int d = lane; d < DK; d += 32) qs[d] = ld_f(q + (long(t) * Hq + h) * q_row + d);
  __syncwarp();
  const int* bt = block_table + long(seq) * table_width;
  const int lo = window > 0 ? max(0, pos - window + 1) : 0;
  const int skip = lo - min(x.keep, lo);             // tokens between the kept first ones and the window
  float m = -INFINITY, l = 0.f, acc[NV];
  if (x.sink) {                                      // as if a key with this score and no value had been seen
    m = x.sink[h];
    l = 1.f;
  }
#pragma unroll
  for (int j = 0; j < NV; ++j) acc[j] = 0.f;
  const int last = pos - skip;                       // places of the visible tokens: 0 .. last
  for (int k0 = 0; k0 <= last; k0 += 32) {
    const int place = k0 + lane, key = place < lo - skip ? place : place + skip;
    long cell = 0;
    float s = -INFINITY;
    if (place <= last) {
      cell = long(bt[key / page]) * page + key % page;
      const T* kr = k_cache + cell * k_cell + long(kvh) * DK;
      float a0 = 0.f, a1 = 0.f;
      int d = 0;
      for (; d + 1 < DK; d += 2) {
        a0 = fmaf(qs[d], ld_f(kr + d), a0);
        a1 = fmaf(qs[d + 1], ld_f(kr + d + 1), a1);
      }
      if (d < DK) a0 = fmaf(qs[d], ld_f(kr + d), a0);
      s = (a0 + a1) * scale;
      if (cap > 0.f) s = cap * tanhf(s / cap);
    }
    float mx = s;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
    const float mn = fmaxf(m, mx);
    const float p = place <= last ? expf(s - mn) : 0.f;
    const float alpha = m == -INFINITY ? 0.f : expf(m - mn);
    m = mn;
    l = l * alpha + warp_sum_f(p);
#pragma unroll
    for (int j = 0; j < NV; ++j) acc[j] *= alpha;
    const int n = min(32, last - k0 + 1);
    for (int i = 0; i < n; ++i) {
      const float pi = __shfl_sync(0xffffffffu, p, i);
      const long ci = __shfl_sync(0xffffffffu, cell, i);
      const T* vr = v_cache + ci * v_cell + long(kvh) * DV;
#pragma unroll
      for (int j = 0; j < NV; ++j) {
        const int d = lane + 32 * j;
        if (d < DV) acc[j] = fmaf(pi, ld_f(vr + d), acc[j]);
      }
    }
  }
  float f = l > 0.f ? x.out_scale / l : 0.f;
  if (x.gate) f *= sigmoid_f(ld_f(static_cast<const T*>(x.gate) + t * x.ld_gate + h));
  T* orow = x.on ? out + t * x.ldo + long(h) * DV : out + (long(t) * Hq + h) * DV;
#pragma unroll
  for (int j = 0; j < NV; ++j) {
    const int d = lane + 32 * j;
    if (d < DV) st_f(orow + d, acc[j] * f);
  }
}

template <typename T>
int attn_t(const void* q, long q_row, const void* k, const void* v, long k_cell, long v_cell, const int* cu_q, const int* ctx_lens,
           const int* bt, int tw, int page, int n_seqs, int nT, int Hq, int Hkv, int DK, int DV, float scale, float cap,
           int window, void* out, const AttnExtra& x, cudaStream_t s) {
  const long warps = long(nT) * Hq;
  const dim3 grid(unsigned((warps + 3) / 4));
  const size_t smem = size_t(4) * DK * 4;
  if (smem > 40 * 1024) return 1;
#define LB_NV(N)                                                                                                       \
  if (DV <= 32 * N)                                                                                                    \
    return launch_pdl(paged_attn_general_kernel<T, N>, grid, dim3(128), smem, s, static_cast<const T*>(q), q_row,      \
                      static_cast<const T*>(k), static_cast<const T*>(v), k_cell, v_cell, cu_q, ctx_lens, bt, tw,      \
                      page, n_seqs, nT, Hq, Hkv, DK, DV, scale, cap, window, static_cast<T*>(out), x) != cudaSuccess;
  LB_NV(2) LB_NV(4) LB_NV(8) LB_NV(16) LB_NV(32)
#undef LB_NV
  return 1;
}

}  // namespace

int qkv_norm_append_launch(const void* q, const void* k, const void* v, long ld, const float* qw, const float* kw,
                           float eps, const long* slots, void* q_out, void* k_cache, void* v_cache, long k_cell,
                           long v_cell, int T, int Hq, int Hkv, int DK, int DV, bool f32, cudaStream_t s) {
  if (T <= 0) return 0;
  const long warps = long(T) * (Hq + 2 * Hkv);
  const dim3 grid(unsigned((warps * 32 + 127) / 128));
#define LB_T(TT)                                                                                                       \
  return launch_pdl(qkv_norm_append_kernel<TT>, grid, dim3(128), 0, s, static_cast<const TT*>(q),                      \
                    static_cast<const TT*>(k), static_cast<const TT*>(v), ld, qw, kw, eps, slots,                      \
                    static_cast<TT*>(q_out), static_cast<TT*>(k_cache), static_cast<TT*>(v_cache), k_cell, v_cell, T,  \
                    Hq, Hkv, DK, DV) != cudaSuccess;
  if (f32) { LB_T(float) } else { LB_T(__nv_bfloat16) }
#undef LB_T
}

int paged_attn_general_launch(const void* q, long q_row, const void* k_cache, const void* v_cache, long k_cell, long v_cell,
                              const int* cu_q, const int* ctx_lens, const int* block_table, int table_width, int page,
                              int n_seqs, int T, int Hq, int Hkv, int DK, int DV, float scale, float softcap, int window,
                              void* out, bool f32, cudaStream_t s, const AttnExtra& x) {
  if (T <= 0 || n_seqs <= 0) return 0;
  if (page <= 0 || Hkv <= 0 || Hq % Hkv || x.keep < 0) return 1;
  return f32 ? attn_t<float>(q, q_row, k_cache, v_cache, k_cell, v_cell, cu_q, ctx_lens, block_table, table_width, page, n_seqs,
                             T, Hq, Hkv, DK, DV, scale, softcap, window, out, x, s)
             : attn_t<__nv_bfloat16>(q, q_row, k_cache, v_cache, k_cell, v_cell, cu_q, ctx_lens, block_table, table_width, page,
                                     n_seqs, T, Hq, Hkv, DK, DV, scale, softcap, window, out, x, s);
}

}  // namespace lb
