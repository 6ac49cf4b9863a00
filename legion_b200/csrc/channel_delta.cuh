// Pieces shared by the kernels of the gated delta rule with a decay per key channel (channel_delta.cu, channel_delta_mma.cu).
#pragma once
#include "act_type.cuh"
#include "common.cuh"
#include "layers.h"

namespace lb {

// Blocks of BT tokens of a slice [lo, hi) of the step's rows: sequence i begins at block (rows of the slice in front of it) /
// BT + i, which leaves room for every sequence's last, partial block. Returns false where a block number has no tokens.
struct DeltaBlock { int seq, t0, n, seq0; };  // sequence, first row, tokens, first row of the sequence
__device__ __forceinline__ int clamp_i(int v, int lo, int hi) { return v < lo ? lo : v > hi ? hi : v; }
template <int BT>
__device__ __forceinline__ bool find_block(const int* cu, int n_seqs, int lo, int hi, int blk, DeltaBlock& b) {
  int a = 0, z = n_seqs;                      // last sequence whose first block is <= blk
  while (z - a > 1) {
    const int m = (a + z) >> 1;
    if ((clamp_i(cu[m], lo, hi) - lo) / BT + m <= blk) a = m; else z = m;
  }
  const int s0 = clamp_i(cu[a], lo, hi), s1 = clamp_i(cu[a + 1], lo, hi);
  const int t0 = s0 + (blk - ((s0 - lo) / BT + a)) * BT;
  if (t0 >= s1) return false;
  b.seq = a; b.t0 = t0; b.n = min(BT, s1 - t0); b.seq0 = cu[a];
  return true;
}

template <typename T>
__device__ __forceinline__ float silu_t(float z) {
  if constexpr (sizeof(T) == 2) return __fdividef(z, 1.f + __expf(-z));
  else return silu_f(z);
}
template <typename T>
__device__ __forceinline__ float sigmoid_t(float z) {
  if constexpr (sizeof(T) == 2) return __fdividef(1.f, 1.f + __expf(-z));
  else return sigmoid_f(z);
}
// exp(A softplus(raw)). bf16: log(1 + e) from the hardware logarithm, by its series where e is small (|error| < 4e-6 of it)
template <typename T>
__device__ __forceinline__ float decay_t(float raw, float A) {
  if constexpr (sizeof(T) == 2) {
    const float e = __expf(-fabsf(raw));
    const float l = e < 0.0625f ? e * fmaf(e, fmaf(e, fmaf(e, -0.25f, 1.f / 3.f), -0.5f), 1.f) : __logf(1.f + e);
    return __expf(A * (fmaxf(raw, 0.f) + l));
  } else {
    return expf(A * softplus_f(raw));
  }
}

// Sum over the warp of 32 values per lane; lane L gets value L.
__device__ __forceinline__ float transpose_sum(float (&v)[32]) {
  const int lane = threadIdx.x & 31;
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    const bool up = lane & o;
#pragma unroll
    for (int i = 0; i < o; ++i) {
      const float send = up ? v[i] : v[i + o], keep = up ? v[i + o] : v[i];
      v[i] = keep + __shfl_xor_sync(0xffffffffu, send, o);
    }
  }
  return v[0];
}

// bf16 prompts with key heads of at most 128 columns (channel_delta_mma.cu)
bool channel_delta_mma_ok(const ChannelDeltaArgs& a);
int channel_delta_mma_launch(const ChannelDeltaArgs& a, float* rec, long rec_floats, int* status, cudaStream_t s);
long channel_delta_mma_floats(int H, int DK, int DV);     // scratch per eight tokens (and per sequence)

}  // namespace lb
