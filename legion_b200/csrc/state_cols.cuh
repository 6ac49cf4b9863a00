// Columns of a recurrent state [value column][key channel] in registers: eight lanes per column, pairs of channels packed for
// the two-wide fp32 instructions.
#pragma once
#include <cuda_runtime.h>
#include <stdint.h>

namespace lb {

__device__ __forceinline__ uint64_t p2(float lo, float hi) {
  uint64_t r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(lo), "f"(hi));
  return r;
}
__device__ __forceinline__ void u2(uint64_t v, float& lo, float& hi) { asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(v)); }
__device__ __forceinline__ uint64_t fma2(uint64_t a, uint64_t b, uint64_t c) {
  uint64_t d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
  return d;
}
__device__ __forceinline__ uint64_t mul2(uint64_t a, uint64_t b) {
  uint64_t d;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}
__device__ __forceinline__ void ld4(const float* p, uint64_t& lo, uint64_t& hi) {
  const ulonglong2 v = *reinterpret_cast<const ulonglong2*>(p);
  lo = v.x;
  hi = v.y;
}

// State rows of a lane: 32 i + 4 (lane & 7) + 0..3 of a column, pairs packed
template <int NI>
__device__ __forceinline__ void load_state(const float* col, int r, int DK, bool ok, uint64_t (&S)[2 * NI]) {
#pragma unroll
  for (int i = 0; i < NI; ++i) {
    const int c = 32 * i + 4 * r;
    float v[4] = {0.f, 0.f, 0.f, 0.f};
    if (ok) {
      if (DK % 4 == 0) {
        if (c < DK) {
          const float4 f = *reinterpret_cast<const float4*>(col + c);
          v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w;
        }
      } else {
#pragma unroll
        for (int j = 0; j < 4; ++j)
          if (c + j < DK) v[j] = col[c + j];
      }
    }
    S[2 * i] = p2(v[0], v[1]);
    S[2 * i + 1] = p2(v[2], v[3]);
  }
}
template <int NI>
__device__ __forceinline__ void store_state(float* col, int r, int DK, const uint64_t (&S)[2 * NI]) {
#pragma unroll
  for (int i = 0; i < NI; ++i) {
    const int c = 32 * i + 4 * r;
    float v[4];
    u2(S[2 * i], v[0], v[1]);
    u2(S[2 * i + 1], v[2], v[3]);
    if (DK % 4 == 0) {
      if (c < DK) *reinterpret_cast<float4*>(col + c) = make_float4(v[0], v[1], v[2], v[3]);
    } else {
#pragma unroll
      for (int j = 0; j < 4; ++j)
        if (c + j < DK) col[c + j] = v[j];
    }
  }
}

}  // namespace lb
