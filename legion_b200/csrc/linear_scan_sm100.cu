// Chunked form of the decayed linear-attention state on tcgen05 (bf16 activations, prompt-sized steps):
//   S_t = a_t S_(t-1) + w_t k_t v_t^T,   o_t = S_t^T q_t          (w_t: the step size of a selective layer, else 1)
// With c_i = sum_{j <= i} log a_j inside a chunk of C = 128 tokens:
//   dS   = sum_j exp(c_C - c_j) w_j k_j v_j^T                     STATES kernel, one CTA per (chunk, head, value tile)
//   S_0' = exp(c_C) S_0 + dS                                      CARRY kernel, elementwise over the chunks of a sequence
//   O_i  = exp(c_i) S_0^T q_i + sum_{j <= i} exp(c_i - c_j) w_j (q_i . k_j) v_j
//                                                                 OUTPUT kernel, one CTA per (chunk, head, value tile)
// Only the elementwise CARRY walks the chunks in order; both contractions run for all chunks at once. The state between
// chunks stays fp32, and whatever enters a contraction beside the bf16 projections (decayed keys, decayed scores, the
// state) is split into two bf16 terms, high part and remainder, so it contributes with about 16 significant bits; the
// decay exp(c_i) of the carried part is applied to the fp32 accumulator. The layout [P, N] of the state makes it the
// K-major B operand of the output product; keys and values are read as MN-major operands from the tiles they were
// loaded into. Tiles are built by the threads (activation, decay and split on the way into swizzled shared memory), so
// any head size and pitch works; head sizes are padded to 64-column halves with zeros.
#include "common.cuh"
#include "layers.h"

namespace lb {
namespace {

constexpr int C = 128;                    // tokens per chunk
constexpr int HALF = C * 128;             // bytes of one 64-column half of a 128-row tile
constexpr float LOG2E = 1.4426950408889634f;

__device__ __forceinline__ void tmem_st16(uint32_t taddr, const uint32_t (&r)[16]) {
  asm volatile(
      "tcgen05.st.sync.aligned.32x32b.x16.b32 [%0], "
      "{%1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, %16};"
      ::"r"(taddr), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]),
      "r"(r[8]), "r"(r[9]), "r"(r[10]), "r"(r[11]), "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15])
      : "memory");
}
__device__ __forceinline__ void tmem_st_wait() { asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory"); }
// A operand (bf16 pairs in 32-bit cells, row = lane) from tensor memory
__device__ __forceinline__ void umma_f16_ts(uint32_t d_tmem, uint32_t a_tmem, uint64_t bdesc, uint32_t idesc,
                                            uint32_t accumulate) {
  asm volatile(
      "{\n\t.reg .pred p;\n\t"
      "setp.ne.b32 p, %4, 0;\n\t"
      "tcgen05.mma.cta_group::1.kind::f16 [%0], [%1], %2, %3, p;\n\t}\n"
      ::"r"(d_tmem), "r"(a_tmem), "l"(bdesc), "r"(idesc), "r"(accumulate)
      : "memory");
}

struct ChunkArgs {
  LinScanArgs L;
  const int* chunk_t0; const int* chunk_n;
  float* dS;                              // [chunks, H, P, N]: chunk contributions, then the state in front of each chunk
  float* gC;                              // [chunks, H] decay over the whole chunk
  int vec_q, vec_k, vec_v, vec_o;         // 16-byte accesses are aligned
  int* status;
};

__device__ __forceinline__ float silu_fast(float z) { return z / (1.f + __expf(-z)); }

__device__ __forceinline__ void unpack8(const uint4& u, float (&v)[8]) {
  const __nv_bfloat162* p = reinterpret_cast<const __nv_bfloat162*>(&u);
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    const float2 f = __bfloat1622float2(p[j]);
    v[2 * j] = f.x;
    v[2 * j + 1] = f.y;
  }
}

// Eight columns of a row as floats (zeros outside), activation applied and rounded to bf16 where the layer has one.
__device__ __forceinline__ void load8(const __nv_bfloat16* row, int col, int width, bool row_ok, bool vec, bool silu,
                                      float (&v)[8]) {
#pragma unroll
  for (int j = 0; j < 8; ++j) v[j] = 0.f;
  if (!row_ok || col >= width) return;
  if (vec && col + 8 <= width) {
    unpack8(__ldg(reinterpret_cast<const uint4*>(row + col)), v);
  } else {
#pragma unroll
    for (int j = 0; j < 8; ++j)
      if (col + j < width) v[j] = __bfloat162float(row[col + j]);
  }
  if (silu) {
#pragma unroll
    for (int j = 0; j < 8; ++j) v[j] = silu_fast(v[j]);
  }
}
__device__ __forceinline__ uint4 pack8(const float (&v)[8]) {
  return make_uint4(pack_bf16x2(v[0], v[1]), pack_bf16x2(v[2], v[3]), pack_bf16x2(v[4], v[5]), pack_bf16x2(v[6], v[7]));
}
// v -> high bf16 part (packed) and the remainder left in v
__device__ __forceinline__ uint4 split8(float (&v)[8]) {
  const uint4 hi = pack8(v);
  const __nv_bfloat162* p = reinterpret_cast<const __nv_bfloat162*>(&hi);
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    const float2 f = __bfloat1622float2(p[j]);
    v[2 * j] -= f.x;
    v[2 * j + 1] -= f.y;
  }
  return hi;
}

// A [128 token rows] x [HALVES * 64 columns] tile, eight columns of a row at a time: put(row, byte offset in the
// K-major 128-byte-swizzled tile, values). With aligned rows all of a thread's loads are issued before the first is used.
template <int HALVES, typename Put>
__device__ __forceinline__ void each8(const __nv_bfloat16* src, long ld, int width, int nval, bool vec, bool silu, Put put) {
  constexpr int IT = C * HALVES * 8 / 256;
  auto at = [](int i, int& row, int& c8) {
    const int e = threadIdx.x + 256 * i;
    row = e / (HALVES * 8);
    c8 = e % (HALVES * 8);
  };
  auto off = [](int row, int c8) { return (c8 >> 3) * HALF + row * 128 + (((c8 & 7) ^ (row & 7)) << 4); };
  if (vec) {
    uint4 raw[IT];
#pragma unroll
    for (int i = 0; i < IT; ++i) {
      int row, c8;
      at(i, row, c8);
      raw[i] = (row < nval && c8 * 8 < width) ? __ldg(reinterpret_cast<const uint4*>(src + long(row) * ld + c8 * 8))
                                              : make_uint4(0u, 0u, 0u, 0u);
    }
#pragma unroll
    for (int i = 0; i < IT; ++i) {
      int row, c8;
      at(i, row, c8);
      float v[8];
      unpack8(raw[i], v);
      if (silu) {
#pragma unroll
        for (int j = 0; j < 8; ++j) v[j] = silu_fast(v[j]);
      }
      put(row, off(row, c8), v);
    }
  } else {
#pragma unroll 1
    for (int i = 0; i < IT; ++i) {
      int row, c8;
      at(i, row, c8);
      float v[8];
      load8(src + long(row) * ld, c8 * 8, width, row < nval, false, silu, v);
      put(row, off(row, c8), v);
    }
  }
}
template <int HALVES>
__device__ __forceinline__ void load_tile(uint8_t* dst, const __nv_bfloat16* src, long ld, int width, int nval, bool vec,
                                          bool silu) {
  each8<HALVES>(src, ld, width, nval, vec, silu,
                [&](int, int off, float (&v)[8]) { *reinterpret_cast<uint4*>(dst + off) = pack8(v); });
}

// log2 of a constant decay; decays sit close to 1, where log1p keeps the relative accuracy that a plain logarithm loses
__device__ __forceinline__ float log2_decay(float d) { return fmaxf(log1pf(d - 1.f) * LOG2E, -1e4f); }

// cumulative log2 decay c (inclusive) and input weight w of the chunk's tokens; needs 4 floats of scratch
__device__ __forceinline__ void chunk_decay(const ChunkArgs& a, int h, int t0, int nval, float* cs, float* ws, float* tmp) {
  const LinScanArgs& L = a.L;
  const int i = threadIdx.x, lane = i & 31;
  float g = 0.f, w = 0.f;
  if (i < C) {
    if (i < nval) {
      w = 1.f;
      if (L.decay) {
        g = log2_decay(L.decay[h]);
      } else {
        const float raw = __bfloat162float(static_cast<const __nv_bfloat16*>(L.dt)[long(t0 + i) * L.lddt + h]) + L.dt_bias[h];
        w = raw > 20.f ? raw : log1pf(expf(raw));
        g = w * L.A[h] * LOG2E;
      }
    }
    ws[i] = w;
  }
  if (L.decay) {                           // constant decay: multiples of one logarithm, no sums to round
    if (i < C) cs[i] = g != 0.f || i < nval ? g * float(i + 1) : log2_decay(L.decay[h]) * float(nval);
    __syncthreads();
    return;
  }
  float c = g;
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const float n = __shfl_up_sync(0xffffffffu, c, o);
    if (lane >= o) c += n;
  }
  if (i < C && lane == 31) tmp[i >> 5] = c;
  __syncthreads();
  if (i < C) {
    for (int k = 0; k < (i >> 5); ++k) c += tmp[k];
    cs[i] = c;
  }
  __syncthreads();
}

// ---------------------------------------------------------------------------------------------------------------
// STATES: dS[p, n] = sum_j (v_j[p]) (w_j exp(c_C - c_j) k_j[n]); A = V^T (MN-major), B = K' (MN-major), M = value columns
// ---------------------------------------------------------------------------------------------------------------
template <int NH, int PH>
constexpr int states_smem() { return (PH + 2 * NH) * HALF + 2 * C * 4 + 1024 + 128; }

template <int NH, int PH>
__global__ void __launch_bounds__(256) chunk_states_kernel(const ChunkArgs a) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* v_s = smem;
  uint8_t* kh_s = v_s + PH * HALF;
  uint8_t* kl_s = kh_s + NH * HALF;
  float* cs = reinterpret_cast<float*>(kl_s + NH * HALF);
  float* ws = cs + C;
  uint64_t* done = reinterpret_cast<uint64_t*>(ws + C);
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(done + 1);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  float* tmp = reinterpret_cast<float*>(tmem_slot + 2);
  const LinScanArgs& L = a.L;
  const int chunk = blockIdx.x, h = blockIdx.y, p0 = blockIdx.z * PH * 64;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int g = h / (L.H / L.G);
  if (threadIdx.x == 0) {
    mbar_init(done, 1);
    *abort_flag = 0;
    mbar_fence_init();
  }
  if (warp == 1) {
    tmem_alloc(tmem_slot, NH * 64);
    tmem_relinquish();
  }
  griddep_wait();
  griddep_launch();
  const int t0 = a.chunk_t0[chunk], nval = a.chunk_n[chunk];
  chunk_decay(a, h, t0, nval, cs, ws, tmp);
  const float cC = cs[C - 1];
  const auto* vp = static_cast<const __nv_bfloat16*>(L.v) + long(t0) * L.ldv + long(h) * L.P + p0;
  const auto* kp = static_cast<const __nv_bfloat16*>(L.k) + long(t0) * L.ldk + long(g) * L.N;
  load_tile<PH>(v_s, vp, L.ldv, L.P - p0, nval, a.vec_v, L.silu_in);
  each8<NH>(kp, L.ldk, L.N, nval, a.vec_k, L.silu_in, [&](int row, int off, float (&v)[8]) {
    const float f = exp2f(cC - cs[row]) * ws[row];
#pragma unroll
    for (int j = 0; j < 8; ++j) v[j] = (L.silu_in ? __bfloat162float(__float2bfloat16(v[j])) : v[j]) * f;
    *reinterpret_cast<uint4*>(kh_s + off) = split8(v);
    *reinterpret_cast<uint4*>(kl_s + off) = pack8(v);
  });
  fence_proxy_async_smem();
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_slot;
  if (threadIdx.x == 0) {
    constexpr uint32_t idesc = umma_idesc(128, NH * 64, 1, 1, 1, 1);
    const uint32_t va = smem_u32(v_s), kh = smem_u32(kh_s), kl = smem_u32(kl_s);
    const uint32_t lbo = PH == 1 ? 0u : uint32_t(HALF);    // 64 value columns: the only group is read twice, the copy dropped
#pragma unroll
    for (int k = 0; k < C / 16; ++k) {
      const uint64_t ad = umma_desc_mn_sw128(va + k * 16 * 128, lbo, 1024);
      umma_f16(tmem, ad, umma_desc_mn_sw128(kh + k * 16 * 128, HALF, 1024), idesc, k ? 1u : 0u);
      umma_f16(tmem, ad, umma_desc_mn_sw128(kl + k * 16 * 128, HALF, 1024), idesc, 1u);
    }
    umma_commit(done);
    if (blockIdx.z == 0) a.gC[long(chunk) * L.H + h] = exp2f(cC);
  }
  const bool ok = mbar_wait(done, 0, abort_flag);
  if (!ok) { *abort_flag = 1; atomicCAS(a.status, 0, ST_TIMEOUT_TMEM_FULL | SITE_CHUNK_STATES); }
  __syncwarp();
  tc_fence_after();
  if (__all_sync(0xffffffffu, ok)) {
    const int p = p0 + (warp & 3) * 32 + lane;
    const bool p_ok = (warp & 3) * 32 + lane < PH * 64 && p < L.P;
    float* dst = a.dS + ((long(chunk) * L.H + h) * L.P + p) * L.N;
#pragma unroll 1
    for (int c = (warp >> 2) * (NH * 32); c < ((warp >> 2) + 1) * (NH * 32); c += 32) {
      uint32_t r[32];
      tmem_ld32(tmem + (uint32_t((warp & 3) * 32) << 16) + c, r);
      tmem_ld_wait();
      if (p_ok) {
        if (L.N % 4 == 0) {
#pragma unroll
          for (int j = 0; j < 32; j += 4)
            if (c + j < L.N)
              *reinterpret_cast<float4*>(dst + c + j) = make_float4(__uint_as_float(r[j]), __uint_as_float(r[j + 1]),
                                                                    __uint_as_float(r[j + 2]), __uint_as_float(r[j + 3]));
        } else {
#pragma unroll
          for (int j = 0; j < 32; ++j)
            if (c + j < L.N) dst[c + j] = __uint_as_float(r[j]);
        }
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem, NH * 64);
  }
}

// ---------------------------------------------------------------------------------------------------------------
// CARRY: the contributions become the state in front of each chunk; the pool gets the state behind the last one.
// ---------------------------------------------------------------------------------------------------------------
template <int VEC>
__global__ void __launch_bounds__(256) chunk_carry_kernel(const ChunkArgs a, const int* __restrict__ seq_chunk0,
                                                          const int* __restrict__ seq_nchunk) {
  griddep_wait();
  griddep_launch();
  const LinScanArgs& L = a.L;
  const int h = blockIdx.y, seq = blockIdx.z, slot = L.slots[seq];
  const long e = (long(blockIdx.x) * 256 + threadIdx.x) * VEC, PN = long(L.P) * L.N;
  const int n = seq_nchunk[seq], c0 = seq_chunk0[seq];
  if (e >= PN || n <= 0 || slot < 0) return;
  float* st = L.state + (long(slot) * L.H + h) * PN + e;
  float s[VEC];
  auto ld = [&](const float* p, float (&v)[VEC]) {
    if constexpr (VEC == 4) {
      const float4 f = *reinterpret_cast<const float4*>(p);
      v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w;
    } else {
      v[0] = *p;
    }
  };
  auto stv = [&](float* p, const float (&v)[VEC]) {
    if constexpr (VEC == 4) *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
    else *p = v[0];
  };
  ld(st, s);
  constexpr int U = 8;                      // contributions in flight
  for (int b = 0; b < n; b += U) {
    float d[U][VEC], gc[U];
#pragma unroll
    for (int u = 0; u < U; ++u)
      if (b + u < n) {
        const long row = long(c0 + b + u) * L.H + h;
        ld(a.dS + row * PN + e, d[u]);
        gc[u] = a.gC[row];
      }
#pragma unroll
    for (int u = 0; u < U; ++u)
      if (b + u < n) {
        stv(a.dS + (long(c0 + b + u) * L.H + h) * PN + e, s);
#pragma unroll
        for (int j = 0; j < VEC; ++j) s[j] = fmaf(gc[u], s[j], d[u][j]);
      }
  }
  if (L.write_state) stv(st, s);
}

// ---------------------------------------------------------------------------------------------------------------
// OUTPUT
// ---------------------------------------------------------------------------------------------------------------
template <int NH, int PH>
constexpr int output_smem() { return 2 * NH * HALF + PH * HALF + 2 * NH * (PH * 64 * 128) + 2 * C * 4 + 1024 + 128; }

template <int NH, int PH>
__global__ void __launch_bounds__(256) chunk_output_kernel(const ChunkArgs a) {
  constexpr int PW = PH * 64;
  constexpr int SHALF = PW * 128;           // bytes of one 64-column half of the state tile
  constexpr int TM_COLS = PH == 1 ? 256 : 512;   // scores 128 (later high parts and remainders), two accumulators
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* q_s = smem;
  uint8_t* k_s = q_s + NH * HALF;
  uint8_t* v_s = k_s + NH * HALF;
  uint8_t* sh_s = v_s + PH * HALF;
  uint8_t* sl_s = sh_s + NH * SHALF;
  float* cs = reinterpret_cast<float*>(sl_s + NH * SHALF);
  float* ws = cs + C;
  uint64_t* s_done = reinterpret_cast<uint64_t*>(ws + C);
  uint64_t* o_done = s_done + 1;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(s_done + 2);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  float* tmp = reinterpret_cast<float*>(tmem_slot + 2);
  const LinScanArgs& L = a.L;
  const int chunk = blockIdx.x, h = blockIdx.y, p0 = blockIdx.z * PW;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int g = h / (L.H / L.G);
  if (threadIdx.x == 0) {
    mbar_init(s_done, 1);
    mbar_init(o_done, 1);
    *abort_flag = 0;
    mbar_fence_init();
  }
  if (warp == 1) {
    tmem_alloc(tmem_slot, TM_COLS);
    tmem_relinquish();
  }
  griddep_wait();
  griddep_launch();
  const int t0 = a.chunk_t0[chunk], nval = a.chunk_n[chunk];
  const auto* qp = static_cast<const __nv_bfloat16*>(L.q) + long(t0) * L.ldq + long(g) * L.N;
  const auto* kp = static_cast<const __nv_bfloat16*>(L.k) + long(t0) * L.ldk + long(g) * L.N;
  const auto* vp = static_cast<const __nv_bfloat16*>(L.v) + long(t0) * L.ldv + long(h) * L.P + p0;
  load_tile<NH>(q_s, qp, L.ldq, L.N, nval, a.vec_q, L.silu_in);
  load_tile<NH>(k_s, kp, L.ldk, L.N, nval, a.vec_k, L.silu_in);
  fence_proxy_async_smem();
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_slot;
  const uint32_t tm_s = tmem, tm_lo = tmem + 64, tm_x = tmem + 128, tm_o = tmem + 128 + PW;
  const uint32_t qa = smem_u32(q_s), ka = smem_u32(k_s), va = smem_u32(v_s);
  if (threadIdx.x == 0) {
    constexpr uint32_t idesc_s = umma_idesc(128, 128, 1, 1, 0, 0);
#pragma unroll
    for (int k = 0; k < NH * 4; ++k) {
      const uint32_t off = (k >> 2) * HALF + (k & 3) * 32;
      umma_f16(tm_s, umma_desc_k_sw128(qa + off), umma_desc_k_sw128(ka + off), idesc_s, k ? 1u : 0u);
    }
    umma_commit(s_done);
  }
  __syncwarp();
  // values and the state in front of the chunk while the scores are computed
  load_tile<PH>(v_s, vp, L.ldv, L.P - p0, nval, a.vec_v, L.silu_in);
  {
    const float* S0 = a.dS + ((long(chunk) * L.H + h) * L.P + p0) * L.N;
    auto put = [&](int row, int c8, float (&v)[8]) {
      const int off = (c8 >> 3) * SHALF + row * 128 + (((c8 & 7) ^ (row & 7)) << 4);
      *reinterpret_cast<uint4*>(sh_s + off) = split8(v);
      *reinterpret_cast<uint4*>(sl_s + off) = pack8(v);
    };
    constexpr int IT = PW * NH * 8 / 256, B = IT < 4 ? IT : 4;       // B pieces of 32 bytes in flight per thread
    if (L.N % 8 == 0) {
#pragma unroll
      for (int i0 = 0; i0 < IT; i0 += B) {
        float4 f[B][2];
#pragma unroll
        for (int i = 0; i < B; ++i) {
          const int e = threadIdx.x + 256 * (i0 + i), row = e / (NH * 8), col = (e % (NH * 8)) * 8;
          f[i][0] = f[i][1] = make_float4(0.f, 0.f, 0.f, 0.f);
          if (p0 + row < L.P && col < L.N) {
            const float4* src = reinterpret_cast<const float4*>(S0 + long(row) * L.N + col);
            f[i][0] = src[0];
            f[i][1] = src[1];
          }
        }
#pragma unroll
        for (int i = 0; i < B; ++i) {
          const int e = threadIdx.x + 256 * (i0 + i);
          float v[8] = {f[i][0].x, f[i][0].y, f[i][0].z, f[i][0].w, f[i][1].x, f[i][1].y, f[i][1].z, f[i][1].w};
          put(e / (NH * 8), e % (NH * 8), v);
        }
      }
    } else {
#pragma unroll 1
      for (int e = threadIdx.x; e < PW * NH * 8; e += 256) {
        const int row = e / (NH * 8), col = (e % (NH * 8)) * 8;
        float v[8];
#pragma unroll
        for (int j = 0; j < 8; ++j) v[j] = (p0 + row < L.P && col + j < L.N) ? S0[long(row) * L.N + col + j] : 0.f;
        put(row, col >> 3, v);
      }
    }
  }
  chunk_decay(a, h, t0, nval, cs, ws, tmp);
  bool ok = mbar_wait(s_done, 0, abort_flag);
  if (!ok) { *abort_flag = 1; atomicCAS(a.status, 0, ST_TIMEOUT_TMEM_FULL | SITE_CHUNK_SCORES); }
  __syncwarp();
  tc_fence_after();
  const int row = (warp & 3) * 32 + lane;                 // token of the chunk
  const uint32_t lane_off = uint32_t((warp & 3) * 32) << 16;
  const int wg = warp >> 2;                               // warpgroup: half of the columns
  const float ci = cs[row];
  // decayed scores: both warpgroups read their half of the columns before either writes over them
  uint32_t hi[32], lo[32];
#pragma unroll
  for (int b = 0; b < 2; ++b) {
    const int c = wg * 64 + b * 32;
    uint32_t r[32];
    tmem_ld32(tm_s + lane_off + c, r);
    tmem_ld_wait();
#pragma unroll
    for (int j = 0; j < 32; j += 2) {
      float x[2];
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int t = c + j + e;
        x[e] = t <= row ? __uint_as_float(r[j + e]) * exp2f(ci - cs[t]) * ws[t] : 0.f;
      }
      const uint32_t ph = pack_bf16x2(x[0], x[1]);
      const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&ph));
      hi[b * 16 + j / 2] = ph;
      lo[b * 16 + j / 2] = pack_bf16x2(x[0] - f.x, x[1] - f.y);
    }
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
#pragma unroll
  for (int b = 0; b < 2; ++b) {
    tmem_st16(tm_s + lane_off + wg * 32 + b * 16, *reinterpret_cast<uint32_t(*)[16]>(&hi[b * 16]));
    tmem_st16(tm_lo + lane_off + wg * 32 + b * 16, *reinterpret_cast<uint32_t(*)[16]>(&lo[b * 16]));
  }
  tmem_st_wait();
  fence_proxy_async_smem();
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  if (threadIdx.x == 0) {
    constexpr uint32_t idesc_x = umma_idesc(128, PW, 1, 1, 0, 0);
    constexpr uint32_t idesc_o = umma_idesc(128, PW, 1, 1, 0, 1);
    const uint32_t sh = smem_u32(sh_s), sl = smem_u32(sl_s);
#pragma unroll
    for (int k = 0; k < C / 16; ++k) {
      const uint64_t bd = umma_desc_mn_sw128(va + k * 16 * 128, HALF, 1024);
      umma_f16_ts(tm_o, tm_s + k * 8, bd, idesc_o, k ? 1u : 0u);
      umma_f16_ts(tm_o, tm_lo + k * 8, bd, idesc_o, 1u);
    }
#pragma unroll
    for (int k = 0; k < NH * 4; ++k) {
      const uint64_t ad = umma_desc_k_sw128(qa + (k >> 2) * HALF + (k & 3) * 32);
      const uint32_t off = (k >> 2) * SHALF + (k & 3) * 32;
      umma_f16(tm_x, ad, umma_desc_k_sw128(sh + off), idesc_x, k ? 1u : 0u);
      umma_f16(tm_x, ad, umma_desc_k_sw128(sl + off), idesc_x, 1u);
    }
    umma_commit(o_done);
  }
  __syncwarp();
  ok = mbar_wait(o_done, 0, abort_flag);
  if (!ok) { *abort_flag = 1; atomicCAS(a.status, 0, ST_TIMEOUT_TMEM_FULL | SITE_CHUNK_OUTPUT); }
  __syncwarp();
  tc_fence_after();
  if (__all_sync(0xffffffffu, ok)) {
    const float ei = exp2f(ci);
    const float Dh = L.D ? L.D[h] : 0.f;
    const long t = t0 + row;
    __nv_bfloat16* orow = static_cast<__nv_bfloat16*>(L.out) + t * L.ldo + long(h) * L.P + p0;
    const __nv_bfloat16* zrow = L.z ? static_cast<const __nv_bfloat16*>(L.z) + t * L.ldz + long(h) * L.P + p0 : nullptr;
    const __nv_bfloat16* vrow = vp + long(row) * L.ldv;
#pragma unroll 1
    for (int c = wg * (PW / 2); c < (wg + 1) * (PW / 2); c += 32) {
      uint32_t x[32], o[32];
      tmem_ld32(tm_x + lane_off + c, x);
      tmem_ld32(tm_o + lane_off + c, o);
      tmem_ld_wait();
      if (row < nval) {
#pragma unroll
        for (int b = 0; b < 4; ++b) {
          const int col = c + b * 8;
          float y[8], z[8], vv[8];
          if (p0 + col >= L.P) continue;
          if (L.D) load8(vrow, col, L.P - p0, true, a.vec_v, L.silu_in, vv);
          if (zrow) load8(zrow, col, L.P - p0, true, a.vec_o, true, z);
#pragma unroll
          for (int j = 0; j < 8; ++j) {
            y[j] = fmaf(ei, __uint_as_float(x[b * 8 + j]), __uint_as_float(o[b * 8 + j]));
            if (L.D) y[j] = fmaf(Dh, vv[j], y[j]);
            if (zrow) y[j] *= z[j];
          }
          if (a.vec_o && p0 + col + 8 <= L.P) {
            *reinterpret_cast<uint4*>(orow + col) = pack8(y);
          } else {
#pragma unroll
            for (int j = 0; j < 8; ++j)
              if (p0 + col + j < L.P) orow[col + j] = __float2bfloat16(y[j]);
          }
        }
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem, TM_COLS);
  }
}

template <int NH, int PH>
int launch_np(const ChunkArgs& a, int n_chunks, const int* seq_chunk0, const int* seq_nchunk, cudaStream_t s) {
  constexpr int SA = states_smem<NH, PH>(), SC = output_smem<NH, PH>();
  static_assert(SC <= 227 * 1024, "shared memory budget");
  auto ks = chunk_states_kernel<NH, PH>;
  auto ko = chunk_output_kernel<NH, PH>;
  static bool attr = false;
  if (!attr) {
    if (cudaFuncSetAttribute(ks, cudaFuncAttributeMaxDynamicSharedMemorySize, SA) != cudaSuccess ||
        cudaFuncSetAttribute(ko, cudaFuncAttributeMaxDynamicSharedMemorySize, SC) != cudaSuccess)
      return 1;
    attr = true;
  }
  const LinScanArgs& L = a.L;
  const dim3 grid(n_chunks, L.H, (L.P + PH * 64 - 1) / (PH * 64));
  if (launch_pdl(ks, grid, dim3(256), SA, s, a) != cudaSuccess) return 1;
  const long PN = long(L.P) * L.N;
  const int vec = L.N % 4 == 0 ? 4 : 1;
  const dim3 gc(unsigned((PN + 256 * vec - 1) / (256 * vec)), L.H, L.n_seqs);
  if ((vec == 4 ? launch_pdl(chunk_carry_kernel<4>, gc, dim3(256), 0, s, a, seq_chunk0, seq_nchunk)
                : launch_pdl(chunk_carry_kernel<1>, gc, dim3(256), 0, s, a, seq_chunk0, seq_nchunk)) != cudaSuccess)
    return 1;
  return launch_pdl(ko, grid, dim3(256), SC, s, a) != cudaSuccess;
}

}  // namespace

bool linear_chunk_ok(int N, int P) { return N >= 1 && N <= 128 && P >= 1 && P <= 1024; }

size_t linear_chunk_scratch_bytes(int n_chunks, int H, int N, int P) {
  return size_t(n_chunks) * H * (size_t(N) * P + 1) * 4 + 256;
}

int linear_chunk_launch(const LinScanArgs& L, const int* chunk_t0, const int* chunk_n, const int* chunk_seq, int n_chunks,
                        const int* seq_chunk0, const int* seq_nchunk, void* scratch, int* status, cudaStream_t s) {
  (void)chunk_seq;
  if (L.n_seqs <= 0 || n_chunks <= 0) return 0;
  if (!linear_chunk_ok(L.N, L.P) || L.G <= 0 || L.H % L.G || L.H > 65535 || L.n_seqs > 65535) return 1;
  ChunkArgs a{};
  a.L = L;
  a.chunk_t0 = chunk_t0; a.chunk_n = chunk_n; a.status = status;
  a.dS = static_cast<float*>(scratch);
  a.gC = a.dS + size_t(n_chunks) * L.H * L.N * L.P;
  auto al = [](const void* p, long ld, int w) { return reinterpret_cast<uintptr_t>(p) % 16 == 0 && ld % 8 == 0 && w % 8 == 0; };
  a.vec_q = al(L.q, L.ldq, L.N);
  a.vec_k = al(L.k, L.ldk, L.N);
  a.vec_v = al(L.v, L.ldv, L.P);
  a.vec_o = al(L.out, L.ldo, L.P) && (!L.z || al(L.z, L.ldz, L.P));
  if (L.N <= 64) return L.P <= 64 ? launch_np<1, 1>(a, n_chunks, seq_chunk0, seq_nchunk, s)
                                  : launch_np<1, 2>(a, n_chunks, seq_chunk0, seq_nchunk, s);
  return L.P <= 64 ? launch_np<2, 1>(a, n_chunks, seq_chunk0, seq_nchunk, s)
                   : launch_np<2, 2>(a, n_chunks, seq_chunk0, seq_nchunk, s);
}

}  // namespace lb
