// Chunked form of the HGRN2 state on tcgen05 (bf16 activations, prompt-sized steps):
//   F_t = lower + (1 - lower) sigmoid(f_t + b) (per key channel),  S_t = diag(F_t) S_(t-1) + (1 - F_t) v_t^T,  o_t = S_t^T silu(q_t)
// In chunks of C = 128 tokens, with F_(i..j] the product of the gates of tokens i + 1 .. j:
//   dS   = sum_j (F_(j..C] (1 - F_j)) v_j^T                       STATES kernel, one CTA per (chunk, head)
//   S_0' = F_(0..C] S_0 + dS                                      CARRY kernel, elementwise over the chunks of a sequence
//   o_i  = S_0^T (F_(0..i] q_i) + sum_{j <= i} A_ij v_j           OUTPUT kernel, one CTA per (chunk, head)
//   A_ij = q_i . (F_(j..i] (1 - F_j))
// A gate that is a vector does not factor out of A. Between two halves of a block of 2 s tokens it does, with the boundary b
// between them as reference: A_ij = (F_(b..i] q_i) . (F_(j..b] (1 - F_j)) for j <= b < i. So A is put together from such
// products for s = 64, 32, 16, 8 (all blocks of a size in one 128 x 128 product, of which only the blocks below the diagonal
// are read) and, inside blocks of 8 tokens, from inner products on FMA units. All products of gates run forward in time, each
// factor at most 1: no quotient and no logarithm of a gate appears, and gates near 0 and near 1 keep their accuracy.
//
// A thread owns two neighbouring channels of 16 tokens; what a level or the carry needs from other segments of the same channels
// are their total products, shared once. The state between chunks stays fp32; whatever enters a contraction beside the bf16
// projections and the activated queries (decayed writes, A, the state) is split into two bf16 terms, so it contributes with
// about 16 bits. The norm per head ends the OUTPUT kernel.
#include "act_type.cuh"
#include "common.cuh"
#include "layers.h"

namespace lb {
namespace {

constexpr int C = 128;                    // tokens per chunk
constexpr int HALF = C * 128;             // bytes of one 64-column half of a 128-row tile
constexpr int SEG = 16, SEGS = C / SEG;   // tokens of a thread, segments of a chunk

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

struct ForgetChunkArgs {
  ForgetScanArgs L;
  const int* chunk_t0; const int* chunk_n;
  float* dS;                              // [chunks, H, P, N]: chunk contributions, then the state in front of each chunk
  float* gC;                              // [chunks, H, N]: product of the chunk's gates
  int pair_q, pair_f, vec_v, vec_o;       // 4-byte pairs / 16-byte vectors are aligned
  int* status;
};

__device__ __forceinline__ float sigmoid_fast(float z) { return __fdividef(1.f, 1.f + __expf(-z)); }

__device__ __forceinline__ float2 bf2(uint32_t u) {
  return make_float2(__uint_as_float(u << 16), __uint_as_float(u & 0xffff0000u));
}
// columns c, c + 1 of a row (zero from `width` on)
__device__ __forceinline__ uint32_t ld_pair(const __nv_bfloat16* row, int c, int width, bool pair) {
  if (pair && c + 1 < width) return __ldg(reinterpret_cast<const unsigned int*>(row + c));
  uint32_t u = 0;
  if (c < width) u = __bfloat16_as_ushort(row[c]);
  if (c + 1 < width) u |= uint32_t(__bfloat16_as_ushort(row[c + 1])) << 16;
  return u;
}
// byte offset of column pair p of a row in a K-major tile of 64-column halves, 128-byte swizzle
__device__ __forceinline__ int pair_off(int row, int p) {
  return (p >> 5) * HALF + row * 128 + ((((p & 31) >> 2) ^ (row & 7)) << 4) + (p & 3) * 4;
}
// high bf16 parts and remainders of two values
__device__ __forceinline__ void split2(float x, float y, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16x2(x, y);
  const float2 f = bf2(hi);
  lo = pack_bf16x2(x - f.x, y - f.y);
}

// What a thread writes per token of its segment: 1 - F of its two channels (0 past the chunk's tokens).
__device__ __forceinline__ void load_writes(const ForgetChunkArgs& a, int h, int t0, int nval, int p, int seg, float2 (&w)[SEG]) {
  const ForgetScanArgs& L = a.L;
  const int c = 2 * p;
  const auto* fp = static_cast<const __nv_bfloat16*>(L.f) + long(t0 + seg * SEG) * L.ldf + long(h) * L.N;
  uint32_t raw[SEG];
#pragma unroll
  for (int i = 0; i < SEG; ++i) raw[i] = seg * SEG + i < nval ? ld_pair(fp + i * L.ldf, c, L.N, a.pair_f) : 0u;
  float2 b = make_float2(0.f, 0.f), open = b;               // bias, 1 - lower (0 past the head's channels)
  if (c < L.N) { b.x = L.f_b[h * L.N + c]; open.x = 1.f - L.lower[h * L.N + c]; }
  if (c + 1 < L.N) { b.y = L.f_b[h * L.N + c + 1]; open.y = 1.f - L.lower[h * L.N + c + 1]; }
#pragma unroll
  for (int i = 0; i < SEG; ++i) {
    const float2 z = bf2(raw[i]);
    const bool in = seg * SEG + i < nval;
    w[i].x = in ? open.x * sigmoid_fast(-(z.x + b.x)) : 0.f;
    w[i].y = in ? open.y * sigmoid_fast(-(z.y + b.y)) : 0.f;
  }
}
__device__ __forceinline__ float2 total_of(const float2 (&w)[SEG]) {
  float2 g = make_float2(1.f, 1.f);
#pragma unroll
  for (int i = 0; i < SEG; ++i) { g.x *= 1.f - w[i].x; g.y *= 1.f - w[i].y; }
  return g;
}
// product of the totals of segments lo .. hi - 1 of channel pair p
template <int PAIRS>
__device__ __forceinline__ float2 totals(const float2* g_s, int p, int lo, int hi) {
  float2 m = make_float2(1.f, 1.f);
  for (int s = lo; s < hi; ++s) {
    const float2 g = g_s[s * PAIRS + p];
    m.x *= g.x;
    m.y *= g.y;
  }
  return m;
}

// Values of the chunk as a tile [128 tokens][PH * 64 columns]
template <int PH, int NT>
__device__ __forceinline__ void load_values(const ForgetChunkArgs& a, int h, int t0, int nval, uint8_t* dst) {
  const ForgetScanArgs& L = a.L;
  const auto* vp = static_cast<const __nv_bfloat16*>(L.v) + long(t0) * L.ldv + long(h) * L.P;
  constexpr int IT = C * PH * 8 / NT;
  uint4 raw[IT];
#pragma unroll
  for (int i = 0; i < IT; ++i) {
    const int e = threadIdx.x + NT * i, row = e / (PH * 8), c = (e % (PH * 8)) * 8;
    raw[i] = make_uint4(0u, 0u, 0u, 0u);
    if (row >= nval || c >= L.P) continue;
    const __nv_bfloat16* src = vp + long(row) * L.ldv;
    if (a.vec_v) {
      raw[i] = __ldg(reinterpret_cast<const uint4*>(src + c));
    } else {
      raw[i].x = ld_pair(src, c, L.P, false); raw[i].y = ld_pair(src, c + 2, L.P, false);
      raw[i].z = ld_pair(src, c + 4, L.P, false); raw[i].w = ld_pair(src, c + 6, L.P, false);
    }
  }
#pragma unroll
  for (int i = 0; i < IT; ++i) {
    const int e = threadIdx.x + NT * i, row = e / (PH * 8), c8 = e % (PH * 8);
    *reinterpret_cast<uint4*>(dst + (c8 >> 3) * HALF + row * 128 + (((c8 & 7) ^ (row & 7)) << 4)) = raw[i];
  }
}

// ---------------------------------------------------------------------------------------------------------------
// STATES: dS[p, n] = sum_j v_j[p] (F_(j..C] (1 - F_j))[n]; A = V^T (MN-major), B = decayed writes (MN-major)
// ---------------------------------------------------------------------------------------------------------------
template <int NH, int PH>
constexpr int states_smem() { return (PH + 2 * NH) * HALF + SEGS * NH * 32 * 8 + 1024 + 64; }

template <int NH, int PH>
__global__ void __launch_bounds__(NH * 256) forget_states_kernel(const ForgetChunkArgs a) {
  constexpr int NT = NH * 256, PAIRS = NH * 32;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* v_s = smem;
  uint8_t* kh_s = v_s + PH * HALF;
  uint8_t* kl_s = kh_s + NH * HALF;
  float2* g_s = reinterpret_cast<float2*>(kl_s + NH * HALF);             // [SEGS][PAIRS]
  uint64_t* done = reinterpret_cast<uint64_t*>(g_s + SEGS * PAIRS);
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(done + 1);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  const ForgetScanArgs& L = a.L;
  const int chunk = blockIdx.x, h = blockIdx.y;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int p = threadIdx.x % PAIRS, seg = threadIdx.x / PAIRS;
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
  load_values<PH, NT>(a, h, t0, nval, v_s);
  {
    float2 w[SEG];
    load_writes(a, h, t0, nval, p, seg, w);
    g_s[seg * PAIRS + p] = total_of(w);
    __syncthreads();
    float2 m = totals<PAIRS>(g_s, p, seg + 1, SEGS);
#pragma unroll
    for (int i = SEG - 1; i >= 0; --i) {
      const int off = pair_off(seg * SEG + i, p);
      uint32_t hi, lo;
      split2(w[i].x * m.x, w[i].y * m.y, hi, lo);
      *reinterpret_cast<uint32_t*>(kh_s + off) = hi;
      *reinterpret_cast<uint32_t*>(kl_s + off) = lo;
      m.x *= 1.f - w[i].x;
      m.y *= 1.f - w[i].y;
    }
    if (seg == 0) {                        // (the product now spans the chunk)
      float* g = a.gC + (long(chunk) * L.H + h) * L.N + 2 * p;
      if (2 * p < L.N) g[0] = m.x;
      if (2 * p + 1 < L.N) g[1] = m.y;
    }
  }
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
  }
  __syncwarp();
  const bool ok = mbar_wait(done, 0, abort_flag);
  if (!ok) { *abort_flag = 1; atomicCAS(a.status, 0, ST_TIMEOUT_TMEM_FULL | SITE_FORGET_STATES); }
  __syncwarp();
  tc_fence_after();
  if (__all_sync(0xffffffffu, ok)) {
    const int v = (warp & 3) * 32 + lane, c = (warp >> 2) * 32;          // value column; a warpgroup per 32 channels
    const bool v_ok = v < PH * 64 && v < L.P;
    float* dst = a.dS + ((long(chunk) * L.H + h) * L.P + v) * L.N;
    uint32_t r[32];
    tmem_ld32(tmem + (uint32_t((warp & 3) * 32) << 16) + c, r);
    tmem_ld_wait();
    if (v_ok) {
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
__global__ void __launch_bounds__(256) forget_carry_kernel(const ForgetChunkArgs a, const int* __restrict__ seq_chunk0,
                                                           const int* __restrict__ seq_nchunk) {
  griddep_wait();
  griddep_launch();
  const ForgetScanArgs& L = a.L;
  const int h = blockIdx.y, seq = blockIdx.z, slot = L.slots[seq];
  const long PN = long(L.P) * L.N, e = (long(blockIdx.x) * 256 + threadIdx.x) * VEC;
  const int n = seq_nchunk[seq], c0 = seq_chunk0[seq];
  if (e >= PN || n <= 0 || slot < 0) return;
  const int ch = int(e % L.N);                                           // first key channel
  float* st = L.state + (long(slot) * L.H + h) * PN + e;
  float s[VEC];
  ld_vec<VEC>(st, s);
  constexpr int U = 4;                      // contributions in flight
  for (int b = 0; b < n; b += U) {
    float d[U][VEC], g[U][VEC];
#pragma unroll
    for (int u = 0; u < U; ++u)
      if (b + u < n) {
        const long row = long(c0 + b + u) * L.H + h;
        ld_vec<VEC>(a.dS + row * PN + e, d[u]);
        ld_vec<VEC>(a.gC + row * L.N + ch, g[u]);
      }
#pragma unroll
    for (int u = 0; u < U; ++u)
      if (b + u < n) {
        st_vec<VEC>(a.dS + (long(c0 + b + u) * L.H + h) * PN + e, s);
#pragma unroll
        for (int j = 0; j < VEC; ++j) s[j] = fmaf(g[u][j], s[j], d[u][j]);
      }
  }
  if (L.write_state) st_vec<VEC>(st, s);
}

// ---------------------------------------------------------------------------------------------------------------
// OUTPUT
// ---------------------------------------------------------------------------------------------------------------
// One level: halves of S tokens. Rows of a right half get their decayed queries in the q tile, rows of a left half their
// decayed writes in the k tiles; the other rows of either tile are not read back.
template <int S, int PAIRS>
__device__ __forceinline__ void build_level(const float2 (&q)[SEG], const float2 (&w)[SEG], const float2* g_s, int p, int seg,
                                            uint8_t* q_s, uint8_t* kh_s, uint8_t* kl_s) {
  auto put_q = [&](int i, float2 m) {
    *reinterpret_cast<uint32_t*>(q_s + pair_off(seg * SEG + i, p)) = pack_bf16x2(q[i].x * m.x, q[i].y * m.y);
  };
  auto put_k = [&](int i, float2 m) {
    const int off = pair_off(seg * SEG + i, p);
    uint32_t hi, lo;
    split2(w[i].x * m.x, w[i].y * m.y, hi, lo);
    *reinterpret_cast<uint32_t*>(kh_s + off) = hi;
    *reinterpret_cast<uint32_t*>(kl_s + off) = lo;
  };
  if constexpr (S >= SEG) {
    constexpr int HS = S / SEG;             // segments of a half
    const int at = seg % HS, half0 = seg - at;
    if ((seg / HS) & 1) {
      float2 m = totals<PAIRS>(g_s, p, half0, seg);
#pragma unroll
      for (int i = 0; i < SEG; ++i) {
        m.x *= 1.f - w[i].x;
        m.y *= 1.f - w[i].y;
        put_q(i, m);
      }
    } else {
      float2 m = totals<PAIRS>(g_s, p, seg + 1, half0 + HS);
#pragma unroll
      for (int i = SEG - 1; i >= 0; --i) {
        put_k(i, m);
        m.x *= 1.f - w[i].x;
        m.y *= 1.f - w[i].y;
      }
    }
  } else {
#pragma unroll
    for (int b = 0; b < SEG; b += 2 * S) {
      float2 m = make_float2(1.f, 1.f);
#pragma unroll
      for (int i = b + S - 1; i >= b; --i) {
        put_k(i, m);
        m.x *= 1.f - w[i].x;
        m.y *= 1.f - w[i].y;
      }
      m = make_float2(1.f, 1.f);
#pragma unroll
      for (int i = b + S; i < b + 2 * S; ++i) {
        m.x *= 1.f - w[i].x;
        m.y *= 1.f - w[i].y;
        put_q(i, m);
      }
    }
  }
}

template <int NH, int PH>
constexpr int output_smem() {
  return (3 * NH + PH) * HALF + 2 * NH * (PH * 64 * 128) + SEGS * NH * 32 * 8 + NH * C * 8 * 4 + 2 * NH * C * 4 + 1024 + 128;
}

template <int NH, int PH>
__global__ void __launch_bounds__(NH * 256, 1) forget_output_kernel(const ForgetChunkArgs a) {
  constexpr int NT = NH * 256, PAIRS = NH * 32, WGS = NT / 128;
  constexpr int PW = PH * 64;
  constexpr int SHALF = PW * 128;           // bytes of one 64-column half of the state tile
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* q_s = smem;
  uint8_t* kh_s = q_s + NH * HALF;
  uint8_t* kl_s = kh_s + NH * HALF;
  uint8_t* v_s = kl_s + NH * HALF;
  uint8_t* sh_s = v_s + PH * HALF;
  uint8_t* sl_s = sh_s + NH * SHALF;
  float2* g_s = reinterpret_cast<float2*>(sl_s + NH * SHALF);            // [SEGS][PAIRS] totals
  float* diag_s = reinterpret_cast<float*>(g_s + SEGS * PAIRS);          // [NH][C][8] A inside blocks of 8, a plane per 64 channels
  float* red_s = diag_s + NH * C * 8;                                    // [WGS][C] sums of squares
  uint64_t* bars = reinterpret_cast<uint64_t*>(red_s + WGS * C);         // [4] levels, [1] output
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 5);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  const ForgetScanArgs& L = a.L;
  const int chunk = blockIdx.x, h = blockIdx.y;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int p = threadIdx.x % PAIRS, seg = threadIdx.x / PAIRS;
  if (threadIdx.x == 0) {
    for (int i = 0; i < 5; ++i) mbar_init(&bars[i], 1);
    *abort_flag = 0;
    mbar_fence_init();
  }
  if (warp == 1) {
    tmem_alloc(tmem_slot, 512);
    tmem_relinquish();
  }
  griddep_wait();
  griddep_launch();
  const int t0 = a.chunk_t0[chunk], nval = a.chunk_n[chunk];
  float2 q[SEG], w[SEG];
  {
    const auto* qp = static_cast<const __nv_bfloat16*>(L.q) + long(t0 + seg * SEG) * L.ldq + long(h) * L.N;
    uint32_t raw[SEG];
#pragma unroll
    for (int i = 0; i < SEG; ++i) raw[i] = seg * SEG + i < nval ? ld_pair(qp + i * L.ldq, 2 * p, L.N, a.pair_q) : 0u;
    load_writes(a, h, t0, nval, p, seg, w);
#pragma unroll
    for (int i = 0; i < SEG; ++i) {
      const float2 z = bf2(raw[i]);
      q[i] = make_float2(z.x * sigmoid_fast(z.x), z.y * sigmoid_fast(z.y));
    }
  }
  g_s[seg * PAIRS + p] = total_of(w);
  __syncthreads();
  const uint32_t tmem = *tmem_slot;
  // high parts and remainders of A (bf16 pairs), two level accumulators, the output
  const uint32_t tm_hi = tmem, tm_lo = tmem + 64, tm_d = tmem + 128, tm_o = tmem + 384;
  const uint32_t qa = smem_u32(q_s), kh = smem_u32(kh_s), kl = smem_u32(kl_s), va = smem_u32(v_s);
  const int wq = warp & 3, wg = warp >> 2;                // 32 tokens (rows of tensor memory), warpgroup
  const uint32_t lane_off = uint32_t(wq * 32) << 16;
  bool ok = true;
  // products of a level, once all its rows are in place
  auto level_mma = [&](int lv) {
    fence_proxy_async_smem();
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    if (threadIdx.x == 0) {
      constexpr uint32_t idesc = umma_idesc(128, 128, 1, 1, 0, 0);
#pragma unroll
      for (int k = 0; k < NH * 4; ++k) {
        const uint32_t off = (k >> 2) * HALF + (k & 3) * 32;
        const uint64_t ad = umma_desc_k_sw128(qa + off);
        umma_f16(tm_d + (lv & 1) * 128, ad, umma_desc_k_sw128(kh + off), idesc, k ? 1u : 0u);
        umma_f16(tm_d + (lv & 1) * 128, ad, umma_desc_k_sw128(kl + off), idesc, 1u);
      }
      umma_commit(&bars[lv]);
    }
    __syncwarp();
  };
  auto level_wait = [&](int lv) {
    if (!mbar_wait(&bars[lv], 0, abort_flag)) {
      *abort_flag = 1;
      atomicCAS(a.status, 0, ST_TIMEOUT_TMEM_FULL | SITE_FORGET_LEVEL);
      ok = false;
    }
    __syncwarp();
    tc_fence_after();
  };
  // 32 columns of A (group g) of the warp's rows, high parts and remainders, into tensor memory
  auto store_group = [&](int g, const float (&x)[32]) {
    uint32_t hi[16], lo[16];
#pragma unroll
    for (int j = 0; j < 16; ++j) split2(x[2 * j], x[2 * j + 1], hi[j], lo[j]);
    tmem_st16(tm_hi + lane_off + g * 16, hi);
    tmem_st16(tm_lo + lane_off + g * 16, lo);
  };
  auto copy_group = [&](int g, int lv) {
    uint32_t r[32];
    float x[32];
    tmem_ld32(tm_d + (lv & 1) * 128 + lane_off + g * 32, r);
    tmem_ld_wait();
#pragma unroll
    for (int j = 0; j < 32; ++j) x[j] = __uint_as_float(r[j]);
    store_group(g, x);
  };
  const int diag_wg = wq % WGS;                           // the warpgroup that puts this warp's diagonal group together

  build_level<64, PAIRS>(q, w, g_s, p, seg, q_s, kh_s, kl_s);
  level_mma(0);
  load_values<PH, NT>(a, h, t0, nval, v_s);
  // blocks of 8 tokens: A_ij summed over the thread's channels, then over the warp's
#pragma unroll
  for (int b = 0; b < SEG; b += 8) {
    float2 c[8];                                          // decayed writes of the block's tokens, as token i sees them
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      float s[8];
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        s[j] = 0.f;
        if (j < i) {
          c[j].x *= 1.f - w[b + i].x;
          c[j].y *= 1.f - w[b + i].y;
        }
        if (j == i) c[j] = w[b + i];
        if (j <= i) s[j] = fmaf(q[b + i].x, c[j].x, q[b + i].y * c[j].y);
      }
#pragma unroll
      for (int o = 4; o > 0; o >>= 1) {                   // lane l gets sum l & 7 of four lanes each
        const bool up = lane & o;
#pragma unroll
        for (int j = 0; j < o; ++j) {
          const float send = up ? s[j] : s[j + o], keep = up ? s[j + o] : s[j];
          s[j] = keep + __shfl_xor_sync(0xffffffffu, send, o);
        }
      }
      s[0] += __shfl_xor_sync(0xffffffffu, s[0], 8);
      s[0] += __shfl_xor_sync(0xffffffffu, s[0], 16);
      if (lane < 8) diag_s[((NH == 2 ? (warp & 1) : 0) * C + seg * SEG + b + i) * 8 + lane] = s[0];
    }
  }
  level_wait(0);
  __syncthreads();                                        // the tiles are free again
  build_level<32, PAIRS>(q, w, g_s, p, seg, q_s, kh_s, kl_s);
  level_mma(1);
  // groups of columns 0 .. 63 for the rows of the right half; what lies above the diagonal is zero
#pragma unroll
  for (int g = 0; g < 4; ++g) {
    if (g % WGS != wg) continue;
    if (g < 2 && wq >= 2) copy_group(g, 0);
    if (g > wq) {
      const float zero[32] = {};
      store_group(g, zero);
    }
  }
  level_wait(1);
  __syncthreads();
  build_level<16, PAIRS>(q, w, g_s, p, seg, q_s, kh_s, kl_s);
  level_mma(2);
  if ((wq == 1 && wg == 0) || (wq == 3 && wg == 2 % WGS)) copy_group(wq - 1, 1);
  // the state in front of the chunk, high parts and remainders
  {
    const float* S0 = a.dS + (long(chunk) * L.H + h) * L.P * L.N;
    constexpr int IT = PW * NH * 8 / NT;
    auto put = [&](int row, int c8, const float (&v)[8]) {
      const int off = (c8 >> 3) * SHALF + row * 128 + (((c8 & 7) ^ (row & 7)) << 4);
      uint4 hi, lo;
      split2(v[0], v[1], hi.x, lo.x);
      split2(v[2], v[3], hi.y, lo.y);
      split2(v[4], v[5], hi.z, lo.z);
      split2(v[6], v[7], hi.w, lo.w);
      *reinterpret_cast<uint4*>(sh_s + off) = hi;
      *reinterpret_cast<uint4*>(sl_s + off) = lo;
    };
#pragma unroll
    for (int i = 0; i < IT; ++i) {
      const int e = threadIdx.x + NT * i, row = e / (NH * 8), c8 = e % (NH * 8), col = c8 * 8;
      float v[8];
#pragma unroll
      for (int j = 0; j < 8; ++j) v[j] = 0.f;
      if (row < L.P) {
        if (L.N % 8 == 0) {
          if (col < L.N) {
            const float4* src = reinterpret_cast<const float4*>(S0 + long(row) * L.N + col);
            const float4 f0 = src[0], f1 = src[1];
            v[0] = f0.x; v[1] = f0.y; v[2] = f0.z; v[3] = f0.w;
            v[4] = f1.x; v[5] = f1.y; v[6] = f1.z; v[7] = f1.w;
          }
        } else {
#pragma unroll
          for (int j = 0; j < 8; ++j)
            if (col + j < L.N) v[j] = S0[long(row) * L.N + col + j];
        }
      }
      put(row, c8, v);
    }
  }
  level_wait(2);
  float x16[16];                                          // columns 0 .. 15 of the diagonal group, for its lower half
  if (wg == diag_wg) {
    uint32_t r[16];
    tmem_ld16(tm_d + lane_off + wq * 32, r);
    tmem_ld_wait();
#pragma unroll
    for (int j = 0; j < 16; ++j) x16[j] = __uint_as_float(r[j]);
  }
  __syncthreads();
  build_level<8, PAIRS>(q, w, g_s, p, seg, q_s, kh_s, kl_s);
  level_mma(3);
  level_wait(3);
  if (wg == diag_wg) {
    uint32_t r[32];
    float x[32];
    tmem_ld32(tm_d + 128 + lane_off + wq * 32, r);
    tmem_ld_wait();
    const int blk = lane >> 3;                            // block of 8 tokens inside the group
    const float* dr = diag_s + (wq * 32 + lane) * 8;
    float d[8];
    {
      const float4 d0 = *reinterpret_cast<const float4*>(dr), d1 = *reinterpret_cast<const float4*>(dr + 4);
      d[0] = d0.x; d[1] = d0.y; d[2] = d0.z; d[3] = d0.w;
      d[4] = d1.x; d[5] = d1.y; d[6] = d1.z; d[7] = d1.w;
      if constexpr (NH == 2) {
        const float4 e0 = *reinterpret_cast<const float4*>(dr + C * 8), e1 = *reinterpret_cast<const float4*>(dr + C * 8 + 4);
        d[0] += e0.x; d[1] += e0.y; d[2] += e0.z; d[3] += e0.w;
        d[4] += e1.x; d[5] += e1.y; d[6] += e1.z; d[7] += e1.w;
      }
    }
#pragma unroll
    for (int c = 0; c < 32; ++c) {
      const int cb = c >> 3;
      float v = 0.f;
      if (cb == blk) v = (c & 7) <= (lane & 7) ? d[c & 7] : 0.f;
      else if ((cb == 0 && blk == 1) || (cb == 2 && blk == 3)) v = __uint_as_float(r[c]);
      else if (cb < 2 && blk >= 2) v = x16[c & 15];
      x[c] = v;
    }
    store_group(wq, x);
  }
  __syncthreads();                                        // the q tile is free
  {
    float2 m = totals<PAIRS>(g_s, p, 0, seg);             // queries decayed from the chunk's first token on
#pragma unroll
    for (int i = 0; i < SEG; ++i) {
      m.x *= 1.f - w[i].x;
      m.y *= 1.f - w[i].y;
      *reinterpret_cast<uint32_t*>(q_s + pair_off(seg * SEG + i, p)) = pack_bf16x2(q[i].x * m.x, q[i].y * m.y);
    }
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
    for (int k = 0; k < NH * 4; ++k) {
      const uint64_t ad = umma_desc_k_sw128(qa + (k >> 2) * HALF + (k & 3) * 32);
      const uint32_t off = (k >> 2) * SHALF + (k & 3) * 32;
      umma_f16(tm_o, ad, umma_desc_k_sw128(sh + off), idesc_x, k ? 1u : 0u);
      umma_f16(tm_o, ad, umma_desc_k_sw128(sl + off), idesc_x, 1u);
    }
#pragma unroll
    for (int k = 0; k < C / 16; ++k) {
      const uint64_t bd = umma_desc_mn_sw128(va + k * 16 * 128, HALF, 1024);
      umma_f16_ts(tm_o, tm_hi + k * 8, bd, idesc_o, 1u);
      umma_f16_ts(tm_o, tm_lo + k * 8, bd, idesc_o, 1u);
    }
    umma_commit(&bars[4]);
  }
  __syncwarp();
  if (!mbar_wait(&bars[4], 0, abort_flag)) {
    *abort_flag = 1;
    atomicCAS(a.status, 0, ST_TIMEOUT_TMEM_FULL | SITE_FORGET_OUTPUT);
    ok = false;
  }
  __syncwarp();
  tc_fence_after();
  // norm over the head's value columns (those past P are zeros): 32 columns per warp, sums joined through shared memory
  const int row = wq * 32 + lane;
  constexpr int GROUPS = PW / 32, PER = (GROUPS + WGS - 1) / WGS;        // column groups, and of them per warpgroup
  float y[PER][32];
  float ss = 0.f;
  const bool all_ok = __all_sync(0xffffffffu, ok);
#pragma unroll
  for (int i = 0; i < PER; ++i) {
    const int g = wg + i * WGS;
    if (all_ok && g < GROUPS) {
      uint32_t r[32];
      tmem_ld32(tm_o + lane_off + g * 32, r);
      tmem_ld_wait();
#pragma unroll
      for (int j = 0; j < 32; ++j) {
        y[i][j] = __uint_as_float(r[j]);
        ss = fmaf(y[i][j], y[i][j], ss);
      }
    }
  }
  red_s[wg * C + row] = ss;
  __syncthreads();
  ss = 0.f;
#pragma unroll
  for (int g = 0; g < WGS; ++g) ss += red_s[g * C + row];
  const float inv = L.scale / sqrtf(ss / float(L.P) + L.eps);
  if (all_ok && row < nval) {
    __nv_bfloat16* orow = static_cast<__nv_bfloat16*>(L.out) + long(t0 + row) * L.ldo + long(h) * L.P;
#pragma unroll
    for (int i = 0; i < PER; ++i) {
      const int g = wg + i * WGS;
      if (g >= GROUPS) continue;
#pragma unroll
      for (int j = 0; j < 32; j += 8) {
        const int col = g * 32 + j;
        if (col >= L.P) continue;
        float z[8];
#pragma unroll
        for (int e = 0; e < 8; ++e) z[e] = col + e < L.P ? y[i][j + e] * inv * __ldg(L.norm_w + col + e) : 0.f;
        if (a.vec_o) {
          *reinterpret_cast<uint4*>(orow + col) = make_uint4(pack_bf16x2(z[0], z[1]), pack_bf16x2(z[2], z[3]),
                                                             pack_bf16x2(z[4], z[5]), pack_bf16x2(z[6], z[7]));
        } else {
#pragma unroll
          for (int e = 0; e < 8; ++e)
            if (col + e < L.P) orow[col + e] = __float2bfloat16(z[e]);
        }
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem, 512);
  }
}

template <int NH, int PH>
int launch_np(const ForgetChunkArgs& a, int n_chunks, const int* seq_chunk0, const int* seq_nchunk, cudaStream_t s) {
  constexpr int SA = states_smem<NH, PH>(), SC = output_smem<NH, PH>();
  static_assert(SC <= 227 * 1024, "shared memory budget");
  auto ks = forget_states_kernel<NH, PH>;
  auto ko = forget_output_kernel<NH, PH>;
  static bool attr = false;
  if (!attr) {
    if (cudaFuncSetAttribute(ks, cudaFuncAttributeMaxDynamicSharedMemorySize, SA) != cudaSuccess ||
        cudaFuncSetAttribute(ko, cudaFuncAttributeMaxDynamicSharedMemorySize, SC) != cudaSuccess)
      return 1;
    attr = true;
  }
  const ForgetScanArgs& L = a.L;
  const dim3 grid(n_chunks, L.H);
  if (launch_pdl(ks, grid, dim3(NH * 256), SA, s, a) != cudaSuccess) return 1;
  const long PN = long(L.P) * L.N;
  const int vec = L.N % 4 == 0 ? 4 : 1;
  const dim3 gc(unsigned((PN + 256 * vec - 1) / (256 * vec)), L.H, L.n_seqs);
  if ((vec == 4 ? launch_pdl(forget_carry_kernel<4>, gc, dim3(256), 0, s, a, seq_chunk0, seq_nchunk)
                : launch_pdl(forget_carry_kernel<1>, gc, dim3(256), 0, s, a, seq_chunk0, seq_nchunk)) != cudaSuccess)
    return 1;
  return launch_pdl(ko, grid, dim3(NH * 256), SC, s, a) != cudaSuccess;
}

}  // namespace

bool forget_chunk_ok(int N, int P) { return N >= 1 && N <= 128 && P >= 1 && P <= 128; }

size_t forget_chunk_scratch_bytes(int n_chunks, int H, int N, int P) {
  return size_t(n_chunks) * H * (size_t(N) * P + N) * 4 + 256;
}

int forget_chunk_launch(const ForgetScanArgs& L, const int* chunk_t0, const int* chunk_n, int n_chunks, const int* seq_chunk0,
                        const int* seq_nchunk, void* scratch, int* status, cudaStream_t s) {
  if (L.n_seqs <= 0 || n_chunks <= 0) return 0;
  if (!forget_chunk_ok(L.N, L.P) || L.H < 1 || L.H > 65535 || L.n_seqs > 65535 || (reinterpret_cast<uintptr_t>(L.state) & 15))
    return 1;
  ForgetChunkArgs a{};
  a.L = L;
  a.chunk_t0 = chunk_t0; a.chunk_n = chunk_n; a.status = status;
  a.dS = static_cast<float*>(scratch);
  a.gC = a.dS + size_t(n_chunks) * L.H * L.N * L.P;
  auto al = [](const void* p, long ld, int w, int n) { return reinterpret_cast<uintptr_t>(p) % (2 * n) == 0 && ld % n == 0 && w % n == 0; };
  a.pair_q = al(L.q, L.ldq, L.N, 2);
  a.pair_f = al(L.f, L.ldf, L.N, 2);
  a.vec_v = al(L.v, L.ldv, L.P, 8);
  a.vec_o = al(L.out, L.ldo, L.P, 8);
  if (L.N <= 64) return L.P <= 64 ? launch_np<1, 1>(a, n_chunks, seq_chunk0, seq_nchunk, s)
                                  : launch_np<1, 2>(a, n_chunks, seq_chunk0, seq_nchunk, s);
  return L.P <= 64 ? launch_np<2, 1>(a, n_chunks, seq_chunk0, seq_nchunk, s)
                   : launch_np<2, 2>(a, n_chunks, seq_chunk0, seq_nchunk, s);
}

}  // namespace lb
