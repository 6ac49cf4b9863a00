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
// A thread owns two neighbouring channels of a segment of tokens; what a level or the carry needs from other segments of the same
// channels are their total products, shared once. The state between chunks stays fp32; whatever enters a contraction beside the bf16
// projections and the activated queries (decayed writes, A, the state) is split into two bf16 terms, so it contributes with
// about 16 bits. The norm per head ends the OUTPUT kernel.
#include "act_type.cuh"
#include "common.cuh"
#include "layers.h"
#include "state_cols.cuh"

namespace lb {
namespace {

constexpr int C = 128;                    // tokens per chunk
constexpr int HALF = C * 128;             // bytes of one 64-column half of a 128-row tile
constexpr int SEG = 16, SEGS = C / SEG;   // tokens of a thread, segments of a chunk

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
  int vec_q, vec_f, vec_v, vec_o;         // 16-byte vectors are aligned
  int* status;
};

__device__ __forceinline__ float sigmoid_fast(float z) {
  float e, r;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(e) : "f"(z * -1.4426950408889634f));
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(1.f + e));
  return r;
}

__device__ __forceinline__ float2 bf2(uint32_t u) {
  return make_float2(__uint_as_float(u << 16), __uint_as_float(u & 0xffff0000u));
}
// columns c, c + 1 of a row (zero from `width` on)
__device__ __forceinline__ uint32_t ld_pair(const __nv_bfloat16* row, int c, int width) {
  uint32_t u = 0;
  if (c < width) u = __bfloat16_as_ushort(row[c]);
  if (c + 1 < width) u |= uint32_t(__bfloat16_as_ushort(row[c + 1])) << 16;
  return u;
}
// 16 bytes global -> shared, zeros without `in`
__device__ __forceinline__ void cp_async16(void* dst, const void* src, bool in) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(dst)), "l"(src), "r"(in ? 16 : 0) : "memory");
}
__device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_all;" ::: "memory"); }
// A chunk's rows of a head, W8 * 8 columns (zeros past `width` and past its tokens), by asynchronous copies where rows are
// aligned; off(row, 8-column piece): byte offset of a piece.
template <int W8, int NT, typename Off>
__device__ __forceinline__ void stage_rows(uint8_t* dst, const __nv_bfloat16* src, long ld, int width, int nval, bool vec, Off off) {
#pragma unroll
  for (int i = 0; i < C * W8 / NT; ++i) {
    const int e = threadIdx.x + NT * i, row = e / W8, c8 = e % W8;
    const bool in = row < nval && c8 * 8 < width;
    const __nv_bfloat16* r = src + (in ? row * ld + c8 * 8 : 0);
    uint8_t* to = dst + off(row, c8);
    if (vec) {
      cp_async16(to, r, in);
    } else {
      uint32_t u[4];
#pragma unroll
      for (int j = 0; j < 4; ++j) u[j] = in ? ld_pair(r, 2 * j, width - c8 * 8) : 0u;
      *reinterpret_cast<uint4*>(to) = make_uint4(u[0], u[1], u[2], u[3]);
    }
  }
}
__device__ __forceinline__ int tile_off(int row, int c8) { return (c8 >> 3) * HALF + row * 128 + (((c8 & 7) ^ (row & 7)) << 4); }
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

// What a thread writes per token of its segment: 1 - F of its two channels (0 past the chunk's tokens); f_s: the staged rows.
__device__ __forceinline__ void load_writes(const ForgetChunkArgs& a, const uint32_t* f_s, int pairs, int h, int nval, int p, int seg,
                                            float2 (&w)[SEG]) {
  const ForgetScanArgs& L = a.L;
  const int c = 2 * p;
  float2 b = make_float2(0.f, 0.f), open = b;               // bias, 1 - lower (0 past the head's channels)
  if (c < L.N) { b.x = L.f_b[h * L.N + c]; open.x = 1.f - L.lower[h * L.N + c]; }
  if (c + 1 < L.N) { b.y = L.f_b[h * L.N + c + 1]; open.y = 1.f - L.lower[h * L.N + c + 1]; }
#pragma unroll
  for (int i = 0; i < SEG; ++i) {
    const float2 z = bf2(f_s[(seg * SEG + i) * pairs + p]);
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

// Values of the chunk as a tile [128 tokens][PH * 64 columns] (asynchronous copies: wait for them)
template <int PH, int NT>
__device__ __forceinline__ void load_values(const ForgetChunkArgs& a, int h, int t0, int nval, uint8_t* dst) {
  const ForgetScanArgs& L = a.L;
  stage_rows<PH * 8, NT>(dst, static_cast<const __nv_bfloat16*>(L.v) + long(t0) * L.ldv + long(h) * L.P, L.ldv, L.P, nval, a.vec_v,
                         tile_off);
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
  uint8_t* smem = smem_raw + ((1024u - (smem_u32(smem_raw) & 1023u)) & 1023u);   // (an offset: the address space stays known)
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
  stage_rows<NH * 8, NT>(kl_s, static_cast<const __nv_bfloat16*>(L.f) + long(t0) * L.ldf + long(h) * L.N, L.ldf, L.N, nval, a.vec_f,
                         [](int row, int c8) { return row * (NH * 128) + c8 * 16; });
  load_values<PH, NT>(a, h, t0, nval, v_s);
  {
    cp_async_wait();
    __syncthreads();
    float2 w[SEG];
    load_writes(a, reinterpret_cast<const uint32_t*>(kl_s), PAIRS, h, nval, p, seg, w);
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
// OUTPUT: a thread owns two neighbouring channels of 8 tokens, with -(1 - F) in registers: a product moves on by one fused
// multiply-add. The code of a level is the same for all of them (a loop, so that it stays in the instruction cache).
// ---------------------------------------------------------------------------------------------------------------
constexpr int OSEG = 8, OSEGS = C / OSEG;
constexpr int imax(int a, int b) { return a > b ? a : b; }

// Levels: q tile | high parts | remainders. Beside them first 1 - F (fp32) and the queries' projections (bf16) by token for the blocks of 8,
// later the values and the state in front of the chunk.
template <int NH, int PH>
struct OutSmem {
  static constexpr int TILES = 3 * NH * HALF;
  static constexpr int SHALF = PH * 64 * 128;                 // bytes of one 64-column half of the state tile
  static constexpr int SHARE = imax(PH * HALF + 2 * NH * SHALF, NH * 64 * C * 4 + NH * HALF);
  static constexpr int BYTES = TILES + SHARE + OSEGS * NH * 32 * 8 + C * 8 * 4 + NH * 4 * C * 4 + 1024 + 128;
  static_assert(BYTES <= 227 * 1024, "shared memory budget");
};

__device__ __forceinline__ void tmem_ld8(uint32_t taddr, uint32_t (&r)[8]) {
  asm volatile("tcgen05.ld.sync.aligned.32x32b.x8.b32 {%0, %1, %2, %3, %4, %5, %6, %7}, [%8];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7])
               : "r"(taddr) : "memory");
}
__device__ __forceinline__ void tmem_st4(uint32_t taddr, const uint32_t (&r)[4]) {
  asm volatile("tcgen05.st.sync.aligned.32x32b.x4.b32 [%0], {%1, %2, %3, %4};"
               ::"r"(taddr), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]) : "memory");
}

template <int NH, int PH>
__global__ void __launch_bounds__(NH * 512, 1) forget_output_kernel(const ForgetChunkArgs a) {
  using Sm = OutSmem<NH, PH>;
  constexpr int NT = NH * 512, PAIRS = NH * 32, WGS = NT / 128, PW = PH * 64, SHALF = Sm::SHALF;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = smem_raw + ((1024u - (smem_u32(smem_raw) & 1023u)) & 1023u);   // (an offset: the address space stays known)
  uint8_t* q_s = smem;
  uint8_t* kh_s = q_s + NH * HALF;
  uint8_t* kl_s = kh_s + NH * HALF;
  uint8_t* share = smem + Sm::TILES;
  float* nw_s = reinterpret_cast<float*>(share);                         // [C][NH * 64] -(1 - F)
  uint32_t* qb_s = reinterpret_cast<uint32_t*>(share + NH * 64 * C * 4); // [C][PAIRS] queries before silu, pairs of bf16
  uint8_t* v_s = share;
  uint8_t* sh_s = v_s + PH * HALF;
  uint8_t* sl_s = sh_s + NH * SHALF;
  uint64_t* g_s = reinterpret_cast<uint64_t*>(share + Sm::SHARE);        // [OSEGS][PAIRS] products of the segments' gates
  float* diag_s = reinterpret_cast<float*>(g_s + OSEGS * PAIRS);         // [C][8] A inside blocks of 8
  float* red_s = diag_s + C * 8;                                         // [WGS][C] sums of squares
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
  uint64_t q[OSEG], nw[OSEG];
  {
    auto rows = [](int row, int c8) { return row * (NH * 128) + c8 * 16; };
    stage_rows<NH * 8, NT>(reinterpret_cast<uint8_t*>(qb_s), static_cast<const __nv_bfloat16*>(L.q) + long(t0) * L.ldq + long(h) * L.N,
                           L.ldq, L.N, nval, a.vec_q, rows);
    stage_rows<NH * 8, NT>(kh_s, static_cast<const __nv_bfloat16*>(L.f) + long(t0) * L.ldf + long(h) * L.N, L.ldf, L.N, nval, a.vec_f,
                           rows);
    float2 b = make_float2(0.f, 0.f), open = b;               // bias, 1 - lower (0 past the head's channels)
    if (2 * p < L.N) { b.x = L.f_b[h * L.N + 2 * p]; open.x = 1.f - L.lower[h * L.N + 2 * p]; }
    if (2 * p + 1 < L.N) { b.y = L.f_b[h * L.N + 2 * p + 1]; open.y = 1.f - L.lower[h * L.N + 2 * p + 1]; }
    cp_async_wait();
    __syncthreads();
    const uint32_t* f_s = reinterpret_cast<const uint32_t*>(kh_s);
    uint64_t g = p2(1.f, 1.f);
#pragma unroll
    for (int i = 0; i < OSEG; ++i) {
      const int t = seg * OSEG + i;
      const float2 z = bf2(qb_s[t * PAIRS + p]), e = bf2(f_s[t * PAIRS + p]);
      const float qx = z.x * sigmoid_fast(z.x), qy = z.y * sigmoid_fast(z.y);
      q[i] = p2(qx, qy);
      nw[i] = t < nval ? p2(-open.x * sigmoid_fast(-(e.x + b.x)), -open.y * sigmoid_fast(-(e.y + b.y))) : 0ull;
      g = fma2(nw[i], g, g);
      *reinterpret_cast<uint64_t*>(nw_s + t * (NH * 64) + 2 * p) = nw[i];
    }
    g_s[seg * PAIRS + p] = g;
  }
  __syncthreads();
  const uint32_t tmem = *tmem_slot;
  // high parts and remainders of A (bf16 pairs), two level accumulators, the output
  const uint32_t tm_hi = tmem, tm_lo = tmem + 64, tm_d = tmem + 128, tm_o = tmem + 384;
  const uint32_t qa = smem_u32(q_s), kh = smem_u32(kh_s), kl = smem_u32(kl_s);
  const int wq = warp & 3, wg = warp >> 2;                // 32 tokens (rows of tensor memory), warpgroup
  const uint32_t lane_off = uint32_t(wq * 32) << 16;
  const uint32_t tile0 = (p >> 5) * HALF + seg * OSEG * 128 + ((p & 31) >> 2) * 16 + (p & 3) * 4;   // token 0 of the segment
  auto at = [&](int i) { return (tile0 ^ (i << 4)) + i * 128; };          // (swizzle: 16-byte chunk xor token mod 8)
  auto product = [&](int lo, int hi) {                    // of the gates of segments lo .. hi - 1
    uint64_t m = p2(1.f, 1.f);
#pragma unroll 1
    for (int s = lo; s < hi; ++s) m = mul2(m, g_s[s * PAIRS + p]);
    return m;
  };
  auto put_queries = [&](uint64_t m) {                    // decayed from the front of the segment on, m in front of it
#pragma unroll
    for (int i = 0; i < OSEG; ++i) {
      m = fma2(nw[i], m, m);
      float x, y;
      u2(mul2(q[i], m), x, y);
      *reinterpret_cast<uint32_t*>(q_s + at(i)) = pack_bf16x2(x, y);
    }
  };
  bool ok = true;
  auto wait = [&](int bar, int site) {                    // one warp polls; the barrier behind it is the others' wait
    if (warp == 0) {
      if (!mbar_wait(&bars[bar], 0, abort_flag)) {
        *abort_flag = 1;
        atomicCAS(a.status, 0, ST_TIMEOUT_TMEM_FULL | site);
      }
      __syncwarp();
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    ok = ok && !*abort_flag;
  };
  // eight columns of A from column c on: high parts and remainders into tensor memory
  auto store8 = [&](int c, const float (&x)[8]) {
    uint32_t hi[4], lo[4];
#pragma unroll
    for (int j = 0; j < 4; ++j) split2(x[2 * j], x[2 * j + 1], hi[j], lo[j]);
    tmem_st4(tm_hi + lane_off + c / 2, hi);
    tmem_st4(tm_lo + lane_off + c / 2, lo);
  };

#pragma unroll 1
  for (int lv = 0; lv < 4; ++lv) {
    // halves of 8, 4, 2, 1 segments: rows of a right half get their decayed queries in the q tile, rows of a left half their
    // decayed writes in the k tiles; the other rows of either tile are not read back
    const int hs = 8 >> lv, half0 = seg & ~(hs - 1);
    if (seg & hs) {
      put_queries(product(half0, seg));
    } else {
      uint64_t m = product(seg + 1, half0 + hs);
#pragma unroll
      for (int i = OSEG - 1; i >= 0; --i) {
        float x, y;
        uint32_t hi, lo;
        u2(mul2(nw[i], m), x, y);
        split2(-x, -y, hi, lo);
        *reinterpret_cast<uint32_t*>(kh_s + at(i)) = hi;
        *reinterpret_cast<uint32_t*>(kl_s + at(i)) = lo;
        m = fma2(nw[i], m, m);
      }
    }
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
    if (lv == 0) {
      // blocks of 8 tokens: a warp takes the tokens of one place in several blocks, CG lanes share a token's channels
      constexpr int CG = NH * 4, TPW = 32 / CG;
      const int i8 = warp & 7, t = ((warp >> 3) * TPW + lane / CG) * 8 + i8, cg = lane % CG;
      uint64_t qv[8], D[8];
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        const uint2 u = *reinterpret_cast<const uint2*>(qb_s + t * PAIRS + 2 * (cg + CG * k));
        const float2 x = bf2(u.x), y = bf2(u.y);
        qv[2 * k] = p2(x.x * sigmoid_fast(x.x), x.y * sigmoid_fast(x.y));
        qv[2 * k + 1] = p2(y.x * sigmoid_fast(y.x), y.y * sigmoid_fast(y.y));
        D[2 * k] = D[2 * k + 1] = p2(1.f, 1.f);
      }
#pragma unroll 1
      for (int j = i8; j >= 0; --j) {
        const float* wr = nw_s + (t - i8 + j) * (NH * 64) + 4 * cg;
        uint64_t acc = 0ull;
#pragma unroll
        for (int k = 0; k < 4; ++k) {
          uint64_t w0, w1;
          ld4(wr + 4 * CG * k, w0, w1);
          acc = fma2(mul2(w0, D[2 * k]), qv[2 * k], acc);
          acc = fma2(mul2(w1, D[2 * k + 1]), qv[2 * k + 1], acc);
          D[2 * k] = fma2(w0, D[2 * k], D[2 * k]);
          D[2 * k + 1] = fma2(w1, D[2 * k + 1], D[2 * k + 1]);
        }
        float x, y;
        u2(acc, x, y);
        x += y;
#pragma unroll
        for (int o = CG / 2; o > 0; o >>= 1) x += __shfl_xor_sync(0xffffffffu, x, o);
        if (cg == 0) diag_s[t * 8 + j] = -x;
      }
    } else if (lv == 1) {
      load_values<PH, NT>(a, h, t0, nval, v_s);           // (1 - F and the queries by token have been read)
#pragma unroll 1
      for (int c = wg * 16; c < C; c += WGS * 16)
#pragma unroll 1
        for (int e = c; e < c + 16; e += 8) {
          float x[8];
          if (wq >= 2 && c < 64) {                        // rows of the right half, columns of the left one
            uint32_t r[8];
            tmem_ld8(tm_d + lane_off + e, r);
            tmem_ld_wait();
#pragma unroll
            for (int j = 0; j < 8; ++j) x[j] = __uint_as_float(r[j]);
            store8(e, x);
          } else if (c / 32 > wq) {                       // above the diagonal
#pragma unroll
            for (int j = 0; j < 8; ++j) x[j] = 0.f;
            store8(e, x);
          }
        }
    } else if (lv == 2) {
      // the state in front of the chunk, high parts and remainders
      const float* S0 = a.dS + (long(chunk) * L.H + h) * L.P * L.N;
      constexpr int IT = PW * NH * 8 / NT;
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
        const int off = (c8 >> 3) * SHALF + row * 128 + (((c8 & 7) ^ (row & 7)) << 4);
        uint4 hi, lo;
        split2(v[0], v[1], hi.x, lo.x);
        split2(v[2], v[3], hi.y, lo.y);
        split2(v[4], v[5], hi.z, lo.z);
        split2(v[6], v[7], hi.w, lo.w);
        *reinterpret_cast<uint4*>(sh_s + off) = hi;
        *reinterpret_cast<uint4*>(sl_s + off) = lo;
      }
#pragma unroll 1
      for (int c = wg * 16; c < C; c += WGS * 16)
        if ((wq & 1) && c / 32 == wq - 1) {               // the second 32 rows of either half against the first
#pragma unroll 1
          for (int e = c; e < c + 16; e += 8) {
            uint32_t r[8];
            float x[8];
            tmem_ld8(tm_d + 128 + lane_off + e, r);
            tmem_ld_wait();
#pragma unroll
            for (int j = 0; j < 8; ++j) x[j] = __uint_as_float(r[j]);
            store8(e, x);
          }
        }
    }
    wait(lv, SITE_FORGET_LEVEL);                          // the tiles are free, accumulators two levels back have been read
  }
  put_queries(product(0, seg));                           // decayed from the chunk's first token on
  // the 32 columns on the diagonal: levels of 16 and of 8 and the blocks of 8
#pragma unroll 1
  for (int c = wg * 16; c < C; c += WGS * 16)
    if (c / 32 == wq) {
#pragma unroll 1
      for (int e = c; e < c + 16; e += 8) {
        const int cb = (e >> 3) & 3, blk = lane >> 3;     // blocks of 8 of the columns and of the lane's token
        uint32_t r16[8], r8[8];
        tmem_ld8(tm_d + lane_off + e, r16);
        tmem_ld8(tm_d + 128 + lane_off + e, r8);
        const float4 d0 = *reinterpret_cast<const float4*>(diag_s + (wq * 32 + lane) * 8);
        const float4 d1 = *reinterpret_cast<const float4*>(diag_s + (wq * 32 + lane) * 8 + 4);
        const float d[8] = {d0.x, d0.y, d0.z, d0.w, d1.x, d1.y, d1.z, d1.w};
        tmem_ld_wait();
        float x[8];
#pragma unroll
        for (int j = 0; j < 8; ++j)
          x[j] = cb == blk                       ? (j <= (lane & 7) ? d[j] : 0.f)
                 : !(cb & 1) && blk == cb + 1    ? __uint_as_float(r8[j])
                 : cb < 2 && blk >= 2            ? __uint_as_float(r16[j])
                                                 : 0.f;
        store8(e, x);
      }
    }
  tmem_st_wait();
  cp_async_wait();                                        // the values
  fence_proxy_async_smem();
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  if (threadIdx.x == 0) {
    constexpr uint32_t idesc_x = umma_idesc(128, PW, 1, 1, 0, 0);
    constexpr uint32_t idesc_o = umma_idesc(128, PW, 1, 1, 0, 1);
    const uint32_t sh = smem_u32(sh_s), sl = smem_u32(sl_s), va = smem_u32(v_s);
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
  wait(4, SITE_FORGET_OUTPUT);
  // norm over the head's value columns (those past P are zeros): 16 columns per warp and turn, sums joined in shared memory
  const int row = wq * 32 + lane;
  constexpr int GROUPS = PW / 16, PER = (GROUPS + WGS - 1) / WGS;        // column groups, and of them per warpgroup
  uint32_t y[PER][16];
  float ss = 0.f;
  const bool all_ok = ok;                                 // (the same for the whole CTA)
#pragma unroll
  for (int i = 0; i < PER; ++i) {
    const int g = wg + i * WGS;
    if (all_ok && g < GROUPS) {
      tmem_ld16(tm_o + lane_off + g * 16, y[i]);
      tmem_ld_wait();
#pragma unroll
      for (int j = 0; j < 16; ++j) ss = fmaf(__uint_as_float(y[i][j]), __uint_as_float(y[i][j]), ss);
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
      for (int j = 0; j < 16; j += 8) {
        const int col = g * 16 + j;
        if (col >= L.P) continue;
        float z[8];
#pragma unroll
        for (int e = 0; e < 8; ++e) z[e] = col + e < L.P ? __uint_as_float(y[i][j + e]) * inv * __ldg(L.norm_w + col + e) : 0.f;
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
  constexpr int SA = states_smem<NH, PH>(), SC = OutSmem<NH, PH>::BYTES;
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
  return launch_pdl(ko, grid, dim3(NH * 512), SC, s, a) != cudaSuccess;
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
  a.vec_q = al(L.q, L.ldq, L.N, 8);
  a.vec_f = al(L.f, L.ldf, L.N, 8);
  a.vec_v = al(L.v, L.ldv, L.P, 8);
  a.vec_o = al(L.out, L.ldo, L.P, 8);
  if (L.N <= 64) return L.P <= 64 ? launch_np<1, 1>(a, n_chunks, seq_chunk0, seq_nchunk, s)
                                  : launch_np<1, 2>(a, n_chunks, seq_chunk0, seq_nchunk, s);
  return L.P <= 64 ? launch_np<2, 1>(a, n_chunks, seq_chunk0, seq_nchunk, s)
                   : launch_np<2, 2>(a, n_chunks, seq_chunk0, seq_nchunk, s);
}

}  // namespace lb
