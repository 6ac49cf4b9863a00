// Gated delta rule with a decay per key channel, bf16 prompts: blocks of eight tokens, products with the state on tensor cores.
// The algebra is that of channel_delta.cu. With G_j = g_1 .. g_j inside a block and S_0 the state in front of it,
//   d_j = S_0^T (beta_j G_j k_j),   e_j = S_0^T (G_j q_j)
//   u_j = beta_j v_j - d_j - sum_{i<j} c_ij u_i,     c_ij = beta_j k_i . (g_{i+1} .. g_j k_j)
//   o_j = e_j + sum_{i<=j} m_ij u_i,                 m_ij = k_i . (g_{i+1} .. g_j q_j)
//   S_8 = G_8 S_0 + sum_i (g_{i+1} .. g_8 k_i) u_i^T
// PREP writes a record per (head, block), all blocks in parallel. SCAN walks the blocks of a sequence: a warp owns 16 state
// columns and keeps them as the fp32 accumulator fragments of m16n8 tiles (16 value columns x 8 key channels). Those are at
// the same time, tile pair by tile pair, the A operand of the products d and e (16 x 128 times 128 x 16), and the update
// accumulates onto them (16 x 8 tokens times 8 tokens x 8 channels), so the state never leaves the registers and no value is
// exchanged between lanes but the 16 results of a column. Decays, norms, inner products, the decay of the state and the
// solution for u are fp32; what enters a product (state, decayed vectors, u) is split into two bf16 terms, high part and
// remainder, and the three leading products are summed (about 16 significant bits, fp32 accumulation).
//
// The record holds the operands in fragment order (a lane's registers side by side), so the consumer reads 16 bytes per lane
// without bank conflicts; records are built in shared memory and leave, and come, as bulk copies.
#include "channel_delta.cuh"

namespace lb {
namespace {

constexpr int BT = 8;                      // tokens per block
constexpr int CPC = 64;                    // state columns per SCAN CTA (four warps of sixteen)
constexpr int STAGES = 4;

// record: KS = padded key channels / 16
__host__ __device__ constexpr int dot_bytes(int ks) { return ks * 1024; }        // [ks][2 tiles of 8 vectors][32 lanes][hi b0 b1, lo b0 b1]
__host__ __device__ constexpr int up_bytes(int ks) { return ks * 512; }          // [ks][32 lanes][tile 0 hi lo, tile 1 hi lo]
__host__ __device__ constexpr int dec_bytes(int ks) { return ks * 64; }          // [ks][4][tile 0 pair, tile 1 pair] of G_8
constexpr int SC_BYTES = 512;                                                    // c [8][8] (row j), m [8][8] (row j)
__host__ __device__ constexpr int head_bytes(int ks) { return dot_bytes(ks) + up_bytes(ks) + dec_bytes(ks) + SC_BYTES; }
__host__ __device__ constexpr int pad16(int n) { return (n + 15) / 16 * 16; }
__host__ __device__ constexpr int rec_bytes(int ks, int dv) { return head_bytes(ks) + pad16(dv) * 32; }   // + beta v [column][8]
__host__ __device__ constexpr int steps_of(int dk) { return dk <= 32 ? 2 : dk <= 64 ? 4 : 8; }

__device__ __forceinline__ float bf_hi(float v) { return __bfloat162float(__float2bfloat16(v)); }

// N columns at p (n_ok of them exist); VEC: aligned, all or none exist
template <int N, bool VEC>
__device__ __forceinline__ void ld_cols(const __nv_bfloat16* p, int n_ok, float (&v)[N]) {
  if constexpr (VEC && N == 4) {
    if (n_ok >= 4) ld_f4(p, v);
    else v[0] = v[1] = v[2] = v[3] = 0.f;
  } else if constexpr (VEC && N == 2) {
    float2 f = make_float2(0.f, 0.f);
    if (n_ok >= 2) f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p));
    v[0] = f.x;
    v[1] = f.y;
  } else {
#pragma unroll
    for (int j = 0; j < N; ++j) v[j] = j < n_ok ? __bfloat162float(p[j]) : 0.f;
  }
}

// Convolution + silu of N neighbouring channels for the block's tokens. hist: [taps - 1] rows C apart; w: taps rows ws apart
template <int N, int KC, bool VEC>
__device__ __forceinline__ void conv_cols(const __nv_bfloat16* x, long ld, const float* hist, long C, const float* w, int ws,
                                          int taps, int n_ok, const DeltaBlock& b, float (&y)[BT][N]) {
  if constexpr (KC > 0) {
    float u[KC - 1 + BT][N];
#pragma unroll
    for (int i = 0; i < KC - 1 + BT; ++i) {
      const int s = b.t0 - (KC - 1) + i;
      if (s < b.seq0) {
#pragma unroll
        for (int j = 0; j < N; ++j) u[i][j] = j < n_ok ? hist[((KC - 1) + (s - b.seq0)) * C + j] : 0.f;
      } else {
        ld_cols<N, VEC>(x + long(s) * ld, i - (KC - 1) < b.n ? n_ok : 0, u[i]);
      }
    }
#pragma unroll
    for (int t = 0; t < BT; ++t)
#pragma unroll
      for (int j = 0; j < N; ++j) y[t][j] = 0.f;
#pragma unroll
    for (int k = 0; k < KC; ++k)
#pragma unroll
      for (int j = 0; j < N; ++j) {
        const float wk = j < n_ok ? w[k * ws + j] : 0.f;
#pragma unroll
        for (int t = 0; t < BT; ++t) y[t][j] = fmaf(wk, u[t + k][j], y[t][j]);
      }
  } else {
#pragma unroll
    for (int t = 0; t < BT; ++t) {
#pragma unroll
      for (int j = 0; j < N; ++j) {
        float acc = 0.f;
        for (int k = 0; k < taps && t < b.n && j < n_ok; ++k) {
          const int s = b.t0 + t - (taps - 1) + k;
          acc = fmaf(w[k * ws + j], s >= b.seq0 ? __bfloat162float(x[long(s) * ld + j]) : hist[((taps - 1) + (s - b.seq0)) * C + j], acc);
        }
        y[t][j] = acc;
      }
    }
  }
#pragma unroll
  for (int t = 0; t < BT; ++t)
#pragma unroll
    for (int j = 0; j < N; ++j) y[t][j] = t < b.n ? silu_t<__nv_bfloat16>(y[t][j]) : 0.f;
}

__device__ __forceinline__ void bulk_store(void* gdst, const void* smem_src, uint32_t bytes) {
  asm volatile("cp.async.bulk.global.shared::cta.bulk_group [%0], [%1], %2;" ::"l"(reinterpret_cast<uint64_t>(gdst)),
               "r"(smem_u32(smem_src)), "r"(bytes)
               : "memory");
  asm volatile("cp.async.bulk.commit_group;" ::: "memory");
}

// What a lane holds after the three transposed sums: kind 0 c, 1 m, 2 |q|^2, 3 |k|^2, 7 nothing; i and j
struct Cell { int kind, i, j; };
__host__ __device__ constexpr Cell cell_of(int batch, int lane) {
  if (batch == 0) {                                   // |q_j|^2, |k_j|^2, m_0j, c_0j
    if (lane < 8) return {2, 0, lane};
    if (lane < 16) return {3, 0, lane - 8};
    if (lane < 24) return {1, 0, lane - 16};
    if (lane < 31) return {0, 0, lane - 23};
    return {7, 0, 0};
  }
  int n = 0;
  for (int x = 0; x < (batch == 1 ? 4 : 3); ++x) {    // rows 1, 2, 7, 6 | 3, 4, 5
    const int i = batch == 1 ? (x == 0 ? 1 : x == 1 ? 2 : x == 2 ? 7 : 6) : 3 + x;
    for (int j = i; j < 8; ++j, ++n)
      if (n == lane) return {1, i, j};
    for (int j = i + 1; j < 8; ++j, ++n)
      if (n == lane) return {0, i, j};
  }
  return {7, 0, 0};
}
struct CellTable { uint8_t v[3][32]; };
constexpr CellTable make_cells() {
  CellTable t{};
  for (int b = 0; b < 3; ++b)
    for (int l = 0; l < 32; ++l) {
      const Cell c = cell_of(b, l);
      t.v[b][l] = uint8_t((c.kind == 7 ? 3 : c.kind) << 6 | c.i << 3 | c.j);
    }
  return t;
}
__constant__ CellTable CELLS = make_cells();

constexpr int PREP_BLOCKS = 4;             // blocks per warp

// One warp per (head, block); a lane holds NC neighbouring key channels.
template <int KS, int KC, bool VEC>
__global__ void __launch_bounds__(128, 2) delta_prep8_kernel(const ChannelDeltaArgs a, int lo, int hi, int n_blocks, uint8_t* rec) {
  using T = __nv_bfloat16;
  constexpr int NC = KS / 2, DKP = KS * 16;
  extern __shared__ __align__(128) uint8_t smem[];
  const int h = blockIdx.y, DK = a.DK, DV = a.DV, W = 2 * DK + DV, taps = a.KC;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int hk = h / (a.H / a.G);
  const int q0 = hk * DK, k0 = a.G * DK + hk * DK, v0 = 2 * a.G * DK + h * DV, C = 2 * a.G * DK + a.H * DV;
  const int R = rec_bytes(KS, DV);
  uint8_t* r = smem + warp * R;
  float* w_s = reinterpret_cast<float*>(smem + 4 * R);      // taps of the head's q | k | v channels, [taps][2 dk + dv]
  for (int i = threadIdx.x; i < W * taps; i += 128) {
    const int c = i % W, j = i / W;
    w_s[i] = a.conv_w[long(j) * C + (c < DK ? q0 + c : c < 2 * DK ? k0 + c - DK : v0 + c - 2 * DK)];
  }
  griddep_wait();
  griddep_launch();
  __syncthreads();
  const float Ah = a.A[h];
  const T* x = static_cast<const T*>(a.qkv);
  const int c0 = lane * NC, n_ok = max(0, min(NC, DK - c0));
  const T* ap = static_cast<const T*>(a.a) + long(h) * DK + c0;
  float db[NC];
#pragma unroll
  for (int j = 0; j < NC; ++j) db[j] = j < n_ok ? a.dt_bias[long(h) * DK + c0 + j] : 0.f;
  float* sc = reinterpret_cast<float*>(r + dot_bytes(KS) + up_bytes(KS) + dec_bytes(KS));
  for (int i = lane; i < SC_BYTES / 4; i += 32) sc[i] = 0.f;                     // above the diagonals
  const int blk0 = (blockIdx.x * 4 + warp) * PREP_BLOCKS;
  for (int blk = blk0; blk < min(n_blocks, blk0 + PREP_BLOCKS); ++blk) {
    DeltaBlock b;
    if (!find_block<BT>(a.cu, a.n_seqs, lo, hi, blk, b)) continue;
    const float* hist = a.conv_state + long(a.slots[b.seq]) * C * (taps - 1);
    float q[BT][NC], k[BT][NC], g[BT][NC];
    conv_cols<NC, KC, VEC>(x + q0 + c0, a.ld, hist + q0 + c0, C, w_s + c0, W, taps, n_ok, b, q);
    conv_cols<NC, KC, VEC>(x + k0 + c0, a.ld, hist + k0 + c0, C, w_s + DK + c0, W, taps, n_ok, b, k);
#pragma unroll
    for (int t = 0; t < BT; ++t) {
      float z[NC];
      ld_cols<NC, VEC>(ap + long(b.t0 + t) * a.lda, t < b.n ? n_ok : 0, z);
#pragma unroll
      for (int j = 0; j < NC; ++j) g[t][j] = t < b.n && j < n_ok ? decay_t<T>(z[j] + db[j], Ah) : 1.f;
    }
    const float be = lane < b.n && lane < BT ? sigmoid_t<T>(ld_f(static_cast<const T*>(a.b) + long(b.t0 + lane) * a.ldb + h)) : 0.f;
    // the record this warp wrote before has left its shared memory
    if (lane == 0) asm volatile("cp.async.bulk.wait_group.read 0;" ::: "memory");
    __syncwarp();
    // ---- inner products
    float rq[BT], rk[BT], bb[BT];
#pragma unroll
    for (int t = 0; t < BT; ++t) bb[t] = __shfl_sync(0xffffffffu, be, t);
    auto products = [&](int i, float* m, float* c) {      // m[j - i] for j >= i, c[j - i - 1] for j > i
      float kd[NC];
#pragma unroll
      for (int n = 0; n < NC; ++n) {
        kd[n] = k[i][n];
        m[0] = fmaf(kd[n], q[i][n], n ? m[0] : 0.f);
      }
#pragma unroll
      for (int j = 0; j < BT; ++j)
        if (j > i) {
          float sm_ = 0.f, sc_ = 0.f;
#pragma unroll
          for (int n = 0; n < NC; ++n) {
            kd[n] *= g[j][n];
            sm_ = fmaf(kd[n], q[j][n], sm_);
            sc_ = fmaf(kd[n], k[j][n], sc_);
          }
          m[j - i] = sm_;
          c[j - i - 1] = sc_;
        }
    };
    auto place = [&](int batch, float v) {                 // the lane's sum into its cell
      const int e = CELLS.v[batch][lane], kind = e >> 6, i = (e >> 3) & 7, j = e & 7;
      float ri = 0.f, kj = 0.f, qj = 0.f, bj = 0.f;
#pragma unroll
      for (int t = 0; t < BT; ++t) {
        if (t == i) ri = rk[t];
        if (t == j) { kj = rk[t]; qj = rq[t]; bj = bb[t]; }
      }
      if (kind == 0) sc[j * 8 + i] = v * ri * kj * bj;
      else if (kind == 1) sc[64 + j * 8 + i] = v * ri * qj;
    };
    {
      float s[32];
#pragma unroll
      for (int t = 0; t < BT; ++t) {
        s[t] = s[8 + t] = 0.f;
#pragma unroll
        for (int n = 0; n < NC; ++n) {
          s[t] = fmaf(q[t][n], q[t][n], s[t]);
          s[8 + t] = fmaf(k[t][n], k[t][n], s[8 + t]);
        }
      }
      products(0, s + 16, s + 24);
      s[31] = 0.f;
      const float v = transpose_sum(s);
      const float inv = 1.f / sqrtf(v + a.l2_eps);
#pragma unroll
      for (int t = 0; t < BT; ++t) {
        rq[t] = __shfl_sync(0xffffffffu, inv, t) * a.scale;
        rk[t] = __shfl_sync(0xffffffffu, inv, 8 + t);
      }
      place(0, v);
    }
    {
      float s[32];
      products(1, s, s + 7);
      products(2, s + 13, s + 19);
      products(7, s + 24, s + 25);
      products(6, s + 25, s + 27);
#pragma unroll
      for (int i = 28; i < 32; ++i) s[i] = 0.f;
      place(1, transpose_sum(s));
    }
    {
      float s[32];
      products(3, s, s + 5);
      products(4, s + 9, s + 13);
      products(5, s + 16, s + 19);
#pragma unroll
      for (int i = 21; i < 32; ++i) s[i] = 0.f;
      place(2, transpose_sum(s));
    }
    // ---- operands in fragment order; 16-byte chunks of a step s are permuted by s (lane chunk ^ s), which keeps both the
    // writes here and the reads of the consumer off each other's banks
    float G[NC];
#pragma unroll
    for (int n = 0; n < NC; ++n) G[n] = 1.f;
    auto put_dot = [&](int vec, const float (&v)[NC]) {
#pragma unroll
      for (int n = 0; n < NC; n += (NC >= 2 ? 2 : 1)) {
        const int c = c0 + n, s = c >> 4, kk = c & 15;
        uint8_t* p = r + (s * 2 + (vec >> 3)) * 512 + ((((vec & 7) * 4 + ((kk & 7) >> 1)) ^ (s & 7)) << 4) + (kk >> 3) * 4;
        if constexpr (NC >= 2) {
          const float h0 = bf_hi(v[n]), h1 = bf_hi(v[n + 1]);
          *reinterpret_cast<uint32_t*>(p) = pack_bf16x2(v[n], v[n + 1]);
          *reinterpret_cast<uint32_t*>(p + 8) = pack_bf16x2(v[n] - h0, v[n + 1] - h1);
        } else {
          *reinterpret_cast<__nv_bfloat16*>(p + (kk & 1) * 2) = __float2bfloat16(v[n]);
          *reinterpret_cast<__nv_bfloat16*>(p + 8 + (kk & 1) * 2) = __float2bfloat16(v[n] - bf_hi(v[n]));
        }
      }
    };
#pragma unroll
    for (int t = 0; t < BT; ++t) {
      float vd[NC], ve[NC];
      const float fd = bb[t] * rk[t];
#pragma unroll
      for (int n = 0; n < NC; ++n) {
        G[n] *= g[t][n];
        vd[n] = G[n] * (k[t][n] * fd);
        ve[n] = G[n] * (q[t][n] * rq[t]);
      }
      put_dot(2 * t, vd);
      put_dot(2 * t + 1, ve);
    }
#pragma unroll
    for (int n = 0; n < NC; ++n) {
      const int c = c0 + n, s = c >> 4, kk = c & 15;
      *reinterpret_cast<float*>(r + dot_bytes(KS) + up_bytes(KS) + s * 64 + ((kk & 7) >> 1) * 16 + (kk >> 3) * 8 + (kk & 1) * 4) = G[n];
      float D = 1.f, u[BT];
#pragma unroll
      for (int t = BT - 1; t >= 0; --t) {
        u[t] = D * (k[t][n] * rk[t]);
        D *= g[t][n];
      }
#pragma unroll
      for (int p = 0; p < BT / 2; ++p) {                   // token pair p of channel c: tile kk / 8 of step s, lane (kk % 8) * 4 + p
        const float h0 = bf_hi(u[2 * p]), h1 = bf_hi(u[2 * p + 1]);
        *reinterpret_cast<uint2*>(r + dot_bytes(KS) + s * 512 + ((((kk & 7) * 4 + p) ^ (s & 7)) << 4) + (kk >> 3) * 8) =
            make_uint2(pack_bf16x2(u[2 * p], u[2 * p + 1]), pack_bf16x2(u[2 * p] - h0, u[2 * p + 1] - h1));
      }
    }
    // ---- beta v
    float* vs = reinterpret_cast<float*>(r + head_bytes(KS));
    for (int c = 2 * lane; c < pad16(DV); c += 64) {
      float v[BT][2];
      conv_cols<2, KC, VEC>(x + v0 + c, a.ld, hist + v0 + c, C, w_s + 2 * DK + c, W, taps, max(0, min(2, DV - c)), b, v);
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int f = 0; f < 2; ++f)
          *reinterpret_cast<float4*>(vs + (c + n) * 8 + 4 * f) =
              make_float4(bb[4 * f] * v[4 * f][n], bb[4 * f + 1] * v[4 * f + 1][n], bb[4 * f + 2] * v[4 * f + 2][n],
                          bb[4 * f + 3] * v[4 * f + 3][n]);
    }
    fence_proxy_async_smem();
    __syncwarp();
    if (lane == 0) bulk_store(rec + (long(h) * n_blocks + blk) * R, r, R);
  }
  if (lane == 0) asm volatile("cp.async.bulk.wait_group 0;" ::: "memory");
}

__device__ __forceinline__ void mma16(float (&d)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
               : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void mma8(float (&d)[4], uint32_t a0, uint32_t a1, uint32_t b0) {
  asm volatile("mma.sync.aligned.m16n8k8.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5}, {%6}, {%0, %1, %2, %3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
               : "r"(a0), "r"(a1), "r"(b0));
}
// high bf16 parts of two values, and their remainders
__device__ __forceinline__ void split2(float x, float y, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16x2(x, y);
  lo = pack_bf16x2(x - __uint_as_float(hi << 16), y - __uint_as_float(hi & 0xffff0000u));
}

// grid (H * column groups, sequences), 160 threads: warps 0..3 own sixteen columns each, warp 4 copies the records.
template <int KS>
__global__ void __launch_bounds__(160) delta_scan8_kernel(const ChannelDeltaArgs a, int lo, int hi, int n_blocks, const uint8_t* rec,
                                                          int* status) {
  constexpr int HEAD = head_bytes(KS), STAGE = HEAD + CPC * 32;
  extern __shared__ __align__(128) uint8_t smem[];         // [STAGES][STAGE]
  __shared__ __align__(8) uint64_t full[STAGES], empty[STAGES];
  __shared__ int abort_s;
  volatile int* abort_flag = &abort_s;
  const int DK = a.DK, DV = a.DV, groups = (DV + CPC - 1) / CPC;
  const int h = blockIdx.x / groups, col0 = (blockIdx.x % groups) * CPC, seq = blockIdx.y;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int n_warps = min(4, (DV - col0 + 15) / 16);       // warps with columns
  if (threadIdx.x == 0) {
    for (int i = 0; i < STAGES; ++i) {
      mbar_init(&full[i], 1);
      mbar_init(&empty[i], n_warps);
    }
    abort_s = 0;
    mbar_fence_init();
  }
  __syncthreads();
  griddep_wait();
  griddep_launch();
  const int s0 = clamp_i(a.cu[seq], lo, hi), s1 = clamp_i(a.cu[seq + 1], lo, hi);
  const int slot = a.slots[seq];
  if (s1 <= s0 || slot < 0) return;
  const int n_blk = (s1 - s0 + BT - 1) / BT;
  const int R = rec_bytes(KS, DV);
  const uint8_t* r0 = rec + (long(h) * n_blocks + (s0 - lo) / BT + seq) * R;
  if (warp == 4) {
    if (lane == 0) {
      const int vbytes = min(CPC, pad16(DV) - col0) * 32;
      int i = 0;
      for (; i < n_blk; ++i) {
        const int s = i % STAGES;
        if (i >= STAGES && !mbar_wait(&empty[s], ((i / STAGES) - 1) & 1, abort_flag)) {
          *abort_flag = 1;
          atomicCAS(status, 0, ST_TIMEOUT_EMPTY | SITE_DELTA_SCAN);
          break;
        }
        const uint8_t* src = r0 + long(i) * R;
        mbar_expect_tx(&full[s], HEAD + vbytes);
        bulk_load(smem + s * STAGE, src, HEAD, &full[s]);
        bulk_load(smem + s * STAGE + HEAD, src + HEAD + col0 * 32, vbytes, &full[s]);
      }
      // copies in flight land before the CTA ends: the consumers wait for every one, unless they gave up
      if (*abort_flag) {
        volatile int no = 0;
        for (int j = max(0, i - STAGES); j < i; ++j) mbar_wait(&full[j % STAGES], (j / STAGES) & 1, &no, 1000000ull);
      }
    }
    return;
  }
  if (warp >= n_warps) return;
  const int q = lane & 3, ca = col0 + warp * 16 + (lane >> 2), cb = ca + 8;
  float* st = a.state + (long(slot) * a.H + h) * DV * DK;
  // S[t]: key channels 8 t + 2 q, + 1 of columns ca (0, 1) and cb (2, 3)
  float S[2 * KS][4];
#pragma unroll
  for (int t = 0; t < 2 * KS; ++t)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int c = e < 2 ? ca : cb, k = 8 * t + 2 * q + (e & 1);
      S[t][e] = c < DV && k < DK ? st[long(c) * DK + k] : 0.f;
    }
  auto* out = static_cast<__nv_bfloat16*>(a.out) + long(h) * DV;
  for (int i = 0; i < n_blk; ++i) {
    const int sg = i % STAGES;
    if (!__all_sync(0xffffffffu, mbar_wait(&full[sg], (i / STAGES) & 1, abort_flag))) {
      *abort_flag = 1;
      if (lane == 0) atomicCAS(status, 0, ST_TIMEOUT_FULL | SITE_DELTA_SCAN);
      break;
    }
    const uint8_t* v = smem + sg * STAGE;
    // ---- d and e: vector 2 q of tile n is d_{q + 4 n}, vector 2 q + 1 is e_{q + 4 n}
    float acc[2][3][4];
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int p = 0; p < 3; ++p)
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[n][p][e] = 0.f;
#pragma unroll
    for (int s = 0; s < KS; ++s) {
      uint32_t h0, h1, h2, h3, l0, l1, l2, l3;
      split2(S[2 * s][0], S[2 * s][1], h0, l0);
      split2(S[2 * s][2], S[2 * s][3], h1, l1);
      split2(S[2 * s + 1][0], S[2 * s + 1][1], h2, l2);
      split2(S[2 * s + 1][2], S[2 * s + 1][3], h3, l3);
#pragma unroll
      for (int n = 0; n < 2; ++n) {
        const uint4 f = *reinterpret_cast<const uint4*>(v + (s * 2 + n) * 512 + ((lane ^ (s & 7)) << 4));
        mma16(acc[n][0], h0, h1, h2, h3, f.x, f.y);
        mma16(acc[n][1], h0, h1, h2, h3, f.z, f.w);
        mma16(acc[n][2], l0, l1, l2, l3, f.x, f.y);
      }
    }
    float x[2][4];
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) x[n][e] = acc[n][0][e] + (acc[n][1][e] + acc[n][2][e]);
    // ---- u of both columns, on every lane of the quad
    const float* sc = reinterpret_cast<const float*>(v + dot_bytes(KS) + up_bytes(KS) + dec_bytes(KS));
    const float* vv = reinterpret_cast<const float*>(v + HEAD) + (warp * 16 + (lane >> 2)) * 8;
    float ua[BT], ub[BT];
    {
      float va[BT], vb[BT];
#pragma unroll
      for (int f = 0; f < 2; ++f) {
        const float4 p = *reinterpret_cast<const float4*>(vv + 4 * f), r = *reinterpret_cast<const float4*>(vv + 64 + 4 * f);
        va[4 * f] = p.x; va[4 * f + 1] = p.y; va[4 * f + 2] = p.z; va[4 * f + 3] = p.w;
        vb[4 * f] = r.x; vb[4 * f + 1] = r.y; vb[4 * f + 2] = r.z; vb[4 * f + 3] = r.w;
      }
#pragma unroll
      for (int j = 0; j < BT; ++j) {
        va[j] -= __shfl_sync(0xffffffffu, x[j >> 2][0], (lane & 28) + (j & 3));
        vb[j] -= __shfl_sync(0xffffffffu, x[j >> 2][2], (lane & 28) + (j & 3));
      }
#pragma unroll
      for (int j = 0; j < BT; ++j) {
        float c[BT];
        if (j > 0) {
          const float4 p = *reinterpret_cast<const float4*>(sc + j * 8);
          c[0] = p.x; c[1] = p.y; c[2] = p.z; c[3] = p.w;
        }
        if (j > 4) {
          const float4 p = *reinterpret_cast<const float4*>(sc + j * 8 + 4);
          c[4] = p.x; c[5] = p.y; c[6] = p.z; c[7] = p.w;
        }
        float sa = va[j], sb = vb[j];
#pragma unroll
        for (int k = 0; k < j; ++k) {
          sa = fmaf(-c[k], ua[k], sa);
          sb = fmaf(-c[k], ub[k], sb);
        }
        ua[j] = sa;
        ub[j] = sb;
      }
    }
    // ---- outputs of tokens q and q + 4
#pragma unroll
    for (int n = 0; n < 2; ++n) {
      const float4 p = *reinterpret_cast<const float4*>(sc + 64 + (q + 4 * n) * 8);
      float oa = fmaf(p.x, ua[0], x[n][1]), ob = fmaf(p.x, ub[0], x[n][3]);
      oa = fmaf(p.y, ua[1], oa); ob = fmaf(p.y, ub[1], ob);
      oa = fmaf(p.z, ua[2], oa); ob = fmaf(p.z, ub[2], ob);
      oa = fmaf(p.w, ua[3], oa); ob = fmaf(p.w, ub[3], ob);
      if (n == 1) {
        const float4 r = *reinterpret_cast<const float4*>(sc + 64 + (q + 4) * 8 + 4);
        oa = fmaf(r.x, ua[4], oa); ob = fmaf(r.x, ub[4], ob);
        oa = fmaf(r.y, ua[5], oa); ob = fmaf(r.y, ub[5], ob);
        oa = fmaf(r.z, ua[6], oa); ob = fmaf(r.z, ub[6], ob);
        oa = fmaf(r.w, ua[7], oa); ob = fmaf(r.w, ub[7], ob);
      }
      const int t = s0 + i * BT + q + 4 * n;
      if (t < s1) {
        if (ca < DV) out[long(t) * a.ldo + ca] = __float2bfloat16(oa);
        if (cb < DV) out[long(t) * a.ldo + cb] = __float2bfloat16(ob);
      }
    }
    // ---- state: decay, then the eight writes. A operand: tokens 2 q, 2 q + 1 of both columns, high parts and remainders
    const float a0 = q == 0 ? ua[0] : q == 1 ? ua[2] : q == 2 ? ua[4] : ua[6], a1 = q == 0 ? ua[1] : q == 1 ? ua[3] : q == 2 ? ua[5] : ua[7];
    const float b0 = q == 0 ? ub[0] : q == 1 ? ub[2] : q == 2 ? ub[4] : ub[6], b1 = q == 0 ? ub[1] : q == 1 ? ub[3] : q == 2 ? ub[5] : ub[7];
    uint32_t ah, al, bh, bl;
    split2(a0, a1, ah, al);
    split2(b0, b1, bh, bl);
#pragma unroll
    for (int s = 0; s < KS; ++s) {
      const float4 g = *reinterpret_cast<const float4*>(v + dot_bytes(KS) + up_bytes(KS) + s * 64 + q * 16);
      const uint4 f = *reinterpret_cast<const uint4*>(v + dot_bytes(KS) + s * 512 + ((lane ^ (s & 7)) << 4));
      S[2 * s][0] *= g.x; S[2 * s][1] *= g.y; S[2 * s][2] *= g.x; S[2 * s][3] *= g.y;
      S[2 * s + 1][0] *= g.z; S[2 * s + 1][1] *= g.w; S[2 * s + 1][2] *= g.z; S[2 * s + 1][3] *= g.w;
      mma16(S[2 * s], ah, bh, al, bl, f.x, f.x);
      mma8(S[2 * s], ah, bh, f.y);
      mma16(S[2 * s + 1], ah, bh, al, bl, f.z, f.z);
      mma8(S[2 * s + 1], ah, bh, f.w);
    }
    __syncwarp();
    if (lane == 0) mbar_arrive(&empty[sg]);
  }
  if (a.write_state && !*abort_flag) {
#pragma unroll
    for (int t = 0; t < 2 * KS; ++t)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int c = e < 2 ? ca : cb, k = 8 * t + 2 * q + (e & 1);
        if (c < DV && k < DK) st[long(c) * DK + k] = S[t][e];
      }
  }
}

template <int KS, int KC>
int prep_k(const ChannelDeltaArgs& a, int lo, int hi, int nb, uint8_t* rec, bool vec, cudaStream_t s) {
  const dim3 grid((nb + 4 * PREP_BLOCKS - 1) / (4 * PREP_BLOCKS), a.H);
  const int smem = 4 * rec_bytes(KS, a.DV) + (2 * a.DK + a.DV) * a.KC * 4;
  auto k1 = delta_prep8_kernel<KS, KC, true>;
  auto k0 = delta_prep8_kernel<KS, KC, false>;
  auto kfn = vec ? k1 : k0;
  if (smem > 200 * 1024 || cudaFuncSetAttribute(kfn, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess) return 1;
  return launch_pdl(kfn, grid, dim3(128), smem, s, a, lo, hi, nb, rec) != cudaSuccess;
}

template <int KS>
int slice_k(const ChannelDeltaArgs& a, int lo, int hi, int nb, uint8_t* rec, bool vec, int* status, cudaStream_t s) {
  int rc;
  if (a.KC == 4) rc = prep_k<KS, 4>(a, lo, hi, nb, rec, vec, s);
  else if (a.KC == 3) rc = prep_k<KS, 3>(a, lo, hi, nb, rec, vec, s);
  else if (a.KC == 2) rc = prep_k<KS, 2>(a, lo, hi, nb, rec, vec, s);
  else rc = prep_k<KS, 0>(a, lo, hi, nb, rec, vec, s);
  if (rc) return 1;
  const int smem = STAGES * (head_bytes(KS) + CPC * 32);
  auto kfn = delta_scan8_kernel<KS>;
  if (cudaFuncSetAttribute(kfn, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess) return 1;
  return launch_pdl(kfn, dim3(a.H * ((a.DV + CPC - 1) / CPC), a.n_seqs), dim3(160), smem, s, a, lo, hi, nb,
                    static_cast<const uint8_t*>(rec), status) != cudaSuccess;
}

}  // namespace

bool channel_delta_mma_ok(const ChannelDeltaArgs& a) {
  return a.DK <= 128 && 4 * rec_bytes(steps_of(a.DK), a.DV) + (2 * a.DK + a.DV) * a.KC * 4 <= 200 * 1024;
}

long channel_delta_mma_floats(int H, int DK, int DV) { return DK > 128 ? 0 : long(rec_bytes(steps_of(DK), DV)) / 4 * H; }

int channel_delta_mma_launch(const ChannelDeltaArgs& a, float* rec, long rec_floats, int* status, cudaStream_t s) {
  const int ks = steps_of(a.DK), nc = ks / 2;
  const long blocks = rec_floats / channel_delta_mma_floats(a.H, a.DK, a.DV);       // records the scratch holds, per head
  const long tokens = (blocks - a.n_seqs) * BT;
  if (tokens < BT || (tokens < a.T && !a.write_state)) return 1;      // slices hand the state on through the pool
  auto al = [](const void* p, size_t n) { return reinterpret_cast<uintptr_t>(p) % n == 0; };
  const int m = nc < 2 ? 2 : nc;
  const bool vec = a.DK % m == 0 && a.DV % 2 == 0 && a.ld % m == 0 && a.lda % m == 0 && (2L * a.G * a.DK) % m == 0 &&
                   al(a.qkv, 2 * m) && al(a.a, 2 * m);
  for (int lo = 0; lo < a.T;) {
    const int hi = int(long(a.T) - lo <= tokens ? a.T : lo + tokens);
    const int nb = (hi - lo) / BT + a.n_seqs;
    auto* r = reinterpret_cast<uint8_t*>(rec);
    const int rc = ks == 2 ? slice_k<2>(a, lo, hi, nb, r, vec, status, s)
                           : ks == 4 ? slice_k<4>(a, lo, hi, nb, r, vec, status, s) : slice_k<8>(a, lo, hi, nb, r, vec, status, s);
    if (rc) return 1;
    lo = hi;
  }
  return 0;
}

}  // namespace lb
