// Gated delta rule with a decay per key channel, bf16 prompts: blocks of eight tokens, products with the state on tensor cores.
// With G_j = g_1 .. g_j inside a block and S_0 the state in front of it, the delta rule of the block is (see channel_delta.cu)
//   u_j = beta_j v_j - S_0^T (beta_j G_j k_j) - sum_{i<j} c_ij u_i,   c_ij = beta_j k_i . (g_{i+1} .. g_j k_j)
//   o_j = S_0^T (G_j q_j) + sum_{i<=j} m_ij u_i,                      m_ij = k_i . (g_{i+1} .. g_j q_j)
//   S_8 = G_8 S_0 + sum_i (g_{i+1} .. g_8 k_i) u_i^T
// The triangular system does not involve the state, so it is solved beforehand, for the vectors and for the values:
//   w_j = beta_j G_j k_j - sum_{i<j} c_ij w_i,    x_j = beta_j v_j - sum_{i<j} c_ij x_i
//   r_j = G_j q_j - sum_{i<=j} m_ij w_i,          y_j = sum_{i<=j} m_ij x_i
//   u_j = x_j - S_0^T w_j,                        o_j = y_j + S_0^T r_j
// PREP writes a record per (head, block) with w, r, x, y, the decayed keys and G_8, all blocks in parallel. SCAN walks the
// blocks of a sequence: a warp owns 16 state columns and keeps them as the fp32 accumulator fragments of m16n8 tiles (16 value
// columns x 8 key channels). Those are at the same time, tile pair by tile pair, the A operand of the products with w and r
// (16 x 128 times 128 x 16); the results arrive in the places the update needs u in as its A operand, and the update
// accumulates onto the state (16 x 8 tokens times 8 tokens x 8 channels): the state never leaves the registers, and the lanes
// of a warp exchange nothing. The walk is a chain of dependent steps: where there are fewer column groups than the machine
// has schedulers, two or four warps share a group, each with its part of the key channels, and add up their partial results
// through shared memory. Decays, norms, inner products, the triangular solution and the decay of the state are fp32; what
// enters a product (state, vectors, u) is split into two bf16 terms, high part and remainder, and the three leading products
// are summed (about 16 significant bits, fp32 accumulation).
//
// The record holds the operands in fragment order (a lane's registers side by side), so the consumer reads 16 bytes per lane
// without bank conflicts; records are built in shared memory and leave, and come, as bulk copies.
#include "channel_delta.cuh"

namespace lb {
namespace {

constexpr int BT = 8;                      // tokens per block
constexpr int stages_of(int split) { return split == 1 ? 4 : 6; }      // two CTAs per SM

// record: KS = padded key channels / 16
__host__ __device__ constexpr int dot_bytes(int ks) { return ks * 1024; }        // [ks][2 tiles of 8 vectors][32 lanes][hi b0 b1, lo b0 b1]
__host__ __device__ constexpr int up_bytes(int ks) { return ks * 512; }          // [ks][32 lanes][tile 0 hi lo, tile 1 hi lo]
__host__ __device__ constexpr int dec_bytes(int ks) { return ks * 64; }          // [ks][4][tile 0 pair, tile 1 pair] of G_8
__host__ __device__ constexpr int head_bytes(int ks) { return dot_bytes(ks) + up_bytes(ks) + dec_bytes(ks); }
__host__ __device__ constexpr int pad16(int n) { return (n + 15) / 16 * 16; }
// + per 16 columns: [x, y][32 lanes][columns ca pair, cb pair of tokens 2 q, 2 q + 1]
__host__ __device__ constexpr int rec_bytes(int ks, int dv) { return head_bytes(ks) + pad16(dv) * 64; }
constexpr int SC_FLOATS = 128;                                                   // c [8][8] (row j), m [8][8] (row j), PREP only
// place of a lane's 16 bytes in its column group's part (both sides stay off each other's banks)
__device__ __forceinline__ int val_chunk(int lane, int group) { return lane ^ (lane >> 3) ^ ((group & 1) << 2); }
__host__ __device__ constexpr int steps_of(int dk) { return dk <= 32 ? 2 : dk <= 64 ? 4 : 8; }

// Two neighbouring columns as loaded: a bf16 pair. n_ok of them exist; VEC: aligned, both or none exist
template <bool VEC>
__device__ __forceinline__ uint32_t ld_pair(const __nv_bfloat16* p, int n_ok) {
  if constexpr (VEC) return n_ok > 0 ? *reinterpret_cast<const uint32_t*>(p) : 0u;
  const uint32_t lo = n_ok > 0 ? *reinterpret_cast<const uint16_t*>(p) : 0u;
  return n_ok > 1 ? lo | uint32_t(*reinterpret_cast<const uint16_t*>(p + 1)) << 16 : lo;
}
__device__ __forceinline__ float2 un_pair(uint32_t v) { return make_float2(__uint_as_float(v << 16), __uint_as_float(v & 0xffff0000u)); }

// The block's window of two channels: rows t0 - (KC - 1) .. t0 + 7; rows in front of the sequence come from its history
// ([KC - 1] rows C apart, bf16 values in fp32). KC 0: nothing is loaded ahead.
template <int KC>
struct Window { uint32_t u[KC > 0 ? KC - 1 + BT : 1]; };
template <int KC, bool VEC>
__device__ __forceinline__ void load_window(const __nv_bfloat16* x, long ld, const float* hist, long C, int n_ok, const DeltaBlock& b,
                                            Window<KC>& w) {
  if constexpr (KC > 0) {
    if (VEC && b.n == BT && b.t0 - (KC - 1) >= b.seq0) {      // all rows are there
      const __nv_bfloat16* p = x + long(b.t0 - (KC - 1)) * ld;
#pragma unroll
      for (int i = 0; i < KC - 1 + BT; ++i) {
        w.u[i] = n_ok > 0 ? *reinterpret_cast<const uint32_t*>(p) : 0u;
        p += ld;
      }
      return;
    }
#pragma unroll
    for (int i = 0; i < KC - 1 + BT; ++i) {
      const int s = b.t0 - (KC - 1) + i;
      if (s < b.seq0) {
        const float* p = hist + ((KC - 1) + (s - b.seq0)) * C;
        w.u[i] = pack_bf16x2(n_ok > 0 ? p[0] : 0.f, n_ok > 1 ? p[1] : 0.f);
      } else {
        w.u[i] = i - (KC - 1) < b.n ? ld_pair<VEC>(x + long(s) * ld, n_ok) : 0u;
      }
    }
  }
}
// Convolution + silu of the two channels for the block's tokens. taps: rows ws apart
template <int KC>
__device__ __forceinline__ void conv_pair(const Window<KC>& win, const __nv_bfloat16* x, long ld, const float* hist, long C,
                                          const float* w, int ws, int taps, int n_ok, const DeltaBlock& b, float (&y)[BT][2]) {
  if constexpr (KC > 0) {
#pragma unroll
    for (int t = 0; t < BT; ++t) y[t][0] = y[t][1] = 0.f;
#pragma unroll
    for (int k = 0; k < KC; ++k) {
      const float w0 = n_ok > 0 ? w[k * ws] : 0.f, w1 = n_ok > 1 ? w[k * ws + 1] : 0.f;
#pragma unroll
      for (int t = 0; t < BT; ++t) {
        const float2 u = un_pair(win.u[t + k]);
        y[t][0] = fmaf(w0, u.x, y[t][0]);
        y[t][1] = fmaf(w1, u.y, y[t][1]);
      }
    }
  } else {
#pragma unroll
    for (int t = 0; t < BT; ++t)
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        float acc = 0.f;
        for (int k = 0; k < taps && t < b.n && j < n_ok; ++k) {
          const int s = b.t0 + t - (taps - 1) + k;
          acc = fmaf(w[k * ws + j], s >= b.seq0 ? __bfloat162float(x[long(s) * ld + j]) : hist[((taps - 1) + (s - b.seq0)) * C + j], acc);
        }
        y[t][j] = acc;
      }
  }
#pragma unroll
  for (int t = 0; t < BT; ++t)
#pragma unroll
    for (int j = 0; j < 2; ++j) y[t][j] = t < b.n ? silu_t<__nv_bfloat16>(y[t][j]) : 0.f;
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

constexpr int PREP_BLOCKS = 4;             // blocks per warp (pair)

// A lane holds two neighbouring key channels; one warp per (head, block), or two (WPB) where a head has 128 of them.
template <int KS, int KC, bool VEC>
__global__ void __launch_bounds__(128, 4) delta_prep8_kernel(const ChannelDeltaArgs a, int lo, int hi, int n_blocks, uint8_t* rec) {
  using T = __nv_bfloat16;
  constexpr int WPB = KS == 8 ? 2 : 1, NB = 4 / WPB;        // blocks in flight per CTA
  extern __shared__ __align__(128) uint8_t smem[];
  __shared__ float part[NB][WPB][3][32];
  const int h = blockIdx.y, DK = a.DK, DV = a.DV, W = 2 * DK + DV, taps = a.KC;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, grp = warp / WPB, wp = warp % WPB;
  const int hk = h / (a.H / a.G);
  const int q0 = hk * DK, k0 = a.G * DK + hk * DK, v0 = 2 * a.G * DK + h * DV, C = 2 * a.G * DK + a.H * DV;
  const int R = rec_bytes(KS, DV);
  uint8_t* r = smem + grp * R;
  float* sc = reinterpret_cast<float*>(smem + NB * R) + grp * SC_FLOATS;
  float* w_s = reinterpret_cast<float*>(smem + NB * R) + NB * SC_FLOATS;      // taps of the head's q | k | v channels, [taps][2 dk + dv]
  for (int i = threadIdx.x; i < W * taps; i += 128) {
    const int c = i % W, j = i / W;
    w_s[i] = a.conv_w[long(j) * C + (c < DK ? q0 + c : c < 2 * DK ? k0 + c - DK : v0 + c - 2 * DK)];
  }
  auto group_sync = [&] {
    if constexpr (WPB == 1) __syncwarp();
    else asm volatile("bar.sync %0, 64;" ::"r"(1 + grp) : "memory");
  };
  griddep_wait();
  __syncthreads();
  const float Ah = a.A[h];
  const T* x = static_cast<const T*>(a.qkv);
  const int c0 = (wp * 32 + lane) * 2, n_ok = max(0, min(2, DK - c0));
  const bool has = c0 < KS * 16;                            // (32 channels: half of the lanes have none)
  const T* ap = static_cast<const T*>(a.a) + long(h) * DK + c0;
  const float db0 = n_ok > 0 ? a.dt_bias[long(h) * DK + c0] : 0.f, db1 = n_ok > 1 ? a.dt_bias[long(h) * DK + c0 + 1] : 0.f;
  if (wp == 0)
    for (int i = lane; i < SC_FLOATS; i += 32) sc[i] = 0.f;                      // above the diagonals
  const int blk0 = (blockIdx.x * NB + grp) * PREP_BLOCKS, blk1 = min(n_blocks, blk0 + PREP_BLOCKS);
  for (int blk = blk0; blk < blk1; ++blk) {
    DeltaBlock b;
    if (!find_block<BT>(a.cu, a.n_seqs, lo, hi, blk, b)) continue;
    const float* hist = a.conv_state + long(a.slots[b.seq]) * C * (taps - 1);
    float q[BT][2], k[BT][2], g[BT][2];
    {
      Window<KC> wq, wk;
      uint32_t ra[BT];
      load_window<KC, VEC>(x + q0 + c0, a.ld, hist + q0 + c0, C, n_ok, b, wq);
      load_window<KC, VEC>(x + k0 + c0, a.ld, hist + k0 + c0, C, n_ok, b, wk);
#pragma unroll
      for (int t = 0; t < BT; ++t) ra[t] = t < b.n ? ld_pair<VEC>(ap + long(b.t0 + t) * a.lda, n_ok) : 0u;
      conv_pair<KC>(wq, x + q0 + c0, a.ld, hist + q0 + c0, C, w_s + c0, W, taps, n_ok, b, q);
      conv_pair<KC>(wk, x + k0 + c0, a.ld, hist + k0 + c0, C, w_s + DK + c0, W, taps, n_ok, b, k);
#pragma unroll
      for (int t = 0; t < BT; ++t) {
        const float2 z = un_pair(ra[t]);
        g[t][0] = t < b.n && n_ok > 0 ? decay_t<T>(z.x + db0, Ah) : 1.f;
        g[t][1] = t < b.n && n_ok > 1 ? decay_t<T>(z.y + db1, Ah) : 1.f;
      }
    }
    const float be = lane < b.n && lane < BT ? sigmoid_t<T>(ld_f(static_cast<const T*>(a.b) + long(b.t0 + lane) * a.ldb + h)) : 0.f;
    // ---- inner products
    auto products = [&](int i, float* m, float* c) {      // m[j - i] for j >= i, c[j - i - 1] for j > i
      float kd0 = k[i][0], kd1 = k[i][1];
      m[0] = fmaf(kd0, q[i][0], kd1 * q[i][1]);
#pragma unroll
      for (int j = 0; j < BT; ++j)
        if (j > i) {
          kd0 *= g[j][0];
          kd1 *= g[j][1];
          m[j - i] = fmaf(kd0, q[j][0], kd1 * q[j][1]);
          c[j - i - 1] = fmaf(kd0, k[j][0], kd1 * k[j][1]);
        }
    };
    float sum[3];
    {
      float s[32];
#pragma unroll
      for (int t = 0; t < BT; ++t) {
        s[t] = fmaf(q[t][0], q[t][0], q[t][1] * q[t][1]);
        s[8 + t] = fmaf(k[t][0], k[t][0], k[t][1] * k[t][1]);
      }
      products(0, s + 16, s + 24);
      s[31] = 0.f;
      sum[0] = transpose_sum(s);
    }
    {
      float s[32];
      products(1, s, s + 7);
      products(2, s + 13, s + 19);
      products(7, s + 24, s + 25);
      products(6, s + 25, s + 27);
#pragma unroll
      for (int i = 28; i < 32; ++i) s[i] = 0.f;
      sum[1] = transpose_sum(s);
    }
    {
      float s[32];
      products(3, s, s + 5);
      products(4, s + 9, s + 13);
      products(5, s + 16, s + 19);
#pragma unroll
      for (int i = 21; i < 32; ++i) s[i] = 0.f;
      sum[2] = transpose_sum(s);
    }
    // the record this group wrote before has left its shared memory
    if (wp == 0 && lane == 0) asm volatile("cp.async.bulk.wait_group.read 0;" ::: "memory");
    if constexpr (WPB == 2) {
#pragma unroll
      for (int e = 0; e < 3; ++e) part[grp][wp][e][lane] = sum[e];
    }
    group_sync();
    if constexpr (WPB == 2) {
#pragma unroll
      for (int e = 0; e < 3; ++e) sum[e] = part[grp][0][e][lane] + part[grp][1][e][lane];
    }
    float rq[BT], rk[BT], bb[BT];
    {
      const float inv = 1.f / sqrtf(sum[0] + a.l2_eps);
#pragma unroll
      for (int t = 0; t < BT; ++t) {
        rq[t] = __shfl_sync(0xffffffffu, inv, t) * a.scale;
        rk[t] = __shfl_sync(0xffffffffu, inv, 8 + t);
        bb[t] = __shfl_sync(0xffffffffu, be, t);
      }
    }
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
    if (wp == 0) place(0, sum[0]);
    if (wp == WPB - 1) place(1, sum[1]);
    if (wp == 0) place(2, sum[2]);
    // the values: the loads go out here
    const int vc = 2 * (wp * 32 + lane), v_ok = max(0, min(2, DV - vc));
    Window<KC> wv;
    load_window<KC, VEC>(x + v0 + vc, a.ld, hist + v0 + vc, C, v_ok, b, wv);
    group_sync();
    // row j of c and m, on every lane
    auto row8 = [&](const float* p, float (&v)[BT]) {
      const float4 f = *reinterpret_cast<const float4*>(p), e = *reinterpret_cast<const float4*>(p + 4);
      v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w;
      v[4] = e.x; v[5] = e.y; v[6] = e.z; v[7] = e.w;
    };
    // ---- operands in fragment order; 16-byte chunks of a step s are permuted by s (lane chunk ^ s), which keeps both the
    // writes here and the reads of the consumer off each other's banks
    const int ks = c0 >> 4, kk = c0 & 15;                  // the lane's step, first channel inside it (even)
    if (has) {
      float G0 = 1.f, G1 = 1.f;
      uint8_t* dot = r + ks * 1024 + (kk >> 3) * 4;
      auto put_dot = [&](int vec, float v0_, float v1_) {
        uint8_t* p = dot + (vec >> 3) * 512 + ((((vec & 7) * 4 + ((kk & 7) >> 1)) ^ (ks & 7)) << 4);
        const uint32_t hi_ = pack_bf16x2(v0_, v1_);
        const float2 hf = un_pair(hi_);
        *reinterpret_cast<uint32_t*>(p) = hi_;
        *reinterpret_cast<uint32_t*>(p + 8) = pack_bf16x2(v0_ - hf.x, v1_ - hf.y);
      };
      float w0[BT], w1[BT];
#pragma unroll
      for (int t = 0; t < BT; ++t) {
        const float fd = bb[t] * rk[t];
        float cr[BT], mr[BT];
        row8(sc + t * 8, cr);
        row8(sc + 64 + t * 8, mr);
        G0 *= g[t][0];
        G1 *= g[t][1];
        w0[t] = G0 * (k[t][0] * fd);
        w1[t] = G1 * (k[t][1] * fd);
        float r0 = G0 * (q[t][0] * rq[t]), r1 = G1 * (q[t][1] * rq[t]);
#pragma unroll
        for (int i = 0; i < t; ++i) {
          w0[t] = fmaf(-cr[i], w0[i], w0[t]);
          w1[t] = fmaf(-cr[i], w1[i], w1[t]);
        }
#pragma unroll
        for (int i = 0; i <= t; ++i) {
          r0 = fmaf(-mr[i], w0[i], r0);
          r1 = fmaf(-mr[i], w1[i], r1);
        }
        put_dot(t, w0[t], w1[t]);
        put_dot(8 + t, r0, r1);
      }
      *reinterpret_cast<float2*>(r + dot_bytes(KS) + up_bytes(KS) + ks * 64 + ((kk & 7) >> 1) * 16 + (kk >> 3) * 8) = make_float2(G0, G1);
#pragma unroll
      for (int n = 0; n < 2; ++n) {
        float D = 1.f, u[BT];
#pragma unroll
        for (int t = BT - 1; t >= 0; --t) {
          u[t] = D * (k[t][n] * rk[t]);
          D *= g[t][n];
        }
#pragma unroll
        for (int p = 0; p < BT / 2; ++p) {                 // token pair p of the channel: tile kk / 8 of the step, lane (channel % 8) * 4 + p
          const uint32_t hi_ = pack_bf16x2(u[2 * p], u[2 * p + 1]);
          const float2 hf = un_pair(hi_);
          *reinterpret_cast<uint2*>(r + dot_bytes(KS) + ks * 512 + (((((kk & 7) + n) * 4 + p) ^ (ks & 7)) << 4) + (kk >> 3) * 8) =
              make_uint2(hi_, pack_bf16x2(u[2 * p] - hf.x, u[2 * p + 1] - hf.y));
        }
      }
    }
    for (int c = vc; c < pad16(DV); c += 64 * WPB) {
      const int ok = max(0, min(2, DV - c));
      if (c != vc) load_window<KC, VEC>(x + v0 + c, a.ld, hist + v0 + c, C, ok, b, wv);
      float v[BT][2], y[BT][2];
      conv_pair<KC>(wv, x + v0 + c, a.ld, hist + v0 + c, C, w_s + 2 * DK + c, W, taps, ok, b, v);
#pragma unroll
      for (int t = 0; t < BT; ++t) {
        float cr[BT], mr[BT];
        row8(sc + t * 8, cr);
        row8(sc + 64 + t * 8, mr);
#pragma unroll
        for (int n = 0; n < 2; ++n) {
          v[t][n] *= bb[t];
#pragma unroll
          for (int i = 0; i < t; ++i) v[t][n] = fmaf(-cr[i], v[i][n], v[t][n]);
          y[t][n] = mr[0] * v[0][n];
#pragma unroll
          for (int i = 1; i <= t; ++i) y[t][n] = fmaf(mr[i], v[i][n], y[t][n]);
        }
      }
      const int cg = c >> 4;
      uint8_t* vp = r + head_bytes(KS) + cg * 1024 + ((c >> 3) & 1) * 8;
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int p = 0; p < BT / 2; ++p) {
          uint8_t* d = vp + val_chunk(((c & 7) + n) * 4 + p, cg) * 16;
          *reinterpret_cast<float2*>(d) = make_float2(v[2 * p][n], v[2 * p + 1][n]);
          *reinterpret_cast<float2*>(d + 512) = make_float2(y[2 * p][n], y[2 * p + 1][n]);
        }
    }
    fence_proxy_async_smem();
    group_sync();
    if (wp == 0 && lane == 0) bulk_store(rec + (long(h) * n_blocks + blk) * R, r, R);
  }
  if (wp == 0 && lane == 0) asm volatile("cp.async.bulk.wait_group 0;" ::: "memory");
  griddep_launch();      // not earlier: waiting CTAs of SCAN would take this kernel's shared memory
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

// grid (H * column groups, sequences), 160 threads: SPLIT of warps 0..3 own sixteen columns each, warp 4 copies the records.
template <int KS, int SPLIT>
__global__ void __launch_bounds__(160) delta_scan8_kernel(const ChannelDeltaArgs a, int lo, int hi, int n_blocks, const uint8_t* rec,
                                                          int* status) {
  constexpr int CPC = 64 / SPLIT, HEAD = head_bytes(KS), STAGE = HEAD + CPC * 64;
  constexpr int NS = KS / SPLIT;                           // steps of sixteen key channels per warp
  constexpr int STAGES = stages_of(SPLIT);
  extern __shared__ __align__(128) uint8_t smem[];         // [STAGES][STAGE]
  __shared__ __align__(8) uint64_t full[STAGES], empty[STAGES];
  __shared__ int abort_s;
  __shared__ float4 xs[SPLIT > 1 ? 4 / SPLIT : 1][2][SPLIT][2][32];      // partial results: [group][parity][part][tile][lane]
  volatile int* abort_flag = &abort_s;
  const int DK = a.DK, DV = a.DV, groups = (DV + CPC - 1) / CPC;
  const int h = blockIdx.x / groups, col0 = (blockIdx.x % groups) * CPC, seq = blockIdx.y;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int n_warps = min(4, (DV - col0 + 15) / 16 * SPLIT);      // warps with columns
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
      const int vbytes = min(CPC, pad16(DV) - col0) * 64;
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
        bulk_load(smem + s * STAGE + HEAD, src + HEAD + col0 * 64, vbytes, &full[s]);
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
  const int grp = warp / SPLIT, part = warp % SPLIT;
  const int q = lane & 3, ca = col0 + grp * 16 + (lane >> 2), cb = ca + 8;
  float* st = a.state + (long(slot) * a.H + h) * DV * DK;
  // S[t]: key channels k0 + 8 t + 2 q, + 1 of columns ca (0, 1) and cb (2, 3)
  const int k0 = part * NS * 16;
  float S[2 * NS][4];
#pragma unroll
  for (int t = 0; t < 2 * NS; ++t)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int c = e < 2 ? ca : cb, k = k0 + 8 * t + 2 * q + (e & 1);
      S[t][e] = c < DV && k < DK ? st[long(c) * DK + k] : 0.f;
    }
  bool ok = true;      // a wait that runs out does not leave the loop: the warps of a group keep meeting at their barrier
  auto* out = static_cast<__nv_bfloat16*>(a.out) + long(h) * DV;
  auto stage = [&](int i) -> const uint8_t* {              // block i's record, once it has landed
    if (ok && !__all_sync(0xffffffffu, mbar_wait(&full[i % STAGES], (i / STAGES) & 1, abort_flag))) {
      *abort_flag = 1;
      if (lane == 0) atomicCAS(status, 0, ST_TIMEOUT_FULL | SITE_DELTA_SCAN);
      ok = false;
    }
    return smem + (i % STAGES) * STAGE;
  };
  // a block's operands; warps with few steps fetch those of the next block while they wait for each other
  constexpr bool AHEAD = NS <= 2;
  struct Ops {
    uint4 dot[AHEAD ? NS : 1][2], up[AHEAD ? NS : 1];
    float4 g[AHEAD ? NS : 1], xv, yv;
  };
  auto dot_of = [&](const uint8_t* v, int gs, int n) { return *reinterpret_cast<const uint4*>(v + (gs * 2 + n) * 512 + ((lane ^ (gs & 7)) << 4)); };
  auto up_of = [&](const uint8_t* v, int gs) { return *reinterpret_cast<const uint4*>(v + dot_bytes(KS) + gs * 512 + ((lane ^ (gs & 7)) << 4)); };
  auto dec_of = [&](const uint8_t* v, int gs) { return *reinterpret_cast<const float4*>(v + dot_bytes(KS) + up_bytes(KS) + gs * 64 + q * 16); };
  const int val_off = HEAD + grp * 1024 + val_chunk(lane, (col0 >> 4) + grp) * 16;
  const int comp = (part >> 1) * 2 + (part & 1);           // with four warps: the output (column, token) that is this warp's
  auto fetch = [&](const uint8_t* v, Ops& o) {
    if constexpr (AHEAD) {
#pragma unroll
      for (int s = 0; s < NS; ++s) {
        o.dot[s][0] = dot_of(v, part * NS + s, 0);
        o.dot[s][1] = dot_of(v, part * NS + s, 1);
      }
    }
    o.xv = *reinterpret_cast<const float4*>(v + val_off);
    if constexpr (SPLIT == 4) o.yv.x = *reinterpret_cast<const float*>(v + val_off + 512 + comp * 4);
    else o.yv = *reinterpret_cast<const float4*>(v + val_off + 512);
    if constexpr (AHEAD) {
#pragma unroll
      for (int s = 0; s < NS; ++s) {
        o.up[s] = up_of(v, part * NS + s);
        o.g[s] = dec_of(v, part * NS + s);
      }
    }
  };
  auto block = [&](int i, Ops& o, Ops& next) {
    const uint8_t* v = smem + (i % STAGES) * STAGE;
    // ---- products with w (tile 0) and r (tile 1): a lane gets tokens 2 q, 2 q + 1 of columns ca (0, 1) and cb (2, 3)
    float acc[2][3][4];
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int p = 0; p < 3; ++p)
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[n][p][e] = 0.f;
#pragma unroll
    for (int s = 0; s < NS; ++s) {
      const int gs = part * NS + s;                        // step of the head
      uint32_t h0, h1, h2, h3, l0, l1, l2, l3;
      split2(S[2 * s][0], S[2 * s][1], h0, l0);
      split2(S[2 * s][2], S[2 * s][3], h1, l1);
      split2(S[2 * s + 1][0], S[2 * s + 1][1], h2, l2);
      split2(S[2 * s + 1][2], S[2 * s + 1][3], h3, l3);
#pragma unroll
      for (int n = 0; n < 2; ++n) {
        const uint4 f = AHEAD ? o.dot[AHEAD ? s : 0][n] : dot_of(v, gs, n);
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
    if constexpr (SPLIT > 1) {
#pragma unroll
      for (int n = 0; n < 2; ++n) xs[grp][i & 1][part][n][lane] = make_float4(x[n][0], x[n][1], x[n][2], x[n][3]);
      asm volatile("bar.sync %0, %1;" ::"r"(1 + grp), "n"(32 * SPLIT) : "memory");
      float4 f[SPLIT], r[SPLIT];
#pragma unroll
      for (int p = 0; p < SPLIT; ++p) {
        f[p] = xs[grp][i & 1][p][0][lane];
        if constexpr (SPLIT == 4) r[p].x = reinterpret_cast<const float*>(&xs[grp][i & 1][p][1][lane])[comp];
        else r[p] = xs[grp][i & 1][p][1][lane];
      }
#pragma unroll
      for (int p = 1; p < SPLIT; ++p) {                    // the same order on every warp
        f[0].x += f[p].x; f[0].y += f[p].y; f[0].z += f[p].z; f[0].w += f[p].w;
        r[0].x += r[p].x;
        if constexpr (SPLIT != 4) { r[0].y += r[p].y; r[0].z += r[p].z; r[0].w += r[p].w; }
      }
      x[0][0] = f[0].x; x[0][1] = f[0].y; x[0][2] = f[0].z; x[0][3] = f[0].w;
      x[1][0] = r[0].x; x[1][1] = r[0].y; x[1][2] = r[0].z; x[1][3] = r[0].w;
    }
    if (i + 1 < n_blk) fetch(stage(i + 1), next);
    // ---- state: decay, then the eight writes. A operand: u of tokens 2 q, 2 q + 1 of both columns, high parts and remainders
    uint32_t ah, al, bh, bl;
    split2(o.xv.x - x[0][0], o.xv.y - x[0][1], ah, al);
    split2(o.xv.z - x[0][2], o.xv.w - x[0][3], bh, bl);
#pragma unroll
    for (int s = 0; s < NS; ++s) {
      const int gs = part * NS + s;
      const float4 g = AHEAD ? o.g[AHEAD ? s : 0] : dec_of(v, gs);
      const uint4 f = AHEAD ? o.up[AHEAD ? s : 0] : up_of(v, gs);
      S[2 * s][0] *= g.x; S[2 * s][1] *= g.y; S[2 * s][2] *= g.x; S[2 * s][3] *= g.y;
      S[2 * s + 1][0] *= g.z; S[2 * s + 1][1] *= g.w; S[2 * s + 1][2] *= g.z; S[2 * s + 1][3] *= g.w;
      mma16(S[2 * s], ah, bh, al, bl, f.x, f.x);
      mma8(S[2 * s], ah, bh, f.y);
      mma16(S[2 * s + 1], ah, bh, al, bl, f.z, f.z);
      mma8(S[2 * s + 1], ah, bh, f.w);
    }
    __syncwarp();
    if (lane == 0) mbar_arrive(&empty[i % STAGES]);
    // ---- outputs, shared out among the warps of the group: by column with two, by column and token with four
    const int t = s0 + i * BT + 2 * q;
    auto put = [&](int tok, int col, float val) {
      if (tok < s1 && col < DV) out[long(tok) * a.ldo + col] = __float2bfloat16(val);
    };
    if constexpr (SPLIT == 4) {
      put(t + (part & 1), part < 2 ? ca : cb, o.yv.x + x[1][0]);
    } else {
      if (SPLIT == 1 || part == 0) {
        put(t, ca, o.yv.x + x[1][0]);
        put(t + 1, ca, o.yv.y + x[1][1]);
      }
      if (SPLIT == 1 || part == 1) {
        put(t, cb, o.yv.z + x[1][2]);
        put(t + 1, cb, o.yv.w + x[1][3]);
      }
    }
  };
  Ops even, odd;
  fetch(stage(0), even);
  for (int i = 0; i < n_blk; i += 2) {
    block(i, even, odd);
    if (i + 1 < n_blk) block(i + 1, odd, even);
  }
  if (a.write_state && !*abort_flag) {
#pragma unroll
    for (int t = 0; t < 2 * NS; ++t)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int c = e < 2 ? ca : cb, k = k0 + 8 * t + 2 * q + (e & 1);
        if (c < DV && k < DK) st[long(c) * DK + k] = S[t][e];
      }
  }
}

constexpr long SPLIT4_GROUPS = 300, SPLIT2_GROUPS = 1200;
constexpr int in_flight(int ks) { return ks == 8 ? 2 : 4; }      // blocks per PREP CTA

template <int KS, int KC>
int prep_k(const ChannelDeltaArgs& a, int lo, int hi, int nb, uint8_t* rec, bool vec, cudaStream_t s) {
  constexpr int NB = in_flight(KS);
  const dim3 grid((nb + NB * PREP_BLOCKS - 1) / (NB * PREP_BLOCKS), a.H);
  const int smem = NB * (rec_bytes(KS, a.DV) + SC_FLOATS * 4) + (2 * a.DK + a.DV) * a.KC * 4;
  auto k1 = delta_prep8_kernel<KS, KC, true>;
  auto k0 = delta_prep8_kernel<KS, KC, false>;
  auto kfn = vec ? k1 : k0;
  if (smem > 200 * 1024 || cudaFuncSetAttribute(kfn, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess) return 1;
  return launch_pdl(kfn, grid, dim3(128), smem, s, a, lo, hi, nb, rec) != cudaSuccess;
}

template <int KS, int SPLIT>
int scan_k(const ChannelDeltaArgs& a, int lo, int hi, int nb, const uint8_t* rec, int* status, cudaStream_t s) {
  constexpr int CPC = 64 / SPLIT;
  const int smem = stages_of(SPLIT) * (head_bytes(KS) + CPC * 64);
  auto kfn = delta_scan8_kernel<KS, SPLIT>;
  if (cudaFuncSetAttribute(kfn, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess) return 1;
  return launch_pdl(kfn, dim3(a.H * ((a.DV + CPC - 1) / CPC), a.n_seqs), dim3(160), smem, s, a, lo, hi, nb, rec, status) !=
         cudaSuccess;
}

template <int KS>
int slice_k(const ChannelDeltaArgs& a, int lo, int hi, int nb, uint8_t* rec, bool vec, int* status, cudaStream_t s) {
  int rc;
  if (a.KC == 4) rc = prep_k<KS, 4>(a, lo, hi, nb, rec, vec, s);
  else if (a.KC == 3) rc = prep_k<KS, 3>(a, lo, hi, nb, rec, vec, s);
  else if (a.KC == 2) rc = prep_k<KS, 2>(a, lo, hi, nb, rec, vec, s);
  else rc = prep_k<KS, 0>(a, lo, hi, nb, rec, vec, s);
  if (rc) return 1;
  // a warp per column group, or two or four while there are schedulers without one
  const long groups = long(a.H) * (pad16(a.DV) / 16) * a.n_seqs;
  if (KS >= 4 && groups <= SPLIT4_GROUPS) return scan_k<KS, (KS >= 4 ? 4 : 2)>(a, lo, hi, nb, rec, status, s);
  if (groups <= SPLIT2_GROUPS) return scan_k<KS, 2>(a, lo, hi, nb, rec, status, s);
  return scan_k<KS, 1>(a, lo, hi, nb, rec, status, s);
}

}  // namespace

bool channel_delta_mma_ok(const ChannelDeltaArgs& a) {
  return a.DK <= 128 && in_flight(steps_of(a.DK)) * (rec_bytes(steps_of(a.DK), a.DV) + SC_FLOATS * 4) + (2 * a.DK + a.DV) * a.KC * 4 <= 200 * 1024;
}

long channel_delta_mma_floats(int H, int DK, int DV) { return DK > 128 ? 0 : long(rec_bytes(steps_of(DK), DV)) / 4 * H; }

int channel_delta_mma_launch(const ChannelDeltaArgs& a, float* rec, long rec_floats, int* status, cudaStream_t s) {
  const int ks = steps_of(a.DK);
  const long blocks = rec_floats / channel_delta_mma_floats(a.H, a.DK, a.DV);       // records the scratch holds, per head
  const long tokens = (blocks - a.n_seqs) * BT;
  if (tokens < BT || (tokens < a.T && !a.write_state)) return 1;      // slices hand the state on through the pool
  auto al = [](const void* p, size_t n) { return reinterpret_cast<uintptr_t>(p) % n == 0; };
  const bool vec = a.DK % 2 == 0 && a.DV % 2 == 0 && a.ld % 2 == 0 && a.lda % 2 == 0 && al(a.qkv, 4) && al(a.a, 4);
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
