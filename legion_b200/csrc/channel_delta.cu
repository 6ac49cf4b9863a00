// Gated delta rule with a decay per head and key channel (fp32 state, kept as [value column][key channel]):
//   S = diag(g_t) S,  u = beta_t (v_t - S^T k_t),  S += k_t u^T,  o_t = S^T q_t
// with q, k and v behind a short causal convolution and silu, unit q and k per head, g = exp(A softplus(a + bias)).
//
// Prompts take the tokens in blocks of four. With everything but the state known beforehand, the four updates of a block
// become one: let G_j = g_1 .. g_j inside the block, then
//   d_j = S_0^T (G_j k_j),   e_j = S_0^T (G_j q_j)                       eight products with the state in front of the block
//   u_j = beta_j (v_j - d_j - sum_{i<j} c_ij u_i),  c_ij = k_i . (g_{i+1} .. g_j k_j)
//   o_j = e_j + sum_{i<=j} m_ij u_i,                m_ij = k_i . (g_{i+1} .. g_j q_j)
//   S_4 = G_4 S_0 + sum_i (g_{i+1} .. g_4 k_i) u_i^T
// so one pass over the state serves four tokens, every decay product is at most 1 (nothing can overflow, whatever the decay),
// and all of it is fp32 arithmetic. PREP computes a record per (block, head) for all blocks in parallel: convolution, silu,
// norms, decays, the decayed vectors and the 16 inner products. SCAN walks the blocks of a sequence; columns of the state are
// independent, so a warp owns four of them (eight lanes per column) with the state in registers, and the records stream
// through shared memory by bulk copies. Steps whose records would not fit the scratch run in slices of tokens.
// This file's form serves fp32 and head sizes of any kind; bf16 prompts run the same algebra with blocks of eight tokens and
// the products on tensor cores (channel_delta_mma.cu).
//
// Decode steps are one launch: history and convolution, decays, update, RMS norm per head and output gate.
#include "channel_delta.cuh"
#include "state_cols.cuh"

namespace lb {
namespace {

constexpr int BT = 4;                    // tokens per block
constexpr int NVEC = 13;                 // vectors of a record: G_j k_j, G_j q_j (j = 1..4), G_4, g_{i+1} .. g_4 k_i (i = 1..4)
constexpr int NSCAL = 32;                // scalars of a record: beta 0..3 | c 12 13 14 23 24 34 | m 11 12 13 14 22 23 24 33 34 44
constexpr int COLS = 16;                 // state columns per SCAN CTA (four warps of four)
constexpr int STAGES = 6;

__host__ __device__ constexpr int pad_dk(int dk) { return dk <= 32 ? 32 : dk <= 64 ? 64 : dk <= 128 ? 128 : 256; }
__host__ __device__ constexpr int pad_dv(int dv) { return (dv + COLS - 1) / COLS * COLS; }
__host__ __device__ constexpr long record_floats(int dkp, int dvp) { return long(NVEC) * dkp + NSCAL + BT * dvp; }

// Convolution + silu of one channel for the block's tokens; rows in front of the sequence come from its history (rows hs
// apart). KC 0: any number of taps (taps of a channel ws_stride apart).
template <typename T, int KC>
__device__ __forceinline__ void conv_block(const T* x, long ld, const float* hist, long hs, const float* w, int ws_stride, int taps,
                                           const DeltaBlock& b, float (&y)[BT]) {
  if constexpr (KC > 0) {
    float u[KC - 1 + BT];
#pragma unroll
    for (int i = 0; i < KC - 1 + BT; ++i) {
      const int s = b.t0 - (KC - 1) + i;
      u[i] = s >= b.seq0 ? (i - (KC - 1) < b.n ? ld_f(x + long(s) * ld) : 0.f) : hist[((KC - 1) + (s - b.seq0)) * hs];
    }
#pragma unroll
    for (int t = 0; t < BT; ++t) {
      float acc = 0.f;
#pragma unroll
      for (int j = 0; j < KC; ++j) acc = fmaf(w[j * ws_stride], u[t + j], acc);
      y[t] = silu_t<T>(acc);
    }
  } else {
#pragma unroll
    for (int t = 0; t < BT; ++t) {
      float acc = 0.f;
      for (int j = 0; j < taps && t < b.n; ++j) {
        const int s = b.t0 + t - (taps - 1) + j;
        acc = fmaf(w[j * ws_stride], s >= b.seq0 ? ld_f(x + long(s) * ld) : hist[((taps - 1) + (s - b.seq0)) * hs], acc);
      }
      y[t] = silu_t<T>(acc);
    }
  }
}

constexpr int PREP_BLOCKS = 4;           // blocks per warp

// NC: key channels per lane (channel = lane + 32 i)
template <typename T, int NC, int KC>
__global__ void __launch_bounds__(128) delta_prep_kernel(const ChannelDeltaArgs a, int lo, int hi, int n_blocks, float* rec) {
  extern __shared__ float w_s[];         // taps of the head's q | k | v channels, [taps][2 dk + dv]
  const int h = blockIdx.y, DK = a.DK, DV = a.DV, W = 2 * DK + DV, taps = a.KC;
  const int hk = h / (a.H / a.G), lane = threadIdx.x & 31;
  const int q0 = hk * DK, k0 = a.G * DK + hk * DK, v0 = 2 * a.G * DK + h * DV, C = 2 * a.G * DK + a.H * DV;
  for (int i = threadIdx.x; i < W * taps; i += 128) {
    const int c = i % W, j = i / W;
    const int ch = c < DK ? q0 + c : c < 2 * DK ? k0 + c - DK : v0 + c - 2 * DK;
    w_s[i] = a.conv_w[long(j) * C + ch];
  }
  griddep_wait();
  griddep_launch();
  __syncthreads();
  constexpr int DKP = 32 * NC;
  const int DVP = pad_dv(DV);
  const float Ah = a.A[h];
  const T* x = static_cast<const T*>(a.qkv);
  const T* ap = static_cast<const T*>(a.a) + long(h) * DK;
  const int blk0 = (blockIdx.x * 4 + (threadIdx.x >> 5)) * PREP_BLOCKS;
  for (int blk = blk0; blk < min(n_blocks, blk0 + PREP_BLOCKS); ++blk) {
    DeltaBlock b;
    if (!find_block<BT>(a.cu, a.n_seqs, lo, hi, blk, b)) continue;
    const float* hist = a.conv_state + long(a.slots[b.seq]) * C * (taps - 1);
    float* r = rec + (long(h) * n_blocks + blk) * record_floats(DKP, DVP);
    float q[NC][BT], k[NC][BT], g[NC][BT], s[32];
#pragma unroll
    for (int i = 0; i < 32; ++i) s[i] = 0.f;
#pragma unroll
    for (int i = 0; i < NC; ++i) {
      const int c = lane + 32 * i;
      if (c < DK) {
        conv_block<T, KC>(x + q0 + c, a.ld, hist + q0 + c, C, w_s + c, W, taps, b, q[i]);
        conv_block<T, KC>(x + k0 + c, a.ld, hist + k0 + c, C, w_s + DK + c, W, taps, b, k[i]);
        const float db = a.dt_bias[long(h) * DK + c];
#pragma unroll
        for (int t = 0; t < BT; ++t) {
          if (t < b.n) {
            g[i][t] = decay_t<T>(ld_f(ap + long(b.t0 + t) * a.lda + c) + db, Ah);
          } else {
            q[i][t] = k[i][t] = 0.f;
            g[i][t] = 1.f;
          }
        }
      } else {
#pragma unroll
        for (int t = 0; t < BT; ++t) { q[i][t] = k[i][t] = 0.f; g[i][t] = 1.f; }
      }
      // sums of squares, and the inner products of the raw vectors
      const float g23 = g[i][1] * g[i][2], g34 = g[i][2] * g[i][3], g234 = g23 * g[i][3];
#pragma unroll
      for (int t = 0; t < BT; ++t) {
        s[t] = fmaf(q[i][t], q[i][t], s[t]);
        s[4 + t] = fmaf(k[i][t], k[i][t], s[4 + t]);
      }
      const float k0g2 = k[i][0] * g[i][1], k0g3 = k[i][0] * g23, k0g4 = k[i][0] * g234, k1g3 = k[i][1] * g[i][2],
                  k1g4 = k[i][1] * g34, k2g4 = k[i][2] * g[i][3];
      s[8] = fmaf(k0g2, k[i][1], s[8]);
      s[9] = fmaf(k0g3, k[i][2], s[9]);
      s[10] = fmaf(k0g4, k[i][3], s[10]);
      s[11] = fmaf(k1g3, k[i][2], s[11]);
      s[12] = fmaf(k1g4, k[i][3], s[12]);
      s[13] = fmaf(k2g4, k[i][3], s[13]);
      s[14] = fmaf(k[i][0], q[i][0], s[14]);
      s[15] = fmaf(k0g2, q[i][1], s[15]);
      s[16] = fmaf(k0g3, q[i][2], s[16]);
      s[17] = fmaf(k0g4, q[i][3], s[17]);
      s[18] = fmaf(k[i][1], q[i][1], s[18]);
      s[19] = fmaf(k1g3, q[i][2], s[19]);
      s[20] = fmaf(k1g4, q[i][3], s[20]);
      s[21] = fmaf(k[i][2], q[i][2], s[21]);
      s[22] = fmaf(k2g4, q[i][3], s[22]);
      s[23] = fmaf(k[i][3], q[i][3], s[23]);
    }
    const float mine = transpose_sum(s);
    float rq[BT], rk[BT];
    {
      const float inv = 1.f / sqrtf(mine + a.l2_eps);
#pragma unroll
      for (int t = 0; t < BT; ++t) {
        rq[t] = __shfl_sync(0xffffffffu, inv, t) * a.scale;
        rk[t] = __shfl_sync(0xffffffffu, inv, 4 + t);
      }
    }
    {
      // (i, j) of the products held by lanes 8..23: two bits each
      constexpr uint32_t I = 0u | (0u << 2) | (0u << 4) | (1u << 6) | (1u << 8) | (2u << 10) | (0u << 12) | (0u << 14) |
                             (0u << 16) | (0u << 18) | (1u << 20) | (1u << 22) | (1u << 24) | (2u << 26) | (2u << 28) | (3u << 30);
      constexpr uint32_t J = 1u | (2u << 2) | (3u << 4) | (2u << 6) | (3u << 8) | (3u << 10) | (0u << 12) | (1u << 14) |
                             (2u << 16) | (3u << 18) | (1u << 20) | (2u << 22) | (3u << 24) | (2u << 26) | (3u << 28) | (3u << 30);
      const int p = 2 * ((lane - 8) & 15), i = (I >> p) & 3, j = (J >> p) & 3;
      const float ri = i == 0 ? rk[0] : i == 1 ? rk[1] : i == 2 ? rk[2] : rk[3];
      const float kj = j == 0 ? rk[0] : j == 1 ? rk[1] : j == 2 ? rk[2] : rk[3];
      const float qj = j == 0 ? rq[0] : j == 1 ? rq[1] : j == 2 ? rq[2] : rq[3];
      float* sc = r + NVEC * DKP;
      if (lane >= 8 && lane < 24) sc[lane - 4] = mine * ri * (lane < 14 ? kj : qj);
      if (lane < BT)
        sc[lane] = lane < b.n ? sigmoid_t<T>(ld_f(static_cast<const T*>(a.b) + long(b.t0 + lane) * a.ldb + h)) : 0.f;
    }
#pragma unroll
    for (int i = 0; i < NC; ++i) {
      float* p = r + lane + 32 * i;
      float G = 1.f;
#pragma unroll
      for (int t = 0; t < BT; ++t) {
        G *= g[i][t];
        p[2 * t * DKP] = G * k[i][t] * rk[t];
        p[(2 * t + 1) * DKP] = G * q[i][t] * rq[t];
      }
      p[8 * DKP] = G;
      float D = 1.f;
#pragma unroll
      for (int t = BT - 1; t >= 0; --t) {
        p[(9 + t) * DKP] = D * k[i][t] * rk[t];
        D *= g[i][t];
      }
    }
    float* rv = r + NVEC * DKP + NSCAL;
    for (int c = lane; c < DVP; c += 32) {
      float v[BT] = {0.f, 0.f, 0.f, 0.f};
      if (c < DV) conv_block<T, KC>(x + v0 + c, a.ld, hist + v0 + c, C, w_s + 2 * DK + c, W, taps, b, v);
#pragma unroll
      for (int t = 0; t < BT; ++t) rv[t * DVP + c] = v[t];
    }
  }
}

// grid (H * column tiles, sequences), 160 threads: warps 0..3 own four columns each, warp 4 copies the records.
template <typename T, int NI>
__global__ void __launch_bounds__(160) delta_scan_kernel(const ChannelDeltaArgs a, int lo, int hi, int n_blocks, const float* rec, int* status) {
  constexpr int DKP = 32 * NI;
  constexpr int HEAD = NVEC * DKP + NSCAL;               // floats of a record that every column tile reads
  constexpr int STAGE = HEAD + BT * COLS;
  extern __shared__ __align__(128) float st_s[];         // [STAGES][STAGE]
  __shared__ __align__(8) uint64_t full[STAGES], empty[STAGES];
  __shared__ int abort_s;
  volatile int* abort_flag = &abort_s;
  const int DK = a.DK, DV = a.DV, DVP = pad_dv(DV), tiles = DVP / COLS;
  const int h = blockIdx.x / tiles, tile = blockIdx.x % tiles, seq = blockIdx.y;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (threadIdx.x == 0) {
    for (int i = 0; i < STAGES; ++i) {
      mbar_init(&full[i], 1);
      mbar_init(&empty[i], 4);
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
  const long pitch = record_floats(DKP, DVP);
  const float* r0 = rec + (long(h) * n_blocks + (s0 - lo) / BT + seq) * pitch;
  if (warp == 4) {
    if (lane == 0) {
      int i = 0;
      for (; i < n_blk; ++i) {
        const int s = i % STAGES;
        if (i >= STAGES && !mbar_wait(&empty[s], ((i / STAGES) - 1) & 1, abort_flag)) {
          *abort_flag = 1;
          atomicCAS(status, 0, ST_TIMEOUT_EMPTY | SITE_DELTA_SCAN);
          break;
        }
        float* dst = st_s + s * STAGE;
        const float* src = r0 + i * pitch;
        mbar_expect_tx(&full[s], STAGE * 4);
        bulk_load(dst, src, HEAD * 4, &full[s]);
#pragma unroll
        for (int t = 0; t < BT; ++t)
          bulk_load(dst + HEAD + t * COLS, src + HEAD + t * DVP + tile * COLS, COLS * 4, &full[s]);
      }
      // copies in flight land before the CTA ends: the consumers wait for every one, unless they gave up
      if (*abort_flag) {
        volatile int no = 0;
        for (int j = max(0, i - STAGES); j < i; ++j) mbar_wait(&full[j % STAGES], (j / STAGES) & 1, &no, 1000000ull);
      }
    }
    return;
  }
  const int r = lane & 7, ct = warp * 4 + (lane >> 3), col = tile * COLS + ct;
  const bool ok = col < DV;
  float* sp = a.state + ((long(slot) * a.H + h) * DV + (ok ? col : 0)) * DK;
  uint64_t S[2 * NI];
  load_state<NI>(sp, r, DK, ok, S);
  T* out = static_cast<T*>(a.out) + long(h) * DV + col;
  for (int i = 0; i < n_blk; ++i) {
    const int s = i % STAGES;
    if (!__all_sync(0xffffffffu, mbar_wait(&full[s], (i / STAGES) & 1, abort_flag))) {
      *abort_flag = 1;
      if (lane == 0) atomicCAS(status, 0, ST_TIMEOUT_FULL | SITE_DELTA_SCAN);
      break;
    }
    const float* v = st_s + s * STAGE;
    // value index: 0..3 = d_1 .. d_4, 4..7 = e_1 .. e_4
    uint64_t acc[8];
#pragma unroll
    for (int x = 0; x < 8; ++x) acc[x] = 0ull;
#pragma unroll
    for (int n = 0; n < NI; ++n) {
#pragma unroll
      for (int x = 0; x < 8; ++x) {
        uint64_t p, q;
        ld4(v + ((x & 3) * 2 + (x >> 2)) * DKP + 32 * n + 4 * r, p, q);
        acc[x] = fma2(S[2 * n], p, acc[x]);
        acc[x] = fma2(S[2 * n + 1], q, acc[x]);
      }
    }
    float f[8];
#pragma unroll
    for (int x = 0; x < 8; ++x) {
      float p, q;
      u2(acc[x], p, q);
      f[x] = p + q;
    }
#pragma unroll
    for (int o = 4; o > 0; o >>= 1) {                    // lane r of the column gets value r
      const bool up = r & o;
#pragma unroll
      for (int x = 0; x < o; ++x) {
        const float send = up ? f[x] : f[x + o], keep = up ? f[x + o] : f[x];
        f[x] = keep + __shfl_xor_sync(0xffffffffu, send, o);
      }
    }
    const float* sc = v + NVEC * DKP;
    const float4 be = *reinterpret_cast<const float4*>(sc);
    const float4 c0 = *reinterpret_cast<const float4*>(sc + 4), c1 = *reinterpret_cast<const float4*>(sc + 8);
    const float4 m0 = *reinterpret_cast<const float4*>(sc + 12), m1 = *reinterpret_cast<const float4*>(sc + 16);
    const int base = lane & 24;
    const float* vv = v + HEAD + ct;
    // c 12 13 14 23 | 24 34, m 11 12 | 13 14 22 23 | 24 33 34 44
    const float u1 = be.x * (vv[0] - __shfl_sync(0xffffffffu, f[0], base));
    const float u2_ = be.y * (vv[COLS] - __shfl_sync(0xffffffffu, f[0], base + 1) - c0.x * u1);
    const float u3 = be.z * (vv[2 * COLS] - __shfl_sync(0xffffffffu, f[0], base + 2) - c0.y * u1 - c0.w * u2_);
    const float u4 = be.w * (vv[3 * COLS] - __shfl_sync(0xffffffffu, f[0], base + 3) - c0.z * u1 - c1.x * u2_ - c1.y * u3);
    const uint64_t U1 = p2(u1, u1), U2 = p2(u2_, u2_), U3 = p2(u3, u3), U4 = p2(u4, u4);
#pragma unroll
    for (int n = 0; n < NI; ++n) {
      const float* w = v + 8 * DKP + 32 * n + 4 * r;
      uint64_t p, q;
      ld4(w, p, q);
      S[2 * n] = mul2(S[2 * n], p);
      S[2 * n + 1] = mul2(S[2 * n + 1], q);
      ld4(w + DKP, p, q);
      S[2 * n] = fma2(p, U1, S[2 * n]);
      S[2 * n + 1] = fma2(q, U1, S[2 * n + 1]);
      ld4(w + 2 * DKP, p, q);
      S[2 * n] = fma2(p, U2, S[2 * n]);
      S[2 * n + 1] = fma2(q, U2, S[2 * n + 1]);
      ld4(w + 3 * DKP, p, q);
      S[2 * n] = fma2(p, U3, S[2 * n]);
      S[2 * n + 1] = fma2(q, U3, S[2 * n + 1]);
      ld4(w + 4 * DKP, p, q);
      S[2 * n] = fma2(p, U4, S[2 * n]);
      S[2 * n + 1] = fma2(q, U4, S[2 * n + 1]);
    }
    // lane 4 + j holds e_{j+1}: o = e + sum over i <= j of m_ij u_i
    const int j = r & 3;
    float o = f[0];
    o = fmaf(j == 0 ? c1.z : j == 1 ? c1.w : j == 2 ? m0.x : m0.y, u1, o);
    if (j >= 1) o = fmaf(j == 1 ? m0.z : j == 2 ? m0.w : m1.x, u2_, o);
    if (j >= 2) o = fmaf(j == 2 ? m1.y : m1.z, u3, o);
    if (j >= 3) o = fmaf(m1.w, u4, o);
    __syncwarp();
    if (lane == 0) mbar_arrive(&empty[s]);
    const int t = s0 + i * BT + j;
    if (r >= 4 && ok && t < s1) st_f(out + long(t) * a.ldo, o);
  }
  if (a.write_state && ok && !*abort_flag) store_state<NI>(sp, r, DK, S);
}

// New convolution history of the sequences that end inside the slice (their rows are all there; the old history has been
// read by the kernels in front).
template <typename T>
__global__ void __launch_bounds__(128) delta_history_kernel(const ChannelDeltaArgs a) {
  griddep_wait();
  griddep_launch();
  const int C = 2 * a.G * a.DK + a.H * a.DV, c = blockIdx.x * 128 + threadIdx.x, seq = blockIdx.y, K1 = a.KC - 1;
  if (c >= C) return;
  const int t0 = a.cu[seq], t1 = a.cu[seq + 1];
  if (t1 <= t0 || a.slots[seq] < 0) return;
  float* st = a.conv_state + long(a.slots[seq]) * C * K1 + c;
  const T* x = static_cast<const T*>(a.qkv) + c;
  for (int j = 0; j < K1; ++j) {           // position j takes what was behind it: never read after written
    const int s = t1 - K1 + j;
    st[long(j) * C] = s >= t0 ? ld_f(x + long(s) * a.ld) : st[long(K1 + (s - t0)) * C];
  }
}

// ---------------------------------------------------------------------------------------------------------------
// Decode: one CTA per (head, sequence), one token per sequence. q / k channels may serve several heads: the last of them to have read the
// old history (an arrival counter per sequence and key head) replaces it.
// ---------------------------------------------------------------------------------------------------------------
constexpr int DEC_IT = 4;                // column groups of a warp whose loads are in flight together

template <typename T, int NI, int KC>
__global__ void __launch_bounds__(256) delta_decode_kernel(const ChannelDeltaArgs a, const T* gate, long ldg, const float* norm_w,
                                                           float eps, unsigned int* ctr) {
  constexpr int DKP = 32 * NI, K1C = KC > 0 ? KC - 1 : 0;
  extern __shared__ float sm[];          // g k | g q | g | k [DKP each] | v [DV] | o [DV]
  __shared__ float red[3][8];
  __shared__ int s_last;
  const int DK = a.DK, DV = a.DV, H = a.H, G = a.G, hpg = H / G;
  const int h = blockIdx.x, n = blockIdx.y, hk = h / hpg;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, r = lane & 7, tid = threadIdx.x;
  const int slot = a.slots[n];
  float* gk = sm, *gq = sm + DKP, *gs = sm + 2 * DKP, *ks = sm + 3 * DKP, *vs = sm + 4 * DKP, *os = vs + DV;
  float* state = a.state + (long(slot < 0 ? 0 : slot) * H + h) * DV * DK;
  const int n_it = (DV + 31) / 32;       // groups of 32 columns
  const int K1 = a.KC - 1, C = 2 * G * DK + H * DV, W = 2 * DK + DV;
  float* hist = a.conv_state + long(slot < 0 ? 0 : slot) * C * K1;
  auto channel = [&](int i) { return i < DK ? hk * DK + i : i < 2 * DK ? G * DK + hk * DK + i - DK : 2 * G * DK + h * DV + i - 2 * DK; };
  // Nothing of this step writes weights, state or history in front of this launch: their loads go out before the wait for
  // the projections (the first two turns of the convolution's loop, all of the decay's and the norm's for usual sizes).
  uint64_t S[DEC_IT][2 * NI];
  auto column = [&](int it) { return it * 32 + warp * 4 + (lane >> 3); };
  float tw[2][K1C + 1], th[2][K1C > 0 ? K1C : 1];
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    const int i = tid + 256 * e;
    if (KC > 0 && i < W) {
      const int c = channel(i);
#pragma unroll
      for (int j = 0; j <= K1C; ++j) tw[e][j] = a.conv_w[long(j) * C + c];
#pragma unroll
      for (int j = 0; j < K1C; ++j) th[e][j] = hist[long(j) * C + c];
    }
  }
  const float db = tid < DK ? a.dt_bias[long(h) * DK + tid] : 0.f, Ah = a.A[h], nw = tid < DV ? norm_w[tid] : 0.f;
  if (slot >= 0) {
#pragma unroll
    for (int it = 0; it < DEC_IT; ++it)
      if (it < n_it) load_state<NI>(state + long(min(column(it), DV - 1)) * DK, r, DK, column(it) < DV, S[it]);
  }
  griddep_wait();
  griddep_launch();
  if (slot < 0) return;
  const T* x = static_cast<const T*>(a.qkv) + long(n) * a.ld;
  const T* ap = static_cast<const T*>(a.a) + long(n) * a.lda + long(h) * DK;
  const T* gr = gate + long(n) * ldg + long(h) * DV;
  float tx[2];
#pragma unroll
  for (int e = 0; e < 2; ++e) tx[e] = tid + 256 * e < W ? ld_f(x + channel(tid + 256 * e)) : 0.f;
  const float ta = tid < DK ? ld_f(ap + tid) : 0.f, tg = tid < DV ? ld_f(gr + tid) : 0.f;
  const float beta = sigmoid_t<T>(ld_f(static_cast<const T*>(a.b) + long(n) * a.ldb + h));
  float qq = 0.f, kk = 0.f;
  auto one = [&](int i, float xv, const float* w, const float* hv) {       // a channel: convolution, silu, history
    const int c = channel(i);
    const bool own = hpg == 1 || i >= 2 * DK;
    float* hc = hist + c;
    float acc;
    if constexpr (KC > 0) {
      acc = w[K1C] * xv;
#pragma unroll
      for (int j = 0; j < K1C; ++j) acc = fmaf(w[j], hv[j], acc);
      if (own) {
#pragma unroll
        for (int j = 1; j < K1C; ++j) hc[long(j - 1) * C] = hv[j];
        if (K1C > 0) hc[long(K1C - 1) * C] = xv;
      }
    } else {
      const float* wc = a.conv_w + c;
      acc = wc[long(K1) * C] * xv;
      for (int j = 0; j < K1; ++j) {
        const float v = hc[long(j) * C];
        acc = fmaf(wc[long(j) * C], v, acc);
        if (own && j > 0) hc[long(j - 1) * C] = v;
      }
      if (own && K1 > 0) hc[long(K1 - 1) * C] = xv;
    }
    const float y = silu_t<T>(acc);
    if (i < DK) { gq[i] = y; qq = fmaf(y, y, qq); }
    else if (i < 2 * DK) { ks[i - DK] = y; kk = fmaf(y, y, kk); }
    else vs[i - 2 * DK] = y;
  };
#pragma unroll
  for (int e = 0; e < 2; ++e)
    if (tid + 256 * e < W) one(tid + 256 * e, tx[e], tw[e], th[e]);
  for (int i = tid + 512; i < W; i += 256) {
    float w[K1C + 1], hv[K1C > 0 ? K1C : 1];
    if constexpr (KC > 0) {
      const int c = channel(i);
#pragma unroll
      for (int j = 0; j <= K1C; ++j) w[j] = a.conv_w[long(j) * C + c];
#pragma unroll
      for (int j = 0; j < K1C; ++j) hv[j] = hist[long(j) * C + c];
    }
    one(i, ld_f(x + channel(i)), w, hv);
  }
  qq = warp_sum_f(qq);
  kk = warp_sum_f(kk);
  if (lane == 0) { red[0][warp] = qq; red[1][warp] = kk; }
  if (hpg > 1) __threadfence();
  __syncthreads();
  if (hpg > 1 && K1 > 0) {
    if (threadIdx.x == 0) {
      const unsigned int old = atomicAdd(&ctr[long(n) * G + hk], 1u);
      s_last = old == unsigned(hpg) - 1u;
      if (s_last) ctr[long(n) * G + hk] = 0u;
    }
    __syncthreads();
    if (s_last) {
      __threadfence();
      for (int i = threadIdx.x; i < 2 * DK; i += 256) {
        const int c = channel(i);
        float* hc = hist + c;
        for (int j = 0; j + 1 < K1; ++j) hc[long(j) * C] = __ldcg(&hc[long(j + 1) * C]);
        hc[long(K1 - 1) * C] = ld_f(x + c);
      }
    }
  }
  qq = kk = 0.f;
#pragma unroll
  for (int w = 0; w < 8; ++w) { qq += red[0][w]; kk += red[1][w]; }
  const float rq = a.scale / sqrtf(qq + a.l2_eps), rk = 1.f / sqrtf(kk + a.l2_eps);
  float kq = 0.f;
  for (int c = threadIdx.x; c < DKP; c += 256) {
    float g = 1.f, kv = 0.f, qv = 0.f;
    if (c < DK) {
      g = decay_t<T>(ta + db, Ah);        // (256 channels at most: one turn)
      kv = ks[c] * rk;
      qv = gq[c] * rq;
    }
    kq = fmaf(kv, qv, kq);
    gk[c] = g * kv;
    gq[c] = g * qv;
    gs[c] = g;
    ks[c] = kv;
  }
  kq = warp_sum_f(kq);
  if (lane == 0) red[2][warp] = kq;
  __syncthreads();
  kq = 0.f;
#pragma unroll
  for (int w = 0; w < 8; ++w) kq += red[2][w];
  float oo = 0.f;
  for (int it0 = 0; it0 < n_it; it0 += DEC_IT) {
    if (it0 > 0) {
#pragma unroll
      for (int it = 0; it < DEC_IT; ++it)
        if (it0 + it < n_it)
          load_state<NI>(state + long(min(column(it0 + it), DV - 1)) * DK, r, DK, column(it0 + it) < DV, S[it]);
    }
#pragma unroll
    for (int it = 0; it < DEC_IT; ++it) {
      if (it0 + it < n_it) {
        const int col = column(it0 + it);
        uint64_t d2 = 0ull, e2 = 0ull;
#pragma unroll
        for (int i = 0; i < NI; ++i) {
          uint64_t p, q;
          ld4(gk + 32 * i + 4 * r, p, q);
          d2 = fma2(S[it][2 * i], p, d2);
          d2 = fma2(S[it][2 * i + 1], q, d2);
          ld4(gq + 32 * i + 4 * r, p, q);
          e2 = fma2(S[it][2 * i], p, e2);
          e2 = fma2(S[it][2 * i + 1], q, e2);
        }
        float d, e, t;
        u2(d2, d, t);
        d += t;
        u2(e2, e, t);
        e += t;
#pragma unroll
        for (int o = 4; o > 0; o >>= 1) {
          d += __shfl_xor_sync(0xffffffffu, d, o);
          e += __shfl_xor_sync(0xffffffffu, e, o);
        }
        const float u = col < DV ? beta * (vs[col] - d) : 0.f;
        const float o = fmaf(kq, u, e);
        const uint64_t U = p2(u, u);
#pragma unroll
        for (int i = 0; i < NI; ++i) {
          uint64_t p, q;
          ld4(gs + 32 * i + 4 * r, p, q);
          S[it][2 * i] = mul2(S[it][2 * i], p);
          S[it][2 * i + 1] = mul2(S[it][2 * i + 1], q);
          ld4(ks + 32 * i + 4 * r, p, q);
          S[it][2 * i] = fma2(p, U, S[it][2 * i]);
          S[it][2 * i + 1] = fma2(q, U, S[it][2 * i + 1]);
        }
        if (col < DV) {
          store_state<NI>(state + long(col) * DK, r, DK, S[it]);
          if (r == 0) {
            os[col] = o;
            oo = fmaf(o, o, oo);
          }
        }
      }
    }
  }
  oo = warp_sum_f(oo);
  if (lane == 0) red[0][warp] = oo;
  __syncthreads();
  oo = 0.f;
#pragma unroll
  for (int w = 0; w < 8; ++w) oo += red[0][w];
  const float inv = 1.f / sqrtf(oo / float(DV) + eps);
  T* out = static_cast<T*>(a.out) + long(n) * a.ldo + long(h) * DV;
  if (tid < DV) st_f(out + tid, os[tid] * inv * nw * sigmoid_t<T>(tg));
  for (int c = tid + 256; c < DV; c += 256) st_f(out + c, os[c] * inv * norm_w[c] * sigmoid_t<T>(ld_f(gr + c)));
}

// RMS norm of each head, times w, times sigmoid(gate): one warp per (row, head)
template <typename T, int VEC>
__global__ void __launch_bounds__(256) head_norm_gate_kernel(const T* __restrict__ o, long ldo, const T* __restrict__ gate, long ldg,
                                                             const float* __restrict__ w, float eps, int H, int D, long n,
                                                             T* __restrict__ out, long ldout) {
  griddep_wait();
  griddep_launch();
  const long i = long(blockIdx.x) * 8 + (threadIdx.x >> 5);
  if (i >= n) return;
  const int lane = threadIdx.x & 31, h = int(i % H);
  const long t = i / H;
  const T* x = o + t * ldo + long(h) * D;
  const T* g = gate + t * ldg + long(h) * D;
  float ss = 0.f;
  for (int c = lane * VEC; c < D; c += 32 * VEC) {
    float v[VEC];
    ld_vec<VEC>(x + c, v);
#pragma unroll
    for (int j = 0; j < VEC; ++j) ss = fmaf(v[j], v[j], ss);
  }
  const float inv = 1.f / sqrtf(warp_sum_f(ss) / float(D) + eps);
  for (int c = lane * VEC; c < D; c += 32 * VEC) {
    float v[VEC], z[VEC];
    ld_vec<VEC>(x + c, v);
    ld_vec<VEC>(g + c, z);
#pragma unroll
    for (int j = 0; j < VEC; ++j) v[j] = v[j] * inv * w[c + j] * sigmoid_t<T>(z[j]);
    st_vec<VEC>(out + t * ldout + long(h) * D + c, v);
  }
}

template <typename T, int NC>
int prep_t(const ChannelDeltaArgs& a, int lo, int hi, int n_blocks, float* rec, cudaStream_t s) {
  const dim3 grid((n_blocks + 4 * PREP_BLOCKS - 1) / (4 * PREP_BLOCKS), a.H);
  const size_t smem = size_t(2 * a.DK + a.DV) * a.KC * 4;
  if (smem > 48 * 1024) return 1;
#define LB_KC(K_) \
  if (a.KC == K_) return launch_pdl(delta_prep_kernel<T, NC, K_>, grid, dim3(128), smem, s, a, lo, hi, n_blocks, rec) != cudaSuccess;
  LB_KC(1) LB_KC(2) LB_KC(3) LB_KC(4)
#undef LB_KC
  return launch_pdl(delta_prep_kernel<T, NC, 0>, grid, dim3(128), smem, s, a, lo, hi, n_blocks, rec) != cudaSuccess;
}

template <typename T, int NI>
int scan_t(const ChannelDeltaArgs& a, int lo, int hi, int n_blocks, const float* rec, int* status, cudaStream_t s) {
  const int smem = STAGES * (NVEC * 32 * NI + NSCAL + BT * COLS) * 4;
  auto kfn = delta_scan_kernel<T, NI>;
  static bool attr = false;
  if (!attr) {
    if (cudaFuncSetAttribute(kfn, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess) return 1;
    attr = true;
  }
  return launch_pdl(kfn, dim3(a.H * (pad_dv(a.DV) / COLS), a.n_seqs), dim3(160), smem, s, a, lo, hi, n_blocks, rec, status) != cudaSuccess;
}

template <typename T>
int scan_all(const ChannelDeltaArgs& a, float* rec, long rec_floats, int* status, cudaStream_t s) {
  const int DKP = pad_dk(a.DK);
  const long per = record_floats(DKP, pad_dv(a.DV)) * a.H;
  const long blocks = rec_floats / per;                  // records the scratch holds, per head
  const long tokens = (blocks - a.n_seqs) * BT;
  if (tokens < BT || (tokens < a.T && !a.write_state)) return 1;      // slices hand the state on through the pool
  for (int lo = 0; lo < a.T;) {
    const int hi = int(long(a.T) - lo <= tokens ? a.T : lo + tokens);
    const int nb = (hi - lo) / BT + a.n_seqs;
    int rc = 1;
#define LB_NI(N_) \
  if (DKP == 32 * N_) rc = prep_t<T, N_>(a, lo, hi, nb, rec, s) || scan_t<T, N_>(a, lo, hi, nb, rec, status, s);
    LB_NI(1) LB_NI(2) LB_NI(4) LB_NI(8)
#undef LB_NI
    if (rc) return 1;
    lo = hi;
  }
  return 0;
}

template <typename T>
int history_t(const ChannelDeltaArgs& a, cudaStream_t s) {
  if (a.write_state && a.KC > 1)
    return launch_pdl(delta_history_kernel<T>, dim3((2 * a.G * a.DK + a.H * a.DV + 127) / 128, a.n_seqs), dim3(128), 0, s, a) !=
           cudaSuccess;
  return 0;
}

template <typename T>
int decode_t(const ChannelDeltaArgs& a, const void* gate, long ldg, const float* norm_w, float eps, unsigned int* ctr,
             cudaStream_t s) {
  const int DKP = pad_dk(a.DK);
  const size_t smem = size_t(4 * DKP + 2 * a.DV) * 4;
  if (smem > 48 * 1024) return 1;
#define LB_K(N_, K_)                                                                                                          \
  return launch_pdl(delta_decode_kernel<T, N_, K_>, dim3(a.H, a.n_seqs), dim3(256), smem, s, a, static_cast<const T*>(gate), ldg, \
                    norm_w, eps, ctr) != cudaSuccess;
#define LB_NI(N_)               \
  if (DKP == 32 * N_) {         \
    if (a.KC == 4) { LB_K(N_, 4) } \
    if (a.KC == 3) { LB_K(N_, 3) } \
    LB_K(N_, 0)                 \
  }
  LB_NI(1) LB_NI(2) LB_NI(4) LB_NI(8)
#undef LB_NI
#undef LB_K
  return 1;
}

template <typename T>
int norm_gate_t(const void* o, long ldo, const void* gate, long ldg, const float* w, float eps, int H, int D, int rows, void* out,
                long ldout, cudaStream_t s) {
  const long n = long(rows) * H;
  const bool v4 = D % 4 == 0 && ldo % 4 == 0 && ldg % 4 == 0 && ldout % 4 == 0 &&
                  ((reinterpret_cast<uintptr_t>(o) | reinterpret_cast<uintptr_t>(gate) | reinterpret_cast<uintptr_t>(out)) %
                   (4 * sizeof(T))) == 0;
  return launch_pdl(v4 ? head_norm_gate_kernel<T, 4> : head_norm_gate_kernel<T, 1>, dim3(unsigned((n + 7) / 8)), dim3(256), 0, s,
                    static_cast<const T*>(o), ldo, static_cast<const T*>(gate), ldg, w, eps, H, D, n, static_cast<T*>(out),
                    ldout) != cudaSuccess;
}

bool shape_ok(const ChannelDeltaArgs& a) {
  return a.G > 0 && a.H % a.G == 0 && a.DK >= 1 && a.DK <= 256 && a.DV >= 1 && a.KC >= 1 && a.n_seqs <= 65535;
}

}  // namespace

long channel_delta_record_floats(int H, int DK, int DV, bool f32) {
  // per four tokens; records of eight tokens count half
  const long four = record_floats(pad_dk(DK), pad_dv(DV)) * H;
  return f32 || DK > 128 ? four : max(four, (channel_delta_mma_floats(H, DK, DV) + 1) / 2);
}

int channel_delta_launch(const ChannelDeltaArgs& a, float* rec, long rec_floats, int* status, bool f32, cudaStream_t s) {
  if (a.n_seqs <= 0 || a.T <= 0) return 0;
  if (!shape_ok(a) || (reinterpret_cast<uintptr_t>(rec) & 127) || (reinterpret_cast<uintptr_t>(a.state) & 15)) return 1;
  if (f32) return scan_all<float>(a, rec, rec_floats, status, s) || history_t<float>(a, s);
  const int rc = channel_delta_mma_ok(a) ? channel_delta_mma_launch(a, rec, rec_floats, status, s)
                                         : scan_all<__nv_bfloat16>(a, rec, rec_floats, status, s);
  return rc || history_t<__nv_bfloat16>(a, s);
}

int channel_delta_decode_launch(const ChannelDeltaArgs& a, const void* gate, long ldg, const float* norm_w, float eps,
                                unsigned int* ctr, bool f32, cudaStream_t s) {
  if (a.n_seqs <= 0) return 0;
  if (!shape_ok(a) || (reinterpret_cast<uintptr_t>(a.state) & 15)) return 1;
  return f32 ? decode_t<float>(a, gate, ldg, norm_w, eps, ctr, s) : decode_t<__nv_bfloat16>(a, gate, ldg, norm_w, eps, ctr, s);
}

int head_norm_gate_launch(const void* o, long ldo, const void* gate, long ldg, const float* w, float eps, int H, int D, int rows,
                          void* out, long ldout, bool f32, cudaStream_t s) {
  if (rows <= 0) return 0;
  return f32 ? norm_gate_t<float>(o, ldo, gate, ldg, w, eps, H, D, rows, out, ldout, s)
             : norm_gate_t<__nv_bfloat16>(o, ldo, gate, ldg, w, eps, H, D, rows, out, ldout, s);
}

}  // namespace lb
