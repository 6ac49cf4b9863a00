// One fp32 residual whose sublayers run between two RMS norms, with a short causal convolution in front of each:
//   x' = x + norm(y) * post_w            (y: the sublayer's output; the first launch of a step starts from the embedding)
//   n  = norm(x') * norm_w               (the next sublayer's norm; both norms work in `groups` equal parts of the row)
//   h_t = n_t + sum_j taps[j] n_(t - K + 1 + j)                     (per channel; n before the sequence's start is zero)
// in one launch per sublayer, so that the residual and the sublayer output are read once. The last K - 1 rows of n are a
// sequence's history; the launch reads and replaces it.
//
// A norm never leaves its group, so a CTA takes one group of columns and walks up to `tok` consecutive tokens of one
// sequence with the previous rows of n in registers: one warp for groups of up to 512 columns (no barrier at all), several
// for wider ones. A tile in the middle of a sequence recomputes n of the K - 1 tokens in front of it from x and y (the new
// residual goes to a second buffer, so these are still there). Only the first tile of a sequence touches the history: it
// reads it, and replaces it with the rows of the sequence's last tokens, recomputed when they lie in another tile. So no
// launch waits and no two CTAs meet in the state.
#include <algorithm>

#include "act_type.cuh"
#include "common.cuh"
#include "layers.h"

namespace lb {
namespace {

struct Tile { int seq, t0, t1, ta; };

constexpr int RING = 4;          // tokens whose rows are on the way to shared memory

template <int BYTES>
__device__ __forceinline__ void copy_async(void* smem, const void* src) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], %2;" ::"r"(smem_u32(smem)), "l"(src), "n"(BYTES) : "memory");
}

// The sequence and first token of tile `idx` when every sequence is cut into tiles of `tok` tokens (warp-wide; seq < 0:
// no such tile).
__device__ __forceinline__ Tile find_tile(const int* __restrict__ cu, int n_seqs, int tok, int idx) {
  const int lane = threadIdx.x & 31;
  int before = 0;
  for (int b = 0; b < n_seqs; b += 32) {
    const int s = b + lane;
    const int c0 = s < n_seqs ? cu[s] : 0, c1 = s < n_seqs ? cu[s + 1] : 0;
    const int n = (c1 - c0 + tok - 1) / tok;
    int inc = n;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const int v = __shfl_up_sync(0xffffffffu, inc, o);
      if (lane >= o) inc += v;
    }
    const unsigned hit = __ballot_sync(0xffffffffu, before + inc > idx);
    if (hit) {
      const int l = __ffs(hit) - 1;
      const int first = before + __shfl_sync(0xffffffffu, inc - n, l);
      Tile t;
      t.seq = b + l;
      t.t0 = __shfl_sync(0xffffffffu, c0, l);
      t.t1 = __shfl_sync(0xffffffffu, c1, l);
      t.ta = t.t0 + (idx - first) * tok;
      return t;
    }
    before += __shfl_sync(0xffffffffu, inc, 31);
  }
  return Tile{-1, 0, 0, 0};
}

// K: taps; 0: any number up to 16 (a.taps_n). FULL: the group is exactly VEC * NC columns per thread.
template <typename T, int VEC, int NC, int K, bool ONE_WARP, bool FULL>
__global__ void __launch_bounds__(ONE_WARP ? 32 : 512, ONE_WARP && NC * VEC <= 16 && K > 0 ? 12 : 1)
    resid_step_kernel(const ResidStepArgs a) {
  __shared__ float part_s[2][16];
  const int tid = threadIdx.x, nt = ONE_WARP ? 32 : blockDim.x, H = a.H, gs = FULL ? nt * NC * VEC : H / a.groups;
  const int tile = blockIdx.x / a.groups, col0 = (blockIdx.x % a.groups) * gs + tid * VEC;
  constexpr int R = K > 0 ? (K > 1 ? K - 1 : 1) : 15;     // rows of history in registers
  const int K1 = K > 0 ? K - 1 : a.taps_n - 1;
  const bool start = a.x_in == nullptr;
  auto on = [&](int c) { return FULL || (c * nt + tid) * VEC < gs; };
  griddep_wait();
  griddep_launch();
  Tile tl;
  if (a.tok >= a.max_len) {
    tl.seq = tile;
    tl.t0 = tl.ta = a.cu ? a.cu[tl.seq] : tile;
    tl.t1 = a.cu ? a.cu[tl.seq + 1] : tl.t0 + 1;
  } else {
    tl = find_tile(a.cu, a.n_seqs, a.tok, tile);
  }
  if (tl.seq < 0 || tl.ta >= tl.t1) return;
  const int tb = min(tl.t1, tl.ta + a.tok);
  const float gs_inv = 1.f / float(gs);
  const int step = nt * VEC;                              // columns between a thread's vectors

  // Four columns at a time: a token's rows come through a ring in shared memory, every thread copying what it reads itself
  extern __shared__ __align__(16) uint8_t ring_s[];
  constexpr bool ASYNC = VEC == 4;
  constexpr int YB = 4 * int(sizeof(T));
  uint8_t* ring_x = ring_s + tid * 16;
  uint8_t* ring_y = ring_s + size_t(RING * NC * nt) * 16 + tid * YB;
  auto emb_row = [&](int t) {
    long row = t;
    if (a.ids) {
      const int id = a.ids[t];
      row = (id < 0 || id >= a.vocab) ? 0 : id;
    }
    return static_cast<const T*>(a.emb) + row * a.ld_emb + col0;
  };
  auto issue = [&](int t, bool real, int stage) {
    if constexpr (ASYNC) {
      if (real && !a.direct) {
        const T* yp = start ? emb_row(t) : static_cast<const T*>(a.y) + long(t) * a.ldy + col0;
        uint8_t* sy = ring_y + stage * (NC * nt * YB);
#pragma unroll
        for (int c = 0; c < NC; ++c)
          if (on(c)) copy_async<YB>(sy + c * (nt * YB), yp + c * step);
        if (!start) {
          const float* xp = a.x_in + long(t) * H + col0;
          uint8_t* sx = ring_x + stage * (NC * nt * 16);
#pragma unroll
          for (int c = 0; c < NC; ++c)
            if (on(c)) copy_async<16>(sx + c * (nt * 16), xp + c * step);
        }
      }
      asm volatile("cp.async.commit_group;" ::: "memory");
    }
  };
  // the token's rows: embedding in x, or residual in x and sublayer output in y
  float x[NC][VEC], y[NC][VEC];
  auto take = [&](int t, int stage) {
    const bool ring = ASYNC && !a.direct;
    if constexpr (ASYNC) asm volatile("cp.async.wait_group %0;" ::"n"(RING - 1) : "memory");
    const T* yp = ring ? reinterpret_cast<const T*>(ring_y + stage * (NC * nt * YB))
                       : (start ? emb_row(t) : static_cast<const T*>(a.y) + long(t) * a.ldy + col0);
    const int ys = ring ? nt * 4 : step;
    if (start) {
#pragma unroll
      for (int c = 0; c < NC; ++c)
        if (on(c)) ld_vec<VEC>(yp + c * ys, x[c]);
      return;
    }
    const float* xp = ring ? reinterpret_cast<const float*>(ring_x + stage * (NC * nt * 16)) : a.x_in + long(t) * H + col0;
#pragma unroll
    for (int c = 0; c < NC; ++c)
      if (on(c)) {
        ld_vec<VEC>(yp + c * ys, y[c]);
        ld_vec<VEC>(xp + c * ys, x[c]);
      }
  };
  auto inv_rms = [&](const float (&v)[NC][VEC], int buf) {
    float ss = 0.f;
#pragma unroll
    for (int c = 0; c < NC; ++c)
      if (on(c)) {
#pragma unroll
        for (int j = 0; j < VEC; ++j) ss = fmaf(v[c][j], v[c][j], ss);
      }
    ss = warp_sum_f(ss);
    if constexpr (!ONE_WARP) {
      if ((tid & 31) == 0) part_s[buf][tid >> 5] = ss;
      __syncthreads();
      ss = 0.f;
      for (int i = 0; i < nt / 32; ++i) ss += part_s[buf][i];
    }
    return rsqrtf(fmaf(ss, gs_inv, a.eps));
  };
  // x becomes n; the new residual is written when the token is this tile's own
  const float* post_w = a.post_w + col0;
  const float* norm_w = a.norm_w + col0;
  auto advance = [&](int t, bool own) {
    if (start) {
      if constexpr (!ONE_WARP) __syncthreads();            // with one norm per token its buffer is written every time
#pragma unroll
      for (int c = 0; c < NC; ++c)
#pragma unroll
        for (int j = 0; j < VEC; ++j) x[c][j] *= a.emb_scale;
    } else {
      const float inv = inv_rms(y, 0);
#pragma unroll
      for (int c = 0; c < NC; ++c) {
        float w[VEC];
        if (on(c)) ld_vec<VEC>(post_w + c * step, w);
#pragma unroll
        for (int j = 0; j < VEC; ++j) x[c][j] = fmaf(y[c][j] * inv, w[j], x[c][j]);
      }
    }
    if (own) {
      float* xo = a.x_out + long(t) * H + col0;
#pragma unroll
      for (int c = 0; c < NC; ++c)
        if (on(c)) st_vec<VEC>(xo + c * step, x[c]);
    }
    const float inv = inv_rms(x, 1);
#pragma unroll
    for (int c = 0; c < NC; ++c) {
      float w[VEC];
      if (on(c)) ld_vec<VEC>(norm_w + c * step, w);
#pragma unroll
      for (int j = 0; j < VEC; ++j) x[c][j] *= inv * w[j];
    }
  };

  // hist[R - 1] is the row before the current token; with K == 0 rows older than K1 are not used
  float hist[R][NC][VEC];
  auto used = [&](int i) { return K > 1 || (K == 0 && i >= R - K1); };
  auto push = [&]() {
    if constexpr (K != 1) {
#pragma unroll
      for (int c = 0; c < NC; ++c)
#pragma unroll
        for (int j = 0; j < VEC; ++j) {
#pragma unroll
          for (int i = 0; i + 1 < R; ++i) hist[i][c][j] = hist[i + 1][c][j];
          hist[R - 1][c][j] = x[c][j];
        }
    }
  };
  float* st = (K != 1 && a.hist) ? a.hist + long(a.slots[tl.seq]) * K1 * H + col0 : nullptr;
  const bool first = tl.ta == tl.t0;
  if constexpr (K != 1) {
#pragma unroll
    for (int i = 0; i < R; ++i)
#pragma unroll
      for (int c = 0; c < NC; ++c) {
#pragma unroll
        for (int j = 0; j < VEC; ++j) hist[i][c][j] = 0.f;
        if (first && used(i) && on(c)) ld_vec<VEC>(st + long(i - (R - K1)) * H + c * step, hist[i][c]);
      }
  }
  const int tw = first ? tl.ta : tl.ta - K1;                // rows in front of the tile come first
  // rows [tw, tb), and behind them, where this tile owns the history, the sequence's last rows
  const bool tail = K != 1 && first && a.write_state && K1 > 0 && tb < tl.t1;
  const int n_rows = tb - tw, n_all = n_rows + (tail ? K1 : 0);
  auto row_at = [&](int i) { return i < n_rows ? tw + i : tl.t1 - K1 + (i - n_rows); };
#pragma unroll 1
  for (int i = 0; i < RING - 1; ++i) issue(row_at(i), i < n_all, i);
#pragma unroll 1
  for (int i = 0; i < n_all; ++i) {
    const int t = row_at(i);
    issue(row_at(i + RING - 1), i + RING - 1 < n_all, (i + RING - 1) % RING);
    take(t, i % RING);
    const bool own = i < n_rows && t >= tl.ta;
    advance(t, own);
    if (own) {
      T* hr = static_cast<T*>(a.h) + long(t) * a.ldh + col0;
#pragma unroll
      for (int c = 0; c < NC; ++c)
        if (on(c)) {
          float o[VEC];
#pragma unroll
          for (int j = 0; j < VEC; ++j) o[j] = x[c][j];
          if (a.taps) {
            const float* tp = a.taps + col0 + c * step;
            float w[VEC];
            ld_vec<VEC>(tp + long(K1) * H, w);
#pragma unroll
            for (int j = 0; j < VEC; ++j) o[j] = fmaf(w[j], x[c][j], o[j]);
            if constexpr (K != 1) {
#pragma unroll
              for (int i2 = 0; i2 < R; ++i2)
                if (used(i2)) {
                  ld_vec<VEC>(tp + long(i2 - (R - K1)) * H, w);
#pragma unroll
                  for (int j = 0; j < VEC; ++j) o[j] = fmaf(w[j], hist[i2][c][j], o[j]);
                }
            }
          }
          st_vec<VEC>(hr + c * step, o);
        }
    }
    push();
  }
  if constexpr (K != 1) {
    if (first && a.write_state && K1 > 0) {
#pragma unroll
      for (int i = 0; i < R; ++i)
        if (used(i)) {
#pragma unroll
          for (int c = 0; c < NC; ++c)
            if (on(c)) st_vec<VEC>(st + long(i - (R - K1)) * H + c * step, hist[i][c]);
        }
    }
  }
}

// Decode: one token per sequence, everything a CTA reads is asked for at once. A thread holds one vector of columns.
template <typename T, int VEC, int K>
__global__ void __launch_bounds__(1024) resid_token_kernel(const ResidStepArgs a) {
  __shared__ float part_s[2][32];
  const int tid = threadIdx.x, H = a.H, gs = H / a.groups;
  const int seq = blockIdx.x / a.groups, d = (blockIdx.x % a.groups) * gs + tid * VEC;
  const bool on = tid * VEC < gs, start = a.x_in == nullptr;
  constexpr int K1 = K - 1;
  float nw[VEC], pw[VEC], w[K][VEC];
  if (on) {                                                 // weights do not depend on the launches before
    ld_vec<VEC>(a.norm_w + d, nw);
    if (!start) ld_vec<VEC>(a.post_w + d, pw);
    if (a.taps) {
#pragma unroll
      for (int j = 0; j < K; ++j) ld_vec<VEC>(a.taps + long(j) * H + d, w[j]);
    }
  }
  griddep_wait();
  griddep_launch();
  const int t = a.cu ? a.cu[seq] : seq;
  if (a.cu && a.cu[seq + 1] <= t) return;
  float* st = a.hist ? a.hist + long(a.slots[seq]) * K1 * H + d : nullptr;
  float x[VEC], y[VEC], h[K][VEC];
  if (on) {
    if (start) {
      long row = t;
      if (a.ids) {
        const int id = a.ids[t];
        row = (id < 0 || id >= a.vocab) ? 0 : id;
      }
      ld_vec<VEC>(static_cast<const T*>(a.emb) + row * a.ld_emb + d, x);
    } else {
      ld_vec<VEC>(a.x_in + long(t) * H + d, x);
      ld_vec<VEC>(static_cast<const T*>(a.y) + long(t) * a.ldy + d, y);
    }
    if (a.taps) {
#pragma unroll
      for (int j = 0; j < K1; ++j) ld_vec<VEC>(st + long(j) * H, h[j]);
    }
  }
  auto inv_rms = [&](const float (&v)[VEC], float* part) {
    float ss = 0.f;
    if (on) {
#pragma unroll
      for (int j = 0; j < VEC; ++j) ss = fmaf(v[j], v[j], ss);
    }
    ss = warp_sum_f(ss);
    if (blockDim.x > 32) {
      if ((tid & 31) == 0) part[tid >> 5] = ss;
      __syncthreads();
      ss = 0.f;
      for (int i = 0; i < int(blockDim.x) / 32; ++i) ss += part[i];
    }
    return rsqrtf(fmaf(ss, 1.f / float(gs), a.eps));
  };
  if (start) {
#pragma unroll
    for (int j = 0; j < VEC; ++j) x[j] *= a.emb_scale;
  } else {
    const float inv = inv_rms(y, part_s[0]);
#pragma unroll
    for (int j = 0; j < VEC; ++j) x[j] += y[j] * inv * pw[j];
  }
  if (on) st_vec<VEC>(a.x_out + long(t) * H + d, x);
  const float inv = inv_rms(x, part_s[1]);
  if (!on) return;
  float o[VEC];
#pragma unroll
  for (int j = 0; j < VEC; ++j) o[j] = h[K1][j] = x[j] * inv * nw[j];
  if (a.taps) {
#pragma unroll
    for (int i = 0; i < K; ++i)
#pragma unroll
      for (int j = 0; j < VEC; ++j) o[j] = fmaf(w[i][j], h[i][j], o[j]);
    if (a.write_state) {
#pragma unroll
      for (int i = 0; i < K1; ++i) st_vec<VEC>(st + long(i) * H, h[i + 1]);
    }
  }
  st_vec<VEC>(static_cast<T*>(a.h) + long(t) * a.ldh + d, o);
}

template <typename T, int VEC>
int launch_token(const ResidStepArgs& a, int nt, dim3 grid, cudaStream_t s) {
  const int K = a.taps ? a.taps_n : 1;
#define LB_K(N)                                                                                                        \
  if (K == N) return launch_pdl(resid_token_kernel<T, VEC, N>, grid, dim3(nt), 0, s, a) != cudaSuccess;
  LB_K(1) LB_K(2) LB_K(3) LB_K(4) LB_K(5)
#undef LB_K
  return -1;
}

template <typename T, int VEC, int NC, bool ONE, bool FULL = false>
int launch_k(ResidStepArgs a, int nt, dim3 grid, cudaStream_t s) {
  const int K = a.taps ? a.taps_n : 1;
  size_t smem = VEC == 4 ? size_t(RING) * NC * nt * (16 + 4 * sizeof(T)) : 0;
  a.direct = smem > 200 * 1024;                             // groups too wide for the ring: plain loads
  if (a.direct) smem = 0;
  if (!a.taps) a.taps_n = 1;
#define LB_K(N)                                                                                                        \
  if (K == N || (N == 0 && K <= 16)) {                                                                                 \
    auto k = resid_step_kernel<T, VEC, NC, N, ONE, FULL>;                                                              \
    if (smem > 40 * 1024 &&                                                                                            \
        cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, int(smem)) != cudaSuccess)                \
      return 1;                                                                                                        \
    return launch_pdl(k, grid, dim3(nt), smem, s, a) != cudaSuccess;                                                   \
  }
  if constexpr (FULL) {
    LB_K(1) LB_K(3) LB_K(4)
    return launch_k<T, VEC, NC, ONE, false>(a, nt, grid, s);
  } else {
    LB_K(1) LB_K(4) LB_K(0)
    return 1;
  }
#undef LB_K
}

template <typename T>
int dispatch(const ResidStepArgs& a, cudaStream_t s) {
  const size_t es = sizeof(T);
  auto al = [&](const void* p, size_t n) { return p == nullptr || reinterpret_cast<uintptr_t>(p) % n == 0; };
  const int gs = a.H / a.groups;
  const bool v4 = gs % 4 == 0 && al(a.x_in, 16) && al(a.x_out, 16) && al(a.emb, 4 * es) && al(a.y, 4 * es) &&
                  al(a.h, 4 * es) && al(a.post_w, 16) && al(a.norm_w, 16) && al(a.taps, 16) && al(a.hist, 16) &&
                  a.ld_emb % 4 == 0 && a.ldy % 4 == 0 && a.ldh % 4 == 0;
  const long tiles = a.tok >= a.max_len ? (a.cu ? a.n_seqs : a.rows) : a.rows / a.tok + a.n_seqs;
  if (tiles * a.groups > 0x7fffffffL) return 1;
  const dim3 grid(static_cast<unsigned>(tiles * a.groups));
  const int need = v4 ? gs / 4 : gs;                        // threads with one vector each
  const int nt = std::min(512, (need + 127) / 128 * 32), nc = (need + nt - 1) / nt;     // up to 4 vectors per thread
  if (a.max_len <= 1 && need <= 1024) {
    const int rc = v4 ? launch_token<T, 4>(a, (need + 31) / 32 * 32, grid, s) : launch_token<T, 1>(a, (need + 31) / 32 * 32, grid, s);
    if (rc >= 0) return rc;
  }
  if (v4) {
    if (need <= 32) return launch_k<T, 4, 1, true>(a, 32, grid, s);
    if (gs == 256) return launch_k<T, 4, 2, true, true>(a, 32, grid, s);
    if (gs == 512) return launch_k<T, 4, 4, true, true>(a, 32, grid, s);
    if (nt == 32) return launch_k<T, 4, 4, true>(a, 32, grid, s);
    if (gs % 256 == 0 && gs <= 4096) return launch_k<T, 4, 2, false, true>(a, gs / 8, grid, s);
    if (nt * 16 == gs) return launch_k<T, 4, 4, false, true>(a, nt, grid, s);
    if (nc <= 4) return launch_k<T, 4, 4, false>(a, nt, grid, s);
    if (nc <= 8) return launch_k<T, 4, 8, false>(a, nt, grid, s);
  } else {
    if (nt == 32) return launch_k<T, 1, 4, true>(a, 32, grid, s);
    if (nc <= 4) return launch_k<T, 1, 4, false>(a, nt, grid, s);
    if (nc <= 8) return launch_k<T, 1, 8, false>(a, nt, grid, s);
  }
  return 1;
}

}  // namespace

int resid_step_launch(const ResidStepArgs& a, bool f32, cudaStream_t s) {
  if (a.rows <= 0) return 0;
  if (a.groups < 1 || a.H < 1 || a.H % a.groups || a.tok < 1) return 1;
  if (a.taps && (a.taps_n < 1 || a.tok < (a.tok >= a.max_len ? 1 : a.taps_n - 1))) return 1;
  return f32 ? dispatch<float>(a, s) : dispatch<__nv_bfloat16>(a, s);
}

}  // namespace lb
