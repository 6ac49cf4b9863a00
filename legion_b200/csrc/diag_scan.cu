// Diagonal gated linear recurrence (RG-LRU): per channel
//   r = sigmoid(gate_r + bias), i = sigmoid(gate_i + bias), log a = r * log_decay,
//   S_t = a S_(t-1) + sqrt(1 - a^2) i u,   out = S gelu(y + y_b)
// with u from a short convolution and the gates from a block-diagonal product of u. State and everything that enters it
// besides u are fp32.
//
// Three forms:
//   decode   one launch per step: history and convolution, the block-diagonal products, recurrence and output
//   chunks   prompts: chunk summaries (product of a, state from zero) of all chunks in parallel, a carry over the chunks,
//            outputs of all chunks in parallel. The first pass leaves a and the input term in the gate buffer, so the
//            transcendental functions run once.
//   tokens   short portions: one thread per channel walks its sequence
#include "act_type.cuh"
#include "common.cuh"
#include "layers.h"

namespace lb {
namespace {

// bf16 activations: hardware exponential and reciprocal (about 2^-21), far below the rounding of u
template <typename T>
__device__ __forceinline__ float gate_sigmoid(float z) {
  if constexpr (sizeof(T) == 2) return __fdividef(1.f, 1.f + __expf(-z));
  else return sigmoid_f(z);
}
// a and the input term of one token; zr, zi: gates with bias
template <typename T>
__device__ __forceinline__ float2 recur_terms(float zr, float zi, float u, float log_decay) {
  const float la = gate_sigmoid<T>(zr) * log_decay;
  const float a = sizeof(T) == 2 ? __expf(la) : expf(la);
  const float b2 = -expm1f(2.f * la);                    // 1 - a^2 without cancellation
  return make_float2(a, (sizeof(T) == 2 ? __fsqrt_rn(b2) : sqrtf(b2)) * gate_sigmoid<T>(zi) * u);
}
template <typename T>
__device__ __forceinline__ float gelu_branch(float z) {
  if constexpr (sizeof(T) == 2) {
    const float k = 1.5957691216057308f * (z + 0.044715f * z * z * z);       // z sigmoid(2 sqrt(2 / pi) (...)) = gelu_tanh(z)
    return z * gate_sigmoid<T>(k);
  } else {
    return gelu_tanh_f(z);
  }
}

struct Chan { long r, i; };      // places of a channel's two gates within a token's row of 2 W
__device__ __forceinline__ Chan gate_of(int c, int d) {
  const long r = long(c / d) * 2 * d + c % d;
  return Chan{r, r + d};
}

template <typename T>
__global__ void __launch_bounds__(128) diag_tokens_kernel(const DiagScanArgs a) {
  griddep_wait();
  griddep_launch();
  const int c = blockIdx.x * 128 + threadIdx.x, seq = blockIdx.y;
  if (c >= a.W) return;
  const int t0 = a.cu[seq], t1 = a.cu[seq + 1];
  if (t1 <= t0 || (a.max_tokens > 0 && t1 - t0 > a.max_tokens)) return;
  const Chan g = gate_of(c, a.W / a.blocks);
  const float br = a.gates_b[g.r], bi = a.gates_b[g.i], ld = a.log_decay[c], yb = a.y_b[c];
  float* st = a.state + long(a.slots[seq]) * a.W + c;
  float S = *st;
  const float* gt = a.gates + long(t0) * 2 * a.W;
  const T* u = static_cast<const T*>(a.u) + t0 * a.ldu + c;
  const T* y = static_cast<const T*>(a.y) + t0 * a.ldy + c;
  T* out = static_cast<T*>(a.out) + t0 * a.ldo + c;
  for (int t = t0; t < t1; ++t, gt += 2 * a.W, u += a.ldu, y += a.ldy, out += a.ldo) {
    const float2 ab = recur_terms<T>(gt[g.r] + br, gt[g.i] + bi, ld_f(u), ld);
    S = fmaf(ab.x, S, ab.y);
    st_f(out, S * gelu_branch<T>(ld_f(y) + yb));
  }
  if (a.write_state) *st = S;
}

constexpr int UN = 8;            // tokens whose loads are in flight together

template <typename T>
__global__ void __launch_bounds__(128) diag_chunk_terms_kernel(const DiagScanArgs a, const int* __restrict__ chunk_t0,
                                                               const int* __restrict__ chunk_n, float* __restrict__ ends) {
  griddep_wait();
  griddep_launch();
  const int c = blockIdx.x * 128 + threadIdx.x, ch = blockIdx.y;
  if (c >= a.W) return;
  const int n = chunk_n[ch];
  const long t0 = chunk_t0[ch];
  const Chan g = gate_of(c, a.W / a.blocks);
  const float br = a.gates_b[g.r], bi = a.gates_b[g.i], ld = a.log_decay[c];
  float* gt = a.gates + t0 * 2 * a.W;
  const T* u = static_cast<const T*>(a.u) + t0 * a.ldu + c;
  float A = 1.f, B = 0.f;
  for (int t = 0; t < n; t += UN) {
    float zr[UN], zi[UN], uv[UN];
#pragma unroll
    for (int k = 0; k < UN; ++k)
      if (t + k < n) {
        zr[k] = gt[long(t + k) * 2 * a.W + g.r];
        zi[k] = gt[long(t + k) * 2 * a.W + g.i];
        uv[k] = ld_f(u + (t + k) * a.ldu);
      }
#pragma unroll
    for (int k = 0; k < UN; ++k)
      if (t + k < n) {
        const float2 ab = recur_terms<T>(zr[k] + br, zi[k] + bi, uv[k], ld);
        gt[long(t + k) * 2 * a.W + g.r] = ab.x;
        gt[long(t + k) * 2 * a.W + g.i] = ab.y;
        A *= ab.x;
        B = fmaf(ab.x, B, ab.y);
      }
  }
  ends[long(ch) * 2 * a.W + c] = A;
  ends[(long(ch) * 2 + 1) * a.W + c] = B;
}

// state in front of every chunk, in place of its product of a
__global__ void __launch_bounds__(128) diag_chunk_carry_kernel(const DiagScanArgs a, const int* __restrict__ seq_chunk0,
                                                               const int* __restrict__ seq_nchunk, float* __restrict__ ends) {
  griddep_wait();
  griddep_launch();
  const int c = blockIdx.x * 128 + threadIdx.x, seq = blockIdx.y;
  if (c >= a.W) return;
  const int n = seq_nchunk[seq];
  if (n <= 0) return;
  float* st = a.state + long(a.slots[seq]) * a.W + c;
  float* e = ends + long(seq_chunk0[seq]) * 2 * a.W + c;
  float S = *st;
  for (int k0 = 0; k0 < n; k0 += UN) {
    float A[UN], B[UN];
#pragma unroll
    for (int k = 0; k < UN; ++k)
      if (k0 + k < n) {
        A[k] = e[long(k0 + k) * 2 * a.W];
        B[k] = e[(long(k0 + k) * 2 + 1) * a.W];
      }
#pragma unroll
    for (int k = 0; k < UN; ++k)
      if (k0 + k < n) {
        e[long(k0 + k) * 2 * a.W] = S;
        S = fmaf(A[k], S, B[k]);
      }
  }
  if (a.write_state) *st = S;
}

template <typename T>
__global__ void __launch_bounds__(128) diag_chunk_out_kernel(const DiagScanArgs a, const int* __restrict__ chunk_t0,
                                                             const int* __restrict__ chunk_n,
                                                             const float* __restrict__ ends) {
  griddep_wait();
  griddep_launch();
  const int c = blockIdx.x * 128 + threadIdx.x, ch = blockIdx.y;
  if (c >= a.W) return;
  const int n = chunk_n[ch];
  const long t0 = chunk_t0[ch];
  const Chan g = gate_of(c, a.W / a.blocks);
  const float yb = a.y_b[c];
  const float* gt = a.gates + t0 * 2 * a.W;
  const T* y = static_cast<const T*>(a.y) + t0 * a.ldy + c;
  T* out = static_cast<T*>(a.out) + t0 * a.ldo + c;
  float S = ends[long(ch) * 2 * a.W + c];
  for (int t = 0; t < n; t += UN) {
    float A[UN], B[UN], yv[UN];
#pragma unroll
    for (int k = 0; k < UN; ++k)
      if (t + k < n) {
        A[k] = gt[long(t + k) * 2 * a.W + g.r];
        B[k] = gt[long(t + k) * 2 * a.W + g.i];
        yv[k] = ld_f(y + (t + k) * a.ldy);
      }
#pragma unroll
    for (int k = 0; k < UN; ++k)
      if (t + k < n) {
        S = fmaf(A[k], S, B[k]);
        st_f(out + (t + k) * a.ldo, S * gelu_branch<T>(yv[k] + yb));
      }
  }
}

template <typename T>
int chunk_t(const DiagScanArgs& a, const int* chunk_t0, const int* chunk_n, int n_chunks, const int* seq_chunk0,
            const int* seq_nchunk, float* ends, cudaStream_t s) {
  const int cb = (a.W + 127) / 128;
  if (n_chunks > 65535 || a.n_seqs > 65535) return 1;
  if (launch_pdl(diag_chunk_terms_kernel<T>, dim3(cb, n_chunks), dim3(128), 0, s, a, chunk_t0, chunk_n, ends) != cudaSuccess)
    return 1;
  if (launch_pdl(diag_chunk_carry_kernel, dim3(cb, a.n_seqs), dim3(128), 0, s, a, seq_chunk0, seq_nchunk, ends) != cudaSuccess)
    return 1;
  return launch_pdl(diag_chunk_out_kernel<T>, dim3(cb, n_chunks), dim3(128), 0, s, a, chunk_t0, chunk_n,
                    static_cast<const float*>(ends)) != cudaSuccess;
}

// One decode step, one token per sequence: x + in_bias through the convolution with its history, the two block-diagonal
// products, recurrence, output. A CTA takes `SEQ` sequences and 32 of a block's channels: it evaluates u of the whole block
// (every CTA of the block does, from the same history), multiplies its rows of the two gate matrices with it, one warp
// per 4 rows of each, and updates its channels' state. The history of a block is replaced by the last of the block's CTAs
// to have read it (an arrival counter per block and sequence tile; nothing waits).
constexpr int DEC_SEQ = DIAG_DECODE_SEQ;
constexpr int DEC_CH = 32;

template <typename T>
__global__ void __launch_bounds__(256) diag_decode_kernel(const DiagDecodeArgs a) {
  extern __shared__ float u_s[];                       // [DEC_SEQ][d]
  __shared__ int last_s;
  __shared__ float z_s[DEC_SEQ][2][DEC_CH];
  griddep_wait();
  griddep_launch();
  const DiagScanArgs& r = a.s;
  const int d = r.W / r.blocks, parts = (d + DEC_CH - 1) / DEC_CH;
  const int b = blockIdx.x / parts, part = blockIdx.x % parts;
  const int s0 = blockIdx.y * DEC_SEQ, ns = min(DEC_SEQ, r.n_seqs - s0);
  const int K1 = a.KC - 1;
  const T* x = static_cast<const T*>(a.x);
  for (int i = threadIdx.x; i < ns * d; i += blockDim.x) {
    const int q = i / d, c = b * d + i % d, seq = s0 + q;
    const float* h = a.conv_state + (long(r.slots[seq]) * r.W + c) * K1;
    const float* w = a.conv_w + long(c) * a.KC;
    float acc = a.conv_b ? a.conv_b[c] : 0.f;
    for (int j = 0; j < K1; ++j) acc = fmaf(w[j], h[j], acc);
    acc = fmaf(w[K1], ld_f(x + seq * a.ldx + c) + a.in_bias[c], acc);
    T ur;                                               // the prompt form keeps u in the activation type
    st_f(&ur, acc);
    u_s[q * d + i % d] = ld_f(&ur);
  }
  __syncthreads();
  if (K1 > 0 && r.write_state) {
    if (threadIdx.x == 0) {
      __threadfence();
      unsigned int* ctr = a.ctr + blockIdx.y * r.blocks + b;
      const unsigned int old = atomicAdd(ctr, 1u);
      last_s = old == unsigned(parts - 1);
      if (last_s) *ctr = 0;
    }
    __syncthreads();
    if (last_s) {
      __threadfence();
      for (int i = threadIdx.x; i < ns * d; i += blockDim.x) {
        const int q = i / d, c = b * d + i % d, seq = s0 + q;
        float* h = a.conv_state + (long(r.slots[seq]) * r.W + c) * K1;
        for (int j = 0; j + 1 < K1; ++j) h[j] = h[j + 1];
        h[K1 - 1] = ld_f(x + seq * a.ldx + c) + a.in_bias[c];
      }
    }
  }
  // gates: warp w takes rows w, w + 8, ... of the part's 2 x DEC_CH rows
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const T* gw = static_cast<const T*>(a.gates_w) + long(b) * 2 * d * d;
  for (int row = warp; row < 2 * DEC_CH; row += 8) {
    const int which = row / DEC_CH, j = part * DEC_CH + row % DEC_CH;
    if (j >= d) continue;
    const T* wr = gw + (long(which) * d + j) * d;
    float acc[DEC_SEQ];
#pragma unroll
    for (int q = 0; q < DEC_SEQ; ++q) acc[q] = 0.f;
    if (a.vec) {
      for (int k = lane * 4; k < d; k += 128) {
        float w[4];
        ld_f4(wr + k, w);
#pragma unroll
        for (int q = 0; q < DEC_SEQ; ++q)
          if (q < ns) {
            const float4 u = *reinterpret_cast<const float4*>(u_s + q * d + k);
            acc[q] = fmaf(w[0], u.x, fmaf(w[1], u.y, fmaf(w[2], u.z, fmaf(w[3], u.w, acc[q]))));
          }
      }
    } else {
      for (int k = lane; k < d; k += 32) {
        const float w = ld_f(wr + k);
#pragma unroll
        for (int q = 0; q < DEC_SEQ; ++q)
          if (q < ns) acc[q] = fmaf(w, u_s[q * d + k], acc[q]);
      }
    }
#pragma unroll
    for (int q = 0; q < DEC_SEQ; ++q) {
      const float v = warp_sum_f(acc[q]);
      if (lane == 0) z_s[q][which][row % DEC_CH] = v;
    }
  }
  __syncthreads();
  for (int i = threadIdx.x; i < ns * DEC_CH; i += blockDim.x) {
    const int q = i / DEC_CH, j = part * DEC_CH + i % DEC_CH;
    if (j >= d) continue;
    const int c = b * d + j, seq = s0 + q;
    const Chan g = gate_of(c, d);
    const float2 ab = recur_terms<T>(z_s[q][0][i % DEC_CH] + r.gates_b[g.r], z_s[q][1][i % DEC_CH] + r.gates_b[g.i],
                                     u_s[q * d + j], r.log_decay[c]);
    float* st = r.state + long(r.slots[seq]) * r.W + c;
    const float S = fmaf(ab.x, *st, ab.y);
    if (r.write_state) *st = S;
    st_f(static_cast<T*>(r.out) + seq * r.ldo + c,
         S * gelu_branch<T>(ld_f(static_cast<const T*>(r.y) + seq * r.ldy + c) + r.y_b[c]));
  }
}

// The same step for bf16 and blocks of 32 to 256 channels (multiples of 32): the d / 32 CTAs of a block form a cluster.
// Each evaluates u of its own 32 channels - so it owns their history - and hands it to the others through distributed
// shared memory; its gate weights are on the way before the launch in front of this one has finished.
// SEQ sequences per CTA, eight at a time through the products, which run on mma.sync (u is rounded to bf16 anyway): four
// tiles of 16 of the CTA's 64 gate rows, each shared by two warps that take half of the columns.
__device__ __forceinline__ void mma_16x8x16(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
template <int NK, int SEQ>
__global__ void __launch_bounds__(256) diag_decode_cluster_kernel(const DiagDecodeArgs a, const int d) {
  constexpr int PER = (SEQ * DEC_CH + 255) / 256;        // (sequence, channel) pairs per thread: sequence q + 8 p
  constexpr int KS = 4 * NK;                             // steps of 16 columns per warp, at most
  constexpr int PITCH = 128 * NK + 8;                    // so that the eight rows of a fragment lie in different banks
  constexpr int ROWS = SEQ < 8 ? 8 : SEQ;
  __shared__ __align__(16) __nv_bfloat16 u_s[ROWS][PITCH];
  __shared__ float z_s[2][2 * DEC_CH][ROWS + 1];         // column half, gate row, sequence
  using T = __nv_bfloat16;
  const DiagScanArgs& r = a.s;
  const int parts = d / DEC_CH, b = blockIdx.x / parts, part = blockIdx.x % parts;
  const int s0 = blockIdx.y * SEQ, ns = min(SEQ, r.n_seqs - s0);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g4 = lane >> 2, t4 = lane & 3;
  asm volatile("barrier.cluster.arrive.relaxed.aligned;" ::: "memory");
  const T* gw = static_cast<const T*>(a.gates_w) + long(b) * 2 * d * d;
  const int half = d / 2, k0 = (warp >> 2) * half, row0 = (warp & 3) * 16;
  uint32_t w[KS][4];
#pragma unroll
  for (int i = 0; i < 4; ++i) {                          // fragment i: rows + 8 for odd i, columns + 8 for i >= 2
    const int row = row0 + g4 + (i & 1) * 8;
    const T* wr = gw + (long(row / DEC_CH) * d + part * DEC_CH + row % DEC_CH) * d + k0 + (i >> 1) * 8 + 2 * t4;
#pragma unroll
    for (int n = 0; n < KS; ++n) w[n][i] = n * 16 < half ? *reinterpret_cast<const uint32_t*>(wr + n * 16) : 0u;
  }
  const int c = b * d + part * DEC_CH + lane, K1 = a.KC - 1;
  const Chan g = gate_of(c, d);
  const float br = r.gates_b[g.r], bi = r.gates_b[g.i], ld = r.log_decay[c], yb = r.y_b[c], ib = a.in_bias[c];
  const float cb = a.conv_b ? a.conv_b[c] : 0.f;
  griddep_wait();
  griddep_launch();
  float u[PER], S[PER], yv[PER];
  float* st[PER];
#pragma unroll
  for (int p = 0; p < PER; ++p) {
    const int q = warp + 8 * p;
    u[p] = 0.f;
    st[p] = nullptr;
    if (q < ns) {
      const int seq = s0 + q, slot = r.slots[seq];
      float* h = a.conv_state + (long(slot) * r.W + c) * K1;
      const float* cw = a.conv_w + long(c) * a.KC;
      st[p] = r.state + long(slot) * r.W + c;
      const float xv = ld_f(static_cast<const T*>(a.x) + seq * a.ldx + c) + ib;
      S[p] = *st[p];
      yv[p] = ld_f(static_cast<const T*>(r.y) + seq * r.ldy + c) + yb;
      float acc = cb;
      if (K1 <= 4) {                                     // all loads before the first store
        float hv[4];
#pragma unroll
        for (int j = 0; j < 4; ++j) hv[j] = j < K1 ? h[j] : 0.f;
#pragma unroll
        for (int j = 0; j < 4; ++j)
          if (j < K1) {
            acc = fmaf(cw[j], hv[j], acc);
            h[j] = j + 1 < K1 ? hv[(j + 1) & 3] : xv;
          }
      } else {
        for (int j = 0; j < K1; ++j) {
          const float hv = h[j];
          acc = fmaf(cw[j], hv, acc);
          if (j > 0) h[j - 1] = hv;
        }
        h[K1 - 1] = xv;
      }
      u[p] = __bfloat162float(__float2bfloat16(fmaf(cw[K1], xv, acc)));
    }
  }
  asm volatile("barrier.cluster.wait.aligned;" ::: "memory");        // every CTA of the cluster has started
#pragma unroll
  for (int p = 0; p < PER; ++p) {
    const int q = warp + 8 * p;                          // rows past the last sequence hold zeros
    const uint32_t two = pack_bf16x2(u[p], __shfl_down_sync(0xffffffffu, u[p], 1));
    if (q < ROWS && !(lane & 1)) {
      const uint32_t local = smem_u32(&u_s[q][part * DEC_CH + lane]);
      for (int k = 0; k < parts; ++k) {
        uint32_t remote;
        asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(remote) : "r"(local), "r"(k));
        asm volatile("st.shared::cluster.u32 [%0], %1;" ::"r"(remote), "r"(two) : "memory");
      }
    }
  }
  asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory");
  asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory");
#pragma unroll
  for (int q0 = 0; q0 < ROWS; q0 += 8) {
    if (q0 >= ns) break;
    float acc[4] = {0.f, 0.f, 0.f, 0.f};
    const T* ub = &u_s[q0 + g4][k0 + 2 * t4];
#pragma unroll
    for (int n = 0; n < KS; ++n)
      if (n * 16 < half)
        mma_16x8x16(acc, w[n], *reinterpret_cast<const uint32_t*>(ub + n * 16), *reinterpret_cast<const uint32_t*>(ub + n * 16 + 8));
    float (*z)[ROWS + 1] = z_s[warp >> 2];
    z[row0 + g4][q0 + 2 * t4] = acc[0];
    z[row0 + g4][q0 + 2 * t4 + 1] = acc[1];
    z[row0 + g4 + 8][q0 + 2 * t4] = acc[2];
    z[row0 + g4 + 8][q0 + 2 * t4 + 1] = acc[3];
  }
  __syncthreads();
#pragma unroll
  for (int p = 0; p < PER; ++p) {
    const int q = warp + 8 * p;
    if (q < ns) {
      const float zr = z_s[0][lane][q] + z_s[1][lane][q], zi = z_s[0][DEC_CH + lane][q] + z_s[1][DEC_CH + lane][q];
      const float2 ab = recur_terms<T>(zr + br, zi + bi, u[p], ld);
      const float Sn = fmaf(ab.x, S[p], ab.y);
      *st[p] = Sn;
      st_f(static_cast<T*>(r.out) + (s0 + q) * r.ldo + c, Sn * gelu_branch<T>(yv[p]));
    }
  }
}

template <int NK, int SEQ>
int decode_cluster(const DiagDecodeArgs& a, int d, cudaStream_t s) {
  const int parts = d / DEC_CH;
  cudaLaunchConfig_t cfg{};
  cfg.gridDim = dim3(a.s.blocks * parts, (a.s.n_seqs + SEQ - 1) / SEQ);
  cfg.blockDim = dim3(256);
  cfg.stream = s;
  cudaLaunchAttribute attr[2];
  attr[0].id = cudaLaunchAttributeClusterDimension;
  attr[0].val.clusterDim.x = parts;
  attr[0].val.clusterDim.y = attr[0].val.clusterDim.z = 1;
  cfg.numAttrs = 1;
  if (pdl_enabled()) {
    attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[1].val.programmaticStreamSerializationAllowed = 1;
    cfg.numAttrs = 2;
  }
  cfg.attrs = attr;
  return cudaLaunchKernelEx(&cfg, diag_decode_cluster_kernel<NK, SEQ>, a, d) != cudaSuccess;
}
template <int NK>
int decode_cluster_n(const DiagDecodeArgs& a, int d, cudaStream_t s) {
  // as many sequences per CTA as leave about one wave of two CTAs per SM
  const long ctas = long(a.s.W / DEC_CH) * ((a.s.n_seqs + 7) / 8);
  if (ctas <= 296) return decode_cluster<NK, 8>(a, d, s);
  if (ctas <= 592) return decode_cluster<NK, 16>(a, d, s);
  return decode_cluster<NK, 32>(a, d, s);
}

template <typename T>
int decode_t(DiagDecodeArgs a, cudaStream_t s) {
  const int d = a.s.W / a.s.blocks, parts = (d + DEC_CH - 1) / DEC_CH;
  const size_t smem = size_t(DEC_SEQ) * d * 4;
  a.vec = d % 4 == 0 && reinterpret_cast<uintptr_t>(a.gates_w) % (4 * sizeof(T)) == 0;
  if constexpr (sizeof(T) == 2) {
    if (d % DEC_CH == 0 && d <= 256 && a.s.write_state && reinterpret_cast<uintptr_t>(a.gates_w) % 8 == 0)
      return d <= 128 ? decode_cluster_n<1>(a, d, s) : decode_cluster_n<2>(a, d, s);
  }
  if (smem > 200 * 1024) return 1;
  auto k = diag_decode_kernel<T>;
  if (smem > 40 * 1024 && cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, int(smem)) != cudaSuccess) return 1;
  return launch_pdl(k, dim3(a.s.blocks * parts, (a.s.n_seqs + DEC_SEQ - 1) / DEC_SEQ), dim3(256), smem, s, a) != cudaSuccess;
}

}  // namespace

int diag_scan_launch(const DiagScanArgs& a, bool f32, cudaStream_t s) {
  if (a.n_seqs <= 0 || a.T <= 0) return 0;
  if (a.blocks < 1 || a.W % a.blocks || a.n_seqs > 65535) return 1;
  const dim3 grid((a.W + 127) / 128, a.n_seqs);
  return (f32 ? launch_pdl(diag_tokens_kernel<float>, grid, dim3(128), 0, s, a)
              : launch_pdl(diag_tokens_kernel<__nv_bfloat16>, grid, dim3(128), 0, s, a)) != cudaSuccess;
}

int diag_chunk_launch(const DiagScanArgs& a, const int* chunk_t0, const int* chunk_n, int n_chunks, const int* seq_chunk0,
                      const int* seq_nchunk, float* ends, bool f32, cudaStream_t s) {
  if (a.n_seqs <= 0 || n_chunks <= 0) return 0;
  if (a.blocks < 1 || a.W % a.blocks) return 1;
  return f32 ? chunk_t<float>(a, chunk_t0, chunk_n, n_chunks, seq_chunk0, seq_nchunk, ends, s)
             : chunk_t<__nv_bfloat16>(a, chunk_t0, chunk_n, n_chunks, seq_chunk0, seq_nchunk, ends, s);
}

int diag_decode_launch(const DiagDecodeArgs& a, bool f32, cudaStream_t s) {
  if (a.s.n_seqs <= 0) return 0;
  if (a.s.blocks < 1 || a.s.W % a.s.blocks || a.KC < 1) return 1;
  return f32 ? decode_t<float>(a, s) : decode_t<__nv_bfloat16>(a, s);
}

}  // namespace lb
