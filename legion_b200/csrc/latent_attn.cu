// Pieces of latent attention for any sizes, bf16 and fp32, around the attention over the cached rows (attn_mla_sm100.cu;
// attn_general.cu for fp32): cache rows and rotated query parts, the output gate, the gather of a prompt's cached latents
// for its per-head form (keys and values of every head written out, attn_prefill_sm100.cu), and the two fused launches of
// a decode step - queries into the latent space with the cache append, and split merge with value projection and gate.
#include "act_type.cuh"
#include "common.cuh"
#include "layers.h"

namespace lb {
namespace {

// Column i of a vector whose first `rot` columns turn in neighbouring pairs; cs: cos | sin of the token's position.
template <typename T>
__device__ __forceinline__ float rotated(const T* v, int i, const float* cs, int rot) {
  const float x = ld_f(v + i);
  if (i >= rot) return x;
  const float c = cs[i >> 1], s = cs[(rot >> 1) + (i >> 1)];
  return (i & 1) ? x * c + ld_f(v + i - 1) * s : x * c - ld_f(v + i + 1) * s;
}

// Norm of the latent and rotation of the shared key part of one token, to its cache cell (one CTA of 128 threads).
template <typename T>
__device__ __forceinline__ void append_row(const LatentPrepArgs& a, int t, float* red) {
  const T* row = static_cast<const T*>(a.kv) + t * a.ldkv;
  float ss = 0.f;
  for (int i = threadIdx.x; i < a.L; i += blockDim.x) {
    const float v = ld_f(row + i);
    ss = fmaf(v, v, ss);
  }
  ss = warp_sum_f(ss);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
  __syncthreads();
  const long slot = a.slots[t];
  if (slot < 0) return;
  float tot = 0.f;
  for (int i = 0; i < int(blockDim.x) / 32; ++i) tot += red[i];
  const float inv = 1.f / sqrtf(tot / float(a.L) + a.eps);
  T* dst = static_cast<T*>(a.cache) + slot * a.cell;
  for (int i = threadIdx.x; i < a.L; i += blockDim.x) st_f(dst + i, ld_f(row + i) * inv * a.norm_w[i]);
  const float* cs = a.cos_sin + long(a.positions[t]) * a.rot;
  for (int i = threadIdx.x; i < a.R; i += blockDim.x) st_f(dst + a.L + i, rotated(row + a.L, i, cs, a.rot));
}

// Rotated part of a token's queries to their rows in the latent space.
template <typename T>
__device__ __forceinline__ void rotate_queries(const LatentPrepArgs& a, int t) {
  const float* cs = a.cos_sin + long(a.positions[t]) * a.rot;
  for (int i = threadIdx.x; i < a.heads * a.R; i += blockDim.x) {
    const int h = i / a.R, j = i % a.R;
    const T* q = static_cast<const T*>(a.q) + t * a.ldq + long(h) * (a.dim + a.R) + a.dim;
    st_f(static_cast<T*>(a.q_abs) + (long(t) * a.heads + h) * a.q_row + a.L + j, rotated(q, j, cs, a.rot));
  }
}

template <typename T>
__global__ void __launch_bounds__(128) latent_prep_kernel(const LatentPrepArgs a) {
  __shared__ float red[4];
  griddep_wait();
  griddep_launch();
  const int t = blockIdx.x;
  append_row<T>(a, t, red);
  rotate_queries<T>(a, t);
}

// 16 bytes of a row, neighbouring pairs turned; cs: cos of the first pair, sn: its sin
__device__ __forceinline__ uint4 rotate8(uint4 v, const float* c, const float* sn) {
  __nv_bfloat162* p = reinterpret_cast<__nv_bfloat162*>(&v);
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const float2 f = __bfloat1622float2(p[i]);
    p[i] = __floats2bfloat162_rn(f.x * c[i] - f.y * sn[i], f.y * c[i] + f.x * sn[i]);
  }
  return v;
}

// Prompts: queries as they are, their rotated part turned, [T, heads, dim + R] (bf16, dim and R multiples of 8, all of R
// rotated), and the token's cache row.
__global__ void __launch_bounds__(128) latent_prompt_prep_kernel(const LatentPrepArgs a) {
  __shared__ float red[4];
  griddep_wait();
  griddep_launch();
  const int t = blockIdx.x;
  using T = __nv_bfloat16;
  const float* cs = a.cos_sin + long(a.positions[t]) * a.rot;
  const int per = (a.dim + a.R) / 8, nd = a.dim / 8;
  const uint4* src = reinterpret_cast<const uint4*>(static_cast<const T*>(a.q) + t * a.ldq);
  uint4* dst = reinterpret_cast<uint4*>(static_cast<T*>(a.q_abs) + long(t) * a.heads * (a.dim + a.R));
  for (int i = threadIdx.x; i < a.heads * per; i += 128) {
    const int j = i % per - nd;
    const uint4 v = src[i];
    dst[i] = j < 0 ? v : rotate8(v, cs + 4 * j, cs + (a.rot >> 1) + 4 * j);
  }
  append_row<T>(a, t, red);
}

// Cached rows of the sequences of a step, 64 rows a page of the expanded buffers: latents to lat [rows, L], the shared key
// part behind every head's keys, k [rows, heads, dim + R]. Rows past a sequence's end become zero. One warp per row.
__global__ void __launch_bounds__(256) latent_gather_kernel(const LatentGatherArgs a) {
  griddep_wait();
  griddep_launch();
  const int row = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  const int pg = row >> 6, seq = a.page_seq[pg], pos = a.page_pos[pg] + (row & 63);
  const bool ok = pos < a.ctx_lens[seq];
  const __nv_bfloat16* src = static_cast<const __nv_bfloat16*>(a.cache);
  if (ok) src += (long(a.block_table[long(seq) * a.table_width + pos / a.page]) * a.page + pos % a.page) * a.cell;
  const uint4 zero = make_uint4(0u, 0u, 0u, 0u);
  uint4* lat = reinterpret_cast<uint4*>(static_cast<__nv_bfloat16*>(a.lat) + long(row) * a.L);
  for (int i = lane; i < a.L / 8; i += 32) lat[i] = ok ? reinterpret_cast<const uint4*>(src)[i] : zero;
  const int nr = a.R / 8;
  __nv_bfloat16* k = static_cast<__nv_bfloat16*>(a.k) + long(row) * a.heads * (a.dim + a.R) + a.dim;
  for (int i = lane; i < a.heads * nr; i += 32) {
    const int h = i / nr, j = i % nr;
    *reinterpret_cast<uint4*>(k + long(h) * (a.dim + a.R) + j * 8) = ok ? reinterpret_cast<const uint4*>(src + a.L)[j] : zero;
  }
}

// Sum over the lanes of 32 values per lane: lane l ends up with value l.
__device__ __forceinline__ float reduce_scatter32(float (&v)[32], int lane) {
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
__device__ __forceinline__ void unpack4(uint2 u, float (&f)[4]) {
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.x));
  const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.y));
  f[0] = a.x; f[1] = a.y; f[2] = b.x; f[3] = b.y;
}

// Decode, in front of the attention. CTA (head, 64 latent columns): q_abs = q W_uk for up to 16 tokens, its weights (8 rows
// per warp, 4 columns of every 128 per lane) on the way before the launch in front of this one has finished; the CTAs
// behind those: one token's cache row and the rotated part of its queries.
constexpr int LQ_TOK = 16;
template <int NK>
__global__ void __launch_bounds__(256) latent_decode_q_kernel(const LatentPrepArgs a, const __nv_bfloat16* __restrict__ uk) {
  __shared__ float red[8];
  using T = __nv_bfloat16;
  const int slices = (a.L + 63) / 64, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (int(blockIdx.x) >= a.heads * slices) {
    griddep_wait();
    griddep_launch();
    const int t = int(blockIdx.x) - a.heads * slices + int(blockIdx.y) * LQ_TOK;
    if (t < a.T) {
      append_row<T>(a, t, red);
      rotate_queries<T>(a, t);
    }
    return;
  }
  const int h = blockIdx.x / slices, l0 = (blockIdx.x % slices) * 64 + warp * 8;
  uint2 w[8][NK];
#pragma unroll
  for (int i = 0; i < 8; ++i)
#pragma unroll
    for (int n = 0; n < NK; ++n) {
      const int k = n * 128 + lane * 4;
      w[i][n] = (l0 + i < a.L && k < a.dim) ? *reinterpret_cast<const uint2*>(uk + (long(h) * a.L + l0 + i) * a.dim + k)
                                            : make_uint2(0u, 0u);
    }
  griddep_wait();
  griddep_launch();
  const int t_end = min(a.T, int(blockIdx.y + 1) * LQ_TOK);
  const T* q = static_cast<const T*>(a.q) + long(h) * (a.dim + a.R);
  T* out = static_cast<T*>(a.q_abs) + long(h) * a.q_row;
#pragma unroll 1
  for (int t0 = blockIdx.y * LQ_TOK; t0 < t_end; t0 += 4) {
    float v[32];
#pragma unroll
    for (int i = 0; i < 32; ++i) v[i] = 0.f;
#pragma unroll
    for (int n = 0; n < NK; ++n) {
      const int k = n * 128 + lane * 4;
      float x[4][4];
#pragma unroll
      for (int s = 0; s < 4; ++s) {
        const bool ok = t0 + s < t_end && k < a.dim;
        unpack4(ok ? *reinterpret_cast<const uint2*>(q + (t0 + s) * a.ldq + k) : make_uint2(0u, 0u), x[s]);
      }
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        float f[4];
        unpack4(w[i][n], f);
#pragma unroll
        for (int s = 0; s < 4; ++s)
          v[i * 4 + s] = fmaf(f[0], x[s][0], fmaf(f[1], x[s][1], fmaf(f[2], x[s][2], fmaf(f[3], x[s][3], v[i * 4 + s]))));
      }
    }
    const float r = reduce_scatter32(v, lane);
    const int l = l0 + lane / 4, t = t0 + lane % 4;
    if (l < a.L && t < t_end) out[long(t) * a.heads * a.q_row + l] = __float2bfloat16(r);
  }
}

// Decode, behind the attention. CTA (head, 32 value columns, up to 4 tokens): the key splits merged into shared memory, the
// value projection (4 rows per warp, weights on the way early) and the output gate.
constexpr int LV_TOK = 4;
template <int NK>
__global__ void __launch_bounds__(256) latent_decode_v_kernel(const LatentValueArgs a) {
  extern __shared__ float o_s[];                       // [LV_TOK][L]
  __shared__ float w_s[LV_TOK][64];
  using T = __nv_bfloat16;
  const int parts = (a.V + 31) / 32, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int h = blockIdx.x / parts, v0 = (blockIdx.x % parts) * 32 + warp * 4;
  const int t0 = blockIdx.y * LV_TOK, nt = min(LV_TOK, a.T - t0);
  const T* uv = static_cast<const T*>(a.uv) + long(h) * a.V * a.L;
  uint2 w[4][NK];
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int n = 0; n < NK; ++n) {
      const int k = n * 128 + lane * 4;
      w[i][n] = (v0 + i < a.V && k < a.L) ? *reinterpret_cast<const uint2*>(uv + long(v0 + i) * a.L + k) : make_uint2(0u, 0u);
    }
  griddep_wait();
  griddep_launch();
  if (a.n_splits > 1) {
    if (warp < nt) {                                    // share of every split in the merged row
      const float* ml = a.ml_part + (long(t0 + warp) * a.heads + h) * a.n_splits * 2;
      float m = -INFINITY;
      for (int s = lane; s < a.n_splits; s += 32) m = fmaxf(m, ml[2 * s]);
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, o));
      float sum = 0.f;
      for (int s = lane; s < a.n_splits; s += 32) {
        const float e = ml[2 * s] == -INFINITY ? 0.f : expf(ml[2 * s] - m);
        w_s[warp][s] = e;
        sum = fmaf(e, ml[2 * s + 1], sum);
      }
      sum = warp_sum_f(sum);
      const float inv = sum > 0.f ? 1.f / sum : 0.f;
      for (int s = lane; s < a.n_splits; s += 32) w_s[warp][s] *= inv;
    }
    __syncthreads();
    for (int i = threadIdx.x * 4; i < nt * a.L; i += 1024) {
      const int q = i / a.L, c = i % a.L;
      const float* o = a.o_part + (long(t0 + q) * a.heads + h) * a.n_splits * a.L + c;
      float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 4
      for (int s = 0; s < a.n_splits; ++s) {
        const float e = w_s[q][s];
        const float4 v = *reinterpret_cast<const float4*>(o + long(s) * a.L);
        if (e != 0.f) { acc.x = fmaf(e, v.x, acc.x); acc.y = fmaf(e, v.y, acc.y); acc.z = fmaf(e, v.z, acc.z); acc.w = fmaf(e, v.w, acc.w); }
      }
      *reinterpret_cast<float4*>(o_s + i) = acc;
    }
  } else {
    for (int i = threadIdx.x * 4; i < nt * a.L; i += 1024) {
      const int q = i / a.L, c = i % a.L;
      float f[4];
      ld_f4(static_cast<const T*>(a.o_lat) + (long(t0 + q) * a.heads + h) * a.L + c, f);
      *reinterpret_cast<float4*>(o_s + i) = make_float4(f[0], f[1], f[2], f[3]);
    }
  }
  for (int i = nt * a.L + threadIdx.x; i < LV_TOK * a.L; i += 256) o_s[i] = 0.f;
  __syncthreads();
  float v[16];
#pragma unroll
  for (int i = 0; i < 16; ++i) v[i] = 0.f;
#pragma unroll
  for (int n = 0; n < NK; ++n) {
    const int k = n * 128 + lane * 4;
    if (k < a.L) {
      float4 x[LV_TOK];
#pragma unroll
      for (int s = 0; s < LV_TOK; ++s) x[s] = *reinterpret_cast<const float4*>(o_s + s * a.L + k);
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        float f[4];
        unpack4(w[i][n], f);
#pragma unroll
        for (int s = 0; s < LV_TOK; ++s)
          v[i * 4 + s] = fmaf(f[0], x[s].x, fmaf(f[1], x[s].y, fmaf(f[2], x[s].z, fmaf(f[3], x[s].w, v[i * 4 + s]))));
      }
    }
  }
#pragma unroll
  for (int o = 8; o > 0; o >>= 1) {
    const bool up = lane & o;
#pragma unroll
    for (int i = 0; i < o; ++i) {
      const float send = up ? v[i] : v[i + o], keep = up ? v[i + o] : v[i];
      v[i] = keep + __shfl_xor_sync(0xffffffffu, send, o);
    }
  }
  const float r = v[0] + __shfl_xor_sync(0xffffffffu, v[0], 16);
  const int c = v0 + (lane & 15) / 4, q = lane % 4, t = t0 + q;
  if (lane < 16 && c < a.V && q < nt) {
    float g = 1.f;
    if (a.gate) g = sigmoid_f(ld_f(static_cast<const T*>(a.gate) + t * a.ldg + (a.per_head ? h : h * a.V + c)));
    static_cast<T*>(a.out)[long(t) * a.heads * a.V + h * a.V + c] = __float2bfloat16(r * g);
  }
}

template <typename T, int VEC>
__global__ void __launch_bounds__(256) latent_gate_kernel(T* __restrict__ x, const T* __restrict__ gate, long ldg,
                                                          int per_head, int vdim, int N, long n) {
  griddep_wait();
  griddep_launch();
  const long i = (long(blockIdx.x) * 256 + threadIdx.x) * VEC;
  if (i >= n) return;
  const long t = i / N;
  const int c = int(i % N);
  float v[VEC], g[VEC];
  ld_vec<VEC>(x + i, v);
  if (per_head) {
    const float s = sigmoid_f(ld_f(gate + t * ldg + c / vdim));
#pragma unroll
    for (int j = 0; j < VEC; ++j) v[j] *= s;
  } else {
    ld_vec<VEC>(gate + t * ldg + c, g);
#pragma unroll
    for (int j = 0; j < VEC; ++j) v[j] *= sigmoid_f(g[j]);
  }
  st_vec<VEC>(x + i, v);
}

template <typename T>
int gate_t(void* x, const void* gate, long ldg, int per_head, int vdim, int N, int T_, cudaStream_t s) {
  const long n = long(T_) * N;
  const bool v = vdim % 4 == 0 && reinterpret_cast<uintptr_t>(x) % (4 * sizeof(T)) == 0 &&
                 (per_head || (ldg % 4 == 0 && reinterpret_cast<uintptr_t>(gate) % (4 * sizeof(T)) == 0));
  const int vec = v ? 4 : 1;
  const dim3 grid(unsigned((n / vec + 255) / 256));
  return (v ? launch_pdl(latent_gate_kernel<T, 4>, grid, dim3(256), 0, s, static_cast<T*>(x), static_cast<const T*>(gate), ldg,
                         per_head, vdim, N, n)
            : launch_pdl(latent_gate_kernel<T, 1>, grid, dim3(256), 0, s, static_cast<T*>(x), static_cast<const T*>(gate), ldg,
                         per_head, vdim, N, n)) != cudaSuccess;
}

}  // namespace

int latent_prep_launch(const LatentPrepArgs& a, bool f32, cudaStream_t s) {
  if (a.T <= 0) return 0;
  if (a.rot % 2 || a.rot > a.R) return 1;
  return (f32 ? launch_pdl(latent_prep_kernel<float>, dim3(a.T), dim3(128), 0, s, a)
              : launch_pdl(latent_prep_kernel<__nv_bfloat16>, dim3(a.T), dim3(128), 0, s, a)) != cudaSuccess;
}

int latent_gate_launch(void* x, const void* gate, long ldg, int per_head, int vdim, int N, int T, bool f32, cudaStream_t s) {
  if (T <= 0 || N <= 0) return 0;
  return f32 ? gate_t<float>(x, gate, ldg, per_head, vdim, N, T, s)
             : gate_t<__nv_bfloat16>(x, gate, ldg, per_head, vdim, N, T, s);
}

int latent_prompt_prep_launch(const LatentPrepArgs& a, cudaStream_t s) {
  if (a.T <= 0) return 0;
  if (a.rot != a.R || a.R % 8 || a.dim % 8 || a.ldq % 8 || reinterpret_cast<uintptr_t>(a.q) % 16) return 1;
  return launch_pdl(latent_prompt_prep_kernel, dim3(a.T), dim3(128), 0, s, a) != cudaSuccess;
}

int latent_gather_launch(const LatentGatherArgs& a, cudaStream_t s) {
  if (a.pages <= 0) return 0;
  if (a.L % 8 || a.R % 8 || a.dim % 8 || a.cell % 8) return 1;
  return launch_pdl(latent_gather_kernel, dim3(a.pages * 8), dim3(256), 0, s, a) != cudaSuccess;
}

int latent_decode_q_launch(const LatentPrepArgs& a, const void* uk, cudaStream_t s) {
  if (a.T <= 0) return 0;
  if (a.rot % 2 || a.rot > a.R || a.dim % 4 || a.dim > 256 || a.ldq % 4 || (a.dim + a.R) % 4 ||
      (reinterpret_cast<uintptr_t>(a.q) | reinterpret_cast<uintptr_t>(uk)) % 8)
    return 1;
  const dim3 grid(a.heads * ((a.L + 63) / 64) + LQ_TOK, (a.T + LQ_TOK - 1) / LQ_TOK);
  auto k = a.dim <= 128 ? latent_decode_q_kernel<1> : latent_decode_q_kernel<2>;
  return launch_pdl(k, grid, dim3(256), 0, s, a, static_cast<const __nv_bfloat16*>(uk)) != cudaSuccess;
}

int latent_decode_v_launch(const LatentValueArgs& a, cudaStream_t s) {
  if (a.T <= 0) return 0;
  if (a.L % 4 || a.L > 512 || a.n_splits > 64 || reinterpret_cast<uintptr_t>(a.uv) % 8 || reinterpret_cast<uintptr_t>(a.o_lat) % 8)
    return 1;
  const dim3 grid(a.heads * ((a.V + 31) / 32), (a.T + LV_TOK - 1) / LV_TOK);
  const size_t smem = size_t(LV_TOK) * a.L * 4;
  auto k = a.L <= 128 ? latent_decode_v_kernel<1> : (a.L <= 256 ? latent_decode_v_kernel<2> : latent_decode_v_kernel<4>);
  return launch_pdl(k, grid, dim3(256), smem, s, a) != cudaSuccess;
}

}  // namespace lb
