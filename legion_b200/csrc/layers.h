// Launch interface of the layer kernels that work on bf16 and on fp32 activations (hyper.cu, sgemm.cu, attn_general.cu,
// linear_scan.cu, linear_scan_sm100.cu). Pointers are device pointers; f32 selects the activation type of the `void*`
// operands. Every function returns 0 on success and enqueues without synchronising.
#pragma once
#include <cuda_runtime.h>
#include <stddef.h>

#include "attn_extra.h"

namespace lb {

// Hyper-connections with static weights (hyper.cu). X [rows, S, H] fp32.
struct HyperArgs {
  const float* x_in;               // streams before the sublayer; nullptr: every stream starts as the embedding row
                                   // (normed with pre_w, if given)
  float* x_out;                    // streams after it (may be x_in)
  const void* emb; const int* ids; // start: embedding table and token ids (ids == nullptr: row t of emb)
  long ld_emb; int vocab;
  const void* y0; long ldy0; float c0;   // sublayer output: c0 * (sum of y_rows consecutive rows of y0) + c1 * y1
  const void* y1; long ldy1; float c1;
  int y_rows;
  const float* mix;                // [S from, S to]; nullptr: identity
  const float* out_w;              // [S]; nullptr: all ones
  const float* in_w;               // [S] weights of the next sublayer's input (nullptr: all ones)
  const float* norm_w; float eps, w_offset;
  void* h; long ldh;               // norm of the next input, activation type; nullptr: none
  const float* pre_w;              // start: norm of the embedding rows, nullptr: none
  void* raw; long ldraw;           // next input without the norm, activation type; nullptr: none
  int rows, S, H;
};
int hyper_launch(const HyperArgs& a, bool f32, cudaStream_t s);

// Parallel sublayers on one fp32 residual, with gates and depth average (depth_step.cu).
constexpr int DEPTH_AHEAD = 3;     // layers for which a pass over all earlier results sums up ahead
struct DepthStepArgs {
  const float* x;                  // [T, H] the layer's input
  float* x_out;                    // [n_rows, H] the next one's (may be x without rows)
  const float* hist; long hist_stride; int n_hist;   // earlier results to sum up, hist_stride floats apart
  const float* part;               // [T, H] sum of those before them; nullptr: none
  float* hist_out;                 // [T, H] takes the layer's result; nullptr: not kept
  const float* coef;               // [n_hist + 1] of hist's results and of the layer's own; nullptr: no average
  int n_ahead; float* ahead_out;   // [n_ahead] tensors [T, H], hist_stride apart: the same sums with other coefficients
  const float* ahead_coef[DEPTH_AHEAD];
  const void* y1; long ldy1;       // mixer output, activation type
  const void* y2; long ldy2; int y2_rows; const float* y2_b;   // feed-forward output, the sum of y2_rows consecutive rows
                                   // (nullptr: none), and its bias
  const void* g1; const void* g2; long ldg; const float* b1; const float* b2;   // gates before bias and sigmoid; nullptr: open
  const float* norm_w; float eps, w_offset;
  void* h; long ldh;               // [n_rows, H]
  const long* rows;                // tokens whose next input is wanted; nullptr: all
  int n_rows, H;
};
int depth_step_launch(const DepthStepArgs& a, bool f32, cudaStream_t s);

// One fp32 residual between grouped norms, with the next sublayer's input convolution (resid_step.cu).
struct ResidStepArgs {
  const float* x_in;               // [rows, H]; nullptr: start from the embedding
  float* x_out;                    // [rows, H], not x_in
  const void* emb; const int* ids; // start: embedding table and token ids (ids == nullptr: row t of emb), times emb_scale
  long ld_emb; int vocab; float emb_scale;
  const void* y; long ldy;         // sublayer output, activation type
  const float* post_w;             // its norm
  const float* norm_w;             // the next norm
  float eps; int groups;
  const float* taps; int taps_n;   // [taps_n, H], oldest token first; nullptr: h = n
  float* hist;                     // [slots, taps_n - 1, H]
  const int* cu; const int* slots; // without a convolution cu may be nullptr: every row is a sequence
  int n_seqs, max_len, tok;        // tok: tokens per CTA, at least taps_n - 1 where sequences are longer than it
  int write_state;
  void* h; long ldh;
  int rows, H;
  int direct;                      // set by the launcher
};
int resid_step_launch(const ResidStepArgs& a, bool f32, cudaStream_t s);

// Latent attention of any sizes (latent_attn.cu). kv rows: latent [L] | shared key part [R]; q rows: heads of [dim | R].
struct LatentPrepArgs {
  const void* q; long ldq;
  const void* kv; long ldkv;
  const float* norm_w; float eps;
  const float* cos_sin; int rot;   // [positions, rot]: cos | sin of rot / 2 pairs of neighbouring columns
  const int* positions; const long* slots;
  void* cache; long cell;          // elements between cache cells
  void* q_abs; long q_row;         // [T, heads] rows of q_row elements; columns [L, L + R) are written here
  int T, heads, dim, R, L;
};
int latent_prep_launch(const LatentPrepArgs& a, bool f32, cudaStream_t s);
// Prompts in the per-head form (bf16): q_abs takes [T, heads, dim + R] with the last R columns rotated; cache as above
int latent_prompt_prep_launch(const LatentPrepArgs& a, cudaStream_t s);
struct LatentGatherArgs {
  const void* cache; long cell;
  const int* block_table; int table_width, page; const int* ctx_lens;
  const int* page_seq; const int* page_pos;   // [pages] of 64 expanded rows: sequence and first position
  void* lat;                       // [pages * 64, L]
  void* k;                         // [pages * 64, heads, dim + R]; columns [dim, dim + R) are written
  int pages, heads, dim, R, L;
};
int latent_gather_launch(const LatentGatherArgs& a, cudaStream_t s);
// Decode (bf16): latent_prep and the queries' way into the latent space, uk [heads, L, dim], in one launch
int latent_decode_q_launch(const LatentPrepArgs& a, const void* uk, cudaStream_t s);
// Decode (bf16): merge of the key splits (n_splits > 1) or attended latents, value projection and gate
struct LatentValueArgs {
  const float* o_part; const float* ml_part; int n_splits;   // [T * heads, n_splits, L], [.., 2]
  const void* o_lat;               // n_splits == 1: [T, heads, L]
  const void* uv;                  // [heads, V, L]
  const void* gate; long ldg; int per_head;                  // nullptr: none
  void* out;                       // [T, heads * V]
  int T, heads, L, V;
};
int latent_decode_v_launch(const LatentValueArgs& a, cudaStream_t s);
// x[t, n] *= sigmoid(gate[t, per_head ? n / vdim : n]) in place
int latent_gate_launch(void* x, const void* gate, long ldg, int per_head, int vdim, int N, int T, bool f32, cudaStream_t s);

// Diagonal gated recurrence (diag_scan.cu): a = exp(sigmoid(r) log_decay), S = a S + sqrt(1 - a^2) sigmoid(i) u,
// out = S gelu(y + y_b). gates: [T, blocks, 2, W / blocks] fp32 before bias and sigmoid.
struct DiagScanArgs {
  const void* u; long ldu;
  float* gates;                    // overwritten by the chunked form
  const float* gates_b; const float* log_decay;
  const void* y; long ldy; const float* y_b;
  float* state;                    // [slots, W]
  const int* cu; const int* slots;
  int n_seqs, T, W, blocks;
  void* out; long ldo;
  int write_state;
  int max_tokens;                  // sequential form: sequences with more tokens are left alone (0: all run)
};
int diag_scan_launch(const DiagScanArgs& a, bool f32, cudaStream_t s);
// chunk tables as of linear_chunk_launch; ends: scratch of n_chunks * 2 * W floats
int diag_chunk_launch(const DiagScanArgs& a, const int* chunk_t0, const int* chunk_n, int n_chunks, const int* seq_chunk0,
                      const int* seq_nchunk, float* ends, bool f32, cudaStream_t s);
// One decode step with the convolution and the gate products in front of it
struct DiagDecodeArgs {
  const void* x; long ldx;         // [n, W] input of the convolution before in_bias
  const float* in_bias;
  const float* conv_w; const float* conv_b; float* conv_state; int KC;   // [W, KC], [slots, W, KC - 1]
  const void* gates_w;             // [blocks, 2, d, d], activation type
  DiagScanArgs s;                  // u and gates unused
  unsigned int* ctr;               // [sequence tiles, blocks] zeroed arrival counters, left zero
  int vec;                         // set by the launcher
};
int diag_decode_launch(const DiagDecodeArgs& a, bool f32, cudaStream_t s);
constexpr int DIAG_DECODE_SEQ = 4;  // sequences per tile

// Plain FMA GEMM (sgemm.cu): out[t, n] = sum_k x[t, k] w[n, k] in fp32, any sizes and pitches. Token tiles of
// SGEMM_BN rows; the grouped form takes the tile tables of the tcgen05 GEMM.
constexpr int SGEMM_BN = 32;
struct SgemmArgs {
  const void* x; long ldx;
  const void* w; long ldw;
  void* out; long ldo; int out_f32;
  const void* residual; long ldr;  // activation type
  const float* tok_scale;          // per activation row (grouped) multiplier
  const int* out_rows;             // activation row -> output row (negative: drop)
  int T, K, N;
  int dual; long dual_offset; int act;   // act(gate) * up, rows dual_offset apart; act 0 silu, 1 gelu (tanh), 2 relu^2
                                         // (no up), 3 xIELU (no up) with act_ab
  const float* act_ab;             // [2]
  const float* bias;               // dual: [2 * N] added to gate and up ahead of the activation
  int heads; long x_head_col, out_head_col;  // heads > 1: head z reads x columns from z * x_head_col and weight rows from
                                             // z * rows_per_group, and writes output columns from z * out_head_col
  const int* tile_group; const int* tile_tok0; const int* tile_ntok; const int* n_tiles; int max_tiles;
  long rows_per_group;
};
int sgemm_launch(const SgemmArgs& a, bool f32, cudaStream_t s);

// q / k head norms (optional) and the append of k and v to the paged cache, any head sizes (attn_general.cu)
int qkv_norm_append_launch(const void* q, const void* k, const void* v, long ld, const float* qw, const float* kw,
                           float eps, const long* slots, void* q_out, void* k_cache, void* v_cache, long k_cell,
                           long v_cell, int T, int Hq, int Hkv, int DK, int DV, bool f32, cudaStream_t s);
// What lies between a q | k | v projection and the scores (qkv_conv.cu): bias, short causal convolution with carried
// history, RMS norm of q and k over each head or the whole, rotation, append of k and v. All but the append optional.
struct QkvConvArgs {
  const void* x; long ld;          // [T, Hq * DK | Hkv * DK | Hkv * DV]
  const float* in_b;               // [columns]; the history holds x + in_b
  const float* conv_w; int KC;     // [KC, columns]; nullptr: none
  float* conv_state;               // [slots, KC - 1, columns]
  const int* cu; const int* state_slots; int n_seqs;
  const float* qw; const float* kw; int norm_all; float eps;   // weights [DK], or [Hq * DK] / [Hkv * DK] with norm_all
  const float* cos_sin; int rot; int rot_half;                 // [positions, rot]; rot_half: column i turns with i + rot / 2
  const int* positions; const long* slots;
  void* q_out; void* k_cache; void* v_cache; long k_cell, v_cell;
  int T, Hq, Hkv, DK, DV;
  int max_len;                     // longest sequence of the step
  int write_state;
  int tok, one;                    // set by the launcher: tokens per CTA; every sequence has one token
};
int qkv_conv_append_launch(QkvConvArgs a, bool f32, cudaStream_t s);

// Gated delta rule with a decay per key channel (channel_delta.cu)
struct ChannelDeltaArgs {
  const void* qkv; long ld;        // [T, G * DK | G * DK | H * DV] in front of the convolution
  const float* conv_w; int KC; float* conv_state;              // [KC, columns], [slots, KC - 1, columns]
  const void* a; long lda;         // [T, H * DK]: decay exp(A softplus(a + dt_bias))
  const float* A; const float* dt_bias;                        // [H], [H * DK]
  const void* b; long ldb;         // [T, H]: beta = sigmoid(b)
  float* state;                    // [slots, H, DV, DK]
  const int* cu; const int* slots;
  int n_seqs, T, H, G, DK, DV;
  float scale, l2_eps;
  void* out; long ldo;             // [T, H * DV]
  int write_state;
};
// floats of scratch per four tokens (and per sequence); rec: 128-byte aligned, for at least n_seqs + 1 of them
long channel_delta_record_floats(int H, int DK, int DV, bool f32);
int channel_delta_launch(const ChannelDeltaArgs& a, float* rec, long rec_floats, int* status, bool f32, cudaStream_t s);
// One decode step with the norm per head (times norm_w, times sigmoid(gate)) behind it; ctr: [n_seqs, G] zeroed arrival
// counters, left zero
int channel_delta_decode_launch(const ChannelDeltaArgs& a, const void* gate, long ldg, const float* norm_w, float eps,
                                unsigned int* ctr, bool f32, cudaStream_t s);
int head_norm_gate_launch(const void* o, long ldo, const void* gate, long ldg, const float* w, float eps, int H, int D, int rows,
                          void* out, long ldout, bool f32, cudaStream_t s);

// Paged causal attention on FMA units, one warp per (token, query head); value heads up to 1024 wide; q_row: elements
// between query heads
int paged_attn_general_launch(const void* q, long q_row, const void* k_cache, const void* v_cache, long k_cell, long v_cell,
                              const int* cu_q, const int* ctx_lens, const int* block_table, int table_width, int page,
                              int n_seqs, int T, int Hq, int Hkv, int DK, int DV, float scale, float softcap, int window,
                              void* out, bool f32, cudaStream_t s, const AttnExtra& x = AttnExtra{});

// Decayed outer-product state S_t = a_t S_(t-1) + k_t v_t^T, o_t = S_t^T q_t (linear_scan.cu, linear_scan_sm100.cu).
struct LinScanArgs {
  const void* q; long ldq;         // [T, G, N]
  const void* k; long ldk;
  const void* v; long ldv;         // [T, H, P]
  int silu_in;                     // q, k and v pass silu first
  const float* decay;              // [H] constant decay per head, or nullptr: the selective form below
  const void* dt; long lddt;       // [T, H] raw step sizes: dt = softplus(raw + dt_bias), a = exp(dt * A), v is scaled by dt
  const float* dt_bias; const float* A;
  const float* D;                  // [H] skip: o += D v (unscaled v); nullptr: none
  const void* z; long ldz;         // [T, H, P] gate: o *= silu(z); nullptr: none
  float* state;                    // [slots, H, P, N] fp32
  const int* cu; const int* slots;
  int n_seqs, T, H, G, N, P;
  void* out; long ldo;
  int write_state;
  int max_tokens;                  // linear_scan: sequences with more tokens are left alone (0: all run)
};
int linear_scan_launch(const LinScanArgs& a, bool f32, cudaStream_t s);

// Chunked form on tcgen05 (bf16): host-side tables of 128-token chunks. chunk_t0 / chunk_n: first token row and valid
// tokens; seq_chunk0 / seq_nchunk: chunk range of each sequence. scratch: linear_chunk_scratch_bytes, 256-byte aligned.
bool linear_chunk_ok(int N, int P);
size_t linear_chunk_scratch_bytes(int n_chunks, int H, int N, int P);
int linear_chunk_launch(const LinScanArgs& a, const int* chunk_t0, const int* chunk_n, const int* chunk_seq,
                        int n_chunks, const int* seq_chunk0, const int* seq_nchunk, void* scratch, int* status,
                        cudaStream_t s);

// HGRN2 (forget_scan.cu, forget_scan_sm100.cu): F = lower + (1 - lower) sigmoid(f + f_b), S_t = diag(F_t) S_(t-1) +
// (1 - F_t) v_t^T, o_t = S_t^T silu(q_t), out = o / rms(o) * norm_w * scale per head.
struct ForgetScanArgs {
  const void* q; const void* f; const void* v; long ldq, ldf, ldv;   // [T, H * N], [T, H * N], [T, H * P]
  const float* f_b; const float* lower;   // [H * N]
  float* state;                    // [slots, H, P, N]
  const int* cu; const int* slots;
  int n_seqs, T, H, N, P;
  const float* norm_w; float eps, scale;
  void* out; long ldo;             // [T, H * P]
  int write_state;
  int max_tokens;                  // forget_scan: sequences with more tokens are left alone (0: all run)
};
int forget_scan_launch(const ForgetScanArgs& a, bool f32, cudaStream_t s);
// Chunked form on tcgen05 (bf16), chunk tables as of linear_chunk_launch; scratch: forget_chunk_scratch_bytes, 256-byte aligned
bool forget_chunk_ok(int N, int P);
size_t forget_chunk_scratch_bytes(int n_chunks, int H, int N, int P);
int forget_chunk_launch(const ForgetScanArgs& a, const int* chunk_t0, const int* chunk_n, int n_chunks, const int* seq_chunk0,
                        const int* seq_nchunk, void* scratch, int* status, cudaStream_t s);

// One decode step of a Mamba-2 mixer: convolution with history update, step size, state update, skip and gate.
struct SsdDecodeArgs {
  const void* xbc; long ldx;       // [n, H * P + 2 * G * N] input projection columns x | B | C
  const float* conv_w; const float* conv_b; float* conv_state; int KC;
  LinScanArgs s;                   // q / k / v unused
  unsigned int* ctr;               // [n, G] zeroed arrival counters, left zero
};
int ssd_decode_launch(const SsdDecodeArgs& a, bool f32, cudaStream_t s);

// y normed in `groups` equal parts, times w, times sigmoid(gate) when a gate is given
int group_norm_gate_launch(const void* y, long ldy, const void* gate, long ldg, const float* w, float eps, int groups,
                           int C, int rows, void* out, long ldo, bool f32, cudaStream_t s);

// Causal depth-wise convolution (+ silu) with carried history, any number of taps (conv_any.cu); in_bias is added to x first
int conv_silu_any_launch(const void* x, long ldx, const float* w, const float* bias, float* conv_state,
                         const int* cu_seq, const int* slots, int n_seqs, int T, int C, int KC, void* out, long ldo,
                         int write_state, const float* in_bias, int silu, bool f32, cudaStream_t s);

// x = cap * tanh(x * scale / cap) in place (logits.cu)
int softcap_launch(float* x, float scale, float cap, long n, cudaStream_t s);

}  // namespace lb
