// Bindings of the layer kernels that take bf16 and fp32 activations (layers.h), and of the short convolution.
#include <ATen/cuda/CUDAContext.h>
#include <c10/cuda/CUDAGuard.h>
#include <torch/extension.h>

#include <cmath>

#include "gdn.h"
#include "layers.h"

namespace {
using torch::Tensor;
using OptT = c10::optional<Tensor>;

// text of the launch error behind a failed call, if there is one
std::string cuda_error() {
  const cudaError_t e = cudaGetLastError();
  return e == cudaSuccess ? std::string() : std::string(" (") + cudaGetErrorString(e) + ")";
}

cudaStream_t cur_stream() { return at::cuda::getCurrentCUDAStream().stream(); }

template <typename T>
T* optp(const OptT& t) {
  return t.has_value() ? reinterpret_cast<T*>(t->data_ptr()) : nullptr;
}

// activation type of a tensor: fp32 or bf16, innermost dimension contiguous
bool is_f32(const Tensor& t, const char* name) {
  TORCH_CHECK(t.is_cuda() && (t.scalar_type() == at::kFloat || t.scalar_type() == at::kBFloat16), name,
              " must be a float32 or bfloat16 CUDA tensor");
  TORCH_CHECK(t.stride(-1) == 1 || t.size(-1) == 1, name, " must be contiguous in its last dimension");
  return t.scalar_type() == at::kFloat;
}
void same(const Tensor& t, bool f32, const char* name) {
  TORCH_CHECK(is_f32(t, name) == f32, name, " must have the activation type");
}
void f32c(const Tensor& t, int64_t n, const char* name) {
  TORCH_CHECK(t.is_cuda() && t.scalar_type() == at::kFloat && t.is_contiguous() && t.numel() >= n, name,
              " must be a contiguous float32 tensor of at least ", n, " elements");
}

lb::LinScanArgs scan_args(const Tensor& q, const Tensor& k, const Tensor& v, bool silu_in, const OptT& decay,
                          const OptT& dt, const OptT& dt_bias, const OptT& A, const OptT& D, const OptT& z,
                          Tensor& state, const Tensor& cu, const Tensor& slots, int64_t H, int64_t G, int64_t N,
                          int64_t P, Tensor& out, bool write_state) {
  const bool f32 = is_f32(q, "q");
  same(k, f32, "k");
  same(v, f32, "v");
  same(out, f32, "out");
  const int64_t T = q.size(0);
  TORCH_CHECK(q.dim() == 2 && k.dim() == 2 && v.dim() == 2 && q.size(1) >= G * N && k.size(1) >= G * N && v.size(1) >= H * P &&
                  k.size(0) == T && v.size(0) == T && out.dim() == 2 && out.size(0) == T && out.size(1) >= H * P,
              "linear scan: q, k [T, G * N], v and out [T, H * P]");
  TORCH_CHECK(state.is_contiguous() && state.scalar_type() == at::kFloat && state.dim() == 4 && state.size(1) == H &&
                  state.size(2) == P && state.size(3) == N, "linear scan: state [slots, H, P, N] float32");
  TORCH_CHECK(cu.scalar_type() == at::kInt && slots.scalar_type() == at::kInt && cu.numel() == slots.numel() + 1,
              "linear scan: int32 sequence bounds and slots");
  lb::LinScanArgs a{};
  a.q = q.data_ptr(); a.ldq = q.stride(0); a.k = k.data_ptr(); a.ldk = k.stride(0); a.v = v.data_ptr(); a.ldv = v.stride(0);
  a.silu_in = silu_in;
  if (decay.has_value()) {
    f32c(*decay, H, "decay");
    a.decay = decay->data_ptr<float>();
  } else {
    TORCH_CHECK(dt.has_value() && dt_bias.has_value() && A.has_value(), "linear scan: step sizes, their bias and A");
    same(*dt, f32, "dt");
    TORCH_CHECK(dt->size(0) == T && dt->size(1) >= H, "linear scan: dt [T, H]");
    f32c(*dt_bias, H, "dt_bias");
    f32c(*A, H, "A");
    a.dt = dt->data_ptr(); a.lddt = dt->stride(0);
    a.dt_bias = dt_bias->data_ptr<float>(); a.A = A->data_ptr<float>();
  }
  if (D.has_value()) {
    f32c(*D, H, "D");
    a.D = D->data_ptr<float>();
  }
  if (z.has_value()) {
    same(*z, f32, "z");
    TORCH_CHECK(z->size(0) == T && z->size(1) >= H * P, "linear scan: z [T, H * P]");
    a.z = z->data_ptr(); a.ldz = z->stride(0);
  }
  a.state = state.data_ptr<float>();
  a.cu = cu.data_ptr<int>(); a.slots = slots.data_ptr<int>();
  a.n_seqs = int(slots.numel()); a.T = int(T); a.H = int(H); a.G = int(G); a.N = int(N); a.P = int(P);
  a.out = out.data_ptr(); a.ldo = out.stride(0);
  a.write_state = write_state;
  return a;
}

lb::DiagScanArgs diag_args(int64_t T, int64_t W, const Tensor& gates_b, const Tensor& log_decay, const Tensor& y,
                           const Tensor& y_b, Tensor& state, const Tensor& cu, const Tensor& slots, int64_t blocks,
                           Tensor& out, bool f32) {
  same(y, f32, "y");
  same(out, f32, "out");
  TORCH_CHECK(blocks >= 1 && W % blocks == 0 && y.dim() == 2 && y.size(0) == T && y.size(1) == W && out.dim() == 2 &&
                  out.size(0) == T && out.size(1) == W, "diag_scan: y and out [T, W], W in equal blocks");
  f32c(gates_b, 2 * W, "gate bias");
  f32c(log_decay, W, "log decay");
  f32c(y_b, W, "y bias");
  TORCH_CHECK(state.scalar_type() == at::kFloat && state.is_contiguous() && state.dim() == 2 && state.size(1) == W,
              "diag_scan: state [slots, W] float32");
  TORCH_CHECK(cu.scalar_type() == at::kInt && slots.scalar_type() == at::kInt && cu.numel() == slots.numel() + 1,
              "diag_scan: int32 sequence bounds and slots");
  lb::DiagScanArgs a{};
  a.gates_b = gates_b.data_ptr<float>(); a.log_decay = log_decay.data_ptr<float>();
  a.y = y.data_ptr(); a.ldy = y.stride(0); a.y_b = y_b.data_ptr<float>();
  a.state = state.data_ptr<float>(); a.cu = cu.data_ptr<int>(); a.slots = slots.data_ptr<int>();
  a.n_seqs = int(slots.numel()); a.T = int(T); a.W = int(W); a.blocks = int(blocks);
  a.out = out.data_ptr(); a.ldo = out.stride(0);
  return a;
}

lb::ChannelDeltaArgs delta_args(const Tensor& qkv, const Tensor& conv_w, Tensor& conv_state, const Tensor& a_raw, const Tensor& A,
                                const Tensor& dt_bias, const Tensor& b_raw, Tensor& state, const Tensor& cu, const Tensor& slots,
                                int64_t H, int64_t G, int64_t DK, int64_t DV, Tensor& out, bool f32) {
  const int64_t T = qkv.size(0), C = 2 * G * DK + H * DV;
  same(a_raw, f32, "decay projection");
  same(b_raw, f32, "beta projection");
  same(out, f32, "out");
  TORCH_CHECK(G >= 1 && H % G == 0 && qkv.dim() == 2 && qkv.size(1) == C && a_raw.size(0) == T && a_raw.size(1) == H * DK &&
                  b_raw.size(0) == T && b_raw.size(1) == H && out.size(0) == T && out.size(1) == H * DV,
              "channel_delta: q | k | v [T, columns], decays [T, H * DK], beta [T, H], out [T, H * DV]");
  f32c(conv_w, 0, "conv_w");
  TORCH_CHECK(conv_w.dim() == 2 && conv_w.size(1) == C, "channel_delta: conv_w [taps, columns]");
  TORCH_CHECK(conv_state.scalar_type() == at::kFloat && conv_state.is_contiguous() && conv_state.dim() == 3 &&
                  conv_state.size(2) == C && conv_state.size(1) == conv_w.size(0) - 1, "channel_delta: history [slots, taps - 1, columns]");
  f32c(A, H, "A");
  f32c(dt_bias, H * DK, "dt_bias");
  TORCH_CHECK(state.scalar_type() == at::kFloat && state.is_contiguous() && state.dim() == 4 && state.size(1) == H &&
                  state.size(2) == DV && state.size(3) == DK, "channel_delta: state [slots, H, DV, DK] float32");
  TORCH_CHECK(cu.scalar_type() == at::kInt && slots.scalar_type() == at::kInt && cu.numel() == slots.numel() + 1,
              "channel_delta: int32 sequence bounds and slots");
  lb::ChannelDeltaArgs a{};
  a.qkv = qkv.data_ptr(); a.ld = qkv.stride(0);
  a.conv_w = conv_w.data_ptr<float>(); a.KC = int(conv_w.size(0)); a.conv_state = conv_state.data_ptr<float>();
  a.a = a_raw.data_ptr(); a.lda = a_raw.stride(0); a.A = A.data_ptr<float>(); a.dt_bias = dt_bias.data_ptr<float>();
  a.b = b_raw.data_ptr(); a.ldb = b_raw.stride(0);
  a.state = state.data_ptr<float>(); a.cu = cu.data_ptr<int>(); a.slots = slots.data_ptr<int>();
  a.n_seqs = int(slots.numel()); a.T = int(T); a.H = int(H); a.G = int(G); a.DK = int(DK); a.DV = int(DV);
  a.scale = 1.f / std::sqrt(float(DK)); a.l2_eps = 1e-6f;
  a.out = out.data_ptr(); a.ldo = out.stride(0);
  return a;
}
}  // namespace

void bind_layers(pybind11::module_& m) {
  m.def("hyper_step", [](const OptT& x_in, Tensor& x_out, const OptT& emb, const OptT& ids, const OptT& y0, double c0,
                         int64_t y_rows, const OptT& y1, double c1, const OptT& mix, const OptT& out_w, const OptT& in_w,
                         const Tensor& norm_w, double eps, double w_offset, Tensor& h) {
    const bool f32 = is_f32(h, "h");
    TORCH_CHECK(x_out.dim() == 3 && x_out.is_contiguous() && x_out.scalar_type() == at::kFloat,
                "hyper_step: streams are contiguous float32 [rows, streams, width]");
    const int64_t R = x_out.size(0), S = x_out.size(1), H = x_out.size(2);
    TORCH_CHECK(h.dim() == 2 && h.size(0) == R && h.size(1) == H, "hyper_step: h [rows, width]");
    lb::HyperArgs a{};
    a.x_out = x_out.data_ptr<float>();
    if (x_in.has_value()) {
      TORCH_CHECK(x_in->sizes() == x_out.sizes() && x_in->is_contiguous() && x_in->scalar_type() == at::kFloat,
                  "hyper_step: x_in like x_out");
      TORCH_CHECK(y0.has_value() && mix.has_value() && out_w.has_value(), "hyper_step: sublayer output and its weights");
      same(*y0, f32, "y0");
      TORCH_CHECK(y0->dim() == 2 && y0->size(1) == H && y0->size(0) >= R * y_rows && y_rows >= 1,
                  "hyper_step: y0 [rows * y_rows, width]");
      f32c(*mix, S * S, "mix");
      f32c(*out_w, S, "out_w");
      a.x_in = x_in->data_ptr<float>();
      a.y0 = y0->data_ptr(); a.ldy0 = y0->stride(0);
      if (y1.has_value()) {
        same(*y1, f32, "y1");
        TORCH_CHECK(y1->dim() == 2 && y1->size(1) == H && y1->size(0) >= R, "hyper_step: y1 [rows, width]");
        a.y1 = y1->data_ptr(); a.ldy1 = y1->stride(0);
      }
      a.mix = mix->data_ptr<float>(); a.out_w = out_w->data_ptr<float>();
    } else {
      TORCH_CHECK(emb.has_value() && emb->dim() == 2 && emb->size(1) == H, "hyper_step: embedding rows");
      same(*emb, f32, "emb");
      a.emb = emb->data_ptr(); a.ld_emb = emb->stride(0); a.vocab = int(emb->size(0));
      if (ids.has_value()) {
        TORCH_CHECK(ids->scalar_type() == at::kInt && ids->is_contiguous() && ids->numel() == R, "hyper_step: int32 ids");
        a.ids = ids->data_ptr<int>();
      } else {
        TORCH_CHECK(emb->size(0) >= R, "hyper_step: one embedding row per token");
      }
    }
    if (in_w.has_value()) {
      f32c(*in_w, S, "in_w");
      a.in_w = in_w->data_ptr<float>();
    }
    f32c(norm_w, H, "norm_w");
    a.norm_w = norm_w.data_ptr<float>(); a.eps = float(eps); a.w_offset = float(w_offset);
    a.c0 = float(c0); a.c1 = float(c1); a.y_rows = int(y_rows);
    a.h = h.data_ptr(); a.ldh = h.stride(0); a.rows = int(R); a.S = int(S); a.H = int(H);
    c10::cuda::CUDAGuard guard(h.device());
    TORCH_CHECK(lb::hyper_launch(a, f32, cur_stream()) == 0, "hyper_step: at most 16 streams of 51200 columns", cuda_error());
  });
  m.def("prenorm_step", [](const OptT& x_in, Tensor& x_out, const OptT& emb, const OptT& ids, const OptT& pre_w, const OptT& y0,
                           double c0, int64_t y_rows, const OptT& y1, double c1, const OptT& norm_w, double eps, double w_offset,
                           const OptT& h, const OptT& raw) {
    // one stream of the hyper-connection launch without mix weights
    TORCH_CHECK(h.has_value() || raw.has_value(), "prenorm_step: nothing to write for the next sublayer");
    const bool f32 = is_f32(h.has_value() ? *h : *raw, "h");
    TORCH_CHECK(x_out.dim() == 2 && x_out.is_contiguous() && x_out.scalar_type() == at::kFloat,
                "prenorm_step: the stream is contiguous float32 [rows, width]");
    const int64_t R = x_out.size(0), H = x_out.size(1);
    lb::HyperArgs a{};
    a.x_out = x_out.data_ptr<float>();
    a.y_rows = 1;
    if (x_in.has_value()) {
      TORCH_CHECK(x_in->sizes() == x_out.sizes() && x_in->is_contiguous() && x_in->scalar_type() == at::kFloat,
                  "prenorm_step: x_in like x_out");
      a.x_in = x_in->data_ptr<float>();
      if (y0.has_value()) {
        same(*y0, f32, "y0");
        TORCH_CHECK(y0->dim() == 2 && y0->size(1) == H && y_rows >= 1 && y0->size(0) >= R * y_rows, "prenorm_step: y0 [rows * y_rows, width]");
        a.y0 = y0->data_ptr(); a.ldy0 = y0->stride(0); a.y_rows = int(y_rows);
      }
      if (y1.has_value()) {
        same(*y1, f32, "y1");
        TORCH_CHECK(y1->dim() == 2 && y1->size(1) == H && y1->size(0) >= R, "prenorm_step: y1 [rows, width]");
        a.y1 = y1->data_ptr(); a.ldy1 = y1->stride(0);
      }
    } else {
      TORCH_CHECK(emb.has_value() && emb->dim() == 2 && emb->size(1) == H, "prenorm_step: embedding rows");
      same(*emb, f32, "emb");
      a.emb = emb->data_ptr(); a.ld_emb = emb->stride(0); a.vocab = int(emb->size(0));
      if (ids.has_value()) {
        TORCH_CHECK(ids->scalar_type() == at::kInt && ids->is_contiguous() && ids->numel() == R, "prenorm_step: int32 ids");
        a.ids = ids->data_ptr<int>();
      } else {
        TORCH_CHECK(emb->size(0) >= R, "prenorm_step: one embedding row per token");
      }
      if (pre_w.has_value()) {
        f32c(*pre_w, H, "pre_w");
        a.pre_w = pre_w->data_ptr<float>();
      }
    }
    if (h.has_value()) {
      TORCH_CHECK(norm_w.has_value() && h->dim() == 2 && h->size(0) == R && h->size(1) == H, "prenorm_step: h [rows, width] and its norm");
      f32c(*norm_w, H, "norm_w");
      a.norm_w = norm_w->data_ptr<float>();
      a.h = h->data_ptr(); a.ldh = h->stride(0);
    }
    if (raw.has_value()) {
      same(*raw, f32, "raw");
      TORCH_CHECK(raw->dim() == 2 && raw->size(0) == R && raw->size(1) == H, "prenorm_step: raw [rows, width]");
      a.raw = raw->data_ptr(); a.ldraw = raw->stride(0);
    }
    a.c0 = float(c0); a.c1 = float(c1); a.eps = float(eps); a.w_offset = float(w_offset);
    a.rows = int(R); a.S = 1; a.H = int(H);
    c10::cuda::CUDAGuard guard(x_out.device());
    TORCH_CHECK(lb::hyper_launch(a, f32, cur_stream()) == 0, "prenorm_step: rows of at most 51200 columns", cuda_error());
  });
  // first: index of the first earlier result to sum up (those before it are in `part`); coefs: of this layer and, for the sums
  // that `ahead` takes, of the layers behind it
  m.def("depth_step", [](const Tensor& x, Tensor& x_out, const OptT& hist, int64_t layer, int64_t first, const OptT& part, bool keep,
                         const Tensor& y1, const OptT& g1, const OptT& b1, const OptT& y2, int64_t y2_rows, const OptT& g2,
                         const OptT& b2, const OptT& y2_b, const std::vector<Tensor>& coefs, const OptT& ahead,
                         const Tensor& norm_w, double eps, double w_offset, Tensor& h, const OptT& rows) {
    const bool f32 = is_f32(h, "h");
    same(y1, f32, "y1");
    const int64_t T = x.size(0), H = x.size(1), R = h.size(0);
    TORCH_CHECK(x.dim() == 2 && x.is_contiguous() && x.scalar_type() == at::kFloat && x_out.is_contiguous() && x_out.dim() == 2 &&
                    x_out.scalar_type() == at::kFloat && x_out.size(0) == R && x_out.size(1) == H && h.size(1) == H &&
                    y1.dim() == 2 && y1.size(0) == T && y1.size(1) == H, "depth_step: x, y1 [rows, width], x_out and h alike");
    lb::DepthStepArgs a{};
    a.x = x.data_ptr<float>(); a.x_out = x_out.data_ptr<float>();
    a.y1 = y1.data_ptr(); a.ldy1 = y1.stride(0); a.y2_rows = 1;
    if (hist.has_value()) {
      TORCH_CHECK(hist->is_contiguous() && hist->scalar_type() == at::kFloat && hist->dim() == 3 && hist->size(0) > layer + 1 &&
                      hist->size(1) == T && hist->size(2) == H && layer >= 0 && first >= 0 && first <= layer + 1 && !coefs.empty(),
                  "depth_step: hist [layers + 1, rows, width]");
      a.hist = hist->data_ptr<float>() + first * T * H; a.hist_stride = T * H; a.n_hist = int(layer + 1 - first);
      f32c(coefs[0], layer + 2, "depth average");
      a.coef = coefs[0].data_ptr<float>() + first;
      if (keep) a.hist_out = hist->data_ptr<float>() + (layer + 1) * T * H;
      if (part.has_value()) {
        f32c(*part, T * H, "partial sum");
        a.part = part->data_ptr<float>();
      }
      if (ahead.has_value()) {
        a.n_ahead = int(coefs.size()) - 1;
        TORCH_CHECK(a.n_ahead <= lb::DEPTH_AHEAD && first == 0, "depth_step: sums ahead");
        f32c(*ahead, a.n_ahead * T * H, "sums ahead");
        a.ahead_out = ahead->data_ptr<float>();
        for (int s = 0; s < a.n_ahead; ++s) {
          f32c(coefs[s + 1], layer + 2, "depth average");
          a.ahead_coef[s] = coefs[s + 1].data_ptr<float>();
        }
      }
    }
    if (y2.has_value()) {
      same(*y2, f32, "y2");
      TORCH_CHECK(y2->dim() == 2 && y2->size(1) == H && y2_rows >= 1 && y2->size(0) >= T * y2_rows, "depth_step: y2 [rows * y2_rows, width]");
      a.y2 = y2->data_ptr(); a.ldy2 = y2->stride(0); a.y2_rows = int(y2_rows);
      if (y2_b.has_value()) {
        f32c(*y2_b, H, "feed-forward bias");
        a.y2_b = y2_b->data_ptr<float>();
      }
    }
    auto gate = [&](const OptT& g, const OptT& b, const void*& gp, const float*& bp) {
      if (!g.has_value()) return;
      same(*g, f32, "gate");
      TORCH_CHECK(b.has_value() && g->dim() == 2 && g->size(0) == T && g->size(1) == H && (!a.ldg || a.ldg == g->stride(0)),
                  "depth_step: gates [rows, width] of one projection, with bias");
      f32c(*b, H, "gate bias");
      gp = g->data_ptr(); bp = b->data_ptr<float>(); a.ldg = g->stride(0);
    };
    gate(g1, b1, a.g1, a.b1);
    if (y2.has_value()) gate(g2, b2, a.g2, a.b2);
    if (rows.has_value()) {
      TORCH_CHECK(rows->scalar_type() == at::kLong && rows->is_contiguous() && rows->numel() == R && x_out.data_ptr() != x.data_ptr(),
                  "depth_step: int64 rows, an output of their own");
      a.rows = reinterpret_cast<const long*>(rows->data_ptr());
    } else {
      TORCH_CHECK(R == T, "depth_step: a row per token");
    }
    f32c(norm_w, H, "norm_w");
    a.norm_w = norm_w.data_ptr<float>(); a.eps = float(eps); a.w_offset = float(w_offset);
    a.h = h.data_ptr(); a.ldh = h.stride(0); a.n_rows = int(R); a.H = int(H);
    c10::cuda::CUDAGuard guard(x.device());
    TORCH_CHECK(lb::depth_step_launch(a, f32, cur_stream()) == 0, "depth_step: rows of at most 25600 columns", cuda_error());
  });
  auto forget_args = [](const Tensor& q, const Tensor& f, const Tensor& v, const Tensor& f_b, const Tensor& lower, Tensor& state,
                        const Tensor& cu, const Tensor& slots, int64_t H, int64_t N, int64_t P, const Tensor& norm_w, double eps,
                        double scale, Tensor& out, bool write_state) {
    const bool f32 = is_f32(q, "q");
    same(f, f32, "f");
    same(v, f32, "v");
    same(out, f32, "out");
    const int64_t T = q.size(0);
    TORCH_CHECK(q.dim() == 2 && f.dim() == 2 && v.dim() == 2 && out.dim() == 2 && q.size(1) == H * N && f.size(1) == H * N &&
                    v.size(1) == H * P && out.size(1) == H * P && f.size(0) == T && v.size(0) == T && out.size(0) == T,
                "forget scan: q, f [T, H * N], v and out [T, H * P]");
    f32c(f_b, H * N, "forget bias");
    f32c(lower, H * N, "lower bounds");
    f32c(norm_w, P, "norm weight");
    TORCH_CHECK(state.is_contiguous() && state.scalar_type() == at::kFloat && state.dim() == 4 && state.size(1) == H &&
                    state.size(2) == P && state.size(3) == N, "forget scan: state [slots, H, P, N] float32");
    TORCH_CHECK(cu.scalar_type() == at::kInt && slots.scalar_type() == at::kInt && cu.numel() == slots.numel() + 1,
                "forget scan: int32 sequence bounds and slots");
    lb::ForgetScanArgs a{};
    a.q = q.data_ptr(); a.ldq = q.stride(0); a.f = f.data_ptr(); a.ldf = f.stride(0); a.v = v.data_ptr(); a.ldv = v.stride(0);
    a.f_b = f_b.data_ptr<float>(); a.lower = lower.data_ptr<float>(); a.state = state.data_ptr<float>();
    a.cu = cu.data_ptr<int>(); a.slots = slots.data_ptr<int>();
    a.n_seqs = int(slots.numel()); a.T = int(T); a.H = int(H); a.N = int(N); a.P = int(P);
    a.norm_w = norm_w.data_ptr<float>(); a.eps = float(eps); a.scale = float(scale);
    a.out = out.data_ptr(); a.ldo = out.stride(0); a.write_state = write_state;
    return a;
  };
  m.def("forget_scan", [forget_args](const Tensor& q, const Tensor& f, const Tensor& v, const Tensor& f_b, const Tensor& lower,
                                     Tensor& state, const Tensor& cu, const Tensor& slots, int64_t H, int64_t N, int64_t P,
                                     const Tensor& norm_w, double eps, double scale, Tensor& out, bool write_state,
                                     int64_t max_tokens) {
    auto a = forget_args(q, f, v, f_b, lower, state, cu, slots, H, N, P, norm_w, eps, scale, out, write_state);
    a.max_tokens = int(max_tokens);
    c10::cuda::CUDAGuard guard(q.device());
    TORCH_CHECK(lb::forget_scan_launch(a, q.scalar_type() == at::kFloat, cur_stream()) == 0,
                "forget scan: key heads of at most 512 columns, value heads of at most 4096", cuda_error());
  });
  m.def("forget_chunk_ok", [](int64_t N, int64_t P) { return lb::forget_chunk_ok(int(N), int(P)); });
  m.def("forget_chunk_scratch_bytes", [](int64_t n_chunks, int64_t H, int64_t N, int64_t P) {
    return int64_t(lb::forget_chunk_scratch_bytes(int(n_chunks), int(H), int(N), int(P)));
  });
  m.def("forget_chunk", [forget_args](const Tensor& q, const Tensor& f, const Tensor& v, const Tensor& f_b, const Tensor& lower,
                                      Tensor& state, const Tensor& cu, const Tensor& slots, int64_t H, int64_t N, int64_t P,
                                      const Tensor& norm_w, double eps, double scale, Tensor& out, bool write_state,
                                      const Tensor& tab, int64_t n_chunks, Tensor& scratch, Tensor& status) {
    auto a = forget_args(q, f, v, f_b, lower, state, cu, slots, H, N, P, norm_w, eps, scale, out, write_state);
    TORCH_CHECK(q.scalar_type() == at::kBFloat16, "forget_chunk: bf16 activations");
    TORCH_CHECK(tab.scalar_type() == at::kInt && tab.is_contiguous() && tab.numel() >= 3 * n_chunks + 2 * a.n_seqs, "forget_chunk: chunk tables");
    TORCH_CHECK(scratch.is_contiguous() && size_t(scratch.numel() * scratch.element_size()) >=
                    lb::forget_chunk_scratch_bytes(int(n_chunks), int(H), int(N), int(P)), "forget_chunk: scratch");
    const int* t = tab.data_ptr<int>();
    c10::cuda::CUDAGuard guard(q.device());
    TORCH_CHECK(lb::forget_chunk_launch(a, t, t + n_chunks, int(n_chunks), t + 3 * n_chunks, t + 3 * n_chunks + a.n_seqs,
                                        scratch.data_ptr(), reinterpret_cast<int*>(status.data_ptr()), cur_stream()) == 0,
                "forget_chunk: heads of at most 128 columns", cuda_error());
  });
  m.def("qkv_conv_append", [](const Tensor& x, const OptT& in_b, const OptT& conv_w, const OptT& conv_state, const Tensor& cu,
                              const Tensor& state_slots, const OptT& qw, const OptT& kw, bool norm_all, double eps,
                              const OptT& cos_sin, bool rot_half, const Tensor& positions, const Tensor& slots, Tensor& q_out,
                              Tensor& k_cache, Tensor& v_cache, int64_t max_len, bool write_state) {
    const bool f32 = is_f32(x, "x");
    same(q_out, f32, "q_out");
    same(k_cache, f32, "k_cache");
    same(v_cache, f32, "v_cache");
    lb::QkvConvArgs a{};
    const int64_t T = q_out.size(0), Hq = q_out.size(1), DK = q_out.size(2), Hkv = k_cache.size(-2), DV = v_cache.size(-1);
    const int64_t C = (Hq + Hkv) * DK + Hkv * DV;
    TORCH_CHECK(x.dim() == 2 && x.size(0) == T && x.size(1) == C && k_cache.size(-1) == DK && v_cache.size(-2) == Hkv &&
                    q_out.is_contiguous() && k_cache.is_contiguous() && v_cache.is_contiguous(), "qkv_conv_append: q | k | v columns");
    TORCH_CHECK(cu.scalar_type() == at::kInt && state_slots.scalar_type() == at::kInt && cu.numel() == state_slots.numel() + 1 &&
                    positions.scalar_type() == at::kInt && positions.numel() == T && slots.scalar_type() == at::kLong &&
                    slots.numel() == T, "qkv_conv_append: int32 bounds, slots and positions, int64 cells");
    a.x = x.data_ptr(); a.ld = x.stride(0);
    if (in_b.has_value()) {
      f32c(*in_b, C, "bias");
      a.in_b = in_b->data_ptr<float>();
    }
    a.KC = 1;
    if (conv_w.has_value()) {
      f32c(*conv_w, 0, "conv_w");
      TORCH_CHECK(conv_w->dim() == 2 && conv_w->size(1) == C, "qkv_conv_append: conv_w [taps, columns]");
      a.conv_w = conv_w->data_ptr<float>();
      a.KC = int(conv_w->size(0));
      if (a.KC > 1) {
        TORCH_CHECK(conv_state.has_value() && conv_state->scalar_type() == at::kFloat && conv_state->is_contiguous() &&
                        conv_state->dim() == 3 && conv_state->size(2) == C && conv_state->size(1) == a.KC - 1,
                    "qkv_conv_append: history [slots, taps - 1, columns]");
        a.conv_state = conv_state->data_ptr<float>();
      }
    }
    a.cu = cu.data_ptr<int>(); a.state_slots = state_slots.data_ptr<int>(); a.n_seqs = int(state_slots.numel());
    TORCH_CHECK(qw.has_value() == kw.has_value(), "qkv_conv_append: norms of q and k go together");
    if (qw.has_value()) {
      f32c(*qw, norm_all ? Hq * DK : DK, "q norm");
      f32c(*kw, norm_all ? Hkv * DK : DK, "k norm");
      a.qw = qw->data_ptr<float>(); a.kw = kw->data_ptr<float>();
    }
    a.norm_all = norm_all; a.eps = float(eps);
    if (cos_sin.has_value()) {
      f32c(*cos_sin, 0, "cos_sin");
      a.cos_sin = cos_sin->data_ptr<float>();
      a.rot = int(cos_sin->size(1));
    }
    a.rot_half = rot_half;
    a.positions = positions.data_ptr<int>(); a.slots = reinterpret_cast<const long*>(slots.data_ptr());
    a.q_out = q_out.data_ptr(); a.k_cache = k_cache.data_ptr(); a.v_cache = v_cache.data_ptr();
    a.k_cell = Hkv * DK; a.v_cell = Hkv * DV;
    a.T = int(T); a.Hq = int(Hq); a.Hkv = int(Hkv); a.DK = int(DK); a.DV = int(DV);
    a.max_len = int(max_len); a.write_state = write_state;
    c10::cuda::CUDAGuard guard(x.device());
    TORCH_CHECK(lb::qkv_conv_append_launch(a, f32, cur_stream()) == 0,
                "qkv_conv_append: at most 51200 query and key columns, rotation within a head", cuda_error());
  });
  m.def("channel_delta_record_floats", [](int64_t H, int64_t DK, int64_t DV, bool f32) {
    return int64_t(lb::channel_delta_record_floats(int(H), int(DK), int(DV), f32));
  });
  m.def("channel_delta", [](const Tensor& qkv, const Tensor& conv_w, Tensor& conv_state, const Tensor& a_raw, const Tensor& A,
                            const Tensor& dt_bias, const Tensor& b_raw, Tensor& state, const Tensor& cu, const Tensor& slots,
                            int64_t H, int64_t G, int64_t DK, int64_t DV, Tensor& out, bool write_state, const Tensor& rec,
                            Tensor& status) {
    const bool f32 = is_f32(qkv, "qkv");
    auto a = delta_args(qkv, conv_w, conv_state, a_raw, A, dt_bias, b_raw, state, cu, slots, H, G, DK, DV, out, f32);
    a.write_state = write_state;
    f32c(rec, 0, "scratch");
    c10::cuda::CUDAGuard guard(qkv.device());
    TORCH_CHECK(lb::channel_delta_launch(a, rec.data_ptr<float>(), rec.numel(), reinterpret_cast<int*>(status.data_ptr()), f32,
                                         cur_stream()) == 0,
                "channel_delta: key heads of at most 256 columns, heads a multiple of the key heads", cuda_error());
  });
  m.def("channel_delta_decode", [](const Tensor& qkv, const Tensor& conv_w, Tensor& conv_state, const Tensor& a_raw, const Tensor& A,
                                   const Tensor& dt_bias, const Tensor& b_raw, Tensor& state, const Tensor& cu,
                                   const Tensor& slots, int64_t H, int64_t G, int64_t DK, int64_t DV, const Tensor& gate,
                                   const Tensor& norm_w, double eps, Tensor& ctr, Tensor& out) {
    const bool f32 = is_f32(qkv, "qkv");
    auto a = delta_args(qkv, conv_w, conv_state, a_raw, A, dt_bias, b_raw, state, cu, slots, H, G, DK, DV, out, f32);
    a.write_state = 1;
    same(gate, f32, "gate");
    f32c(norm_w, DV, "norm weight");
    TORCH_CHECK(qkv.size(0) == slots.numel() && gate.size(0) == qkv.size(0) && gate.size(1) == H * DV && ctr.element_size() == 4 &&
                    ctr.numel() >= slots.numel() * G, "channel_delta_decode: one token per sequence, gate like the output");
    c10::cuda::CUDAGuard guard(qkv.device());
    TORCH_CHECK(lb::channel_delta_decode_launch(a, gate.data_ptr(), gate.stride(0), norm_w.data_ptr<float>(), float(eps),
                                                reinterpret_cast<unsigned int*>(ctr.data_ptr()), f32, cur_stream()) == 0,
                "channel_delta_decode: key heads of at most 256 columns, heads a multiple of the key heads", cuda_error());
  });
  m.def("head_norm_gate", [](const Tensor& o, const Tensor& gate, const Tensor& w, double eps, int64_t H, Tensor& out) {
    const bool f32 = is_f32(o, "o");
    same(gate, f32, "gate");
    same(out, f32, "out");
    const int64_t R = o.size(0), C = o.size(1);
    TORCH_CHECK(H > 0 && C % H == 0 && gate.size(0) == R && gate.size(1) == C && out.size(0) == R && out.size(1) == C,
                "head_norm_gate: o, gate and out [rows, heads * d]");
    f32c(w, C / H, "norm weight");
    c10::cuda::CUDAGuard guard(o.device());
    TORCH_CHECK(lb::head_norm_gate_launch(o.data_ptr(), o.stride(0), gate.data_ptr(), gate.stride(0), w.data_ptr<float>(),
                                          float(eps), int(H), int(C / H), int(R), out.data_ptr(), out.stride(0), f32,
                                          cur_stream()) == 0, "head_norm_gate failed", cuda_error());
  });
  m.def("sgemm", [](const Tensor& w, const Tensor& x, Tensor& out, const OptT& residual, const OptT& tok_scale,
                    const OptT& out_rows, int64_t n_feat, bool dual, int64_t dual_offset, int64_t act,
                    const OptT& tile_group, const OptT& tile_tok0, const OptT& tile_ntok, const OptT& meta,
                    int64_t max_tiles, int64_t rows_per_group, int64_t n_tok, const OptT& act_ab, const OptT& bias) {
    const bool f32 = is_f32(x, "x");
    same(w, f32, "w");
    TORCH_CHECK(w.dim() == 2 && x.dim() == 2 && out.dim() == 2 && w.size(1) == x.size(1), "sgemm: K mismatch");
    if (act_ab.has_value()) f32c(*act_ab, 2, "activation numbers");
    TORCH_CHECK(act != 3 || (act_ab.has_value() && !dual), "sgemm: xIELU takes two numbers");
    is_f32(out, "out");
    TORCH_CHECK(out.size(1) >= n_feat && w.size(0) >= n_feat + (dual ? dual_offset : 0), "sgemm: shapes");
    lb::SgemmArgs a{};
    a.x = x.data_ptr(); a.ldx = x.stride(0); a.w = w.data_ptr(); a.ldw = w.stride(0);
    a.out = out.data_ptr(); a.ldo = out.stride(0); a.out_f32 = out.scalar_type() == at::kFloat;
    if (residual.has_value()) {
      same(*residual, f32, "residual");
      a.residual = residual->data_ptr(); a.ldr = residual->stride(0);
    }
    a.tok_scale = optp<float>(tok_scale); a.out_rows = optp<int>(out_rows);
    a.T = int(n_tok); a.K = int(x.size(1)); a.N = int(n_feat);
    a.dual = dual; a.dual_offset = dual_offset; a.act = int(act); a.act_ab = optp<float>(act_ab);
    if (bias.has_value()) {
      TORCH_CHECK(dual && !tile_group.has_value(), "sgemm: biases of an ungrouped gate/up product");
      f32c(*bias, 2 * n_feat, "bias");
      a.bias = bias->data_ptr<float>();
    }
    a.tile_group = optp<int>(tile_group); a.tile_tok0 = optp<int>(tile_tok0); a.tile_ntok = optp<int>(tile_ntok);
    a.n_tiles = optp<int>(meta); a.max_tiles = int(max_tiles); a.rows_per_group = rows_per_group;
    TORCH_CHECK(!a.tile_group || (a.tile_tok0 && a.tile_ntok && a.n_tiles), "sgemm: incomplete tile tables");
    TORCH_CHECK(a.tile_group || x.size(0) >= n_tok, "sgemm: too few rows");
    c10::cuda::CUDAGuard guard(x.device());
    TORCH_CHECK(lb::sgemm_launch(a, f32, cur_stream()) == 0, "sgemm failed", cuda_error());
  }, pybind11::arg("w"), pybind11::arg("x"), pybind11::arg("out"), pybind11::arg("residual"), pybind11::arg("tok_scale"),
     pybind11::arg("out_rows"), pybind11::arg("n_feat"), pybind11::arg("dual"), pybind11::arg("dual_offset"), pybind11::arg("act"),
     pybind11::arg("tile_group"), pybind11::arg("tile_tok0"), pybind11::arg("tile_ntok"), pybind11::arg("meta"),
     pybind11::arg("max_tiles"), pybind11::arg("rows_per_group"), pybind11::arg("n_tok"), pybind11::arg("act_ab"),
     pybind11::arg("bias") = pybind11::none());
  m.def("qkv_norm_append", [](const Tensor& q, const Tensor& k, const Tensor& v, const OptT& qw, const OptT& kw, double eps,
                              const Tensor& slots, Tensor& q_out, Tensor& k_cache, Tensor& v_cache) {
    const bool f32 = is_f32(q, "q");
    same(k, f32, "k");
    same(v, f32, "v");
    same(k_cache, f32, "k_cache");
    same(v_cache, f32, "v_cache");
    same(q_out, f32, "q_out");
    const int64_t T = q_out.size(0), Hq = q_out.size(1), DK = q_out.size(2), Hkv = k_cache.size(-2), DV = v_cache.size(-1);
    TORCH_CHECK(q.size(0) == T && q.size(1) == Hq * DK && k.size(1) == Hkv * DK && v.size(1) == Hkv * DV &&
                    k_cache.size(-1) == DK && v_cache.size(-2) == Hkv, "qkv_norm_append: shapes");
    TORCH_CHECK(q.stride(0) == k.stride(0) && q.stride(0) == v.stride(0), "qkv_norm_append: column slices of one projection");
    TORCH_CHECK(slots.scalar_type() == at::kLong && slots.numel() == T, "qkv_norm_append: slots int64 [T]");
    TORCH_CHECK(q_out.is_contiguous() && k_cache.is_contiguous() && v_cache.is_contiguous(), "qkv_norm_append: contiguous");
    if (qw.has_value()) f32c(*qw, DK, "q norm");
    if (kw.has_value()) f32c(*kw, DK, "k norm");
    c10::cuda::CUDAGuard guard(q.device());
    TORCH_CHECK(lb::qkv_norm_append_launch(q.data_ptr(), k.data_ptr(), v.data_ptr(), q.stride(0), optp<float>(qw),
                                           optp<float>(kw), float(eps), reinterpret_cast<const long*>(slots.data_ptr()),
                                           q_out.data_ptr(), k_cache.data_ptr(), v_cache.data_ptr(), Hkv * DK, Hkv * DV,
                                           int(T), int(Hq), int(Hkv), int(DK), int(DV), f32, cur_stream()) == 0,
                "qkv_norm_append failed", cuda_error());
  });
  m.def("paged_attn_general", [](const Tensor& q, const Tensor& k_cache, const Tensor& v_cache, const Tensor& cu_q,
                                 const Tensor& ctx_lens, const Tensor& block_table, double scale, int64_t window,
                                 Tensor& out, double softcap, int64_t keep, const OptT& sink, const OptT& gate, double out_scale) {
    const bool f32 = is_f32(q, "q");
    same(k_cache, f32, "k_cache");
    same(v_cache, f32, "v_cache");
    same(out, f32, "out");
    const int64_t T = q.size(0), Hq = q.size(1), DK = q.size(2), Hkv = k_cache.size(-2), DV = v_cache.size(-1);
    lb::AttnExtra x;
    if (out.dim() == 2) {              // rows may lie apart; sinks, kept first tokens, output gate and scale
      TORCH_CHECK(out.size(0) == T && out.size(1) == Hq * DV && keep >= 0, "paged_attn_general: out [T, heads * value head size]");
      x.on = 1; x.keep = int(keep); x.out_scale = float(out_scale); x.ldo = out.stride(0);
      if (sink.has_value()) {
        f32c(*sink, Hq, "sinks");
        x.sink = sink->data_ptr<float>();
      }
      if (gate.has_value()) {
        same(*gate, f32, "gate");
        TORCH_CHECK(gate->size(0) == T && gate->size(1) == Hq, "paged_attn_general: gate [T, heads]");
        x.gate = gate->data_ptr(); x.ld_gate = gate->stride(0);
      }
    } else {
      TORCH_CHECK(out.dim() == 3 && out.is_contiguous() && out.size(0) == T && out.size(1) == Hq && out.size(2) == DV && !keep &&
                      !sink.has_value() && !gate.has_value() && out_scale == 1., "paged_attn_general: out [T, heads, size]");
    }
    TORCH_CHECK(q.is_contiguous() && k_cache.is_contiguous() && v_cache.is_contiguous() && k_cache.size(-1) == DK,
                "paged_attn_general: shapes");
    TORCH_CHECK(cu_q.scalar_type() == at::kInt && ctx_lens.scalar_type() == at::kInt && block_table.scalar_type() == at::kInt &&
                    cu_q.numel() == ctx_lens.numel() + 1 && block_table.stride(1) == 1, "paged_attn_general: int32 tables");
    c10::cuda::CUDAGuard guard(q.device());
    TORCH_CHECK(lb::paged_attn_general_launch(q.data_ptr(), DK, k_cache.data_ptr(), v_cache.data_ptr(), Hkv * DK, Hkv * DV,
                                              cu_q.data_ptr<int>(), ctx_lens.data_ptr<int>(), block_table.data_ptr<int>(),
                                              int(block_table.stride(0)), int(k_cache.size(-3)), int(ctx_lens.numel()),
                                              int(T), int(Hq), int(Hkv), int(DK), int(DV), float(scale), float(softcap),
                                              int(window), out.data_ptr(), f32, cur_stream(), x) == 0,
                "paged_attn_general: value heads of at most 1024 columns, key heads of at most 2560", cuda_error());
  }, pybind11::arg("q"), pybind11::arg("k_cache"), pybind11::arg("v_cache"), pybind11::arg("cu_q"), pybind11::arg("ctx_lens"),
     pybind11::arg("block_table"), pybind11::arg("scale"), pybind11::arg("window"), pybind11::arg("out"), pybind11::arg("softcap"),
     pybind11::arg("keep") = 0, pybind11::arg("sink") = pybind11::none(), pybind11::arg("gate") = pybind11::none(),
     pybind11::arg("out_scale") = 1.);
  m.def("linear_scan", [](const Tensor& q, const Tensor& k, const Tensor& v, bool silu_in, const OptT& decay, const OptT& dt,
                          const OptT& dt_bias, const OptT& A, const OptT& D, const OptT& z, Tensor& state, const Tensor& cu,
                          const Tensor& slots, int64_t H, int64_t G, int64_t N, int64_t P, Tensor& out, bool write_state,
                          int64_t max_tokens) {
    auto a = scan_args(q, k, v, silu_in, decay, dt, dt_bias, A, D, z, state, cu, slots, H, G, N, P, out, write_state);
    a.max_tokens = int(max_tokens);
    c10::cuda::CUDAGuard guard(q.device());
    TORCH_CHECK(lb::linear_scan_launch(a, q.scalar_type() == at::kFloat, cur_stream()) == 0,
                "linear scan: at most 512 state columns, heads a multiple of the groups", cuda_error());
  });
  m.def("ssd_decode", [](const Tensor& xbc, const Tensor& conv_w, const OptT& conv_b, Tensor& conv_state, const Tensor& dt,
                         const Tensor& dt_bias, const Tensor& A, const OptT& D, const OptT& z, Tensor& state,
                         const Tensor& cu, const Tensor& slots, int64_t H, int64_t G, int64_t N, int64_t P, Tensor& ctr,
                         Tensor& out) {
    const int64_t inner = H * P, n = slots.numel();
    TORCH_CHECK(xbc.dim() == 2 && xbc.size(0) == n && xbc.size(1) == inner + 2 * G * N, "ssd_decode: x | B | C columns");
    const Tensor x = xbc.narrow(1, 0, inner), B = xbc.narrow(1, inner, G * N), Cm = xbc.narrow(1, inner + G * N, G * N);
    lb::SsdDecodeArgs a{};
    a.s = scan_args(Cm, B, x, false, c10::nullopt, dt, dt_bias, A, D, z, state, cu, slots, H, G, N, P, out, true);
    f32c(conv_w, conv_w.numel(), "conv_w");
    TORCH_CHECK(conv_w.dim() == 2 && conv_w.size(0) == xbc.size(1), "ssd_decode: conv_w [channels, taps]");
    a.xbc = xbc.data_ptr(); a.ldx = xbc.stride(0);
    a.conv_w = conv_w.data_ptr<float>(); a.conv_b = optp<float>(conv_b); a.KC = int(conv_w.size(1));
    TORCH_CHECK(conv_state.scalar_type() == at::kFloat && conv_state.is_contiguous() && conv_state.dim() == 3 &&
                    conv_state.size(1) == xbc.size(1) && conv_state.size(2) == a.KC - 1, "ssd_decode: history [slots, C, taps - 1]");
    a.conv_state = conv_state.data_ptr<float>();
    TORCH_CHECK(ctr.numel() >= n * G && ctr.element_size() == 4 && ctr.is_contiguous(), "ssd_decode: counters [n, G]");
    a.ctr = reinterpret_cast<unsigned int*>(ctr.data_ptr());
    c10::cuda::CUDAGuard guard(xbc.device());
    TORCH_CHECK(lb::ssd_decode_launch(a, xbc.scalar_type() == at::kFloat, cur_stream()) == 0, "ssd_decode: unsupported sizes", cuda_error());
  });
  m.def("linear_chunk_ok", [](int64_t N, int64_t P) { return lb::linear_chunk_ok(int(N), int(P)); });
  m.def("linear_chunk_scratch_bytes", [](int64_t n_chunks, int64_t H, int64_t N, int64_t P) {
    return int64_t(lb::linear_chunk_scratch_bytes(int(n_chunks), int(H), int(N), int(P)));
  });
  m.def("linear_chunk", [](const Tensor& q, const Tensor& k, const Tensor& v, bool silu_in, const OptT& decay, const OptT& dt,
                           const OptT& dt_bias, const OptT& A, const OptT& D, const OptT& z, Tensor& state,
                           const Tensor& cu, const Tensor& slots, int64_t H, int64_t G, int64_t N, int64_t P, Tensor& out,
                           bool write_state, const Tensor& tables, int64_t n_chunks, Tensor& scratch, Tensor& status) {
    const auto a = scan_args(q, k, v, silu_in, decay, dt, dt_bias, A, D, z, state, cu, slots, H, G, N, P, out, write_state);
    TORCH_CHECK(q.scalar_type() == at::kBFloat16, "linear_chunk: bf16 activations");
    TORCH_CHECK(tables.scalar_type() == at::kInt && tables.is_contiguous() && tables.numel() >= 3 * n_chunks + 2 * a.n_seqs,
                "linear_chunk: tables = chunk_t0 | chunk_n | chunk_seq | seq_chunk0 | seq_nchunk");
    TORCH_CHECK(size_t(scratch.numel()) * scratch.element_size() >=
                    lb::linear_chunk_scratch_bytes(int(n_chunks), int(H), int(N), int(P)), "linear_chunk: scratch too small");
    const int* tb = tables.data_ptr<int>();
    c10::cuda::CUDAGuard guard(q.device());
    TORCH_CHECK(lb::linear_chunk_launch(a, tb, tb + n_chunks, tb + 2 * n_chunks, int(n_chunks), tb + 3 * n_chunks,
                                        tb + 3 * n_chunks + a.n_seqs, scratch.data_ptr(),
                                        reinterpret_cast<int*>(status.data_ptr()), cur_stream()) == 0,
                "linear_chunk: unsupported sizes", cuda_error());
  });
  m.def("group_norm_gate", [](const Tensor& y, const OptT& gate, const Tensor& w, double eps, int64_t groups, Tensor& out) {
    const bool f32 = is_f32(y, "y");
    same(out, f32, "out");
    const int64_t R = y.size(0), C = y.size(1);
    TORCH_CHECK(y.dim() == 2 && out.size(0) == R && out.size(1) == C && groups > 0 && C % groups == 0, "group_norm_gate: shapes");
    f32c(w, C, "norm weight");
    if (gate.has_value()) {
      same(*gate, f32, "gate");
      TORCH_CHECK(gate->size(0) == R && gate->size(1) == C, "group_norm_gate: gate like y");
    }
    c10::cuda::CUDAGuard guard(y.device());
    TORCH_CHECK(lb::group_norm_gate_launch(y.data_ptr(), y.stride(0), gate.has_value() ? gate->data_ptr() : nullptr,
                                           gate.has_value() ? gate->stride(0) : 0, w.data_ptr<float>(), float(eps),
                                           int(groups), int(C), int(R), out.data_ptr(), out.stride(0), f32, cur_stream()) == 0,
                "group_norm_gate failed", cuda_error());
  });
  m.def("conv1d_silu", [](const Tensor& x, const Tensor& w, const OptT& bias, Tensor& conv_state, const Tensor& cu_seq,
                          const Tensor& slots, Tensor& out, bool write_state, int64_t max_len, const OptT& in_bias,
                          bool silu) {
    c10::cuda::CUDAGuard guard(x.device());
    TORCH_CHECK(x.scalar_type() == at::kBFloat16 && w.scalar_type() == at::kFloat, "conv1d_silu dtypes");
    if (in_bias.has_value()) f32c(*in_bias, x.size(1), "input bias");
    TORCH_CHECK(lb::conv1d_silu_launch(x.data_ptr(), x.stride(0), w.data_ptr<float>(), optp<float>(bias),
                                       conv_state.data_ptr<float>(), cu_seq.data_ptr<int>(), slots.data_ptr<int>(),
                                       int(slots.numel()), int(x.size(1)), int(w.size(1)), out.data_ptr(),
                                       out.stride(0), write_state ? 1 : 0, cur_stream(), int(max_len),
                                       optp<float>(in_bias), silu) == 0,
                "conv1d_silu: unsupported kernel width");
  });
  m.def("conv_silu_any", [](const Tensor& x, const Tensor& w, const OptT& bias, Tensor& conv_state, const Tensor& cu,
                            const Tensor& slots, Tensor& out, bool write_state, const OptT& in_bias, bool silu) {
    const bool f32 = is_f32(x, "x");
    if (in_bias.has_value()) f32c(*in_bias, x.size(1), "input bias");
    same(out, f32, "out");
    const int64_t T = x.size(0), C = x.size(1), KC = w.size(1);
    TORCH_CHECK(w.size(0) == C && out.size(0) == T && out.size(1) == C && conv_state.is_contiguous() &&
                    conv_state.size(1) == C && conv_state.size(2) == KC - 1, "conv_silu_any: shapes");
    f32c(w, C * KC, "conv weight");
    if (bias.has_value()) f32c(*bias, C, "conv bias");
    c10::cuda::CUDAGuard guard(x.device());
    TORCH_CHECK(lb::conv_silu_any_launch(x.data_ptr(), x.stride(0), w.data_ptr<float>(), optp<float>(bias),
                                         conv_state.data_ptr<float>(), cu.data_ptr<int>(), slots.data_ptr<int>(),
                                         int(slots.numel()), int(T), int(C), int(KC), out.data_ptr(), out.stride(0),
                                         write_state, optp<float>(in_bias), silu, f32, cur_stream()) == 0,
                "conv_silu_any: at most 65535 tokens per step", cuda_error());
  });
  // per-head products: out[t, h * out_col + n] = sum_k x[t, h * x_col + k] w[h * rows + n, k]
  m.def("sgemm_heads", [](const Tensor& w, const Tensor& x, Tensor& out, int64_t heads, int64_t rows, int64_t n_feat, int64_t K,
                          int64_t x_col, int64_t out_col) {
    const bool f32 = is_f32(x, "x");
    same(w, f32, "w");
    is_f32(out, "out");
    TORCH_CHECK(heads >= 1 && heads <= 65535 && w.dim() == 2 && x.dim() == 2 && out.dim() == 2 && w.size(1) == K &&
                    w.size(0) >= (heads - 1) * rows + n_feat && x.size(1) >= (heads - 1) * x_col + K &&
                    out.size(0) == x.size(0) && out.size(1) >= (heads - 1) * out_col + n_feat, "sgemm_heads: shapes");
    lb::SgemmArgs a{};
    a.x = x.data_ptr(); a.ldx = x.stride(0); a.w = w.data_ptr(); a.ldw = w.stride(0);
    a.out = out.data_ptr(); a.ldo = out.stride(0); a.out_f32 = out.scalar_type() == at::kFloat;
    a.T = int(x.size(0)); a.K = int(K); a.N = int(n_feat);
    a.heads = int(heads); a.x_head_col = x_col; a.out_head_col = out_col; a.rows_per_group = rows;
    c10::cuda::CUDAGuard guard(x.device());
    TORCH_CHECK(lb::sgemm_launch(a, f32, cur_stream()) == 0, "sgemm_heads failed", cuda_error());
  });
  m.def("resid_step", [](const OptT& x_in, Tensor& x_out, const OptT& emb, const OptT& ids, double emb_scale, const OptT& y,
                         const OptT& post_w, const Tensor& norm_w, int64_t groups, double eps, const OptT& taps,
                         const OptT& hist, const OptT& cu, const OptT& slots, bool write_state, int64_t max_len, int64_t tok,
                         Tensor& h) {
    const bool f32 = is_f32(h, "h");
    TORCH_CHECK(x_out.dim() == 2 && x_out.is_contiguous() && x_out.scalar_type() == at::kFloat,
                "resid_step: the residual is contiguous float32 [rows, width]");
    const int64_t R = x_out.size(0), H = x_out.size(1);
    TORCH_CHECK(h.dim() == 2 && h.size(0) == R && h.size(1) == H, "resid_step: h [rows, width]");
    TORCH_CHECK(groups >= 1 && H % groups == 0, "resid_step: the width must divide into ", groups, " groups");
    lb::ResidStepArgs a{};
    a.x_out = x_out.data_ptr<float>();
    if (x_in.has_value()) {
      TORCH_CHECK(x_in->sizes() == x_out.sizes() && x_in->is_contiguous() && x_in->scalar_type() == at::kFloat &&
                      x_in->data_ptr() != x_out.data_ptr(), "resid_step: x_in like x_out, in a buffer of its own");
      TORCH_CHECK(y.has_value() && post_w.has_value(), "resid_step: sublayer output and its norm");
      same(*y, f32, "y");
      TORCH_CHECK(y->dim() == 2 && y->size(0) == R && y->size(1) == H, "resid_step: y [rows, width]");
      f32c(*post_w, H, "post norm");
      a.x_in = x_in->data_ptr<float>();
      a.y = y->data_ptr(); a.ldy = y->stride(0); a.post_w = post_w->data_ptr<float>();
    } else {
      TORCH_CHECK(emb.has_value() && emb->dim() == 2 && emb->size(1) == H, "resid_step: embedding rows");
      same(*emb, f32, "emb");
      a.emb = emb->data_ptr(); a.ld_emb = emb->stride(0); a.vocab = int(emb->size(0)); a.emb_scale = float(emb_scale);
      if (ids.has_value()) {
        TORCH_CHECK(ids->scalar_type() == at::kInt && ids->is_contiguous() && ids->numel() == R, "resid_step: int32 ids");
        a.ids = ids->data_ptr<int>();
      } else {
        TORCH_CHECK(emb->size(0) >= R, "resid_step: one embedding row per token");
      }
    }
    f32c(norm_w, H, "norm_w");
    a.norm_w = norm_w.data_ptr<float>(); a.eps = float(eps); a.groups = int(groups);
    a.rows = int(R); a.H = int(H);
    a.h = h.data_ptr(); a.ldh = h.stride(0);
    a.n_seqs = int(R); a.max_len = 1; a.tok = 1;
    if (taps.has_value()) {
      TORCH_CHECK(taps->dim() == 2 && taps->size(1) == H && cu.has_value() && slots.has_value() && hist.has_value(),
                  "resid_step: taps [taps, width], history, bounds and slots");
      const int64_t K = taps->size(0);
      f32c(*taps, K * H, "taps");
      TORCH_CHECK(hist->scalar_type() == at::kFloat && hist->is_contiguous() && hist->dim() == 3 && hist->size(1) == K - 1 &&
                      hist->size(2) == H, "resid_step: history [slots, taps - 1, width] float32");
      TORCH_CHECK(cu->scalar_type() == at::kInt && slots->scalar_type() == at::kInt && cu->numel() == slots->numel() + 1,
                  "resid_step: int32 sequence bounds and slots");
      a.taps = taps->data_ptr<float>(); a.taps_n = int(K); a.hist = hist->data_ptr<float>();
      a.cu = cu->data_ptr<int>(); a.slots = slots->data_ptr<int>(); a.n_seqs = int(slots->numel());
      a.max_len = int(max_len); a.tok = int(tok);
    }
    a.write_state = write_state;
    c10::cuda::CUDAGuard guard(h.device());
    TORCH_CHECK(lb::resid_step_launch(a, f32, cur_stream()) == 0, "resid_step: width ", H, ", ", groups, " groups, ",
                a.taps_n, " taps, ", a.tok, " tokens per block", cuda_error());
  });
  // the cache append and the queries: rot part only (latent space rows), with uk also their way into the latent space;
  // prompt: q_abs takes the queries themselves, [T, heads, dim + rot]
  m.def("latent_prep", [](const Tensor& q, const Tensor& kv, const Tensor& norm_w, double eps, const Tensor& cos_sin,
                          const Tensor& positions, const Tensor& slots, Tensor& cache, Tensor& q_abs, int64_t dim, int64_t rot,
                          const OptT& uk, bool prompt) {
    const bool f32 = is_f32(q, "q");
    same(kv, f32, "kv");
    same(cache, f32, "cache");
    same(q_abs, f32, "q_abs");
    const int64_t T = q.size(0), H = q_abs.size(1), L = norm_w.numel();
    TORCH_CHECK(q.dim() == 2 && kv.dim() == 2 && kv.size(0) == T && q.size(1) >= H * (dim + rot) && kv.size(1) >= L + rot,
                "latent_prep: q [T, heads * (dim + rot)], kv [T, rank + rot]");
    TORCH_CHECK(q_abs.dim() == 3 && q_abs.is_contiguous() && q_abs.size(0) == T &&
                    (prompt ? q_abs.size(2) == dim + rot : q_abs.size(2) >= L + rot) && cache.is_contiguous() &&
                    cache.size(-1) >= L + rot, "latent_prep: rows of rank + rot columns");
    f32c(norm_w, L, "norm");
    TORCH_CHECK(cos_sin.dim() == 2 && cos_sin.size(1) <= rot && cos_sin.size(1) % 2 == 0, "latent_prep: table [positions, rotated columns]");
    f32c(cos_sin, 0, "cos_sin");
    TORCH_CHECK(positions.scalar_type() == at::kInt && slots.scalar_type() == at::kLong && positions.numel() == T &&
                    slots.numel() == T, "latent_prep: positions int32, slots int64");
    lb::LatentPrepArgs a{};
    a.q = q.data_ptr(); a.ldq = q.stride(0); a.kv = kv.data_ptr(); a.ldkv = kv.stride(0);
    a.norm_w = norm_w.data_ptr<float>(); a.eps = float(eps);
    a.cos_sin = cos_sin.data_ptr<float>(); a.rot = int(cos_sin.size(1));
    a.positions = positions.data_ptr<int>(); a.slots = reinterpret_cast<const long*>(slots.data_ptr());
    a.cache = cache.data_ptr(); a.cell = cache.size(-1); a.q_abs = q_abs.data_ptr(); a.q_row = q_abs.size(2);
    a.T = int(T); a.heads = int(H); a.dim = int(dim); a.R = int(rot); a.L = int(L);
    c10::cuda::CUDAGuard guard(q.device());
    if (uk.has_value()) {
      TORCH_CHECK(!f32 && !is_f32(*uk, "uk") && uk->is_contiguous() && uk->numel() == H * L * dim, "latent_prep: uk [heads * rank, dim]");
      TORCH_CHECK(lb::latent_decode_q_launch(a, uk->data_ptr(), cur_stream()) == 0, "latent decode queries failed", cuda_error());
    } else if (prompt) {
      TORCH_CHECK(!f32, "latent_prep: the prompt form is bf16");
      TORCH_CHECK(lb::latent_prompt_prep_launch(a, cur_stream()) == 0, "latent prompt queries failed", cuda_error());
    } else {
      TORCH_CHECK(lb::latent_prep_launch(a, f32, cur_stream()) == 0, "latent_prep failed", cuda_error());
    }
  });
  m.def("latent_gather", [](const Tensor& cache, const Tensor& block_table, const Tensor& ctx_lens, const Tensor& pages,
                            Tensor& lat, Tensor& k, int64_t dim, int64_t rot) {
    TORCH_CHECK(!is_f32(cache, "cache") && !is_f32(lat, "lat") && !is_f32(k, "k"), "latent_gather: bf16");
    const int64_t n = pages.size(1), L = lat.size(1), H = k.size(1);
    TORCH_CHECK(pages.scalar_type() == at::kInt && pages.is_contiguous() && pages.size(0) == 2 && lat.is_contiguous() &&
                    k.is_contiguous() && lat.size(0) == n * 64 && k.size(0) == n * 64 && k.size(2) == dim + rot &&
                    cache.is_contiguous() && cache.dim() == 4 && cache.size(3) >= L + rot, "latent_gather: shapes");
    TORCH_CHECK(block_table.scalar_type() == at::kInt && ctx_lens.scalar_type() == at::kInt && block_table.stride(1) == 1,
                "latent_gather: int32 tables");
    lb::LatentGatherArgs a{};
    a.cache = cache.data_ptr(); a.cell = cache.size(3); a.page = int(cache.size(1));
    a.block_table = block_table.data_ptr<int>(); a.table_width = int(block_table.stride(0)); a.ctx_lens = ctx_lens.data_ptr<int>();
    a.page_seq = pages.data_ptr<int>(); a.page_pos = pages.data_ptr<int>() + n;
    a.lat = lat.data_ptr(); a.k = k.data_ptr();
    a.pages = int(n); a.heads = int(H); a.dim = int(dim); a.R = int(rot); a.L = int(L);
    c10::cuda::CUDAGuard guard(cache.device());
    TORCH_CHECK(lb::latent_gather_launch(a, cur_stream()) == 0, "latent_gather failed", cuda_error());
  });
  m.def("latent_decode_v", [](const OptT& o_part, const OptT& ml_part, int64_t n_splits, const OptT& o_lat, const Tensor& uv,
                              const OptT& gate, int64_t heads, int64_t L, Tensor& out) {
    TORCH_CHECK(!is_f32(uv, "uv") && !is_f32(out, "out") && uv.is_contiguous() && uv.size(1) == L && out.is_contiguous() &&
                    uv.size(0) % heads == 0 && out.size(1) == uv.size(0), "latent_decode_v: uv [heads * V, rank], out [T, heads * V]");
    const int64_t T = out.size(0), V = uv.size(0) / heads;
    lb::LatentValueArgs a{};
    a.n_splits = int(n_splits);
    if (n_splits > 1) {
      TORCH_CHECK(o_part.has_value() && ml_part.has_value(), "latent_decode_v: partials");
      f32c(*o_part, T * heads * n_splits * L, "o_part");
      f32c(*ml_part, T * heads * n_splits * 2, "ml_part");
      a.o_part = o_part->data_ptr<float>(); a.ml_part = ml_part->data_ptr<float>();
    } else {
      TORCH_CHECK(o_lat.has_value() && !is_f32(*o_lat, "o_lat") && o_lat->is_contiguous() && o_lat->numel() == T * heads * L,
                  "latent_decode_v: o_lat [T, heads, rank]");
      a.o_lat = o_lat->data_ptr();
    }
    a.uv = uv.data_ptr();
    if (gate.has_value()) {
      TORCH_CHECK(!is_f32(*gate, "gate") && gate->dim() == 2 && gate->size(0) == T && (gate->size(1) == heads * V || gate->size(1) == heads),
                  "latent_decode_v: one gate per column or per head");
      a.gate = gate->data_ptr(); a.ldg = gate->stride(0); a.per_head = gate->size(1) != heads * V;
    }
    a.out = out.data_ptr(); a.T = int(T); a.heads = int(heads); a.L = int(L); a.V = int(V);
    c10::cuda::CUDAGuard guard(out.device());
    TORCH_CHECK(lb::latent_decode_v_launch(a, cur_stream()) == 0, "latent_decode_v failed", cuda_error());
  });
  m.def("latent_attn_general", [](const Tensor& q_abs, const Tensor& cache, const Tensor& cu_q, const Tensor& ctx_lens,
                                  const Tensor& block_table, double scale, int64_t rank, int64_t rot, Tensor& out) {
    const bool f32 = is_f32(q_abs, "q_abs");
    same(cache, f32, "cache");
    same(out, f32, "out");
    const int64_t T = q_abs.size(0), H = q_abs.size(1), cell = cache.size(-1);
    TORCH_CHECK(q_abs.dim() == 3 && q_abs.is_contiguous() && cache.is_contiguous() && cache.dim() == 4 && cell >= rank + rot &&
                    q_abs.size(2) >= rank + rot && out.is_contiguous() && out.numel() == T * H * rank,
                "latent_attn_general: rows of rank + rot columns");
    TORCH_CHECK(cu_q.scalar_type() == at::kInt && ctx_lens.scalar_type() == at::kInt && block_table.scalar_type() == at::kInt &&
                    block_table.stride(1) == 1 && cu_q.numel() == ctx_lens.numel() + 1, "latent_attn_general: int32 tables");
    c10::cuda::CUDAGuard guard(q_abs.device());
    TORCH_CHECK(lb::paged_attn_general_launch(q_abs.data_ptr(), q_abs.size(2), cache.data_ptr(), cache.data_ptr(), cell, cell,
                                              cu_q.data_ptr<int>(), ctx_lens.data_ptr<int>(), block_table.data_ptr<int>(),
                                              int(block_table.stride(0)), int(cache.size(1)), int(ctx_lens.numel()), int(T),
                                              int(H), 1, int(rank + rot), int(rank), float(scale), 0.f, 0, out.data_ptr(), f32,
                                              cur_stream()) == 0,
                "latent_attn_general: latents of at most 1024 columns", cuda_error());
  });
  m.def("latent_gate", [](Tensor& x, const Tensor& gate, int64_t heads) {
    const bool f32 = is_f32(x, "x");
    same(gate, f32, "gate");
    const int64_t T = x.size(0), N = x.size(1);
    TORCH_CHECK(x.dim() == 2 && x.is_contiguous() && gate.dim() == 2 && gate.size(0) == T && N % heads == 0 &&
                    (gate.size(1) == N || gate.size(1) == heads), "latent_gate: one gate per column or per head");
    c10::cuda::CUDAGuard guard(x.device());
    TORCH_CHECK(lb::latent_gate_launch(x.data_ptr(), gate.data_ptr(), gate.stride(0), gate.size(1) != N, int(N / heads), int(N),
                                       int(T), f32, cur_stream()) == 0, "latent_gate failed", cuda_error());
  });
  m.def("diag_scan", [](const Tensor& u, Tensor& gates, const Tensor& gates_b, const Tensor& log_decay, const Tensor& y,
                        const Tensor& y_b, Tensor& state, const Tensor& cu, const Tensor& slots, int64_t blocks, Tensor& out,
                        bool write_state, int64_t max_tokens, const OptT& tables, int64_t n_chunks, const OptT& ends) {
    const bool f32 = is_f32(u, "u");
    lb::DiagScanArgs a = diag_args(u.size(0), u.size(1), gates_b, log_decay, y, y_b, state, cu, slots, blocks, out, f32);
    f32c(gates, u.size(0) * 2 * u.size(1), "gates");
    a.u = u.data_ptr(); a.ldu = u.stride(0); a.gates = gates.data_ptr<float>();
    a.write_state = write_state; a.max_tokens = int(max_tokens);
    c10::cuda::CUDAGuard guard(u.device());
    if (!tables.has_value()) {
      TORCH_CHECK(lb::diag_scan_launch(a, f32, cur_stream()) == 0, "diag_scan failed", cuda_error());
      return;
    }
    TORCH_CHECK(tables->scalar_type() == at::kInt && tables->is_contiguous() && tables->numel() == 3 * n_chunks + 2 * a.n_seqs &&
                    ends.has_value(), "diag_scan: chunk tables");
    f32c(*ends, n_chunks * 2 * u.size(1), "chunk ends");
    const int* t = tables->data_ptr<int>();
    TORCH_CHECK(lb::diag_chunk_launch(a, t, t + n_chunks, int(n_chunks), t + 3 * n_chunks, t + 3 * n_chunks + a.n_seqs,
                                      ends->data_ptr<float>(), f32, cur_stream()) == 0, "diag_scan failed", cuda_error());
  });
  m.def("diag_decode", [](const Tensor& x, const Tensor& in_bias, const Tensor& conv_w, const OptT& conv_b, Tensor& conv_state,
                          const Tensor& gates_w, const Tensor& gates_b, const Tensor& log_decay, const Tensor& y,
                          const Tensor& y_b, Tensor& state, const Tensor& cu, const Tensor& slots, int64_t blocks, Tensor& ctr,
                          Tensor& out) {
    const bool f32 = is_f32(x, "x");
    const int64_t n = x.size(0), W = x.size(1), K = conv_w.size(1);
    TORCH_CHECK(n == slots.numel(), "diag_decode: one token per sequence");
    lb::DiagDecodeArgs a{};
    a.s = diag_args(n, W, gates_b, log_decay, y, y_b, state, cu, slots, blocks, out, f32);
    a.s.write_state = 1;
    same(gates_w, f32, "gate weights");
    TORCH_CHECK(gates_w.is_contiguous() && gates_w.numel() == 2 * W * (W / blocks), "diag_decode: gate weights [blocks, 2, d, d]");
    f32c(conv_w, W * K, "conv weight");
    f32c(in_bias, W, "input bias");
    if (conv_b.has_value()) f32c(*conv_b, W, "conv bias");
    TORCH_CHECK(conv_state.scalar_type() == at::kFloat && conv_state.is_contiguous() && conv_state.dim() == 3 &&
                    conv_state.size(1) == W && conv_state.size(2) == K - 1, "diag_decode: history [slots, W, taps - 1]");
    TORCH_CHECK(ctr.scalar_type() == at::kInt && ctr.is_contiguous() &&
                    ctr.numel() >= (n + lb::DIAG_DECODE_SEQ - 1) / lb::DIAG_DECODE_SEQ * blocks, "diag_decode: counters");
    a.x = x.data_ptr(); a.ldx = x.stride(0); a.in_bias = in_bias.data_ptr<float>();
    a.conv_w = conv_w.data_ptr<float>(); a.conv_b = optp<float>(conv_b); a.conv_state = conv_state.data_ptr<float>();
    a.KC = int(K); a.gates_w = gates_w.data_ptr();
    a.ctr = reinterpret_cast<unsigned int*>(ctr.data_ptr());
    c10::cuda::CUDAGuard guard(x.device());
    TORCH_CHECK(lb::diag_decode_launch(a, f32, cur_stream()) == 0, "diag_decode failed", cuda_error());
  });
  m.def("softcap", [](Tensor& x, double scale, double cap) {
    f32c(x, 0, "logits");
    c10::cuda::CUDAGuard guard(x.device());
    TORCH_CHECK(lb::softcap_launch(x.data_ptr<float>(), float(scale), float(cap), x.numel(), cur_stream()) == 0, "softcap failed",
                cuda_error());
  });
}
