// Optional parts of the paged attention kernels beside scale, window and soft cap.
#pragma once

namespace lb {

struct AttnExtra {
  int on = 0;                      // 0: none of it
  const float* sink = nullptr;     // [Hq] natural-log units: exp(sink) joins the softmax's denominator, without key or value
  int keep = 0;                    // first tokens of the sequence that a window leaves visible
  const void* gate = nullptr;      // [T, Hq], activation type: the head's output times sigmoid(gate)
  long ld_gate = 0;
  float out_scale = 1.f;           // factor of the output
  long ldo = 0;                    // elements between output rows
};

// Modes of the tensor-core attention kernels; only ATTN_EXT carries the optional parts among its arguments.
enum : int { ATTN_PLAIN = 0, ATTN_CAP = 1, ATTN_EXT = 2 };
template <int MODE>
struct AttnExtraArg {};
template <>
struct AttnExtraArg<ATTN_EXT> : AttnExtra {
  AttnExtraArg() = default;
  explicit AttnExtraArg(const AttnExtra& x) : AttnExtra(x) {}
};

}  // namespace lb
