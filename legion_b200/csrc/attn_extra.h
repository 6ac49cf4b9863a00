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

}  // namespace lb
