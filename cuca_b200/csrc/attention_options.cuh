// What the paged attention kernels take besides queries, pages and sizes; passed by address from Python (keep the layout
// in step with kernels/ops.py:AttentionOptions).
//
// A query at position P sees the keys j <= P with P - j < window (window 0: all of them) or j < keep (beside a window the
// first `keep` positions of a request stay visible). The score of head a is scale * (q . k), with softcap c > 0 made
// c tanh(s / c), less slopes[a] * (P - j). The softmax's denominator holds one more term with `sink`: exp(0), or
// exp(sink_val[a]), neither scaled nor capped. With `key_scale` the values are the keys: the pool's rows hold both, a score's
// q . k is multiplied by the key row's own factor before anything else, and the value is the row as it is. With `gate` the result is multiplied by sigmoid(gate[row, a dv + i]).
#pragma once

struct CucaAttnOptions {
  float scale;
  int window;
  int keep;
  float softcap;
  int sink;
  int gate_stride;        // values between rows of `gate`
  const float* sink_val;  // [nh] or null
  const float* slopes;    // [nh] or null: no distance bias
  const void* gate;       // rows of the output's type, or null
  float* key_scale;       // [pages][key heads][positions of a page] or null (written only by kernels that store keys)
};

#define CUCA_LOG2E 1.4426950408889634f
