// Host API of the kernels around sublayers with several residual streams, and of per-head query / key preparation with rotation
// (streams.cu, rotary.cu).
#pragma once
#include <cuda_runtime.h>
#include <stdint.h>

namespace tdb {

// One pass over the streams between two sublayers: what the last sublayer adds, and the normed input of the next.
//     x_t <- sum_s mix[s, t] x_s + out[t] y          (ids: x_t <- table[id] instead, y null: unchanged)
//     h    = RMSNorm(sum_t in[t] x_t) * w
// The output of a sublayer of two branches is y = (RMSNorm(y) y_w + RMSNorm(y2) y2_w) / 2.
struct HyperArgs {
  float* x;               // [T, S, W] fp32
  const int64_t* ids;     // [T]
  const void* table;      // [vocab, W]
  int64_t vocab;
  const void* y;          // [T, W]
  const void* y2;         // null: y itself is the output
  const float* y_w;       // [W]
  const float* y2_w;
  const float* mix;       // [S, S], from x to
  const float* out;       // [S]
  const float* in;        // [S]
  const float* w;         // [W]
  void* h;                // [n, W]; null: streams only
  const int64_t* rows;    // [n] tokens; null = all
  int store;              // write the streams
  int64_t n;
  int64_t T;
  int S, W, n_real;       // S <= 16; W a multiple of 8, columns from n_real on are zero and do not count
  float eps;
  int is_f32;             // dtype of table, y, y2, h
};
cudaError_t launch_hyper_step(const HyperArgs& a, cudaStream_t s);

// Queries and keys of a step: RMS norm per head with a weight, rotation of the first `rot` elements, RMS norm without one; keys and
// values go to their cache rows.  D a multiple of 32, at most 1024.
struct HeadPrepArgs {
  const void* z;          // [T, ld]: q [H, D], k [G, D], v [G, D]
  int64_t ld;
  const float* q_w;       // [D] null = no norm before the rotation
  const float* k_w;
  const float* cos_sin;   // [n_pos, rot_ld]: cos, sin of pair i at columns 2i, 2i + 1
  int64_t n_pos;
  int rot, rot_ld;
  int interleaved;        // pair i is (2i, 2i + 1), else (i, i + rot / 2)
  int unit;               // norm after the rotation
  const int64_t* pos;     // [T]
  void* q_out;            // [T, H, D]
  void* k_cache;          // [cap, G, D]
  void* v_cache;
  const int64_t* rows;    // [T], rows outside [0, cap) are not written
  int64_t cap;
  int64_t T;
  int H, G, D, d_real;    // d_real: divisor of the norms
  float eps;
  int is_f32;
};
cudaError_t launch_head_prep(const HeadPrepArgs& a, cudaStream_t s);

// out = act(gate) * up for rows [gate | up] of 2 F columns.  act 0: silu, 1: gelu (tanh form).
cudaError_t launch_gated_act(const void* in, void* out, int64_t rows, int F, int act, int is_f32, cudaStream_t s);

}  // namespace tdb
