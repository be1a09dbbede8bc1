// Host API of attention over a sliding window (window_attn.cu, window_attn_sm100.cu) and of the preparation of its queries, keys and
// values (qkv_prep.cu).  Position i sees the positions j with 0 <= i - j < window (window 0: every j <= i).
//
// Two kinds of weights:
//   sigmoid        w = sigmoid(scale q.k + bias[head][i - j]), not normalised over the keys
//   differential   two maps of scores over the same values, a softmax each: o = a1 - lambda a2, o <- RMSNorm(o) * out_scale
// and an output gate with one number per head, o <- o * sigmoid(gate), where given.
//
// Queries [T, H maps, dk], keys [rows, G maps, dk], values [rows, G, dv]; head h uses key head h / (H / G); the maps of a head lie side
// by side.  A sequence keeps the last min(window, max_length) tokens in a ring, position p at row p % R of its slot.  A decode step
// reads the ring.  A prompt reads a packed copy: what the ring held of earlier steps and the new tokens, sequence after sequence.
#pragma once
#include <cuda_runtime.h>
#include <stdint.h>

namespace tdb {

struct WindowAttnArgs {
  const void* q;
  const void* k;
  const void* v;
  void* out;                 // [T, H, dv]
  int64_t T;
  int64_t rows;              // rows of k and v
  int H, G, maps, dk, dv;
  float scale;
  int is_f32;
  const float* bias;         // sigmoid form: fp32 [H, bias_n], added to the score at that distance; null = differential (maps = 2)
  int64_t bias_n;
  float lambda;              // differential form
  float out_scale, eps;
  int dv_real;               // divisor of its norm
  const void* gate;          // [T, ld_gate], logit of head h in column h; null = no gate
  int64_t ld_gate;
  // simple form: token t sees the rows row0[t] .. + n_keys[t]; row0 + newest holds the token itself, rows after it are the oldest
  const int64_t* row0;
  const int32_t* n_keys;
  const int32_t* newest;
  // decode form: token t at position pos[t] of the sequence in slots[t], ring rows a slot
  const int32_t* slots;
  const int64_t* pos;
  int ring;
  int splits;
  float* workspace;          // window_decode_workspace(...) floats when splits > 1
  uint32_t* counters;        // [T * G * head chunks] zero, left zero
  // prompt form: position p of sequence b at packed row p + shift[b]
  const int32_t* cu;         // [N + 1]
  const int32_t* q_pos0;     // [N]
  const int32_t* shift;      // [N]
  int N, max_q, window;
  int* error_flag;           // set when a bounded wait gave up
};
cudaError_t launch_window_simple(const WindowAttnArgs& a, cudaStream_t s);    // fp32 arithmetic, dk and dv up to 1024
cudaError_t launch_window_decode(const WindowAttnArgs& a, cudaStream_t s);    // bf16, dk and dv 64 or 128
cudaError_t launch_window_prompt(const WindowAttnArgs& a, cudaStream_t s);    // bf16, dk and dv 64 or 128, scale > 0
int window_head_chunks(int H, int G, int maps);                               // of one key head, in the decode form
int64_t window_decode_workspace(int64_t T, int G, int chunks, int splits, int dv);

// Projected q | k | v of a step: biases, an RMS norm over the whole of q and of k with weights, rotation of the first `rot` elements
// of every head of q and k (element i with i + rot / 2); keys and values go to up to two places.
struct QkvPrepArgs {
  const void* z;             // [T, ld]: q [Hq, dk], k [Gk, dk], v [G, dv]
  int64_t ld;
  const float* bias;         // [Hq dk + Gk dk + G dv] null = none
  const float* q_w;          // [Hq dk] null = no norm
  const float* k_w;          // [Gk dk]
  int nq_real, nk_real;      // divisors of the means
  const float* sumsq;        // [T, 2] sums of squares of q and k over all ranks; null: taken here
  float eps;
  const float* cos_sin;      // [n_pos, rot_ld]: cos, sin of pair i at columns 2i, 2i + 1
  int64_t n_pos;
  int rot, rot_ld;
  const int64_t* pos;        // [T]
  void* q_out;               // [T, Hq, dk]
  void* k_a;                 // [cap_a, Gk, dk]; rows outside [0, cap) are not written
  void* v_a;                 // [cap_a, G, dv]
  const int64_t* rows_a;
  int64_t cap_a;
  void* k_b;                 // second place, null = none
  void* v_b;
  const int64_t* rows_b;
  int64_t cap_b;
  int64_t T;
  int Hq, Gk, G, dk, dv;     // dk and dv multiples of 8
  int is_f32;
};
cudaError_t launch_qkv_prep(const QkvPrepArgs& a, cudaStream_t s);

}  // namespace tdb
