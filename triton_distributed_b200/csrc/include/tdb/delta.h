// Host API of the serving form of the gated delta rule (delta.cu, delta_chunk.cu): short convolutions, unit norms, decay, recurrence
// with carried state, head norm and output gate.  Per value head, with the fp32 state S [dk, dv] and k, q of unit length:
//
//     S <- g S;   u = beta (v - S^T k);   S <- S + k u^T;   o = S^T q;   y = RMSNorm(o) * w * silu(gate)
//
// Value head h uses key head h / (H / G).  Sizes are padded with zeros (dk, dv multiples of 16).
#pragma once
#include <cuda_runtime.h>
#include <stdint.h>

namespace tdb {

struct DeltaArgs {
  const void* z;             // [T, ld] projections: q [G, dk], k [G, dk], v [H, dv], output gate [H, dv]
  int64_t ld;
  const float* ab;           // [T, 2 H]: decay input a, then step-size input b
  const float* conv_w;       // [C, taps], C = 2 G dk + H dv; the last column belongs to the current token
  const float* a_log;        // [H]   log decay = -exp(a_log) * softplus(a + dt_bias)
  const float* dt_bias;      // [H]
  const float* norm_w;       // [dv]
  float* state;              // [slots, H, dk, dv]
  void* conv;                // [slots, taps, C] activation dtype: the convolutions' input of position p is at row p % taps
  const int32_t* slots;      // [N]
  const int64_t* pos0;       // [N] position of the sequence's first token of this call: what lies before position 0 is zero
  const int32_t* cu;         // [N + 1] token ranges (null: token n is sequence n)
  void* out;                 // [T, H dv] activation dtype
  int64_t T;
  int N, G, H, dk, dv, taps;
  int dv_real;               // divisor of the head norm
  float q_scale, unit_eps, eps;
  int is_f32;
  // tables of the 64-token chunks (prompts)
  const int32_t* chunk_seq;  // [NC] sequence of every chunk
  const int32_t* chunk_t0;   // [NC] first token
  const int32_t* seq_chunk0; // [N + 1] first chunk of every sequence
  int NC;
  // scratch of the prompt forms: per token and head the log decay and the step size ...
  float* log_g;              // [T, H]
  float* beta;               // [T, H]
  // ... and the convolved, normed inputs: recurrent form fp32, chunk form bf16 (q and k as a high and a low part)
  void* q;                   // [T, G, dk]
  void* k;
  void* q_lo;                // chunk form only
  void* k_lo;
  void* v;                   // [T, H, dv]
  float* o_raw;              // recurrent form: [T, H, dv]
  // chunk form, see delta_chunk.cu: what a chunk does to the state and to the outputs, and the states between the chunks
  void* trans;               // [NC, H, dk, dk] bf16 pairs
  float* inject;             // [NC, H, dk, dv]
  void* read;                // [NC, H, 64, dk] bf16 pairs
  float* local;              // [NC, H, 64, dv]
  void* states;              // [NC, H, dk, dv] bf16 pairs
  float* decay;              // [NC, H]
};
cudaError_t launch_delta_decode(const DeltaArgs& a, cudaStream_t s);      // one token per sequence, everything in one launch
cudaError_t launch_delta_recurrent(const DeltaArgs& a, cudaStream_t s);   // prompts token by token
cudaError_t launch_delta_chunk(const DeltaArgs& a, cudaStream_t s);       // prompts in 64-token chunks (bf16)
bool delta_chunk_supported(int dk, int dv);
// Pieces of the prompt forms: convolutions, norms, decays and step sizes of all tokens; the convolution inputs that are kept.
cudaError_t launch_delta_prepare(const DeltaArgs& a, bool split, cudaStream_t s);
cudaError_t launch_delta_keep(const DeltaArgs& a, cudaStream_t s);

}  // namespace tdb
