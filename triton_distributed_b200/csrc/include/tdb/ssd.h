// Host API of the state space layer in its serving form (ssd.cu, ssd_chunk.cu): short convolutions with biases, step sizes, one decay per
// head and token, recurrence with carried state, skip; and the gate with the norm over groups of its output.  Per head, with the fp32
// state S [dk, dv], input x [dv], and B, C [dk] of the head's group:
//
//     S <- exp(-exp(a_log) dt) S + dt B x^T;   y = S^T C + D x;   dt = softplus(dt_in + dt_bias)
//
// Head h uses group h / (H / G).  Sizes are padded with zeros (dk, dv multiples of 8, in the chunk form of 16).
#pragma once
#include <cuda_runtime.h>
#include <stdint.h>

namespace tdb {

struct SsdArgs {
  const void* z;             // [T, ld] projections: x [H, dv], B [G, dk], C [G, dk] from column 0, dt [H] from column dt_col
  int64_t ld;
  int dt_col;
  const float* conv_w;       // [channels, taps], channels = H dv + 2 G dk; the last column belongs to the current token
  const float* conv_b;       // [channels]
  const float* a_log;        // [H]
  const float* dt_bias;      // [H]
  const float* skip;         // [H] D
  float* state;              // [slots, H, dk, dv]
  void* conv;                // [slots, taps, channels] activation dtype: the convolutions' input of position p is at row p % taps
  const int32_t* slots;      // [N]
  const int64_t* pos0;       // [N] position of the sequence's first token of this call: what lies before position 0 is zero
  const int32_t* cu;         // [N + 1] token ranges (null: token n is sequence n)
  void* out;                 // [T, H dv] y, activation dtype
  int64_t T;
  int N, G, H, dk, dv, taps;
  int is_f32;
  // tables of the 64-token chunks (prompts)
  const int32_t* chunk_seq;  // [NC] sequence of every chunk
  const int32_t* chunk_t0;   // [NC] first token
  const int32_t* seq_chunk0; // [N + 1] first chunk of every sequence
  int NC;
  // scratch of the prompt forms
  void* xbc;                 // [T, channels] convolved inputs, activation dtype
  float* dt;                 // [T, H] step sizes
  float* log_g;              // [T, H] log decays, summed from the chunk's start
  float* inject;             // chunk form: [NC, H, dk, dv] what a chunk adds to the state, then the state before it, see ssd_chunk.cu
};
cudaError_t launch_ssd_decode(const SsdArgs& a, cudaStream_t s);      // one token per sequence, everything in one launch
cudaError_t launch_ssd_recurrent(const SsdArgs& a, cudaStream_t s);   // prompts token by token
cudaError_t launch_ssd_chunk(const SsdArgs& a, cudaStream_t s);       // prompts in 64-token chunks (bf16)
bool ssd_chunk_supported(int dk, int dv);
// Pieces of the prompt forms: convolutions, step sizes and decays of all tokens; the convolution inputs that are kept.
cudaError_t launch_ssd_prepare(const SsdArgs& a, cudaStream_t s);
cudaError_t launch_ssd_keep(const SsdArgs& a, cudaStream_t s);

// out = RMSNorm of every part of y * silu(gate), times w.  The H dv_real real elements of a row are cut into `parts` equal parts; a head
// takes dv columns in memory.
struct GatedNormArgs {
  const void* y;             // [T, H dv]
  const void* gate;          // [T, ld_gate]
  int64_t ld_gate;
  const float* w;            // [H dv]
  void* out;                 // [T, H dv]
  int64_t T;
  int H, dv, dv_real, parts;
  float eps;
  int is_f32;
};
cudaError_t launch_gated_norm(const GatedNormArgs& a, cudaStream_t s);

}  // namespace tdb
