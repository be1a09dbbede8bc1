// Host API of the kernels that layered ("hybrid") decoders add: an fp32 residual stream with norms on the sublayers'
// outputs or on the stream itself (parallel layers), whole-projection q / k norms over a tied KV cache, routers, pair-wise
// expert GEMV, gated linear attention.  `is_f32` selects fp32 activations / weights, else bf16; everything that says fp32 is fp32 in both.
#pragma once
#include <cuda_runtime.h>
#include <stdint.h>

namespace tdb {

// ---- residual stream (stream_ops.cu); W a multiple of 8, columns >= n_real are zero and do not count in the norms
// x[t] = scale * table[ids[t]] in fp32, and its bf16 copy xb (null = none).
cudaError_t launch_embed_stream(const int64_t* ids, const void* table, float* x, void* xb, int64_t T, int W, int64_t vocab,
                                float scale, int is_f32, cudaStream_t s);
struct PostNormArgs {
  float* x;               // [T, W] residual stream, updated in place: x += rmsnorm(y) * w
  void* xb;               // [T, W] bf16 copy of the new x, null = none
  const void* y;          // [T * rows_per_token, W]: the rows of a token are summed first
  int y_f32;              // dtype of y and shared
  int rows_per_token;
  const void* shared;     // [T, W] added to the sum, times shared_gate[t]; null = none
  const float* shared_gate;
  const float* w;         // [W] fp32
  int64_t T;
  int W, n_real;
  float eps;
};
cudaError_t launch_postnorm_add(const PostNormArgs& a, cudaStream_t s);
// out[t] = sum of the token's rows + gate * shared, without norm (what tensor-parallel ranks exchange).
cudaError_t launch_combine_rows(const PostNormArgs& a, void* out, cudaStream_t s);
// out[i] = rmsnorm(x[rows[i]]) * w (rows null: identity), fp32 or bf16 output.
// Parallel layers, x += mixer + feed-forward, and the two norms of the new x that the next layer reads.
struct ParallelAddArgs {
  float* x;               // [T, W]
  const void* mix;        // [T, W] activation dtype, null = none
  const void* y;          // [T * rows, W]: rows of a token are summed; null = none
  int y_f32, rows;
  const int32_t* ids;     // [T, rows] experts of the rows (null = all rows count): a row with an id outside [0, experts) is
  const float* weights;   // not read, weights * hin stands in for it
  int experts;
  const void* hin;        // [T, W] activation dtype
  const void* shared;     // [T, W] activation dtype, null = none
  const float* bias;      // [W] fp32, null = none
  float* sum_out;         // non-null: the sum goes there and nothing else happens (what tensor-parallel ranks exchange)
  const float* w1;        // [W] fp32: h1 = rmsnorm(x) * w1 ...
  void* h1;               // activation dtype; null = no norm
  const float* w2;        // ... and h2 (null = one norm only)
  void* h2;
  int act_f32;
  int64_t T;
  int W, n_real;
  float eps;
};
cudaError_t launch_parallel_add(const ParallelAddArgs& a, cudaStream_t s);
// A sublayer between two norms: x += rmsnorm(y) * post, then h = rmsnorm(x) * pre, the input of the next one.
struct SandwichArgs {
  float* x;               // [T, W]
  const int64_t* ids;     // [T] start: x = scale * table[id] instead of reading it; null = x as it is
  const void* table;      // [vocab, W]
  int64_t vocab;
  float scale;
  const void* y;          // [T, W], null = nothing is added
  const float* post;      // [post_n]; one number for all coordinates (post_n = 1) or one each (post_n = W)
  int post_n;
  const float* pre;
  int pre_n;
  void* h;                // [n, W], null = stream only
  const int64_t* rows;    // [n] tokens, null = all
  int store;              // write x
  int64_t n;
  int W, n_real;          // W a multiple of 8, columns from n_real on are zero and do not count
  float eps;
  int is_f32;             // dtype of table, y, h
};
cudaError_t launch_sandwich(const SandwichArgs& a, cudaStream_t s);
cudaError_t launch_stream_norm(const float* x, const int64_t* rows, const float* w, void* out, int64_t n, int W, int n_real,
                               float eps, int out_f32, cudaStream_t s);

// ---- q / k norm over whole projections + tied cache write (tied_kv.cu)
struct QkNormArgs {
  const void* qk;         // [T, ld]: q in columns [0, Nq), k in [Nq, Nq + Nk)
  int64_t ld;
  const float* qw;        // [Nq] fp32: everything that multiplies the normed q (its weight, the key norm's weight, scale)
  void* q_out;            // [T, Nq]
  void* k_a;              // raw k row of token t goes to row rows_a[t] of k_a / scale_a ...
  float* scale_a;
  const int64_t* rows_a;
  int64_t cap_a;          // rows of k_a; rows outside [0, cap) are not written
  void* k_b;              // ... and to row rows_b[t] of k_b / scale_b (null = no second destination)
  float* scale_b;
  const int64_t* rows_b;
  int64_t cap_b;
  const float* sumsq;     // [T, 2] sums of squares of q and k over all ranks; null: taken here
  int64_t T;
  int Nq, Nk;             // columns held here (multiples of 8)
  int nq_real, nk_real;   // divisors of the means
  float eps;
  int is_f32;
};
cudaError_t launch_qk_norm_tied(const QkNormArgs& a, cudaStream_t s);
cudaError_t launch_qk_sumsq(const QkNormArgs& a, float* out, cudaStream_t s);

// ---- narrow linear layers with fp32 outputs (router.cu)
struct NarrowLinearArgs {
  const void* x;          // [T, K]
  int64_t ldx;
  const void* w;          // [N, K]
  float* out;             // [T, N]
  int64_t T;
  int N, K;
  int is_f32;
  // router mode (top >= 1): columns [0, E) are expert logits, column E (when has_gate) the shared expert's gate
  int top, E, has_gate;
  int32_t* ids;           // [T, top]
  float* weights;         // [T, top] sigmoid scores of the chosen experts
  float* gate;            // [T] sigmoid of the gate logit
  // scores: independent sigmoids, or a softmax over the E logits; the choice is by score + correction[e] (null = 0), only
  // inside the `keep` best of `groups` equal groups of neighbours (a group counts as its best choice score; 0 = no groups).
  // The weights are the scores without the correction.
  int softmax;
  const float* correction;
  int groups, keep;
  uint32_t* counters;     // one per 16 tokens, zero; left zero
};
cudaError_t launch_narrow_linear(const NarrowLinearArgs& a, cudaStream_t s);

// ---- experts (moe_gemv.cu): y = W_down relu(W_up (w h))^2, or gated y = w W_down (silu(W_gate h) * (W_up h))
// in place or to out: out = (relu(w[row] * in + bias))^2; weight null = 1, bias null = 0
cudaError_t launch_relu2(const void* in, const float* row_weight, const float* bias, void* out, int64_t rows, int F, int is_f32,
                         cudaStream_t s);
struct ExpertGemvArgs {
  const void* x;          // [T, K]
  int gated;              // up then holds [E, 2 F, K]: gate rows before up rows (shared_up likewise)
  const void* up;         // [E, F, K]
  const void* down;       // [E, K, F]
  const int32_t* ids;     // [T, top]
  const float* weights;   // [T, top]: multiplies the expert's input (gated: its output)
  int identity;           // ids E .. E + identity - 1 are experts whose output is x itself (gated form) ...
  int skip_identity;      // ... and that another rank adds
  const void* shared_up;  // [Fs, K] or null
  const void* shared_down;  // [K, Fs]
  const float* shared_gate; // [T]
  void* act;              // scratch [T, top * F + Fs]
  float* y;               // [T, K] fp32
  int64_t T;
  int K, F, Fs, top, E;
  int is_f32;
};
cudaError_t launch_expert_gemv(const ExpertGemvArgs& a, cudaStream_t s);

// ---- gated linear attention (gla.cu, gla_chunk.cu)
struct GlaArgs {
  const void* qkvg;       // [T, ld]: q [H, dk], k [H, dk], v [H, dv], output gate [H, dv]
  int64_t ld;
  const float* a;         // [T, R] fp32 low-rank decay input
  int R;
  const float* a2;        // [R, H * dk] fp32
  const float* a2_b;      // [H * dk] fp32
  float inv_tau;          // log decay = logsigmoid(z) * inv_tau
  const float* norm_w;    // [dv] fp32
  float* state;           // [slots, H, dk, dv] fp32
  const int32_t* slots;   // [N] state row of every sequence
  const int64_t* pos0;    // [N] position of the sequence's first token of this call: 0 = the state starts at zero
  const int32_t* cu;      // [N + 1] token ranges (null: token n is sequence n)
  void* out;              // [T, H * dv]
  float* log_decay;       // scratch [T, H, dk] fp32 (not used by the decode form)
  float* o_raw;           // scratch [T, H, dv] fp32 (recurrent form only)
  int64_t T;
  int N, H, dk, dv, dv_real;
  float q_scale, eps;
  int is_f32;
  // chunk-parallel form (bf16): tables of the 64-token chunks and scratch
  const int32_t* chunk_seq;   // [NC]
  const int32_t* chunk_t0;    // [NC] first token
  const int32_t* seq_chunk0;  // [N + 1]
  int NC;
  float* chunk_state;         // [NC, H, dk, dv]
  float* chunk_decay;         // [NC, H, dk]
};
cudaError_t launch_gla_decode(const GlaArgs& a, cudaStream_t s);      // one token per sequence, everything fused
cudaError_t launch_gla_recurrent(const GlaArgs& a, cudaStream_t s);   // token by token, any lengths
cudaError_t launch_gla_chunk(const GlaArgs& a, cudaStream_t s);       // 64-token chunks in parallel, bf16
bool gla_chunk_supported(int dk, int dv);

}  // namespace tdb
