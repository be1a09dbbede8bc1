// Host API of the latent-attention kernels (latent.cu, latent_sm100.cu).  A token is cached as ONE row [R + r] shared by all
// heads: the normed latent c and the rotated key part.  Head h's key is [W_uk c | rotated part] and its value W_uv c.
//
//   absorbed form   q' = [W_uk^T q_unrotated | q_rotated] scores cached rows directly, the attention output is a mixture of
//                   latents, and W_uv is applied after the softmax: one KV "head", no per-head keys or values (decoding)
//   expanded form   keys and values of the visible tokens are materialised by two GEMMs (prompts)
//
// All sizes are padded to multiples of eight (zero columns).  T is bf16 or fp32 (is_f32).
#pragma once
#include <cuda_runtime.h>
#include <stdint.h>

namespace tdb {

struct LatentPrepArgs {
  void* z;                  // [tokens, ld]: q in columns [0, H (d + r)), then (own_kv) the latent projection [R + r]
  int64_t ld;
  int64_t T;
  int H, d, r, R;
  int own_kv;               // 0: the layer uses another layer's rows and projects none
  int R_real;               // divisor of the latent's norm
  float eps;
  const float* norm_w;      // [R]
  const float* cos_sin;     // [n_pos, r]: cos, sin of pair i at columns 2i, 2i + 1
  int64_t n_pos;
  const int64_t* pos;       // [T]
  void* cache;              // rows [R + r]; row rows[t] is written (rows outside [0, cap) are not)
  const int64_t* rows;
  int64_t cap;
  void* ctx;                // second destination, null = none
  const int64_t* ctx_rows;
  int64_t ctx_cap;
  const void* uk_t;         // absorbed form: [H, R, d] = W_uk^T per head
  void* q_eff;              // absorbed form: [T, H, R + r]
  int is_f32;
};
// Expanded form: rotates the queries in place and writes the cache rows.
cudaError_t launch_latent_rotate(const LatentPrepArgs& a, cudaStream_t s);
// Absorbed form: writes q_eff and the cache rows in one launch; z is left alone.
cudaError_t launch_latent_absorb(const LatentPrepArgs& a, cudaStream_t s);

// out[t, h] = sigmoid(gate[t, h]) * W_uv[h] o[t, h] with o the merge of `splits` partials (ml null: one normed partial).
struct LatentOutArgs {
  const float* o;           // [T, H, splits, R] fp32
  const float* ml;          // [T, H, splits, 2]: reference maximum (log2 domain) and sum of every partial
  int splits;
  const void* uv;           // [H, dv, R]
  const void* gate;         // [T, ld_gate], head h at columns [h dv, (h + 1) dv)
  int64_t ld_gate;
  void* out;                // [T, H dv]
  int64_t T;
  int H, R, dv;
  int is_f32;
};
cudaError_t launch_latent_out(const LatentOutArgs& a, cudaStream_t s);

// Decoding on tcgen05: one query token per sequence over the cached rows (bf16, R <= 512, r <= 64).
struct LatentDecodeArgs {
  const void* q_eff;        // [B, H, R + r]
  const void* cache;        // [slots, max_len, R + r]
  const int32_t* slots;     // [B]
  const int32_t* kv_lens;   // [B]
  float* o;                 // [B, H, splits, R]
  float* ml;                // [B, H, splits, 2]
  int B, H, R, r, num_slots, max_len, splits;
  float scale;
  int* error_flag;
};
cudaError_t launch_latent_decode(const LatentDecodeArgs& a, cudaStream_t s);

// Prompts on tcgen05 (bf16, d <= 128, r <= 64, dv <= 128): causal, var-len.  Sequence b's visible tokens are rows
// [ctx0[b], ctx0[b] + kv_lens[b]) of k / ctx and columns of vt.
struct LatentPrefillArgs {
  const void* q;            // [T, ld_q], head h at columns [h (d + r), ...): unrotated | rotated part
  int64_t ld_q;
  const void* k;            // [L, H d] unrotated keys
  const void* ctx;          // [L, R + r]: the rotated key part is at column R
  const void* vt;           // [H dv, L] values, transposed
  const int32_t* cu;        // [B + 1] query ranges
  const int32_t* q_pos0;    // [B] position of the first query
  const int32_t* kv_lens;   // [B]
  const int32_t* ctx0;      // [B] multiples of eight
  const void* gate;         // [T, ld_gate]
  int64_t ld_gate;
  void* out;                // [T, H dv]
  int64_t T, L;
  int B, H, d, r, R, dv, max_q;
  float scale;
  int* error_flag;
};
cudaError_t launch_latent_prefill(const LatentPrefillArgs& a, cudaStream_t s);

}  // namespace tdb
