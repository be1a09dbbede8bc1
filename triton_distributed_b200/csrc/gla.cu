// Gated linear attention with a decay per key channel.  Per head, with the state S [dk x dv] in fp32:
//     S   <- diag(alpha_t) S + k_t v_t^T          alpha_t = sigmoid(z_t)^(1/tau), z_t = A2 a_t + b   (a_t = A1 x_t)
//     o_t  = q_scale S^T q_t
//     y_t  = RMSNorm(o_t) * w * silu(g_t)
//
//   gla_decode_kernel     one token per sequence: decay, state update, output, norm and gate in one launch; the state is
//                         read and written once with 16-byte accesses (what the step is bound by)
//   gla_log_decay_kernel  log alpha of every token and channel, for the recurrent form
//   gla_recurrent_kernel  token by token with the state in registers (a CTA owns 32 columns of one head of one sequence;
//                         every column is shared by four lanes): the 32-bit path
//   gla_norm_gate_kernel  norm and gate of its outputs
// The chunk-parallel form for bf16 prefill is in gla_chunk.cu.  A sequence whose call starts at position 0 starts from a
// zero state whatever its state row holds, so rows can be handed to a new sequence without clearing.
#include "tdb/gla.cuh"
#include "tdb/hybrid.h"
#include "tdb/launch.cuh"
#include "tdb/vec.cuh"

namespace tdb {

namespace {

constexpr int kDecodeThreads = 512;
constexpr int kMaxParts = 16;

template <typename T>
__global__ void __launch_bounds__(kDecodeThreads, 1) gla_decode_kernel(const GlaArgs p) {
  extern __shared__ __align__(16) float sm[];
  __shared__ float red[32];
  float* s_q = sm;                 // [dk]
  float* s_k = s_q + p.dk;         // [dk]
  float* s_d = s_k + p.dk;         // [dk] decay
  float* s_v = s_d + p.dk;         // [dv]
  float* s_o = s_v + p.dv;         // [row groups][dv]
  float* s_z = s_o;                // [parts][dk], before s_o is used
  const int h = blockIdx.x, n = blockIdx.y;
  pdl_wait();
  pdl_launch_dependents();
  // the state rows this thread starts with are requested first: the decays are computed while they travel
  const int dv4 = p.dv >> 2;
  const int groups = kDecodeThreads / dv4;           // rows processed side by side
  const int c4 = threadIdx.x % dv4, rg = threadIdx.x / dv4;
  const bool fresh = p.pos0[n] == 0;
  float4* S = reinterpret_cast<float4*>(p.state + ((static_cast<int64_t>(p.slots[n]) * p.H + h) * p.dk) * p.dv) + c4;
  constexpr int U = 8;
  float4 s[U];
  auto fetch = [&](int r0) {
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int r = r0 + u * groups;
      s[u] = (r < p.dk && !fresh) ? S[static_cast<int64_t>(r) * dv4] : make_float4(0.f, 0.f, 0.f, 0.f);
    }
  };
  if (rg < groups) fetch(rg);
  const T* row = reinterpret_cast<const T*>(p.qkvg) + n * p.ld;
  const int Hk = p.H * p.dk, Hv = p.H * p.dv;
  // z = a2^T a + b: the threads of a channel share the low-rank dimension, so its loads are all in flight at once
  const int parts = max(1, min(kDecodeThreads / p.dk, kMaxParts));
  for (int i = threadIdx.x; i < parts * p.dk; i += kDecodeThreads) {
    const int c = i % p.dk, part = i / p.dk;
    float z = 0.f;
#pragma unroll 4
    for (int r = part; r < p.R; r += parts)
      z = fmaf(p.a2[static_cast<int64_t>(r) * Hk + h * p.dk + c], p.a[static_cast<int64_t>(n) * p.R + r], z);
    s_z[part * p.dk + c] = z;
  }
  for (int c = threadIdx.x; c < p.dk; c += kDecodeThreads) {
    s_q[c] = to_f32(row[h * p.dk + c]) * p.q_scale;
    s_k[c] = to_f32(row[Hk + h * p.dk + c]);
  }
  for (int c = threadIdx.x; c < p.dv; c += kDecodeThreads) s_v[c] = to_f32(row[2 * Hk + h * p.dv + c]);
  __syncthreads();
  for (int c = threadIdx.x; c < p.dk; c += kDecodeThreads) {
    float z = p.a2_b[h * p.dk + c];
    for (int i = 0; i < parts; ++i) z += s_z[i * p.dk + c];
    s_d[c] = expf(gla_log_decay(z, p.inv_tau));
  }
  __syncthreads();
  float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
  if (rg < groups) {
    const float4 v = reinterpret_cast<const float4*>(s_v)[c4];
    for (int r0 = rg; r0 < p.dk; r0 += groups * U) {
      if (r0 != rg) fetch(r0);
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int r = r0 + u * groups;
        if (r < p.dk) {
          const float d = s_d[r], k = s_k[r], q = s_q[r];
          s[u].x = fmaf(d, s[u].x, k * v.x); s[u].y = fmaf(d, s[u].y, k * v.y);
          s[u].z = fmaf(d, s[u].z, k * v.z); s[u].w = fmaf(d, s[u].w, k * v.w);
          o.x = fmaf(q, s[u].x, o.x); o.y = fmaf(q, s[u].y, o.y);
          o.z = fmaf(q, s[u].z, o.z); o.w = fmaf(q, s[u].w, o.w);
          S[static_cast<int64_t>(r) * dv4] = s[u];
        }
      }
    }
    reinterpret_cast<float4*>(s_o + rg * p.dv)[c4] = o;
  }
  __syncthreads();
  float ss = 0.f;
  for (int c = threadIdx.x; c < p.dv; c += kDecodeThreads) {
    float t = 0.f;
    for (int i = 0; i < groups; ++i) t += s_o[i * p.dv + c];
    s_v[c] = t;
    ss += t * t;
  }
  const float inv = 1.f / sqrtf(block_reduce_sum(ss, red) / p.dv_real + p.eps);
  T* out = reinterpret_cast<T*>(p.out) + static_cast<int64_t>(n) * Hv + h * p.dv;
  for (int c = threadIdx.x; c < p.dv; c += kDecodeThreads) {
    const float g = to_f32(row[2 * Hk + Hv + h * p.dv + c]);
    out[c] = from_f32<T>(s_v[c] * inv * p.norm_w[c] * g * sigmoid_f32(g));
  }
}

constexpr int kDecayTok = 16;
__global__ void __launch_bounds__(256) gla_log_decay_kernel(const GlaArgs p) {
  extern __shared__ float s_a[];       // [kDecayTok][R]
  pdl_wait();
  pdl_launch_dependents();
  const int64_t t0 = static_cast<int64_t>(blockIdx.y) * kDecayTok;
  const int nt = static_cast<int>(min(static_cast<int64_t>(kDecayTok), p.T - t0));
  for (int i = threadIdx.x; i < nt * p.R; i += 256) s_a[i] = p.a[t0 * p.R + i];
  __syncthreads();
  const int C = p.H * p.dk, c = blockIdx.x * 256 + threadIdx.x;
  if (c >= C) return;
  float z[kDecayTok];
  const float b = p.a2_b[c];
#pragma unroll
  for (int i = 0; i < kDecayTok; ++i) z[i] = b;
  for (int r = 0; r < p.R; ++r) {
    const float w = p.a2[static_cast<int64_t>(r) * C + c];
#pragma unroll
    for (int i = 0; i < kDecayTok; ++i)
      if (i < nt) z[i] = fmaf(w, s_a[i * p.R + r], z[i]);
  }
#pragma unroll
  for (int i = 0; i < kDecayTok; ++i)
    if (i < nt) p.log_decay[(t0 + i) * C + c] = gla_log_decay(z[i], p.inv_tau);
}

constexpr int kRecTok = 16;      // tokens staged at a time
constexpr int kRecCols = 32;     // columns of dv per CTA
template <typename T, int KP>    // KP rows of dk per lane, dk <= 4 KP
__global__ void __launch_bounds__(4 * kRecCols) gla_recurrent_kernel(const GlaArgs p) {
  extern __shared__ __align__(16) float sm[];
  constexpr int kDkp = 4 * KP;
  float* s_q = sm;                          // [kRecTok][kDkp]
  float* s_k = s_q + kRecTok * kDkp;
  float* s_d = s_k + kRecTok * kDkp;
  float* s_v = s_d + kRecTok * kDkp;        // [kRecTok][kRecCols]
  const int v0 = blockIdx.x * kRecCols, h = blockIdx.y, n = blockIdx.z;
  const int col = threadIdx.x >> 2, part = threadIdx.x & 3;
  pdl_wait();
  pdl_launch_dependents();
  const int64_t tb = p.cu != nullptr ? p.cu[n] : n, te = p.cu != nullptr ? p.cu[n + 1] : n + 1;
  const int Hk = p.H * p.dk, Hv = p.H * p.dv;
  const bool col_ok = v0 + col < p.dv, fresh = p.pos0[n] == 0;
  float* st = p.state + ((static_cast<int64_t>(p.slots[n]) * p.H + h) * p.dk) * p.dv + v0 + col;
  float S[KP];
#pragma unroll
  for (int i = 0; i < KP; ++i) {
    const int r = part + 4 * i;
    S[i] = (!fresh && col_ok && r < p.dk) ? st[static_cast<int64_t>(r) * p.dv] : 0.f;
  }
  for (int64_t t0 = tb; t0 < te; t0 += kRecTok) {
    const int nt = static_cast<int>(min(static_cast<int64_t>(kRecTok), te - t0));
    __syncthreads();
    for (int i = threadIdx.x; i < nt * kDkp; i += 4 * kRecCols) {
      const int j = i / kDkp, c = i - j * kDkp;
      const T* row = reinterpret_cast<const T*>(p.qkvg) + (t0 + j) * p.ld;
      const bool ok = c < p.dk;
      s_q[i] = ok ? to_f32(row[h * p.dk + c]) * p.q_scale : 0.f;
      s_k[i] = ok ? to_f32(row[Hk + h * p.dk + c]) : 0.f;
      s_d[i] = ok ? expf(p.log_decay[(t0 + j) * Hk + h * p.dk + c]) : 0.f;
    }
    for (int i = threadIdx.x; i < nt * kRecCols; i += 4 * kRecCols) {
      const int j = i / kRecCols, c = i - j * kRecCols;
      s_v[i] = v0 + c < p.dv ? to_f32(reinterpret_cast<const T*>(p.qkvg)[(t0 + j) * p.ld + 2 * Hk + h * p.dv + v0 + c]) : 0.f;
    }
    __syncthreads();
    for (int j = 0; j < nt; ++j) {
      const float v = s_v[j * kRecCols + col];
      float o = 0.f;
#pragma unroll
      for (int i = 0; i < KP; ++i) {
        const int r = j * kDkp + part + 4 * i;
        S[i] = fmaf(s_d[r], S[i], s_k[r] * v);
        o = fmaf(s_q[r], S[i], o);
      }
      o += __shfl_xor_sync(0xffffffffu, o, 1);
      o += __shfl_xor_sync(0xffffffffu, o, 2);
      if (part == 0 && col_ok) p.o_raw[(t0 + j) * Hv + h * p.dv + v0 + col] = o;
    }
  }
#pragma unroll
  for (int i = 0; i < KP; ++i) {
    const int r = part + 4 * i;
    if (col_ok && r < p.dk) st[static_cast<int64_t>(r) * p.dv] = S[i];
  }
}

template <typename T>
__global__ void __launch_bounds__(128) gla_norm_gate_kernel(const GlaArgs p) {
  pdl_wait();
  pdl_launch_dependents();
  const int64_t wid = static_cast<int64_t>(blockIdx.x) * 4 + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (wid >= p.T * p.H) return;
  const int64_t t = wid / p.H;
  const int h = static_cast<int>(wid - t * p.H);
  const float* o = p.o_raw + wid * p.dv;
  float ss = 0.f;
  for (int c = lane; c < p.dv; c += 32) ss += o[c] * o[c];
  const float inv = 1.f / sqrtf(warp_sum(ss) / p.dv_real + p.eps);
  const T* gate = reinterpret_cast<const T*>(p.qkvg) + t * p.ld + 2 * p.H * p.dk + p.H * p.dv + h * p.dv;
  T* out = reinterpret_cast<T*>(p.out) + wid * p.dv;
  for (int c = lane; c < p.dv; c += 32) {
    const float g = to_f32(gate[c]);
    out[c] = from_f32<T>(o[c] * inv * p.norm_w[c] * g * sigmoid_f32(g));
  }
}

template <typename T, int KP>
cudaError_t launch_rec(const GlaArgs& a, cudaStream_t s) {
  static SmemOptIn opt;
  const int smem = (3 * kRecTok * 4 * KP + kRecTok * kRecCols) * 4;
  cudaError_t e = opt.ensure(gla_recurrent_kernel<T, KP>, smem);
  if (e != cudaSuccess) return e;
  return launch_pdl(gla_recurrent_kernel<T, KP>, dim3((a.dv + kRecCols - 1) / kRecCols, a.H, a.N), dim3(4 * kRecCols),
                    static_cast<size_t>(smem), s, a);
}
template <typename T>
cudaError_t launch_rec_t(const GlaArgs& a, cudaStream_t s) {
  cudaError_t e = a.dk <= 32    ? launch_rec<T, 8>(a, s)
                  : a.dk <= 64  ? launch_rec<T, 16>(a, s)
                  : a.dk <= 128 ? launch_rec<T, 32>(a, s)
                  : a.dk <= 256 ? launch_rec<T, 64>(a, s)
                                : launch_rec<T, 128>(a, s);
  if (e != cudaSuccess) return e;
  return launch_pdl(gla_norm_gate_kernel<T>, dim3(static_cast<unsigned>((a.T * a.H + 3) / 4)), dim3(128), 0, s, a);
}

bool args_ok(const GlaArgs& a) {
  return a.N >= 0 && a.H >= 1 && a.dk >= 1 && a.dk <= 512 && a.dv >= 4 && a.dv % 4 == 0 && a.dv <= 1024 && a.dv_real >= 1 &&
         a.R >= 1 && a.R <= 512;
}

cudaError_t launch_gla_log_decay(const GlaArgs& a, cudaStream_t s) {
  const int64_t tiles = (a.T + kDecayTok - 1) / kDecayTok;
  if (tiles > 65535) return cudaErrorInvalidValue;
  return launch_pdl(gla_log_decay_kernel, dim3((a.H * a.dk + 255) / 256, static_cast<unsigned>(tiles)), dim3(256),
                    static_cast<size_t>(kDecayTok * a.R * 4), s, a);
}

}  // namespace

cudaError_t launch_gla_decode(const GlaArgs& a, cudaStream_t s) {
  if (!args_ok(a)) return cudaErrorInvalidValue;
  if (a.N == 0) return cudaSuccess;
  const int groups = kDecodeThreads / (a.dv / 4);
  const int tail = groups * a.dv > kDecodeThreads + a.dk ? groups * a.dv : kDecodeThreads + a.dk;   // s_o, or s_z before it
  const size_t smem = static_cast<size_t>(3 * a.dk + a.dv + tail) * 4;
  const dim3 grid(a.H, a.N), block(kDecodeThreads);
  return a.is_f32 ? launch_pdl(gla_decode_kernel<float>, grid, block, smem, s, a)
                  : launch_pdl(gla_decode_kernel<__nv_bfloat16>, grid, block, smem, s, a);
}

cudaError_t launch_gla_recurrent(const GlaArgs& a, cudaStream_t s) {
  if (!args_ok(a) || a.log_decay == nullptr || a.o_raw == nullptr) return cudaErrorInvalidValue;
  if (a.T == 0 || a.N == 0) return cudaSuccess;
  cudaError_t e = launch_gla_log_decay(a, s);
  if (e != cudaSuccess) return e;
  return a.is_f32 ? launch_rec_t<float>(a, s) : launch_rec_t<__nv_bfloat16>(a, s);
}

}  // namespace tdb
