// Gated delta rule with its neighbours, serving form (tdb/delta.h states the recurrence).
//
//   delta_decode_kernel    one token per sequence: convolutions, unit norms, decay, state update, read-out, head norm and gate in
//                          one launch.  The state is read and written once: S^T k and S^T q come from the same pass, and
//                          S_new^T q = g S^T q + (k . q) u
//   delta_prepare_kernel   prompts: convolutions, activations, unit norms, decays and step sizes of all tokens
//   delta_keep_kernel      prompts: the last inputs of the convolutions go to the state
//   delta_recurrent_kernel prompts token by token with the state in registers (a CTA owns 32 columns of one head of one sequence,
//                          four lanes share a column): the 32-bit path, and sizes the chunk form does not take
//   delta_norm_gate_kernel norm and gate of its outputs
// The chunk-parallel form is in delta_chunk.cu.
//
// The inputs of the convolutions are kept in a ring of `taps` rows per sequence.  A decode step reads the `taps - 1` positions before
// its own and writes its own to the row of position p - taps, which nobody reads: the CTAs of a step need no order, and a repeated
// step writes the same values.  Nothing before position 0 is ever read, so slots are reused without clearing.
#include "tdb/delta.h"
#include "tdb/launch.cuh"
#include "tdb/vec.cuh"

namespace tdb {

namespace {

TDB_DEVICE float softplus_f32(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
TDB_DEVICE float silu_f32(float z) { return z * sigmoid_f32(z); }
TDB_DEVICE float delta_log_decay(const DeltaArgs& p, float a, int h) {
  return -expf(p.a_log[h]) * softplus_f32(a + p.dt_bias[h]);
}

// ---------------------------------------------------------------------------------------------------- decode

// Convolution of channel c at the sequence's newest token, followed by silu.
template <typename T>
TDB_DEVICE float conv_now(const DeltaArgs& p, const T* zrow, const T* ring, int64_t pos, int C, int c) {
  const float* w = p.conv_w + static_cast<int64_t>(c) * p.taps + p.taps - 1;
  float acc = w[0] * to_f32(zrow[c]);
  for (int j = 1; j < p.taps; ++j)
    if (pos - j >= 0) acc = fmaf(w[-j], to_f32(ring[((pos - j) % p.taps) * C + c]), acc);
  return silu_f32(acc);
}

// U rows of the state per thread are in flight (or held in registers, when that is all of them).
template <typename T, int THREADS, int U>
__global__ void __launch_bounds__(THREADS) delta_decode_kernel(const DeltaArgs p) {
  extern __shared__ __align__(16) float sm[];
  __shared__ float red[3][32];
  float* s_q = sm;                 // [dk]
  float* s_k = s_q + p.dk;         // [dk]
  float* s_v = s_k + p.dk;         // [dv] value, then u
  float* s_o = s_v + p.dv;         // [dv]
  float* s_p = s_o + p.dv;         // [row groups][2][dv] partial S^T k and S^T q
  const int h = blockIdx.x, n = blockIdx.y;
  pdl_wait();
  pdl_launch_dependents();
  const int dv4 = p.dv >> 2;
  const int groups = THREADS / dv4;           // rows processed side by side
  const int c4 = threadIdx.x % dv4, rg = threadIdx.x / dv4;
  const int64_t pos = p.pos0[n], slot = p.slots[n];
  const bool fresh = pos == 0;
  float4* S = reinterpret_cast<float4*>(p.state + ((slot * p.H + h) * p.dk) * p.dv) + c4;
  float4 s[U];
  auto fetch = [&](int r0) {
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int r = r0 + u * groups;
      s[u] = (r < p.dk && !fresh) ? S[static_cast<int64_t>(r) * dv4] : make_float4(0.f, 0.f, 0.f, 0.f);
    }
  };
  if (rg < groups) fetch(rg);
  // inputs, while the state travels
  const int share = p.H / p.G, g = h / share;
  const int Gk = p.G * p.dk, Hv = p.H * p.dv, C = 2 * Gk + Hv;
  const T* zrow = reinterpret_cast<const T*>(p.z) + n * p.ld;
  T* ring = reinterpret_cast<T*>(p.conv) + slot * p.taps * C;
  T* keep = ring + (pos % p.taps) * C;
  float qq = 0.f, kk = 0.f, qk = 0.f;
  for (int i = threadIdx.x; i < 2 * p.dk + p.dv; i += THREADS) {
    const bool is_v = i >= 2 * p.dk;
    const int c = is_v ? 2 * Gk + h * p.dv + i - 2 * p.dk : (i < p.dk ? g * p.dk + i : Gk + g * p.dk + i - p.dk);
    sm[i] = conv_now(p, zrow, ring, pos, C, c);
    if (is_v || h % share == 0) keep[c] = zrow[c];
  }
  __syncthreads();
  for (int i = threadIdx.x; i < p.dk; i += THREADS) {
    const float q = s_q[i], k = s_k[i];
    qq += q * q; kk += k * k; qk += q * k;
  }
  const float fq = rsqrtf(block_reduce_sum(qq, red[0]) + p.unit_eps) * p.q_scale;
  const float fk = rsqrtf(block_reduce_sum(kk, red[1]) + p.unit_eps);
  qk = block_reduce_sum(qk, red[2]) * fq * fk;
  const float decay = expf(delta_log_decay(p, p.ab[static_cast<int64_t>(n) * 2 * p.H + h], h));
  const float beta = sigmoid_f32(p.ab[static_cast<int64_t>(n) * 2 * p.H + p.H + h]);
  // S^T k and S^T q
  if (rg < groups) {
    float4 a = make_float4(0.f, 0.f, 0.f, 0.f), b = a;
    for (int r0 = rg; r0 < p.dk; r0 += groups * U) {
      if (r0 != rg) fetch(r0);
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int r = r0 + u * groups;
        if (r < p.dk) {
          const float k = s_k[r], q = s_q[r];
          a.x = fmaf(k, s[u].x, a.x); a.y = fmaf(k, s[u].y, a.y); a.z = fmaf(k, s[u].z, a.z); a.w = fmaf(k, s[u].w, a.w);
          b.x = fmaf(q, s[u].x, b.x); b.y = fmaf(q, s[u].y, b.y); b.z = fmaf(q, s[u].z, b.z); b.w = fmaf(q, s[u].w, b.w);
        }
      }
    }
    reinterpret_cast<float4*>(s_p + (2 * rg) * p.dv)[c4] = a;
    reinterpret_cast<float4*>(s_p + (2 * rg + 1) * p.dv)[c4] = b;
  }
  __syncthreads();
  float ss = 0.f;
  for (int c = threadIdx.x; c < p.dv; c += THREADS) {
    float a = 0.f, b = 0.f;
    for (int i = 0; i < groups; ++i) {
      a += s_p[(2 * i) * p.dv + c];
      b += s_p[(2 * i + 1) * p.dv + c];
    }
    const float u = beta * (s_v[c] - decay * fk * a);
    const float o = fmaf(decay * fq, b, qk * u);
    s_v[c] = u * fk;                                  // the state gets k u^T, and s_k holds k before its norm
    s_o[c] = o;
    ss += o * o;
  }
  const float inv = 1.f / sqrtf(block_reduce_sum(ss, red[0]) / p.dv_real + p.eps);
  if (rg < groups) {
    const float4 v = reinterpret_cast<const float4*>(s_v)[c4];
    const bool held = rg + groups * U >= p.dk;        // all rows of this thread are still in registers
    for (int r0 = rg; r0 < p.dk; r0 += groups * U) {
      if (!held) fetch(r0);
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int r = r0 + u * groups;
        if (r < p.dk) {
          const float k = s_k[r];
          S[static_cast<int64_t>(r) * dv4] = make_float4(fmaf(decay, s[u].x, k * v.x), fmaf(decay, s[u].y, k * v.y),
                                                         fmaf(decay, s[u].z, k * v.z), fmaf(decay, s[u].w, k * v.w));
        }
      }
    }
  }
  T* out = reinterpret_cast<T*>(p.out) + static_cast<int64_t>(n) * Hv + h * p.dv;
  for (int c = threadIdx.x; c < p.dv; c += THREADS)
    out[c] = from_f32<T>(s_o[c] * inv * p.norm_w[c] * silu_f32(to_f32(zrow[C + h * p.dv + c])));
}

// ---------------------------------------------------------------------------------------------------- inputs of prompts
constexpr int kPrepTok = 32;      // tokens per CTA
constexpr int kPrepThreads = 256;

// V = 4 or 8 neighbouring elements.
TDB_DEVICE void load_n(const __nv_bfloat16* p, float (&f)[8]) { load8(p, f); }
TDB_DEVICE void load_n(const float* p, float (&f)[8]) { load8(p, f); }
TDB_DEVICE void load_n(const __nv_bfloat16* p, float (&f)[4]) {
  const uint2 v = *reinterpret_cast<const uint2*>(p);
  const float2 a = unpack_bf16x2(v.x), b = unpack_bf16x2(v.y);
  f[0] = a.x; f[1] = a.y; f[2] = b.x; f[3] = b.y;
}
TDB_DEVICE void load_n(const float* p, float (&f)[4]) {
  const float4 v = *reinterpret_cast<const float4*>(p);
  f[0] = v.x; f[1] = v.y; f[2] = v.z; f[3] = v.w;
}
TDB_DEVICE void store_n(__nv_bfloat16* p, const float (&f)[8]) { store8(p, f); }
TDB_DEVICE void store_n(float* p, const float (&f)[8]) { store8(p, f); }
TDB_DEVICE void store_n(__nv_bfloat16* p, const float (&f)[4]) {
  *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(f[0], f[1]), pack_bf16x2(f[2], f[3]));
}
TDB_DEVICE void store_n(float* p, const float (&f)[4]) { *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]); }

template <int V>
TDB_DEVICE void store_split(__nv_bfloat16* hi, __nv_bfloat16* lo, const float (&f)[V]) {
  float l[V];
#pragma unroll
  for (int i = 0; i < V; ++i) l[i] = f[i] - __bfloat162float(__float2bfloat16(f[i]));
  store_n(hi, f);
  store_n(lo, l);
}

// P lanes (a power of two) share a unit, one head of q, k or v: V channels per lane.  TAPS > 0: convolutions of at most TAPS taps,
// weights and the last inputs in registers; 0: any number.
template <typename T, bool SPLIT, int TAPS, int V>
__global__ void __launch_bounds__(kPrepThreads) delta_prepare_kernel(const DeltaArgs p, int P) {
  pdl_wait();
  pdl_launch_dependents();
  const int per_block = kPrepThreads / P, units = 2 * p.G + p.H;
  const int unit = blockIdx.y * per_block + threadIdx.x / P, lane = threadIdx.x % P;
  const int n = p.chunk_seq[blockIdx.x];
  const int64_t c0 = p.chunk_t0[blockIdx.x], begin = p.cu[n], end = p.cu[n + 1], before = p.pos0[n] - begin;
  const int64_t t0 = c0 + blockIdx.z * kPrepTok, t1 = min(min(t0 + kPrepTok, c0 + 64), end);
  if (t0 >= t1) return;
  const int Gk = p.G * p.dk, C = 2 * Gk + p.H * p.dv;
  const bool live = unit < units;
  const int kind = unit < p.G ? 0 : unit < 2 * p.G ? 1 : 2;
  const int dim = kind == 2 ? p.dv : p.dk;
  const int head = unit - kind * p.G;
  const int d = lane * V, c = (kind == 2 ? 2 * Gk + head * p.dv : kind * Gk + head * p.dk) + d;
  const bool ok = live && d < dim;
  const T* z = reinterpret_cast<const T*>(p.z);
  const T* ring = reinterpret_cast<const T*>(p.conv) + static_cast<int64_t>(p.slots[n]) * p.taps * C;
  // input of channel group c at (packed) token t, zero before the sequence
  auto input = [&](int64_t t, float (&f)[V]) {
    const int64_t pos = before + t;
    if (t >= begin) {
      load_n(z + t * p.ld + c, f);
    } else if (pos >= 0) {
      load_n(ring + (pos % p.taps) * C + c, f);
    } else {
#pragma unroll
      for (int i = 0; i < V; ++i) f[i] = 0.f;
    }
  };
  constexpr int kWin = TAPS > 0 ? TAPS : 1;
  constexpr int kBatch = 4;           // tokens whose inputs are requested together
  float w[kWin][V], x[kWin + kBatch - 1][V];       // x[j]: input of token (first of the batch) + kBatch - 1 - j
#pragma unroll
  for (int j = 0; j < kWin + kBatch - 1; ++j)
#pragma unroll
    for (int i = 0; i < V; ++i) x[j][i] = 0.f;
  if (TAPS > 0 && ok) {
#pragma unroll
    for (int j = 0; j < kWin; ++j) {
#pragma unroll
      for (int i = 0; i < V; ++i) w[j][i] = j < p.taps ? p.conv_w[static_cast<int64_t>(c + i) * p.taps + p.taps - 1 - j] : 0.f;
      if (j + 1 < p.taps && j + 1 < kWin) input(t0 - 1 - j, x[j]);          // shifted into place below
    }
  }
  auto finish = [&](int64_t t, float (&acc)[V]) {
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < V; ++i) {
      acc[i] = __fdividef(acc[i], 1.f + __expf(-acc[i]));
      ss += ok ? acc[i] * acc[i] : 0.f;
    }
    for (int o = P >> 1; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    if (!ok || t >= t1) return;
    if (kind == 2) {
      if (SPLIT) store_n(reinterpret_cast<__nv_bfloat16*>(p.v) + (t * p.H + head) * p.dv + d, acc);
      else store_n(reinterpret_cast<float*>(p.v) + (t * p.H + head) * p.dv + d, acc);
      return;
    }
    const float f = rsqrtf(ss + p.unit_eps) * (kind == 0 ? p.q_scale : 1.f);
#pragma unroll
    for (int i = 0; i < V; ++i) acc[i] *= f;
    const int64_t at = (t * p.G + head) * p.dk + d;
    void* dst = kind == 0 ? p.q : p.k;
    if (SPLIT)
      store_split<V>(reinterpret_cast<__nv_bfloat16*>(dst) + at, reinterpret_cast<__nv_bfloat16*>(kind == 0 ? p.q_lo : p.k_lo) + at, acc);
    else
      store_n(reinterpret_cast<float*>(dst) + at, acc);
  };
  for (int64_t b = t0; b < t1; b += kBatch) {
    if constexpr (TAPS > 0) {
      if (ok) {
#pragma unroll
        for (int j = kWin - 2; j >= 0; --j)
#pragma unroll
          for (int i = 0; i < V; ++i) x[j + kBatch][i] = x[j][i];
#pragma unroll
        for (int j = 0; j < kBatch; ++j)
          if (b + j < t1) load_n(z + (b + j) * p.ld + c, x[kBatch - 1 - j]);
      }
#pragma unroll
      for (int k = 0; k < kBatch; ++k) {
        float acc[V] = {};
#pragma unroll
        for (int j = 0; j < kWin; ++j)
#pragma unroll
          for (int i = 0; i < V; ++i) acc[i] = fmaf(w[j][i], x[kBatch - 1 - k + j][i], acc[i]);
        finish(b + k, acc);
      }
    } else {
      for (int k = 0; k < kBatch; ++k) {
        float acc[V] = {};
        if (ok && b + k < t1)
          for (int j = 0; j < p.taps; ++j) {
            float f[V];
            input(b + k - j, f);
            const float* wj = p.conv_w + static_cast<int64_t>(c) * p.taps + p.taps - 1 - j;
#pragma unroll
            for (int i = 0; i < V; ++i) acc[i] = fmaf(wj[i * p.taps], f[i], acc[i]);
          }
        finish(b + k, acc);
      }
    }
  }
  if (blockIdx.y == 0)                 // decays and step sizes of these tokens
    for (int64_t i = threadIdx.x; i < (t1 - t0) * p.H; i += kPrepThreads) {
      const int64_t t = t0 + i / p.H;
      const int h = static_cast<int>(i % p.H);
      p.log_g[t * p.H + h] = delta_log_decay(p, p.ab[t * 2 * p.H + h], h);
      p.beta[t * p.H + h] = sigmoid_f32(p.ab[t * 2 * p.H + p.H + h]);
    }
}
template <typename T, bool SPLIT, int V>
cudaError_t launch_prepare_v(const DeltaArgs& a, cudaStream_t s) {
  int P = 1;
  while (P * V < a.dk || P * V < a.dv) P *= 2;
  const int per_block = kPrepThreads / P, units = 2 * a.G + a.H;
  const dim3 grid(a.NC, (units + per_block - 1) / per_block, 64 / kPrepTok), block(kPrepThreads);
  return a.taps <= 2   ? launch_pdl(delta_prepare_kernel<T, SPLIT, 2, V>, grid, block, 0, s, a, P)
         : a.taps <= 4 ? launch_pdl(delta_prepare_kernel<T, SPLIT, 4, V>, grid, block, 0, s, a, P)
                       : launch_pdl(delta_prepare_kernel<T, SPLIT, 0, V>, grid, block, 0, s, a, P);
}
template <typename T, bool SPLIT>
cudaError_t launch_prepare(const DeltaArgs& a, cudaStream_t s) {
  return a.dk <= 128 && a.dv <= 128 ? launch_prepare_v<T, SPLIT, 4>(a, s) : launch_prepare_v<T, SPLIT, 8>(a, s);
}

template <typename T>
__global__ void __launch_bounds__(256) delta_keep_kernel(const DeltaArgs p) {
  pdl_wait();
  pdl_launch_dependents();
  const int n = blockIdx.y, C = 2 * p.G * p.dk + p.H * p.dv;
  const int c = (blockIdx.x * 256 + threadIdx.x) * 8;
  if (c >= C) return;
  const int64_t begin = p.cu[n], end = p.cu[n + 1];
  T* ring = reinterpret_cast<T*>(p.conv) + static_cast<int64_t>(p.slots[n]) * p.taps * C;
  for (int j = 0; j < p.taps - 1 && end - 1 - j >= begin; ++j) {
    const int64_t t = end - 1 - j, pos = p.pos0[n] + t - begin;
    float f[8];
    load8(reinterpret_cast<const T*>(p.z) + t * p.ld + c, f);
    store8(ring + (pos % p.taps) * C + c, f);
  }
}

// ---------------------------------------------------------------------------------------------------- token by token
constexpr int kRecTok = 16;      // tokens staged at a time
constexpr int kRecCols = 32;     // columns of dv per CTA
template <int KP>                // KP rows of dk per lane, dk <= 4 KP
__global__ void __launch_bounds__(4 * kRecCols) delta_recurrent_kernel(const DeltaArgs p) {
  extern __shared__ __align__(16) float sm[];
  constexpr int kDkp = 4 * KP;
  float* s_q = sm;                          // [kRecTok][kDkp]
  float* s_k = s_q + kRecTok * kDkp;
  float* s_v = s_k + kRecTok * kDkp;        // [kRecTok][kRecCols]
  float* s_g = s_v + kRecTok * kRecCols;    // [kRecTok] decay
  float* s_b = s_g + kRecTok;               // [kRecTok] step size
  const int v0 = blockIdx.x * kRecCols, h = blockIdx.y, n = blockIdx.z;
  const int col = threadIdx.x >> 2, part = threadIdx.x & 3;
  pdl_wait();
  pdl_launch_dependents();
  const int g = h / (p.H / p.G);
  const int64_t tb = p.cu[n], te = p.cu[n + 1];
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
      const int64_t at = ((t0 + j) * p.G + g) * p.dk + c;
      s_q[i] = c < p.dk ? reinterpret_cast<const float*>(p.q)[at] : 0.f;
      s_k[i] = c < p.dk ? reinterpret_cast<const float*>(p.k)[at] : 0.f;
    }
    for (int i = threadIdx.x; i < nt * kRecCols; i += 4 * kRecCols) {
      const int j = i / kRecCols, c = i - j * kRecCols;
      s_v[i] = v0 + c < p.dv ? reinterpret_cast<const float*>(p.v)[((t0 + j) * p.H + h) * p.dv + v0 + c] : 0.f;
    }
    if (threadIdx.x < nt) {
      s_g[threadIdx.x] = expf(p.log_g[(t0 + threadIdx.x) * p.H + h]);
      s_b[threadIdx.x] = p.beta[(t0 + threadIdx.x) * p.H + h];
    }
    __syncthreads();
    for (int j = 0; j < nt; ++j) {
      const float decay = s_g[j];
      float r = 0.f;
#pragma unroll
      for (int i = 0; i < KP; ++i) {
        S[i] *= decay;
        r = fmaf(S[i], s_k[j * kDkp + part + 4 * i], r);
      }
      r += __shfl_xor_sync(0xffffffffu, r, 1);
      r += __shfl_xor_sync(0xffffffffu, r, 2);
      const float u = s_b[j] * (s_v[j * kRecCols + col] - r);
      float o = 0.f;
#pragma unroll
      for (int i = 0; i < KP; ++i) {
        const int c = j * kDkp + part + 4 * i;
        S[i] = fmaf(s_k[c], u, S[i]);
        o = fmaf(s_q[c], S[i], o);
      }
      o += __shfl_xor_sync(0xffffffffu, o, 1);
      o += __shfl_xor_sync(0xffffffffu, o, 2);
      if (part == 0 && col_ok) p.o_raw[((t0 + j) * p.H + h) * p.dv + v0 + col] = o;
    }
  }
#pragma unroll
  for (int i = 0; i < KP; ++i) {
    const int r = part + 4 * i;
    if (col_ok && r < p.dk) st[static_cast<int64_t>(r) * p.dv] = S[i];
  }
}

template <typename T>
__global__ void __launch_bounds__(128) delta_norm_gate_kernel(const DeltaArgs p) {
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
  const T* gate = reinterpret_cast<const T*>(p.z) + t * p.ld + 2 * p.G * p.dk + p.H * p.dv + h * p.dv;
  T* out = reinterpret_cast<T*>(p.out) + wid * p.dv;
  for (int c = lane; c < p.dv; c += 32) out[c] = from_f32<T>(o[c] * inv * p.norm_w[c] * silu_f32(to_f32(gate[c])));
}

template <int KP>
cudaError_t launch_rec(const DeltaArgs& a, cudaStream_t s) {
  static SmemOptIn opt;
  const int smem = (2 * kRecTok * 4 * KP + kRecTok * kRecCols + 2 * kRecTok) * 4;
  cudaError_t e = opt.ensure(delta_recurrent_kernel<KP>, smem);
  if (e != cudaSuccess) return e;
  return launch_pdl(delta_recurrent_kernel<KP>, dim3((a.dv + kRecCols - 1) / kRecCols, a.H, a.N), dim3(4 * kRecCols),
                    static_cast<size_t>(smem), s, a);
}

template <int THREADS, int U>
cudaError_t launch_decode(const DeltaArgs& a, cudaStream_t s) {
  const int groups = THREADS / (a.dv / 4);
  const size_t smem = static_cast<size_t>(2 * a.dk + 2 * a.dv + 2 * groups * a.dv) * 4;
  const dim3 grid(a.H, a.N), block(THREADS);
  return a.is_f32 ? launch_pdl(delta_decode_kernel<float, THREADS, U>, grid, block, smem, s, a)
                  : launch_pdl(delta_decode_kernel<__nv_bfloat16, THREADS, U>, grid, block, smem, s, a);
}

bool args_ok(const DeltaArgs& a) {
  return a.N >= 0 && a.G >= 1 && a.H >= 1 && a.H % a.G == 0 && a.dk >= 8 && a.dk % 8 == 0 && a.dk <= 256 && a.dv >= 8 && a.dv % 8 == 0 &&
         a.dv <= 256 && a.dv_real >= 1 && a.taps >= 1 && a.ld % 8 == 0 && a.H <= 65535 && a.N <= 65535;
}

}  // namespace

cudaError_t launch_delta_decode(const DeltaArgs& a, cudaStream_t s) {
  if (!args_ok(a)) return cudaErrorInvalidValue;
  if (a.N == 0) return cudaSuccess;
  // the small form holds states of up to 8192 elements in registers, the large one of up to 16384
  return a.dk * a.dv <= 8192 ? launch_decode<256, 8>(a, s) : launch_decode<512, 8>(a, s);
}

cudaError_t launch_delta_prepare(const DeltaArgs& a, bool split, cudaStream_t s) {
  if (!args_ok(a) || a.cu == nullptr || (split && a.is_f32)) return cudaErrorInvalidValue;
  if (a.NC == 0) return cudaSuccess;
  if (a.is_f32) return launch_prepare<float, false>(a, s);
  return split ? launch_prepare<__nv_bfloat16, true>(a, s) : launch_prepare<__nv_bfloat16, false>(a, s);
}

cudaError_t launch_delta_keep(const DeltaArgs& a, cudaStream_t s) {
  if (!args_ok(a) || a.cu == nullptr) return cudaErrorInvalidValue;
  if (a.N == 0 || a.taps == 1) return cudaSuccess;
  const dim3 grid(((2 * a.G * a.dk + a.H * a.dv) / 8 + 255) / 256, a.N), block(256);
  return a.is_f32 ? launch_pdl(delta_keep_kernel<float>, grid, block, 0, s, a)
                  : launch_pdl(delta_keep_kernel<__nv_bfloat16>, grid, block, 0, s, a);
}

cudaError_t launch_delta_recurrent(const DeltaArgs& a, cudaStream_t s) {
  if (!args_ok(a) || a.o_raw == nullptr || a.cu == nullptr) return cudaErrorInvalidValue;
  if (a.T == 0 || a.N == 0) return cudaSuccess;
  cudaError_t e = launch_delta_prepare(a, false, s);
  if (e == cudaSuccess) e = launch_delta_keep(a, s);
  if (e == cudaSuccess)
    e = a.dk <= 32 ? launch_rec<8>(a, s) : a.dk <= 64 ? launch_rec<16>(a, s) : a.dk <= 128 ? launch_rec<32>(a, s) : launch_rec<64>(a, s);
  if (e != cudaSuccess) return e;
  const dim3 grid(static_cast<unsigned>((a.T * a.H + 3) / 4)), block(128);
  return a.is_f32 ? launch_pdl(delta_norm_gate_kernel<float>, grid, block, 0, s, a)
                  : launch_pdl(delta_norm_gate_kernel<__nv_bfloat16>, grid, block, 0, s, a);
}

}  // namespace tdb
