// State space layer with its neighbours, serving form (tdb/ssd.h states the recurrence).
//
//   ssd_decode_kernel      one token per sequence: convolutions, step size, decay, state update, read-out and skip in one launch; the
//                          state is read and written once
//   ssd_prepare_kernel     prompts: convolutions with their activation, step sizes and summed log decays of all tokens
//   ssd_keep_kernel        prompts: the last inputs of the convolutions go to the state
//   ssd_recurrent_kernel   prompts token by token with the state in registers (a CTA owns 32 columns of one head of one sequence, four
//                          lanes share a column): the 32-bit path, and sizes the chunk form does not take
//   gated_norm_kernel      gate and norm over groups of the output
// The chunk-parallel form is in ssd_chunk.cu.
//
// The inputs of the convolutions are kept in a ring of `taps` rows per sequence, as in delta.cu: a decode step reads the `taps - 1`
// positions before its own and writes its own to a row that nobody reads; nothing before position 0 is ever read.
#include "tdb/launch.cuh"
#include "tdb/ssd.h"
#include "tdb/vec.cuh"

namespace tdb {

namespace {

TDB_DEVICE float softplus_f32(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
TDB_DEVICE float silu_f32(float z) { return z * sigmoid_f32(z); }
// silu of an activation of type T: to fp32 accuracy where that is what comes out.
template <typename T>
TDB_DEVICE float silu_act(float z) {
  if constexpr (sizeof(T) == 4) return silu_f32(z);
  else return __fdividef(z, 1.f + __expf(-z));
}
// exp(-exp(a_log) dt).  An error of the rate counts once per token for as long as the state lives, so the 32-bit path rounds once, at the end.
template <typename T>
TDB_DEVICE float decay_of(float a_log, float dt) {
  if constexpr (sizeof(T) == 4) return static_cast<float>(exp(-exp(static_cast<double>(a_log)) * dt));
  else return expf(-expf(a_log) * dt);
}
__host__ __device__ __forceinline__ int ssd_channels(const SsdArgs& p) { return p.H * p.dv + 2 * p.G * p.dk; }
template <typename T>
TDB_DEVICE float step_size(const SsdArgs& p, int64_t t, int h) {
  return softplus_f32(to_f32(reinterpret_cast<const T*>(p.z)[t * p.ld + p.dt_col + h]) + p.dt_bias[h]);
}

// ---------------------------------------------------------------------------------------------------- decode
// Convolution of channel c at the sequence's newest token, followed by silu.
template <typename T>
TDB_DEVICE float conv_now(const SsdArgs& p, const T* zrow, const T* ring, int64_t pos, int C, int c) {
  const float* w = p.conv_w + static_cast<int64_t>(c) * p.taps + p.taps - 1;
  float acc = fmaf(w[0], to_f32(zrow[c]), p.conv_b[c]);
  for (int j = 1; j < p.taps; ++j)
    if (pos - j >= 0) acc = fmaf(w[-j], to_f32(ring[((pos - j) % p.taps) * C + c]), acc);
  return silu_f32(acc);
}

constexpr int kDecThreads = 256;
constexpr int kDecRows = 8;        // rows of the state per thread in flight

template <typename T>
__global__ void __launch_bounds__(kDecThreads) ssd_decode_kernel(const SsdArgs p) {
  extern __shared__ __align__(16) float sm[];
  float* s_b = sm;                 // [dk] dt B
  float* s_c = s_b + p.dk;         // [dk]
  float* s_x = s_c + p.dk;         // [dv]
  float* s_p = s_x + p.dv;         // [row groups][dv] partial read-outs
  const int h = blockIdx.x, n = blockIdx.y;
  pdl_wait();
  pdl_launch_dependents();
  const int dv4 = p.dv >> 2, groups = kDecThreads / dv4;
  const int c4 = threadIdx.x % dv4, rg = threadIdx.x / dv4;
  const int64_t pos = p.pos0[n], slot = p.slots[n];
  const bool fresh = pos == 0;
  float4* S = reinterpret_cast<float4*>(p.state + ((slot * p.H + h) * p.dk) * p.dv) + c4;
  float4 s[kDecRows];
  auto fetch = [&](int r0) {
#pragma unroll
    for (int u = 0; u < kDecRows; ++u) {
      const int r = r0 + u * groups;
      s[u] = (r < p.dk && !fresh) ? S[static_cast<int64_t>(r) * dv4] : make_float4(0.f, 0.f, 0.f, 0.f);
    }
  };
  if (rg < groups) fetch(rg);
  // inputs, while the state travels
  const int share = p.H / p.G, g = h / share, Hv = p.H * p.dv, Gk = p.G * p.dk, C = ssd_channels(p);
  const T* zrow = reinterpret_cast<const T*>(p.z) + n * p.ld;
  T* ring = reinterpret_cast<T*>(p.conv) + slot * p.taps * C;
  T* keep = ring + (pos % p.taps) * C;
  const float dt = step_size<T>(p, n, h), decay = decay_of<T>(p.a_log[h], dt);
  for (int i = threadIdx.x; i < 2 * p.dk + p.dv; i += kDecThreads) {
    const bool is_x = i >= 2 * p.dk;
    const int c = is_x ? h * p.dv + i - 2 * p.dk : Hv + (i < p.dk ? g * p.dk + i : Gk + g * p.dk + i - p.dk);
    const float v = conv_now(p, zrow, ring, pos, C, c);
    sm[i] = i < p.dk ? v * dt : v;
    if (is_x || h % share == 0) keep[c] = zrow[c];
  }
  __syncthreads();
  if (rg < groups) {
    const float4 x = reinterpret_cast<const float4*>(s_x)[c4];
    float4 y = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int r0 = rg; r0 < p.dk; r0 += groups * kDecRows) {
      if (r0 != rg) fetch(r0);
#pragma unroll
      for (int u = 0; u < kDecRows; ++u) {
        const int r = r0 + u * groups;
        if (r < p.dk) {
          const float b = s_b[r], c = s_c[r];
          float4 v = s[u];
          v.x = fmaf(decay, v.x, b * x.x); v.y = fmaf(decay, v.y, b * x.y);
          v.z = fmaf(decay, v.z, b * x.z); v.w = fmaf(decay, v.w, b * x.w);
          S[static_cast<int64_t>(r) * dv4] = v;
          y.x = fmaf(c, v.x, y.x); y.y = fmaf(c, v.y, y.y); y.z = fmaf(c, v.z, y.z); y.w = fmaf(c, v.w, y.w);
        }
      }
    }
    reinterpret_cast<float4*>(s_p + rg * p.dv)[c4] = y;
  }
  __syncthreads();
  T* out = reinterpret_cast<T*>(p.out) + static_cast<int64_t>(n) * Hv + h * p.dv;
  for (int c = threadIdx.x; c < p.dv; c += kDecThreads) {
    float y = p.skip[h] * s_x[c];
    for (int i = 0; i < groups; ++i) y += s_p[i * p.dv + c];
    out[c] = from_f32<T>(y);
  }
}

// ---------------------------------------------------------------------------------------------------- inputs of prompts
constexpr int kPrepTok = 32;      // tokens per CTA
constexpr int kPrepThreads = 128;
constexpr int kBatch = 8;         // tokens whose inputs are requested together
constexpr int kV = 4;             // channels of a thread

TDB_DEVICE void load_v(const __nv_bfloat16* p, float (&f)[kV]) {
  const uint2 v = *reinterpret_cast<const uint2*>(p);
  const float2 a = unpack_bf16x2(v.x), b = unpack_bf16x2(v.y);
  f[0] = a.x; f[1] = a.y; f[2] = b.x; f[3] = b.y;
}
TDB_DEVICE void load_v(const float* p, float (&f)[kV]) {
  const float4 v = *reinterpret_cast<const float4*>(p);
  f[0] = v.x; f[1] = v.y; f[2] = v.z; f[3] = v.w;
}
TDB_DEVICE void store_v(__nv_bfloat16* p, const float (&f)[kV]) {
  *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(f[0], f[1]), pack_bf16x2(f[2], f[3]));
}
TDB_DEVICE void store_v(float* p, const float (&f)[kV]) { *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]); }

// A thread owns kV channels.  TAPS > 0: convolutions of at most TAPS taps, weights and the last inputs in registers; 0: any number.
// The last row of blocks takes the step sizes and decays.
template <typename T, int TAPS>
__global__ void __launch_bounds__(kPrepThreads) ssd_prepare_kernel(const SsdArgs p) {
  pdl_wait();
  pdl_launch_dependents();
  const int n = p.chunk_seq[blockIdx.x], C = ssd_channels(p);
  const int64_t c0 = p.chunk_t0[blockIdx.x], begin = p.cu[n], end = min(static_cast<int64_t>(p.cu[n + 1]), c0 + 64);
  if (blockIdx.y == gridDim.y - 1) {
    for (int h = blockIdx.z * kPrepThreads + threadIdx.x; h < p.H; h += gridDim.z * kPrepThreads) {
      const float rate = -expf(p.a_log[h]);
      float g = 0.f;
#pragma unroll 8
      for (int64_t t = c0; t < end; ++t) {
        const float dt = step_size<T>(p, t, h);
        g = fmaf(rate, dt, g);
        p.dt[t * p.H + h] = dt;
        p.log_g[t * p.H + h] = g;
      }
    }
    return;
  }
  const int64_t t0 = c0 + blockIdx.z * kPrepTok, t1 = min(t0 + kPrepTok, end), before = p.pos0[n] - begin;
  const int c = (blockIdx.y * kPrepThreads + threadIdx.x) * kV;
  if (t0 >= t1 || c >= C) return;
  const T* z = reinterpret_cast<const T*>(p.z);
  const T* ring = reinterpret_cast<const T*>(p.conv) + static_cast<int64_t>(p.slots[n]) * p.taps * C;
  auto input = [&](int64_t t, float (&f)[kV]) {           // of (packed) token t, zero before the sequence
    const int64_t pos = before + t;
    if (t >= begin) {
      load_v(z + t * p.ld + c, f);
    } else if (pos >= 0) {
      load_v(ring + (pos % p.taps) * C + c, f);
    } else {
#pragma unroll
      for (int i = 0; i < kV; ++i) f[i] = 0.f;
    }
  };
  float bias[kV];
  load_v(p.conv_b + c, bias);
  auto finish = [&](int64_t t, float (&acc)[kV]) {
#pragma unroll
    for (int i = 0; i < kV; ++i) acc[i] = silu_act<T>(acc[i]);
    store_v(reinterpret_cast<T*>(p.xbc) + t * C + c, acc);
  };
  if constexpr (TAPS > 0) {
    float w[TAPS][kV], x[TAPS + kBatch - 1][kV];           // x[j]: input of token (first of the batch) + kBatch - 1 - j
#pragma unroll
    for (int j = 0; j < TAPS; ++j) {
#pragma unroll
      for (int i = 0; i < kV; ++i) {
        w[j][i] = j < p.taps ? p.conv_w[static_cast<int64_t>(c + i) * p.taps + p.taps - 1 - j] : 0.f;
        x[j][i] = 0.f;
      }
      if (j + 1 < TAPS && j + 1 < p.taps) input(t0 - 1 - j, x[j]);       // shifted into place below
    }
    for (int64_t b = t0; b < t1; b += kBatch) {
#pragma unroll
      for (int j = TAPS - 2; j >= 0; --j)
#pragma unroll
        for (int i = 0; i < kV; ++i) x[j + kBatch][i] = x[j][i];
#pragma unroll
      for (int j = 0; j < kBatch; ++j) {
        if (b + j < t1) {
          load_v(z + (b + j) * p.ld + c, x[kBatch - 1 - j]);
        } else {
#pragma unroll
          for (int i = 0; i < kV; ++i) x[kBatch - 1 - j][i] = 0.f;
        }
      }
#pragma unroll
      for (int k = 0; k < kBatch; ++k) {
        if (b + k >= t1) break;
        float acc[kV];
#pragma unroll
        for (int i = 0; i < kV; ++i) acc[i] = bias[i];
#pragma unroll
        for (int j = 0; j < TAPS; ++j)
#pragma unroll
          for (int i = 0; i < kV; ++i) acc[i] = fmaf(w[j][i], x[kBatch - 1 - k + j][i], acc[i]);
        finish(b + k, acc);
      }
    }
  } else {
    for (int64_t t = t0; t < t1; ++t) {
      float acc[kV];
#pragma unroll
      for (int i = 0; i < kV; ++i) acc[i] = bias[i];
      for (int j = 0; j < p.taps; ++j) {
        float f[kV];
        input(t - j, f);
        const float* wj = p.conv_w + static_cast<int64_t>(c) * p.taps + p.taps - 1 - j;
#pragma unroll
        for (int i = 0; i < kV; ++i) acc[i] = fmaf(wj[i * p.taps], f[i], acc[i]);
      }
      finish(t, acc);
    }
  }
}

template <typename T>
cudaError_t launch_prepare(const SsdArgs& a, cudaStream_t s) {
  const dim3 grid(a.NC, (ssd_channels(a) / kV + kPrepThreads - 1) / kPrepThreads + 1, 64 / kPrepTok), block(kPrepThreads);
  return a.taps <= 2   ? launch_pdl(ssd_prepare_kernel<T, 2>, grid, block, 0, s, a)
         : a.taps <= 4 ? launch_pdl(ssd_prepare_kernel<T, 4>, grid, block, 0, s, a)
                       : launch_pdl(ssd_prepare_kernel<T, 0>, grid, block, 0, s, a);
}

template <typename T>
__global__ void __launch_bounds__(256) ssd_keep_kernel(const SsdArgs p) {
  pdl_wait();
  pdl_launch_dependents();
  const int n = blockIdx.y, C = ssd_channels(p);
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
template <typename T, int KP>    // KP rows of dk per lane, dk <= 4 KP
__global__ void __launch_bounds__(4 * kRecCols) ssd_recurrent_kernel(const SsdArgs p) {
  extern __shared__ __align__(16) float sm[];
  constexpr int kDkp = 4 * KP;
  float* s_b = sm;                          // [kRecTok][kDkp]
  float* s_c = s_b + kRecTok * kDkp;
  float* s_x = s_c + kRecTok * kDkp;        // [kRecTok][kRecCols]
  float* s_g = s_x + kRecTok * kRecCols;    // [kRecTok] decay
  float* s_d = s_g + kRecTok;               // [kRecTok] step size
  const int v0 = blockIdx.x * kRecCols, h = blockIdx.y, n = blockIdx.z;
  const int col = threadIdx.x >> 2, part = threadIdx.x & 3;
  pdl_wait();
  pdl_launch_dependents();
  const int g = h / (p.H / p.G), Hv = p.H * p.dv, Gk = p.G * p.dk, C = ssd_channels(p);
  const int64_t tb = p.cu[n], te = p.cu[n + 1];
  const bool col_ok = v0 + col < p.dv, fresh = p.pos0[n] == 0;
  const float a_log = p.a_log[h], skip = p.skip[h];
  const T* xbc = reinterpret_cast<const T*>(p.xbc);
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
      const T* row = xbc + (t0 + j) * C + Hv + g * p.dk + c;
      s_b[i] = c < p.dk ? to_f32(row[0]) : 0.f;
      s_c[i] = c < p.dk ? to_f32(row[Gk]) : 0.f;
    }
    for (int i = threadIdx.x; i < nt * kRecCols; i += 4 * kRecCols) {
      const int j = i / kRecCols, c = i - j * kRecCols;
      s_x[i] = v0 + c < p.dv ? to_f32(xbc[(t0 + j) * C + h * p.dv + v0 + c]) : 0.f;
    }
    if (threadIdx.x < nt) {
      const float dt = p.dt[(t0 + threadIdx.x) * p.H + h];
      s_d[threadIdx.x] = dt;
      s_g[threadIdx.x] = decay_of<T>(a_log, dt);
    }
    __syncthreads();
    for (int j = 0; j < nt; ++j) {
      const float decay = s_g[j], x = s_x[j * kRecCols + col], u = s_d[j] * x;
      float y = 0.f;
#pragma unroll
      for (int i = 0; i < KP; ++i) {
        const int c = j * kDkp + part + 4 * i;
        S[i] = fmaf(decay, S[i], s_b[c] * u);
        y = fmaf(s_c[c], S[i], y);
      }
      y += __shfl_xor_sync(0xffffffffu, y, 1);
      y += __shfl_xor_sync(0xffffffffu, y, 2);
      if (part == 0 && col_ok) reinterpret_cast<T*>(p.out)[(t0 + j) * Hv + h * p.dv + v0 + col] = from_f32<T>(fmaf(skip, x, y));
    }
  }
#pragma unroll
  for (int i = 0; i < KP; ++i) {
    const int r = part + 4 * i;
    if (col_ok && r < p.dk) st[static_cast<int64_t>(r) * p.dv] = S[i];
  }
}

template <typename T, int KP>
cudaError_t launch_rec(const SsdArgs& a, cudaStream_t s) {
  static SmemOptIn opt;
  const int smem = (2 * kRecTok * 4 * KP + kRecTok * kRecCols + 2 * kRecTok) * 4;
  cudaError_t e = opt.ensure(ssd_recurrent_kernel<T, KP>, smem);
  if (e != cudaSuccess) return e;
  return launch_pdl(ssd_recurrent_kernel<T, KP>, dim3((a.dv + kRecCols - 1) / kRecCols, a.H, a.N), dim3(4 * kRecCols), static_cast<size_t>(smem), s, a);
}
template <typename T>
cudaError_t launch_rec_t(const SsdArgs& a, cudaStream_t s) {
  return a.dk <= 32 ? launch_rec<T, 8>(a, s) : a.dk <= 64 ? launch_rec<T, 16>(a, s) : a.dk <= 128 ? launch_rec<T, 32>(a, s) : launch_rec<T, 64>(a, s);
}

// ---------------------------------------------------------------------------------------------------- gate and norm
// One block per (token, part).  PLAIN: no padding between heads and parts of a multiple of eight elements; a thread keeps NCH groups of
// eight in registers.
template <typename T, bool PLAIN, int NCH>
__global__ void __launch_bounds__(512) gated_norm_kernel(const GatedNormArgs p) {
  __shared__ float red[32];
  pdl_wait();
  pdl_launch_dependents();
  const int64_t t = blockIdx.x;
  const int part = blockIdx.y, size = p.H * p.dv_real / p.parts, cols = p.H * p.dv;
  const T* y = reinterpret_cast<const T*>(p.y) + t * cols;
  const T* gate = reinterpret_cast<const T*>(p.gate) + t * p.ld_gate;
  T* out = reinterpret_cast<T*>(p.out) + t * cols;
  float ss = 0.f;
  if constexpr (PLAIN) {
    float f[NCH][8];
#pragma unroll
    for (int k = 0; k < NCH; ++k) {
      const int e = (threadIdx.x + k * blockDim.x) * 8;
      if (e >= size) continue;
      float g[8];
      load8(y + part * size + e, f[k]);
      load8(gate + part * size + e, g);
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        f[k][i] *= silu_act<T>(g[i]);
        ss += f[k][i] * f[k][i];
      }
    }
    const float inv = 1.f / sqrtf(block_reduce_sum(ss, red) / size + p.eps);
#pragma unroll
    for (int k = 0; k < NCH; ++k) {
      const int e = (threadIdx.x + k * blockDim.x) * 8;
      if (e >= size) continue;
      float w[8];
      load8(p.w + part * size + e, w);
#pragma unroll
      for (int i = 0; i < 8; ++i) f[k][i] *= inv * w[i];
      store8(out + part * size + e, f[k]);
    }
  } else {
    auto at = [&](int e) { return (e / p.dv_real) * p.dv + e % p.dv_real; };
    auto gated = [&](int c) {
      const float g = to_f32(gate[c]);
      return to_f32(y[c]) * silu_f32(g);
    };
    for (int e = threadIdx.x; e < size; e += blockDim.x) {
      const float f = gated(at(part * size + e));
      ss += f * f;
    }
    const float inv = 1.f / sqrtf(block_reduce_sum(ss, red) / size + p.eps);
    for (int e = threadIdx.x; e < size; e += blockDim.x) {
      const int c = at(part * size + e);
      out[c] = from_f32<T>(gated(c) * inv * p.w[c]);
    }
    const int pad = p.dv - p.dv_real;
    if (part == 0)
      for (int i = threadIdx.x; i < p.H * pad; i += blockDim.x) out[(i / pad) * p.dv + p.dv_real + i % pad] = from_f32<T>(0.f);
  }
}

template <typename T>
cudaError_t launch_gated_norm_t(const GatedNormArgs& a, cudaStream_t s) {
  const int size = a.H * a.dv_real / a.parts;
  const dim3 grid(static_cast<unsigned>(a.T), a.parts);
  if (a.dv != a.dv_real || size % 8 != 0 || size > 32768) return launch_pdl(gated_norm_kernel<T, false, 1>, grid, dim3(size >= 1024 ? 256 : 64), 0, s, a);
  const int vec = size / 8;
  if (vec <= 256) return launch_pdl(gated_norm_kernel<T, true, 1>, grid, dim3((vec + 31) / 32 * 32), 0, s, a);
  if (vec <= 1024) return launch_pdl(gated_norm_kernel<T, true, 2>, grid, dim3(512), 0, s, a);
  return launch_pdl(gated_norm_kernel<T, true, 8>, grid, dim3(512), 0, s, a);
}

bool args_ok(const SsdArgs& a) {
  return a.N >= 0 && a.G >= 1 && a.H >= 1 && a.H % a.G == 0 && a.dk >= 8 && a.dk % 8 == 0 && a.dk <= 256 && a.dv >= 8 && a.dv % 8 == 0 && a.dv <= 256 &&
         a.taps >= 1 && a.ld % 8 == 0 && a.H <= 65535 && a.N <= 65535;
}

}  // namespace

cudaError_t launch_ssd_decode(const SsdArgs& a, cudaStream_t s) {
  if (!args_ok(a)) return cudaErrorInvalidValue;
  if (a.N == 0) return cudaSuccess;
  const int groups = kDecThreads / (a.dv / 4);
  const size_t smem = static_cast<size_t>(2 * a.dk + a.dv + groups * a.dv) * 4;
  const dim3 grid(a.H, a.N), block(kDecThreads);
  return a.is_f32 ? launch_pdl(ssd_decode_kernel<float>, grid, block, smem, s, a) : launch_pdl(ssd_decode_kernel<__nv_bfloat16>, grid, block, smem, s, a);
}

cudaError_t launch_ssd_prepare(const SsdArgs& a, cudaStream_t s) {
  if (!args_ok(a) || a.cu == nullptr) return cudaErrorInvalidValue;
  if (a.NC == 0) return cudaSuccess;
  return a.is_f32 ? launch_prepare<float>(a, s) : launch_prepare<__nv_bfloat16>(a, s);
}

cudaError_t launch_ssd_keep(const SsdArgs& a, cudaStream_t s) {
  if (!args_ok(a) || a.cu == nullptr) return cudaErrorInvalidValue;
  if (a.N == 0 || a.taps == 1) return cudaSuccess;
  const dim3 grid((ssd_channels(a) / 8 + 255) / 256, a.N), block(256);
  return a.is_f32 ? launch_pdl(ssd_keep_kernel<float>, grid, block, 0, s, a) : launch_pdl(ssd_keep_kernel<__nv_bfloat16>, grid, block, 0, s, a);
}

cudaError_t launch_ssd_recurrent(const SsdArgs& a, cudaStream_t s) {
  if (!args_ok(a) || a.cu == nullptr) return cudaErrorInvalidValue;
  if (a.T == 0 || a.N == 0) return cudaSuccess;
  cudaError_t e = launch_ssd_prepare(a, s);
  if (e == cudaSuccess) e = launch_ssd_keep(a, s);
  if (e == cudaSuccess) e = a.is_f32 ? launch_rec_t<float>(a, s) : launch_rec_t<__nv_bfloat16>(a, s);
  return e;
}

cudaError_t launch_gated_norm(const GatedNormArgs& a, cudaStream_t s) {
  if (a.H < 1 || a.dv < a.dv_real || a.dv_real < 1 || a.dv % 8 != 0 || a.parts < 1 || a.parts > 65535 || (a.H * a.dv_real) % a.parts != 0 || a.ld_gate % 8 != 0)
    return cudaErrorInvalidValue;
  if (a.T == 0) return cudaSuccess;
  return a.is_f32 ? launch_gated_norm_t<float>(a, s) : launch_gated_norm_t<__nv_bfloat16>(a, s);
}

}  // namespace tdb
