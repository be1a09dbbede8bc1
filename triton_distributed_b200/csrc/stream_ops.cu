// Residual-stream kernels of decoders that keep the stream in fp32 and norm a sublayer's OUTPUT before adding it:
// embedding into the stream, x += RMSNorm(y) * w (y summed over a token's expert rows and a gated shared row on the
// way), and the norm in front of the head.  Of parallel layers that norm the stream itself: x += mixer + feed-forward and both
// norms of the next layer in one pass.  The stream has a bf16 copy that the next sublayer's GEMMs read.
// One block per token, 32-byte accesses, the row is kept in shared memory between the two passes.
#include "tdb/hybrid.h"
#include "tdb/launch.cuh"
#include "tdb/vec.cuh"

namespace tdb {

namespace {

template <typename T>
__global__ void embed_stream_kernel(const int64_t* __restrict__ ids, const T* __restrict__ table, float* __restrict__ x,
                                    T* __restrict__ xb, int W, int64_t vocab, float scale) {
  const int64_t t = blockIdx.x;
  int64_t id = ids[t];
  if (id < 0 || id >= vocab) id = 0;
  for (int c = threadIdx.x * 8; c < W; c += blockDim.x * 8) {
    float f[8];
    load8(table + id * W + c, f);
#pragma unroll
    for (int i = 0; i < 8; ++i) f[i] *= scale;
    store8(x + t * W + c, f);
    if (xb != nullptr) store8(xb + t * W + c, f);
  }
}

// Sum of a token's contributions, columns [c, c + 8).
template <typename TY>
TDB_DEVICE void token_sum(const TY* y, int rows, const TY* shared, float gate, int64_t t, int W, int c, float (&acc)[8]) {
  load8(y + t * rows * W + c, acc);
  for (int r = 1; r < rows; ++r) {
    float f[8];
    load8(y + (t * rows + r) * W + c, f);
#pragma unroll
    for (int i = 0; i < 8; ++i) acc[i] += f[i];
  }
  if (shared != nullptr) {
    float f[8];
    load8(shared + t * W + c, f);
#pragma unroll
    for (int i = 0; i < 8; ++i) acc[i] += gate * f[i];
  }
}

template <typename TY>
__global__ void postnorm_add_kernel(const PostNormArgs p) {
  __shared__ float red[32];
  extern __shared__ float row[];       // [W]
  pdl_wait();
  pdl_launch_dependents();
  const int64_t t = blockIdx.x;
  const TY* y = reinterpret_cast<const TY*>(p.y);
  const TY* sh = reinterpret_cast<const TY*>(p.shared);
  const float gate = (sh != nullptr && p.shared_gate != nullptr) ? p.shared_gate[t] : 1.f;
  float ss = 0.f;
  for (int c = threadIdx.x * 8; c < p.W; c += blockDim.x * 8) {
    float a[8];
    token_sum(y, p.rows_per_token, sh, gate, t, p.W, c, a);
#pragma unroll
    for (int i = 0; i < 8; ++i) ss += a[i] * a[i];
    store8(row + c, a);
  }
  const float inv = 1.f / sqrtf(block_reduce_sum(ss, red) / p.n_real + p.eps);
  __nv_bfloat16* xb = reinterpret_cast<__nv_bfloat16*>(p.xb);
  for (int c = threadIdx.x * 8; c < p.W; c += blockDim.x * 8) {
    float a[8], w[8], x[8];
    load8(row + c, a);
    load8(p.w + c, w);
    load8(p.x + t * p.W + c, x);
#pragma unroll
    for (int i = 0; i < 8; ++i) x[i] += a[i] * inv * w[i];
    store8(p.x + t * p.W + c, x);
    if (xb != nullptr) store8(xb + t * p.W + c, x);
  }
}

template <typename TY>
__global__ void combine_rows_kernel(const PostNormArgs p, TY* out) {
  pdl_wait();
  pdl_launch_dependents();
  const int64_t t = blockIdx.x;
  const TY* sh = reinterpret_cast<const TY*>(p.shared);
  const float gate = (sh != nullptr && p.shared_gate != nullptr) ? p.shared_gate[t] : 1.f;
  for (int c = threadIdx.x * 8; c < p.W; c += blockDim.x * 8) {
    float a[8];
    token_sum(reinterpret_cast<const TY*>(p.y), p.rows_per_token, sh, gate, t, p.W, c, a);
    store8(out + t * p.W + c, a);
  }
}

template <typename TO>
__global__ void stream_norm_kernel(const float* __restrict__ x, const int64_t* __restrict__ rows, const float* __restrict__ w,
                                   TO* __restrict__ out, int W, int n_real, float eps) {
  __shared__ float red[32];
  pdl_wait();
  pdl_launch_dependents();
  const int64_t i = blockIdx.x;
  const float* xr = x + (rows != nullptr ? rows[i] : i) * W;
  float ss = 0.f;
  for (int c = threadIdx.x * 8; c < W; c += blockDim.x * 8) {
    float a[8];
    load8(xr + c, a);
#pragma unroll
    for (int j = 0; j < 8; ++j) ss += a[j] * a[j];
  }
  const float inv = 1.f / sqrtf(block_reduce_sum(ss, red) / n_real + eps);
  for (int c = threadIdx.x * 8; c < W; c += blockDim.x * 8) {
    float a[8], g[8];
    load8(xr + c, a);
    load8(w + c, g);
#pragma unroll
    for (int j = 0; j < 8; ++j) a[j] *= inv * g[j];
    store8(out + i * W + c, a);
  }
}

// One block per token; the new row stays in shared memory between the two passes.
template <typename TA, typename TY>
__global__ void parallel_add_kernel(const ParallelAddArgs p) {
  __shared__ float red[32];
  extern __shared__ float row[];       // [W]
  pdl_wait();
  pdl_launch_dependents();
  const int64_t t = blockIdx.x, at = t * p.W;
  const TA* mix = reinterpret_cast<const TA*>(p.mix);
  const TA* shared = reinterpret_cast<const TA*>(p.shared);
  const TA* hin = reinterpret_cast<const TA*>(p.hin);
  const TY* y = reinterpret_cast<const TY*>(p.y) + at * p.rows;
  float ss = 0.f;
  for (int c = threadIdx.x * 8; c < p.W; c += blockDim.x * 8) {
    float a[8] = {}, f[8];
    auto add = [&](float w) {
#pragma unroll
      for (int i = 0; i < 8; ++i) a[i] = fmaf(w, f[i], a[i]);
    };
    if (mix != nullptr) {
      load8(mix + at + c, f);
      add(1.f);
    }
    if (p.y != nullptr)
      for (int r = 0; r < p.rows; ++r) {
        const int e = p.ids != nullptr ? p.ids[t * p.rows + r] : 0;
        if (p.ids == nullptr || (e >= 0 && e < p.experts)) {
          load8(y + static_cast<int64_t>(r) * p.W + c, f);
          add(1.f);
        } else if (hin != nullptr) {
          load8(hin + at + c, f);
          add(p.weights[t * p.rows + r]);
        }
      }
    if (shared != nullptr) {
      load8(shared + at + c, f);
      add(1.f);
    }
    if (p.bias != nullptr) {
      load8(p.bias + c, f);
      add(1.f);
    }
    if (p.sum_out != nullptr) {
      store8(p.sum_out + at + c, a);
      continue;
    }
    load8(p.x + at + c, f);
    add(1.f);
    if (mix != nullptr || p.y != nullptr) store8(p.x + at + c, a);
#pragma unroll
    for (int i = 0; i < 8; ++i) ss += a[i] * a[i];
    store8(row + c, a);
  }
  if (p.sum_out != nullptr || p.h1 == nullptr) return;
  const float inv = 1.f / sqrtf(block_reduce_sum(ss, red) / p.n_real + p.eps);
  for (int c = threadIdx.x * 8; c < p.W; c += blockDim.x * 8) {
    float a[8], w[8], o[8];
    load8(row + c, a);
    load8(p.w1 + c, w);
#pragma unroll
    for (int i = 0; i < 8; ++i) o[i] = a[i] * inv * w[i];
    store8(reinterpret_cast<TA*>(p.h1) + at + c, o);
    if (p.h2 == nullptr) continue;
    load8(p.w2 + c, w);
#pragma unroll
    for (int i = 0; i < 8; ++i) o[i] = a[i] * inv * w[i];
    store8(reinterpret_cast<TA*>(p.h2) + at + c, o);
  }
}

// One block per row; a thread keeps its NCH groups of eight columns in registers through both norms.
template <typename T, int NCH>
__global__ void __launch_bounds__(512) sandwich_kernel(const SandwichArgs p) {
  __shared__ float red[2][32];
  pdl_wait();
  pdl_launch_dependents();
  const int64_t i = blockIdx.x, t = p.rows != nullptr ? p.rows[i] : i;
  float x[NCH][8], y[NCH][8];
  float ss = 0.f;
  int64_t id = 0;
  if (p.ids != nullptr) {
    id = p.ids[t];
    if (id < 0 || id >= p.vocab) id = 0;
  }
#pragma unroll
  for (int k = 0; k < NCH; ++k) {
    const int c = (threadIdx.x + k * blockDim.x) * 8;
    if (c >= p.W) continue;
    if (p.ids != nullptr) {
      load8(reinterpret_cast<const T*>(p.table) + id * p.W + c, x[k]);
#pragma unroll
      for (int e = 0; e < 8; ++e) x[k][e] *= p.scale;
    } else {
      load8(p.x + t * p.W + c, x[k]);
    }
    if (p.y != nullptr) {
      load8(reinterpret_cast<const T*>(p.y) + t * p.W + c, y[k]);
#pragma unroll
      for (int e = 0; e < 8; ++e) ss += y[k][e] * y[k][e];
    }
  }
  auto weight = [&](const float* w, int n, int c, float (&f)[8]) {
    if (n > 1) {
      load8(w + c, f);
    } else {
#pragma unroll
      for (int e = 0; e < 8; ++e) f[e] = w[0];
    }
  };
  const float inv_y = p.y != nullptr ? 1.f / sqrtf(block_reduce_sum(ss, red[0]) / p.n_real + p.eps) : 0.f;
  ss = 0.f;
#pragma unroll
  for (int k = 0; k < NCH; ++k) {
    const int c = (threadIdx.x + k * blockDim.x) * 8;
    if (c >= p.W) continue;
    if (p.y != nullptr) {
      float w[8];
      weight(p.post, p.post_n, c, w);
#pragma unroll
      for (int e = 0; e < 8; ++e) x[k][e] += y[k][e] * inv_y * w[e];
    }
    if (p.store) store8(p.x + t * p.W + c, x[k]);
#pragma unroll
    for (int e = 0; e < 8; ++e) ss += x[k][e] * x[k][e];
  }
  if (p.h == nullptr) return;
  const float inv_x = 1.f / sqrtf(block_reduce_sum(ss, red[1]) / p.n_real + p.eps);
#pragma unroll
  for (int k = 0; k < NCH; ++k) {
    const int c = (threadIdx.x + k * blockDim.x) * 8;
    if (c >= p.W) continue;
    float w[8];
    weight(p.pre, p.pre_n, c, w);
#pragma unroll
    for (int e = 0; e < 8; ++e) x[k][e] *= inv_x * w[e];
    store8(reinterpret_cast<T*>(p.h) + i * p.W + c, x[k]);
  }
}

int row_threads(int W) {
  const int vec = W / 8;
  return vec >= 512 ? 512 : vec >= 256 ? 256 : vec >= 128 ? 128 : 64;
}

}  // namespace

cudaError_t launch_embed_stream(const int64_t* ids, const void* table, float* x, void* xb, int64_t T, int W, int64_t vocab,
                                float scale, int is_f32, cudaStream_t s) {
  if (W % 8 != 0) return cudaErrorInvalidValue;
  if (T == 0) return cudaSuccess;
  if (is_f32)
    embed_stream_kernel<float><<<static_cast<unsigned>(T), row_threads(W), 0, s>>>(
        ids, reinterpret_cast<const float*>(table), x, nullptr, W, vocab, scale);
  else
    embed_stream_kernel<__nv_bfloat16><<<static_cast<unsigned>(T), row_threads(W), 0, s>>>(
        ids, reinterpret_cast<const __nv_bfloat16*>(table), x, reinterpret_cast<__nv_bfloat16*>(xb), W, vocab, scale);
  return cudaGetLastError();
}

cudaError_t launch_postnorm_add(const PostNormArgs& a, cudaStream_t s) {
  if (a.W % 8 != 0 || a.n_real < 1 || a.rows_per_token < 1) return cudaErrorInvalidValue;
  if (a.T == 0) return cudaSuccess;
  const size_t smem = static_cast<size_t>(a.W) * 4;
  if (smem > 200 * 1024) return cudaErrorInvalidValue;
  static SmemOptIn f, b;
  if (smem > 40 * 1024) {
    cudaError_t e = a.y_f32 ? f.ensure(postnorm_add_kernel<float>, 200 * 1024)
                            : b.ensure(postnorm_add_kernel<__nv_bfloat16>, 200 * 1024);
    if (e != cudaSuccess) return e;
  }
  const dim3 grid(static_cast<unsigned>(a.T)), block(row_threads(a.W));
  return a.y_f32 ? launch_pdl(postnorm_add_kernel<float>, grid, block, smem, s, a)
                 : launch_pdl(postnorm_add_kernel<__nv_bfloat16>, grid, block, smem, s, a);
}

cudaError_t launch_combine_rows(const PostNormArgs& a, void* out, cudaStream_t s) {
  if (a.W % 8 != 0 || a.rows_per_token < 1) return cudaErrorInvalidValue;
  if (a.T == 0) return cudaSuccess;
  const dim3 grid(static_cast<unsigned>(a.T)), block(row_threads(a.W));
  return a.y_f32 ? launch_pdl(combine_rows_kernel<float>, grid, block, 0, s, a, reinterpret_cast<float*>(out))
                 : launch_pdl(combine_rows_kernel<__nv_bfloat16>, grid, block, 0, s, a, reinterpret_cast<__nv_bfloat16*>(out));
}

cudaError_t launch_parallel_add(const ParallelAddArgs& a, cudaStream_t s) {
  if (a.W % 8 != 0 || a.n_real < 1 || (a.y != nullptr && a.rows < 1) || (a.act_f32 && a.y != nullptr && !a.y_f32) ||
      (a.ids != nullptr && a.weights == nullptr) || (a.h1 != nullptr && a.w1 == nullptr) || (a.h2 != nullptr && a.w2 == nullptr))
    return cudaErrorInvalidValue;
  if (a.T == 0) return cudaSuccess;
  const size_t smem = static_cast<size_t>(a.W) * 4;
  if (smem > 200 * 1024) return cudaErrorInvalidValue;
  static SmemOptIn ff, bf, bb;
  if (smem > 40 * 1024) {
    cudaError_t e = a.act_f32 ? ff.ensure(parallel_add_kernel<float, float>, 200 * 1024)
                    : a.y_f32 ? bf.ensure(parallel_add_kernel<__nv_bfloat16, float>, 200 * 1024)
                              : bb.ensure(parallel_add_kernel<__nv_bfloat16, __nv_bfloat16>, 200 * 1024);
    if (e != cudaSuccess) return e;
  }
  const dim3 grid(static_cast<unsigned>(a.T)), block(row_threads(a.W));
  return a.act_f32 ? launch_pdl(parallel_add_kernel<float, float>, grid, block, smem, s, a)
         : a.y_f32 ? launch_pdl(parallel_add_kernel<__nv_bfloat16, float>, grid, block, smem, s, a)
                   : launch_pdl(parallel_add_kernel<__nv_bfloat16, __nv_bfloat16>, grid, block, smem, s, a);
}

namespace {
template <typename T>
cudaError_t launch_sandwich_t(const SandwichArgs& a, cudaStream_t s) {
  const dim3 grid(static_cast<unsigned>(a.n));
  const int vec = a.W / 8;
  if (vec <= 512) return launch_pdl(sandwich_kernel<T, 1>, grid, dim3((vec + 31) / 32 * 32), 0, s, a);
  if (vec <= 1024) return launch_pdl(sandwich_kernel<T, 2>, grid, dim3(512), 0, s, a);
  return launch_pdl(sandwich_kernel<T, 8>, grid, dim3(512), 0, s, a);
}
}  // namespace

cudaError_t launch_sandwich(const SandwichArgs& a, cudaStream_t s) {
  auto weight_ok = [&](const float* w, int n) { return w != nullptr && (n == 1 || n == a.W); };
  if (a.W % 8 != 0 || a.W < 8 || a.W > 32768 || a.n_real < 1 || (a.y != nullptr && !weight_ok(a.post, a.post_n)) || (a.h != nullptr && !weight_ok(a.pre, a.pre_n)) ||
      (a.ids != nullptr && a.table == nullptr))
    return cudaErrorInvalidValue;
  if (a.n == 0) return cudaSuccess;
  return a.is_f32 ? launch_sandwich_t<float>(a, s) : launch_sandwich_t<__nv_bfloat16>(a, s);
}

cudaError_t launch_stream_norm(const float* x, const int64_t* rows, const float* w, void* out, int64_t n, int W, int n_real,
                               float eps, int out_f32, cudaStream_t s) {
  if (W % 8 != 0 || n_real < 1) return cudaErrorInvalidValue;
  if (n == 0) return cudaSuccess;
  const dim3 grid(static_cast<unsigned>(n)), block(row_threads(W));
  return out_f32 ? launch_pdl(stream_norm_kernel<float>, grid, block, 0, s, x, rows, w, reinterpret_cast<float*>(out), W,
                              n_real, eps)
                 : launch_pdl(stream_norm_kernel<__nv_bfloat16>, grid, block, 0, s, x, rows, w,
                              reinterpret_cast<__nv_bfloat16*>(out), W, n_real, eps);
}

}  // namespace tdb
