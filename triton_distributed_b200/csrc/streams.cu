// Several residual streams (hyper-connections): one kernel between two sublayers mixes the streams, adds the last sublayer's output
// to each of them and norms the mixture that the next sublayer reads.  One block per token; a column's streams stay in registers, so
// the streams are read and written once.  The first call of a model starts them from the embedding table, the last one sums them
// for the rows that are asked for and stores nothing.
#include "tdb/launch.cuh"
#include "tdb/streams.h"
#include "tdb/vec.cuh"

namespace tdb {

namespace {

template <typename T, int MAXS>
__global__ void hyper_step_kernel(const HyperArgs p) {
  __shared__ float red[32];
  __shared__ float s_mix[MAXS * MAXS], s_out[MAXS], s_in[MAXS];
  extern __shared__ float row[];       // [W]
  pdl_wait();
  pdl_launch_dependents();
  const int64_t t = p.rows != nullptr ? p.rows[blockIdx.x] : blockIdx.x;
  const int S = p.S;
  const T* y = reinterpret_cast<const T*>(p.y) + t * p.W;
  const T* y2 = reinterpret_cast<const T*>(p.y2) + t * p.W;
  for (int i = threadIdx.x; i < S * S; i += blockDim.x) s_mix[i] = p.y != nullptr ? p.mix[i] : 0.f;
  if (threadIdx.x < S) {
    s_out[threadIdx.x] = p.y != nullptr ? p.out[threadIdx.x] : 0.f;
    s_in[threadIdx.x] = p.h != nullptr ? p.in[threadIdx.x] : 0.f;
  }
  float f1 = 1.f, f2 = 0.f;
  if (p.y2 != nullptr) {
    float a = 0.f, b = 0.f;
    for (int c = threadIdx.x * 8; c < p.W; c += blockDim.x * 8) {
      float u[8], v[8];
      load8(y + c, u);
      load8(y2 + c, v);
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        a += u[i] * u[i];
        b += v[i] * v[i];
      }
    }
    f1 = 0.5f / sqrtf(block_reduce_sum(a, red) / p.n_real + p.eps);
    f2 = 0.5f / sqrtf(block_reduce_sum(b, red) / p.n_real + p.eps);
  }
  __syncthreads();
  int64_t id = 0;
  if (p.ids != nullptr) {
    id = p.ids[t];
    if (id < 0 || id >= p.vocab) id = 0;
  }
  float* x = p.x + t * S * p.W;
  float ss = 0.f;
  for (int c = threadIdx.x * 8; c < p.W; c += blockDim.x * 8) {
    float xs[MAXS][8], u[8] = {}, o[8] = {};
    if (p.ids != nullptr) {
      load8(reinterpret_cast<const T*>(p.table) + id * p.W + c, xs[0]);
    } else {
#pragma unroll
      for (int s = 0; s < MAXS; ++s)
        if (s < S) load8(x + static_cast<int64_t>(s) * p.W + c, xs[s]);
    }
    if (p.y != nullptr) {
      load8(y + c, o);
      if (p.y2 != nullptr) {
        float b[8], w1[8], w2[8];
        load8(y2 + c, b);
        load8(p.y_w + c, w1);
        load8(p.y2_w + c, w2);
#pragma unroll
        for (int i = 0; i < 8; ++i) o[i] = o[i] * f1 * w1[i] + b[i] * f2 * w2[i];
      }
    }
#pragma unroll
    for (int d = 0; d < MAXS; ++d) {
      if (d >= S) break;
      float v[8];
      if (p.ids != nullptr) {
#pragma unroll
        for (int i = 0; i < 8; ++i) v[i] = xs[0][i];
      } else if (p.y == nullptr) {
#pragma unroll
        for (int i = 0; i < 8; ++i) v[i] = xs[d][i];
      } else {
        const float w = s_out[d];
#pragma unroll
        for (int i = 0; i < 8; ++i) v[i] = w * o[i];
#pragma unroll
        for (int s = 0; s < MAXS; ++s) {
          if (s >= S) break;
          const float m = s_mix[s * S + d];
#pragma unroll
          for (int i = 0; i < 8; ++i) v[i] = fmaf(m, xs[s][i], v[i]);
        }
      }
      if (p.store) store8(x + static_cast<int64_t>(d) * p.W + c, v);
      const float w = s_in[d];
#pragma unroll
      for (int i = 0; i < 8; ++i) u[i] = fmaf(w, v[i], u[i]);
    }
#pragma unroll
    for (int i = 0; i < 8; ++i) ss += u[i] * u[i];
    store8(row + c, u);
  }
  if (p.h == nullptr) return;
  const float inv = 1.f / sqrtf(block_reduce_sum(ss, red) / p.n_real + p.eps);
  T* h = reinterpret_cast<T*>(p.h) + static_cast<int64_t>(blockIdx.x) * p.W;
  for (int c = threadIdx.x * 8; c < p.W; c += blockDim.x * 8) {
    float a[8], w[8];
    load8(row + c, a);
    load8(p.w + c, w);
#pragma unroll
    for (int i = 0; i < 8; ++i) a[i] *= inv * w[i];
    store8(h + c, a);
  }
}

template <typename T, int MAXS>
cudaError_t launch_s(const HyperArgs& a, cudaStream_t s) {
  const size_t smem = static_cast<size_t>(a.W) * 4;
  static SmemOptIn opt;
  if (smem > 40 * 1024) {
    cudaError_t e = opt.ensure(hyper_step_kernel<T, MAXS>, 200 * 1024);
    if (e != cudaSuccess) return e;
  }
  const int vec = a.W / 8;
  // few tokens: as many loads in flight per token as a block allows
  const int most = a.n <= 148 && MAXS <= 4 ? 512 : 256;
  const int threads = vec >= most ? most : vec >= 256 ? 256 : vec >= 128 ? 128 : 64;
  return launch_pdl(hyper_step_kernel<T, MAXS>, dim3(static_cast<unsigned>(a.n)), dim3(threads), smem, s, a);
}
template <typename T>
cudaError_t launch_t(const HyperArgs& a, cudaStream_t s) {
  switch (a.S) {
    case 1: return launch_s<T, 1>(a, s);
    case 2: return launch_s<T, 2>(a, s);
    case 3: return launch_s<T, 3>(a, s);
    case 4: return launch_s<T, 4>(a, s);
    default: return a.S <= 8 ? launch_s<T, 8>(a, s) : launch_s<T, 16>(a, s);
  }
}

// ---------------------------------------------------------------------------------------------------- gated activations
template <int ACT>
TDB_DEVICE float activate(float z) {
  if constexpr (ACT == 0) return z * sigmoid_f32(z);
  else return gelu_tanh_f32(z);
}

template <typename T, int ACT>
__global__ void __launch_bounds__(256) gated_act_kernel(const T* __restrict__ in, T* __restrict__ out, int64_t rows, int F) {
  pdl_wait();
  pdl_launch_dependents();
  const int nv = F >> 3;
  const int64_t total = rows * nv;
  for (int64_t v = blockIdx.x * static_cast<int64_t>(256) + threadIdx.x; v < total; v += static_cast<int64_t>(gridDim.x) * 256) {
    const int64_t r = v / nv;
    const int c = static_cast<int>(v - r * nv) * 8;
    float g[8], u[8];
    load8(in + r * 2 * F + c, g);
    load8(in + r * 2 * F + F + c, u);
#pragma unroll
    for (int i = 0; i < 8; ++i) g[i] = activate<ACT>(g[i]) * u[i];
    store8(out + r * F + c, g);
  }
}

}  // namespace

cudaError_t launch_hyper_step(const HyperArgs& a, cudaStream_t s) {
  if (a.W % 8 != 0 || a.n_real < 1 || a.S < 1 || a.S > 16 || a.W > 50 * 1024 || (a.y != nullptr && (a.mix == nullptr || a.out == nullptr)) ||
      (a.y2 != nullptr && (a.y == nullptr || a.y_w == nullptr || a.y2_w == nullptr)) || (a.h != nullptr && (a.in == nullptr || a.w == nullptr)) ||
      (a.ids != nullptr && a.y != nullptr) || (a.rows != nullptr && a.store))
    return cudaErrorInvalidValue;
  if (a.n == 0) return cudaSuccess;
  return a.is_f32 ? launch_t<float>(a, s) : launch_t<__nv_bfloat16>(a, s);
}

cudaError_t launch_gated_act(const void* in, void* out, int64_t rows, int F, int act, int is_f32, cudaStream_t s) {
  if (F % 8 != 0 || act < 0 || act > 1) return cudaErrorInvalidValue;
  if (rows == 0) return cudaSuccess;
  const int64_t blocks = (rows * (F / 8) + 255) / 256;
  const dim3 grid(static_cast<unsigned>(blocks < 148 * 16 ? blocks : 148 * 16)), block(256);
  auto go = [&](auto kernel, auto* i, auto* o) { return launch_pdl(kernel, grid, block, 0, s, i, o, rows, F); };
  if (is_f32) {
    auto* i = reinterpret_cast<const float*>(in);
    auto* o = reinterpret_cast<float*>(out);
    return act == 0 ? go(gated_act_kernel<float, 0>, i, o) : go(gated_act_kernel<float, 1>, i, o);
  }
  auto* i = reinterpret_cast<const __nv_bfloat16*>(in);
  auto* o = reinterpret_cast<__nv_bfloat16*>(out);
  return act == 0 ? go(gated_act_kernel<__nv_bfloat16, 0>, i, o) : go(gated_act_kernel<__nv_bfloat16, 1>, i, o);
}

}  // namespace tdb
