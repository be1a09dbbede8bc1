// Experts of two forms with a weight w per (token, expert) pair:
//   squared ReLU  y = W_down relu(W_up (w h))^2: the up projection has no bias, so the weight can scale its OUTPUT
//   gated         y = w W_down (silu(W_gate h) * (W_up h)): the weight goes on the activation; identity experts (y = w h) have
//                 no matrices and are added by the down kernel
//
//   relu2_kernel        (relu(w * in + bias))^2 over rows, between the two grouped GEMMs of a prefill and in dense layers
//   expert_up_kernel    few tokens: one (token, chosen expert or shared expert) pair per blockIdx.y, weight rows streamed
//                       once with 16-byte loads, four rows per warp, activation fused
//   expert_down_kernel  sum over the token's experts and the gated shared expert in one pass, fp32 output
//
// A decode step is bound by the weights of the experts it touches; experts shared by tokens of the batch come from L2.
#include "tdb/hybrid.h"
#include "tdb/launch.cuh"
#include "tdb/vec.cuh"

namespace tdb {

namespace {

TDB_DEVICE float relu2(float v) {
  v = fmaxf(v, 0.f);
  return v * v;
}

template <typename T>
__global__ void relu2_kernel(const T* in, const float* __restrict__ w, const float* __restrict__ bias, T* out, int64_t rows, int F) {
  pdl_wait();
  pdl_launch_dependents();
  const int nv = F >> 3;
  for (int64_t v = blockIdx.x * static_cast<int64_t>(blockDim.x) + threadIdx.x; v < rows * nv;
       v += static_cast<int64_t>(gridDim.x) * blockDim.x) {
    const float s = w != nullptr ? w[v / nv] : 1.f;
    float f[8], b[8] = {};
    load8(in + v * 8, f);
    if (bias != nullptr) load8(bias + (v % nv) * 8, b);
#pragma unroll
    for (int i = 0; i < 8; ++i) f[i] = relu2(fmaf(s, f[i], b[i]));
    store8(out + v * 8, f);
  }
}

// Eight weights on their way from global memory.
template <typename T>
struct Raw8;
template <>
struct Raw8<__nv_bfloat16> {
  uint4 v;
  TDB_DEVICE void load(const __nv_bfloat16* p) { v = ld_nc_v4(p); }
  TDB_DEVICE float dot(const float (&x)[8]) const {
    const float2 a = unpack_bf16x2(v.x), b = unpack_bf16x2(v.y), c = unpack_bf16x2(v.z), d = unpack_bf16x2(v.w);
    return fmaf(a.x, x[0], fmaf(a.y, x[1], fmaf(b.x, x[2], b.y * x[3]))) + fmaf(c.x, x[4], fmaf(c.y, x[5], fmaf(d.x, x[6], d.y * x[7])));
  }
};
template <>
struct Raw8<float> {
  float4 a, b;
  TDB_DEVICE void load(const float* p) {
    a = reinterpret_cast<const float4*>(p)[0];
    b = reinterpret_cast<const float4*>(p)[1];
  }
  TDB_DEVICE float dot(const float (&x)[8]) const {
    return fmaf(a.x, x[0], fmaf(a.y, x[1], fmaf(a.z, x[2], a.w * x[3]))) + fmaf(b.x, x[4], fmaf(b.y, x[5], fmaf(b.z, x[6], b.w * x[7])));
  }
};

constexpr int kWarps = 8;
constexpr int kMaxTop = 64;

// acc[r] += row r of w (R rows, n columns) . xs over the warp's lanes (not reduced)
template <typename T, int R>
TDB_DEVICE void rows_dot(const T* w, int64_t ldw, const T* xs, int n, int rows, float (&acc)[R]) {
  const int lane = threadIdx.x & 31;
  constexpr int U = sizeof(T) == 2 ? 4 : 2;     // steps whose weight loads are in flight together
  for (int c0 = lane * 8; c0 < n; c0 += 256 * U) {
    Raw8<T> v[U][R];
#pragma unroll
    for (int u = 0; u < U; ++u)
#pragma unroll
      for (int r = 0; r < R; ++r)
        if (c0 + u * 256 < n) v[u][r].load(w + (r < rows ? r : 0) * ldw + c0 + u * 256);
#pragma unroll
    for (int u = 0; u < U; ++u) {
      if (c0 + u * 256 >= n) break;
      float x[8];
      load8(xs + c0 + u * 256, x);
#pragma unroll
      for (int r = 0; r < R; ++r) acc[r] += v[u][r].dot(x);
    }
  }
}

// The same for two rows of a gate matrix and the two rows `pair` elements further on: acc[0..1] gate, acc[2..3] up.
template <typename T>
TDB_DEVICE void rows_dot_pair(const T* w, int64_t pair, int64_t ldw, const T* xs, int n, int rows, float (&acc)[4]) {
  const int lane = threadIdx.x & 31;
  constexpr int U = sizeof(T) == 2 ? 4 : 2;
  for (int c0 = lane * 8; c0 < n; c0 += 256 * U) {
    Raw8<T> v[U][4];
#pragma unroll
    for (int u = 0; u < U; ++u)
#pragma unroll
      for (int r = 0; r < 4; ++r)
        if (c0 + u * 256 < n) v[u][r].load(w + (r >> 1) * pair + ((r & 1) < rows ? (r & 1) : 0) * ldw + c0 + u * 256);
#pragma unroll
    for (int u = 0; u < U; ++u) {
      if (c0 + u * 256 >= n) break;
      float x[8];
      load8(xs + c0 + u * 256, x);
#pragma unroll
      for (int r = 0; r < 4; ++r) acc[r] += v[u][r].dot(x);
    }
  }
}

constexpr int kUpRows = 4;
template <typename T, bool GATED>
__global__ void __launch_bounds__(kWarps * 32) expert_up_kernel(const ExpertGemvArgs p) {
  extern __shared__ __align__(16) uint8_t smem[];
  T* xs = reinterpret_cast<T*>(smem);          // [K]
  const int slots = p.top + (p.shared_up != nullptr ? 1 : 0);
  const int64_t t = blockIdx.y / slots;
  const int s = blockIdx.y - static_cast<int>(t) * slots;
  const bool shared = s == p.top;
  const int F = shared ? p.Fs : p.F;
  constexpr int kRows = GATED ? kUpRows / 2 : kUpRows;      // output rows per warp: a gated one takes two weight rows
  const int r0 = (blockIdx.x * kWarps + (threadIdx.x >> 5)) * kRows;
  pdl_wait();
  pdl_launch_dependents();
  if (blockIdx.x * kWarps * kRows >= F) return;
  int e = 0;
  float wgt = 1.f;
  if (!shared) {
    e = p.ids[t * p.top + s];
    wgt = p.weights[t * p.top + s];
    if (GATED && e >= p.E) return;                            // identity
    if (e < 0 || e >= p.E) e = 0, wgt = 0.f;
  }
  const T* x = reinterpret_cast<const T*>(p.x) + t * p.K;
  for (int c = threadIdx.x * 8; c < p.K; c += kWarps * 256) {
    float f[8];
    load8(x + c, f);
    store8(xs + c, f);
  }
  const T* w = shared ? reinterpret_cast<const T*>(p.shared_up)
                      : reinterpret_cast<const T*>(p.up) + static_cast<int64_t>(e) * p.F * p.K * (GATED ? 2 : 1);
  __syncthreads();
  if (r0 >= F) return;
  const int rows = min(kRows, F - r0);
  T* act = reinterpret_cast<T*>(p.act) + t * (static_cast<int64_t>(p.top) * p.F + p.Fs) + static_cast<int64_t>(s) * p.F;
  if constexpr (GATED) {
    // rows r0, r0 + 1 of the gate and the same rows of up, F rows further down (all loads of the four in flight together)
    float acc[kUpRows] = {};
    rows_dot_pair<T>(w + static_cast<int64_t>(r0) * p.K, static_cast<int64_t>(F) * p.K, p.K, xs, p.K, rows, acc);
#pragma unroll
    for (int r = 0; r < kRows; ++r) {
      const float g = warp_sum(acc[r]), u = warp_sum(acc[kRows + r]);
      if ((threadIdx.x & 31) == r && r < rows) act[r0 + r] = from_f32<T>(wgt * g * sigmoid_f32(g) * u);
    }
    return;
  }
  float acc[kUpRows] = {};
  rows_dot<T, kUpRows>(w + static_cast<int64_t>(r0) * p.K, p.K, xs, p.K, rows, acc);
#pragma unroll
  for (int r = 0; r < kUpRows; ++r) {
    const float v = warp_sum(acc[r]);
    if ((threadIdx.x & 31) == r && r < rows) act[r0 + r] = from_f32<T>(relu2(wgt * v));
  }
}

constexpr int kDownRows = 2;
template <typename T, int U>     // U vectors of eight weights per row in flight: 8 for one or two tokens, where CTAs are few
__global__ void __launch_bounds__(kWarps * 32) expert_down_kernel(const ExpertGemvArgs p) {
  extern __shared__ __align__(16) uint8_t smem[];
  T* as = reinterpret_cast<T*>(smem);          // [top * F + Fs]
  __shared__ int s_ids[kMaxTop];               // -1: identity
  __shared__ float s_self;                     // what multiplies the token's own row
  const int64_t t = blockIdx.y;
  const int n_act = p.top * p.F + p.Fs;
  pdl_wait();
  pdl_launch_dependents();
  if (threadIdx.x < p.top) {
    const int e = p.ids[t * p.top + threadIdx.x];
    // an id out of range got the activation zero; that of an identity expert was not written
    s_ids[threadIdx.x] = (e >= 0 && e < p.E) ? e : (p.identity > 0 && e >= p.E && e < p.E + p.identity) ? -1 : 0;
  }
  if (threadIdx.x == 0) {
    float w = 0.f;
    if (p.identity > 0 && !p.skip_identity)
      for (int s = 0; s < p.top; ++s) {
        const int e = p.ids[t * p.top + s];
        if (e >= p.E && e < p.E + p.identity) w += p.weights[t * p.top + s];
      }
    s_self = w;
  }
  const T* act = reinterpret_cast<const T*>(p.act) + t * n_act;
  for (int c = threadIdx.x * 8; c < n_act; c += kWarps * 256) {
    float f[8];
    load8(act + c, f);
    store8(as + c, f);
  }
  __syncthreads();
  const int r0 = (blockIdx.x * kWarps + (threadIdx.x >> 5)) * kDownRows;
  if (r0 >= p.K) return;
  const int rows = min(kDownRows, p.K - r0);
  const float gate = p.shared_gate != nullptr ? p.shared_gate[t] : 1.f;
  const int n_routed = p.top * p.F;
  float acc[kDownRows] = {};
  // one loop over the activations of all experts of the token, so that the loads of several experts are in flight together
  // (a vector of eight never crosses an expert: F is a multiple of eight)
  for (int c0 = (threadIdx.x & 31) * 8; c0 < n_act; c0 += 256 * U) {
    Raw8<T> v[U][kDownRows];
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int c = c0 + u * 256;
      if (c >= n_act) break;
      const bool routed = c < n_routed;
      const int s = routed ? c / p.F : 0;
      if (routed && s_ids[s] < 0) continue;
      const T* w = routed ? reinterpret_cast<const T*>(p.down) + (static_cast<int64_t>(s_ids[s]) * p.K + r0) * p.F + (c - s * p.F)
                          : reinterpret_cast<const T*>(p.shared_down) + static_cast<int64_t>(r0) * p.Fs + (c - n_routed);
      const int64_t ldw = routed ? p.F : p.Fs;
#pragma unroll
      for (int r = 0; r < kDownRows; ++r) v[u][r].load(w + (r < rows ? r : 0) * ldw);
    }
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int c = c0 + u * 256;
      if (c >= n_act) break;
      if (c < n_routed && s_ids[c / p.F] < 0) continue;
      const float f = c < n_routed ? 1.f : gate;
      float x[8];
      load8(as + c, x);
#pragma unroll
      for (int r = 0; r < kDownRows; ++r) acc[r] = fmaf(f, v[u][r].dot(x), acc[r]);
    }
  }
#pragma unroll
  for (int r = 0; r < kDownRows; ++r) {
    float v = warp_sum(acc[r]);
    if ((threadIdx.x & 31) == r && r < rows) {
      if (s_self != 0.f) v = fmaf(s_self, to_f32(reinterpret_cast<const T*>(p.x)[t * p.K + r0 + r]), v);
      p.y[t * p.K + r0 + r] = v;
    }
  }
}

template <typename T>
cudaError_t launch_experts(const ExpertGemvArgs& a, cudaStream_t s) {
  const int slots = a.top + (a.shared_up != nullptr ? 1 : 0);
  const size_t smem_up = static_cast<size_t>(a.K) * sizeof(T);
  const size_t smem_dn = static_cast<size_t>(a.top * a.F + a.Fs) * sizeof(T);
  if (smem_up > 200 * 1024 || smem_dn > 200 * 1024) return cudaErrorInvalidValue;
  const bool few = a.T <= 2 && sizeof(T) == 2;
  static SmemOptIn up, upg, dn, dn8;
  cudaError_t e = a.gated ? upg.ensure(expert_up_kernel<T, true>, 200 * 1024) : up.ensure(expert_up_kernel<T, false>, 200 * 1024);
  if (e != cudaSuccess) return e;
  e = few ? dn8.ensure(expert_down_kernel<T, 8>, 200 * 1024) : dn.ensure(expert_down_kernel<T, 4>, 200 * 1024);
  if (e != cudaSuccess) return e;
  const int fmax = a.F > a.Fs ? a.F : a.Fs;
  const int per_up = kWarps * kUpRows / (a.gated ? 2 : 1), per_dn = kWarps * kDownRows;
  const dim3 grid_up((fmax + per_up - 1) / per_up, static_cast<unsigned>(a.T * slots));
  e = a.gated ? launch_pdl(expert_up_kernel<T, true>, grid_up, dim3(kWarps * 32), smem_up, s, a)
              : launch_pdl(expert_up_kernel<T, false>, grid_up, dim3(kWarps * 32), smem_up, s, a);
  if (e != cudaSuccess) return e;
  const dim3 grid_dn((a.K + per_dn - 1) / per_dn, static_cast<unsigned>(a.T));
  return few ? launch_pdl(expert_down_kernel<T, 8>, grid_dn, dim3(kWarps * 32), smem_dn, s, a)
             : launch_pdl(expert_down_kernel<T, 4>, grid_dn, dim3(kWarps * 32), smem_dn, s, a);
}

}  // namespace

cudaError_t launch_relu2(const void* in, const float* row_weight, const float* bias, void* out, int64_t rows, int F, int is_f32,
                         cudaStream_t s) {
  if (F % 8 != 0) return cudaErrorInvalidValue;
  if (rows == 0) return cudaSuccess;
  const int64_t blocks = (rows * (F / 8) + 255) / 256;
  const dim3 grid(static_cast<unsigned>(blocks < 148 * 16 ? blocks : 148 * 16));
  return is_f32 ? launch_pdl(relu2_kernel<float>, grid, dim3(256), 0, s, reinterpret_cast<const float*>(in), row_weight, bias,
                             reinterpret_cast<float*>(out), rows, F)
                : launch_pdl(relu2_kernel<__nv_bfloat16>, grid, dim3(256), 0, s, reinterpret_cast<const __nv_bfloat16*>(in),
                             row_weight, bias, reinterpret_cast<__nv_bfloat16*>(out), rows, F);
}

cudaError_t launch_expert_gemv(const ExpertGemvArgs& a, cudaStream_t s) {
  if (a.K % 8 != 0 || a.F % 8 != 0 || a.Fs % 8 != 0 || a.top < 1 || a.top > kMaxTop) return cudaErrorInvalidValue;
  if ((a.shared_up == nullptr) != (a.shared_down == nullptr) || (a.shared_up == nullptr && a.Fs != 0)) return cudaErrorInvalidValue;
  if (a.T * (a.top + 1) > 65535 || (a.identity > 0 && !a.gated)) return cudaErrorInvalidValue;
  if (a.T == 0) return cudaSuccess;
  return a.is_f32 ? launch_experts<float>(a, s) : launch_experts<__nv_bfloat16>(a, s);
}

}  // namespace tdb
