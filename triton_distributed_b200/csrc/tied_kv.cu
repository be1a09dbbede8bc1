// Attention over a tied KV cache: the values of a token are its keys as projected, before the key norm, and the norm runs
// over the whole projection (all heads at once).  A normed key is then raw_key * f * weight with ONE factor f per token,
// so the cache stores the raw key once plus the fp32 factor: the key norm's weight is folded into the query, the factor
// multiplies the token's score, and the same bytes serve as the value.  That halves the cache and the decode stream.
//
//   qk_norm_tied_kernel     one block per token: both sums of squares, the scaled query, the raw key row and its factor
//                           into up to two cache destinations
//   tied_attn_simple_kernel fp32 arithmetic, one warp per (token, head), any head dim up to 1024, fp32 or bf16 tensors:
//                           the 32-bit path and the check of the tensor-core kernels in attn.cu / attn_sm100.cu; values
//                           may be a leading part of the row (latent attention)
#include "tdb/attn.h"
#include "tdb/hybrid.h"
#include "tdb/launch.cuh"
#include "tdb/vec.cuh"

namespace tdb {

namespace {

template <typename T>
TDB_DEVICE float row_sumsq(const T* row, int n) {
  float ss = 0.f;
  for (int c = threadIdx.x * 8; c < n; c += blockDim.x * 8) {
    float f[8];
    load8(row + c, f);
#pragma unroll
    for (int i = 0; i < 8; ++i) ss += f[i] * f[i];
  }
  return ss;
}

template <typename T>
__global__ void qk_norm_tied_kernel(const QkNormArgs p) {
  __shared__ float red[32];
  pdl_wait();
  pdl_launch_dependents();
  const int64_t t = blockIdx.x;
  const T* q = reinterpret_cast<const T*>(p.qk) + t * p.ld;
  const T* k = q + p.Nq;
  float sq, sk;
  if (p.sumsq != nullptr) {
    sq = p.sumsq[2 * t];
    sk = p.sumsq[2 * t + 1];
  } else {
    sq = block_reduce_sum(row_sumsq(q, p.Nq), red);
    sk = block_reduce_sum(row_sumsq(k, p.Nk), red);
  }
  const float fq = 1.f / sqrtf(sq / p.nq_real + p.eps);
  const float fk = 1.f / sqrtf(sk / p.nk_real + p.eps);
  T* qo = reinterpret_cast<T*>(p.q_out) + t * p.Nq;
  for (int c = threadIdx.x * 8; c < p.Nq; c += blockDim.x * 8) {
    float f[8], w[8];
    load8(q + c, f);
    load8(p.qw + c, w);
#pragma unroll
    for (int i = 0; i < 8; ++i) f[i] *= fq * w[i];
    store8(qo + c, f);
  }
  const int64_t ra = p.rows_a[t];
  const int64_t rb = p.k_b != nullptr ? p.rows_b[t] : -1;
  const bool oka = ra >= 0 && ra < p.cap_a, okb = rb >= 0 && rb < p.cap_b;
  T* ka = reinterpret_cast<T*>(p.k_a) + ra * p.Nk;
  T* kb = reinterpret_cast<T*>(p.k_b) + rb * p.Nk;
  for (int c = threadIdx.x * 8; c < p.Nk; c += blockDim.x * 8) {
    float f[8];
    load8(k + c, f);
    if (oka) store8(ka + c, f);
    if (okb) store8(kb + c, f);
  }
  if (threadIdx.x == 0) {
    if (oka) p.scale_a[ra] = fk;
    if (okb) p.scale_b[rb] = fk;
  }
}

template <typename T>
__global__ void qk_sumsq_kernel(const QkNormArgs p, float* out) {
  __shared__ float red[32];
  const int64_t t = blockIdx.x;
  const T* q = reinterpret_cast<const T*>(p.qk) + t * p.ld;
  const float sq = block_reduce_sum(row_sumsq(q, p.Nq), red);
  const float sk = block_reduce_sum(row_sumsq(q + p.Nq, p.Nk), red);
  if (threadIdx.x == 0) {
    out[2 * t] = sq;
    out[2 * t + 1] = sk;
  }
}

constexpr int kSimpleMaxD = 1024;

template <typename T, typename TO, int kPer>     // kPer elements of a row per lane
__global__ void __launch_bounds__(128) tied_attn_simple_kernel(const TiedSimpleArgs p) {
  pdl_wait();
  pdl_launch_dependents();
  const int64_t wid = static_cast<int64_t>(blockIdx.x) * 4 + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (wid >= p.T * p.Hq) return;
  const int64_t t = wid / p.Hq;
  const int h = static_cast<int>(wid - t * p.Hq);
  const int hkv = h / (p.Hq / p.Hkv);
  const int per = (p.D + 31) / 32;
  const T* q = reinterpret_cast<const T*>(p.q) + wid * p.D;
  float qf[kPer], o[kPer];
#pragma unroll
  for (int i = 0; i < kPer; ++i) {
    const int d = lane + 32 * i;
    qf[i] = (i < per && d < p.D) ? to_f32(q[d]) : 0.f;
    o[i] = 0.f;
  }
  const int64_t row0 = p.row0[t];
  const int n = p.n_keys[t];
  // the sink is simply where the running maximum and the denominator start
  float m = p.epi.sink != nullptr ? p.epi.sink[h] : -INFINITY;
  float l = p.epi.sink != nullptr ? 1.f : 0.f;
  for (int j = 0; j < n; ++j) {
    const T* kr = reinterpret_cast<const T*>(p.k) + ((row0 + j) * p.Hkv + hkv) * p.D;
    float kf[kPer];
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < kPer; ++i) {
      const int d = lane + 32 * i;
      kf[i] = (i < per && d < p.D) ? to_f32(kr[d]) : 0.f;
      s = fmaf(qf[i], kf[i], s);
    }
    s = warp_sum(s) * (p.k_scale != nullptr ? p.k_scale[row0 + j] * p.scale : p.scale);
    if (p.softcap > 0.f) s = p.softcap * tanhf(s / p.softcap);
    if (p.v != nullptr) {
      const T* vr = reinterpret_cast<const T*>(p.v) + ((row0 + j) * p.Hkv + hkv) * p.Dv;
#pragma unroll
      for (int i = 0; i < kPer; ++i) {
        const int d = lane + 32 * i;
        kf[i] = (i < per && d < p.Dv) ? to_f32(vr[d]) : 0.f;
      }
    }
    const float mn = fmaxf(m, s);
    const float corr = expf(m - mn), e = expf(s - mn);   // m = -inf -> 0
    l = l * corr + e;
    m = mn;
#pragma unroll
    for (int i = 0; i < kPer; ++i) o[i] = fmaf(e, kf[i], o[i] * corr);
  }
  const float inv = l > 0.f ? 1.f / l : 0.f;
  TO* out = reinterpret_cast<TO*>(p.out) + wid * p.Dv;
  const T* gate = p.epi.gate != nullptr
                      ? reinterpret_cast<const T*>(p.epi.gate) + t * p.epi.ld_gate + static_cast<int64_t>(h) * p.Dv
                      : nullptr;
#pragma unroll
  for (int i = 0; i < kPer; ++i) {
    const int d = lane + 32 * i;
    if (i < per && d < p.Dv) {
      const float g = gate != nullptr ? sigmoid_f32(to_f32(gate[d])) : 1.f;
      out[d] = from_f32<TO>(o[i] * inv * g);
    }
  }
}

template <typename T, typename TO>
cudaError_t launch_simple(const TiedSimpleArgs& a, cudaStream_t s) {
  const dim3 grid(static_cast<unsigned>((a.T * a.Hq + 3) / 4));
  return a.D <= 256   ? launch_pdl(tied_attn_simple_kernel<T, TO, 8>, grid, dim3(128), 0, s, a)
         : a.D <= 512 ? launch_pdl(tied_attn_simple_kernel<T, TO, 16>, grid, dim3(128), 0, s, a)
                      : launch_pdl(tied_attn_simple_kernel<T, TO, kSimpleMaxD / 32>, grid, dim3(128), 0, s, a);
}

int norm_threads(int n) { return n >= 2048 ? 256 : n >= 1024 ? 128 : 64; }

bool qk_args_ok(const QkNormArgs& a) {
  return a.Nq % 8 == 0 && a.Nk % 8 == 0 && a.ld % 8 == 0 && a.nq_real > 0 && a.nk_real > 0;
}

}  // namespace

cudaError_t launch_qk_norm_tied(const QkNormArgs& a, cudaStream_t s) {
  if (!qk_args_ok(a) || a.rows_a == nullptr || (a.k_b != nullptr && a.rows_b == nullptr)) return cudaErrorInvalidValue;
  if (a.T == 0) return cudaSuccess;
  const dim3 grid(static_cast<unsigned>(a.T)), block(norm_threads(a.Nq));
  return a.is_f32 ? launch_pdl(qk_norm_tied_kernel<float>, grid, block, 0, s, a)
                  : launch_pdl(qk_norm_tied_kernel<__nv_bfloat16>, grid, block, 0, s, a);
}

cudaError_t launch_qk_sumsq(const QkNormArgs& a, float* out, cudaStream_t s) {
  if (!qk_args_ok(a)) return cudaErrorInvalidValue;
  if (a.T == 0) return cudaSuccess;
  if (a.is_f32)
    qk_sumsq_kernel<float><<<static_cast<unsigned>(a.T), norm_threads(a.Nq), 0, s>>>(a, out);
  else
    qk_sumsq_kernel<__nv_bfloat16><<<static_cast<unsigned>(a.T), norm_threads(a.Nq), 0, s>>>(a, out);
  return cudaGetLastError();
}

cudaError_t launch_tied_attn_simple(const TiedSimpleArgs& a, cudaStream_t s) {
  if (a.D < 1 || a.D > kSimpleMaxD || a.Dv < 1 || a.Dv > a.D || a.softcap < 0.f || a.Hkv < 1 || a.Hq % a.Hkv != 0) return cudaErrorInvalidValue;
  if (a.T == 0) return cudaSuccess;
  if (a.is_f32) return launch_simple<float, float>(a, s);
  return a.out_f32 ? launch_simple<__nv_bfloat16, float>(a, s) : launch_simple<__nv_bfloat16, __nv_bfloat16>(a, s);
}

}  // namespace tdb
