// Query / key preparation per head: RMS norm with a weight, rotation of the leading part of a head (either pairing, angles from a
// table), RMS norm without a weight; keys and values go straight to their cache rows.  One warp per (token, head), a lane holds
// D / 32 neighbouring elements; partners of the split-half pairing come through shared memory.
#include "tdb/launch.cuh"
#include "tdb/streams.h"
#include "tdb/vec.cuh"

namespace tdb {

namespace {

constexpr int kWarps = 4;

template <int E>
TDB_DEVICE void load_e(const __nv_bfloat16* p, float (&f)[E]) {
  if constexpr (E >= 8) {
#pragma unroll
    for (int i = 0; i < E; i += 8) load8(p + i, *reinterpret_cast<float (*)[8]>(f + i));
  } else if constexpr (E >= 2) {
#pragma unroll
    for (int i = 0; i < E; i += 2) {
      const float2 v = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(p + i));
      f[i] = v.x; f[i + 1] = v.y;
    }
  } else {
    f[0] = __bfloat162float(p[0]);
  }
}
template <int E>
TDB_DEVICE void load_e(const float* p, float (&f)[E]) {
#pragma unroll
  for (int i = 0; i < E; ++i) f[i] = p[i];
}
template <int E>
TDB_DEVICE void store_e(__nv_bfloat16* p, const float (&f)[E]) {
  if constexpr (E >= 8) {
#pragma unroll
    for (int i = 0; i < E; i += 8) store8(p + i, *reinterpret_cast<const float (*)[8]>(f + i));
  } else if constexpr (E >= 2) {
#pragma unroll
    for (int i = 0; i < E; i += 2) *reinterpret_cast<uint32_t*>(p + i) = pack_bf16x2(f[i], f[i + 1]);
  } else {
    p[0] = __float2bfloat16(f[0]);
  }
}
template <int E>
TDB_DEVICE void store_e(float* p, const float (&f)[E]) {
#pragma unroll
  for (int i = 0; i < E; ++i) p[i] = f[i];
}

template <typename T, int E>
__global__ void __launch_bounds__(kWarps * 32) head_prep_kernel(const HeadPrepArgs p) {
  __shared__ float sm[kWarps][32 * E];
  pdl_wait();
  pdl_launch_dependents();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int heads = p.H + 2 * p.G;
  const int64_t wid = static_cast<int64_t>(blockIdx.x) * kWarps + warp;
  if (wid >= p.T * heads) return;
  const int64_t t = wid / heads;
  const int u = static_cast<int>(wid - t * heads);
  const bool is_q = u < p.H, is_v = u >= p.H + p.G;
  const int64_t row = p.rows[t];
  T* dst;
  if (is_q) {
    dst = reinterpret_cast<T*>(p.q_out) + (t * p.H + u) * p.D;
  } else {
    if (row < 0 || row >= p.cap) return;
    dst = reinterpret_cast<T*>(is_v ? p.v_cache : p.k_cache) + (row * p.G + (u - p.H - (is_v ? p.G : 0))) * p.D;
  }
  const int d0 = lane * E;
  float x[E];
  load_e<E>(reinterpret_cast<const T*>(p.z) + t * p.ld + static_cast<int64_t>(u) * p.D + d0, x);
  if (!is_v) {
    const float* w = is_q ? p.q_w : p.k_w;
    if (w != nullptr) {
      float ss = 0.f;
#pragma unroll
      for (int i = 0; i < E; ++i) ss += x[i] * x[i];
      const float f = 1.f / sqrtf(warp_sum(ss) / p.d_real + p.eps);
#pragma unroll
      for (int i = 0; i < E; ++i) x[i] *= f * w[d0 + i];
    }
    if (p.rot > 0) {
      float* s = sm[warp];
#pragma unroll
      for (int i = 0; i < E; ++i) s[d0 + i] = x[i];
      __syncwarp();
      int64_t pos = p.pos[t];
      if (pos < 0 || pos >= p.n_pos) pos = 0;
      const float* cs = p.cos_sin + pos * p.rot_ld;
      const int half = p.rot >> 1;
#pragma unroll
      for (int i = 0; i < E; ++i) {
        const int d = d0 + i;
        if (d >= p.rot) continue;
        const bool second = p.interleaved ? (d & 1) : d >= half;
        const int pair = p.interleaved ? d >> 1 : (second ? d - half : d);
        const float other = s[p.interleaved ? d ^ 1 : (second ? d - half : d + half)];
        const float c = cs[2 * pair], sn = cs[2 * pair + 1];
        x[i] = second ? x[i] * c + other * sn : x[i] * c - other * sn;
      }
    }
    if (p.unit) {
      float ss = 0.f;
#pragma unroll
      for (int i = 0; i < E; ++i) ss += x[i] * x[i];
      const float f = 1.f / sqrtf(warp_sum(ss) / p.d_real + p.eps);
#pragma unroll
      for (int i = 0; i < E; ++i) x[i] *= f;
    }
  }
  store_e<E>(dst + d0, x);
}

template <typename T>
cudaError_t launch_prep(const HeadPrepArgs& a, cudaStream_t s) {
  const int64_t warps = a.T * (a.H + 2 * a.G);
  const dim3 grid(static_cast<unsigned>((warps + kWarps - 1) / kWarps)), block(kWarps * 32);
  switch (a.D / 32) {
    case 1: return launch_pdl(head_prep_kernel<T, 1>, grid, block, 0, s, a);
    case 2: return launch_pdl(head_prep_kernel<T, 2>, grid, block, 0, s, a);
    case 4: return launch_pdl(head_prep_kernel<T, 4>, grid, block, 0, s, a);
    case 8: return launch_pdl(head_prep_kernel<T, 8>, grid, block, 0, s, a);
    case 16: return launch_pdl(head_prep_kernel<T, 16>, grid, block, 0, s, a);
    case 32: return launch_pdl(head_prep_kernel<T, 32>, grid, block, 0, s, a);
    default: return cudaErrorInvalidValue;
  }
}

}  // namespace

cudaError_t launch_head_prep(const HeadPrepArgs& a, cudaStream_t s) {
  if (a.D % 32 != 0 || a.H < 1 || a.G < 1 || a.rot % 2 != 0 || a.rot > a.D || a.rot > a.rot_ld || a.d_real < 1 || a.ld % 8 != 0 ||
      (a.rot > 0 && a.cos_sin == nullptr))
    return cudaErrorInvalidValue;
  if (a.T == 0) return cudaSuccess;
  return a.is_f32 ? launch_prep<float>(a, s) : launch_prep<__nv_bfloat16>(a, s);
}

}  // namespace tdb
