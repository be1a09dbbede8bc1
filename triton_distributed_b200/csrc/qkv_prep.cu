// Projected queries, keys and values -> what attention reads, in one launch: biases, RMS norms over the whole projection, rotation,
// and the rows of the cache (and of a packed copy).  One block per token, a thread holds eight neighbouring elements; the partner
// of a rotated element is recomputed from the projection instead of being exchanged.
#include "tdb/launch.cuh"
#include "tdb/vec.cuh"
#include "tdb/window.h"

namespace tdb {

namespace {

// Eight elements of a projection row with their bias.
template <typename T>
TDB_DEVICE void load_biased(const T* z, const float* bias, float (&f)[8]) {
  load8(z, f);
  if (bias != nullptr) {
    float b[8];
    load8(bias, b);
#pragma unroll
    for (int i = 0; i < 8; ++i) f[i] += b[i];
  }
}

template <typename T>
__global__ void qkv_prep_kernel(const QkvPrepArgs p) {
  __shared__ float red[2][32];
  pdl_wait();
  pdl_launch_dependents();
  const int64_t t = blockIdx.x;
  const int Nq = p.Hq * p.dk, Nk = p.Gk * p.dk, Nv = p.G * p.dv;
  const T* z = reinterpret_cast<const T*>(p.z) + t * p.ld;
  float fq = 1.f, fk = 1.f;
  if (p.q_w != nullptr) {
    float sq = 0.f, sk = 0.f;
    if (p.sumsq != nullptr) {
      sq = p.sumsq[2 * t];
      sk = p.sumsq[2 * t + 1];
    } else {
      for (int c = threadIdx.x * 8; c < Nq + Nk; c += blockDim.x * 8) {
        float f[8], s = 0.f;
        load_biased(z + c, p.bias != nullptr ? p.bias + c : nullptr, f);
#pragma unroll
        for (int i = 0; i < 8; ++i) s += f[i] * f[i];
        if (c < Nq) sq += s;
        else sk += s;
      }
      sq = block_reduce_sum(sq, red[0]);
      sk = block_reduce_sum(sk, red[1]);
    }
    fq = 1.f / sqrtf(sq / p.nq_real + p.eps);
    fk = 1.f / sqrtf(sk / p.nk_real + p.eps);
  }
  const int64_t ra = p.rows_a[t], rb = p.k_b != nullptr ? p.rows_b[t] : -1;
  const bool oka = ra >= 0 && ra < p.cap_a, okb = rb >= 0 && rb < p.cap_b;
  const float* cs = nullptr;
  if (p.rot > 0) {
    int64_t pos = p.pos[t];
    if (pos < 0 || pos >= p.n_pos) pos = 0;
    cs = p.cos_sin + pos * p.rot_ld;
  }
  const int half = p.rot >> 1;
  for (int c = threadIdx.x * 8; c < Nq + Nk + Nv; c += blockDim.x * 8) {
    float f[8];
    load_biased(z + c, p.bias != nullptr ? p.bias + c : nullptr, f);
    if (c >= Nq + Nk) {
      const int cv = c - Nq - Nk;
      if (oka) store8(reinterpret_cast<T*>(p.v_a) + ra * Nv + cv, f);
      if (okb) store8(reinterpret_cast<T*>(p.v_b) + rb * Nv + cv, f);
      continue;
    }
    const bool is_q = c < Nq;
    const float* w = is_q ? p.q_w : p.k_w;
    const int cw = is_q ? c : c - Nq;             // inside q or k
    const float n = is_q ? fq : fk;
    if (w != nullptr) {
      float g[8];
      load8(w + cw, g);
#pragma unroll
      for (int i = 0; i < 8; ++i) f[i] *= n * g[i];
    }
    const int d0 = cw % p.dk;
    if (d0 < p.rot) {
      auto turn = [&](int i, float other, int pair, bool second) {
        const float co = cs[2 * pair], si = cs[2 * pair + 1];
        f[i] = second ? f[i] * co + other * si : f[i] * co - other * si;
      };
      if (half % 8 == 0) {                        // the eight partners are neighbours as well
        const bool second = d0 >= half;
        const int off = second ? -half : half;
        float o[8];
        load_biased(z + c + off, p.bias != nullptr ? p.bias + c + off : nullptr, o);
        if (w != nullptr) {
          float g[8];
          load8(w + cw + off, g);
#pragma unroll
          for (int i = 0; i < 8; ++i) o[i] *= n * g[i];
        }
#pragma unroll
        for (int i = 0; i < 8; ++i) turn(i, o[i], d0 + i - (second ? half : 0), second);
      } else {
#pragma unroll
        for (int i = 0; i < 8; ++i) {
          const int d = d0 + i;
          if (d >= p.rot) continue;
          const bool second = d >= half;
          const int off = second ? -half : half;
          float other = to_f32(z[c + i + off]);
          if (p.bias != nullptr) other += p.bias[c + i + off];
          if (w != nullptr) other *= n * w[cw + i + off];
          turn(i, other, second ? d - half : d, second);
        }
      }
    }
    if (is_q) {
      store8(reinterpret_cast<T*>(p.q_out) + t * Nq + cw, f);
    } else {
      if (oka) store8(reinterpret_cast<T*>(p.k_a) + ra * Nk + cw, f);
      if (okb) store8(reinterpret_cast<T*>(p.k_b) + rb * Nk + cw, f);
    }
  }
}

}  // namespace

cudaError_t launch_qkv_prep(const QkvPrepArgs& a, cudaStream_t s) {
  if (a.dk < 8 || a.dv < 8 || a.dk % 8 != 0 || a.dv % 8 != 0 || a.ld % 8 != 0 || a.Hq < 1 || a.Gk < 1 || a.G < 1 || a.rot % 2 != 0 || a.rot < 0 ||
      a.rot > a.dk || (a.rot > 0 && (a.cos_sin == nullptr || a.rot > a.rot_ld)) || (a.q_w == nullptr) != (a.k_w == nullptr) ||
      (a.q_w != nullptr && (a.nq_real < 1 || a.nk_real < 1)) || a.rows_a == nullptr || (a.k_b != nullptr && a.rows_b == nullptr))
    return cudaErrorInvalidValue;
  if (a.T == 0) return cudaSuccess;
  const int n = (a.Hq + a.Gk) * a.dk + a.G * a.dv;
  const dim3 grid(static_cast<unsigned>(a.T)), block(n >= 4096 ? 256 : n >= 1024 ? 128 : 64);
  return a.is_f32 ? launch_pdl(qkv_prep_kernel<float>, grid, block, 0, s, a) : launch_pdl(qkv_prep_kernel<__nv_bfloat16>, grid, block, 0, s, a);
}

}  // namespace tdb
