// Latent attention: what surrounds the attention kernels (see latent.h for the two forms).
//
//   latent_rotate_kernel   prompts: one block per token.  Warp 0 norms the latent, rotates the shared key part and writes the
//                          row to the cache and to the step's packed context; the other warps rotate the queries in place.
//   latent_absorb_kernel   decoding: per-head linear map q' = W_uk^T q on mma.sync, 16 tokens x 64 latent columns per CTA; one
//                          more CTA per head rotates its queries (head 0's also norms the latent and writes the cache row).
//   latent_out_kernel      decoding: merge of the split partials, per-head linear map W_uv, output gate.
//
// The per-head maps stream their weights straight from global memory (every weight is used by one CTA per 16 tokens; the
// first loads are issued before the wait on the previous kernel), the activations go through shared memory.  K positions are
// assigned to fragment slots in the order 16-byte loads deliver them.
#include "tdb/attn_device.cuh"
#include "tdb/latent.h"
#include "tdb/launch.cuh"
#include "tdb/vec.cuh"

namespace tdb {

namespace {

constexpr int kTok = 16;      // tokens per CTA
constexpr int kCols = 64;     // output columns per CTA: eight warps of eight
constexpr int kThreads = 256;
constexpr int kMaxSplits = 64;

// Four neighbouring pairs turn by their angles: (u, v) -> (u cos - v sin, v cos + u sin).
template <typename T>
TDB_DEVICE void rotate8(const T* in, const float* cs, T* out) {
  float x[8], c[8];
  load8(in, x);
  load8(cs, c);
#pragma unroll
  for (int i = 0; i < 8; i += 2) {
    const float u = x[i], v = x[i + 1];
    x[i] = u * c[i] - v * c[i + 1];
    x[i + 1] = v * c[i] + u * c[i + 1];
  }
  store8(out, x);
}

TDB_DEVICE const float* angles(const LatentPrepArgs& p, int64_t t) {
  int64_t pos = p.pos[t];
  if (pos < 0 || pos >= p.n_pos) pos = 0;
  return p.cos_sin + pos * p.r;
}

// One warp: the cached row of token t.
template <typename T>
TDB_DEVICE void latent_row(const LatentPrepArgs& p, int64_t t) {
  const int lane = threadIdx.x & 31;
  const T* c = reinterpret_cast<const T*>(p.z) + t * p.ld + static_cast<int64_t>(p.H) * (p.d + p.r);
  float ss = 0.f;
  for (int i = lane * 8; i < p.R; i += 256) {
    float f[8];
    load8(c + i, f);
#pragma unroll
    for (int j = 0; j < 8; ++j) ss += f[j] * f[j];
  }
  const float inv = 1.f / sqrtf(warp_sum(ss) / p.R_real + p.eps);
  const int64_t ra = p.rows[t], rb = p.ctx != nullptr ? p.ctx_rows[t] : -1;
  const int W = p.R + p.r;
  T* a = ra >= 0 && ra < p.cap ? reinterpret_cast<T*>(p.cache) + ra * W : nullptr;
  T* b = rb >= 0 && rb < p.ctx_cap ? reinterpret_cast<T*>(p.ctx) + rb * W : nullptr;
  for (int i = lane * 8; i < p.R; i += 256) {
    float f[8], w[8];
    load8(c + i, f);
    load8(p.norm_w + i, w);
#pragma unroll
    for (int j = 0; j < 8; ++j) f[j] *= inv * w[j];
    if (a != nullptr) store8(a + i, f);
    if (b != nullptr) store8(b + i, f);
  }
  const float* cs = angles(p, t);
  for (int i = lane * 8; i < p.r; i += 256) {
    if (a != nullptr) rotate8(c + p.R + i, cs + i, a + p.R + i);
    if (b != nullptr) rotate8(c + p.R + i, cs + i, b + p.R + i);
  }
}

template <typename T>
__global__ void __launch_bounds__(128) latent_rotate_kernel(const LatentPrepArgs p) {
  pdl_wait();
  pdl_launch_dependents();
  const int64_t t = blockIdx.x;
  if (threadIdx.x < 32) {
    if (p.own_kv) latent_row<T>(p, t);
    return;
  }
  const float* cs = angles(p, t);
  T* q = reinterpret_cast<T*>(p.z) + t * p.ld;
  const int per = p.r / 8;
  for (int i = threadIdx.x - 32; i < p.H * per; i += 96) {
    const int h = i / per, c = (i - h * per) * 8;
    T* at = q + static_cast<int64_t>(h) * (p.d + p.r) + p.d + c;
    rotate8(at, cs + c, at);
  }
}

// ---- per-head linear map of 16 tokens, bf16: c += rows g, g + 8 of as (shared memory, [16][pitch]) times row g of w
struct HeadWeights {          // this lane's 16-byte pieces of its weight row, four 32-element blocks at a time
  uint4 v[4];
  TDB_DEVICE void load(const __nv_bfloat16* row, int k0, int K, int t) {
#pragma unroll
    for (int b = 0; b < 4; ++b) {
      const int kk = k0 + b * 32 + t * 8;
      v[b] = (row != nullptr && kk < K) ? ld_nc_v4(row + kk) : make_uint4(0u, 0u, 0u, 0u);
    }
  }
};
TDB_DEVICE void head_blocks(float (&c)[4], const __nv_bfloat16* as, int pitch, const HeadWeights& w, int k0, int K, int g, int t) {
#pragma unroll
  for (int b = 0; b < 4; ++b) {
    const int kk = k0 + b * 32 + t * 8;
    if (k0 + b * 32 >= K) break;
    // pieces beyond K meet zero weights; the row's tail in shared memory is zero as well
    const uint4 lo = *reinterpret_cast<const uint4*>(as + g * pitch + kk);
    const uint4 hi = *reinterpret_cast<const uint4*>(as + (g + 8) * pitch + kk);
    const uint32_t a0[4] = {lo.x, hi.x, lo.y, hi.y}, a1[4] = {lo.z, hi.z, lo.w, hi.w};
    attn::mma_bf16(c, a0, w.v[b].x, w.v[b].y);
    attn::mma_bf16(c, a1, w.v[b].z, w.v[b].w);
  }
}
TDB_DEVICE int head_pitch(int K) { return (K + 31) / 32 * 32 + 32; }
__host__ __device__ inline size_t head_smem(int K, bool f32) { return static_cast<size_t>(kTok) * ((K + 31) / 32 * 32 + 32) * (f32 ? 4 : 2); }

// Groups of threads that share the partials of a token in latent_out_kernel.
__host__ __device__ inline int merge_groups(int n_tok, int splits) {
  return n_tok > 2 || splits < 8 ? 1 : n_tok == 2 ? 2 : 4;
}

// The map itself.  `stage` fills as[16][pitch] (after the previous kernel's results are visible), `put(token, column, value)`
// takes the products; w [n_cols, K] are the head's weights.
template <typename T, typename Stage, typename Put>
TDB_DEVICE void head_linear(const T* w, int n_cols, int K, int n0, T* as, Stage stage, Put put) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
  const int pitch = head_pitch(K);
  if constexpr (sizeof(T) == 2) {
    const int col = n0 + warp * 8 + g;
    const T* row = col < n_cols ? w + static_cast<int64_t>(col) * K : nullptr;
    HeadWeights hw;
    hw.load(row, 0, K, t);
    stage();
    __syncthreads();
    float c[4] = {0.f, 0.f, 0.f, 0.f};
    for (int k0 = 0; k0 < K; k0 += 128) {
      HeadWeights next;
      if (k0 + 128 < K) next.load(row, k0 + 128, K, t);
      head_blocks(c, as, pitch, hw, k0, K, g, t);
      if (k0 + 128 < K) hw = next;
    }
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int n = n0 + warp * 8 + 2 * t + (e & 1);
      if (n < n_cols) put(g + (e >> 1) * 8, n, c[e]);
    }
  } else {
    stage();
    __syncthreads();
    const int n = n0 + (threadIdx.x & 63), i0 = (threadIdx.x >> 6) * 4;
    if (n >= n_cols) return;
    float c[4] = {0.f, 0.f, 0.f, 0.f};
    for (int k = 0; k < K; k += 8) {
      float f[8];
      load8(w + static_cast<int64_t>(n) * K + k, f);
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 8; ++j) c[i] = fmaf(as[(i0 + i) * pitch + k + j], f[j], c[i]);
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) put(i0 + i, n, c[i]);
  }
}

// grid (ceil(R / 64) + 1, H, ceil(T / 16))
template <typename T>
__global__ void __launch_bounds__(kThreads) latent_absorb_kernel(const LatentPrepArgs p) {
  extern __shared__ __align__(16) uint8_t smem[];
  T* as = reinterpret_cast<T*>(smem);
  const int h = blockIdx.y;
  const int64_t t0 = static_cast<int64_t>(blockIdx.z) * kTok;
  const int n_tok = static_cast<int>(min(static_cast<int64_t>(kTok), p.T - t0));
  const int W = p.R + p.r;
  const T* z = reinterpret_cast<const T*>(p.z) + static_cast<int64_t>(h) * (p.d + p.r);
  T* qe = reinterpret_cast<T*>(p.q_eff) + static_cast<int64_t>(h) * W;
  if (blockIdx.x == gridDim.x - 1) {
    pdl_wait();
    pdl_launch_dependents();
    const int per = p.r / 8;
    for (int i = threadIdx.x; i < n_tok * per; i += kThreads) {
      const int64_t t = t0 + i / per;
      const int c = (i % per) * 8;
      rotate8(z + t * p.ld + p.d + c, angles(p, t) + c, qe + t * p.H * W + p.R + c);
    }
    if (h == 0 && p.own_kv)
      for (int i = threadIdx.x >> 5; i < n_tok; i += kThreads / 32) latent_row<T>(p, t0 + i);
    return;
  }
  const int pitch = head_pitch(p.d);
  head_linear<T>(
      reinterpret_cast<const T*>(p.uk_t) + static_cast<int64_t>(h) * p.R * p.d, p.R, p.d, blockIdx.x * kCols, as,
      [&] {
        pdl_wait();
        pdl_launch_dependents();
        for (int i = threadIdx.x; i < kTok * (pitch / 8); i += kThreads) {
          const int r = i / (pitch / 8), c = (i % (pitch / 8)) * 8;
          float f[8] = {};
          if (r < n_tok && c < p.d) load8(z + (t0 + r) * p.ld + c, f);
          store8(as + r * pitch + c, f);
        }
      },
      [&](int r, int n, float v) {
        if (r < n_tok) qe[(t0 + r) * p.H * W + n] = from_f32<T>(v);
      });
}

// grid (ceil(dv / 64), H, ceil(T / 16))
template <typename T>
__global__ void __launch_bounds__(kThreads) latent_out_kernel(const LatentOutArgs p) {
  extern __shared__ __align__(16) uint8_t smem[];
  __shared__ float wsplit[kTok][kMaxSplits];
  T* as = reinterpret_cast<T*>(smem);
  const int h = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int64_t t0 = static_cast<int64_t>(blockIdx.z) * kTok;
  const int n_tok = static_cast<int>(min(static_cast<int64_t>(kTok), p.T - t0));
  const int pitch = head_pitch(p.R);
  T* out = reinterpret_cast<T*>(p.out) + static_cast<int64_t>(h) * p.dv;
  const T* gate = reinterpret_cast<const T*>(p.gate) + static_cast<int64_t>(h) * p.dv;
  head_linear<T>(
      reinterpret_cast<const T*>(p.uv) + static_cast<int64_t>(h) * p.dv * p.R, p.dv, p.R, blockIdx.x * kCols, as,
      [&] {
        pdl_wait();
        pdl_launch_dependents();
        // factor of every partial: exp2(m - max) / sum of all
        for (int i = warp; i < n_tok; i += kThreads / 32) {
          if (p.ml == nullptr) {
            if (lane == 0) wsplit[i][0] = 1.f;
            continue;
          }
          const float2* ml = reinterpret_cast<const float2*>(p.ml) + ((t0 + i) * p.H + h) * p.splits;
          float2 a[2];
          float m = -INFINITY;
#pragma unroll
          for (int j = 0; j < 2; ++j) {
            const int s = lane + 32 * j;
            a[j] = s < p.splits ? ml[s] : make_float2(-INFINITY, 0.f);
            if (a[j].y > 0.f) m = fmaxf(m, a[j].x);
          }
          m = warp_max(m);
          float w[2], l = 0.f;
#pragma unroll
          for (int j = 0; j < 2; ++j) {
            w[j] = a[j].y > 0.f ? exp2f(a[j].x - m) : 0.f;
            l += w[j] * a[j].y;
          }
          l = warp_sum(l);
#pragma unroll
          for (int j = 0; j < 2; ++j)
            if (lane + 32 * j < p.splits) wsplit[i][lane + 32 * j] = l > 0.f ? w[j] / l : 0.f;
        }
        __syncthreads();
        // few tokens: the partials of a token are dealt out to groups of threads, so that all loads are in flight together
        const int per_row = pitch / 8, groups = merge_groups(n_tok, p.splits);
        float* part = reinterpret_cast<float*>(smem + head_smem(p.R, sizeof(T) == 4));      // [groups][n_tok][R]
        const int n_items = (groups > 1 ? n_tok : kTok) * per_row;
        for (int i = threadIdx.x; i < n_items * groups; i += kThreads) {
          const int grp = i / n_items, r = (i % n_items) / per_row, c = (i % per_row) * 8;
          float acc[8] = {};
          if (r < n_tok && c < p.R) {
            const float* o = p.o + ((t0 + r) * p.H + h) * static_cast<int64_t>(p.splits) * p.R + c;
            for (int s0 = grp; s0 < p.splits; s0 += groups * 4) {
              float f[4][8], w[4];
#pragma unroll
              for (int u = 0; u < 4; ++u) {
                const int s = s0 + u * groups;
                w[u] = s < p.splits ? wsplit[r][s] : 0.f;
                if (w[u] != 0.f) load8(o + static_cast<int64_t>(s) * p.R, f[u]);      // an empty partial was never written
              }
#pragma unroll
              for (int u = 0; u < 4; ++u)
                if (w[u] != 0.f)
#pragma unroll
                  for (int j = 0; j < 8; ++j) acc[j] = fmaf(w[u], f[u][j], acc[j]);
            }
          }
          if (groups == 1) store8(as + r * pitch + c, acc);
          else if (c < p.R) store8(part + (grp * n_tok + r) * p.R + c, acc);
        }
        if (groups > 1) {
          __syncthreads();
          for (int i = threadIdx.x; i < kTok * per_row; i += kThreads) {
            const int r = i / per_row, c = (i % per_row) * 8;
            float acc[8] = {}, f[8];
            if (r < n_tok && c < p.R)
              for (int g = 0; g < groups; ++g) {
                load8(part + (g * n_tok + r) * p.R + c, f);
#pragma unroll
                for (int j = 0; j < 8; ++j) acc[j] += f[j];
              }
            store8(as + r * pitch + c, acc);
          }
        }
      },
      [&](int r, int n, float v) {
        if (r >= n_tok) return;
        const int64_t t = t0 + r;
        out[t * p.H * p.dv + n] = from_f32<T>(v * sigmoid_f32(to_f32(gate[t * p.ld_gate + n])));
      });
}

bool prep_ok(const LatentPrepArgs& a) {
  return a.H >= 1 && a.d % 8 == 0 && a.r % 8 == 0 && a.R % 8 == 0 && a.ld % 8 == 0 && a.d > 0 && a.r > 0 && a.R > 0 && a.n_pos > 0 &&
         (!a.own_kv || (a.cache != nullptr && a.rows != nullptr && a.R_real > 0)) && (a.ctx == nullptr || a.ctx_rows != nullptr);
}

}  // namespace

cudaError_t launch_latent_rotate(const LatentPrepArgs& a, cudaStream_t s) {
  if (!prep_ok(a)) return cudaErrorInvalidValue;
  if (a.T == 0) return cudaSuccess;
  const dim3 grid(static_cast<unsigned>(a.T));
  return a.is_f32 ? launch_pdl(latent_rotate_kernel<float>, grid, dim3(128), 0, s, a)
                  : launch_pdl(latent_rotate_kernel<__nv_bfloat16>, grid, dim3(128), 0, s, a);
}

cudaError_t launch_latent_absorb(const LatentPrepArgs& a, cudaStream_t s) {
  const size_t smem = head_smem(a.d, a.is_f32);
  const int64_t tiles = (a.T + kTok - 1) / kTok;
  if (!prep_ok(a) || a.uk_t == nullptr || a.q_eff == nullptr || smem > 200 * 1024 || tiles > 65535) return cudaErrorInvalidValue;
  if (a.T == 0) return cudaSuccess;
  static SmemOptIn f, b;
  cudaError_t e = a.is_f32 ? f.ensure(latent_absorb_kernel<float>, 200 * 1024) : b.ensure(latent_absorb_kernel<__nv_bfloat16>, 200 * 1024);
  if (e != cudaSuccess) return e;
  const dim3 grid((a.R + kCols - 1) / kCols + 1, a.H, static_cast<unsigned>(tiles));
  return a.is_f32 ? launch_pdl(latent_absorb_kernel<float>, grid, dim3(kThreads), smem, s, a)
                  : launch_pdl(latent_absorb_kernel<__nv_bfloat16>, grid, dim3(kThreads), smem, s, a);
}

cudaError_t launch_latent_out(const LatentOutArgs& a, cudaStream_t s) {
  // (a tail of one or two tokens behind full tiles merges in groups as well: room for the largest case)
  const size_t smem = head_smem(a.R, a.is_f32) + static_cast<size_t>(a.splits < 8 ? 0 : 4) * a.R * 4;
  const int64_t tiles = (a.T + kTok - 1) / kTok;
  if (a.R % 8 != 0 || a.dv < 1 || a.H < 1 || a.splits < 1 || a.splits > kMaxSplits || (a.ml == nullptr && a.splits != 1) ||
      smem > 200 * 1024 || tiles > 65535)
    return cudaErrorInvalidValue;
  if (a.T == 0) return cudaSuccess;
  static SmemOptIn f, b;
  cudaError_t e = a.is_f32 ? f.ensure(latent_out_kernel<float>, 200 * 1024) : b.ensure(latent_out_kernel<__nv_bfloat16>, 200 * 1024);
  if (e != cudaSuccess) return e;
  const dim3 grid((a.dv + kCols - 1) / kCols, a.H, static_cast<unsigned>(tiles));
  return a.is_f32 ? launch_pdl(latent_out_kernel<float>, grid, dim3(kThreads), smem, s, a)
                  : launch_pdl(latent_out_kernel<__nv_bfloat16>, grid, dim3(kThreads), smem, s, a);
}

}  // namespace tdb
