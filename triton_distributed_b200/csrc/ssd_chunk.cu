// State space layer, chunk-parallel form for bf16 activations (recurrence in tdb/ssd.h).
//
// With G_t the log decay summed from a 64-token chunk's start (inclusive, one number per head) and S the state before the chunk:
//     y_t   = e^{G_t} S^T C_t  +  sum_{j <= t} (C_t . B_j) e^{G_t - G_j} dt_j x_j  +  D x_t
//     S_end = e^{G_63} S + sum_j B_j (e^{G_63 - G_j} dt_j x_j)^T
// Three launches behind the convolutions:
//   inject_kernel  one CTA per (chunk, heads of one group): what the chunk adds to the states; the group's B is loaded once
//   scan_kernel    the sequential part, element-wise: turns contributions into the state BEFORE every chunk (in place) and writes the
//                  sequence's final state
//   out_kernel     one CTA per (chunk, heads of one group): the scores C B^T once for all its heads, then outputs head by head
// Contributions and states are stored tile by tile in the order in which the lanes of a warp hold the B fragments of m16n8k16, as in
// gla_chunk.cu: the scan turns each value into its bf16 high and low part, the output kernel loads ready fragments.
//
// Exponentials are of differences that cannot be positive.  The decay being one number per token and head, it multiplies B, the scores and
// rows of the first product's result, so C and x enter the tensor cores as the bf16 numbers they are; what counts as fp32 (states, scaled
// B, scaled scores) enters as a high and a low part: two products each.
#include "tdb/attn_device.cuh"
#include "tdb/chunk.cuh"
#include "tdb/launch.cuh"
#include "tdb/ssd.h"
#include "tdb/vec.cuh"

namespace tdb {

namespace {

using attn::cp_async_commit;
using attn::cp_async_wait;
using attn::ldmatrix_x4_trans;
using attn::mma_bf16;
using chunk::ChunkPos;
using chunk::HiLo;
using chunk::chunk_pos;
using chunk::kC;
using chunk::ld2;
using chunk::ldmatrix_x4;
using chunk::split2;

constexpr int kThreads = 256;

__host__ __device__ __forceinline__ int channels(const SsdArgs& p) { return p.H * p.dv + 2 * p.G * p.dk; }

// ---------------------------------------------------------------------------------------------------- contributions
size_t inject_smem(int dk, int dv) { return static_cast<size_t>(kC) * (dk + 8) * 2 + 2 * (static_cast<size_t>(kC) * (dv + 8) * 2 + kC * 4); }

__global__ void __launch_bounds__(kThreads) inject_kernel(const SsdArgs p, int heads) {
  extern __shared__ __align__(16) uint8_t smem[];
  const int kp = p.dk + 8, vp = p.dv + 8;
  __nv_bfloat16* bs = reinterpret_cast<__nv_bfloat16*>(smem);     // [64][kp]
  __nv_bfloat16* xs = bs + kC * kp;                               // [2][64][vp] inputs of this head and the next
  float* fs = reinterpret_cast<float*>(xs + 2 * kC * vp);         // [2][64] factors of the tokens
  const int chunk = blockIdx.x, h0 = blockIdx.y * heads, g = h0 / (p.H / p.G);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  pdl_wait();
  pdl_launch_dependents();
  const ChunkPos cp = chunk_pos(p, chunk);
  const int C = channels(p), Hv = p.H * p.dv;
  const __nv_bfloat16* base = reinterpret_cast<const __nv_bfloat16*>(p.xbc) + cp.t0 * C;
  chunk::load_tile(bs, kp, base + Hv + g * p.dk, C, p.dk, cp.n, kThreads);
  auto load_head = [&](int h) {
    const int s = (h - h0) & 1;
    chunk::load_tile(xs + s * kC * vp, vp, base + h * p.dv, C, p.dv, cp.n, kThreads);
    cp_async_commit();
    if (threadIdx.x < kC) {
      const int64_t at = cp.t0 * p.H + h;
      const float last = p.log_g[at + static_cast<int64_t>(cp.n - 1) * p.H];
      const int64_t mine = at + static_cast<int64_t>(min(static_cast<int>(threadIdx.x), cp.n - 1)) * p.H;
      fs[s * kC + threadIdx.x] = static_cast<int>(threadIdx.x) < cp.n ? __expf(last - p.log_g[mine]) * p.dt[mine] : 0.f;
    }
  };
  load_head(h0);
  const int nb = (p.dv + 63) / 64, units = (p.dk / 16) * nb;
  const int mat = lane >> 3, mr = lane & 7, gr = lane >> 2, t4 = lane & 3;
  for (int h = h0; h < h0 + heads; ++h) {
    cp_async_wait<0>();
    __syncthreads();
    if (h + 1 < h0 + heads) load_head(h + 1);      // into the buffers that were read before the barrier
    const __nv_bfloat16* x = xs + ((h - h0) & 1) * kC * vp;
    const float* f = fs + ((h - h0) & 1) * kC;
    // units of 16 rows x 64 columns of the state; A = B^T (read transposed), scaled by the tokens' factors and cut into two parts
    float4* out = reinterpret_cast<float4*>(p.inject) + (static_cast<int64_t>(chunk) * p.H + h) * p.dk * (p.dv / 4);
    for (int u = warp; u < units; u += kThreads / 32) {
      const int c0 = (u / nb) * 16, n0 = (u % nb) * 64;
      float acc[8][4];
#pragma unroll
      for (int i = 0; i < 8; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
#pragma unroll
      for (int ks = 0; ks < kC / 16; ++ks) {
        uint32_t a[4], ah[4], al[4];
        ldmatrix_x4_trans(a, bs + (ks * 16 + (mat >> 1) * 8 + mr) * kp + c0 + (mat & 1) * 8);
        const float2 f0 = *reinterpret_cast<const float2*>(f + ks * 16 + 2 * t4), f1 = *reinterpret_cast<const float2*>(f + ks * 16 + 8 + 2 * t4);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const float2 b = unpack_bf16x2(a[i]);
          const HiLo v = split2(b.x * (i < 2 ? f0.x : f1.x), b.y * (i < 2 ? f0.y : f1.y));
          ah[i] = v.hi;
          al[i] = v.lo;
        }
#pragma unroll
        for (int j = 0; j < 8; j += 2) {
          if (n0 + j * 8 >= p.dv) break;
          uint32_t v[4];
          ldmatrix_x4_trans(v, x + (ks * 16 + (mat & 1) * 8 + mr) * vp + n0 + j * 8 + (mat >> 1) * 8);
          mma_bf16(acc[j], ah, v[0], v[1]);
          mma_bf16(acc[j], al, v[0], v[1]);
          mma_bf16(acc[j + 1], ah, v[2], v[3]);
          mma_bf16(acc[j + 1], al, v[2], v[3]);
        }
      }
      // accumulator layout (row g, columns 2t, 2t + 1; row g + 8) -> B-fragment layout (rows 2t, 2t + 1, + 8; column g)
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        if (n0 + j * 8 >= p.dv) break;
        const int src = 8 * t4 + (gr >> 1);         // lane that holds row 2 t4 and the pair of columns with g in it
        float4 v;
        float a0 = __shfl_sync(0xffffffffu, acc[j][0], src), a1 = __shfl_sync(0xffffffffu, acc[j][1], src);
        v.x = (gr & 1) ? a1 : a0;
        a0 = __shfl_sync(0xffffffffu, acc[j][0], src + 4), a1 = __shfl_sync(0xffffffffu, acc[j][1], src + 4);
        v.y = (gr & 1) ? a1 : a0;
        a0 = __shfl_sync(0xffffffffu, acc[j][2], src), a1 = __shfl_sync(0xffffffffu, acc[j][3], src);
        v.z = (gr & 1) ? a1 : a0;
        a0 = __shfl_sync(0xffffffffu, acc[j][2], src + 4), a1 = __shfl_sync(0xffffffffu, acc[j][3], src + 4);
        v.w = (gr & 1) ? a1 : a0;
        out[((c0 / 16) * (p.dv / 8) + n0 / 8 + j) * 32 + lane] = v;
      }
    }
  }
}

// ---------------------------------------------------------------------------------------------------- scan over the chunks
// Thread = one lane's fragment of one 16 x 8 tile of one head's state.
__global__ void __launch_bounds__(256) scan_kernel(const SsdArgs p) {
  const int n = blockIdx.y;
  const int64_t per = static_cast<int64_t>(p.H) * p.dk * (p.dv >> 2);      // fragments of one chunk
  const int64_t e = static_cast<int64_t>(blockIdx.x) * 256 + threadIdx.x;
  pdl_wait();
  pdl_launch_dependents();
  if (e >= per) return;
  const int per_head = p.dk * (p.dv >> 2);
  const int h = static_cast<int>(e / per_head), f = static_cast<int>(e - static_cast<int64_t>(h) * per_head);
  const int lane = f & 31, tile = f >> 5, nt8 = p.dv >> 3;
  const int row = (tile / nt8) * 16 + 2 * (lane & 3), col = (tile % nt8) * 8 + (lane >> 2);
  float* st = p.state + ((static_cast<int64_t>(p.slots[n]) * p.H + h) * p.dk + row) * p.dv + col;
  float4* cs = reinterpret_cast<float4*>(p.inject) + e;
  float4 S = make_float4(0.f, 0.f, 0.f, 0.f);
  if (p.pos0[n] != 0) S = make_float4(st[0], st[p.dv], st[8 * p.dv], st[9 * p.dv]);
  const int c0 = p.seq_chunk0[n], c1 = p.seq_chunk0[n + 1];
  const int64_t first = p.cu[n], end = p.cu[n + 1];
  constexpr int U = 8;
  for (int c = c0; c < c1; c += U) {
    float4 v[U];
    float d[U];
#pragma unroll
    for (int u = 0; u < U; ++u) {
      if (c + u < c1) {
        v[u] = cs[(c + u) * per];
        const int64_t last = min(first + static_cast<int64_t>(c + u - c0 + 1) * kC, end) - 1;      // last token of the chunk
        d[u] = p.log_g[last * p.H + h];
      }
    }
#pragma unroll
    for (int u = 0; u < U; ++u) {
      if (c + u < c1) {
        const HiLo b0 = split2(S.x, S.y), b1 = split2(S.z, S.w);
        reinterpret_cast<uint4*>(cs)[(c + u) * per] = make_uint4(b0.hi, b1.hi, b0.lo, b1.lo);
        const float k = __expf(d[u]);
        S.x = fmaf(k, S.x, v[u].x); S.y = fmaf(k, S.y, v[u].y);
        S.z = fmaf(k, S.z, v[u].z); S.w = fmaf(k, S.w, v[u].w);
      }
    }
  }
  st[0] = S.x; st[p.dv] = S.y; st[8 * p.dv] = S.z; st[9 * p.dv] = S.w;
}

// ---------------------------------------------------------------------------------------------------- outputs
constexpr int kAp = kC + 4;       // pitch of the score matrix (fp32)
constexpr int kWp = kC + 8;       // pitch of a head's weights (bf16)
size_t out_smem(int dk, int dv) {
  return 2 * static_cast<size_t>(kC) * (dk + 8) * 2 + static_cast<size_t>(kC) * (dv + 8) * 2 + static_cast<size_t>(kC) * kAp * 4 +
         2 * static_cast<size_t>(kC) * kWp * 2 + 2 * kC * 4;
}

template <int TW>     // 8-column tiles per warp: dv <= 64 TW
__global__ void __launch_bounds__(kThreads, TW <= 2 ? 2 : 1) out_kernel(const SsdArgs p, int heads) {
  extern __shared__ __align__(16) uint8_t smem[];
  const int kp = p.dk + 8, vp = p.dv + 8;
  __nv_bfloat16* cs = reinterpret_cast<__nv_bfloat16*>(smem);     // [64][kp]
  __nv_bfloat16* bs = cs + kC * kp;
  __nv_bfloat16* xs = bs + kC * kp;                               // [64][vp]
  __nv_bfloat16* wh = xs + kC * vp;                               // [64][kWp] a head's weights, high parts
  __nv_bfloat16* wl = wh + kC * kWp;
  float* A = reinterpret_cast<float*>(wl + kC * kWp);             // [64][kAp] scores of the group
  float* G = A + kC * kAp;                                        // [64] log decays of the head
  float* D = G + kC;                                              // [64] step sizes
  const int chunk = blockIdx.x, h0 = blockIdx.y * heads, g = h0 / (p.H / p.G);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gr = lane >> 2, t4 = lane & 3;
  const int mat = lane >> 3, mr = lane & 7;
  pdl_wait();
  pdl_launch_dependents();
  const ChunkPos cp = chunk_pos(p, chunk);
  const int C = channels(p), Hv = p.H * p.dv, Gk = p.G * p.dk;
  const __nv_bfloat16* base = reinterpret_cast<const __nv_bfloat16*>(p.xbc) + cp.t0 * C;
  chunk::load_tile(bs, kp, base + Hv + g * p.dk, C, p.dk, cp.n, kThreads);
  chunk::load_tile(cs, kp, base + Hv + Gk + g * p.dk, C, p.dk, cp.n, kThreads);
  cp_async_commit();
  auto load_head = [&](int h) {
    chunk::load_tile(xs, vp, base + h * p.dv, C, p.dv, cp.n, kThreads);
    if (threadIdx.x < kC) {                         // rows beyond the sequence repeat the last one and write nothing
      const int64_t at = (cp.t0 + min(static_cast<int>(threadIdx.x), cp.n - 1)) * p.H + h;
      G[threadIdx.x] = p.log_g[at];
      D[threadIdx.x] = static_cast<int>(threadIdx.x) < cp.n ? p.dt[at] : 0.f;
    }
    cp_async_commit();
  };
  load_head(h0);
  cp_async_wait<0>();
  __syncthreads();
  // scores: the ten 16 x 16 blocks on and below the diagonal, over the eight warps
  for (int u = warp; u < 10; u += kThreads / 32) {
    const int bi = u < 1 ? 0 : u < 3 ? 1 : u < 6 ? 2 : 3, bj = u - bi * (bi + 1) / 2;
    float acc[2][4] = {};
    for (int k0 = 0; k0 < p.dk; k0 += 16) {
      uint32_t a[4], b[4];
      ldmatrix_x4(a, cs + (bi * 16 + (mat & 1) * 8 + mr) * kp + k0 + (mat >> 1) * 8);
      ldmatrix_x4(b, bs + (bj * 16 + (mat >> 1) * 8 + mr) * kp + k0 + (mat & 1) * 8);
      mma_bf16(acc[0], a, b[0], b[1]);
      mma_bf16(acc[1], a, b[2], b[3]);
    }
#pragma unroll
    for (int nt = 0; nt < 2; ++nt) {
      float* a0 = A + (bi * 16 + gr) * kAp + bj * 16 + nt * 8 + 2 * t4;
      a0[0] = acc[nt][0]; a0[1] = acc[nt][1];
      a0[8 * kAp] = acc[nt][2]; a0[8 * kAp + 1] = acc[nt][3];
    }
  }
  __syncthreads();
  constexpr int kAhead = 4;
  const int tiles = p.dv / 8, tile0 = warp * TW, ksteps = p.dk / 16;
  for (int h = h0; h < h0 + heads; ++h) {
    // the head's first state fragments travel while its weights are formed
    const uint4* S = reinterpret_cast<const uint4*>(p.inject) + (static_cast<int64_t>(chunk) * p.H + h) * p.dk * (p.dv / 4) + lane;
    uint4 sf[kAhead][TW];
    auto fetch = [&](int u, int step) {
#pragma unroll
      for (int j = 0; j < TW; ++j)
        if (step < ksteps && tile0 + j < tiles) sf[u][j] = S[(step * tiles + tile0 + j) * 32];
    };
#pragma unroll
    for (int u = 0; u < kAhead; ++u) fetch(u, u);
    for (int i = threadIdx.x; i < kC * (kC / 2); i += kThreads) {
      const int t = i / (kC / 2), j = (i - t * (kC / 2)) * 2;
      if (j / 16 > t / 16) continue;                // blocks above the diagonal are not read
      const float gt = G[t];
      const float w0 = j <= t ? A[t * kAp + j] * __expf(gt - G[j]) * D[j] : 0.f;
      const float w1 = j + 1 <= t ? A[t * kAp + j + 1] * __expf(gt - G[j + 1]) * D[j + 1] : 0.f;
      const HiLo s = split2(w0, w1);
      *reinterpret_cast<uint32_t*>(wh + t * kWp + j) = s.hi;
      *reinterpret_cast<uint32_t*>(wl + t * kWp + j) = s.lo;
    }
    __syncthreads();
    float acc[4][TW][4];
#pragma unroll
    for (int r = 0; r < 4; ++r)
#pragma unroll
      for (int j = 0; j < TW; ++j) acc[r][j][0] = acc[r][j][1] = acc[r][j][2] = acc[r][j][3] = 0.f;
    if (tile0 < tiles) {
      // a warp owns TW tiles of 8 columns for all 64 tokens, so a fragment of the state is loaded once per CTA
      for (int s0 = 0; s0 < ksteps; s0 += kAhead) {
#pragma unroll
        for (int u = 0; u < kAhead; ++u) {
          if (s0 + u >= ksteps) break;
          const int off = (mat >> 1) * 8 + (s0 + u) * 16;
#pragma unroll
          for (int r = 0; r < 4; ++r) {
            uint32_t a[4];
            ldmatrix_x4(a, cs + (r * 16 + (mat & 1) * 8 + mr) * kp + off);
#pragma unroll
            for (int j = 0; j < TW; ++j) {
              const uint4 b = sf[u][j];             // high parts of both halves of k, then the low parts
              mma_bf16(acc[r][j], a, b.x, b.y);
              mma_bf16(acc[r][j], a, b.z, b.w);
            }
          }
          fetch(u, s0 + kAhead + u);
        }
      }
#pragma unroll
      for (int r = 0; r < 4; ++r) {
        const float e0 = __expf(G[r * 16 + gr]), e1 = __expf(G[r * 16 + gr + 8]);
#pragma unroll
        for (int j = 0; j < TW; ++j) {
          acc[r][j][0] *= e0; acc[r][j][1] *= e0;
          acc[r][j][2] *= e1; acc[r][j][3] *= e1;
        }
      }
#pragma unroll
      for (int kb = 0; kb < 4; ++kb) {
        uint32_t vb[(TW + 1) / 2][4];
#pragma unroll
        for (int j = 0; j < TW; j += 2)             // a single tile reads 8 columns past it: another warp's, or the row's padding
          ldmatrix_x4_trans(vb[j / 2], xs + (kb * 16 + (mat & 1) * 8 + mr) * vp + min(tile0 + j, tiles - 1) * 8 + (mat >> 1) * 8);
#pragma unroll
        for (int r = kb; r < 4; ++r) {
          uint32_t ah[4], al[4];
          const int at = (r * 16 + (mat & 1) * 8 + mr) * kWp + kb * 16 + (mat >> 1) * 8;
          ldmatrix_x4(ah, wh + at);
          ldmatrix_x4(al, wl + at);
#pragma unroll
          for (int j = 0; j < TW; ++j) {
            const uint32_t b0 = vb[j / 2][(j & 1) * 2], b1 = vb[j / 2][(j & 1) * 2 + 1];
            mma_bf16(acc[r][j], ah, b0, b1);
            mma_bf16(acc[r][j], al, b0, b1);
          }
        }
      }
      const float skip = p.skip[h];
#pragma unroll
      for (int r = 0; r < 4; ++r)
#pragma unroll
        for (int rr = 0; rr < 2; ++rr) {
          const int t = r * 16 + rr * 8 + gr;
          if (t >= cp.n) continue;
          __nv_bfloat16* out = reinterpret_cast<__nv_bfloat16*>(p.out) + (cp.t0 + t) * Hv + h * p.dv;
#pragma unroll
          for (int j = 0; j < TW; ++j)
            if (tile0 + j < tiles) {
              const int c = (tile0 + j) * 8 + 2 * t4;
              const float2 x = ld2(xs + t * vp + c);
              *reinterpret_cast<uint32_t*>(out + c) = pack_bf16x2(fmaf(skip, x.x, acc[r][j][2 * rr]), fmaf(skip, x.y, acc[r][j][2 * rr + 1]));
            }
        }
    }
    __syncthreads();                                // everything of this head has been read
    if (h + 1 < h0 + heads) {
      load_head(h + 1);
      cp_async_wait<0>();
      __syncthreads();
    }
  }
}

template <int TW>
cudaError_t launch_out(const SsdArgs& a, int heads, cudaStream_t s) {
  static SmemOptIn opt;
  cudaError_t e = opt.ensure(out_kernel<TW>, 227 * 1024);
  if (e != cudaSuccess) return e;
  return launch_pdl(out_kernel<TW>, dim3(a.NC, a.H / heads), dim3(kThreads), out_smem(a.dk, a.dv), s, a, heads);
}

}  // namespace

bool ssd_chunk_supported(int dk, int dv) {
  return dk % 16 == 0 && dv % 16 == 0 && dk >= 16 && dv >= 16 && dk <= 256 && dv <= 256 && out_smem(dk, dv) <= 227 * 1024 && inject_smem(dk, dv) <= 227 * 1024;
}

cudaError_t launch_ssd_chunk(const SsdArgs& a, cudaStream_t s) {
  if (a.is_f32 || !ssd_chunk_supported(a.dk, a.dv) || a.cu == nullptr || a.H > 65535) return cudaErrorInvalidValue;
  if (a.T == 0 || a.N == 0) return cudaSuccess;
  cudaError_t e = launch_ssd_prepare(a, s);
  if (e == cudaSuccess) e = launch_ssd_keep(a, s);
  if (e != cudaSuccess) return e;
  // heads of a group that share a CTA: as many as leave a few CTAs for every SM
  int heads = 1;
  while (heads < 8 && (a.H / a.G) % (2 * heads) == 0 && static_cast<int64_t>(a.NC) * (a.H / (2 * heads)) >= 148 * 4) heads *= 2;
  static SmemOptIn opt;
  e = opt.ensure(inject_kernel, 227 * 1024);
  if (e != cudaSuccess) return e;
  e = launch_pdl(inject_kernel, dim3(a.NC, a.H / heads), dim3(kThreads), inject_smem(a.dk, a.dv), s, a, heads);
  if (e != cudaSuccess) return e;
  const int64_t per = static_cast<int64_t>(a.H) * a.dk * (a.dv / 4);
  e = launch_pdl(scan_kernel, dim3(static_cast<unsigned>((per + 255) / 256), a.N), dim3(256), 0, s, a);
  if (e != cudaSuccess) return e;
  if (a.dv <= 64) return launch_out<1>(a, heads, s);
  if (a.dv <= 128) return launch_out<2>(a, heads, s);
  return launch_out<4>(a, heads, s);
}

}  // namespace tdb
