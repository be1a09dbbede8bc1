// Gated linear attention, chunk-parallel form for bf16 activations (recurrence in gla.cu).
//
// With G_t the cumulative log decay inside a 64-token chunk (per key channel, inclusive) and S the state before it:
//     o_t   = q_scale ( (q_t e^{G_t}) S  +  sum_{j <= t} A_tj v_j ),   A_tj = sum_c q_tc k_jc e^{G_tc - G_jc}
//     S_end = e^{G_63} S + sum_j (k_j e^{G_63 - G_j}) v_j^T
// Four launches:
//   chunk_decay_kernel G of every token and channel
//   chunk_kv_kernel    one CTA per (chunk, head): the chunk's own contribution to the state and its total decay
//   chunk_scan_kernel  the sequential part, element-wise: turns contributions into the state BEFORE every chunk (in place)
//                      and writes the sequence's final state; a stream of fp32 values, split over all state elements
//   chunk_out_kernel   one CTA per (chunk, head): A, outputs, head norm and output gate
// Contributions and states are stored tile by tile in the order in which the lanes of a warp hold the B fragments of
// m16n8k16, four fp32 values per lane: the contribution kernel writes 512 bytes per tile and warp, the scan reads and
// writes 16 bytes per thread, and turns each value into its bf16 high and low part on the way, so that the output kernel
// loads one ready fragment (both parts) with one 16-byte load.
//
// Decays can be arbitrarily strong, so an exponential is only ever taken of a difference that is <= 0: A between two
// 16-token blocks uses the later block's start as the reference of both factors (q_t e^{G_t - G_ref}, k_j e^{G_ref - G_j}),
// a 16-token diagonal block is cut once more the same way, and its two 8-token triangles are summed pair by pair.
//
// The state and everything that enters it count as fp32, so the tensor cores (mma.sync bf16, fp32 accumulate) get every
// fp32 operand as a high and a low bf16 part: two products where one side is bf16 anyway (v), three where both are fp32.
#include "tdb/attn_device.cuh"
#include "tdb/chunk.cuh"
#include "tdb/gla.cuh"
#include "tdb/hybrid.h"
#include "tdb/launch.cuh"
#include "tdb/vec.cuh"

namespace tdb {

namespace {

using attn::cp_async16;
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

TDB_DEVICE void load_tile(__nv_bfloat16* dst, int pitch, const __nv_bfloat16* src, int64_t ld, int cols, int n) {
  chunk::load_tile(dst, pitch, src, ld, cols, n, kThreads);
}

// The chunk's cumulative log decays of one head into G [64][dk + 8] (asynchronous, 16-byte copies) ...
TDB_DEVICE int g_pitch(int dk) { return dk + 8; }
TDB_DEVICE void load_decays(const GlaArgs& p, const ChunkPos& cp, int h, float* G) {
  const int C = p.H * p.dk, vec = p.dk >> 2;
  const float* src = p.log_decay + cp.t0 * C + h * p.dk;
  for (int i = threadIdx.x; i < kC * vec; i += kThreads) {
    const int r = i / vec, c = (i - r * vec) * 4;
    cp_async16(G + r * g_pitch(p.dk) + c, src + (r < cp.n ? static_cast<int64_t>(r) * C : 0) + c, r < cp.n);
  }
}
// ... and, once they are there (needs a barrier before and after when n < 64): rows beyond the sequence repeat its last row.
TDB_DEVICE void extend_decays(const GlaArgs& p, const ChunkPos& cp, float* G) {
  const int gp = g_pitch(p.dk);
  for (int i = threadIdx.x; i < (kC - cp.n) * p.dk; i += kThreads) {
    const int r = cp.n + i / p.dk, c = i % p.dk;
    G[r * gp + c] = G[(cp.n - 1) * gp + c];
  }
}

// ---------------------------------------------------------------------------------------------------- cumulative decays
constexpr int kDecayTok = 16;
__global__ void __launch_bounds__(256) chunk_decay_kernel(const GlaArgs p) {
  extern __shared__ float s_a[];       // [kDecayTok][R]
  pdl_wait();
  pdl_launch_dependents();
  const ChunkPos cp = chunk_pos(p, blockIdx.y);
  const int C = p.H * p.dk, c = blockIdx.x * 256 + threadIdx.x;
  float g = 0.f;
  for (int b = 0; b < cp.n; b += kDecayTok) {
    const int nt = min(kDecayTok, cp.n - b);
    __syncthreads();
    for (int i = threadIdx.x; i < nt * p.R; i += 256) s_a[i] = p.a[(cp.t0 + b) * p.R + i];
    __syncthreads();
    if (c >= C) continue;
    float z[kDecayTok];
    const float bias = p.a2_b[c];
#pragma unroll
    for (int i = 0; i < kDecayTok; ++i) z[i] = bias;
#pragma unroll 4
    for (int r = 0; r < p.R; ++r) {
      const float w = p.a2[static_cast<int64_t>(r) * C + c];
#pragma unroll
      for (int i = 0; i < kDecayTok; ++i)
        if (i < nt) z[i] = fmaf(w, s_a[i * p.R + r], z[i]);
    }
#pragma unroll
    for (int i = 0; i < kDecayTok; ++i) {
      if (i < nt) {
        g += gla_log_decay(z[i], p.inv_tau);
        p.log_decay[(cp.t0 + b + i) * C + c] = g;
      }
    }
  }
}

// ---------------------------------------------------------------------------------------------------- state contributions
size_t kv_smem(int dk, int dv) {
  return static_cast<size_t>(kC) * (dk + 8) * 4 + 2 * static_cast<size_t>(kC) * (dk + 8) * 2 + static_cast<size_t>(kC) * (dv + 8) * 2 + 64;
}

__global__ void __launch_bounds__(kThreads) chunk_kv_kernel(const GlaArgs p) {
  extern __shared__ __align__(16) uint8_t smem[];
  const int kp = p.dk + 8, vp = p.dv + 8, gp = g_pitch(p.dk);
  __nv_bfloat16* kh = reinterpret_cast<__nv_bfloat16*>(smem);     // raw keys, then their scaled high parts in place
  __nv_bfloat16* kl = kh + kC * kp;
  __nv_bfloat16* vs = kl + kC * kp;
  float* G = reinterpret_cast<float*>(vs + kC * vp);
  const int chunk = blockIdx.x, h = blockIdx.y;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  pdl_wait();
  pdl_launch_dependents();
  const ChunkPos cp = chunk_pos(p, chunk);
  const __nv_bfloat16* base = reinterpret_cast<const __nv_bfloat16*>(p.qkvg) + cp.t0 * p.ld;
  const int Hk = p.H * p.dk;
  load_tile(kh, kp, base + Hk + h * p.dk, p.ld, p.dk, cp.n);
  load_decays(p, cp, h, G);
  load_tile(vs, vp, base + 2 * Hk + h * p.dv, p.ld, p.dv, cp.n);
  cp_async_commit();
  cp_async_wait<0>();
  __syncthreads();
  // rows beyond the sequence hold k = 0 and G = 0: their factor e^{G_last} is finite
  const float* gl = G + (cp.n - 1) * gp;
  float* dec = p.chunk_decay + (static_cast<int64_t>(chunk) * p.H + h) * p.dk;
  for (int c = threadIdx.x; c < p.dk; c += kThreads) dec[c] = expf(gl[c]);
  for (int i = threadIdx.x; i < kC * (p.dk / 2); i += kThreads) {
    const int t = i / (p.dk / 2), c = (i - t * (p.dk / 2)) * 2;
    const float2 k = ld2(kh + t * kp + c);
    const HiLo s = split2(k.x * __expf(gl[c] - G[t * gp + c]), k.y * __expf(gl[c + 1] - G[t * gp + c + 1]));
    *reinterpret_cast<uint32_t*>(kh + t * kp + c) = s.hi;
    *reinterpret_cast<uint32_t*>(kl + t * kp + c) = s.lo;
  }
  __syncthreads();
  // units of 16 key channels x 64 value columns; A = K~^T (read transposed), B = V
  float4* out = reinterpret_cast<float4*>(p.chunk_state) + (static_cast<int64_t>(chunk) * p.H + h) * p.dk * (p.dv / 4);
  const int nb = (p.dv + 63) / 64, units = (p.dk / 16) * nb;
  const int mat = lane >> 3, mr = lane & 7, g = lane >> 2, t4 = lane & 3;
  for (int u = warp; u < units; u += kThreads / 32) {
    const int c0 = (u / nb) * 16, n0 = (u % nb) * 64;
    float acc[8][4];
#pragma unroll
    for (int i = 0; i < 8; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
#pragma unroll
    for (int ks = 0; ks < kC / 16; ++ks) {
      // transposed 8x8 blocks: matrix 0 = (tokens 0-7, channels 0-7) -> rows 0-7, k 0-7; 1 = channels 8-15; 2 = tokens
      // 8-15; 3 = both
      uint32_t ah[4], al[4];
      const int row = ks * 16 + (mat >> 1) * 8 + mr, col = c0 + (mat & 1) * 8;
      ldmatrix_x4_trans(ah, kh + row * kp + col);
      ldmatrix_x4_trans(al, kl + row * kp + col);
#pragma unroll
      for (int j = 0; j < 8; j += 2) {
        if (n0 + j * 8 >= p.dv) break;
        uint32_t vb[4];
        ldmatrix_x4_trans(vb, vs + (ks * 16 + (mat & 1) * 8 + mr) * vp + n0 + j * 8 + (mat >> 1) * 8);
        mma_bf16(acc[j], ah, vb[0], vb[1]);
        mma_bf16(acc[j], al, vb[0], vb[1]);
        mma_bf16(acc[j + 1], ah, vb[2], vb[3]);
        mma_bf16(acc[j + 1], al, vb[2], vb[3]);
      }
    }
    // accumulator layout (row g, columns 2t, 2t + 1; row g + 8) -> B-fragment layout (rows 2t, 2t + 1, + 8; column g)
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      if (n0 + j * 8 >= p.dv) break;
      const int src = 8 * t4 + (g >> 1);          // lane that holds row 2 t4 and the pair of columns with g in it
      float4 f;
      float a0 = __shfl_sync(0xffffffffu, acc[j][0], src), a1 = __shfl_sync(0xffffffffu, acc[j][1], src);
      f.x = (g & 1) ? a1 : a0;
      a0 = __shfl_sync(0xffffffffu, acc[j][0], src + 4), a1 = __shfl_sync(0xffffffffu, acc[j][1], src + 4);
      f.y = (g & 1) ? a1 : a0;
      a0 = __shfl_sync(0xffffffffu, acc[j][2], src), a1 = __shfl_sync(0xffffffffu, acc[j][3], src);
      f.z = (g & 1) ? a1 : a0;
      a0 = __shfl_sync(0xffffffffu, acc[j][2], src + 4), a1 = __shfl_sync(0xffffffffu, acc[j][3], src + 4);
      f.w = (g & 1) ? a1 : a0;
      out[((c0 / 16) * (p.dv / 8) + n0 / 8 + j) * 32 + lane] = f;
    }
  }
}

// ---------------------------------------------------------------------------------------------------- scan over the chunks
// Thread = one lane's fragment of one 16 x 8 tile of one head's state.
__global__ void __launch_bounds__(256) chunk_scan_kernel(const GlaArgs p) {
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
  const int64_t nhc = static_cast<int64_t>(p.H) * p.dk;
  const float* dec = p.chunk_decay + h * p.dk + row;
  float4* cs = reinterpret_cast<float4*>(p.chunk_state) + e;
  float4 S = make_float4(0.f, 0.f, 0.f, 0.f);
  if (p.pos0[n] != 0) S = make_float4(st[0], st[p.dv], st[8 * p.dv], st[9 * p.dv]);
  const int c0 = p.seq_chunk0[n], c1 = p.seq_chunk0[n + 1];
  constexpr int U = 8;
  for (int c = c0; c < c1; c += U) {
    float4 v[U];
    float2 da[U], db[U];
#pragma unroll
    for (int u = 0; u < U; ++u) {
      if (c + u < c1) {
        v[u] = cs[(c + u) * per];
        da[u] = *reinterpret_cast<const float2*>(dec + (c + u) * nhc);
        db[u] = *reinterpret_cast<const float2*>(dec + (c + u) * nhc + 8);
      }
    }
#pragma unroll
    for (int u = 0; u < U; ++u) {
      if (c + u < c1) {
        const HiLo b0 = split2(S.x, S.y), b1 = split2(S.z, S.w);
        reinterpret_cast<uint4*>(cs)[(c + u) * per] = make_uint4(b0.hi, b1.hi, b0.lo, b1.lo);
        S.x = fmaf(da[u].x, S.x, v[u].x); S.y = fmaf(da[u].y, S.y, v[u].y);
        S.z = fmaf(db[u].x, S.z, v[u].z); S.w = fmaf(db[u].y, S.w, v[u].w);
      }
    }
  }
  st[0] = S.x; st[p.dv] = S.y; st[8 * p.dv] = S.z; st[9 * p.dv] = S.w;
}

// ---------------------------------------------------------------------------------------------------- outputs
constexpr int kAp = kC + 4;       // pitch of the A matrix (fp32)
size_t out_smem(int dk, int dv) {
  return static_cast<size_t>(kC) * (dk + 8) * 4 + 2 * static_cast<size_t>(kC) * (dk + 8) * 2 + static_cast<size_t>(kC) * (dv + 8) * 2 +
         static_cast<size_t>(kC) * kAp * 4 + 8 * kC * 4 + 64;
}

// A[16 x 16 block (bi, bj)], bj < bi, all channels; the products of the block's start as reference.
TDB_DEVICE void block_scores(const GlaArgs& p, const __nv_bfloat16* qs, const __nv_bfloat16* ks, const float* G, float* A, int bi,
                             int bj) {
  const int kp = p.dk + 8, gp = g_pitch(p.dk);
  const int lane = threadIdx.x & 31, g = lane >> 2, t4 = lane & 3;
  const float* ref = G + (bi * 16 - 1) * gp;
  const int r0 = bi * 16 + g, r1 = r0 + 8;
  float acc[2][4] = {};
  for (int k0 = 0; k0 < p.dk; k0 += 16) {
    uint32_t ah[4], al[4];
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int c = k0 + half * 8 + 2 * t4;
      const float f0 = ref[c], f1 = ref[c + 1];
      const float2 a = ld2(qs + r0 * kp + c), b = ld2(qs + r1 * kp + c);
      const HiLo x = split2(a.x * __expf(G[r0 * gp + c] - f0), a.y * __expf(G[r0 * gp + c + 1] - f1));
      const HiLo y = split2(b.x * __expf(G[r1 * gp + c] - f0), b.y * __expf(G[r1 * gp + c + 1] - f1));
      ah[half * 2] = x.hi; al[half * 2] = x.lo;
      ah[half * 2 + 1] = y.hi; al[half * 2 + 1] = y.lo;
    }
#pragma unroll
    for (int nt = 0; nt < 2; ++nt) {
      const int j = bj * 16 + nt * 8 + g;
      HiLo b[2];
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int c = k0 + half * 8 + 2 * t4;
        const float2 k = ld2(ks + j * kp + c);
        b[half] = split2(k.x * __expf(ref[c] - G[j * gp + c]), k.y * __expf(ref[c + 1] - G[j * gp + c + 1]));
      }
      mma_bf16(acc[nt], ah, b[0].hi, b[1].hi);
      mma_bf16(acc[nt], ah, b[0].lo, b[1].lo);
      mma_bf16(acc[nt], al, b[0].hi, b[1].hi);
    }
  }
#pragma unroll
  for (int nt = 0; nt < 2; ++nt) {
    float* a0 = A + r0 * kAp + bj * 16 + nt * 8 + 2 * t4;
    float* a1 = a0 + 8 * kAp;
    a0[0] = acc[nt][0]; a0[1] = acc[nt][1];
    a1[0] = acc[nt][2]; a1[1] = acc[nt][3];
  }
}

// Rows 8-15 against columns 0-7 of the 16-token diagonal block b, on the tensor core.
TDB_DEVICE void diagonal_half(const GlaArgs& p, const __nv_bfloat16* qs, const __nv_bfloat16* ks, const float* G, float* A, int b) {
  const int kp = p.dk + 8, gp = g_pitch(p.dk);
  const int lane = threadIdx.x & 31, g = lane >> 2, t4 = lane & 3;
  const int o = b * 16, r1 = o + 8 + g, j = o + g;
  const float* ref = G + (o + 7) * gp;
  float acc[4] = {};
  for (int k0 = 0; k0 < p.dk; k0 += 16) {
    uint32_t ah[4] = {}, al[4] = {};
    HiLo kb[2];
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int c = k0 + half * 8 + 2 * t4;
      const float f0 = ref[c], f1 = ref[c + 1];
      const float2 q = ld2(qs + r1 * kp + c), k = ld2(ks + j * kp + c);
      const HiLo x = split2(q.x * __expf(G[r1 * gp + c] - f0), q.y * __expf(G[r1 * gp + c + 1] - f1));
      ah[half * 2 + 1] = x.hi; al[half * 2 + 1] = x.lo;
      kb[half] = split2(k.x * __expf(f0 - G[j * gp + c]), k.y * __expf(f1 - G[j * gp + c + 1]));
    }
    mma_bf16(acc, ah, kb[0].hi, kb[1].hi);
    mma_bf16(acc, ah, kb[0].lo, kb[1].lo);
    mma_bf16(acc, al, kb[0].hi, kb[1].hi);
  }
  A[r1 * kAp + o + 2 * t4] = acc[2];
  A[r1 * kAp + o + 2 * t4 + 1] = acc[3];
}

// The eight 8-token triangles on the diagonal (36 pairs each) pair by pair: four lanes share a pair's channels, a thread
// works on five pairs side by side.  Entries above the diagonal of the 16-token blocks become zero.
TDB_DEVICE void triangle_scores(const GlaArgs& p, const __nv_bfloat16* qs, const __nv_bfloat16* ks, const float* G, float* A) {
  constexpr int kPairs = 8 * 36, kPer = (kPairs + kThreads / 4 - 1) / (kThreads / 4);
  const int kp = p.dk + 8, gp = g_pitch(p.dk);
  for (int i = threadIdx.x; i < 4 * 256; i += kThreads) {
    const int o = (i >> 8) * 16, t = (i >> 4) & 15, j = i & 15;
    if (j > t) A[(o + t) * kAp + o + j] = 0.f;
  }
  const int part = threadIdx.x & 3;
  int tt[kPer], jj[kPer];
  float acc[kPer];
#pragma unroll
  for (int i = 0; i < kPer; ++i) {
    const int idx = min((static_cast<int>(threadIdx.x) >> 2) + i * (kThreads / 4), kPairs - 1);
    const int blk = idx / 36;
    int rem = idx - blk * 36, t = 0;
    while (rem > t) rem -= ++t;                        // row t has t + 1 entries
    tt[i] = blk * 8 + t;
    jj[i] = blk * 8 + rem;
    acc[i] = 0.f;
  }
  for (int c = 2 * part; c < p.dk; c += 8) {
#pragma unroll
    for (int i = 0; i < kPer; ++i) {
      const float2 q = ld2(qs + tt[i] * kp + c), k = ld2(ks + jj[i] * kp + c);
      const float2 gt = *reinterpret_cast<const float2*>(G + tt[i] * gp + c), gj = *reinterpret_cast<const float2*>(G + jj[i] * gp + c);
      acc[i] = fmaf(q.x * k.x, __expf(gt.x - gj.x), acc[i]);
      acc[i] = fmaf(q.y * k.y, __expf(gt.y - gj.y), acc[i]);
    }
  }
#pragma unroll
  for (int i = 0; i < kPer; ++i) {
    acc[i] += __shfl_xor_sync(0xffffffffu, acc[i], 1);
    acc[i] += __shfl_xor_sync(0xffffffffu, acc[i], 2);
    if (part == 0) A[tt[i] * kAp + jj[i]] = acc[i];
  }
}

template <int TW>     // 8-column tiles per warp: dv <= 64 TW
__global__ void __launch_bounds__(kThreads, TW <= 2 ? 2 : 1) chunk_out_kernel(const GlaArgs p) {
  extern __shared__ __align__(16) uint8_t smem[];
  const int kp = p.dk + 8, vp = p.dv + 8, gp = g_pitch(p.dk);
  __nv_bfloat16* qs = reinterpret_cast<__nv_bfloat16*>(smem);
  __nv_bfloat16* ks = qs + kC * kp;
  __nv_bfloat16* vs = ks + kC * kp;
  float* A = reinterpret_cast<float*>(vs + kC * vp);
  float* ssq = A + kC * kAp;            // [8 warps][64]
  float* G = ssq + 8 * kC;
  const int chunk = blockIdx.x, h = blockIdx.y;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t4 = lane & 3;
  const int mat = lane >> 3, mr = lane & 7;
  pdl_wait();
  pdl_launch_dependents();
  const ChunkPos cp = chunk_pos(p, chunk);
  const __nv_bfloat16* base = reinterpret_cast<const __nv_bfloat16*>(p.qkvg) + cp.t0 * p.ld;
  const int Hk = p.H * p.dk, Hv = p.H * p.dv;
  load_tile(qs, kp, base + h * p.dk, p.ld, p.dk, cp.n);
  load_tile(ks, kp, base + Hk + h * p.dk, p.ld, p.dk, cp.n);
  load_decays(p, cp, h, G);
  load_tile(vs, vp, base + 2 * Hk + h * p.dv, p.ld, p.dv, cp.n);
  cp_async_commit();
  cp_async_wait<0>();
  __syncthreads();
  if (cp.n < kC) {
    extend_decays(p, cp, G);
    __syncthreads();
  }
  // scores: warps 0-5 one block below the diagonal each, warps 6 and 7 the halves of the diagonal blocks, then all of them
  // the triangles
  if (warp < 6) {
    const int bi = warp < 1 ? 1 : warp < 3 ? 2 : 3, bj = warp - bi * (bi - 1) / 2;
    block_scores(p, qs, ks, G, A, bi, bj);
  } else {
    diagonal_half(p, qs, ks, G, A, 2 * (warp - 6));
    diagonal_half(p, qs, ks, G, A, 2 * (warp - 6) + 1);
  }
  triangle_scores(p, qs, ks, G, A);
  __syncthreads();
  // outputs: a warp owns TW tiles of 8 columns for all 64 tokens, so a fragment of the state is loaded once per CTA.  The
  // first four steps of it are requested now and travel while the queries are prepared.
  constexpr int kAhead = 4;
  const int tiles = p.dv / 8, tile0 = warp * TW, ksteps = p.dk / 16;
  const uint4* S = reinterpret_cast<const uint4*>(p.chunk_state) + (static_cast<int64_t>(chunk) * p.H + h) * p.dk * (p.dv / 4) + lane;
  uint4 sf[kAhead][TW];
  auto fetch = [&](int u, int step) {
#pragma unroll
    for (int j = 0; j < TW; ++j)
      if (step < ksteps && tile0 + j < tiles) sf[u][j] = S[(step * tiles + tile0 + j) * 32];
  };
#pragma unroll
  for (int u = 0; u < kAhead; ++u) fetch(u, u);
  // q e^G in place: high parts over q, low parts over k
  for (int i = threadIdx.x; i < kC * (p.dk / 2); i += kThreads) {
    const int t = i / (p.dk / 2), c = (i - t * (p.dk / 2)) * 2;
    const float2 q = ld2(qs + t * kp + c), gv = *reinterpret_cast<const float2*>(G + t * gp + c);
    const HiLo x = split2(q.x * __expf(gv.x), q.y * __expf(gv.y));
    *reinterpret_cast<uint32_t*>(qs + t * kp + c) = x.hi;
    *reinterpret_cast<uint32_t*>(ks + t * kp + c) = x.lo;
  }
  __syncthreads();
  float acc[4][TW][4];
#pragma unroll
  for (int r = 0; r < 4; ++r)
#pragma unroll
    for (int j = 0; j < TW; ++j) acc[r][j][0] = acc[r][j][1] = acc[r][j][2] = acc[r][j][3] = 0.f;
  if (tile0 < tiles) {
    for (int s0 = 0; s0 < ksteps; s0 += kAhead) {
#pragma unroll
      for (int u = 0; u < kAhead; ++u) {
        if (s0 + u >= ksteps) break;
        const int off = (mat >> 1) * 8 + (s0 + u) * 16;
#pragma unroll
        for (int r = 0; r < 4; ++r) {
          uint32_t ah[4], al[4];
          ldmatrix_x4(ah, qs + (r * 16 + (mat & 1) * 8 + mr) * kp + off);
          ldmatrix_x4(al, ks + (r * 16 + (mat & 1) * 8 + mr) * kp + off);
#pragma unroll
          for (int j = 0; j < TW; ++j) {
            const uint4 b = sf[u][j];        // high parts of both halves of k, then the low parts
            mma_bf16(acc[r][j], ah, b.x, b.y);
            mma_bf16(acc[r][j], ah, b.z, b.w);
            mma_bf16(acc[r][j], al, b.x, b.y);
          }
        }
        fetch(u, s0 + kAhead + u);
      }
    }
#pragma unroll
    for (int kb = 0; kb < 4; ++kb) {
      uint32_t vb[(TW + 1) / 2][4];
#pragma unroll
      for (int j = 0; j < TW; j += 2)      // a single tile reads 8 columns past it: another warp's, or the row's padding
        ldmatrix_x4_trans(vb[j / 2], vs + (kb * 16 + (mat & 1) * 8 + mr) * vp + min(tile0 + j, tiles - 1) * 8 + (mat >> 1) * 8);
#pragma unroll
      for (int r = kb; r < 4; ++r) {
        const float* a0 = A + (r * 16 + g) * kAp + kb * 16 + 2 * t4;
        const float* a1 = a0 + 8 * kAp;
        const HiLo w0 = split2(a0[0], a0[1]), w1 = split2(a1[0], a1[1]), w2 = split2(a0[8], a0[9]), w3 = split2(a1[8], a1[9]);
        const uint32_t ah[4] = {w0.hi, w1.hi, w2.hi, w3.hi}, al[4] = {w0.lo, w1.lo, w2.lo, w3.lo};
#pragma unroll
        for (int j = 0; j < TW; ++j) {
          const uint32_t b0 = vb[j / 2][(j & 1) * 2], b1 = vb[j / 2][(j & 1) * 2 + 1];
          mma_bf16(acc[r][j], ah, b0, b1);
          mma_bf16(acc[r][j], al, b0, b1);
        }
      }
    }
  }
  // head norm over all columns (warps without columns of their own contribute zero), output gate
#pragma unroll
  for (int r = 0; r < 4; ++r) {
    float q0 = 0.f, q1 = 0.f;
#pragma unroll
    for (int j = 0; j < TW; ++j) {
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[r][j][e] = tile0 + j < tiles ? acc[r][j][e] * p.q_scale : 0.f;
      q0 += acc[r][j][0] * acc[r][j][0] + acc[r][j][1] * acc[r][j][1];
      q1 += acc[r][j][2] * acc[r][j][2] + acc[r][j][3] * acc[r][j][3];
    }
    q0 += __shfl_xor_sync(0xffffffffu, q0, 1); q0 += __shfl_xor_sync(0xffffffffu, q0, 2);
    q1 += __shfl_xor_sync(0xffffffffu, q1, 1); q1 += __shfl_xor_sync(0xffffffffu, q1, 2);
    if (t4 == 0) {
      ssq[warp * kC + r * 16 + g] = q0;
      ssq[warp * kC + r * 16 + g + 8] = q1;
    }
  }
  __syncthreads();
#pragma unroll
  for (int r = 0; r < 4; ++r) {
#pragma unroll
    for (int rr = 0; rr < 2; ++rr) {
      const int t = r * 16 + rr * 8 + g;
      if (t >= cp.n) continue;
      float sum = 0.f;
#pragma unroll
      for (int w = 0; w < 8; ++w) sum += ssq[w * kC + t];
      const float inv = 1.f / sqrtf(sum / p.dv_real + p.eps);
      const __nv_bfloat16* gate = base + t * p.ld + 2 * Hk + Hv + h * p.dv;
      __nv_bfloat16* out = reinterpret_cast<__nv_bfloat16*>(p.out) + (cp.t0 + t) * Hv + h * p.dv;
#pragma unroll
      for (int j = 0; j < TW; ++j) {
        if (tile0 + j < tiles) {
          const int c = (tile0 + j) * 8 + 2 * t4;
          const float2 gt = ld2(gate + c);
          const float o0 = acc[r][j][2 * rr] * inv * p.norm_w[c] * gt.x * sigmoid_f32(gt.x);
          const float o1 = acc[r][j][2 * rr + 1] * inv * p.norm_w[c + 1] * gt.y * sigmoid_f32(gt.y);
          *reinterpret_cast<uint32_t*>(out + c) = pack_bf16x2(o0, o1);
        }
      }
    }
  }
}

template <int TW>
cudaError_t launch_out(const GlaArgs& a, cudaStream_t s) {
  static SmemOptIn opt;
  cudaError_t e = opt.ensure(chunk_out_kernel<TW>, 227 * 1024);
  if (e != cudaSuccess) return e;
  return launch_pdl(chunk_out_kernel<TW>, dim3(a.NC, a.H), dim3(kThreads), out_smem(a.dk, a.dv), s, a);
}

}  // namespace

bool gla_chunk_supported(int dk, int dv) {
  return dk % 16 == 0 && dv % 16 == 0 && dv <= 256 && dk <= 256 && out_smem(dk, dv) <= 227 * 1024 && kv_smem(dk, dv) <= 227 * 1024;
}

cudaError_t launch_gla_chunk(const GlaArgs& a, cudaStream_t s) {
  if (a.is_f32 || !gla_chunk_supported(a.dk, a.dv) || a.ld % 8 != 0 || a.cu == nullptr || a.H > 65535) return cudaErrorInvalidValue;
  if (a.T == 0 || a.N == 0) return cudaSuccess;
  if (a.NC > 65535) return cudaErrorInvalidValue;
  cudaError_t e = launch_pdl(chunk_decay_kernel, dim3((a.H * a.dk + 255) / 256, a.NC), dim3(256),
                             static_cast<size_t>(kDecayTok * a.R * 4), s, a);
  if (e != cudaSuccess) return e;
  static SmemOptIn opt;
  e = opt.ensure(chunk_kv_kernel, 227 * 1024);
  if (e != cudaSuccess) return e;
  e = launch_pdl(chunk_kv_kernel, dim3(a.NC, a.H), dim3(kThreads), kv_smem(a.dk, a.dv), s, a);
  if (e != cudaSuccess) return e;
  const int64_t per = static_cast<int64_t>(a.H) * a.dk * (a.dv / 4);
  e = launch_pdl(chunk_scan_kernel, dim3(static_cast<unsigned>((per + 255) / 256), a.N), dim3(256), 0, s, a);
  if (e != cudaSuccess) return e;
  if (a.dv <= 64) return launch_out<1>(a, s);
  if (a.dv <= 128) return launch_out<2>(a, s);
  return launch_out<4>(a, s);
}

}  // namespace tdb
