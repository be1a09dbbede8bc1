// Gated linear attention, chunk-parallel form for bf16 activations (recurrence in gla.cu).
//
// With G_t the cumulative log decay inside a 64-token chunk (per key channel, inclusive) and S the state before it:
//     o_t   = q_scale ( (q_t e^{G_t}) S  +  sum_{j <= t} A_tj v_j ),   A_tj = sum_c q_tc k_jc e^{G_tc - G_jc}
//     S_end = e^{G_63} S + sum_j (k_j e^{G_63 - G_j}) v_j^T
// Three launches after the log decays:
//   chunk_kv_kernel    one CTA per (chunk, head): the chunk's own contribution to the state and its total decay
//   chunk_scan_kernel  the sequential part, element-wise: turns contributions into the state BEFORE every chunk (in place)
//                      and writes the sequence's final state; a stream of fp32 values, split over all state elements
//   chunk_out_kernel   one CTA per (chunk, head): A, outputs, head norm and output gate
//
// Decays can be arbitrarily strong, so an exponential is only ever taken of a difference that is <= 0: A between two
// 16-token blocks uses the later block's start as the reference of both factors (q_t e^{G_t - G_ref}, k_j e^{G_ref - G_j}),
// a 16-token diagonal block is cut once more the same way, and its two 8-token triangles are summed pair by pair.
//
// The state and everything that enters it count as fp32, so the tensor cores (mma.sync bf16, fp32 accumulate) get every
// fp32 operand as a high and a low bf16 part: two products where one side is bf16 anyway (v), three where both are fp32.
#include "tdb/attn_device.cuh"
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

constexpr int kC = 64;            // tokens per chunk
constexpr int kThreads = 256;

struct HiLo {
  uint32_t hi, lo;
};
// Two fp32 values as packed bf16 high parts and packed bf16 remainders.
TDB_DEVICE HiLo split2(float a, float b) {
  HiLo r;
  r.hi = pack_bf16x2(a, b);
  const float2 h = unpack_bf16x2(r.hi);
  r.lo = pack_bf16x2(a - h.x, b - h.y);
  return r;
}
TDB_DEVICE float2 ld2(const __nv_bfloat16* p) { return unpack_bf16x2(*reinterpret_cast<const uint32_t*>(p)); }

struct ChunkPos {
  int64_t t0;
  int n;       // tokens of the chunk
};
TDB_DEVICE ChunkPos chunk_pos(const GlaArgs& p, int chunk) {
  ChunkPos r;
  r.t0 = p.chunk_t0[chunk];
  const int64_t end = p.cu[p.chunk_seq[chunk] + 1];
  r.n = static_cast<int>(min(static_cast<int64_t>(kC), end - r.t0));
  return r;
}

// Rows [0, 64) of `cols` bf16 columns starting at src (row stride ld) into smem with row pitch `pitch` elements; rows >= n
// are zero.
TDB_DEVICE void load_tile(__nv_bfloat16* dst, int pitch, const __nv_bfloat16* src, int64_t ld, int cols, int n) {
  const int vec = cols >> 3;
  for (int i = threadIdx.x; i < kC * vec; i += kThreads) {
    const int r = i / vec, c = i - r * vec;
    cp_async16(dst + r * pitch + c * 8, src + (r < n ? r * ld : 0) + c * 8, r < n);
  }
}

// Inclusive cumulative sums over the tokens of the log decays of one head into G [64][dk + 1].
TDB_DEVICE void cumulate(const GlaArgs& p, const ChunkPos& cp, int h, float* G) {
  const int C = p.H * p.dk, gp = p.dk + 1;
  const float* src = p.log_decay + cp.t0 * C + h * p.dk;
  for (int c = threadIdx.x; c < p.dk; c += kThreads) {
    float acc = 0.f;
#pragma unroll 8
    for (int t = 0; t < kC; ++t) {
      if (t < cp.n) acc += src[static_cast<int64_t>(t) * C + c];
      G[t * gp + c] = acc;
    }
  }
}

// ---------------------------------------------------------------------------------------------------- state contributions
size_t kv_smem(int dk, int dv) {
  return static_cast<size_t>(kC) * (dk + 1) * 4 + 3 * static_cast<size_t>(kC) * (dk + 8) * 2 + static_cast<size_t>(kC) * (dv + 8) * 2 + 64;
}

__global__ void __launch_bounds__(kThreads) chunk_kv_kernel(const GlaArgs p) {
  extern __shared__ __align__(16) uint8_t smem[];
  const int kp = p.dk + 8, vp = p.dv + 8, gp = p.dk + 1;
  __nv_bfloat16* kr = reinterpret_cast<__nv_bfloat16*>(smem);     // raw keys, then unused
  __nv_bfloat16* kh = kr + kC * kp;
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
  load_tile(kr, kp, base + Hk + h * p.dk, p.ld, p.dk, cp.n);
  load_tile(vs, vp, base + 2 * Hk + h * p.dv, p.ld, p.dv, cp.n);
  cp_async_commit();
  cumulate(p, cp, h, G);
  cp_async_wait<0>();
  __syncthreads();
  const float* gl = G + (kC - 1) * gp;
  float* dec = p.chunk_decay + (static_cast<int64_t>(chunk) * p.H + h) * p.dk;
  for (int c = threadIdx.x; c < p.dk; c += kThreads) dec[c] = expf(gl[c]);
  for (int i = threadIdx.x; i < kC * (p.dk / 2); i += kThreads) {
    const int t = i / (p.dk / 2), c = (i - t * (p.dk / 2)) * 2;
    const float2 k = ld2(kr + t * kp + c);
    const HiLo s = split2(k.x * __expf(gl[c] - G[t * gp + c]), k.y * __expf(gl[c + 1] - G[t * gp + c + 1]));
    *reinterpret_cast<uint32_t*>(kh + t * kp + c) = s.hi;
    *reinterpret_cast<uint32_t*>(kl + t * kp + c) = s.lo;
  }
  __syncthreads();
  // units of 16 key channels x 64 value columns; A = K~^T (read transposed), B = V
  float* out = p.chunk_state + (static_cast<int64_t>(chunk) * p.H + h) * p.dk * p.dv;
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
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      if (n0 + j * 8 >= p.dv) break;
      float* o = out + static_cast<int64_t>(c0 + g) * p.dv + n0 + j * 8 + 2 * t4;
      *reinterpret_cast<float2*>(o) = make_float2(acc[j][0], acc[j][1]);
      *reinterpret_cast<float2*>(o + 8 * p.dv) = make_float2(acc[j][2], acc[j][3]);
    }
  }
}

// ---------------------------------------------------------------------------------------------------- scan over the chunks
__global__ void __launch_bounds__(256) chunk_scan_kernel(const GlaArgs p) {
  const int n = blockIdx.y;
  const int dv4 = p.dv >> 2;
  const int64_t per = static_cast<int64_t>(p.H) * p.dk * dv4;      // float4 elements of one chunk's state
  const int64_t e = static_cast<int64_t>(blockIdx.x) * 256 + threadIdx.x;
  pdl_wait();
  pdl_launch_dependents();
  if (e >= per) return;
  const int64_t hc = e / dv4;                                      // (head, key channel)
  const int64_t nhc = static_cast<int64_t>(p.H) * p.dk;
  float4* st = reinterpret_cast<float4*>(p.state) + static_cast<int64_t>(p.slots[n]) * per + e;
  float4* cs = reinterpret_cast<float4*>(p.chunk_state) + e;
  float4 S = p.pos0[n] == 0 ? make_float4(0.f, 0.f, 0.f, 0.f) : *st;
  const int c0 = p.seq_chunk0[n], c1 = p.seq_chunk0[n + 1];
  constexpr int U = 8;
  for (int c = c0; c < c1; c += U) {
    float4 v[U];
    float d[U];
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const bool ok = c + u < c1;
      v[u] = ok ? cs[(c + u) * per] : make_float4(0.f, 0.f, 0.f, 0.f);
      d[u] = ok ? p.chunk_decay[(c + u) * nhc + hc] : 1.f;
    }
#pragma unroll
    for (int u = 0; u < U; ++u) {
      if (c + u < c1) {
        cs[(c + u) * per] = S;
        S.x = fmaf(d[u], S.x, v[u].x); S.y = fmaf(d[u], S.y, v[u].y);
        S.z = fmaf(d[u], S.z, v[u].z); S.w = fmaf(d[u], S.w, v[u].w);
      }
    }
  }
  *st = S;
}

// ---------------------------------------------------------------------------------------------------- outputs
constexpr int kAp = kC + 4;       // pitch of the A matrix (fp32)
size_t out_smem(int dk, int dv) {
  return static_cast<size_t>(kC) * (dk + 1) * 4 + 2 * static_cast<size_t>(kC) * (dk + 8) * 2 + static_cast<size_t>(kC) * (dv + 8) * 2 +
         static_cast<size_t>(kC) * kAp * 4 + 2 * kC * 4 + 64;
}

// A[16 x 16 block (bi, bj)], bj < bi, all channels; the products of the block's start as reference.
TDB_DEVICE void block_scores(const GlaArgs& p, const __nv_bfloat16* qs, const __nv_bfloat16* ks, const float* G, float* A, int bi,
                             int bj) {
  const int kp = p.dk + 8, gp = p.dk + 1;
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

// The 16-token diagonal block b: rows 8-15 against columns 0-7 on the tensor core, the two 8-token triangles pair by pair.
TDB_DEVICE void diagonal_scores(const GlaArgs& p, const __nv_bfloat16* qs, const __nv_bfloat16* ks, const float* G, float* A, int b) {
  const int kp = p.dk + 8, gp = p.dk + 1;
  const int lane = threadIdx.x & 31, g = lane >> 2, t4 = lane & 3;
  const int o = b * 16;
  for (int i = lane; i < 256; i += 32) A[(o + i / 16) * kAp + o + i % 16] = 0.f;
  __syncwarp();
  {
    const float* ref = G + (o + 7) * gp;
    const int r1 = o + 8 + g, j = o + g;
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
    float* a1 = A + r1 * kAp + o + 2 * t4;
    a1[0] = acc[2];
    a1[1] = acc[3];
  }
#pragma unroll
  for (int i = 0; i < 3; ++i) {
    const int idx = lane + 32 * i;                       // 72 pairs: two lower triangles of 36
    if (idx < 72) {
      const int blk = idx / 36;
      int rem = idx - blk * 36, t = 0;
      while (rem > t) rem -= ++t;                        // row t has t + 1 entries
      const int tt = o + blk * 8 + t, jj = o + blk * 8 + rem;
      const float *gt = G + tt * gp, *gj = G + jj * gp;
      float s = 0.f;
#pragma unroll 4
      for (int c = 0; c < p.dk; c += 2) {
        const float2 q = ld2(qs + tt * kp + c), k = ld2(ks + jj * kp + c);
        s = fmaf(q.x * k.x, __expf(gt[c] - gj[c]), s);
        s = fmaf(q.y * k.y, __expf(gt[c + 1] - gj[c + 1]), s);
      }
      A[tt * kAp + jj] = s;
    }
  }
}

template <int NT>     // 8-column tiles per warp: dv <= 16 NT
__global__ void __launch_bounds__(kThreads) chunk_out_kernel(const GlaArgs p) {
  extern __shared__ __align__(16) uint8_t smem[];
  const int kp = p.dk + 8, vp = p.dv + 8, gp = p.dk + 1;
  __nv_bfloat16* qs = reinterpret_cast<__nv_bfloat16*>(smem);
  __nv_bfloat16* ks = qs + kC * kp;
  __nv_bfloat16* vs = ks + kC * kp;
  float* A = reinterpret_cast<float*>(vs + kC * vp);
  float* ssq = A + kC * kAp;            // [2][64]
  float* G = ssq + 2 * kC;
  const int chunk = blockIdx.x, h = blockIdx.y;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t4 = lane & 3;
  pdl_wait();
  pdl_launch_dependents();
  const ChunkPos cp = chunk_pos(p, chunk);
  const __nv_bfloat16* base = reinterpret_cast<const __nv_bfloat16*>(p.qkvg) + cp.t0 * p.ld;
  const int Hk = p.H * p.dk, Hv = p.H * p.dv;
  load_tile(qs, kp, base + h * p.dk, p.ld, p.dk, cp.n);
  load_tile(ks, kp, base + Hk + h * p.dk, p.ld, p.dk, cp.n);
  load_tile(vs, vp, base + 2 * Hk + h * p.dv, p.ld, p.dv, cp.n);
  cp_async_commit();
  cumulate(p, cp, h, G);
  cp_async_wait<0>();
  __syncthreads();
  // scores: warps 0-3 the diagonal blocks, warps 4-7 the six blocks below them
  if (warp < 4) {
    diagonal_scores(p, qs, ks, G, A, warp);
  } else {
    const int w = warp - 4;
    if (w == 0) { block_scores(p, qs, ks, G, A, 1, 0); block_scores(p, qs, ks, G, A, 3, 0); }
    if (w == 1) { block_scores(p, qs, ks, G, A, 2, 0); block_scores(p, qs, ks, G, A, 3, 1); }
    if (w == 2) block_scores(p, qs, ks, G, A, 2, 1);
    if (w == 3) block_scores(p, qs, ks, G, A, 3, 2);
  }
  __syncthreads();
  // outputs: warp = 16 tokens x half of the columns
  const int rg = warp & 3, half = warp >> 2;
  const int n0 = half * (p.dv / 2), nt_here = p.dv / 16;
  const int r0 = rg * 16 + g, r1 = r0 + 8;
  float acc[NT][4];
#pragma unroll
  for (int i = 0; i < NT; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
  const float* S = p.chunk_state + (static_cast<int64_t>(chunk) * p.H + h) * p.dk * p.dv + n0;
  for (int k0 = 0; k0 < p.dk; k0 += 16) {
    uint32_t ah[4], al[4];
#pragma unroll
    for (int hf = 0; hf < 2; ++hf) {
      const int c = k0 + hf * 8 + 2 * t4;
      const float2 a = ld2(qs + r0 * kp + c), b = ld2(qs + r1 * kp + c);
      const HiLo x = split2(a.x * __expf(G[r0 * gp + c]), a.y * __expf(G[r0 * gp + c + 1]));
      const HiLo y = split2(b.x * __expf(G[r1 * gp + c]), b.y * __expf(G[r1 * gp + c + 1]));
      ah[hf * 2] = x.hi; al[hf * 2] = x.lo;
      ah[hf * 2 + 1] = y.hi; al[hf * 2 + 1] = y.lo;
    }
    const float* s0 = S + static_cast<int64_t>(k0 + 2 * t4) * p.dv + g;
#pragma unroll
    for (int j = 0; j < NT; ++j) {
      if (j < nt_here) {
        const float* s = s0 + j * 8;
        const HiLo b0 = split2(s[0], s[p.dv]);
        const HiLo b1 = split2(s[8 * p.dv], s[9 * p.dv]);
        mma_bf16(acc[j], ah, b0.hi, b1.hi);
        mma_bf16(acc[j], ah, b0.lo, b1.lo);
        mma_bf16(acc[j], al, b0.hi, b1.hi);
      }
    }
  }
  const int mat = lane >> 3, mr = lane & 7;
  for (int kb = 0; kb <= rg; ++kb) {
    const float* a0 = A + r0 * kAp + kb * 16 + 2 * t4;
    const float* a1 = a0 + 8 * kAp;
    const HiLo w0 = split2(a0[0], a0[1]), w1 = split2(a1[0], a1[1]), w2 = split2(a0[8], a0[9]), w3 = split2(a1[8], a1[9]);
    const uint32_t ah[4] = {w0.hi, w1.hi, w2.hi, w3.hi}, al[4] = {w0.lo, w1.lo, w2.lo, w3.lo};
    const __nv_bfloat16* vrow = vs + (kb * 16 + (mat & 1) * 8 + mr) * vp + n0 + (mat >> 1) * 8;
#pragma unroll
    for (int j = 0; j < NT; j += 2) {
      if (j < nt_here) {
        uint32_t vb[4];
        // with an odd number of tiles the last pair reads 8 columns past this half: inside the padded row, not used
        ldmatrix_x4_trans(vb, vrow + j * 8);
        mma_bf16(acc[j], ah, vb[0], vb[1]);
        mma_bf16(acc[j], al, vb[0], vb[1]);
        if (j + 1 < nt_here) {
          mma_bf16(acc[j + 1], ah, vb[2], vb[3]);
          mma_bf16(acc[j + 1], al, vb[2], vb[3]);
        }
      }
    }
  }
  // head norm over both halves, output gate
  float q0 = 0.f, q1 = 0.f;
#pragma unroll
  for (int j = 0; j < NT; ++j) {
    acc[j][0] *= p.q_scale; acc[j][1] *= p.q_scale; acc[j][2] *= p.q_scale; acc[j][3] *= p.q_scale;
    q0 += acc[j][0] * acc[j][0] + acc[j][1] * acc[j][1];
    q1 += acc[j][2] * acc[j][2] + acc[j][3] * acc[j][3];
  }
  q0 += __shfl_xor_sync(0xffffffffu, q0, 1); q0 += __shfl_xor_sync(0xffffffffu, q0, 2);
  q1 += __shfl_xor_sync(0xffffffffu, q1, 1); q1 += __shfl_xor_sync(0xffffffffu, q1, 2);
  if (t4 == 0) {
    ssq[half * kC + r0] = q0;
    ssq[half * kC + r1] = q1;
  }
  __syncthreads();
#pragma unroll
  for (int rr = 0; rr < 2; ++rr) {
    const int r = rr ? r1 : r0;
    if (r >= cp.n) continue;
    const float inv = 1.f / sqrtf((ssq[r] + ssq[kC + r]) / p.dv_real + p.eps);
    const __nv_bfloat16* gate = base + r * p.ld + 2 * Hk + Hv + h * p.dv + n0;
    __nv_bfloat16* out = reinterpret_cast<__nv_bfloat16*>(p.out) + (cp.t0 + r) * Hv + h * p.dv + n0;
#pragma unroll
    for (int j = 0; j < NT; ++j) {
      if (j < nt_here) {
        const int c = j * 8 + 2 * t4;
        const float2 gt = ld2(gate + c);
        const float o0 = acc[j][2 * rr] * inv * p.norm_w[n0 + c] * gt.x * sigmoid_f32(gt.x);
        const float o1 = acc[j][2 * rr + 1] * inv * p.norm_w[n0 + c + 1] * gt.y * sigmoid_f32(gt.y);
        *reinterpret_cast<uint32_t*>(out + c) = pack_bf16x2(o0, o1);
      }
    }
  }
}

template <int NT>
cudaError_t launch_out(const GlaArgs& a, cudaStream_t s) {
  static SmemOptIn opt;
  cudaError_t e = opt.ensure(chunk_out_kernel<NT>, 227 * 1024);
  if (e != cudaSuccess) return e;
  return launch_pdl(chunk_out_kernel<NT>, dim3(a.NC, a.H), dim3(kThreads), out_smem(a.dk, a.dv), s, a);
}

}  // namespace

bool gla_chunk_supported(int dk, int dv) {
  return dk % 16 == 0 && dv % 16 == 0 && dv <= 256 && dk <= 256 && out_smem(dk, dv) <= 227 * 1024 && kv_smem(dk, dv) <= 227 * 1024;
}

cudaError_t launch_gla_chunk(const GlaArgs& a, cudaStream_t s) {
  if (a.is_f32 || !gla_chunk_supported(a.dk, a.dv) || a.ld % 8 != 0 || a.cu == nullptr || a.H > 65535) return cudaErrorInvalidValue;
  if (a.T == 0 || a.N == 0) return cudaSuccess;
  cudaError_t e = launch_gla_log_decay(a, s);
  if (e != cudaSuccess) return e;
  static SmemOptIn opt;
  e = opt.ensure(chunk_kv_kernel, 227 * 1024);
  if (e != cudaSuccess) return e;
  e = launch_pdl(chunk_kv_kernel, dim3(a.NC, a.H), dim3(kThreads), kv_smem(a.dk, a.dv), s, a);
  if (e != cudaSuccess) return e;
  const int64_t per = static_cast<int64_t>(a.H) * a.dk * (a.dv / 4);
  e = launch_pdl(chunk_scan_kernel, dim3(static_cast<unsigned>((per + 255) / 256), a.N), dim3(256), 0, s, a);
  if (e != cudaSuccess) return e;
  if (a.dv <= 64) return launch_out<4>(a, s);
  if (a.dv <= 128) return launch_out<8>(a, s);
  return launch_out<16>(a, s);
}

}  // namespace tdb
