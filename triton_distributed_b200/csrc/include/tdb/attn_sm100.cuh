// Softmax warps of the tcgen05 prompt-attention kernels (attn_sm100.cu, latent_sm100.cu): tiles of 128 query rows, blocks of 64
// keys, S and O in TMEM, P through 128-byte-swizzled shared memory.
#pragma once
#include <cuda_bf16.h>

#include "attn.h"
#include "attn_device.cuh"
#include "ptx.cuh"

namespace tdb {
namespace {

constexpr int kBM = 128;           // query rows per tile
constexpr int kBN = 64;            // KV tokens per block
constexpr uint64_t kWaitNs = 4000000000ull;

__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

struct FwdParams {
  const __nv_bfloat16* q;
  __nv_bfloat16* out;
  float* lse;                  // [Hq, total_q] or null
  const int32_t* cu_seqlens_q;
  const int32_t* q_pos0;
  const int32_t* kv_lens;
  int Hq, Hkv, group, causal;
  int dv;                      // columns of an output row
  float scale_log2;            // scale * log2(e)
  float cap_log2 = 0.f;        // soft cap * log2(e), 0 = none: the score s becomes cap * tanh(s * scale / cap)
  float to_cap = 0.f;          // scale / cap
  int64_t total_q;
  int* error_flag;             // device int, set on a timeout
  AttnEpilogue epi;            // sink / output gate of the rows
};

// What one softmax thread (one query row of one 128-row tile) does over all KV blocks of its tile, then the output row.
struct TileCtx {
  uint64_t* s_full;
  uint64_t* s_free;
  uint64_t* p_full;
  uint64_t* pv_full;
  uint32_t tmem_s, tmem_pv;
  uint8_t* p_smem;             // this tile's P buffer
  int row0, rows_here, nblk;
};

// DV: columns of the output accumulator (a multiple of 32); the rows written have p.dv <= DV columns, a multiple of 8.  CAP: with
// soft cap.
template <int DV, bool CAP = false>
__device__ __forceinline__ void softmax_tile(const FwdParams& p, const TileCtx& t, int warp, int lane, int q_begin, int head,
                                             int kv_len, int pos0, volatile int* abort_flag) {
  uint64_t* s_full = t.s_full;
  uint64_t* s_free = t.s_free;
  uint64_t* p_full = t.p_full;
  uint64_t* pv_full = t.pv_full;
  const uint32_t tmem_s = t.tmem_s, tmem_pv = t.tmem_pv;
  const int row0 = t.row0, rows_here = t.rows_here, nblk = t.nblk;
  const int qd = warp & 3;                       // TMEM lane quarter this warp may access
  const int row = qd * 32 + lane;                // row inside the tile
  const bool row_ok = row < rows_here;
  const int pos = pos0 + row0 + row;             // absolute position of the query
  const int lim = p.causal ? min(kv_len, pos + 1) : kv_len;   // tokens [0, lim) are visible
  const uint32_t lane_off = static_cast<uint32_t>(qd * 32) << 16;
  constexpr float kRescaleStep = 8.f;            // log2: the reference maximum follows the row maximum in steps of 2^8
  float m = -INFINITY, l = 0.f;                  // m: reference maximum the exponentials of this row use
  uint8_t* prow = t.p_smem + row * 128;
  const int sw = row & 7;
  bool ok = true;
  for (int j = 0; j < nblk; ++j) {
    if (!mbar_wait(s_full, j & 1, abort_flag, kWaitNs)) { ok = false; break; }
    tc_fence_after_sync();
    uint32_t s0[32], s1[32];
    tmem_ld_32x32(tmem_s + lane_off, s0);
    tmem_ld_32x32(tmem_s + lane_off + 32, s1);
    tmem_ld_wait();
    tc_fence_before_sync();
    mbar_arrive(s_free);                          // S may be overwritten by the next block's product
    const int t0 = j * kBN;
    // Blocks that every row of the warp sees completely (all but the ones on the causal diagonal and the last one of
    // a sequence) skip the masking; the scale is folded into the exponent (one FMA per element), so an element
    // costs a max, an FMA, an ex2, an add and half a pack.
    const bool full = __all_sync(0xffffffffu, t0 + kBN <= lim);
    if constexpr (CAP) {
      attn::cap_scores(reinterpret_cast<float (&)[32]>(s0), p.to_cap, p.cap_log2);
      attn::cap_scores(reinterpret_cast<float (&)[32]>(s1), p.to_cap, p.cap_log2);
    }
    if (!full) {
#pragma unroll
      for (int c = 0; c < 32; ++c) {
        if (t0 + c >= lim) s0[c] = 0xff800000u;          // -inf
        if (t0 + 32 + c >= lim) s1[c] = 0xff800000u;
      }
    }
    float mx = -INFINITY;
#pragma unroll
    for (int c = 0; c < 32; ++c) mx = fmaxf(mx, fmaxf(__uint_as_float(s0[c]), __uint_as_float(s1[c])));
    const float scale_log2 = CAP ? 1.f : p.scale_log2;    // capped scores are in the log2 domain already
    mx *= scale_log2;                                     // scale > 0: the maximum commutes with it
    // raise the reference only when the row maximum has outgrown it by more than the step (or there is none yet)
    float alpha = 1.f;
    bool raise = false;
    if (mx > m) {
      if (m == -INFINITY) {
        m = mx;                                   // nothing accumulated for this row so far (its P were all zero)
      } else if (mx - m > kRescaleStep) {
        alpha = ex2(m - mx);
        m = mx;
        raise = true;
      }
    }
    const float m_use = (m == -INFINITY) ? 0.f : m;
    // the previous block's PV must have finished: it read the P buffer that is rewritten below, and it wrote the O
    // rows a rescale touches (issued long ago: this wait is normally already satisfied)
    if (j > 0 && !mbar_wait(pv_full, (j - 1) & 1, abort_flag, kWaitNs)) { ok = false; break; }
    if (__any_sync(0xffffffffu, raise)) {
      tc_fence_after_sync();
#pragma unroll
      for (int c = 0; c < DV / 32; ++c) {
        uint32_t r[32];
        tmem_ld_32x32(tmem_pv + lane_off + c * 32, r);
        tmem_ld_wait();
#pragma unroll
        for (int i = 0; i < 32; ++i) r[i] = __float_as_uint(__uint_as_float(r[i]) * alpha);
        tmem_st_32x32(tmem_pv + lane_off + c * 32, r);
      }
      tmem_st_wait();
      tc_fence_before_sync();
    }
    float sum = 0.f;
    // P row: 64 bf16 = eight 16-byte chunks, chunk c stored at (c ^ (row & 7)) (128-byte swizzle)
#pragma unroll
    for (int c8 = 0; c8 < 8; ++c8) {
      uint32_t pk[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int c = c8 * 8 + 2 * e;
        const float x0 = ex2(fmaf(__uint_as_float(c < 32 ? s0[c] : s1[c - 32]), scale_log2, -m_use));
        const float x1 = ex2(fmaf(__uint_as_float(c + 1 < 32 ? s0[c + 1] : s1[c + 1 - 32]), scale_log2, -m_use));
        sum += x0 + x1;
        pk[e] = pack_bf16x2(x0, x1);
      }
      *reinterpret_cast<uint4*>(prow + ((c8 ^ sw) << 4)) = make_uint4(pk[0], pk[1], pk[2], pk[3]);
    }
    l = l * alpha + sum;
    fence_proxy_async_smem();                     // P was written through the generic proxy, the MMA reads it through the async proxy
    mbar_arrive(p_full);
  }
  float o[DV];
#pragma unroll
  for (int i = 0; i < DV; ++i) o[i] = 0.f;
  if (ok && nblk > 0) {
    if (!mbar_wait(pv_full, (nblk - 1) & 1, abort_flag, kWaitNs)) {
      ok = false;
    } else {
      tc_fence_after_sync();
#pragma unroll
      for (int c = 0; c < DV / 32; ++c) {
        uint32_t r[32];
        tmem_ld_32x32(tmem_pv + lane_off + c * 32, r);
        tmem_ld_wait();
#pragma unroll
        for (int i = 0; i < 32; ++i) o[c * 32 + i] = __uint_as_float(r[i]);
      }
      tc_fence_before_sync();
    }
  }
  if (!ok) *abort_flag = 1;
  if (ok && row_ok) {
    float inv = l > 0.f ? 1.f / l : 0.f;
    const int64_t tok = static_cast<int64_t>(q_begin) + row0 + row;
    if (p.epi.sink != nullptr && l > 0.f) {
      const float lse = (m + log2f(l)) * 0.6931471805599453f;
      inv /= 1.f + __expf(p.epi.sink[head] - lse);
    }
    if (p.epi.gate != nullptr) {
      const uint4* g4 = reinterpret_cast<const uint4*>(reinterpret_cast<const __nv_bfloat16*>(p.epi.gate) +
                                                       tok * p.epi.ld_gate + static_cast<int64_t>(head) * p.dv);
#pragma unroll
      for (int c = 0; c < DV / 8; ++c) {
        if (8 * c >= p.dv) break;
        const uint4 u = g4[c];
        const uint32_t w[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float2 z = unpack_bf16x2(w[e]);
          o[8 * c + 2 * e] *= 1.f / (1.f + __expf(-z.x));
          o[8 * c + 2 * e + 1] *= 1.f / (1.f + __expf(-z.y));
        }
      }
    }
    __nv_bfloat16* orow = p.out + (tok * p.Hq + head) * p.dv;
#pragma unroll
    for (int c = 0; c < DV / 8; ++c) {
      if (8 * c >= p.dv) break;
      uint4 v;
      v.x = pack_bf16x2(o[8 * c + 0] * inv, o[8 * c + 1] * inv);
      v.y = pack_bf16x2(o[8 * c + 2] * inv, o[8 * c + 3] * inv);
      v.z = pack_bf16x2(o[8 * c + 4] * inv, o[8 * c + 5] * inv);
      v.w = pack_bf16x2(o[8 * c + 6] * inv, o[8 * c + 7] * inv);
      *reinterpret_cast<uint4*>(orow + 8 * c) = v;
    }
    if (p.lse != nullptr)
      p.lse[static_cast<int64_t>(head) * p.total_q + q_begin + row0 + row] =
          l > 0.f ? (m + log2f(l)) * 0.6931471805599453f : -INFINITY;
  }
}

}  // namespace
}  // namespace tdb
