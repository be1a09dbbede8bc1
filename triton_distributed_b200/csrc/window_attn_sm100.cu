// Prompt attention over a sliding window on the 5th-generation tensor cores (bf16; tdb/window.h states the two kinds).
//
// One CTA works on two tiles of 128 query rows that share every block of 64 values (320 threads: warp 0 TMA, warp 1 MMA, warps 2-5
// and 6-9 the scores of a tile each; while one tile's rows are in their exponentials the other tile's products are on the tensor core):
//   sigmoid        the tiles are neighbouring rows of one head and share the keys too; each has its own range of blocks, because the
//                  window moves with the rows.  Weights need no maximum and no sum.  The distance term of a warp's 32 rows and a
//                  block's 64 keys takes 95 neighbouring values of the head's table, which the warp keeps in shared memory and
//                  requests a block ahead.  Two weights share one reciprocal: 1/a = b/(ab), 1/b = a/(ab).
//   differential   the tiles are the two maps of the same rows of a head.  Softmax with a lagging reference maximum (raised only when
//                  the row maximum has outgrown it by 2^8); at the end the second map's rows go through shared memory to the first
//                  map's threads, which take the difference, norm and gate it and write it.
// Keys and values come straight from the packed rows by TMA: blocks start at the first row that the tile's window touches, values are
// the MN-major operand of the second product, so nothing is transposed or padded in memory.
//
// Every wait is bounded; a timeout is recorded, the CTA stops issuing work, frees its TMEM and returns.
#include <cuda.h>
#include <cuda_bf16.h>

#include <cstring>

#include "tdb/api.h"
#include "tdb/attn_sm100.cuh"
#include "tdb/launch.cuh"
#include "tdb/ptx.cuh"
#include "tdb/window.h"

namespace tdb {

namespace {

constexpr int kThreads = 320;
constexpr int kUmmaK = 16;
constexpr int kQChunk = kBM * 128;      // 128 rows x 64 columns
constexpr int kKChunk = kBN * 128;      // 64 rows x 64 columns
constexpr int kPBytes = kBM * kBN * 2;
constexpr int kBiasRow = 96;            // entries of a warp's slice of the distance table
constexpr float kLog2e = 1.4426950408889634f;
constexpr uint32_t kMajorB = 1u << 16;  // instruction descriptor: B is MN-major

template <bool SIG, int NK, int DV>     // NK chunks of 64 key columns
struct Lay {
  static constexpr int kQ = NK * kQChunk;                            // one tile's queries
  static constexpr int kK = NK * kKChunk;                            // one map's keys
  static constexpr int kMaps = SIG ? 1 : 2;
  static constexpr int kV = DV / 64 * kKChunk;
  static constexpr int kStage = kMaps * kK + kV;
  static constexpr int kFixed = 2 * kQ + 2 * kPBytes + (SIG ? 8 * 2 * kBiasRow * 4 : 0) + 512 + 1024;
  static constexpr int kFit = (227 * 1024 - kFixed) / kStage;
  static constexpr int kStages = kFit < 4 ? kFit : 4;
  static constexpr int kOffKV = 2 * kQ;
  static constexpr int kOffP = kOffKV + kStages * kStage;
  static constexpr int kOffBias = kOffP + 2 * kPBytes;
  static constexpr int kOffBar = kOffBias + (SIG ? 8 * 2 * kBiasRow * 4 : 0);
  static constexpr int kSmem = kOffBar + 512 + 1024;
  static_assert(kStages >= 2 && kSmem <= 227 * 1024, "the prompt kernel must fit one SM");
  static_assert(SIG || DV * kBM * 4 <= kOffP, "the second map's rows must fit into the operands' space");
};

struct Params {
  __nv_bfloat16* out;
  const int32_t* cu;
  const int32_t* q_pos0;
  const int32_t* shift;
  const float* bias;
  int64_t bias_n;
  const __nv_bfloat16* gate;
  int64_t ld_gate;
  int H, group, window;
  float scale_log2;
  float lambda, out_scale, eps;
  int dv_real;
  int* error_flag;
};

// Descriptor of an MN-major operand in 128-byte-swizzled shared memory: rows (K) of 64 elements (MN), groups of eight rows 1024 bytes
// apart, the next 64 elements `mn_stride` bytes away.
__device__ __forceinline__ uint64_t smem_desc_mn(uint32_t smem_addr, uint32_t mn_stride) {
  uint64_t d = 0;
  d |= static_cast<uint64_t>((smem_addr & 0x3FFFF) >> 4);
  d |= static_cast<uint64_t>(mn_stride >> 4) << 16;
  d |= static_cast<uint64_t>(1024 >> 4) << 32;
  d |= static_cast<uint64_t>(1) << 46;
  d |= static_cast<uint64_t>(2) << 61;
  return d;
}

__device__ __forceinline__ float rcp(float x) {
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ void both_tiles_sync() { asm volatile("bar.sync 2, 256;" ::: "memory"); }

// One tile as its score warps see it: blocks [b0, b1) of the CTA's blocks.
struct Tile {
  uint64_t* s_full;
  uint64_t* s_free;
  uint64_t* p_full;
  uint64_t* pv_full;
  uint32_t tmem_s, tmem_pv;
  uint8_t* p_smem;
  int b0, b1;
  int first;               // position of the first key of block 0
  int pos;                 // position of the tile's first query row
};

// Loads S of a block and releases it.
__device__ __forceinline__ bool take_scores(const Tile& t, int n, uint32_t lane_off, uint32_t (&s0)[32], uint32_t (&s1)[32], volatile int* abort_flag) {
  if (!mbar_wait(t.s_full, n & 1, abort_flag, kWaitNs)) return false;
  tc_fence_after_sync();
  tmem_ld_32x32(t.tmem_s + lane_off, s0);
  tmem_ld_32x32(t.tmem_s + lane_off + 32, s1);
  tmem_ld_wait();
  tc_fence_before_sync();
  mbar_arrive(t.s_free);
  return true;
}

// Sigmoid weights of all blocks of a tile.
__device__ __forceinline__ bool sigmoid_tile(const Params& p, const Tile& t, int warp, int lane, const float* table, float* slice, volatile int* abort_flag) {
  const int qd = warp & 3, row = qd * 32 + lane, pos = t.pos + row, sw = row & 7;
  const uint32_t lane_off = static_cast<uint32_t>(qd * 32) << 16;
  const float neg_scale = -p.scale_log2;
  const int oldest = p.window > 0 ? pos - p.window + 1 : -1;        // first position this row sees
  uint8_t* prow = t.p_smem + row * 128;
  float next[3];
  auto request = [&](int j) {                                        // entries of block j: distances d0 + 0 .. 94
    const int d0 = t.pos + qd * 32 - (t.first + j * kBN) - 63;
#pragma unroll
    for (int i = 0; i < 3; ++i) {
      const int d = d0 + lane + 32 * i;
      next[i] = d >= 0 && d < p.bias_n ? __ldg(table + d) : 0.f;
    }
  };
  if (t.b0 < t.b1) request(t.b0);
  for (int j = t.b0; j < t.b1; ++j) {
    const int n = j - t.b0;
    float* bias = slice + (n & 1) * kBiasRow;
#pragma unroll
    for (int i = 0; i < 3; ++i) bias[lane + 32 * i] = next[i] * -kLog2e;
    __syncwarp();
    if (j + 1 < t.b1) request(j + 1);
    uint32_t s0[32], s1[32];
    if (!take_scores(t, n, lane_off, s0, s1, abort_flag)) return false;
    const int t0 = t.first + j * kBN;
    const bool full = __all_sync(0xffffffffu, t0 + kBN - 1 <= pos && t0 >= oldest);
    const float* mine = bias + lane + 63;                            // entry of key c: mine[-c]
    // exponents of 2 of the negated argument, then pairs of weights
#pragma unroll
    for (int c = 0; c < 32; ++c) {
      s0[c] = __float_as_uint(ex2(fminf(fmaf(__uint_as_float(s0[c]), neg_scale, mine[-c]), 60.f)));
      s1[c] = __float_as_uint(ex2(fminf(fmaf(__uint_as_float(s1[c]), neg_scale, mine[-32 - c]), 60.f)));
    }
    uint32_t pk[32];
#pragma unroll
    for (int c = 0; c < 64; c += 2) {
      const float a = 1.f + __uint_as_float(c < 32 ? s0[c & 31] : s1[c & 31]), b = 1.f + __uint_as_float(c < 32 ? s0[(c & 31) + 1] : s1[(c & 31) + 1]);
      const float r = rcp(a * b);
      float x = r * b, y = r * a;
      if (!full) {
        if (t0 + c > pos || t0 + c < oldest) x = 0.f;
        if (t0 + c + 1 > pos || t0 + c + 1 < oldest) y = 0.f;
      }
      pk[c / 2] = pack_bf16x2(x, y);
    }
    // the previous block's product must have finished: it read the buffer that is rewritten now
    if (n > 0 && !mbar_wait(t.pv_full, (n - 1) & 1, abort_flag, kWaitNs)) return false;
#pragma unroll
    for (int c = 0; c < 8; ++c) *reinterpret_cast<uint4*>(prow + ((c ^ sw) << 4)) = make_uint4(pk[4 * c], pk[4 * c + 1], pk[4 * c + 2], pk[4 * c + 3]);
    fence_proxy_async_smem();
    mbar_arrive(t.p_full);
  }
  return true;
}

// Softmax of all blocks of a tile; returns the row's sum in `l`.
template <int DV>
__device__ __forceinline__ bool softmax_map(const Params& p, const Tile& t, int warp, int lane, float& l, volatile int* abort_flag) {
  const int qd = warp & 3, row = qd * 32 + lane, pos = t.pos + row, sw = row & 7;
  const uint32_t lane_off = static_cast<uint32_t>(qd * 32) << 16;
  const int oldest = p.window > 0 ? pos - p.window + 1 : -1;
  uint8_t* prow = t.p_smem + row * 128;
  constexpr float kRescaleStep = 8.f;
  float m = -INFINITY;
  l = 0.f;
  for (int j = t.b0; j < t.b1; ++j) {
    const int n = j - t.b0;
    uint32_t s0[32], s1[32];
    if (!take_scores(t, n, lane_off, s0, s1, abort_flag)) return false;
    const int t0 = t.first + j * kBN;
    if (!__all_sync(0xffffffffu, t0 + kBN - 1 <= pos && t0 >= oldest)) {
#pragma unroll
      for (int c = 0; c < 32; ++c) {
        if (t0 + c > pos || t0 + c < oldest) s0[c] = 0xff800000u;               // -inf
        if (t0 + 32 + c > pos || t0 + 32 + c < oldest) s1[c] = 0xff800000u;
      }
    }
    float mx = -INFINITY;
#pragma unroll
    for (int c = 0; c < 32; ++c) mx = fmaxf(mx, fmaxf(__uint_as_float(s0[c]), __uint_as_float(s1[c])));
    mx *= p.scale_log2;                                              // scale > 0
    float alpha = 1.f;
    bool raise = false;
    if (mx > m) {
      if (m == -INFINITY) {
        m = mx;                                                      // nothing accumulated so far
      } else if (mx - m > kRescaleStep) {
        alpha = ex2(m - mx);
        m = mx;
        raise = true;
      }
    }
    const float m_use = m == -INFINITY ? 0.f : m;
    if (n > 0 && !mbar_wait(t.pv_full, (n - 1) & 1, abort_flag, kWaitNs)) return false;
    if (__any_sync(0xffffffffu, raise)) {
      tc_fence_after_sync();
#pragma unroll
      for (int c = 0; c < DV / 32; ++c) {
        uint32_t r[32];
        tmem_ld_32x32(t.tmem_pv + lane_off + c * 32, r);
        tmem_ld_wait();
#pragma unroll
        for (int i = 0; i < 32; ++i) r[i] = __float_as_uint(__uint_as_float(r[i]) * alpha);
        tmem_st_32x32(t.tmem_pv + lane_off + c * 32, r);
      }
      tmem_st_wait();
      tc_fence_before_sync();
    }
    float sum = 0.f;
#pragma unroll
    for (int c8 = 0; c8 < 8; ++c8) {
      uint32_t pk[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int c = c8 * 8 + 2 * e;
        const float x0 = ex2(fmaf(__uint_as_float(c < 32 ? s0[c & 31] : s1[c & 31]), p.scale_log2, -m_use));
        const float x1 = ex2(fmaf(__uint_as_float(c < 32 ? s0[(c + 1) & 31] : s1[(c + 1) & 31]), p.scale_log2, -m_use));
        sum += x0 + x1;
        pk[e] = pack_bf16x2(x0, x1);
      }
      *reinterpret_cast<uint4*>(prow + ((c8 ^ sw) << 4)) = make_uint4(pk[0], pk[1], pk[2], pk[3]);
    }
    l = l * alpha + sum;
    fence_proxy_async_smem();
    mbar_arrive(t.p_full);
  }
  return true;
}

// The row's accumulator, 32 columns from c * 32 on.
__device__ __forceinline__ void take_out(const Tile& t, uint32_t lane_off, int c, float (&o)[32]) {
  uint32_t r[32];
  tmem_ld_32x32(t.tmem_pv + lane_off + c * 32, r);
  tmem_ld_wait();
#pragma unroll
  for (int i = 0; i < 32; ++i) o[i] = __uint_as_float(r[i]);
}
__device__ __forceinline__ void put_out(__nv_bfloat16* row, const float (&o)[32], float f) {
#pragma unroll
  for (int i = 0; i < 32; i += 8) {
    uint4 v;
    v.x = pack_bf16x2(o[i] * f, o[i + 1] * f);
    v.y = pack_bf16x2(o[i + 2] * f, o[i + 3] * f);
    v.z = pack_bf16x2(o[i + 4] * f, o[i + 5] * f);
    v.w = pack_bf16x2(o[i + 6] * f, o[i + 7] * f);
    *reinterpret_cast<uint4*>(row + i) = v;
  }
}

template <bool SIG, int NK, int DV>
__global__ void __launch_bounds__(kThreads, 1)
window_prompt_kernel(const __grid_constant__ CUtensorMap tq, const __grid_constant__ CUtensorMap tk, const __grid_constant__ CUtensorMap tv,
                     const Params p) {
  extern __shared__ __align__(1024) uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  using L = Lay<SIG, NK, DV>;
  constexpr int kStages = L::kStages, kMaps = L::kMaps, kRows = SIG ? 2 * kBM : kBM;
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + L::kOffBar);
  uint64_t* q_full = bars;
  uint64_t* s_full = bars + 1;        // [2] per tile
  uint64_t* s_free = bars + 3;
  uint64_t* p_full = bars + 5;
  uint64_t* pv_full = bars + 7;
  uint64_t* kv_full = bars + 9;       // [kStages]
  uint64_t* kv_empty = kv_full + kStages;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(kv_empty + kStages);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);

  const int b = blockIdx.z, head = blockIdx.y, hkv = head / p.group;
  const int q_begin = p.cu[b], q_len = p.cu[b + 1] - q_begin;
  const int row0 = static_cast<int>(gridDim.x - 1 - blockIdx.x) * kRows;       // without a window the last tiles are the long ones
  if (row0 >= q_len) return;                      // whole CTA, before any barrier or TMEM use
  const int pos0 = p.q_pos0[b] + row0, shift = p.shift[b];
  const int first = p.window > 0 ? max(0, pos0 - p.window + 1) : 0;            // position of the first key of block 0
  int rows_t[2], b0_t[2], b1_t[2];
#pragma unroll
  for (int t = 0; t < 2; ++t) {
    const int at = SIG ? t * kBM : 0;             // first row of the tile
    rows_t[t] = max(0, min(q_len - row0 - at, kBM));
    const int lo = p.window > 0 ? max(0, pos0 + at - p.window + 1) : 0;
    b0_t[t] = rows_t[t] > 0 ? (lo - first) / kBN : 0;
    b1_t[t] = rows_t[t] > 0 ? (pos0 + at + rows_t[t] - first + kBN - 1) / kBN : 0;
  }
  const int nblk = max(b1_t[0], b1_t[1]);
  const int warp = __shfl_sync(0xffffffffu, threadIdx.x >> 5, 0), lane = threadIdx.x & 31;      // warp-uniform

  if (threadIdx.x == 0) {
    mbar_init(q_full, 1);
    for (int i = 0; i < kStages; ++i) {
      mbar_init(&kv_full[i], 1);
      mbar_init(&kv_empty[i], 1);
    }
    for (int t = 0; t < 2; ++t) {
      mbar_init(&s_full[t], 1);
      mbar_init(&s_free[t], 128);
      mbar_init(&p_full[t], 128);
      mbar_init(&pv_full[t], 1);
    }
    *abort_flag = 0;
    fence_mbar_init();
  }
  if (warp == 1) {
    tmem_alloc(tmem_slot, 512);
    tmem_relinquish();
  }
  tc_fence_before_sync();
  __syncthreads();
  tc_fence_after_sync();
  const uint32_t tmem_base = *tmem_slot;          // tile t: S at columns [256 t, 256 t + 64), O at [256 t + 64, 256 t + 64 + DV)
  pdl_wait();                                     // everything above overlaps the previous kernel's tail
  pdl_launch_dependents();

  if (warp == 0) {
    if (lane == 0) {
      // rows beyond the sequence read the next one's or zeros; they are never written out
      mbar_arrive_expect_tx(q_full, 2 * L::kQ);
#pragma unroll
      for (int t = 0; t < 2; ++t)
#pragma unroll
        for (int c = 0; c < NK; ++c)
          tma_load_2d(smem + t * L::kQ + c * kQChunk, &tq, q_full, (SIG ? head : head * 2 + t) * NK * 64 + c * 64, q_begin + row0 + (SIG ? t * kBM : 0));
      int loaded = 0;
      bool ok = true;
      for (int j = 0; j < nblk; ++j) {
        const int s = j % kStages;
        ok = mbar_wait(&kv_empty[s], ((j / kStages) & 1) ^ 1, abort_flag, kWaitNs);
        if (!ok) break;
        mbar_arrive_expect_tx(&kv_full[s], L::kStage);
        uint8_t* st = smem + L::kOffKV + s * L::kStage;
        const int row = shift + first + j * kBN;
#pragma unroll
        for (int c = 0; c < kMaps * NK; ++c) tma_load_2d(st + c * kKChunk, &tk, &kv_full[s], (hkv * kMaps * NK + c) * 64, row);
#pragma unroll
        for (int c = 0; c < DV / 64; ++c) tma_load_2d(st + kMaps * L::kK + c * kKChunk, &tv, &kv_full[s], hkv * DV + c * 64, row);
        ++loaded;
      }
      if (!ok) {                       // own copies land before the CTA's shared memory goes away
        *abort_flag = 1;
        mbar_wait(q_full, 0, nullptr, kWaitNs);
        for (int j = max(0, loaded - kStages); j < loaded; ++j) mbar_wait(&kv_full[j % kStages], (j / kStages) & 1, nullptr, kWaitNs);
      }
    }
  } else if (warp == 1) {
    constexpr uint32_t idesc_s = make_idesc(1u, kBM, kBN);
    constexpr uint32_t idesc_pv = make_idesc(1u, kBM, DV) | kMajorB;
    bool ok = mbar_wait(q_full, 0, abort_flag, kWaitNs);
    auto issue_s = [&](int t, int j) -> bool {
      const int s = j % kStages, n = j - b0_t[t];
      if (!mbar_wait(&kv_full[s], (j / kStages) & 1, abort_flag, kWaitNs)) return false;
      if (n > 0 && !mbar_wait(&s_free[t], (n - 1) & 1, abort_flag, kWaitNs)) return false;
      tc_fence_after_sync();
      const uint32_t sq = smem_u32(smem + t * L::kQ);
      const uint32_t sk = smem_u32(smem + L::kOffKV + s * L::kStage + (SIG ? 0 : t * L::kK));
#pragma unroll
      for (int c = 0; c < NK; ++c)
#pragma unroll
        for (int k = 0; k < 4; ++k)
          umma_f16_elect(tmem_base + t * 256, make_smem_desc_sw128(sq + c * kQChunk) + 2 * k, make_smem_desc_sw128(sk + c * kKChunk) + 2 * k, idesc_s,
                         c > 0 || k > 0 ? 1u : 0u);
      umma_commit_elect(&s_full[t]);
      return true;
    };
    auto issue_pv = [&](int t, int j) -> bool {
      const int n = j - b0_t[t];
      if (!mbar_wait(&p_full[t], n & 1, abort_flag, kWaitNs)) return false;
      tc_fence_after_sync();
      const uint32_t sp = smem_u32(smem + L::kOffP + t * kPBytes);
      const uint32_t sv = smem_u32(smem + L::kOffKV + (j % kStages) * L::kStage + kMaps * L::kK);
#pragma unroll
      for (int k = 0; k < kBN / kUmmaK; ++k)                          // 16 tokens: 16 rows of 128 bytes
        umma_f16_elect(tmem_base + t * 256 + 64, make_smem_desc_sw128(sp) + 2 * k, smem_desc_mn(sv, kKChunk) + k * (2048 >> 4), idesc_pv,
                       n > 0 || k > 0 ? 1u : 0u);
      umma_commit_elect(&pv_full[t]);
      return true;
    };
    auto in = [&](int t, int j) { return j >= b0_t[t] && j < b1_t[t]; };
    for (int t = 0; t < 2 && ok; ++t)
      if (in(t, 0)) ok = issue_s(t, 0);
    for (int j = 0; j < nblk && ok; ++j) {
      // per tile: S of the next block as soon as this block's S has been read, then this block's P V
      for (int t = 0; t < 2 && ok; ++t) {
        if (in(t, j + 1)) ok = issue_s(t, j + 1);
        if (ok && in(t, j)) ok = issue_pv(t, j);
      }
      if (ok) umma_commit_elect(&kv_empty[j % kStages]);   // every product that reads this stage has been issued before
    }
    if (!ok) *abort_flag = 1;
  } else {
    const int t = (warp - 2) >> 2;                 // warps 2-5: tile 0, warps 6-9: tile 1
    Tile c;
    c.s_full = &s_full[t]; c.s_free = &s_free[t]; c.p_full = &p_full[t]; c.pv_full = &pv_full[t];
    c.tmem_s = tmem_base + t * 256; c.tmem_pv = tmem_base + t * 256 + 64;
    c.p_smem = smem + L::kOffP + t * kPBytes;
    c.b0 = b0_t[t]; c.b1 = b1_t[t];
    c.first = first;
    c.pos = pos0 + (SIG ? t * kBM : 0);
    const int qd = warp & 3, row = qd * 32 + lane;
    const uint32_t lane_off = static_cast<uint32_t>(qd * 32) << 16;
    const bool row_ok = row < rows_t[t];
    const int64_t tok = static_cast<int64_t>(q_begin) + row0 + (SIG ? t * kBM : 0) + row;
    float l = 0.f;
    bool ok;
    if constexpr (SIG) {
      float* slice = reinterpret_cast<float*>(smem + L::kOffBias) + (warp - 2) * 2 * kBiasRow;
      ok = sigmoid_tile(p, c, warp, lane, p.bias + head * p.bias_n, slice, abort_flag);
    } else {
      ok = softmax_map<DV>(p, c, warp, lane, l, abort_flag);
    }
    const int n = c.b1 - c.b0;
    if (ok && n > 0) ok = mbar_wait(c.pv_full, (n - 1) & 1, abort_flag, kWaitNs);
    if (!ok) *abort_flag = 1;
    tc_fence_after_sync();
    float f = 1.f;
    if (row_ok && p.gate != nullptr) f = 1.f / (1.f + __expf(-__bfloat162float(p.gate[tok * p.ld_gate + head])));
    __nv_bfloat16* orow = p.out + (tok * p.H + head) * DV;
    if constexpr (SIG) {
      if (n > 0)                                   // uniform in the tile
#pragma unroll
        for (int k = 0; k < DV / 32; ++k) {
          float o[32];
          take_out(c, lane_off, k, o);
          if (ok && row_ok) put_out(orow + 32 * k, o, f);
        }
    } else {
      // both maps' products are done when both tiles are here: the operands' space takes the second map's rows, column by column
      float* other = reinterpret_cast<float*>(smem) + row;
      const float inv = l > 0.f ? 1.f / l : 0.f;
      both_tiles_sync();
      if (t == 1) {
#pragma unroll
        for (int k = 0; k < DV / 32; ++k) {
          float o[32];
          take_out(c, lane_off, k, o);
#pragma unroll
          for (int i = 0; i < 32; ++i) other[(32 * k + i) * kBM] = o[i] * (inv * p.lambda);
        }
      }
      both_tiles_sync();
      if (t == 0) {
        float ss = 0.f;
#pragma unroll
        for (int k = 0; k < DV / 32; ++k) {
          float o[32];
          take_out(c, lane_off, k, o);
#pragma unroll
          for (int i = 0; i < 32; ++i) {
            const float d = fmaf(o[i], inv, -other[(32 * k + i) * kBM]);
            other[(32 * k + i) * kBM] = d;
            ss = fmaf(d, d, ss);
          }
        }
        f *= p.out_scale / sqrtf(ss / p.dv_real + p.eps);
        if (*abort_flag == 0 && row_ok)
#pragma unroll
          for (int k = 0; k < DV / 32; ++k) {
            float o[32];
#pragma unroll
            for (int i = 0; i < 32; ++i) o[i] = other[(32 * k + i) * kBM];
            put_out(orow + 32 * k, o, f);
          }
      }
    }
    tc_fence_before_sync();
  }

  tc_fence_before_sync();
  __syncthreads();
  if (threadIdx.x == 0 && *abort_flag != 0 && p.error_flag != nullptr) *p.error_flag = 1;
  if (warp == 1) {
    tc_fence_after_sync();
    tmem_dealloc(tmem_base, 512);
  }
}

bool encode(CUtensorMap* m, const void* base, int64_t rows, int64_t cols, int box_rows) {
  TensorMap t;
  if (encode_tensor_map_2d(&t, base, kBF16, static_cast<uint64_t>(rows), static_cast<uint64_t>(cols), static_cast<uint64_t>(cols) * 2, box_rows, 64, 128) != 0)
    return false;
  std::memcpy(m, t.bytes, sizeof(*m));
  return true;
}

template <bool SIG, int NK, int DV>
cudaError_t launch(const WindowAttnArgs& a, const Params& p, cudaStream_t s) {
  CUtensorMap mq, mk, mv;
  if (!encode(&mq, a.q, a.T, static_cast<int64_t>(a.H) * a.maps * a.dk, kBM) || !encode(&mk, a.k, a.rows, static_cast<int64_t>(a.G) * a.maps * a.dk, kBN) ||
      !encode(&mv, a.v, a.rows, static_cast<int64_t>(a.G) * a.dv, kBN))
    return cudaErrorInvalidValue;
  static SmemOptIn opt;
  constexpr int smem = Lay<SIG, NK, DV>::kSmem, rows = SIG ? 2 * kBM : kBM;
  cudaError_t e = opt.ensure(window_prompt_kernel<SIG, NK, DV>, smem);
  if (e != cudaSuccess) return e;
  return launch_pdl(window_prompt_kernel<SIG, NK, DV>, dim3((a.max_q + rows - 1) / rows, a.H, a.N), dim3(kThreads), smem, s, mq, mk, mv, p);
}

}  // namespace

cudaError_t launch_window_prompt(const WindowAttnArgs& a, cudaStream_t s) {
  const bool sig = a.bias != nullptr;
  if (a.is_f32 || a.H < 1 || a.G < 1 || a.H % a.G != 0 || a.maps != (sig ? 1 : 2) || !(a.scale > 0.f) || a.cu == nullptr || a.q_pos0 == nullptr ||
      a.shift == nullptr || a.H > 65535 || a.N > 65535 || (!sig && a.dv_real < 1) || (a.dk != 64 && a.dk != 128) || (a.dv != 64 && a.dv != 128))
    return cudaErrorInvalidValue;
  if (a.T == 0 || a.N == 0 || a.max_q == 0) return cudaSuccess;
  Params p;
  p.out = reinterpret_cast<__nv_bfloat16*>(a.out);
  p.cu = a.cu; p.q_pos0 = a.q_pos0; p.shift = a.shift;
  p.bias = a.bias; p.bias_n = a.bias_n;
  p.gate = reinterpret_cast<const __nv_bfloat16*>(a.gate); p.ld_gate = a.ld_gate;
  p.H = a.H; p.group = a.H / a.G; p.window = a.window;
  p.scale_log2 = a.scale * kLog2e;
  p.lambda = a.lambda; p.out_scale = a.out_scale; p.eps = a.eps; p.dv_real = a.dv_real;
  p.error_flag = a.error_flag;
  const int form = (a.dk == 128 ? 2 : 0) + (a.dv == 128 ? 1 : 0);
  if (sig)
    return form == 0 ? launch<true, 1, 64>(a, p, s) : form == 1 ? launch<true, 1, 128>(a, p, s) : form == 2 ? launch<true, 2, 64>(a, p, s) : launch<true, 2, 128>(a, p, s);
  return form == 0 ? launch<false, 1, 64>(a, p, s) : form == 1 ? launch<false, 1, 128>(a, p, s) : form == 2 ? launch<false, 2, 64>(a, p, s) : launch<false, 2, 128>(a, p, s);
}

}  // namespace tdb
