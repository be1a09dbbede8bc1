// Latent attention on the 5th-generation tensor cores (bf16).
//
// latent_prefill_kernel   prompts, expanded form.  One CTA = 256 query rows of one head as two 128-row tiles that share every
//                         block of 64 keys, as in the two-tile form of attn_sm100.cu (same softmax warps).  A key is
//                         [unrotated | rotated] from two tensors: the head's keys and the rotated part in the packed rows, which
//                         all heads share; queries likewise.  Values arrive transposed from their GEMM.  Keys and values have
//                         rings of their own: scores run a block ahead, so a key buffer is free a block earlier than the values
//                         beside it.  Head sizes that are no multiple of 64 are zero-filled by the TMA boxes.
// latent_decode_kernel    decoding, absorbed form: split-KV, one CTA per (split, 32 heads, sequence).  The cached rows are both
//                         keys and values, so a tile of 64 tokens is loaded once and multiplied twice:
//                           S^T[token, head]  = row . q'            M = 64 tokens, N = 32 heads, K = rank + rotated
//                           O^T[latent, head] += row^T . P^T        M = 128 latents, N = 32 heads, K = 64 tokens
//                         (the second product takes the same shared-memory tile as an MN-major A operand).  Few heads cost few
//                         columns, not idle rows.  The ring holds more than two tiles, so S^T of the next tile runs during the
//                         exponentials and loads never stop.  A softmax thread holds 2 tokens x 8 heads; maxima over tokens are
//                         butterfly-transposed, after which lane h of every warp keeps head h's reference maximum.  Partials
//                         are merged by latent_out_kernel.
//
// Every wait is bounded; a timeout is recorded, the CTA runs through without further waiting, frees its TMEM and returns.
#include <cuda.h>
#include <cuda_bf16.h>

#include <cstring>

#include "tdb/api.h"
#include "tdb/attn_sm100.cuh"
#include "tdb/latent.h"
#include "tdb/launch.cuh"
#include "tdb/ptx.cuh"

namespace tdb {

namespace {

constexpr int kUmmaK = 16;

// Descriptor of an MN-major operand in 128-byte-swizzled shared memory: rows (K) of 64 elements (MN), groups of eight rows
// 1024 bytes apart, the next 64 elements `mn_stride` bytes away.
__device__ __forceinline__ uint64_t make_smem_desc_sw128_mn(uint32_t smem_addr, uint32_t mn_stride) {
  uint64_t d = 0;
  d |= static_cast<uint64_t>((smem_addr & 0x3FFFF) >> 4);
  d |= static_cast<uint64_t>(mn_stride >> 4) << 16;
  d |= static_cast<uint64_t>(1024 >> 4) << 32;
  d |= static_cast<uint64_t>(1) << 46;
  d |= static_cast<uint64_t>(2) << 61;
  return d;
}
constexpr uint32_t kMajorA = 1u << 15;     // instruction descriptor: A is MN-major

// ------------------------------------------------------------------------------------------------------------------
// Prompts
// ------------------------------------------------------------------------------------------------------------------
struct PrefillParams {
  FwdParams f;
  const int32_t* ctx0;
  int d, r;
};
constexpr int kPfThreads = 320;       // warp 0 TMA, warp 1 MMA, warps 2-5 softmax of tile 0, warps 6-9 of tile 1
constexpr int kQChunk = kBM * 128;    // 128 rows x 64 columns
constexpr int kKChunk = kBN * 128;
template <int NC, int DV>             // NC chunks of 64 key columns, the last one the rotated part
struct PfLay {
  static constexpr int kStages = NC == 3 ? 2 : 3;
  static constexpr int kQ = NC * kQChunk, kK = NC * kKChunk, kV = DV * 128, kP = kBM * kBN * 2;
  static constexpr int kOffK = 2 * kQ;
  static constexpr int kOffV = kOffK + kStages * kK;
  static constexpr int kOffP = kOffV + kStages * kV;
  static constexpr int kOffBar = kOffP + 2 * kP;
  static constexpr int kSmem = kOffBar + (4 * kStages + 10) * 8 + 64 + 1024;
};
static_assert(PfLay<3, 128>::kSmem <= 227 * 1024 && PfLay<2, 128>::kSmem <= 227 * 1024, "prompt kernel must fit one SM");

template <int NC, int DV>
__global__ void __launch_bounds__(kPfThreads, 1)
latent_prefill_kernel(const __grid_constant__ CUtensorMap tq, const __grid_constant__ CUtensorMap tqr,
                      const __grid_constant__ CUtensorMap tk, const __grid_constant__ CUtensorMap tkr,
                      const __grid_constant__ CUtensorMap tv, const PrefillParams pp) {
  extern __shared__ __align__(1024) uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  using L = PfLay<NC, DV>;
  constexpr int kStages = L::kStages;
  const FwdParams& p = pp.f;
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + L::kOffBar);
  uint64_t* q_full = bars;
  uint64_t* s_full = bars + 1;        // [2] per tile
  uint64_t* s_free = bars + 3;
  uint64_t* p_full = bars + 5;
  uint64_t* pv_full = bars + 7;
  uint64_t* k_full = bars + 9;                  // [kStages] each
  uint64_t* k_empty = k_full + kStages;
  uint64_t* v_full = k_empty + kStages;
  uint64_t* v_empty = v_full + kStages;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(v_empty + kStages);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);

  const int b = blockIdx.z, head = blockIdx.x;
  const int q_begin = p.cu_seqlens_q[b], q_len = p.cu_seqlens_q[b + 1] - q_begin;
  // the long causal tiles of all heads first (blocks are handed out in order of blockIdx.x, then y): no long tile in the last wave
  const int row0 = static_cast<int>(gridDim.y - 1 - blockIdx.y) * (2 * kBM);
  if (row0 >= q_len) return;                      // whole CTA, before any barrier or TMEM use
  const int kv_len = p.kv_lens[b], pos0 = p.q_pos0[b], base = pp.ctx0[b];
  int rows_t[2], nblk_t[2];
#pragma unroll
  for (int t = 0; t < 2; ++t) {
    rows_t[t] = max(0, min(q_len - (row0 + t * kBM), kBM));
    const int kv_end = max(0, min(kv_len, pos0 + row0 + t * kBM + rows_t[t]));
    nblk_t[t] = rows_t[t] > 0 ? (kv_end + kBN - 1) / kBN : 0;
  }
  const int nblk = max(nblk_t[0], nblk_t[1]);
  const int warp = __shfl_sync(0xffffffffu, threadIdx.x >> 5, 0), lane = threadIdx.x & 31;      // warp-uniform

  if (threadIdx.x == 0) {
    mbar_init(q_full, 1);
    for (int i = 0; i < kStages; ++i) {
      mbar_init(&k_full[i], 1);
      mbar_init(&k_empty[i], 1);
      mbar_init(&v_full[i], 1);
      mbar_init(&v_empty[i], 1);
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

  if (warp == 0) {
    if (lane == 0) {
      // rows beyond the sequence read the next one's or zeros; they are never written out
      mbar_arrive_expect_tx(q_full, 2 * L::kQ);
#pragma unroll
      for (int t = 0; t < 2; ++t) {
        uint8_t* sq = smem + t * L::kQ;
#pragma unroll
        for (int c = 0; c < NC - 1; ++c) tma_load_3d(sq + c * kQChunk, &tq, q_full, c * 64, q_begin + row0 + t * kBM, head);
        tma_load_3d(sq + (NC - 1) * kQChunk, &tqr, q_full, 0, q_begin + row0 + t * kBM, head);
      }
      auto load_k = [&](int j) -> bool {
        const int s = j % kStages;
        if (!mbar_wait(&k_empty[s], ((j / kStages) & 1) ^ 1, abort_flag, kWaitNs)) return false;
        mbar_arrive_expect_tx(&k_full[s], L::kK);
        uint8_t* sk = smem + L::kOffK + s * L::kK;
#pragma unroll
        for (int c = 0; c < NC - 1; ++c) tma_load_3d(sk + c * kKChunk, &tk, &k_full[s], c * 64, base + j * kBN, head);
        tma_load_2d(sk + (NC - 1) * kKChunk, &tkr, &k_full[s], 0, base + j * kBN);
        return true;
      };
      int nk = 0, nv = 0;              // blocks requested so far
      bool ok = nblk == 0 || load_k(nk++);
      for (int j = 0; j < nblk && ok; ++j) {
        if (j + 1 < nblk) {            // keys a block ahead of the values
          ok = load_k(j + 1);
          if (!ok) break;
          ++nk;
        }
        const int s = j % kStages;
        ok = mbar_wait(&v_empty[s], ((j / kStages) & 1) ^ 1, abort_flag, kWaitNs);
        if (!ok) break;
        mbar_arrive_expect_tx(&v_full[s], L::kV);
        tma_load_3d(smem + L::kOffV + s * L::kV, &tv, &v_full[s], base + j * kBN, 0, head);
        ++nv;
      }
      if (!ok) {                       // own copies land before the CTA's shared memory goes away
        *abort_flag = 1;
        mbar_wait(q_full, 0, nullptr, kWaitNs);
        for (int j = max(0, nk - kStages); j < nk; ++j) mbar_wait(&k_full[j % kStages], (j / kStages) & 1, nullptr, kWaitNs);
        for (int j = max(0, nv - kStages); j < nv; ++j) mbar_wait(&v_full[j % kStages], (j / kStages) & 1, nullptr, kWaitNs);
      }
    }
  } else if (warp == 1) {
    constexpr uint32_t idesc_s = make_idesc(1u, kBM, kBN);
    constexpr uint32_t idesc_pv = make_idesc(1u, kBM, DV);
    bool ok = mbar_wait(q_full, 0, abort_flag, kWaitNs);
    // the last tile that block j is multiplied with: the second one sees at least the blocks of the first, unless it is empty
    auto last_tile = [&](int j) { return j < nblk_t[1] ? 1 : 0; };
    auto issue_s = [&](int t, int j) -> bool {
      const int s = j % kStages;
      if (!mbar_wait(&k_full[s], (j / kStages) & 1, abort_flag, kWaitNs)) return false;
      if (j > 0 && !mbar_wait(&s_free[t], (j - 1) & 1, abort_flag, kWaitNs)) return false;
      tc_fence_after_sync();
      const uint32_t sq = smem_u32(smem + t * L::kQ);
      const uint32_t sk = smem_u32(smem + L::kOffK + s * L::kK);
      uint32_t acc = 0;
#pragma unroll
      for (int c = 0; c < NC; ++c) {
        const int cols = c < NC - 1 ? pp.d - c * 64 : pp.r;
#pragma unroll
        for (int k = 0; k < 4; ++k) {
          if (k * kUmmaK >= cols) break;
          umma_f16_elect(tmem_base + t * 256, make_smem_desc_sw128(sq + c * kQChunk) + 2 * k, make_smem_desc_sw128(sk + c * kKChunk) + 2 * k,
                   idesc_s, acc);
          acc = 1;
        }
      }
      umma_commit_elect(&s_full[t]);
      if (t == last_tile(j)) umma_commit_elect(&k_empty[s]);      // both tiles' scores against this block have been issued
      return true;
    };
    auto issue_pv = [&](int t, int j) -> bool {
      if (!mbar_wait(&v_full[j % kStages], (j / kStages) & 1, abort_flag, kWaitNs)) return false;
      if (!mbar_wait(&p_full[t], j & 1, abort_flag, kWaitNs)) return false;
      tc_fence_after_sync();
      const uint32_t sp = smem_u32(smem + L::kOffP + t * L::kP);
      const uint32_t sv = smem_u32(smem + L::kOffV + (j % kStages) * L::kV);
#pragma unroll
      for (int k = 0; k < kBN / kUmmaK; ++k)
        umma_f16_elect(tmem_base + t * 256 + 64, make_smem_desc_sw128(sp) + 2 * k, make_smem_desc_sw128(sv) + 2 * k, idesc_pv,
                 (j > 0 || k > 0) ? 1u : 0u);
      umma_commit_elect(&pv_full[t]);
      if (t == last_tile(j)) umma_commit_elect(&v_empty[j % kStages]);
      return true;
    };
    for (int t = 0; t < 2 && ok; ++t)
      if (nblk_t[t] > 0) ok = issue_s(t, 0);
    for (int j = 0; j < nblk && ok; ++j) {
      // per tile: S of the next block as soon as this block's S has been read, then this block's P V
      for (int t = 0; t < 2 && ok; ++t) {
        if (j + 1 < nblk_t[t]) ok = issue_s(t, j + 1);
        if (ok && j < nblk_t[t]) ok = issue_pv(t, j);
      }
    }
    if (!ok) *abort_flag = 1;
  } else {
    const int t = (warp - 2) >> 2;
    TileCtx c;
    c.s_full = &s_full[t]; c.s_free = &s_free[t]; c.p_full = &p_full[t]; c.pv_full = &pv_full[t];
    c.tmem_s = tmem_base + t * 256; c.tmem_pv = tmem_base + t * 256 + 64;
    c.p_smem = smem + L::kOffP + t * L::kP;
    c.row0 = row0 + t * kBM; c.rows_here = rows_t[t]; c.nblk = nblk_t[t];
    softmax_tile<DV>(p, c, warp, lane, q_begin, head, kv_len, pos0, abort_flag);
  }

  tc_fence_before_sync();
  __syncthreads();
  if (threadIdx.x == 0 && *abort_flag != 0 && p.error_flag != nullptr) *p.error_flag = 1;
  if (warp == 1) {
    tc_fence_after_sync();
    tmem_dealloc(tmem_base, 512);
  }
}

template <int NC, int DV>
cudaError_t launch_prefill_t(const CUtensorMap (&m)[5], const PrefillParams& pp, dim3 grid, cudaStream_t s) {
  static SmemOptIn opt;
  cudaError_t e = opt.ensure(latent_prefill_kernel<NC, DV>, PfLay<NC, DV>::kSmem);
  if (e != cudaSuccess) return e;
  latent_prefill_kernel<NC, DV><<<grid, kPfThreads, PfLay<NC, DV>::kSmem, s>>>(m[0], m[1], m[2], m[3], m[4], pp);
  return cudaGetLastError();
}

bool encode3(CUtensorMap* m, const void* base, uint64_t d2, uint64_t rows, uint64_t cols, uint64_t row_elems, uint64_t d2_elems,
             uint32_t box_rows, uint32_t box_cols) {
  TensorMap t;
  if (encode_tensor_map_3d(&t, base, kBF16, d2, rows, cols, row_elems * 2, d2_elems * 2, box_rows, box_cols, 128) != 0) return false;
  std::memcpy(m, t.bytes, sizeof(*m));
  return true;
}
bool encode2(CUtensorMap* m, const void* base, uint64_t rows, uint64_t cols, uint64_t row_elems, uint32_t box_rows, uint32_t box_cols) {
  TensorMap t;
  if (encode_tensor_map_2d(&t, base, kBF16, rows, cols, row_elems * 2, box_rows, box_cols, 128) != 0) return false;
  std::memcpy(m, t.bytes, sizeof(*m));
  return true;
}

// ------------------------------------------------------------------------------------------------------------------
// Decoding
// ------------------------------------------------------------------------------------------------------------------
constexpr int kNH = 32;                       // heads of a CTA
constexpr int kTile = 64;                     // tokens of a tile
constexpr int kChunk = kTile * 128;           // 64 tokens x 64 columns: 8 KB
constexpr int kPair = 2 * kChunk;             // 128 latent columns: the M of one O^T block
constexpr int kSlots = 10;                    // ring of pairs; rank 512 takes four per tile
constexpr int kDecThreads = 192;              // warp 0 TMA, warp 1 MMA, warps 2-5 softmax
constexpr int kOffRot = kSlots * kPair;       // two rotated parts
constexpr int kOffQ = kOffRot + 2 * kChunk;   // [up to 9 chunks][32 heads x 128 bytes]
constexpr int kQChunkD = kNH * 128;
constexpr int kOffP = kOffQ + 9 * kQChunkD;   // P^T: [32 heads][64 tokens]
constexpr int kOffRed = kOffP + kQChunkD;     // fp32 [4][4 warps][32]: tile maxima (even / odd tiles), reference maxima, rescale factors
constexpr int kOffBar = kOffRed + 4 * 4 * 32 * 4;
constexpr int kDecSmem = kOffBar + (2 * kSlots + 10) * 8 + 64 + 1024;
static_assert(kDecSmem <= 227 * 1024, "decode kernel must fit one SM");
constexpr int kTmemO = 2 * kNH;               // S^T of even / odd tiles: columns [0, 32) / [32, 64); O^T block p: [64 + 32 p, 96 + 32 p)
constexpr int kTmemCols = 256;

struct DecodeParams {
  const int32_t* slots;
  const int32_t* kv_lens;
  float* o;
  float2* ml;
  int B, H, R, r, splits, num_slots, max_len;
  float scale_log2;
  int* error_flag;
};

__device__ __forceinline__ void softmax_warps_sync() { asm volatile("bar.sync 1, 128;" ::: "memory"); }

// v[k] of the lanes with the same lane % 4 -> the reduction over those lanes of element k = lane / 4, in that lane.
template <typename Op>
__device__ __forceinline__ float reduce_transposed(float (&v)[8], int lane, Op op) {
#pragma unroll
  for (int o = 4; o > 0; o >>= 1) {
    const bool up = ((lane >> 2) & o) != 0;
#pragma unroll
    for (int i = 0; i < o; ++i) {
      const float keep = up ? v[i + o] : v[i], send = up ? v[i] : v[i + o];
      v[i] = op(keep, __shfl_xor_sync(0xffffffffu, send, 4 * o));
    }
  }
  return v[0];
}

// grid (splits, ceil(H / 32), B)
__global__ void __launch_bounds__(kDecThreads, 1)
latent_decode_kernel(const __grid_constant__ CUtensorMap tq, const __grid_constant__ CUtensorMap tqr,
                     const __grid_constant__ CUtensorMap tc, const __grid_constant__ CUtensorMap tr, const DecodeParams p) {
  extern __shared__ __align__(1024) uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + kOffBar);
  uint64_t* q_full = bars;
  uint64_t* p_full = bars + 1;
  uint64_t* pv_full = bars + 2;
  uint64_t* rot_full = bars + 3;                // [2] each, even / odd tiles
  uint64_t* rot_empty = bars + 5;
  uint64_t* s_full = bars + 7;
  uint64_t* pair_full = bars + 9;               // [kSlots]
  uint64_t* pair_empty = pair_full + kSlots;    // [kSlots]
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(pair_empty + kSlots);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  const int split = blockIdx.x, h0 = blockIdx.y * kNH, b = blockIdx.z;
  const int warp = __shfl_sync(0xffffffffu, threadIdx.x >> 5, 0), lane = threadIdx.x & 31;      // warp-uniform
  const int n_chunks = (p.R + 63) / 64, n_pairs = (n_chunks + 1) / 2;

  if (threadIdx.x == 0) {
    mbar_init(q_full, 1);
    mbar_init(p_full, 128);
    mbar_init(pv_full, 1);
    for (int i = 0; i < 2; ++i) {
      mbar_init(&rot_full[i], 1);
      mbar_init(&rot_empty[i], 1);
      mbar_init(&s_full[i], 1);
    }
    for (int i = 0; i < kSlots; ++i) {
      mbar_init(&pair_full[i], 1);
      mbar_init(&pair_empty[i], 1);
    }
    *abort_flag = 0;
    fence_mbar_init();
  }
  if (warp == 1) {
    tmem_alloc(tmem_slot, kTmemCols);
    tmem_relinquish();
  }
  tc_fence_before_sync();
  __syncthreads();
  tc_fence_after_sync();
  const uint32_t tmem = *tmem_slot;
  pdl_wait();
  pdl_launch_dependents();
  const int kv_len = min(p.kv_lens[b], p.max_len);
  const int tiles = (kv_len + kTile - 1) / kTile, per = (tiles + p.splits - 1) / p.splits;
  const int first = min(split * per, tiles), n_tiles = min(per, tiles - first);

  if (warp == 0) {
    if (lane == 0 && n_tiles > 0) {
      mbar_arrive_expect_tx(q_full, (n_chunks + 1) * kQChunkD);
      for (int c = 0; c < n_chunks; ++c) tma_load_3d(smem + kOffQ + c * kQChunkD, &tq, q_full, c * 64, h0, b);
      tma_load_3d(smem + kOffQ + n_chunks * kQChunkD, &tqr, q_full, 0, h0, b);
      int slot_row = p.slots[b];
      if (slot_row < 0 || slot_row >= p.num_slots) slot_row = 0;
      int it = 0, rots = 0;
      bool ok = true;
      for (int n = 0; n < n_tiles && ok; ++n) {
        const int tok = (first + n) * kTile;
        for (int q = 0; q < n_pairs && ok; ++q) {
          const int s = it % kSlots;
          ok = mbar_wait(&pair_empty[s], ((it / kSlots) & 1) ^ 1, abort_flag, kWaitNs);
          if (!ok) break;
          mbar_arrive_expect_tx(&pair_full[s], kPair);
          tma_load_3d(smem + s * kPair, &tc, &pair_full[s], q * 128, tok, slot_row);
          tma_load_3d(smem + s * kPair + kChunk, &tc, &pair_full[s], q * 128 + 64, tok, slot_row);
          ++it;
        }
        const int e = n & 1;
        if (ok) ok = mbar_wait(&rot_empty[e], ((n >> 1) & 1) ^ 1, abort_flag, kWaitNs);
        if (!ok) break;
        mbar_arrive_expect_tx(&rot_full[e], kChunk);
        tma_load_3d(smem + kOffRot + e * kChunk, &tr, &rot_full[e], 0, tok, slot_row);
        ++rots;
      }
      if (!ok) {
        *abort_flag = 1;
        mbar_wait(q_full, 0, nullptr, kWaitNs);
        for (int i = max(0, it - kSlots); i < it; ++i) mbar_wait(&pair_full[i % kSlots], (i / kSlots) & 1, nullptr, kWaitNs);
        for (int i = max(0, rots - 2); i < rots; ++i) mbar_wait(&rot_full[i & 1], (i >> 1) & 1, nullptr, kWaitNs);
      }
    }
  } else if (warp == 1) {
    if (n_tiles > 0) {
      constexpr uint32_t idesc_s = make_idesc(1u, kTile, kNH);
      constexpr uint32_t idesc_pv = make_idesc(1u, 128, kNH) | kMajorA;
      // descriptors advance by plain additions (the address field counts 16-byte units and never overflows)
      const uint64_t dq = make_smem_desc_sw128(smem_u32(smem + kOffQ)), dp = make_smem_desc_sw128(smem_u32(smem + kOffP));
      const uint64_t drot = make_smem_desc_sw128(smem_u32(smem + kOffRot));
      const uint64_t dk = make_smem_desc_sw128(smem_u32(smem)), dv = make_smem_desc_sw128_mn(smem_u32(smem), kChunk);
      int s_slot = 0, s_phase = 0, v_slot = 0;       // ring positions of the score and of the value products
      // S^T of tile n; its columns were read before P of tile n - 2 was waited for
      auto issue_s = [&](int n) -> bool {
        const int e = n & 1;
        const uint32_t d = tmem + e * kNH;
        for (int q = 0; q < n_pairs; ++q) {
          if (!mbar_wait(&pair_full[s_slot], s_phase, abort_flag, kWaitNs)) return false;
          tc_fence_after_sync();
          const uint64_t a = dk + s_slot * (kPair >> 4), b = dq + 2 * q * (kQChunkD >> 4);
#pragma unroll
          for (int k = 0; k < 4; ++k) umma_f16_elect(d, a + 2 * k, b + 2 * k, idesc_s, (q > 0 || k > 0) ? 1u : 0u);
          if (2 * q + 1 < n_chunks) {
#pragma unroll
            for (int k = 0; k < 4; ++k) umma_f16_elect(d, a + (kChunk >> 4) + 2 * k, b + (kQChunkD >> 4) + 2 * k, idesc_s, 1u);
          }
          if (++s_slot == kSlots) s_slot = 0, s_phase ^= 1;
        }
        if (!mbar_wait(&rot_full[e], (n >> 1) & 1, abort_flag, kWaitNs)) return false;
        tc_fence_after_sync();
        for (int k = 0; k * kUmmaK < p.r; ++k)
          umma_f16_elect(d, drot + e * (kChunk >> 4) + 2 * k, dq + n_chunks * (kQChunkD >> 4) + 2 * k, idesc_s, 1u);
        umma_commit_elect(&rot_empty[e]);
        umma_commit_elect(&s_full[e]);
        return true;
      };
      bool ok = mbar_wait(q_full, 0, abort_flag, kWaitNs) && issue_s(0);
      for (int n = 0; n < n_tiles && ok; ++n) {
        if (n + 1 < n_tiles) ok = issue_s(n + 1);
        if (ok) ok = mbar_wait(p_full, n & 1, abort_flag, kWaitNs);
        if (!ok) break;
        tc_fence_after_sync();
        for (int q = 0; q < n_pairs; ++q) {
          const uint64_t a = dv + v_slot * (kPair >> 4);
#pragma unroll
          for (int k = 0; k < kTile / kUmmaK; ++k)
            umma_f16_elect(tmem + kTmemO + q * kNH, a + k * (2048 >> 4), dp + 2 * k, idesc_pv, (n > 0 || k > 0) ? 1u : 0u);
          umma_commit_elect(&pair_empty[v_slot]);
          if (++v_slot == kSlots) v_slot = 0;
        }
        umma_commit_elect(pv_full);
      }
      if (!ok) *abort_flag = 1;
    }
  } else {
    float* red = reinterpret_cast<float*>(smem + kOffRed);
    const int qd = warp & 3;              // TMEM lane quarter of this warp
    float* my_m = red + 256 + qd * 32;
    float* my_alpha = red + 384 + qd * 32;
    const uint32_t lane_off = static_cast<uint32_t>(qd * 32) << 16;
    constexpr float kRescaleStep = 8.f;
    const int t0 = qd * 16 + (lane >> 2); // this thread's tokens inside the tile: t0, t0 + 8
    const int h0t = 2 * (lane & 3);       // its heads: element k is head 8 (k / 2) + h0t + k % 2
    const int my_head = 8 * (lane >> 3) + h0t + ((lane >> 2) & 1);     // the head a transposed reduction leaves in this lane
    float m = -INFINITY;                  // reference maximum of head h0 + lane (the same in all four warps)
    float l[8];                           // this thread's share of its heads' sums
#pragma unroll
    for (int k = 0; k < 8; ++k) l[k] = 0.f;
    auto mx = [](float a, float c) { return fmaxf(a, c); };
    // After a timeout the waits return at once and the loop runs through: the warps meet at barriers, so none may leave.
    for (int n = 0; n < n_tiles; ++n) {
      const int e = n & 1;
      if (!mbar_wait(&s_full[e], (n >> 1) & 1, abort_flag, kWaitNs)) *abort_flag = 1;
      __syncwarp();
      tc_fence_after_sync();
      uint32_t s[16];
      tmem_ld_16x256b_x4(tmem + e * kNH + lane_off, s);
      tmem_ld_wait();
      tc_fence_before_sync();
      const int tok = (first + n) * kTile + t0;
      const bool seen0 = tok < kv_len, seen1 = tok + 8 < kv_len;
      float x[16], v[8];                  // x[2 k + i]: head element k, token t0 + 8 i
#pragma unroll
      for (int k = 0; k < 8; ++k) {
        const int at = 4 * (k >> 1) + (k & 1);
        x[2 * k] = seen0 ? __uint_as_float(s[at]) * p.scale_log2 : -INFINITY;
        x[2 * k + 1] = seen1 ? __uint_as_float(s[at + 2]) * p.scale_log2 : -INFINITY;
        v[k] = fmaxf(x[2 * k], x[2 * k + 1]);
      }
      float* red_max = red + e * 128;     // a fast warp may be at the next tile while a slow one still reads this one's
      red_max[qd * 32 + my_head] = reduce_transposed(v, lane, mx);
      softmax_warps_sync();
      const float top = fmaxf(fmaxf(red_max[lane], red_max[32 + lane]), fmaxf(red_max[64 + lane], red_max[96 + lane]));
      float alpha = 1.f;
      bool raise = false;
      if (top > m) {
        if (m == -INFINITY) {
          m = top;
        } else if (top - m > kRescaleStep) {
          alpha = ex2(m - top);
          m = top;
          raise = true;
        }
      }
      const bool any = __any_sync(0xffffffffu, raise);
      my_m[lane] = m == -INFINITY ? 0.f : m;
      my_alpha[lane] = alpha;
      __syncwarp();
      // the previous tile's second product read the P buffer and wrote the O^T columns that a rescale touches
      if (n > 0 && !mbar_wait(pv_full, (n - 1) & 1, abort_flag, kWaitNs)) *abort_flag = 1;
      __syncwarp();
      if (any) {
        tc_fence_after_sync();
        for (int q = 0; q < n_pairs; ++q) {
          uint32_t o[32];
          tmem_ld_32x32(tmem + kTmemO + q * kNH + lane_off, o);
          tmem_ld_wait();
#pragma unroll
          for (int h = 0; h < kNH; ++h) o[h] = __float_as_uint(__uint_as_float(o[h]) * my_alpha[h]);
          tmem_st_32x32(tmem + kTmemO + q * kNH + lane_off, o);
        }
        tmem_st_wait();
        tc_fence_before_sync();
#pragma unroll
        for (int k = 0; k < 8; ++k) l[k] *= my_alpha[8 * (k >> 1) + h0t + (k & 1)];
      }
      // P^T: a head's row of 64 tokens is 128 bytes, swizzled in 16-byte pieces
      uint8_t* prow = smem + kOffP + (t0 & 7) * 2;
      const int piece = t0 >> 3;          // of token t0; token t0 + 8 is in the next one
#pragma unroll
      for (int k = 0; k < 8; ++k) {
        const int h = 8 * (k >> 1) + h0t + (k & 1);
        const float mh = my_m[h], e0 = ex2(x[2 * k] - mh), e1 = ex2(x[2 * k + 1] - mh);
        l[k] += e0 + e1;
        *reinterpret_cast<__nv_bfloat16*>(prow + h * 128 + ((piece ^ (h & 7)) << 4)) = __float2bfloat16(e0);
        *reinterpret_cast<__nv_bfloat16*>(prow + h * 128 + (((piece + 1) ^ (h & 7)) << 4)) = __float2bfloat16(e1);
      }
      fence_proxy_async_smem();
      mbar_arrive(p_full);
    }
    // sums over tokens, then the output columns
    softmax_warps_sync();
    red[qd * 32 + my_head] = reduce_transposed(l, lane, [](float a, float c) { return a + c; });
    softmax_warps_sync();
    if (qd == 0 && h0 + lane < p.H) {
      const float sum = red[lane] + red[32 + lane] + red[64 + lane] + red[96 + lane];
      p.ml[(static_cast<int64_t>(b) * p.H + h0 + lane) * p.splits + split] = make_float2(m, sum);
    }
    if (n_tiles > 0) {
      if (!mbar_wait(pv_full, (n_tiles - 1) & 1, abort_flag, kWaitNs)) *abort_flag = 1;
      __syncwarp();
      tc_fence_after_sync();
      const int nh = min(kNH, p.H - h0);
      for (int q = 0; q < n_pairs; ++q) {
        uint32_t o[32];
        tmem_ld_32x32(tmem + kTmemO + q * kNH + lane_off, o);
        tmem_ld_wait();
        const int c = q * 128 + qd * 32 + lane;
        if (c < p.R) {
          float* dst = p.o + ((static_cast<int64_t>(b) * p.H + h0) * p.splits + split) * p.R + c;
#pragma unroll
          for (int h = 0; h < kNH; ++h)
            if (h < nh) dst[static_cast<int64_t>(h) * p.splits * p.R] = __uint_as_float(o[h]);
        }
      }
      tc_fence_before_sync();
    }
  }

  tc_fence_before_sync();
  __syncthreads();
  if (threadIdx.x == 0 && *abort_flag != 0 && p.error_flag != nullptr) *p.error_flag = 1;
  if (warp == 1) {
    tc_fence_after_sync();
    tmem_dealloc(tmem, kTmemCols);
  }
}

}  // namespace

cudaError_t launch_latent_prefill(const LatentPrefillArgs& a, cudaStream_t s) {
  if (a.d < 8 || a.d > 128 || a.r < 8 || a.r > 64 || a.dv < 8 || a.dv > 128 || a.d % 8 || a.r % 8 || a.dv % 8 || a.R % 8 || a.L % 64 ||
      a.ld_q % 8 || a.ld_gate % 8 || (reinterpret_cast<uintptr_t>(a.gate) & 15u) != 0 || !(a.scale > 0.f))
    return cudaErrorInvalidValue;
  if (a.B == 0 || a.max_q == 0) return cudaSuccess;
  const int nc = a.d > 64 ? 3 : 2, DV = a.dv > 64 ? 128 : 64;
  const __nv_bfloat16* q = reinterpret_cast<const __nv_bfloat16*>(a.q);
  const __nv_bfloat16* ctx = reinterpret_cast<const __nv_bfloat16*>(a.ctx);
  CUtensorMap m[5];
  if (!encode3(&m[0], q, a.H, a.T, a.d, a.ld_q, a.d + a.r, kBM, 64) || !encode3(&m[1], q + a.d, a.H, a.T, a.r, a.ld_q, a.d + a.r, kBM, 64) ||
      !encode3(&m[2], a.k, a.H, a.L, a.d, static_cast<uint64_t>(a.H) * a.d, a.d, kBN, 64) ||
      !encode2(&m[3], ctx + a.R, a.L, a.r, a.R + a.r, kBN, 64) ||
      !encode3(&m[4], a.vt, a.H, a.dv, a.L, a.L, static_cast<uint64_t>(a.L) * a.dv, DV, 64))
    return cudaErrorInvalidValue;
  PrefillParams p = {};
  p.f.out = reinterpret_cast<__nv_bfloat16*>(a.out);
  p.f.cu_seqlens_q = a.cu;
  p.f.q_pos0 = a.q_pos0;
  p.f.kv_lens = a.kv_lens;
  p.f.Hq = p.f.Hkv = a.H;
  p.f.group = 1;
  p.f.causal = 1;
  p.f.dv = a.dv;
  p.f.scale_log2 = a.scale * 1.4426950408889634f;
  p.f.total_q = a.T;
  p.f.error_flag = a.error_flag;
  p.f.epi.gate = a.gate;
  p.f.epi.ld_gate = a.ld_gate;
  p.ctx0 = a.ctx0;
  p.d = a.d;
  p.r = a.r;
  const dim3 grid(a.H, (a.max_q + 2 * kBM - 1) / (2 * kBM), a.B);
  if (nc == 3) return DV == 128 ? launch_prefill_t<3, 128>(m, p, grid, s) : launch_prefill_t<3, 64>(m, p, grid, s);
  return DV == 128 ? launch_prefill_t<2, 128>(m, p, grid, s) : launch_prefill_t<2, 64>(m, p, grid, s);
}

cudaError_t launch_latent_decode(const LatentDecodeArgs& a, cudaStream_t s) {
  if (a.R < 8 || a.R > 512 || a.r < 8 || a.r > 64 || a.R % 8 || a.r % 8 || a.splits < 1 || a.H < 1) return cudaErrorInvalidValue;
  if (a.B == 0) return cudaSuccess;
  const int W = a.R + a.r;
  const __nv_bfloat16* q = reinterpret_cast<const __nv_bfloat16*>(a.q_eff);
  const __nv_bfloat16* c = reinterpret_cast<const __nv_bfloat16*>(a.cache);
  const uint64_t seq = static_cast<uint64_t>(a.max_len) * W;
  CUtensorMap mq, mqr, mc, mr;
  if (!encode3(&mq, q, a.B, a.H, a.R, W, static_cast<uint64_t>(a.H) * W, kNH, 64) ||
      !encode3(&mqr, q + a.R, a.B, a.H, a.r, W, static_cast<uint64_t>(a.H) * W, kNH, 64) ||
      !encode3(&mc, c, a.num_slots, a.max_len, a.R, W, seq, kTile, 64) ||
      !encode3(&mr, c + a.R, a.num_slots, a.max_len, a.r, W, seq, kTile, 64))
    return cudaErrorInvalidValue;
  static SmemOptIn opt;
  cudaError_t e = opt.ensure(latent_decode_kernel, kDecSmem);
  if (e != cudaSuccess) return e;
  DecodeParams p;
  p.slots = a.slots;
  p.kv_lens = a.kv_lens;
  p.o = a.o;
  p.ml = reinterpret_cast<float2*>(a.ml);
  p.B = a.B; p.H = a.H; p.R = a.R; p.r = a.r;
  p.splits = a.splits;
  p.num_slots = a.num_slots;
  p.max_len = a.max_len;
  p.scale_log2 = a.scale * 1.4426950408889634f;
  p.error_flag = a.error_flag;
  const dim3 grid(a.splits, (a.H + kNH - 1) / kNH, a.B);
  return launch_pdl(latent_decode_kernel, grid, dim3(kDecThreads), static_cast<size_t>(kDecSmem), s, mq, mqr, mc, mr, p);
}

}  // namespace tdb
