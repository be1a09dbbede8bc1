// Pieces of the chunk-parallel recurrence kernels (gla_chunk.cu, delta_chunk.cu): fp32 operands as a high and a low bf16 part,
// positions of the 64-token chunks, fragment loads.
#pragma once
#include "attn_device.cuh"
#include "ptx.cuh"

namespace tdb {
namespace chunk {

constexpr int kC = 64;            // tokens per chunk

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
template <typename Args>
TDB_DEVICE ChunkPos chunk_pos(const Args& p, int chunk) {
  ChunkPos r;
  r.t0 = p.chunk_t0[chunk];
  const int64_t end = p.cu[p.chunk_seq[chunk] + 1];
  r.n = static_cast<int>(min(static_cast<int64_t>(kC), end - r.t0));
  return r;
}

TDB_DEVICE void ldmatrix_x4(uint32_t (&r)[4], const void* smem_row) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(smem_u32(smem_row)));
}

// Rows [0, 64) of `cols` bf16 columns starting at src (row stride ld) into smem with row pitch `pitch` elements, by `threads`
// threads; rows >= n are zero.  Asynchronous (cp.async).
TDB_DEVICE void load_tile(__nv_bfloat16* dst, int pitch, const __nv_bfloat16* src, int64_t ld, int cols, int n, int threads) {
  const int vec = cols >> 3;
  for (int i = threadIdx.x; i < kC * vec; i += threads) {
    const int r = i / vec, c = i - r * vec;
    attn::cp_async16(dst + r * pitch + c * 8, src + (r < n ? r * ld : 0) + c * 8, r < n);
  }
}

}  // namespace chunk
}  // namespace tdb
