// Gated delta rule, chunk-parallel form for bf16 activations (recurrence and decode form in delta.cu).
//
// Inside a 64-token chunk, with gc the cumulative log decay (inclusive), S the state before it and rows i, j:
//     L[i][j] = beta_i (k_i . k_j) e^{gc_i - gc_j}  (i > j),     A = (I + L)^-1,     P[i][j] = (q_i . k_j) e^{gc_i - gc_j}  (i >= j)
//     w = A (beta e^{gc} k),   u = A (beta v):       what the tokens write is u - w S
//     S_end = e^{gc_63} S + (k e^{gc_63 - gc})^T (u - w S)     o = (q e^{gc}) S + P (u - w S)
// Everything but S is local to the chunk, so the chunk is reduced to four matrices before S is known:
//     trans  = -(k e^{gc_63 - gc})^T w   [dk, dk]        inject = (k e^{gc_63 - gc})^T u   [dk, dv]
//     read   = q e^{gc} - P w            [64, dk]        local  = P u                      [64, dv]
// and the sequential part of a chunk is ONE product, S <- e^{gc_63} S + trans S + inject.  Three launches after the inputs:
//   delta_local_kernel  one CTA per (chunk, head): the four matrices
//   delta_state_kernel  one CTA per (16 or 32 columns of dv, head, sequence) walks the chunks; the state stays in registers in fp32, the
//                       next chunk's operands travel meanwhile; the state before every chunk is written out
//   delta_out_kernel    one CTA per (chunk, head): read S + local, head norm, output gate
// Operands are stored in the order in which the lanes of a warp hold the fragments of m16n8k16.
//
// Exponentials are only taken of differences that are <= 0.  State and recurrence count as fp32: the tensor cores (mma.sync
// bf16, fp32 accumulate) get every fp32 operand as a high and a low bf16 part, two products where one side is bf16 anyway (v),
// three where both are fp32; the triangular inverse is plain fp32.
#include "tdb/attn_device.cuh"
#include "tdb/chunk.cuh"
#include "tdb/delta.h"
#include "tdb/launch.cuh"
#include "tdb/vec.cuh"

namespace tdb {

namespace {

using attn::cp_async_commit;
using attn::cp_async_wait;
using attn::ldmatrix_x4_trans;
using attn::mma_bf16;
using namespace chunk;

constexpr int kThreads = 256;
constexpr int kFp = kC + 4;       // pitch of fp32 [64][64] matrices
constexpr int kSp = kC + 8;       // pitch of bf16 [64][64] slabs

// ---------------------------------------------------------------------------------------------------- chunk-local matrices
// Lower 16 x 16 block (bi, bj) of a 64 x 64 matrix.
TDB_DEVICE constexpr int lower_block(int bi, int bj) { return bi * (bi + 1) / 2 + bj; }
constexpr int kFrags = 10 * 64;    // uint4 of a lower triangular matrix as A fragments: ten blocks, high and low parts of 32 lanes

struct LocalSmem {
  int kp;                          // pitch of K / Q
  __nv_bfloat16 *kh, *kl, *qh, *ql, *sh, *sl, *vs;
  uint4 *pf, *uf, *wf;             // fragments of P, of A beta and of A beta e^{gc}
  float *A, *gc, *beta;
  __device__ LocalSmem(uint8_t* base, int dk) {
    kp = dk + 8;
    kh = reinterpret_cast<__nv_bfloat16*>(base);
    kl = kh + kC * kp;
    pf = reinterpret_cast<uint4*>(kl + kC * kp);
    uf = pf + kFrags;
    wf = uf + kFrags;
    A = reinterpret_cast<float*>(uf);                     // until its fragments take its place
    gc = reinterpret_cast<float*>(wf + kFrags);
    beta = gc + kC;
    qh = reinterpret_cast<__nv_bfloat16*>(beta + kC);     // only until the scores are there; then the slabs
    ql = qh + kC * kp;
    sh = qh;
    sl = sh + kC * kSp;
    vs = sl + kC * kSp;
  }
};
static_assert(kC * kFp * 4 <= 2 * kFrags * 16, "the fp32 matrix must fit where its fragments go");
size_t local_smem(int dk) {
  const size_t q = 2 * static_cast<size_t>(kC) * (dk + 8) * 2, slabs = 3 * static_cast<size_t>(kC) * kSp * 2;
  return 2 * static_cast<size_t>(kC) * (dk + 8) * 2 + 3 * kFrags * 16 + 2 * kC * 4 + (q > slabs ? q : slabs);
}

// 16 x 16 block (bi, bj) of X K^T with X as (xh, xl): two tiles of eight columns.
TDB_DEVICE void score_block(const LocalSmem& s, const __nv_bfloat16* xh, const __nv_bfloat16* xl, int dk, int bi, int bj, float (&acc)[2][4]) {
  const int lane = threadIdx.x & 31, mat = lane >> 3, mr = lane & 7;
  float lo[2][4];
#pragma unroll
  for (int j = 0; j < 2; ++j) {
    acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
    lo[j][0] = lo[j][1] = lo[j][2] = lo[j][3] = 0.f;
  }
  const int arow = (bi * 16 + (mat & 1) * 8 + mr) * s.kp + (mat >> 1) * 8;
  const int brow = (bj * 16 + (mat >> 1) * 8 + mr) * s.kp + (mat & 1) * 8;
#pragma unroll 2
  for (int k0 = 0; k0 < dk; k0 += 16) {
    uint32_t ah[4], al[4], bh[4], bl[4];
    ldmatrix_x4(ah, xh + arow + k0);
    ldmatrix_x4(bh, s.kh + brow + k0);
    ldmatrix_x4(bl, s.kl + brow + k0);
    ldmatrix_x4(al, xl + arow + k0);
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      mma_bf16(acc[j], ah, bh[2 * j], bh[2 * j + 1]);
      mma_bf16(lo[j], ah, bl[2 * j], bl[2 * j + 1]);
      mma_bf16(lo[j], al, bh[2 * j], bh[2 * j + 1]);
    }
  }
#pragma unroll
  for (int j = 0; j < 2; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) acc[j][e] += lo[j][e];
}

// Two neighbouring accumulator tiles are one A fragment: high and low parts to dst[0] and dst[32].
TDB_DEVICE void store_a_fragment(uint4* dst, const float (&a)[4], const float (&b)[4]) {
  const HiLo r0 = split2(a[0], a[1]), r1 = split2(a[2], a[3]), r2 = split2(b[0], b[1]), r3 = split2(b[2], b[3]);
  dst[0] = make_uint4(r0.hi, r1.hi, r2.hi, r3.hi);
  dst[32] = make_uint4(r0.lo, r1.lo, r2.lo, r3.lo);
}

// A <- (I + A)^-1 for the strictly lower triangular A (blocks above the diagonal are scratch).
TDB_DEVICE void invert_unit_lower(float* A) {
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  if (warp < 4) {                       // the 16 x 16 blocks on the diagonal by substitution, a column per lane
    float* D = A + (warp * 16) * kFp + warp * 16;
    float x[16];
    const int j = lane & 15;
#pragma unroll
    for (int i = 0; i < 16; ++i) {
      float a = (i == j) ? 1.f : 0.f, b = 0.f;
#pragma unroll
      for (int m = 0; m < i; ++m) {
        if (m & 1) a = fmaf(-D[i * kFp + m], x[m], a);
        else b = fmaf(-D[i * kFp + m], x[m], b);
      }
      x[i] = a + b;
    }
    __syncwarp();
    if (lane < 16) {
#pragma unroll
      for (int i = 0; i < 16; ++i) D[i * kFp + j] = i >= j ? x[i] : 0.f;
    }
  }
  __syncthreads();
  // blocks below the diagonal, 16 then 32: A21 = -A22 (L21 A11); the product in brackets goes to the block above the diagonal.
  // A thread owns four neighbouring columns of a row.
#pragma unroll
  for (int n = 16; n <= 32; n *= 2) {
    const int per = n * n / 4, all = 32 / n * per;
    for (int i = tid; i < all; i += kThreads) {
      const int b = (i / per) * 2 * n, r = (i % per) / (n / 4), c = (i % (n / 4)) * 4;
      float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 4
      for (int m = c & ~15; m < n; ++m) {
        const float l = A[(b + n + r) * kFp + b + m];
        const float4 v = *reinterpret_cast<const float4*>(A + (b + m) * kFp + b + c);
        a.x = fmaf(l, v.x, a.x); a.y = fmaf(l, v.y, a.y); a.z = fmaf(l, v.z, a.z); a.w = fmaf(l, v.w, a.w);
      }
      *reinterpret_cast<float4*>(A + (b + r) * kFp + b + n + c) = a;
    }
    __syncthreads();
    for (int i = tid; i < all; i += kThreads) {
      const int b = (i / per) * 2 * n, r = (i % per) / (n / 4), c = (i % (n / 4)) * 4;
      float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 4
      for (int m = 0; m < (r & ~15) + 16; ++m) {
        const float l = -A[(b + n + r) * kFp + b + n + m];
        const float4 v = *reinterpret_cast<const float4*>(A + (b + m) * kFp + b + n + c);
        a.x = fmaf(l, v.x, a.x); a.y = fmaf(l, v.y, a.y); a.z = fmaf(l, v.z, a.z); a.w = fmaf(l, v.w, a.w);
      }
      *reinterpret_cast<float4*>(A + (b + n + r) * kFp + b + c) = a;
    }
    __syncthreads();
  }
}

// Fragments of A beta and A beta e^{gc} take the place of A.
TDB_DEVICE void split_inverse(const LocalSmem& s) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t4 = lane & 3;
  float x[2][8], f[2][4];
#pragma unroll
  for (int u = 0; u < 2; ++u) {
    const int i = warp + 8 * u;
    if (i >= 10) break;
    const int bi = i < 1 ? 0 : i < 3 ? 1 : i < 6 ? 2 : 3, bj = i - lower_block(bi, 0);
    const int c = bj * 16 + 2 * t4;
    const float* a = s.A + (bi * 16 + g) * kFp + c;
    const float* b = a + 8 * kFp;
    const float b0 = s.beta[c], b1 = s.beta[c + 1], b2 = s.beta[c + 8], b3 = s.beta[c + 9];
    x[u][0] = a[0] * b0; x[u][1] = a[1] * b1; x[u][2] = b[0] * b0; x[u][3] = b[1] * b1;
    x[u][4] = a[8] * b2; x[u][5] = a[9] * b3; x[u][6] = b[8] * b2; x[u][7] = b[9] * b3;
    f[u][0] = __expf(s.gc[c]); f[u][1] = __expf(s.gc[c + 1]); f[u][2] = __expf(s.gc[c + 8]); f[u][3] = __expf(s.gc[c + 9]);
  }
  __syncthreads();
#pragma unroll
  for (int u = 0; u < 2; ++u) {
    const int i = warp + 8 * u;
    if (i >= 10) break;
    const float a[4] = {x[u][0], x[u][1], x[u][2], x[u][3]}, b[4] = {x[u][4], x[u][5], x[u][6], x[u][7]};
    store_a_fragment(s.uf + i * 64 + lane, a, b);
    const float c[4] = {a[0] * f[u][0], a[1] * f[u][1], a[2] * f[u][0], a[3] * f[u][1]};
    const float d[4] = {b[0] * f[u][2], b[1] * f[u][3], b[2] * f[u][2], b[3] * f[u][3]};
    store_a_fragment(s.wf + i * 64 + lane, c, d);
  }
  __syncthreads();
}

// Row blocks rb and 3 - rb of (lower triangular X as fragments) x (64 tokens x 16 columns from col of B, bf16 in one or two parts):
// the two together have the same length for every rb.  Columns beyond the tensor yield numbers that nobody uses.
template <bool SPLIT_B>
TDB_DEVICE void lower_product(float (&acc)[2][2][4], const uint4* xf, int rb, const __nv_bfloat16* bh, const __nv_bfloat16* bl, int bp, int col) {
  const int lane = threadIdx.x & 31, mat = lane >> 3, mr = lane & 7;
  float lo[2][2][4];
#pragma unroll
  for (int i = 0; i < 2; ++i)
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      acc[i][j][0] = acc[i][j][1] = acc[i][j][2] = acc[i][j][3] = 0.f;
      lo[i][j][0] = lo[i][j][1] = lo[i][j][2] = lo[i][j][3] = 0.f;
    }
  auto row = [&](int i, int kb, const uint32_t (&b)[4], const uint32_t (&c)[4]) {
    const uint4* x = xf + lower_block(i == 0 ? rb : 3 - rb, kb) * 64 + lane;
    const uint4 h = x[0], l = x[32];
    const uint32_t ah[4] = {h.x, h.y, h.z, h.w}, al[4] = {l.x, l.y, l.z, l.w};
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      mma_bf16(acc[i][j], ah, b[2 * j], b[2 * j + 1]);
      mma_bf16(lo[i][j], al, b[2 * j], b[2 * j + 1]);
      if constexpr (SPLIT_B) mma_bf16(lo[i][j], ah, c[2 * j], c[2 * j + 1]);
    }
  };
  for (int kb = 0; kb <= 3 - rb; ++kb) {
    const int brow = (kb * 16 + (mat & 1) * 8 + mr) * bp + col + (mat >> 1) * 8;
    uint32_t b[4], c[4] = {};
    ldmatrix_x4_trans(b, bh + brow);
    if constexpr (SPLIT_B) ldmatrix_x4_trans(c, bl + brow);
    row(1, kb, b, c);
    if (kb <= rb) row(0, kb, b, c);
  }
#pragma unroll
  for (int i = 0; i < 2; ++i)
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[i][j][e] += lo[i][j][e];
}

__global__ void __launch_bounds__(kThreads, 2) delta_local_kernel(const DeltaArgs p) {
  extern __shared__ __align__(16) uint8_t smem[];
  const LocalSmem s(smem, p.dk);
  const int chunk = blockIdx.x, h = blockIdx.y, g_head = h / (p.H / p.G);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t4 = lane & 3;
  const int mat = lane >> 3, mr = lane & 7;
  pdl_wait();
  pdl_launch_dependents();
  const ChunkPos cp = chunk_pos(p, chunk);
  const int64_t Gk = static_cast<int64_t>(p.G) * p.dk, Hv = static_cast<int64_t>(p.H) * p.dv;
  const int64_t qk_at = cp.t0 * Gk + static_cast<int64_t>(g_head) * p.dk;
  const __nv_bfloat16* qh_g = reinterpret_cast<const __nv_bfloat16*>(p.q) + qk_at;
  const __nv_bfloat16* ql_g = reinterpret_cast<const __nv_bfloat16*>(p.q_lo) + qk_at;
  const __nv_bfloat16* v_g = reinterpret_cast<const __nv_bfloat16*>(p.v) + cp.t0 * Hv + static_cast<int64_t>(h) * p.dv;
  load_tile(s.kh, s.kp, reinterpret_cast<const __nv_bfloat16*>(p.k) + qk_at, Gk, p.dk, cp.n, kThreads);
  load_tile(s.kl, s.kp, reinterpret_cast<const __nv_bfloat16*>(p.k_lo) + qk_at, Gk, p.dk, cp.n, kThreads);
  load_tile(s.qh, s.kp, qh_g, Gk, p.dk, cp.n, kThreads);
  load_tile(s.ql, s.kp, ql_g, Gk, p.dk, cp.n, kThreads);
  cp_async_commit();
  if (warp == 0) {                      // inclusive scan of the log decays, two tokens per lane
    const int t = 2 * lane;
    const float a = t < cp.n ? p.log_g[(cp.t0 + t) * p.H + h] : 0.f;
    const float b = t + 1 < cp.n ? p.log_g[(cp.t0 + t + 1) * p.H + h] : 0.f;
    float pre = a + b;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float x = __shfl_up_sync(0xffffffffu, pre, o);
      if (lane >= o) pre += x;
    }
    s.gc[t] = pre - b;
    s.gc[t + 1] = pre;
    if (lane == 31) p.decay[static_cast<int64_t>(chunk) * p.H + h] = expf(pre);
  } else if (warp == 1) {
    s.beta[lane] = lane < cp.n ? p.beta[(cp.t0 + lane) * p.H + h] : 0.f;
    s.beta[lane + 32] = lane + 32 < cp.n ? p.beta[(cp.t0 + lane + 32) * p.H + h] : 0.f;
  }
  cp_async_wait<0>();
  __syncthreads();
  // scores: the ten lower blocks of K K^T and of Q K^T
  for (int u = warp; u < 20; u += kThreads / 32) {
    const bool is_q = u >= 10;
    const int i = is_q ? u - 10 : u;
    const int bi = i < 1 ? 0 : i < 3 ? 1 : i < 6 ? 2 : 3, bj = i - lower_block(bi, 0);
    float acc[2][4];
    score_block(s, is_q ? s.qh : s.kh, is_q ? s.ql : s.kl, p.dk, bi, bj, acc);
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int r = bi * 16 + g + 8 * (e >> 1), c = bj * 16 + j * 8 + 2 * t4 + (e & 1);
        acc[j][e] = r >= c ? acc[j][e] * __expf(s.gc[r] - s.gc[c]) : 0.f;
        if (!is_q) s.A[r * kFp + c] = r > c ? acc[j][e] * s.beta[r] : 0.f;
      }
    if (is_q) store_a_fragment(s.pf + i * 64 + lane, acc[0], acc[1]);
  }
  __syncthreads();                      // Q is no longer needed: its place takes the slabs
  load_tile(s.vs, kSp, v_g, Hv, min(64, p.dv), cp.n, kThreads);
  cp_async_commit();
  invert_unit_lower(s.A);
  split_inverse(s);

  const int64_t ch = static_cast<int64_t>(chunk) * p.H + h;
  const int ksteps = p.dk >> 4, vtiles = p.dv >> 3;
  uint4* trans = reinterpret_cast<uint4*>(p.trans) + ch * ksteps * ksteps * 64 + lane;
  uint4* read = reinterpret_cast<uint4*>(p.read) + ch * 4 * ksteps * 64 + lane;
  float4* inject = reinterpret_cast<float4*>(p.inject) + ch * ksteps * vtiles * 32 + lane;
  float4* local = reinterpret_cast<float4*>(p.local) + ch * 4 * vtiles * 32 + lane;
  // a warp owns 16 columns of a slab of 64 for two of the four row blocks
  const int rb = warp >> 2, col = (warp & 3) * 16, rows[2] = {rb, 3 - rb};
  const float gl = s.gc[kC - 1];
  const int wslabs = (p.dk + 63) / 64, slabs = wslabs + (p.dv + 63) / 64;
  for (int sl = 0; sl < slabs; ++sl) {
    const bool is_w = sl < wslabs;
    const int col0 = (is_w ? sl : sl - wslabs) * 64, dim = is_w ? p.dk : p.dv;
    const bool live = col0 + col < dim;
    float acc[2][2][4];
    if (is_w) {
      lower_product<true>(acc, s.wf, rb, s.kh, s.kl, s.kp, live ? col0 + col : 0);
    } else {
      cp_async_wait<0>();
      __syncthreads();
      lower_product<false>(acc, s.uf, rb, s.vs, nullptr, kSp, col);
    }
    auto put = [&](bool decayed) {
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int r = rows[i] * 16 + g;
        const float f0 = decayed ? __expf(gl - s.gc[r]) : 1.f, f1 = decayed ? __expf(gl - s.gc[r + 8]) : 1.f;
#pragma unroll
        for (int j = 0; j < 2; ++j) {
          const HiLo a = split2(acc[i][j][0] * f0, acc[i][j][1] * f0), b = split2(acc[i][j][2] * f1, acc[i][j][3] * f1);
          const int at = r * kSp + col + j * 8 + 2 * t4;
          *reinterpret_cast<uint32_t*>(s.sh + at) = a.hi;
          *reinterpret_cast<uint32_t*>(s.sl + at) = a.lo;
          *reinterpret_cast<uint32_t*>(s.sh + at + 8 * kSp) = b.hi;
          *reinterpret_cast<uint32_t*>(s.sl + at + 8 * kSp) = b.lo;
        }
      }
    };
    put(false);
    __syncthreads();
    if (!is_w && sl + 1 < slabs) {      // every warp is done with this slab of v
      load_tile(s.vs, kSp, v_g + col0 + 64, Hv, min(64, p.dv - col0 - 64), cp.n, kThreads);
      cp_async_commit();
    }
    if (live) {
      float o[2][2][4];
      lower_product<true>(o, s.pf, rb, s.sh, s.sl, kSp, col);
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        if (is_w) {
          const int r0 = rows[i] * 16 + g, r1 = r0 + 8;
          const float e0 = __expf(s.gc[r0]), e1 = __expf(s.gc[r1]);
#pragma unroll
          for (int j = 0; j < 2; ++j) {
            const int c = col0 + col + j * 8 + 2 * t4;
            float2 q0 = make_float2(0.f, 0.f), q1 = q0;
            if (r0 < cp.n) {
              const float2 a = ld2(qh_g + r0 * Gk + c), b = ld2(ql_g + r0 * Gk + c);
              q0 = make_float2(a.x + b.x, a.y + b.y);
            }
            if (r1 < cp.n) {
              const float2 a = ld2(qh_g + r1 * Gk + c), b = ld2(ql_g + r1 * Gk + c);
              q1 = make_float2(a.x + b.x, a.y + b.y);
            }
            o[i][j][0] = fmaf(q0.x, e0, -o[i][j][0]); o[i][j][1] = fmaf(q0.y, e0, -o[i][j][1]);
            o[i][j][2] = fmaf(q1.x, e1, -o[i][j][2]); o[i][j][3] = fmaf(q1.y, e1, -o[i][j][3]);
          }
          store_a_fragment(read + (rows[i] * ksteps + (col0 + col) / 16) * 64, o[i][0], o[i][1]);
        } else {
#pragma unroll
          for (int j = 0; j < 2; ++j)
            local[(rows[i] * vtiles + (col0 + col) / 8 + j) * 32] = make_float4(o[i][j][0], o[i][j][1], o[i][j][2], o[i][j][3]);
        }
      }
    }
    __syncthreads();
    put(true);
    __syncthreads();
    // K^T times the decayed slab: a warp computes 32 x 32 (two row blocks, four tiles)
    for (int u = warp; u < ((ksteps + 1) >> 1) * 2; u += kThreads / 32) {
      const int kb = (u >> 1) * 2, hf = (u & 1) * 32;
      const bool two = kb + 1 < ksteps;
      if (col0 + hf >= dim) continue;
      float o[2][4][4];
#pragma unroll
      for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) o[i][j][0] = o[i][j][1] = o[i][j][2] = o[i][j][3] = 0.f;
#pragma unroll
      for (int ks = 0; ks < 4; ++ks) {
        uint32_t ah[2][4], al[2][4];
        const int arow = (ks * 16 + (mat >> 1) * 8 + mr) * s.kp + kb * 16 + (mat & 1) * 8;
        ldmatrix_x4_trans(ah[0], s.kh + arow);
        ldmatrix_x4_trans(al[0], s.kl + arow);
        ldmatrix_x4_trans(ah[1], s.kh + arow + (two ? 16 : 0));
        ldmatrix_x4_trans(al[1], s.kl + arow + (two ? 16 : 0));
        const int brow = (ks * 16 + (mat & 1) * 8 + mr) * kSp + hf + (mat >> 1) * 8;
#pragma unroll
        for (int j = 0; j < 4; j += 2) {
          uint32_t bh[4], bl[4];
          ldmatrix_x4_trans(bh, s.sh + brow + j * 8);
          ldmatrix_x4_trans(bl, s.sl + brow + j * 8);
#pragma unroll
          for (int i = 0; i < 2; ++i) {
            mma_bf16(o[i][j], ah[i], bh[0], bh[1]);
            mma_bf16(o[i][j + 1], ah[i], bh[2], bh[3]);
          }
#pragma unroll
          for (int i = 0; i < 2; ++i) {
            mma_bf16(o[i][j], ah[i], bl[0], bl[1]);
            mma_bf16(o[i][j + 1], ah[i], bl[2], bl[3]);
          }
#pragma unroll
          for (int i = 0; i < 2; ++i) {
            mma_bf16(o[i][j], al[i], bh[0], bh[1]);
            mma_bf16(o[i][j + 1], al[i], bh[2], bh[3]);
          }
        }
      }
      const int pairs = min(dim - col0 - hf, 32) >> 4;           // of tiles
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        if (i == 1 && !two) break;
        if (is_w) {
#pragma unroll
          for (int j = 0; j < 4; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) o[i][j][e] = -o[i][j][e];
#pragma unroll
          for (int j = 0; j < 4; j += 2)
            if (j / 2 < pairs) store_a_fragment(trans + ((kb + i) * ksteps + (col0 + hf) / 16 + j / 2) * 64, o[i][j], o[i][j + 1]);
        } else {
#pragma unroll
          for (int j = 0; j < 4; ++j)
            if (j / 2 < pairs) inject[((kb + i) * vtiles + (col0 + hf) / 8 + j) * 32] = make_float4(o[i][j][0], o[i][j][1], o[i][j][2], o[i][j][3]);
        }
      }
    }
    __syncthreads();
  }
}

// ---------------------------------------------------------------------------------------------------- sequential part
// KS: 16-row blocks of dk, a warp each; NT: tiles of eight columns per CTA.
template <int KS, int NT>
__global__ void __launch_bounds__(32 * KS, 1) delta_state_kernel(const DeltaArgs p) {
  extern __shared__ __align__(16) uint8_t smem[];
  constexpr int kPitch = NT * 8 + 8;
  constexpr bool kAhead = KS <= 8;          // the next chunk's operands wait in registers
  constexpr int ksteps = KS;
  const int vtiles = p.dv >> 3;
  const int tile0 = blockIdx.x * NT, h = blockIdx.y, n = blockIdx.z;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t4 = lane & 3, mat = lane >> 3, mr = lane & 7;
  const int tiles = min(NT, vtiles - tile0);
  pdl_wait();
  pdl_launch_dependents();
  __nv_bfloat16* buf = reinterpret_cast<__nv_bfloat16*>(smem);       // [2][hi, lo][dk][pitch]
  const int part = p.dk * kPitch;
  float* st = p.state + ((static_cast<int64_t>(p.slots[n]) * p.H + h) * p.dk + warp * 16 + g) * p.dv + tile0 * 8 + 2 * t4;
  float S[NT][4];
#pragma unroll
  for (int j = 0; j < NT; ++j) {
    float2 a = make_float2(0.f, 0.f), b = a;
    if (p.pos0[n] != 0 && j < tiles) {
      a = *reinterpret_cast<const float2*>(st + j * 8);
      b = *reinterpret_cast<const float2*>(st + 8 * p.dv + j * 8);
    }
    S[j][0] = a.x; S[j][1] = a.y; S[j][2] = b.x; S[j][3] = b.y;
  }
  const int c0 = p.seq_chunk0[n], c1 = p.seq_chunk0[n + 1];
  const uint4* trans = reinterpret_cast<const uint4*>(p.trans) + static_cast<int64_t>(warp) * ksteps * 64 + lane;
  const float4* inject = reinterpret_cast<const float4*>(p.inject) + (static_cast<int64_t>(warp) * vtiles + tile0) * 32 + lane;
  uint4* states = reinterpret_cast<uint4*>(p.states) + (static_cast<int64_t>(warp) * vtiles + tile0) * 32 + lane;
  const int64_t tr_step = static_cast<int64_t>(ksteps) * ksteps * 64, in_step = static_cast<int64_t>(ksteps) * vtiles * 32;
  uint4 nh[kAhead ? KS : 1], nl[kAhead ? KS : 1];
  float4 ni[NT] = {};
  float nd = 0.f;
  auto fetch = [&](int c) {
    const int64_t ch = static_cast<int64_t>(c) * p.H + h;
    nd = p.decay[ch];
    if constexpr (kAhead) {
#pragma unroll
      for (int ks = 0; ks < KS; ++ks) {
        nh[ks] = trans[ch * tr_step + ks * 64];
        nl[ks] = trans[ch * tr_step + ks * 64 + 32];
      }
    }
#pragma unroll
    for (int j = 0; j < NT; ++j)
      if (j < tiles) ni[j] = inject[ch * in_step + j * 32];
  };
  if (c0 < c1) fetch(c0);
  for (int c = c0; c < c1; ++c) {
    const int64_t ch = static_cast<int64_t>(c) * p.H + h;
    __nv_bfloat16* hi = buf + ((c - c0) & 1) * 2 * part;
    __nv_bfloat16* lo = hi + part;
#pragma unroll
    for (int j = 0; j < NT; ++j) {
      const HiLo a = split2(S[j][0], S[j][1]), b = split2(S[j][2], S[j][3]);
      const int at = (warp * 16 + g) * kPitch + j * 8 + 2 * t4;
      *reinterpret_cast<uint32_t*>(hi + at) = a.hi;
      *reinterpret_cast<uint32_t*>(lo + at) = a.lo;
      *reinterpret_cast<uint32_t*>(hi + at + 8 * kPitch) = b.hi;
      *reinterpret_cast<uint32_t*>(lo + at + 8 * kPitch) = b.lo;
    }
    uint4 th[kAhead ? KS : 1], tl[kAhead ? KS : 1];
    float acc[NT][4], lo1[NT][4], lo2[NT][4];
#pragma unroll
    for (int j = 0; j < NT; ++j) {
      acc[j][0] = fmaf(nd, S[j][0], ni[j].x); acc[j][1] = fmaf(nd, S[j][1], ni[j].y);
      acc[j][2] = fmaf(nd, S[j][2], ni[j].z); acc[j][3] = fmaf(nd, S[j][3], ni[j].w);
      lo1[j][0] = lo1[j][1] = lo1[j][2] = lo1[j][3] = 0.f;
      lo2[j][0] = lo2[j][1] = lo2[j][2] = lo2[j][3] = 0.f;
    }
    if constexpr (kAhead) {
#pragma unroll
      for (int ks = 0; ks < KS; ++ks) {
        th[ks] = nh[ks];
        tl[ks] = nl[ks];
      }
    }
    if (c + 1 < c1) fetch(c + 1);
    __syncthreads();       // the other buffer is free as well: its readers have passed this barrier
#pragma unroll
    for (int ks = 0; ks < KS; ++ks) {
      uint4 fh, fl;
      if constexpr (kAhead) {
        fh = th[ks];
        fl = tl[ks];
      } else {
        fh = trans[ch * tr_step + ks * 64];
        fl = trans[ch * tr_step + ks * 64 + 32];
      }
      const uint32_t ah[4] = {fh.x, fh.y, fh.z, fh.w}, al[4] = {fl.x, fl.y, fl.z, fl.w};
      const int brow = (ks * 16 + (mat & 1) * 8 + mr) * kPitch + (mat >> 1) * 8;
#pragma unroll
      for (int j = 0; j < NT; j += 2) {
        uint32_t bh[4], bl[4];
        ldmatrix_x4_trans(bh, hi + brow + j * 8);
        ldmatrix_x4_trans(bl, lo + brow + j * 8);
        mma_bf16(acc[j], ah, bh[0], bh[1]);
        mma_bf16(acc[j + 1], ah, bh[2], bh[3]);
        mma_bf16(lo1[j], ah, bl[0], bl[1]);
        mma_bf16(lo1[j + 1], ah, bl[2], bl[3]);
        mma_bf16(lo2[j], al, bh[0], bh[1]);
        mma_bf16(lo2[j + 1], al, bh[2], bh[3]);
        if (ks == warp) {          // a warp writes its own rows of the state before this chunk, as B fragments of the read-out
          if (j < tiles) states[ch * in_step + j * 32] = make_uint4(bh[0], bh[1], bl[0], bl[1]);
          if (j + 1 < tiles) states[ch * in_step + (j + 1) * 32] = make_uint4(bh[2], bh[3], bl[2], bl[3]);
        }
      }
    }
#pragma unroll
    for (int j = 0; j < NT; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) S[j][e] = acc[j][e] + (lo1[j][e] + lo2[j][e]);
  }
#pragma unroll
  for (int j = 0; j < NT; ++j) {
    if (j >= tiles) break;
    *reinterpret_cast<float2*>(st + j * 8) = make_float2(S[j][0], S[j][1]);
    *reinterpret_cast<float2*>(st + 8 * p.dv + j * 8) = make_float2(S[j][2], S[j][3]);
  }
}

// ---------------------------------------------------------------------------------------------------- outputs
// Operands come in stages of kOutSteps k-steps (64 rows of the state) through shared memory, two stages in flight; all of it is
// stored in fragment order, so a stage is a plain copy.
constexpr int kOutSteps = 4;
size_t out_stage(int dv) { return static_cast<size_t>(kOutSteps) * (dv / 8 * 32 + 4 * 64) * 16; }

template <int TW>     // tiles of eight columns per warp: dv <= 16 TW
__global__ void __launch_bounds__(kThreads, TW <= 8 ? 2 : 1) delta_out_kernel(const DeltaArgs p) {
  extern __shared__ __align__(16) uint8_t smem[];
  __shared__ float ssq[2][kC];
  const int chunk = blockIdx.x, h = blockIdx.y;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t4 = lane & 3;
  const int rb = warp >> 1, half = warp & 1;
  const int ksteps = p.dk >> 4, vtiles = p.dv >> 3, tile0 = half * TW, tiles = min(TW, vtiles - tile0);
  pdl_wait();
  pdl_launch_dependents();
  const ChunkPos cp = chunk_pos(p, chunk);
  const int64_t ch = static_cast<int64_t>(chunk) * p.H + h;
  const uint4* read = reinterpret_cast<const uint4*>(p.read) + ch * 4 * ksteps * 64;
  const uint4* states = reinterpret_cast<const uint4*>(p.states) + ch * ksteps * vtiles * 32;
  const float4* local = reinterpret_cast<const float4*>(p.local) + ((ch * 4 + rb) * vtiles + tile0) * 32 + lane;
  uint4* bufs = reinterpret_cast<uint4*>(smem);
  const int b_size = kOutSteps * vtiles * 32, stage = b_size + kOutSteps * 4 * 64;     // uint4 of a stage: states, then rows to read with
  const int stages = (ksteps + kOutSteps - 1) / kOutSteps;
  auto fetch = [&](int st) {
    if (st < stages) {
      const int k0 = st * kOutSteps, kn = min(kOutSteps, ksteps - k0);
      uint4* dst = bufs + (st & 1) * stage;
      for (int i = threadIdx.x; i < kn * vtiles * 32; i += kThreads) attn::cp_async16(dst + i, states + k0 * vtiles * 32 + i, true);
      for (int i = threadIdx.x; i < 4 * kn * 64; i += kThreads) {
        const int r = i / (kn * 64), c = i - r * kn * 64;
        attn::cp_async16(dst + b_size + r * kOutSteps * 64 + c, read + (r * ksteps + k0) * 64 + c, true);
      }
    }
    cp_async_commit();
  };
  fetch(0);
  fetch(1);
  float acc[TW][4];
#pragma unroll
  for (int j = 0; j < TW; ++j) {
    float4 f = make_float4(0.f, 0.f, 0.f, 0.f);
    if (j < tiles) f = local[j * 32];
    acc[j][0] = f.x; acc[j][1] = f.y; acc[j][2] = f.z; acc[j][3] = f.w;
  }
  for (int st = 0; st < stages; ++st) {
    cp_async_wait<1>();
    __syncthreads();
    const uint4* B = bufs + (st & 1) * stage + tile0 * 32 + lane;
    const uint4* A = bufs + (st & 1) * stage + b_size + rb * kOutSteps * 64 + lane;
    const int kn = min(kOutSteps, ksteps - st * kOutSteps);
    if (rb * 16 < cp.n) {
      for (int ks = 0; ks < kn; ++ks) {
        const uint4 fh = A[ks * 64], fl = A[ks * 64 + 32];
        const uint32_t ah[4] = {fh.x, fh.y, fh.z, fh.w}, al[4] = {fl.x, fl.y, fl.z, fl.w};
#pragma unroll
        for (int j0 = 0; j0 < TW; j0 += 4) {
          uint4 b[4];
#pragma unroll
          for (int j = 0; j < 4; ++j) b[j] = B[(ks * vtiles + min(j0 + j, tiles - 1)) * 32];       // tiles beyond the last: unused copies
#pragma unroll
          for (int j = 0; j < 4; ++j) mma_bf16(acc[j0 + j], ah, b[j].x, b[j].y);
#pragma unroll
          for (int j = 0; j < 4; ++j) mma_bf16(acc[j0 + j], ah, b[j].z, b[j].w);
#pragma unroll
          for (int j = 0; j < 4; ++j) mma_bf16(acc[j0 + j], al, b[j].x, b[j].y);
        }
      }
    }
    __syncthreads();
    fetch(st + 2);
  }
#pragma unroll
  for (int j = 0; j < TW; ++j)
    if (j >= tiles) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
  float q0 = 0.f, q1 = 0.f;
#pragma unroll
  for (int j = 0; j < TW; ++j) {
    q0 += acc[j][0] * acc[j][0] + acc[j][1] * acc[j][1];
    q1 += acc[j][2] * acc[j][2] + acc[j][3] * acc[j][3];
  }
  q0 += __shfl_xor_sync(0xffffffffu, q0, 1); q0 += __shfl_xor_sync(0xffffffffu, q0, 2);
  q1 += __shfl_xor_sync(0xffffffffu, q1, 1); q1 += __shfl_xor_sync(0xffffffffu, q1, 2);
  if (t4 == 0) {
    ssq[half][rb * 16 + g] = q0;
    ssq[half][rb * 16 + g + 8] = q1;
  }
  __syncthreads();
  const __nv_bfloat16* gate0 = reinterpret_cast<const __nv_bfloat16*>(p.z) + cp.t0 * p.ld + 2 * p.G * p.dk + p.H * p.dv + h * p.dv;
  __nv_bfloat16* out0 = reinterpret_cast<__nv_bfloat16*>(p.out) + cp.t0 * p.H * p.dv + h * p.dv;
#pragma unroll
  for (int rr = 0; rr < 2; ++rr) {
    const int t = rb * 16 + rr * 8 + g;
    if (t >= cp.n) continue;
    const float inv = 1.f / sqrtf((ssq[0][t] + ssq[1][t]) / p.dv_real + p.eps);
#pragma unroll
    for (int j = 0; j < TW; ++j) {
      if (j >= tiles) break;
      const int c = (tile0 + j) * 8 + 2 * t4;
      const float2 gt = ld2(gate0 + t * p.ld + c);
      const float o0 = acc[j][2 * rr] * inv * p.norm_w[c] * gt.x * sigmoid_f32(gt.x);
      const float o1 = acc[j][2 * rr + 1] * inv * p.norm_w[c + 1] * gt.y * sigmoid_f32(gt.y);
      *reinterpret_cast<uint32_t*>(out0 + static_cast<int64_t>(t) * p.H * p.dv + c) = pack_bf16x2(o0, o1);
    }
  }
}

template <int KS, int NT>
cudaError_t launch_state(const DeltaArgs& a, cudaStream_t s) {
  static SmemOptIn opt;
  constexpr int kMax = 2 * 2 * KS * 16 * (NT * 8 + 8) * 2;
  cudaError_t e = opt.ensure(delta_state_kernel<KS, NT>, kMax);
  if (e != cudaSuccess) return e;
  const int vtiles = a.dv / 8;
  return launch_pdl(delta_state_kernel<KS, NT>, dim3((vtiles + NT - 1) / NT, a.H, a.N), dim3(a.dk * 2),
                    static_cast<size_t>(2 * 2 * a.dk * (NT * 8 + 8) * 2), s, a);
}
template <int NT>
cudaError_t launch_state_nt(const DeltaArgs& a, cudaStream_t s) {
  switch (a.dk / 16) {
    case 1: return launch_state<1, NT>(a, s);
    case 2: return launch_state<2, NT>(a, s);
    case 3: return launch_state<3, NT>(a, s);
    case 4: return launch_state<4, NT>(a, s);
    case 5: return launch_state<5, NT>(a, s);
    case 6: return launch_state<6, NT>(a, s);
    case 8: return launch_state<8, NT>(a, s);
    case 12: return launch_state<12, NT>(a, s);
    case 16: return launch_state<16, NT>(a, s);
    default: return cudaErrorInvalidValue;
  }
}
template <int TW>
cudaError_t launch_out(const DeltaArgs& a, cudaStream_t s) {
  static SmemOptIn opt;
  cudaError_t e = opt.ensure(delta_out_kernel<TW>, static_cast<int>(2 * out_stage(16 * TW)));
  if (e != cudaSuccess) return e;
  return launch_pdl(delta_out_kernel<TW>, dim3(a.NC, a.H), dim3(kThreads), 2 * out_stage(a.dv), s, a);
}

}  // namespace

bool delta_chunk_supported(int dk, int dv) {
  const int ks = dk / 16;        // the state kernel is compiled for these numbers of row blocks
  return dk % 16 == 0 && dv % 16 == 0 && dv >= 16 && dv <= 256 && ((ks >= 1 && ks <= 6) || ks == 8 || ks == 12 || ks == 16);
}

cudaError_t launch_delta_chunk(const DeltaArgs& a, cudaStream_t s) {
  if (a.is_f32 || !delta_chunk_supported(a.dk, a.dv) || a.cu == nullptr || a.trans == nullptr) return cudaErrorInvalidValue;
  if (a.T == 0 || a.N == 0) return cudaSuccess;
  cudaError_t e = launch_delta_prepare(a, true, s);
  if (e == cudaSuccess) e = launch_delta_keep(a, s);
  if (e != cudaSuccess) return e;
  static SmemOptIn opt;
  e = opt.ensure(delta_local_kernel, 227 * 1024);
  if (e != cudaSuccess) return e;
  e = launch_pdl(delta_local_kernel, dim3(a.NC, a.H), dim3(kThreads), local_smem(a.dk), s, a);
  if (e != cudaSuccess) return e;
  // every CTA of a head reads the same operands: narrow column tiles only while they still fit one wave
  int dev = 0, sms = 0;
  cudaGetDevice(&dev);
  cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev);
  e = static_cast<int64_t>(a.N) * a.H * ((a.dv + 15) / 16) <= sms ? launch_state_nt<2>(a, s) : launch_state_nt<4>(a, s);
  if (e != cudaSuccess) return e;
  if (a.dv <= 64) return launch_out<4>(a, s);
  if (a.dv <= 128) return launch_out<8>(a, s);
  return launch_out<16>(a, s);
}

}  // namespace tdb
