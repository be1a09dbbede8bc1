// Narrow linear layers (a few to a few hundred output columns) with fp32 outputs, and the router built on one of them.
//
//   out[T, N] = x[T, K] * w[N, K]^T      bf16 or fp32 operands, fp32 accumulation and output
//
// A CTA owns 16 tokens x 8 NT columns; its warps split K (interleaved 32-element blocks) and are summed through shared
// memory.  The bf16 form runs on mma.sync.m16n8k16 with the K positions assigned to fragment slots in the order 16-byte
// loads deliver them, so both operands stream straight from global memory (the x tile is re-read from L2 per column tile).
//
// Router mode: the last column CTA of a 16-token tile to arrive reads the tile's logits back and does the selection, one
// warp per token: scores sigmoid(z), the `top` largest (ties to the lower index) with their scores as weights, not
// renormalised, and sigmoid of the extra column that gates a shared expert.  One launch from activations to routing.
#include "tdb/hybrid.h"
#include "tdb/launch.cuh"
#include "tdb/vec.cuh"

namespace tdb {

namespace {

constexpr int kTok = 16;
constexpr int kMaxPerLane = 16;     // experts per lane in the selection: E <= 512

TDB_DEVICE void mma_16816(float (&c)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}

// Partial products of this warp's K blocks into part[16][8 NT].
template <int NT, int WARPS>
TDB_DEVICE void tile_partial(const NarrowLinearArgs& p, const __nv_bfloat16* x, const __nv_bfloat16* w, int64_t t0, int n0,
                             float* part) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
  const bool lo_ok = t0 + g < p.T, hi_ok = t0 + g + 8 < p.T;
  const __nv_bfloat16* xl = x + (lo_ok ? t0 + g : 0) * p.ldx;
  const __nv_bfloat16* xh = x + (hi_ok ? t0 + g + 8 : 0) * p.ldx;
  float c[NT][4];
#pragma unroll
  for (int i = 0; i < NT; ++i) c[i][0] = c[i][1] = c[i][2] = c[i][3] = 0.f;
  const uint4 zero = make_uint4(0u, 0u, 0u, 0u);
  const int nb = (p.K + 31) >> 5;
#pragma unroll 4
  for (int b = warp; b < nb; b += WARPS) {
    const int kk = b * 32 + t * 8;
    const bool ok = kk < p.K;
    const uint4 al = (ok && lo_ok) ? *reinterpret_cast<const uint4*>(xl + kk) : zero;
    const uint4 ah = (ok && hi_ok) ? *reinterpret_cast<const uint4*>(xh + kk) : zero;
#pragma unroll
    for (int i = 0; i < NT; ++i) {
      const int col = n0 + i * 8 + g;
      const uint4 bv = (ok && col < p.N) ? ld_nc_v4(w + static_cast<int64_t>(col) * p.K + kk) : zero;
      mma_16816(c[i], al.x, ah.x, al.y, ah.y, bv.x, bv.y);
      mma_16816(c[i], al.z, ah.z, al.w, ah.w, bv.z, bv.w);
    }
  }
#pragma unroll
  for (int i = 0; i < NT; ++i) {
    part[g * (8 * NT) + i * 8 + 2 * t] = c[i][0];
    part[g * (8 * NT) + i * 8 + 2 * t + 1] = c[i][1];
    part[(g + 8) * (8 * NT) + i * 8 + 2 * t] = c[i][2];
    part[(g + 8) * (8 * NT) + i * 8 + 2 * t + 1] = c[i][3];
  }
}
template <int NT, int WARPS>
TDB_DEVICE void tile_partial(const NarrowLinearArgs& p, const float* x, const float* w, int64_t t0, int n0, float* part) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  for (int i = 0; i < kTok * 8 * NT; ++i) {
    const int64_t tok = t0 + i / (8 * NT);
    const int col = n0 + i % (8 * NT);
    float s = 0.f;
    if (tok < p.T && col < p.N)
      for (int k = (warp * 32 + lane) * 8; k < p.K; k += WARPS * 256) {
        float a[8], b[8];
        load8(x + tok * p.ldx + k, a);
        load8(w + static_cast<int64_t>(col) * p.K + k, b);
#pragma unroll
        for (int j = 0; j < 8; ++j) s = fmaf(a[j], b[j], s);
      }
    s = warp_sum(s);
    if (lane == 0) part[i] = s;
  }
}

TDB_DEVICE void select_token(const NarrowLinearArgs& p, int64_t t) {
  const int lane = threadIdx.x & 31;
  const float* z = p.out + t * p.N;
  float v[kMaxPerLane];
#pragma unroll
  for (int i = 0; i < kMaxPerLane; ++i) {
    const int e = lane + 32 * i;
    v[i] = e < p.E ? sigmoid_f32(__ldcg(z + e)) : -1.f;    // scores are >= 0, -1 = not a candidate
  }
  float my_w = 0.f;
  int my_id = 0;
  for (int j = 0; j < p.top; ++j) {
    float best = -1.f;
    int bi = 0x7fffffff;
#pragma unroll
    for (int i = 0; i < kMaxPerLane; ++i)
      if (v[i] > best) {
        best = v[i];
        bi = lane + 32 * i;
      }
    for (int o = 16; o > 0; o >>= 1) {
      const float ob = __shfl_xor_sync(0xffffffffu, best, o);
      const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
      if (ob > best || (ob == best && oi < bi)) {
        best = ob;
        bi = oi;
      }
    }
#pragma unroll
    for (int i = 0; i < kMaxPerLane; ++i)
      if (lane + 32 * i == bi) v[i] = -1.f;
    if (lane == j) {
      my_w = best;
      my_id = bi;
    }
  }
  if (lane < p.top) {
    p.ids[t * p.top + lane] = my_id;
    p.weights[t * p.top + lane] = my_w;
  }
  if (p.has_gate && lane == 0) p.gate[t] = sigmoid_f32(__ldcg(z + p.E));
}

template <typename T, int NT, int WARPS>
__global__ void __launch_bounds__(WARPS * 32) narrow_linear_kernel(const NarrowLinearArgs p) {
  __shared__ float part[WARPS][kTok * 8 * NT];
  __shared__ int s_last;
  pdl_wait();
  pdl_launch_dependents();
  const int64_t t0 = static_cast<int64_t>(blockIdx.y) * kTok;
  const int n0 = blockIdx.x * 8 * NT;
  tile_partial<NT, WARPS>(p, reinterpret_cast<const T*>(p.x), reinterpret_cast<const T*>(p.w), t0, n0,
                          part[threadIdx.x >> 5]);
  __syncthreads();
  for (int i = threadIdx.x; i < kTok * 8 * NT; i += WARPS * 32) {
    const int64_t tok = t0 + i / (8 * NT);
    const int col = n0 + i % (8 * NT);
    float s = 0.f;
#pragma unroll
    for (int w = 0; w < WARPS; ++w) s += part[w][i];
    if (tok < p.T && col < p.N) p.out[tok * p.N + col] = s;
  }
  if (p.top < 1) return;
  __threadfence();
  __syncthreads();
  if (threadIdx.x == 0) {
    const uint32_t prev = atomicAdd(p.counters + blockIdx.y, 1u);
    s_last = prev == gridDim.x - 1;
    if (s_last) p.counters[blockIdx.y] = 0;      // every arrival has been counted: clean for the next call
  }
  __syncthreads();
  if (!s_last) return;
  __threadfence();
  for (int i = threadIdx.x >> 5; i < kTok; i += WARPS)
    if (t0 + i < p.T) select_token(p, t0 + i);
}

template <typename T, int NT, int WARPS>
cudaError_t launch_t(const NarrowLinearArgs& a, cudaStream_t s) {
  const dim3 grid((a.N + 8 * NT - 1) / (8 * NT), static_cast<unsigned>((a.T + kTok - 1) / kTok));
  return launch_pdl(narrow_linear_kernel<T, NT, WARPS>, grid, dim3(WARPS * 32), 0, s, a);
}

}  // namespace

cudaError_t launch_narrow_linear(const NarrowLinearArgs& a, cudaStream_t s) {
  if (a.K % 8 != 0 || a.ldx % 8 != 0 || a.N < 1) return cudaErrorInvalidValue;
  if ((a.T + kTok - 1) / kTok > 65535) return cudaErrorInvalidValue;
  if (a.top > 0 && (a.top > 32 || a.top > a.E || a.E > 32 * kMaxPerLane || a.counters == nullptr ||
                    a.N != a.E + (a.has_gate ? 1 : 0)))
    return cudaErrorInvalidValue;
  if (a.T == 0) return cudaSuccess;
  // few tokens: as many CTAs and as much split K as the columns allow; many: wider column tiles re-read x less often
  if (a.is_f32) return launch_t<float, 1, 8>(a, s);
  if (a.T <= 64) return launch_t<__nv_bfloat16, 1, 8>(a, s);
  return launch_t<__nv_bfloat16, 4, 4>(a, s);
}

}  // namespace tdb
