// Narrow linear layers (a few to a few hundred output columns) with fp32 outputs, and the router built on one of them.
//
//   out[T, N] = x[T, K] * w[N, K]^T      bf16 or fp32 operands, fp32 accumulation and output
//
// A CTA owns 16 tokens x 8 NT columns; its warps split K (interleaved 32-element blocks) and are summed through shared
// memory.  The bf16 form runs on mma.sync.m16n8k16 with the K positions assigned to fragment slots in the order 16-byte
// loads deliver them, so both operands stream straight from global memory (the x tile is re-read from L2 per column tile).
//
// Router mode: the last column CTA of a 16-token tile to arrive reads the tile's logits back and does the selection, one
// warp per token: scores sigmoid(z) or softmax(z), the `top` largest choice scores (score + correction, inside the best
// groups; ties to the lower index) with their scores as weights, not renormalised, and sigmoid of the extra column that gates
// a shared expert.  One launch from activations to routing; from 2048 tokens on, where the selection wants more warps than the
// projection has CTAs, two.
#include "tdb/attn_device.cuh"
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
#pragma unroll(NT == 1 ? 8 : 4)
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

// Bit pattern that orders like the float (negative ones too), never 0 for a number.
TDB_DEVICE uint32_t order_key(float v) {
  const uint32_t b = __float_as_uint(v);
  return (b & 0x80000000u) != 0u ? ~b : b | 0x80000000u;
}

// Index of the largest key of the warp, ties to the lower index; lane l holds the keys l, l + 32, ...
template <int PER>
TDB_DEVICE uint32_t best_of(const uint32_t (&key)[PER]) {
  uint32_t best = 0u, mine = 0xffffffffu;
#pragma unroll
  for (int i = 0; i < PER; ++i) best = max(best, key[i]);
  best = __reduce_max_sync(0xffffffffu, best);
#pragma unroll
  for (int i = PER - 1; i >= 0; --i)
    if (key[i] == best) mine = (threadIdx.x & 31) + 32 * i;
  return __reduce_min_sync(0xffffffffu, mine);
}

// Selection of one token by one warp; PER = experts per lane.
template <int PER>
TDB_DEVICE void select_token(const NarrowLinearArgs& p, int64_t t) {
  const int lane = threadIdx.x & 31;
  const float* z = p.out + t * p.N;
  float score[PER];
  uint32_t key[PER];       // orders like the choice score; 0 = not a candidate
  if (p.softmax) {
    float m = -INFINITY, l = 0.f;
#pragma unroll
    for (int i = 0; i < PER; ++i) {
      score[i] = lane + 32 * i < p.E ? __ldcg(z + lane + 32 * i) : -INFINITY;
      m = fmaxf(m, score[i]);
    }
    m = warp_max(m);
#pragma unroll
    for (int i = 0; i < PER; ++i) {
      score[i] = expf(score[i] - m);
      l += score[i];
    }
    l = warp_sum(l);
#pragma unroll
    for (int i = 0; i < PER; ++i) score[i] /= l;
  } else {
#pragma unroll
    for (int i = 0; i < PER; ++i) score[i] = lane + 32 * i < p.E ? sigmoid_f32(__ldcg(z + lane + 32 * i)) : 0.f;
  }
#pragma unroll
  for (int i = 0; i < PER; ++i) {
    const int e = lane + 32 * i;
    key[i] = e < p.E ? order_key(score[i] + (p.correction != nullptr ? p.correction[e] : 0.f)) : 0u;
  }
  if (p.groups > 0 && p.keep < p.groups) {
    // the group of the best expert outside the groups found so far is the next best group
    const int size = p.E / p.groups;
    uint32_t open[PER];
#pragma unroll
    for (int i = 0; i < PER; ++i) open[i] = key[i];
    for (int j = 0; j < p.keep; ++j) {
      const int grp = static_cast<int>(best_of<PER>(open)) / size;
#pragma unroll
      for (int i = 0; i < PER; ++i)
        if ((lane + 32 * i) / size == grp) open[i] = 0u;
    }
#pragma unroll
    for (int i = 0; i < PER; ++i)
      if (open[i] != 0u) key[i] = 0u;
  }
  float my_w = 0.f;
  int my_id = 0;
  for (int j = 0; j < p.top; ++j) {
    const uint32_t id = best_of<PER>(key);
    float w = 0.f;
#pragma unroll
    for (int i = 0; i < PER; ++i)
      if (lane + 32 * i == static_cast<int>(id)) {
        key[i] = 0u;
        w = score[i];
      }
    w = __shfl_sync(0xffffffffu, w, id & 31);
    if (lane == j) {
      my_w = w;
      my_id = static_cast<int>(id);
    }
  }
  if (lane < p.top) {
    p.ids[t * p.top + lane] = my_id;
    p.weights[t * p.top + lane] = my_w;
  }
  if (p.has_gate && lane == 0) p.gate[t] = sigmoid_f32(__ldcg(z + p.E));
}
TDB_DEVICE void select_any(const NarrowLinearArgs& p, int64_t t) {
  if (p.E <= 32) select_token<1>(p, t);
  else if (p.E <= 64) select_token<2>(p, t);
  else if (p.E <= 128) select_token<4>(p, t);
  else select_token<kMaxPerLane>(p, t);
}

// The selection as a launch of its own, one warp per token, after the many-token projection.
__global__ void __launch_bounds__(256) select_kernel(const NarrowLinearArgs p) {
  pdl_wait();
  pdl_launch_dependents();
  const int64_t t = static_cast<int64_t>(blockIdx.x) * 8 + (threadIdx.x >> 5);
  if (t < p.T) select_any(p, t);
}

// Counts this column CTA of token tile `tile` in; true for the last one, whose view of the others' outputs is then complete.
TDB_DEVICE bool columns_arrive_last(const NarrowLinearArgs& p, int tile, int* s_last) {
  __threadfence();
  __syncthreads();
  if (threadIdx.x == 0) {
    const uint32_t prev = atomicAdd(p.counters + tile, 1u);
    *s_last = prev == gridDim.x - 1;
    if (*s_last) p.counters[tile] = 0;      // every arrival has been counted: clean for the next call
  }
  __syncthreads();
  if (!*s_last) return false;
  __threadfence();
  return true;
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
  if (!columns_arrive_last(p, blockIdx.y, &s_last)) return;
  for (int i = threadIdx.x >> 5; i < kTok; i += WARPS)
    if (t0 + i < p.T) select_any(p, t0 + i);
}

// ---- many tokens: 64 tokens x up to 136 columns per CTA, both operands through shared memory (cp.async, two stages of 64
// elements of K), so that the weights are read once per 64 tokens and x once.  Each of the four warps owns 16 tokens.
constexpr int kWideTok = 64, kWideTiles = 17, kWideCols = 8 * kWideTiles, kWideK = 64;
constexpr int kWidePitch = kWideK + 32;     // elements: 16-byte reads of eight rows spread over all banks
constexpr int kWideStage = (kWideTok + kWideCols) * kWidePitch * 2;

__global__ void __launch_bounds__(128) narrow_linear_wide_kernel(const NarrowLinearArgs p, int cols_per_cta) {
  extern __shared__ __align__(16) uint8_t smem[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
  const int64_t t0 = static_cast<int64_t>(blockIdx.y) * kWideTok;
  const int n0 = blockIdx.x * cols_per_cta, nc = min(cols_per_cta, p.N - n0);
  const __nv_bfloat16* x = reinterpret_cast<const __nv_bfloat16*>(p.x);
  const __nv_bfloat16* w = reinterpret_cast<const __nv_bfloat16*>(p.w);
  pdl_wait();
  pdl_launch_dependents();
  auto load = [&](int slab) {
    __nv_bfloat16* xs = reinterpret_cast<__nv_bfloat16*>(smem + (slab & 1) * kWideStage);
    __nv_bfloat16* ws = xs + kWideTok * kWidePitch;
    const int k0 = slab * kWideK;
    for (int i = threadIdx.x; i < (kWideTok + nc) * (kWideK / 8); i += 128) {
      const int r = i / (kWideK / 8), k = k0 + (i % (kWideK / 8)) * 8;
      if (r < kWideTok) {
        const bool ok = k < p.K && t0 + r < p.T;
        attn::cp_async16(xs + r * kWidePitch + (k - k0), x + (ok ? (t0 + r) * p.ldx + k : 0), ok);
      } else {
        const bool ok = k < p.K;
        attn::cp_async16(ws + (r - kWideTok) * kWidePitch + (k - k0), w + (ok ? static_cast<int64_t>(n0 + r - kWideTok) * p.K + k : 0), ok);
      }
    }
    attn::cp_async_commit();
  };
  float c[kWideTiles][4];
#pragma unroll
  for (int i = 0; i < kWideTiles; ++i) c[i][0] = c[i][1] = c[i][2] = c[i][3] = 0.f;
  const int slabs = (p.K + kWideK - 1) / kWideK, tiles = (nc + 7) / 8;
  load(0);
  for (int s = 0; s < slabs; ++s) {
    if (s + 1 < slabs) {
      load(s + 1);
      attn::cp_async_wait<1>();
    } else {
      attn::cp_async_wait<0>();
    }
    __syncthreads();
    const __nv_bfloat16* xs = reinterpret_cast<const __nv_bfloat16*>(smem + (s & 1) * kWideStage);
    const __nv_bfloat16* ws = xs + kWideTok * kWidePitch;
#pragma unroll
    for (int kb = 0; kb < kWideK / 32; ++kb) {
      const uint4 al = *reinterpret_cast<const uint4*>(xs + (warp * 16 + g) * kWidePitch + kb * 32 + t * 8);
      const uint4 ah = *reinterpret_cast<const uint4*>(xs + (warp * 16 + g + 8) * kWidePitch + kb * 32 + t * 8);
#pragma unroll
      for (int i = 0; i < kWideTiles; ++i) {
        if (i < tiles) {     // columns of the last tile beyond nc hold stale data: their products are not stored
          const uint4 bv = *reinterpret_cast<const uint4*>(ws + (i * 8 + g) * kWidePitch + kb * 32 + t * 8);
          mma_16816(c[i], al.x, ah.x, al.y, ah.y, bv.x, bv.y);
          mma_16816(c[i], al.z, ah.z, al.w, ah.w, bv.z, bv.w);
        }
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < kWideTiles; ++i) {
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int64_t tok = t0 + warp * 16 + g + (e >> 1) * 8;
      const int col = i * 8 + 2 * t + (e & 1);
      if (tok < p.T && col < nc) p.out[tok * p.N + n0 + col] = c[i][e];
    }
  }
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
                    a.N != a.E + (a.has_gate ? 1 : 0) ||
                    (a.groups > 0 && (a.E % a.groups != 0 || a.keep < 1 || a.keep > a.groups || a.top > a.E / a.groups * a.keep))))
    return cudaErrorInvalidValue;
  if (a.T == 0) return cudaSuccess;
  // few tokens: as many CTAs and as much split K as the columns allow; many: wider column tiles re-read x less often
  if (a.is_f32) return launch_t<float, 1, 8>(a, s);
  if (a.T <= 64) return launch_t<__nv_bfloat16, 1, 8>(a, s);
  if (a.T >= 2048) {
    static SmemOptIn opt;
    cudaError_t e = opt.ensure(narrow_linear_wide_kernel, 2 * kWideStage);
    if (e != cudaSuccess) return e;
    const int tiles = (a.N + 7) / 8, groups = (tiles + kWideTiles - 1) / kWideTiles;
    const int cols = 8 * ((tiles + groups - 1) / groups);
    e = launch_pdl(narrow_linear_wide_kernel, dim3((a.N + cols - 1) / cols, static_cast<unsigned>((a.T + kWideTok - 1) / kWideTok)),
                      dim3(128), static_cast<size_t>(2 * kWideStage), s, a, cols);
    if (e != cudaSuccess || a.top < 1) return e;
    return launch_pdl(select_kernel, dim3(static_cast<unsigned>((a.T + 7) / 8)), dim3(256), 0, s, a);
  }
  return launch_t<__nv_bfloat16, 4, 4>(a, s);
}

}  // namespace tdb
