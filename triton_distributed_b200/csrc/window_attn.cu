// Attention over a sliding window with sigmoid weights or as the difference of two softmax maps (tdb/window.h): the simple form and
// the decode form.
//
//   window_simple_kernel   fp32 arithmetic, one warp per (token, head), any head dim up to 1024, fp32 or bf16 tensors: the 32-bit path,
//                          sizes beyond the tensor-core kernels, and the check of those
//   window_decode_kernel   bf16, one token per sequence, split-KV on mma.sync: the 16 rows of a tile are query heads of one key head.
//                          Two maps take rows of their own over the concatenated key [map 1 | map 2], each with zeros in the other's
//                          part, so that both maps are one tile against one pass over the keys and values; a thread then holds both
//                          maps of a head.  The last CTA of a (sequence, key head) merges the splits and finishes the heads.
#include "tdb/attn_device.cuh"
#include "tdb/launch.cuh"
#include "tdb/vec.cuh"
#include "tdb/window.h"

namespace tdb {

namespace {

using namespace attn;

constexpr int kSimpleMaxD = 1024;

TDB_DEVICE float gate_logit(const __nv_bfloat16* g, int64_t at) { return __bfloat162float(g[at]); }
TDB_DEVICE float gate_logit(const float* g, int64_t at) { return g[at]; }

// ---------------------------------------------------------------------------------------------------- simple form
template <typename T, int KP, int MAPS>     // KP elements of a row per lane
__global__ void __launch_bounds__(128) window_simple_kernel(const WindowAttnArgs p) {
  pdl_wait();
  pdl_launch_dependents();
  const int64_t wid = static_cast<int64_t>(blockIdx.x) * 4 + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (wid >= p.T * p.H) return;
  const int64_t t = wid / p.H;
  const int h = static_cast<int>(wid - t * p.H), g = h / (p.H / p.G);
  float qf[MAPS][KP], o[MAPS][KP], m[MAPS], l[MAPS];
#pragma unroll
  for (int a = 0; a < MAPS; ++a) {
    const T* q = reinterpret_cast<const T*>(p.q) + (wid * MAPS + a) * p.dk;
    m[a] = -INFINITY;
    l[a] = 0.f;
#pragma unroll
    for (int i = 0; i < KP; ++i) {
      const int d = lane + 32 * i;
      qf[a][i] = d < p.dk ? to_f32(q[d]) : 0.f;
      o[a][i] = 0.f;
    }
  }
  const int64_t row0 = p.row0[t];
  const int n = p.n_keys[t], newest = p.newest[t];
  for (int j = 0; j < n; ++j) {
    const int64_t row = row0 + j;
    float vf[KP];
    const T* vr = reinterpret_cast<const T*>(p.v) + (row * p.G + g) * p.dv;
#pragma unroll
    for (int i = 0; i < KP; ++i) {
      const int d = lane + 32 * i;
      vf[i] = d < p.dv ? to_f32(vr[d]) : 0.f;
    }
#pragma unroll
    for (int a = 0; a < MAPS; ++a) {
      const T* kr = reinterpret_cast<const T*>(p.k) + ((row * p.G + g) * MAPS + a) * p.dk;
      float s = 0.f;
#pragma unroll
      for (int i = 0; i < KP; ++i) {
        const int d = lane + 32 * i;
        s = fmaf(qf[a][i], d < p.dk ? to_f32(kr[d]) : 0.f, s);
      }
      s = warp_sum(s) * p.scale;
      if (MAPS == 1) {
        const int dist = newest - j + (newest < j ? n : 0);
        const float w = sigmoid_f32(s + p.bias[h * p.bias_n + min(static_cast<int64_t>(dist), p.bias_n - 1)]);
#pragma unroll
        for (int i = 0; i < KP; ++i) o[a][i] = fmaf(w, vf[i], o[a][i]);
      } else {
        const float mn = fmaxf(m[a], s), corr = expf(m[a] - mn), e = expf(s - mn);     // m = -inf -> 0
        l[a] = l[a] * corr + e;
        m[a] = mn;
#pragma unroll
        for (int i = 0; i < KP; ++i) o[a][i] = fmaf(e, vf[i], o[a][i] * corr);
      }
    }
  }
  float f = 1.f;
  if (MAPS == 2) {
    const float i0 = l[0] > 0.f ? 1.f / l[0] : 0.f, i1 = l[MAPS - 1] > 0.f ? p.lambda / l[MAPS - 1] : 0.f;
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < KP; ++i) {
      o[0][i] = o[0][i] * i0 - o[MAPS - 1][i] * i1;
      ss += o[0][i] * o[0][i];
    }
    f = p.out_scale / sqrtf(warp_sum(ss) / p.dv_real + p.eps);
  }
  if (p.gate != nullptr) f *= sigmoid_f32(gate_logit(reinterpret_cast<const T*>(p.gate), t * p.ld_gate + h));
  T* out = reinterpret_cast<T*>(p.out) + wid * p.dv;
#pragma unroll
  for (int i = 0; i < KP; ++i) {
    const int d = lane + 32 * i;
    if (d < p.dv) out[d] = from_f32<T>(o[0][i] * f);
  }
}

template <typename T, int MAPS>
cudaError_t launch_simple(const WindowAttnArgs& a, cudaStream_t s) {
  const dim3 grid(static_cast<unsigned>((a.T * a.H + 3) / 4));
  const int d = a.dk > a.dv ? a.dk : a.dv;
  return d <= 64    ? launch_pdl(window_simple_kernel<T, 2, MAPS>, grid, dim3(128), 0, s, a)
         : d <= 256 ? launch_pdl(window_simple_kernel<T, 8, MAPS>, grid, dim3(128), 0, s, a)
                    : launch_pdl(window_simple_kernel<T, kSimpleMaxD / 32, MAPS>, grid, dim3(128), 0, s, a);
}

// ---------------------------------------------------------------------------------------------------- decode form
template <int DK, int DV>       // DK: elements of all maps of a key
struct DecTiles {
  static constexpr int kPitchK = DK * 2 + 16, kPitchV = DV * 2 + 16;
  static constexpr int kK = kBlockN * kPitchK, kStage = kK + kBlockN * kPitchV;
  static constexpr int kRed = 4 * 16 * DV * 4 + 2 * 64 * 4;     // merge of the four warps
  static constexpr int kStages = 4 * kStage <= 112 * 1024 ? 4 : 2;
  static constexpr int kSmem = kStages * kStage > kRed ? kStages * kStage : kRed;
};

template <int DK, int DV, int MAPS>
__global__ void __launch_bounds__(kAttnThreads) window_decode_kernel(const WindowAttnArgs p) {
  extern __shared__ __align__(16) uint8_t smem[];
  using L = DecTiles<DK, DV>;
  constexpr int S = L::kStages, kHeads = 16 / MAPS, kMapK = DK / MAPS;
  constexpr bool kSoft = MAPS == 2;
  __shared__ int s_last;
  const int group = p.H / p.G, chunks = (group + kHeads - 1) / kHeads;
  const int split = blockIdx.x, g = blockIdx.y / chunks, hc = blockIdx.y - g * chunks, b = blockIdx.z;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, lr = lane >> 2, c2 = 2 * (lane & 3);
  pdl_wait();
  pdl_launch_dependents();
  const int64_t pos = p.pos[b], row0 = static_cast<int64_t>(p.slots[b]) * p.ring;
  const int n = static_cast<int>(min(pos + 1, static_cast<int64_t>(p.ring))), newest = static_cast<int>(pos % p.ring);
  const int total = (n + kBlockN - 1) / kBlockN, per = (total + p.splits - 1) / p.splits;
  const int blk0 = min(total, split * per), nblk = min(total, blk0 + per) - blk0;
  const __nv_bfloat16* kc = reinterpret_cast<const __nv_bfloat16*>(p.k) + g * DK;
  const __nv_bfloat16* vc = reinterpret_cast<const __nv_bfloat16*>(p.v) + g * DV;
  const int64_t ldk = static_cast<int64_t>(p.G) * DK, ldv = static_cast<int64_t>(p.G) * DV;
  auto load = [&](int i) {
    uint8_t* sk = smem + (i % S) * L::kStage;
    uint8_t* sv = sk + L::kK;
    const int t0 = (blk0 + i) * kBlockN;
    for (int c = threadIdx.x; c < kBlockN * (DK / 8); c += kAttnThreads) {
      const int r = c / (DK / 8), ch = c - r * (DK / 8);
      const bool ok = t0 + r < n;
      cp_async16(sk + r * L::kPitchK + ch * 16, kc + (ok ? (row0 + t0 + r) * ldk : 0) + ch * 8, ok);
    }
    for (int c = threadIdx.x; c < kBlockN * (DV / 8); c += kAttnThreads) {
      const int r = c / (DV / 8), ch = c - r * (DV / 8);
      const bool ok = t0 + r < n;
      cp_async16(sv + r * L::kPitchV + ch * 16, vc + (ok ? (row0 + t0 + r) * ldv : 0) + ch * 8, ok);
    }
  };
  // query fragments: row lr and row lr + 8; with two maps these are the maps of one head
  const int h_lo = hc * kHeads + lr, h_hi = MAPS == 2 ? h_lo : h_lo + 8;
  const bool ok_lo = h_lo < group, ok_hi = h_hi < group;
  const __nv_bfloat16* q = reinterpret_cast<const __nv_bfloat16*>(p.q) + (static_cast<int64_t>(b) * p.H + g * group) * DK;
  uint32_t qf[DK / 16][4];
#pragma unroll
  for (int ks = 0; ks < DK / 16; ++ks) {
    const bool lo = ok_lo && (MAPS == 1 || 16 * ks < kMapK), hi = ok_hi && (MAPS == 1 || 16 * ks >= kMapK);
    const __nv_bfloat16* ql = q + static_cast<int64_t>(h_lo) * DK + 16 * ks + c2;
    const __nv_bfloat16* qh = q + static_cast<int64_t>(h_hi) * DK + 16 * ks + c2;
    qf[ks][0] = lo ? *reinterpret_cast<const uint32_t*>(ql) : 0u;
    qf[ks][1] = hi ? *reinterpret_cast<const uint32_t*>(qh) : 0u;
    qf[ks][2] = lo ? *reinterpret_cast<const uint32_t*>(ql + 8) : 0u;
    qf[ks][3] = hi ? *reinterpret_cast<const uint32_t*>(qh + 8) : 0u;
  }
  const float* bias_lo = p.bias + static_cast<int64_t>(g * group + min(h_lo, group - 1)) * p.bias_n;
  const float* bias_hi = p.bias + static_cast<int64_t>(g * group + min(h_hi, group - 1)) * p.bias_n;
  float o[DV / 8][4];
#pragma unroll
  for (int i = 0; i < DV / 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
#pragma unroll
  for (int j = 0; j < S - 1; ++j) {
    if (j < nblk) load(j);
    cp_async_commit();
  }
  const bool upper = group - hc * kHeads > 8;            // rows 8-15 hold heads (sigmoid form)
  for (int i = 0; i < nblk; ++i) {
    if (i + S - 1 < nblk) load(i + S - 1);
    cp_async_commit();
    const int tb = warp * 16, t0 = (blk0 + i) * kBlockN + tb;      // each warp takes 16 of the 64 tokens
    float bias[2][4];                                    // on its way while the block arrives
    if constexpr (!kSoft) {
#pragma unroll
      for (int j = 0; j < 2; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int tok = t0 + 8 * j + c2 + (e & 1);
          const int dist = newest - tok + (newest < tok ? p.ring : 0);
          bias[j][e] = tok < n && (e < 2 || upper) ? __ldg((e < 2 ? bias_lo : bias_hi) + min(static_cast<int64_t>(dist), p.bias_n - 1)) : 0.f;
        }
    }
    cp_async_wait<S - 1>();
    __syncthreads();
    const uint8_t* sk = smem + (i % S) * L::kStage;
    const uint8_t* sv = sk + L::kK;
    float s[2][4];
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      s[j][0] = s[j][1] = s[j][2] = s[j][3] = 0.f;
      const uint8_t* kr = sk + (tb + 8 * j + lr) * L::kPitchK;
#pragma unroll
      for (int ks = 0; ks < DK / 16; ++ks)
        mma_bf16(s[j], qf[ks], *reinterpret_cast<const uint32_t*>(kr + (16 * ks + c2) * 2), *reinterpret_cast<const uint32_t*>(kr + (16 * ks + 8 + c2) * 2));
    }
    if constexpr (kSoft) {
      float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
      for (int j = 0; j < 2; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          s[j][e] = t0 + 8 * j + c2 + (e & 1) < n ? s[j][e] * (p.scale * kLog2e) : -INFINITY;
          mx[e >> 1] = fmaxf(mx[e >> 1], s[j][e]);
        }
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 1));
        mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 2));
        const float mn = fmaxf(m[r], mx[r]), base = mn == -INFINITY ? 0.f : mn, corr = exp2f(m[r] - base);
        m[r] = mn;
        l[r] *= corr;
#pragma unroll
        for (int d = 0; d < DV / 8; ++d) {
          o[d][2 * r] *= corr;
          o[d][2 * r + 1] *= corr;
        }
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
          for (int e = 2 * r; e < 2 * r + 2; ++e) {
            s[j][e] = exp2f(s[j][e] - base);
            l[r] += s[j][e];
          }
      }
    } else {
#pragma unroll
      for (int j = 0; j < 2; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float y = fmaf(s[j][e], p.scale, bias[j][e]);
          s[j][e] = t0 + 8 * j + c2 + (e & 1) < n && (e < 2 || upper) ? __fdividef(1.f, 1.f + exp2f(fminf(-y * kLog2e, 100.f))) : 0.f;
        }
    }
    uint32_t pa[4];
    pa[0] = pack_bf16x2(s[0][0], s[0][1]);
    pa[1] = pack_bf16x2(s[0][2], s[0][3]);
    pa[2] = pack_bf16x2(s[1][0], s[1][1]);
    pa[3] = pack_bf16x2(s[1][2], s[1][3]);
    const int mat = lane >> 3, row = lane & 7;
    const uint8_t* vb0 = sv + (tb + (mat & 1) * 8 + row) * L::kPitchV + (mat >> 1) * 16;
#pragma unroll
    for (int d = 0; d < DV / 8; d += 2) {
      uint32_t vb[4];
      ldmatrix_x4_trans(vb, vb0 + d * 16);
      mma_bf16(o[d], pa, vb[0], vb[1]);
      mma_bf16(o[d + 1], pa, vb[2], vb[3]);
    }
    __syncthreads();
  }
  // merge of the four warps: the same rows, other tokens
  float* red_o = reinterpret_cast<float*>(smem);          // [4 warps][16 rows][DV]
  float* red_m = red_o + 4 * 16 * DV;                     // [4][16] maxima (log2 domain), sums
  float* red_l = red_m + 64;
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    const int row = lr + 8 * r;
    l[r] += __shfl_xor_sync(0xffffffffu, l[r], 1);
    l[r] += __shfl_xor_sync(0xffffffffu, l[r], 2);
#pragma unroll
    for (int d = 0; d < DV / 8; ++d)
      *reinterpret_cast<float2*>(red_o + (warp * 16 + row) * DV + 8 * d + c2) = make_float2(o[d][2 * r], o[d][2 * r + 1]);
    if ((lane & 3) == 0) {
      red_m[warp * 16 + row] = m[r];
      red_l[warp * 16 + row] = l[r];
    }
  }
  __syncthreads();
  // thread t: row t / 8, columns (t % 8) * 4 + 32 k
  constexpr int kCols = DV / 32;
  const int row = threadIdx.x >> 3, sl = threadIdx.x & 7;
  const int64_t unit = (static_cast<int64_t>(b) * p.G + g) * chunks + hc;
  float4* part = reinterpret_cast<float4*>(p.workspace) + ((unit * p.splits) * 16 + row) * (DV / 4) + sl;      // + split * 16 * DV / 4
  float2* part_ml = reinterpret_cast<float2*>(p.workspace + static_cast<int64_t>(gridDim.z) * gridDim.y * p.splits * 16 * DV) + unit * p.splits * 16 + row;
  float4 acc[kCols];
  float mm = -INFINITY, ll = 0.f;
  {
    float w[4] = {1.f, 1.f, 1.f, 1.f};
    if (kSoft) {
#pragma unroll
      for (int i = 0; i < 4; ++i) mm = fmaxf(mm, red_m[i * 16 + row]);
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        w[i] = mm == -INFINITY ? 0.f : exp2f(red_m[i * 16 + row] - mm);
        ll += red_l[i * 16 + row] * w[i];
      }
    }
#pragma unroll
    for (int k = 0; k < kCols; ++k) {
      acc[k] = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const float4 v = *reinterpret_cast<const float4*>(red_o + (i * 16 + row) * DV + sl * 4 + 32 * k);
        acc[k].x = fmaf(w[i], v.x, acc[k].x); acc[k].y = fmaf(w[i], v.y, acc[k].y);
        acc[k].z = fmaf(w[i], v.z, acc[k].z); acc[k].w = fmaf(w[i], v.w, acc[k].w);
      }
    }
  }
  if (p.splits > 1) {
#pragma unroll
    for (int k = 0; k < kCols; ++k) __stcg(part + static_cast<int64_t>(split) * 16 * (DV / 4) + 8 * k, acc[k]);
    if (sl == 0) __stcg(part_ml + split * 16, make_float2(mm, ll));
    __threadfence();
    __syncthreads();
    if (threadIdx.x == 0) {
      const uint32_t prev = atomicAdd(p.counters + unit, 1u);
      s_last = prev == static_cast<uint32_t>(p.splits) - 1;
      if (s_last) p.counters[unit] = 0;      // clean for the next call
    }
    __syncthreads();
    if (!s_last) return;
    __threadfence();
    float mt = -INFINITY;
    if (kSoft)
      for (int i = 0; i < p.splits; ++i) mt = fmaxf(mt, __ldcg(part_ml + i * 16).x);
    ll = 0.f;
#pragma unroll
    for (int k = 0; k < kCols; ++k) acc[k] = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 4
    for (int i = 0; i < p.splits; ++i) {
      float w = 1.f;
      if (kSoft) {
        const float2 ml = __ldcg(part_ml + i * 16);
        w = mt == -INFINITY ? 0.f : exp2f(ml.x - mt);
        ll = fmaf(ml.y, w, ll);
      }
#pragma unroll
      for (int k = 0; k < kCols; ++k) {
        const float4 v = __ldcg(part + static_cast<int64_t>(i) * 16 * (DV / 4) + 8 * k);
        acc[k].x = fmaf(w, v.x, acc[k].x); acc[k].y = fmaf(w, v.y, acc[k].y);
        acc[k].z = fmaf(w, v.z, acc[k].z); acc[k].w = fmaf(w, v.w, acc[k].w);
      }
    }
  }
  float f = 1.f;
  const int h = hc * kHeads + row % kHeads, head = g * group + h;
  bool write = h < group;
  if (kSoft) {
    // rows 8-15 hold the second map of the heads of rows 0-7
    __syncthreads();
    const float inv = ll > 0.f ? 1.f / ll : 0.f;
    if (row >= 8) {
#pragma unroll
      for (int k = 0; k < kCols; ++k)
        *reinterpret_cast<float4*>(red_o + (row - 8) * DV + sl * 4 + 32 * k) =
            make_float4(acc[k].x * inv * p.lambda, acc[k].y * inv * p.lambda, acc[k].z * inv * p.lambda, acc[k].w * inv * p.lambda);
    }
    __syncthreads();
    float ss = 0.f;
    if (row < 8) {
#pragma unroll
      for (int k = 0; k < kCols; ++k) {
        const float4 v = *reinterpret_cast<const float4*>(red_o + row * DV + sl * 4 + 32 * k);
        acc[k].x = fmaf(acc[k].x, inv, -v.x); acc[k].y = fmaf(acc[k].y, inv, -v.y);
        acc[k].z = fmaf(acc[k].z, inv, -v.z); acc[k].w = fmaf(acc[k].w, inv, -v.w);
        ss += acc[k].x * acc[k].x + acc[k].y * acc[k].y + acc[k].z * acc[k].z + acc[k].w * acc[k].w;
      }
    }
#pragma unroll
    for (int x = 1; x < 8; x *= 2) ss += __shfl_xor_sync(0xffffffffu, ss, x);
    f = p.out_scale / sqrtf(ss / p.dv_real + p.eps);
    write = write && row < 8;
  }
  if (!write) return;
  if (p.gate != nullptr) f *= sigmoid_f32(gate_logit(reinterpret_cast<const __nv_bfloat16*>(p.gate), b * p.ld_gate + head));
  __nv_bfloat16* out = reinterpret_cast<__nv_bfloat16*>(p.out) + (static_cast<int64_t>(b) * p.H + head) * DV + sl * 4;
#pragma unroll
  for (int k = 0; k < kCols; ++k)
    *reinterpret_cast<uint2*>(out + 32 * k) = make_uint2(pack_bf16x2(acc[k].x * f, acc[k].y * f), pack_bf16x2(acc[k].z * f, acc[k].w * f));
}

template <int DK, int DV, int MAPS>
cudaError_t launch_decode(const WindowAttnArgs& a, int chunks, cudaStream_t s) {
  static SmemOptIn opt;
  constexpr int smem = DecTiles<DK, DV>::kSmem;
  cudaError_t e = opt.ensure(window_decode_kernel<DK, DV, MAPS>, smem);
  if (e != cudaSuccess) return e;
  return launch_pdl(window_decode_kernel<DK, DV, MAPS>, dim3(a.splits, a.G * chunks, static_cast<unsigned>(a.T)), dim3(kAttnThreads), smem, s, a);
}

bool common_ok(const WindowAttnArgs& a) {
  return a.H >= 1 && a.G >= 1 && a.H % a.G == 0 && a.dk >= 1 && a.dv >= 1 && (a.bias != nullptr ? a.maps == 1 && a.bias_n >= 1 : a.maps == 2 && a.dv_real >= 1);
}

}  // namespace

int window_head_chunks(int H, int G, int maps) { return (H / G + 16 / maps - 1) / (16 / maps); }

int64_t window_decode_workspace(int64_t T, int G, int chunks, int splits, int dv) {
  return splits > 1 ? T * G * chunks * splits * 16 * (static_cast<int64_t>(dv) + 2) : 0;
}

cudaError_t launch_window_simple(const WindowAttnArgs& a, cudaStream_t s) {
  if (!common_ok(a) || a.dk > kSimpleMaxD || a.dv > kSimpleMaxD || a.row0 == nullptr || a.n_keys == nullptr || a.newest == nullptr) return cudaErrorInvalidValue;
  if (a.T == 0) return cudaSuccess;
  if (a.is_f32) return a.maps == 1 ? launch_simple<float, 1>(a, s) : launch_simple<float, 2>(a, s);
  return a.maps == 1 ? launch_simple<__nv_bfloat16, 1>(a, s) : launch_simple<__nv_bfloat16, 2>(a, s);
}

cudaError_t launch_window_decode(const WindowAttnArgs& a, cudaStream_t s) {
  if (!common_ok(a) || a.is_f32 || a.ring < 1 || a.splits < 1 || a.slots == nullptr || a.pos == nullptr ||
      (a.splits > 1 && (a.workspace == nullptr || a.counters == nullptr)) || a.T > 65535)
    return cudaErrorInvalidValue;
  if (a.T == 0) return cudaSuccess;
  const int chunks = window_head_chunks(a.H, a.G, a.maps);
  if (static_cast<int64_t>(a.G) * chunks > 65535) return cudaErrorInvalidValue;
  if (a.dk == 64 && a.dv == 64) return a.maps == 1 ? launch_decode<64, 64, 1>(a, chunks, s) : launch_decode<128, 64, 2>(a, chunks, s);
  if (a.dk == 64 && a.dv == 128) return a.maps == 1 ? launch_decode<64, 128, 1>(a, chunks, s) : launch_decode<128, 128, 2>(a, chunks, s);
  if (a.dk == 128 && a.dv == 64) return a.maps == 1 ? launch_decode<128, 64, 1>(a, chunks, s) : launch_decode<256, 64, 2>(a, chunks, s);
  if (a.dk == 128 && a.dv == 128) return a.maps == 1 ? launch_decode<128, 128, 1>(a, chunks, s) : launch_decode<256, 128, 2>(a, chunks, s);
  return cudaErrorInvalidValue;
}

}  // namespace tdb
