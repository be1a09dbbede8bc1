// Python bindings of the kernels in tdb/hybrid.h.
#include <ATen/cuda/CUDAContext.h>
#include <c10/cuda/CUDAGuard.h>
#include <torch/extension.h>

#include "tdb/delta.h"
#include "tdb/hybrid.h"
#include "tdb/latent.h"
#include "tdb/streams.h"

namespace py = pybind11;
using OptTensor = c10::optional<at::Tensor>;

namespace {

cudaStream_t cur_stream() { return at::cuda::getCurrentCUDAStream().stream(); }
void check_cuda(cudaError_t e, const char* what) { TORCH_CHECK(e == cudaSuccess, what, ": ", cudaGetErrorString(e)); }

// Activations / weights are fp32 or bf16; returns 1 for fp32.
int act_f32(const at::Tensor& t, const char* name) {
  TORCH_CHECK(t.is_cuda() && (t.scalar_type() == at::kFloat || t.scalar_type() == at::kBFloat16), name, ": fp32 or bf16 CUDA tensor");
  return t.scalar_type() == at::kFloat ? 1 : 0;
}
int act_f32_of(const at::Tensor& t) { return act_f32(t, "y"); }
void check_same(const at::Tensor& t, const at::Tensor& like, const char* name) {
  TORCH_CHECK(t.is_cuda() && t.scalar_type() == like.scalar_type() && t.is_contiguous(), name, ": contiguous CUDA tensor of the activation dtype");
}
float* f32(const at::Tensor& t, int64_t numel, const char* name) {
  TORCH_CHECK(t.is_cuda() && t.scalar_type() == at::kFloat && t.is_contiguous() && t.numel() >= numel, name,
              ": contiguous fp32 CUDA tensor of at least ", numel, " elements");
  return t.data_ptr<float>();
}
int32_t* i32(const at::Tensor& t, int64_t numel, const char* name) {
  TORCH_CHECK(t.is_cuda() && t.scalar_type() == at::kInt && t.is_contiguous() && t.numel() >= numel, name,
              ": contiguous int32 CUDA tensor of at least ", numel, " elements");
  return t.data_ptr<int32_t>();
}
int64_t* i64(const at::Tensor& t, int64_t numel, const char* name) {
  TORCH_CHECK(t.is_cuda() && t.scalar_type() == at::kLong && t.is_contiguous() && t.numel() >= numel, name,
              ": contiguous int64 CUDA tensor of at least ", numel, " elements");
  return t.data_ptr<int64_t>();
}

void embed_stream(const at::Tensor& ids, const at::Tensor& table, at::Tensor& x, const OptTensor& xb, double scale) {
  const int fp = act_f32(table, "table");
  TORCH_CHECK(table.dim() == 2 && table.is_contiguous(), "embed_stream: contiguous table [V, W]");
  const int64_t T = ids.numel(), W = table.size(1);
  c10::cuda::CUDAGuard guard(table.device());
  void* b = nullptr;
  if (!fp && xb.has_value()) {
    TORCH_CHECK(xb->numel() == T * W, "embed_stream: bf16 copy [T, W]");
    check_same(*xb, table, "xb");
    b = xb->data_ptr();
  }
  check_cuda(tdb::launch_embed_stream(i64(ids, T, "ids"), table.data_ptr(), f32(x, T * W, "x"), b, T, W, table.size(0), scale, fp, cur_stream()),
             "launch_embed_stream");
}

tdb::PostNormArgs post_args(const at::Tensor& y, int64_t T, int64_t W, int64_t rows, const OptTensor& shared, const OptTensor& gate) {
  tdb::PostNormArgs a = {};
  a.y_f32 = act_f32(y, "y");
  TORCH_CHECK(y.is_contiguous() && y.numel() == T * rows * W, "y: contiguous [T * rows, W]");
  a.y = y.data_ptr();
  a.rows_per_token = rows;
  if (shared.has_value()) {
    check_same(*shared, y, "shared");
    TORCH_CHECK(shared->numel() == T * W, "shared: [T, W]");
    a.shared = shared->data_ptr();
    if (gate.has_value()) a.shared_gate = f32(*gate, T, "shared_gate");
  }
  a.T = T;
  a.W = W;
  return a;
}

void postnorm_add(at::Tensor& x, const OptTensor& xb, const at::Tensor& y, const at::Tensor& w, int64_t rows, int64_t n_real,
                  double eps, const OptTensor& shared, const OptTensor& gate) {
  TORCH_CHECK(x.dim() == 2, "postnorm_add: x [T, W]");
  const int64_t T = x.size(0), W = x.size(1);
  c10::cuda::CUDAGuard guard(x.device());
  tdb::PostNormArgs a = post_args(y, T, W, rows, shared, gate);
  a.x = f32(x, T * W, "x");
  if (xb.has_value()) {
    TORCH_CHECK(xb->is_cuda() && xb->scalar_type() == at::kBFloat16 && xb->is_contiguous() && xb->numel() == T * W, "xb: bf16 [T, W]");
    a.xb = xb->data_ptr();
  }
  a.w = f32(w, W, "w");
  a.n_real = n_real;
  a.eps = eps;
  check_cuda(tdb::launch_postnorm_add(a, cur_stream()), "launch_postnorm_add");
}

// x += mix + (rows of y) + shared + bias and up to two norms of the new x: (h1, h2), empty where not asked for.  sum_only: the
// sum alone, fp32 [T, W].
std::vector<at::Tensor> parallel_add(at::Tensor& x, const OptTensor& mix, const OptTensor& y, int64_t rows, const OptTensor& ids,
                                     const OptTensor& weights, int64_t experts, const OptTensor& hin, const OptTensor& shared,
                                     const OptTensor& bias, const OptTensor& w1, const OptTensor& w2, int64_t n_real, double eps,
                                     bool act_f32, bool sum_only) {
  TORCH_CHECK(x.dim() == 2, "parallel_add: x [T, W]");
  const int64_t T = x.size(0), W = x.size(1);
  c10::cuda::CUDAGuard guard(x.device());
  tdb::ParallelAddArgs a = {};
  const auto act = x.options().dtype(act_f32 ? at::kFloat : at::kBFloat16);
  auto in = [&](const OptTensor& t, const char* name) -> const void* {
    if (!t.has_value()) return nullptr;
    TORCH_CHECK(t->is_cuda() && t->scalar_type() == act.dtype() && t->is_contiguous() && t->numel() == T * W, name,
                ": contiguous [T, W] of the activation dtype");
    return t->data_ptr();
  };
  a.x = f32(x, T * W, "x");
  a.mix = in(mix, "mix");
  a.shared = in(shared, "shared");
  a.hin = in(hin, "hin");
  a.rows = rows;
  if (y.has_value()) {
    a.y_f32 = act_f32_of(*y);
    TORCH_CHECK(y->is_contiguous() && y->numel() == T * rows * W, "y: contiguous [T * rows, W]");
    a.y = y->data_ptr();
  }
  if (ids.has_value()) {
    TORCH_CHECK(weights.has_value(), "parallel_add: weights missing");
    a.ids = i32(*ids, T * rows, "ids");
    a.weights = f32(*weights, T * rows, "weights");
    a.experts = experts;
  }
  if (bias.has_value()) a.bias = f32(*bias, W, "bias");
  a.act_f32 = act_f32 ? 1 : 0;
  a.T = T; a.W = W; a.n_real = n_real; a.eps = eps;
  std::vector<at::Tensor> out;
  if (sum_only) {
    out.push_back(at::empty({T, W}, x.options()));
    a.sum_out = out[0].data_ptr<float>();
  } else {
    if (w1.has_value()) {
      out.push_back(at::empty({T, W}, act));
      a.w1 = f32(*w1, W, "w1");
      a.h1 = out[0].data_ptr();
    }
    if (w2.has_value()) {
      TORCH_CHECK(w1.has_value(), "parallel_add: w2 without w1");
      out.push_back(at::empty({T, W}, act));
      a.w2 = f32(*w2, W, "w2");
      a.h2 = out[1].data_ptr();
    }
  }
  check_cuda(tdb::launch_parallel_add(a, cur_stream()), "launch_parallel_add");
  return out;
}

at::Tensor combine_rows(const at::Tensor& y, int64_t T, int64_t rows, const OptTensor& shared, const OptTensor& gate) {
  const int64_t W = y.size(-1);
  c10::cuda::CUDAGuard guard(y.device());
  tdb::PostNormArgs a = post_args(y, T, W, rows, shared, gate);
  at::Tensor out = at::empty({T, W}, y.options());
  check_cuda(tdb::launch_combine_rows(a, out.data_ptr(), cur_stream()), "launch_combine_rows");
  return out;
}

void stream_norm(const at::Tensor& x, const OptTensor& rows, const at::Tensor& w, at::Tensor& out, int64_t n_real, double eps) {
  const int fp = act_f32(out, "out");
  const int64_t W = x.size(-1), n = out.numel() / W;
  TORCH_CHECK(out.is_contiguous() && (rows.has_value() || n == x.numel() / W), "stream_norm: output shape");
  c10::cuda::CUDAGuard guard(x.device());
  check_cuda(tdb::launch_stream_norm(f32(x, 0, "x"), rows.has_value() ? i64(*rows, n, "rows") : nullptr, f32(w, W, "w"),
                                     out.data_ptr(), n, W, n_real, eps, fp, cur_stream()),
             "launch_stream_norm");
}

tdb::QkNormArgs qk_args(const at::Tensor& qk, int64_t Nq, int64_t Nk, int64_t nq_real, int64_t nk_real, double eps) {
  tdb::QkNormArgs a = {};
  a.is_f32 = act_f32(qk, "qk");
  TORCH_CHECK(qk.dim() == 2 && qk.stride(1) == 1 && qk.size(1) >= Nq + Nk, "qk: [T, >= Nq + Nk]");
  a.qk = qk.data_ptr();
  a.ld = qk.stride(0);
  a.T = qk.size(0);
  a.Nq = Nq; a.Nk = Nk;
  a.nq_real = nq_real; a.nk_real = nk_real;
  a.eps = eps;
  return a;
}

at::Tensor qk_norm_tied(const at::Tensor& qk, const at::Tensor& qw, int64_t Nk, int64_t nq_real, int64_t nk_real, double eps,
                        at::Tensor& k_a, at::Tensor& scale_a, const at::Tensor& rows_a, const OptTensor& k_b,
                        const OptTensor& scale_b, const OptTensor& rows_b, const OptTensor& sumsq) {
  const int64_t Nq = qw.numel();
  c10::cuda::CUDAGuard guard(qk.device());
  tdb::QkNormArgs a = qk_args(qk, Nq, Nk, nq_real, nk_real, eps);
  a.qw = f32(qw, Nq, "qw");
  at::Tensor q = at::empty({a.T, Nq}, qk.options());
  a.q_out = q.data_ptr();
  check_same(k_a, qk, "k_a");
  a.k_a = k_a.data_ptr();
  a.cap_a = k_a.numel() / Nk;
  a.scale_a = f32(scale_a, a.cap_a, "scale_a");
  a.rows_a = i64(rows_a, a.T, "rows_a");
  if (k_b.has_value()) {
    check_same(*k_b, qk, "k_b");
    a.k_b = k_b->data_ptr();
    a.cap_b = k_b->numel() / Nk;
    a.scale_b = f32(*scale_b, a.cap_b, "scale_b");
    a.rows_b = i64(*rows_b, a.T, "rows_b");
  }
  if (sumsq.has_value()) a.sumsq = f32(*sumsq, 2 * a.T, "sumsq");
  check_cuda(tdb::launch_qk_norm_tied(a, cur_stream()), "launch_qk_norm_tied");
  return q;
}

at::Tensor qk_sumsq(const at::Tensor& qk, int64_t Nq, int64_t Nk) {
  c10::cuda::CUDAGuard guard(qk.device());
  tdb::QkNormArgs a = qk_args(qk, Nq, Nk, 1, 1, 0.0);
  at::Tensor out = at::empty({a.T, 2}, qk.options().dtype(at::kFloat));
  check_cuda(tdb::launch_qk_sumsq(a, out.data_ptr<float>(), cur_stream()), "launch_qk_sumsq");
  return out;
}

tdb::NarrowLinearArgs narrow_args(const at::Tensor& x, const at::Tensor& w) {
  tdb::NarrowLinearArgs a = {};
  a.is_f32 = act_f32(x, "x");
  TORCH_CHECK(x.dim() == 2 && x.stride(1) == 1, "narrow_linear: x [T, K]");
  check_same(w, x, "w");
  TORCH_CHECK(w.dim() == 2 && w.size(1) == x.size(1), "narrow_linear: w [N, K]");
  a.x = x.data_ptr();
  a.ldx = x.stride(0);
  a.w = w.data_ptr();
  a.T = x.size(0);
  a.N = w.size(0);
  a.K = w.size(1);
  return a;
}

at::Tensor narrow_linear(const at::Tensor& x, const at::Tensor& w) {
  c10::cuda::CUDAGuard guard(x.device());
  tdb::NarrowLinearArgs a = narrow_args(x, w);
  at::Tensor out = at::empty({a.T, a.N}, x.options().dtype(at::kFloat));
  a.out = out.data_ptr<float>();
  check_cuda(tdb::launch_narrow_linear(a, cur_stream()), "launch_narrow_linear");
  return out;
}

// Returns (ids int32 [T, top], scores fp32 [T, top], gate fp32 [T] or empty).
std::vector<at::Tensor> sigmoid_router(const at::Tensor& x, const at::Tensor& w, int64_t top, bool has_gate, const at::Tensor& counters) {
  c10::cuda::CUDAGuard guard(x.device());
  tdb::NarrowLinearArgs a = narrow_args(x, w);
  auto fo = x.options().dtype(at::kFloat);
  at::Tensor z = at::empty({a.T, a.N}, fo);
  at::Tensor ids = at::empty({a.T, top}, x.options().dtype(at::kInt));
  at::Tensor wts = at::empty({a.T, top}, fo);
  at::Tensor gate = at::empty({has_gate ? a.T : 0}, fo);
  a.out = z.data_ptr<float>();
  a.top = top;
  a.has_gate = has_gate ? 1 : 0;
  a.E = a.N - a.has_gate;
  a.ids = ids.data_ptr<int32_t>();
  a.weights = wts.data_ptr<float>();
  a.gate = has_gate ? gate.data_ptr<float>() : nullptr;
  a.counters = reinterpret_cast<uint32_t*>(i32(counters, (a.T + 15) / 16, "counters"));
  check_cuda(tdb::launch_narrow_linear(a, cur_stream()), "launch_narrow_linear(router)");
  return {ids, wts, gate};
}

// softmax scores over all columns of w: returns (ids int32 [T, top], scores fp32 [T, top]).
std::vector<at::Tensor> softmax_router(const at::Tensor& x, const at::Tensor& w, const at::Tensor& correction, int64_t top, int64_t groups,
                                       int64_t keep, const at::Tensor& counters) {
  c10::cuda::CUDAGuard guard(x.device());
  tdb::NarrowLinearArgs a = narrow_args(x, w);
  auto fo = x.options().dtype(at::kFloat);
  at::Tensor z = at::empty({a.T, a.N}, fo);
  at::Tensor ids = at::empty({a.T, top}, x.options().dtype(at::kInt));
  at::Tensor wts = at::empty({a.T, top}, fo);
  a.out = z.data_ptr<float>();
  a.top = top;
  a.E = a.N;
  a.softmax = 1;
  a.correction = f32(correction, a.N, "correction");
  a.groups = groups;
  a.keep = keep;
  a.ids = ids.data_ptr<int32_t>();
  a.weights = wts.data_ptr<float>();
  a.counters = reinterpret_cast<uint32_t*>(i32(counters, (a.T + 15) / 16, "counters"));
  check_cuda(tdb::launch_narrow_linear(a, cur_stream()), "launch_narrow_linear(softmax router)");
  return {ids, wts};
}

at::Tensor relu2(const at::Tensor& in, const OptTensor& row_weight, const OptTensor& bias) {
  const int fp = act_f32(in, "in");
  TORCH_CHECK(in.dim() == 2 && in.is_contiguous(), "relu2: contiguous [rows, F]");
  c10::cuda::CUDAGuard guard(in.device());
  at::Tensor out = at::empty_like(in);
  const float* w = row_weight.has_value() ? f32(*row_weight, in.size(0), "row_weight") : nullptr;
  const float* b = bias.has_value() ? f32(*bias, in.size(1), "bias") : nullptr;
  check_cuda(tdb::launch_relu2(in.data_ptr(), w, b, out.data_ptr(), in.size(0), in.size(1), fp, cur_stream()), "launch_relu2");
  return out;
}

at::Tensor expert_gemv(const at::Tensor& x, const at::Tensor& up, const at::Tensor& down, const at::Tensor& ids, const at::Tensor& weights,
                       const OptTensor& shared_up, const OptTensor& shared_down, const OptTensor& shared_gate, bool gated, int64_t identity,
                       bool skip_identity) {
  tdb::ExpertGemvArgs a = {};
  a.is_f32 = act_f32(x, "x");
  TORCH_CHECK(x.dim() == 2 && x.is_contiguous() && up.dim() == 3 && down.dim() == 3, "expert_gemv: x [T, K], up [E, F, K], down [E, K, F]");
  check_same(up, x, "up");
  check_same(down, x, "down");
  a.gated = gated ? 1 : 0;
  a.identity = identity;
  a.skip_identity = skip_identity ? 1 : 0;
  const int64_t rows = gated ? 2 : 1;
  TORCH_CHECK(up.size(1) % rows == 0, "expert_gemv: gated weights come in pairs of rows");
  a.T = x.size(0); a.K = x.size(1); a.E = up.size(0); a.F = up.size(1) / rows;
  TORCH_CHECK(up.size(2) == a.K && down.size(0) == a.E && down.size(1) == a.K && down.size(2) == a.F, "expert_gemv: shape mismatch");
  TORCH_CHECK(ids.dim() == 2 && ids.size(0) == a.T, "expert_gemv: ids [T, top]");
  a.top = ids.size(1);
  a.ids = i32(ids, a.T * a.top, "ids");
  a.weights = f32(weights, a.T * a.top, "weights");
  if (shared_up.has_value()) {
    TORCH_CHECK(shared_down.has_value(), "expert_gemv: shared_down missing");
    check_same(*shared_up, x, "shared_up");
    check_same(*shared_down, x, "shared_down");
    a.Fs = shared_up->size(0) / rows;
    TORCH_CHECK(shared_up->size(1) == a.K && shared_down->size(0) == a.K && shared_down->size(1) == a.Fs && shared_up->size(0) == a.Fs * rows, "expert_gemv: shared shapes");
    a.shared_up = shared_up->data_ptr();
    a.shared_down = shared_down->data_ptr();
    if (shared_gate.has_value()) a.shared_gate = f32(*shared_gate, a.T, "shared_gate");
  }
  c10::cuda::CUDAGuard guard(x.device());
  a.x = x.data_ptr(); a.up = up.data_ptr(); a.down = down.data_ptr();
  at::Tensor act = at::empty({a.T, static_cast<int64_t>(a.top) * a.F + a.Fs}, x.options());
  at::Tensor y = at::empty({a.T, a.K}, x.options().dtype(at::kFloat));
  a.act = act.data_ptr();
  a.y = y.data_ptr<float>();
  check_cuda(tdb::launch_expert_gemv(a, cur_stream()), "launch_expert_gemv");
  return y;
}

// ---- latent attention
tdb::LatentPrepArgs latent_args(const at::Tensor& z, int64_t H, int64_t d, int64_t r, const OptTensor& norm_w, int64_t R, int64_t R_real,
                                double eps, const at::Tensor& cos_sin, const at::Tensor& pos, const OptTensor& cache, const OptTensor& rows,
                                const OptTensor& ctx, const OptTensor& ctx_rows) {
  tdb::LatentPrepArgs a = {};
  a.is_f32 = act_f32(z, "z");
  TORCH_CHECK(z.dim() == 2 && z.stride(1) == 1, "latent: z [T, columns]");
  a.z = z.data_ptr();
  a.ld = z.stride(0);
  a.T = z.size(0);
  a.H = H; a.d = d; a.r = r; a.R = R; a.R_real = R_real;
  a.eps = eps;
  a.n_pos = cos_sin.size(0);
  TORCH_CHECK(cos_sin.dim() == 2 && cos_sin.size(1) == r, "latent: cos_sin [positions, r]");
  a.cos_sin = f32(cos_sin, a.n_pos * r, "cos_sin");
  a.pos = i64(pos, a.T, "pos");
  a.own_kv = norm_w.has_value() ? 1 : 0;
  TORCH_CHECK(z.size(1) >= H * (d + r) + (a.own_kv ? R + r : 0), "latent: z has too few columns");
  auto dest = [&](const OptTensor& c, const OptTensor& ri, void*& base, const int64_t*& rp, int64_t& cap, const char* name) {
    check_same(*c, z, name);
    TORCH_CHECK(c->size(-1) == R + r && ri.has_value(), name, ": rows of R + r");
    base = c->data_ptr();
    cap = c->numel() / (R + r);
    rp = i64(*ri, a.T, "rows");
  };
  if (a.own_kv) {
    TORCH_CHECK(cache.has_value(), "latent: cache missing");
    a.norm_w = f32(*norm_w, R, "norm_w");
    dest(cache, rows, a.cache, a.rows, a.cap, "cache");
    if (ctx.has_value()) dest(ctx, ctx_rows, a.ctx, a.ctx_rows, a.ctx_cap, "ctx");
  }
  return a;
}

void latent_rotate(at::Tensor& z, int64_t H, int64_t d, int64_t r, const OptTensor& norm_w, int64_t R, int64_t R_real, double eps,
                   const at::Tensor& cos_sin, const at::Tensor& pos, const OptTensor& cache, const OptTensor& rows, const OptTensor& ctx,
                   const OptTensor& ctx_rows) {
  c10::cuda::CUDAGuard guard(z.device());
  tdb::LatentPrepArgs a = latent_args(z, H, d, r, norm_w, R, R_real, eps, cos_sin, pos, cache, rows, ctx, ctx_rows);
  check_cuda(tdb::launch_latent_rotate(a, cur_stream()), "launch_latent_rotate");
}

at::Tensor latent_absorb(const at::Tensor& z, const at::Tensor& uk_t, int64_t r, const OptTensor& norm_w, int64_t R_real, double eps,
                         const at::Tensor& cos_sin, const at::Tensor& pos, const OptTensor& cache, const OptTensor& rows) {
  TORCH_CHECK(uk_t.dim() == 3, "latent_absorb: uk_t [H, R, d]");
  check_same(uk_t, z, "uk_t");
  const int64_t H = uk_t.size(0), R = uk_t.size(1);
  c10::cuda::CUDAGuard guard(z.device());
  tdb::LatentPrepArgs a = latent_args(z, H, uk_t.size(2), r, norm_w, R, R_real, eps, cos_sin, pos, cache, rows, c10::nullopt, c10::nullopt);
  at::Tensor q = at::empty({a.T, H, R + r}, z.options());
  a.uk_t = uk_t.data_ptr();
  a.q_eff = q.data_ptr();
  check_cuda(tdb::launch_latent_absorb(a, cur_stream()), "launch_latent_absorb");
  return q;
}

at::Tensor latent_out(const at::Tensor& o, const OptTensor& ml, const at::Tensor& uv, const at::Tensor& gate) {
  tdb::LatentOutArgs a = {};
  TORCH_CHECK(uv.dim() == 3 && o.dim() >= 3, "latent_out: uv [H, dv, R], o [T, H, splits, R]");
  a.is_f32 = act_f32(uv, "uv");
  check_same(uv, uv, "uv");
  a.H = uv.size(0); a.dv = uv.size(1); a.R = uv.size(2);
  a.T = o.size(0);
  a.splits = o.dim() == 4 ? o.size(2) : 1;
  a.o = f32(o, a.T * a.H * static_cast<int64_t>(a.splits) * a.R, "o");
  TORCH_CHECK(o.size(1) == a.H && o.size(-1) == a.R, "latent_out: o does not fit uv");
  if (ml.has_value()) a.ml = f32(*ml, a.T * a.H * static_cast<int64_t>(a.splits) * 2, "ml");
  TORCH_CHECK(gate.is_cuda() && gate.scalar_type() == uv.scalar_type() && gate.dim() == 2 && gate.stride(1) == 1 && gate.size(0) == a.T &&
                  gate.size(1) >= static_cast<int64_t>(a.H) * a.dv, "latent_out: gate [T, H * dv]");
  a.uv = uv.data_ptr();
  a.gate = gate.data_ptr();
  a.ld_gate = gate.stride(0);
  c10::cuda::CUDAGuard guard(o.device());
  at::Tensor out = at::empty({a.T, static_cast<int64_t>(a.H) * a.dv}, uv.options());
  a.out = out.data_ptr();
  check_cuda(tdb::launch_latent_out(a, cur_stream()), "launch_latent_out");
  return out;
}

// Expanded form on tcgen05.  z holds the (rotated) queries, k [L, H d], ctx [L, R + r], vt [H dv, L].
at::Tensor latent_prefill(const at::Tensor& z, const at::Tensor& k, const at::Tensor& ctx, const at::Tensor& vt, const at::Tensor& cu,
                          const at::Tensor& q_pos0, const at::Tensor& kv_lens, const at::Tensor& ctx0, int64_t max_q, int64_t H, int64_t d,
                          int64_t r, int64_t R, int64_t dv, double scale, const at::Tensor& gate, at::Tensor& error) {
  TORCH_CHECK(z.is_cuda() && z.scalar_type() == at::kBFloat16 && z.dim() == 2 && z.stride(1) == 1 && z.size(1) >= H * (d + r), "latent_prefill: z");
  check_same(k, z, "k");
  check_same(ctx, z, "ctx");
  check_same(vt, z, "vt");
  tdb::LatentPrefillArgs a = {};
  a.T = z.size(0);
  a.L = ctx.size(0);
  TORCH_CHECK(ctx.dim() == 2 && ctx.size(1) == R + r && k.numel() == a.L * H * d && vt.dim() == 2 && vt.size(0) == H * dv && vt.size(1) == a.L,
              "latent_prefill: shapes");
  TORCH_CHECK(gate.is_cuda() && gate.scalar_type() == at::kBFloat16 && gate.dim() == 2 && gate.stride(1) == 1 && gate.size(0) == a.T &&
                  gate.size(1) >= H * dv, "latent_prefill: gate [T, H * dv]");
  a.B = kv_lens.numel();
  a.q = z.data_ptr();
  a.ld_q = z.stride(0);
  a.k = k.data_ptr();
  a.ctx = ctx.data_ptr();
  a.vt = vt.data_ptr();
  a.cu = i32(cu, a.B + 1, "cu");
  a.q_pos0 = i32(q_pos0, a.B, "q_pos0");
  a.kv_lens = i32(kv_lens, a.B, "kv_lens");
  a.ctx0 = i32(ctx0, a.B, "ctx0");
  a.gate = gate.data_ptr();
  a.ld_gate = gate.stride(0);
  a.H = H; a.d = d; a.r = r; a.R = R; a.dv = dv; a.max_q = max_q;
  a.scale = scale;
  a.error_flag = i32(error, 1, "error");
  c10::cuda::CUDAGuard guard(z.device());
  at::Tensor out = at::empty({a.T, H * dv}, z.options());
  a.out = out.data_ptr();
  check_cuda(tdb::launch_latent_prefill(a, cur_stream()), "launch_latent_prefill");
  return out;
}

// Absorbed form on tcgen05, one token per sequence: (partials fp32 [B, H, splits, R], their maxima and sums [B, H, splits, 2]).
std::vector<at::Tensor> latent_decode(const at::Tensor& q, const at::Tensor& cache, const at::Tensor& slots, const at::Tensor& kv_lens,
                                      int64_t R, double scale, int64_t splits, at::Tensor& error) {
  TORCH_CHECK(q.is_cuda() && q.scalar_type() == at::kBFloat16 && q.dim() == 3 && q.is_contiguous(), "latent_decode: q [B, H, R + r] bf16");
  check_same(cache, q, "cache");
  TORCH_CHECK(cache.dim() == 3 && cache.size(2) == q.size(2), "latent_decode: cache [slots, max_len, R + r]");
  tdb::LatentDecodeArgs a = {};
  a.B = q.size(0); a.H = q.size(1); a.R = R; a.r = q.size(2) - R;
  a.q_eff = q.data_ptr();
  a.cache = cache.data_ptr();
  a.slots = i32(slots, a.B, "slots");
  a.kv_lens = i32(kv_lens, a.B, "kv_lens");
  a.num_slots = cache.size(0);
  a.max_len = cache.size(1);
  a.splits = splits;
  a.scale = scale;
  a.error_flag = i32(error, 1, "error");
  c10::cuda::CUDAGuard guard(q.device());
  auto fo = q.options().dtype(at::kFloat);
  at::Tensor o = at::empty({a.B, a.H, splits, R}, fo), ml = at::empty({a.B, a.H, splits, 2}, fo);
  a.o = o.data_ptr<float>();
  a.ml = ml.data_ptr<float>();
  check_cuda(tdb::launch_latent_decode(a, cur_stream()), "launch_latent_decode");
  return {o, ml};
}

// form: 0 decode (one token per sequence), 1 recurrent, 2 chunk-parallel
at::Tensor gla_forward(const at::Tensor& qkvg, const at::Tensor& lowrank, const at::Tensor& a2, const at::Tensor& a2_b, double inv_tau,
                       const at::Tensor& norm_w, at::Tensor& state, const at::Tensor& slots, const at::Tensor& pos0,
                       const OptTensor& cu, int64_t dv_real, double q_scale, double eps, int64_t form, const OptTensor& chunk_seq,
                       const OptTensor& chunk_t0, const OptTensor& seq_chunk0) {
  tdb::GlaArgs a = {};
  a.is_f32 = act_f32(qkvg, "qkvg");
  TORCH_CHECK(qkvg.dim() == 2 && qkvg.stride(1) == 1, "gla: qkvg [T, ld]");
  TORCH_CHECK(state.dim() == 4, "gla: state [slots, H, dk, dv]");
  a.T = qkvg.size(0);
  a.ld = qkvg.stride(0);
  a.H = state.size(1); a.dk = state.size(2); a.dv = state.size(3);
  a.dv_real = dv_real;
  const int64_t Hk = static_cast<int64_t>(a.H) * a.dk, Hv = static_cast<int64_t>(a.H) * a.dv;
  TORCH_CHECK(qkvg.size(1) >= 2 * Hk + 2 * Hv, "gla: qkvg has too few columns");
  a.qkvg = qkvg.data_ptr();
  a.R = lowrank.size(1);
  a.a = f32(lowrank, a.T * a.R, "lowrank");
  TORCH_CHECK(a2.dim() == 2 && a2.size(0) == a.R && a2.size(1) == Hk, "gla: a2 [R, H * dk]");
  a.a2 = f32(a2, a.R * Hk, "a2");
  a.a2_b = f32(a2_b, Hk, "a2_b");
  a.inv_tau = inv_tau;
  a.norm_w = f32(norm_w, a.dv, "norm_w");
  a.state = f32(state, 0, "state");
  a.N = slots.numel();
  a.slots = i32(slots, a.N, "slots");
  a.pos0 = i64(pos0, a.N, "pos0");
  if (cu.has_value()) a.cu = i32(*cu, a.N + 1, "cu");
  a.q_scale = q_scale;
  a.eps = eps;
  c10::cuda::CUDAGuard guard(qkvg.device());
  at::Tensor out = at::empty({a.T, Hv}, qkvg.options());
  a.out = out.data_ptr();
  auto fo = qkvg.options().dtype(at::kFloat);
  if (form == 0) {
    TORCH_CHECK(a.T == a.N, "gla decode: one token per sequence");
    check_cuda(tdb::launch_gla_decode(a, cur_stream()), "launch_gla_decode");
    return out;
  }
  at::Tensor ld = at::empty({a.T, Hk}, fo);
  a.log_decay = ld.data_ptr<float>();
  if (form == 1) {
    at::Tensor o = at::empty({a.T, Hv}, fo);
    a.o_raw = o.data_ptr<float>();
    check_cuda(tdb::launch_gla_recurrent(a, cur_stream()), "launch_gla_recurrent");
    return out;
  }
  TORCH_CHECK(chunk_seq.has_value() && chunk_t0.has_value() && seq_chunk0.has_value() && cu.has_value(), "gla chunk: tables missing");
  a.NC = chunk_seq->numel();
  a.chunk_seq = i32(*chunk_seq, a.NC, "chunk_seq");
  a.chunk_t0 = i32(*chunk_t0, a.NC, "chunk_t0");
  a.seq_chunk0 = i32(*seq_chunk0, a.N + 1, "seq_chunk0");
  at::Tensor cs = at::empty({a.NC, Hk, a.dv}, fo), cd = at::empty({a.NC, Hk}, fo);
  a.chunk_state = cs.data_ptr<float>();
  a.chunk_decay = cd.data_ptr<float>();
  check_cuda(tdb::launch_gla_chunk(a, cur_stream()), "launch_gla_chunk");
  return out;
}

// ---- several residual streams
// One pass between two sublayers (see tdb/streams.h).  ids / table: the streams start; y: what the last sublayer adds; in_w / w: the next
// one's input, which is returned (an empty tensor without them).
at::Tensor hyper_step(at::Tensor& x, const OptTensor& ids, const OptTensor& table, const OptTensor& y, const OptTensor& y2, const OptTensor& y_w,
                      const OptTensor& y2_w, const OptTensor& mix, const OptTensor& out_w, const OptTensor& in_w, const OptTensor& w,
                      const OptTensor& rows, int64_t n_real, double eps, bool act_is_f32) {
  TORCH_CHECK(x.dim() == 3, "hyper_step: x [T, streams, W]");
  tdb::HyperArgs a = {};
  a.T = x.size(0); a.S = x.size(1); a.W = x.size(2);
  a.x = f32(x, a.T * a.S * static_cast<int64_t>(a.W), "x");
  a.is_f32 = act_is_f32 ? 1 : 0;
  a.n_real = n_real;
  a.eps = eps;
  a.n = rows.has_value() ? rows->numel() : a.T;
  a.store = rows.has_value() ? 0 : 1;
  c10::cuda::CUDAGuard guard(x.device());
  const auto act = x.options().dtype(act_is_f32 ? at::kFloat : at::kBFloat16);
  auto in = [&](const at::Tensor& t, const char* name) -> const void* {
    TORCH_CHECK(t.is_cuda() && t.scalar_type() == act.dtype() && t.is_contiguous() && t.size(-1) == a.W, name, ": contiguous [.., W] of the activation dtype");
    return t.data_ptr();
  };
  if (rows.has_value()) a.rows = i64(*rows, a.n, "rows");
  if (ids.has_value()) {
    TORCH_CHECK(table.has_value(), "hyper_step: table missing");
    a.ids = i64(*ids, a.T, "ids");
    a.table = in(*table, "table");
    a.vocab = table->size(0);
  }
  if (y.has_value()) {
    TORCH_CHECK(mix.has_value() && out_w.has_value() && y->numel() == a.T * a.W, "hyper_step: y [T, W] with its weights");
    a.y = in(*y, "y");
    a.mix = f32(*mix, a.S * a.S, "mix");
    a.out = f32(*out_w, a.S, "out");
  }
  if (y2.has_value()) {
    TORCH_CHECK(y.has_value() && y_w.has_value() && y2_w.has_value() && y2->numel() == a.T * a.W, "hyper_step: second branch");
    a.y2 = in(*y2, "y2");
    a.y_w = f32(*y_w, a.W, "y_w");
    a.y2_w = f32(*y2_w, a.W, "y2_w");
  }
  at::Tensor h = at::empty({in_w.has_value() ? a.n : 0, a.W}, act);
  if (in_w.has_value()) {
    TORCH_CHECK(w.has_value(), "hyper_step: norm weight missing");
    a.in = f32(*in_w, a.S, "in");
    a.w = f32(*w, a.W, "w");
    a.h = h.data_ptr();
  }
  check_cuda(tdb::launch_hyper_step(a, cur_stream()), "launch_hyper_step");
  return h;
}

at::Tensor head_prep(const at::Tensor& z, int64_t H, int64_t G, int64_t D, int64_t d_real, const OptTensor& q_w, const OptTensor& k_w, bool unit,
                     double eps, const at::Tensor& cos_sin, int64_t rot, bool interleaved, const at::Tensor& pos, at::Tensor& k_cache,
                     at::Tensor& v_cache, const at::Tensor& rows) {
  tdb::HeadPrepArgs a = {};
  a.is_f32 = act_f32(z, "z");
  TORCH_CHECK(z.dim() == 2 && z.stride(1) == 1 && z.size(1) >= (H + 2 * G) * D, "head_prep: z [T, >= (H + 2 G) D]");
  check_same(k_cache, z, "k_cache");
  check_same(v_cache, z, "v_cache");
  TORCH_CHECK(k_cache.numel() % (G * D) == 0 && v_cache.numel() == k_cache.numel(), "head_prep: caches [rows, G, D]");
  TORCH_CHECK(cos_sin.dim() == 2, "head_prep: cos_sin [positions, width]");
  a.z = z.data_ptr(); a.ld = z.stride(0); a.T = z.size(0);
  a.H = H; a.G = G; a.D = D; a.d_real = d_real;
  if (q_w.has_value()) a.q_w = f32(*q_w, D, "q_w");
  if (k_w.has_value()) a.k_w = f32(*k_w, D, "k_w");
  a.n_pos = cos_sin.size(0);
  a.rot_ld = cos_sin.size(1);
  a.cos_sin = f32(cos_sin, 0, "cos_sin");
  a.rot = rot; a.interleaved = interleaved ? 1 : 0; a.unit = unit ? 1 : 0;
  a.eps = eps;
  a.pos = i64(pos, a.T, "pos");
  a.rows = i64(rows, a.T, "rows");
  a.cap = k_cache.numel() / (G * D);
  a.k_cache = k_cache.data_ptr();
  a.v_cache = v_cache.data_ptr();
  c10::cuda::CUDAGuard guard(z.device());
  at::Tensor q = at::empty({a.T, H, D}, z.options());
  a.q_out = q.data_ptr();
  check_cuda(tdb::launch_head_prep(a, cur_stream()), "launch_head_prep");
  return q;
}

at::Tensor gated_act(const at::Tensor& in, int64_t act) {
  const int fp = act_f32(in, "in");
  TORCH_CHECK(in.dim() == 2 && in.is_contiguous() && in.size(1) % 2 == 0, "gated_act: contiguous [rows, 2 F]");
  c10::cuda::CUDAGuard guard(in.device());
  at::Tensor out = at::empty({in.size(0), in.size(1) / 2}, in.options());
  check_cuda(tdb::launch_gated_act(in.data_ptr(), out.data_ptr(), in.size(0), in.size(1) / 2, act, fp, cur_stream()), "launch_gated_act");
  return out;
}

// Gated delta rule, serving form.  form: 0 decode (one token per sequence), 1 recurrent, 2 chunk-parallel
at::Tensor delta_forward(const at::Tensor& z, const at::Tensor& ab, const at::Tensor& conv_w, const at::Tensor& a_log, const at::Tensor& dt_bias,
                         const at::Tensor& norm_w, at::Tensor& state, at::Tensor& conv, const at::Tensor& slots, const at::Tensor& pos0,
                         const OptTensor& cu, int64_t G, int64_t dv_real, double q_scale, double unit_eps, double eps, int64_t form,
                         const OptTensor& chunk_seq, const OptTensor& chunk_t0, const OptTensor& seq_chunk0) {
  tdb::DeltaArgs a = {};
  a.is_f32 = act_f32(z, "z");
  TORCH_CHECK(z.dim() == 2 && z.stride(1) == 1, "delta: z [T, ld]");
  TORCH_CHECK(state.dim() == 4 && conv.dim() == 3, "delta: state [slots, H, dk, dv], conv [slots, taps, C]");
  a.T = z.size(0); a.ld = z.stride(0);
  a.G = G; a.H = state.size(1); a.dk = state.size(2); a.dv = state.size(3);
  a.taps = conv.size(1);
  const int64_t Gk = G * a.dk, Hv = static_cast<int64_t>(a.H) * a.dv, C = 2 * Gk + Hv;
  TORCH_CHECK(z.size(1) >= C + Hv && conv.size(2) == C && conv.size(0) == state.size(0), "delta: shapes of z and conv");
  TORCH_CHECK(conv_w.dim() == 2 && conv_w.size(0) == C && conv_w.size(1) == a.taps, "delta: conv_w [C, taps]");
  check_same(conv, z, "conv");
  a.z = z.data_ptr();
  a.ab = f32(ab, a.T * 2 * a.H, "ab");
  a.conv_w = f32(conv_w, C * a.taps, "conv_w");
  a.a_log = f32(a_log, a.H, "a_log");
  a.dt_bias = f32(dt_bias, a.H, "dt_bias");
  a.norm_w = f32(norm_w, a.dv, "norm_w");
  a.state = f32(state, 0, "state");
  a.conv = conv.data_ptr();
  a.N = slots.numel();
  a.slots = i32(slots, a.N, "slots");
  a.pos0 = i64(pos0, a.N, "pos0");
  if (cu.has_value()) a.cu = i32(*cu, a.N + 1, "cu");
  a.dv_real = dv_real; a.q_scale = q_scale; a.unit_eps = unit_eps; a.eps = eps;
  c10::cuda::CUDAGuard guard(z.device());
  at::Tensor out = at::empty({a.T, Hv}, z.options());
  a.out = out.data_ptr();
  if (form == 0) {
    TORCH_CHECK(a.T == a.N, "delta decode: one token per sequence");
    check_cuda(tdb::launch_delta_decode(a, cur_stream()), "launch_delta_decode");
    return out;
  }
  TORCH_CHECK(cu.has_value() && chunk_seq.has_value() && chunk_t0.has_value() && seq_chunk0.has_value(), "delta prompt: tables missing");
  a.NC = chunk_seq->numel();
  a.chunk_seq = i32(*chunk_seq, a.NC, "chunk_seq");
  a.chunk_t0 = i32(*chunk_t0, a.NC, "chunk_t0");
  a.seq_chunk0 = i32(*seq_chunk0, a.N + 1, "seq_chunk0");
  const auto fo = z.options().dtype(at::kFloat), bo = z.options().dtype(at::kBFloat16);
  at::Tensor gb = at::empty({2, a.T, a.H}, fo);
  a.log_g = gb.data_ptr<float>();
  a.beta = a.log_g + a.T * a.H;
  if (form == 1) {
    at::Tensor qk = at::empty({2, a.T, Gk}, fo), v = at::empty({2, a.T, Hv}, fo);
    a.q = qk.data_ptr<float>();
    a.k = qk.data_ptr<float>() + a.T * Gk;
    a.v = v.data_ptr<float>();
    a.o_raw = v.data_ptr<float>() + a.T * Hv;
    check_cuda(tdb::launch_delta_recurrent(a, cur_stream()), "launch_delta_recurrent");
    return out;
  }
  at::Tensor qk = at::empty({4, a.T, Gk}, bo), v = at::empty({a.T, Hv}, bo);
  a.q = qk[0].data_ptr(); a.q_lo = qk[1].data_ptr(); a.k = qk[2].data_ptr(); a.k_lo = qk[3].data_ptr();
  a.v = v.data_ptr();
  const int64_t NH = static_cast<int64_t>(a.NC) * a.H;
  at::Tensor trans = at::empty({NH, a.dk, a.dk}, fo), inject = at::empty({NH, a.dk, a.dv}, fo), read = at::empty({NH, 64, a.dk}, fo);
  at::Tensor local = at::empty({NH, 64, a.dv}, fo), states = at::empty({NH, a.dk, a.dv}, fo), decay = at::empty({NH}, fo);
  a.trans = trans.data_ptr(); a.inject = inject.data_ptr<float>(); a.read = read.data_ptr();
  a.local = local.data_ptr<float>(); a.states = states.data_ptr(); a.decay = decay.data_ptr<float>();
  check_cuda(tdb::launch_delta_chunk(a, cur_stream()), "launch_delta_chunk");
  return out;
}

}  // namespace

void bind_hybrid(py::module_& m) {
  m.def("embed_stream", &embed_stream);
  m.def("postnorm_add", &postnorm_add);
  m.def("combine_rows", &combine_rows);
  m.def("stream_norm", &stream_norm);
  m.def("qk_norm_tied", &qk_norm_tied);
  m.def("qk_sumsq", &qk_sumsq);
  m.def("narrow_linear", &narrow_linear);
  m.def("sigmoid_router", &sigmoid_router);
  m.def("softmax_router", &softmax_router);
  m.def("relu2", &relu2, py::arg("in"), py::arg("row_weight"), py::arg("bias") = py::none());
  m.def("expert_gemv", &expert_gemv, py::arg("x"), py::arg("up"), py::arg("down"), py::arg("ids"), py::arg("weights"), py::arg("shared_up"),
        py::arg("shared_down"), py::arg("shared_gate"), py::arg("gated") = false, py::arg("identity") = 0,
        py::arg("skip_identity") = false);
  m.def("parallel_add", &parallel_add);
  m.def("latent_rotate", &latent_rotate);
  m.def("latent_absorb", &latent_absorb);
  m.def("latent_out", &latent_out);
  m.def("latent_prefill", &latent_prefill);
  m.def("latent_decode", &latent_decode);
  m.def("gla_forward", &gla_forward);
  m.def("hyper_step", &hyper_step);
  m.def("head_prep", &head_prep);
  m.def("gated_act", &gated_act);
  m.def("delta_forward", &delta_forward);
  m.def("delta_chunk_supported", &tdb::delta_chunk_supported);
  m.def("gla_chunk_supported", &tdb::gla_chunk_supported);
}
