// Python bindings of the kernels in tdb/hybrid.h.
#include <ATen/cuda/CUDAContext.h>
#include <c10/cuda/CUDAGuard.h>
#include <torch/extension.h>

#include "tdb/hybrid.h"

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

void embed_stream(const at::Tensor& ids, const at::Tensor& table, at::Tensor& x, const OptTensor& xb) {
  const int fp = act_f32(table, "table");
  TORCH_CHECK(table.dim() == 2 && table.is_contiguous(), "embed_stream: contiguous table [V, W]");
  const int64_t T = ids.numel(), W = table.size(1);
  c10::cuda::CUDAGuard guard(table.device());
  void* b = nullptr;
  if (!fp) {
    TORCH_CHECK(xb.has_value() && xb->numel() == T * W, "embed_stream: bf16 copy missing");
    check_same(*xb, table, "xb");
    b = xb->data_ptr();
  }
  check_cuda(tdb::launch_embed_stream(i64(ids, T, "ids"), table.data_ptr(), f32(x, T * W, "x"), b, T, W, table.size(0), fp, cur_stream()),
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

at::Tensor relu2(const at::Tensor& in, const OptTensor& row_weight) {
  const int fp = act_f32(in, "in");
  TORCH_CHECK(in.dim() == 2 && in.is_contiguous(), "relu2: contiguous [rows, F]");
  c10::cuda::CUDAGuard guard(in.device());
  at::Tensor out = at::empty_like(in);
  const float* w = row_weight.has_value() ? f32(*row_weight, in.size(0), "row_weight") : nullptr;
  check_cuda(tdb::launch_relu2(in.data_ptr(), w, out.data_ptr(), in.size(0), in.size(1), fp, cur_stream()), "launch_relu2");
  return out;
}

at::Tensor expert_gemv(const at::Tensor& x, const at::Tensor& up, const at::Tensor& down, const at::Tensor& ids, const at::Tensor& weights,
                       const OptTensor& shared_up, const OptTensor& shared_down, const OptTensor& shared_gate) {
  tdb::ExpertGemvArgs a = {};
  a.is_f32 = act_f32(x, "x");
  TORCH_CHECK(x.dim() == 2 && x.is_contiguous() && up.dim() == 3 && down.dim() == 3, "expert_gemv: x [T, K], up [E, F, K], down [E, K, F]");
  check_same(up, x, "up");
  check_same(down, x, "down");
  a.T = x.size(0); a.K = x.size(1); a.E = up.size(0); a.F = up.size(1);
  TORCH_CHECK(up.size(2) == a.K && down.size(0) == a.E && down.size(1) == a.K && down.size(2) == a.F, "expert_gemv: shape mismatch");
  TORCH_CHECK(ids.dim() == 2 && ids.size(0) == a.T, "expert_gemv: ids [T, top]");
  a.top = ids.size(1);
  a.ids = i32(ids, a.T * a.top, "ids");
  a.weights = f32(weights, a.T * a.top, "weights");
  if (shared_up.has_value()) {
    TORCH_CHECK(shared_down.has_value(), "expert_gemv: shared_down missing");
    check_same(*shared_up, x, "shared_up");
    check_same(*shared_down, x, "shared_down");
    a.Fs = shared_up->size(0);
    TORCH_CHECK(shared_up->size(1) == a.K && shared_down->size(0) == a.K && shared_down->size(1) == a.Fs, "expert_gemv: shared shapes");
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
  m.def("relu2", &relu2);
  m.def("expert_gemv", &expert_gemv);
  m.def("gla_forward", &gla_forward);
  m.def("gla_chunk_supported", &tdb::gla_chunk_supported);
}
