// Python bindings of attention over a sliding window, the state space layer, and sublayers between two norms.
#include <ATen/cuda/CUDAContext.h>
#include <c10/cuda/CUDAGuard.h>
#include <torch/extension.h>

#include "tdb/hybrid.h"
#include "tdb/ssd.h"
#include "tdb/window.h"

namespace py = pybind11;
using OptTensor = c10::optional<at::Tensor>;

namespace {

cudaStream_t cur_stream() { return at::cuda::getCurrentCUDAStream().stream(); }
void check_cuda(cudaError_t e, const char* what) { TORCH_CHECK(e == cudaSuccess, what, ": ", cudaGetErrorString(e)); }

int act_f32(const at::Tensor& t, const char* name) {
  TORCH_CHECK(t.is_cuda() && (t.scalar_type() == at::kFloat || t.scalar_type() == at::kBFloat16), name, ": fp32 or bf16 CUDA tensor");
  return t.scalar_type() == at::kFloat ? 1 : 0;
}
void* same(const at::Tensor& t, const at::Tensor& like, int64_t numel, const char* name) {
  TORCH_CHECK(t.is_cuda() && t.scalar_type() == like.scalar_type() && t.is_contiguous() && (numel < 0 || t.numel() == numel), name,
              ": contiguous CUDA tensor of the activation dtype", numel < 0 ? "" : " and the right size");
  return t.data_ptr();
}
float* f32(const at::Tensor& t, int64_t numel, const char* name) {
  TORCH_CHECK(t.is_cuda() && t.scalar_type() == at::kFloat && t.is_contiguous() && t.numel() >= numel, name, ": contiguous fp32 CUDA tensor of at least ",
              numel, " elements");
  return t.data_ptr<float>();
}
int32_t* i32(const at::Tensor& t, int64_t numel, const char* name) {
  TORCH_CHECK(t.is_cuda() && t.scalar_type() == at::kInt && t.is_contiguous() && t.numel() >= numel, name, ": contiguous int32 CUDA tensor of at least ",
              numel, " elements");
  return t.data_ptr<int32_t>();
}
int64_t* i64(const at::Tensor& t, int64_t numel, const char* name) {
  TORCH_CHECK(t.is_cuda() && t.scalar_type() == at::kLong && t.is_contiguous() && t.numel() >= numel, name, ": contiguous int64 CUDA tensor of at least ",
              numel, " elements");
  return t.data_ptr<int64_t>();
}

// ---- a sublayer between two norms.  Returns the next input (an empty tensor without `pre`).
at::Tensor sandwich(at::Tensor& x, const OptTensor& ids, const OptTensor& table, double scale, const OptTensor& y, const OptTensor& post,
                    const OptTensor& pre, const OptTensor& rows, int64_t n_real, double eps, bool act_is_f32) {
  TORCH_CHECK(x.dim() == 2, "sandwich: x [T, W]");
  tdb::SandwichArgs a = {};
  const int64_t T = x.size(0);
  a.W = x.size(1);
  a.x = f32(x, T * a.W, "x");
  a.is_f32 = act_is_f32 ? 1 : 0;
  a.n_real = n_real;
  a.eps = eps;
  a.n = rows.has_value() ? rows->numel() : T;
  a.store = !rows.has_value() && (ids.has_value() || y.has_value());
  c10::cuda::CUDAGuard guard(x.device());
  const auto act = x.options().dtype(act_is_f32 ? at::kFloat : at::kBFloat16);
  auto in = [&](const at::Tensor& t, const char* name) -> const void* {
    TORCH_CHECK(t.is_cuda() && t.scalar_type() == act.dtype() && t.is_contiguous() && t.size(-1) == a.W, name, ": contiguous [.., W] of the activation dtype");
    return t.data_ptr();
  };
  auto weight = [&](const OptTensor& t, int& n, const char* name) -> const float* {
    TORCH_CHECK(t.has_value() && (t->numel() == 1 || t->numel() == a.W), "sandwich: ", name, " holds one number or one per coordinate");
    n = static_cast<int>(t->numel());
    return f32(*t, n, name);
  };
  if (rows.has_value()) a.rows = i64(*rows, a.n, "rows");
  if (ids.has_value()) {
    TORCH_CHECK(table.has_value(), "sandwich: table missing");
    a.ids = i64(*ids, T, "ids");
    a.table = in(*table, "table");
    a.vocab = table->size(0);
    a.scale = scale;
  }
  if (y.has_value()) {
    TORCH_CHECK(y->numel() == T * a.W, "sandwich: y [T, W]");
    a.y = in(*y, "y");
    a.post = weight(post, a.post_n, "post");
  }
  at::Tensor h = at::empty({pre.has_value() ? a.n : 0, a.W}, act);
  if (pre.has_value()) {
    a.pre = weight(pre, a.pre_n, "pre");
    a.h = h.data_ptr();
  }
  check_cuda(tdb::launch_sandwich(a, cur_stream()), "launch_sandwich");
  return h;
}

// ---- queries, keys and values of attention over a window
at::Tensor qkv_prep(const at::Tensor& z, int64_t Hq, int64_t Gk, int64_t G, int64_t dk, int64_t dv, const OptTensor& bias, const OptTensor& q_w,
                    const OptTensor& k_w, int64_t nq_real, int64_t nk_real, const OptTensor& sumsq, double eps, const OptTensor& cos_sin, int64_t rot,
                    const at::Tensor& pos, at::Tensor& k_a, at::Tensor& v_a, const at::Tensor& rows_a, const OptTensor& k_b, const OptTensor& v_b,
                    const OptTensor& rows_b) {
  tdb::QkvPrepArgs a = {};
  a.is_f32 = act_f32(z, "z");
  const int64_t Nq = Hq * dk, Nk = Gk * dk, Nv = G * dv;
  TORCH_CHECK(z.dim() == 2 && z.stride(1) == 1 && z.size(1) >= Nq + Nk + Nv, "qkv_prep: z [T, >= q | k | v]");
  a.z = z.data_ptr(); a.ld = z.stride(0); a.T = z.size(0);
  a.Hq = Hq; a.Gk = Gk; a.G = G; a.dk = dk; a.dv = dv;
  if (bias.has_value()) a.bias = f32(*bias, Nq + Nk + Nv, "bias");
  if (q_w.has_value()) {
    TORCH_CHECK(k_w.has_value(), "qkv_prep: both norms or none");
    a.q_w = f32(*q_w, Nq, "q_w");
    a.k_w = f32(*k_w, Nk, "k_w");
    if (sumsq.has_value()) a.sumsq = f32(*sumsq, a.T * 2, "sumsq");
  }
  a.nq_real = nq_real; a.nk_real = nk_real; a.eps = eps;
  a.rot = rot;
  if (rot > 0) {
    TORCH_CHECK(cos_sin.has_value() && cos_sin->dim() == 2, "qkv_prep: cos_sin [positions, width]");
    a.cos_sin = f32(*cos_sin, 0, "cos_sin");
    a.n_pos = cos_sin->size(0);
    a.rot_ld = cos_sin->size(1);
  }
  a.pos = i64(pos, a.T, "pos");
  auto place = [&](const at::Tensor& k, const at::Tensor& v, const at::Tensor& rows, void*& kp, void*& vp, const int64_t*& rp, int64_t& cap) {
    kp = same(k, z, -1, "keys");
    vp = same(v, z, -1, "values");
    TORCH_CHECK(k.numel() % Nk == 0 && v.numel() % Nv == 0 && k.numel() / Nk == v.numel() / Nv, "qkv_prep: keys [rows, Gk, dk], values [rows, G, dv]");
    cap = k.numel() / Nk;
    rp = i64(rows, a.T, "rows");
  };
  place(k_a, v_a, rows_a, a.k_a, a.v_a, a.rows_a, a.cap_a);
  if (k_b.has_value()) {
    TORCH_CHECK(v_b.has_value() && rows_b.has_value(), "qkv_prep: second place incomplete");
    place(*k_b, *v_b, *rows_b, a.k_b, a.v_b, a.rows_b, a.cap_b);
  }
  c10::cuda::CUDAGuard guard(z.device());
  at::Tensor q = at::empty({a.T, Hq, dk}, z.options());
  a.q_out = q.data_ptr();
  check_cuda(tdb::launch_qkv_prep(a, cur_stream()), "launch_qkv_prep");
  return q;
}

// ---- attention over a window; bias: the sigmoid form, else the differential one.  k and v are [.., heads, elements]
tdb::WindowAttnArgs window_args(const at::Tensor& q, const at::Tensor& k, const at::Tensor& v, double scale, const OptTensor& bias, double lambda,
                                double out_scale, double eps, int64_t dv_real, const OptTensor& gate, at::Tensor& out) {
  tdb::WindowAttnArgs a = {};
  a.is_f32 = act_f32(q, "q");
  TORCH_CHECK(q.dim() == 3 && q.is_contiguous() && k.dim() >= 3 && v.dim() >= 3 && k.size(-1) == q.size(2), "window attention: q [T, H maps, dk], k [.., G maps, dk], v [.., G, dv]");
  a.maps = bias.has_value() ? 1 : 2;
  a.T = q.size(0);
  a.dk = q.size(2);
  a.G = v.size(-2);
  a.dv = v.size(-1);
  TORCH_CHECK(q.size(1) % a.maps == 0 && k.size(-2) == static_cast<int64_t>(a.G) * a.maps, "window attention: number of heads");
  a.H = q.size(1) / a.maps;
  a.rows = v.numel() / (static_cast<int64_t>(a.G) * a.dv);
  a.q = q.data_ptr();
  a.k = same(k, q, a.rows * a.G * a.maps * a.dk, "k");
  a.v = same(v, q, -1, "v");
  a.scale = scale;
  if (bias.has_value()) {
    TORCH_CHECK(bias->dim() == 2 && bias->size(0) == a.H, "window attention: bias [H, distances]");
    a.bias = f32(*bias, a.H, "bias");
    a.bias_n = bias->size(1);
  }
  a.lambda = lambda; a.out_scale = out_scale; a.eps = eps; a.dv_real = dv_real;
  if (gate.has_value()) {
    TORCH_CHECK(gate->is_cuda() && gate->scalar_type() == q.scalar_type() && gate->dim() == 2 && gate->size(0) == a.T && gate->size(1) >= a.H && gate->stride(1) == 1,
                "window attention: gate [T, >= H] of q's dtype");
    a.gate = gate->data_ptr();
    a.ld_gate = gate->stride(0);
  }
  out = at::empty({a.T, a.H, a.dv}, q.options());
  a.out = out.data_ptr();
  return a;
}

at::Tensor window_simple(const at::Tensor& q, const at::Tensor& k, const at::Tensor& v, double scale, const OptTensor& bias, double lambda, double out_scale,
                         double eps, int64_t dv_real, const OptTensor& gate, const at::Tensor& row0, const at::Tensor& n_keys, const at::Tensor& newest) {
  c10::cuda::CUDAGuard guard(q.device());
  at::Tensor out;
  tdb::WindowAttnArgs a = window_args(q, k, v, scale, bias, lambda, out_scale, eps, dv_real, gate, out);
  a.row0 = i64(row0, a.T, "row0");
  a.n_keys = i32(n_keys, a.T, "n_keys");
  a.newest = i32(newest, a.T, "newest");
  check_cuda(tdb::launch_window_simple(a, cur_stream()), "launch_window_simple");
  return out;
}

at::Tensor window_decode(const at::Tensor& q, const at::Tensor& k, const at::Tensor& v, double scale, const OptTensor& bias, double lambda, double out_scale,
                         double eps, int64_t dv_real, const OptTensor& gate, const at::Tensor& slots, const at::Tensor& pos, int64_t splits,
                         at::Tensor& counters) {
  c10::cuda::CUDAGuard guard(q.device());
  at::Tensor out;
  tdb::WindowAttnArgs a = window_args(q, k, v, scale, bias, lambda, out_scale, eps, dv_real, gate, out);
  TORCH_CHECK(v.dim() == 4, "window_decode: k and v [slots, ring, heads, elements]");
  a.ring = v.size(1);
  a.slots = i32(slots, a.T, "slots");
  a.pos = i64(pos, a.T, "pos");
  a.splits = splits;
  const int chunks = tdb::window_head_chunks(a.H, a.G, a.maps);
  at::Tensor ws = at::empty({tdb::window_decode_workspace(a.T, a.G, chunks, a.splits, a.dv)}, q.options().dtype(at::kFloat));
  a.workspace = ws.data_ptr<float>();
  a.counters = reinterpret_cast<uint32_t*>(i32(counters, a.T * a.G * chunks, "counters"));
  check_cuda(tdb::launch_window_decode(a, cur_stream()), "launch_window_decode");
  return out;
}

// Returns (out, error flag int32 [1]: non-zero if a bounded wait inside the kernel gave up).
std::vector<at::Tensor> window_prompt(const at::Tensor& q, const at::Tensor& k, const at::Tensor& v, double scale, const OptTensor& bias, double lambda,
                                      double out_scale, double eps, int64_t dv_real, const OptTensor& gate, const at::Tensor& cu, const at::Tensor& q_pos0,
                                      const at::Tensor& shift, int64_t max_q, int64_t window) {
  c10::cuda::CUDAGuard guard(q.device());
  at::Tensor out, err = at::zeros({1}, q.options().dtype(at::kInt));
  tdb::WindowAttnArgs a = window_args(q, k, v, scale, bias, lambda, out_scale, eps, dv_real, gate, out);
  a.N = q_pos0.numel();
  a.cu = i32(cu, a.N + 1, "cu");
  a.q_pos0 = i32(q_pos0, a.N, "q_pos0");
  a.shift = i32(shift, a.N, "shift");
  a.max_q = max_q;
  a.window = window;
  a.error_flag = err.data_ptr<int32_t>();
  check_cuda(tdb::launch_window_prompt(a, cur_stream()), "launch_window_prompt");
  return {out, err};
}

// ---- state space layer.  form: 0 decode (one token per sequence), 1 recurrent, 2 chunk-parallel
at::Tensor ssd_forward(const at::Tensor& z, int64_t dt_col, const at::Tensor& conv_w, const at::Tensor& conv_b, const at::Tensor& a_log,
                       const at::Tensor& dt_bias, const at::Tensor& skip, at::Tensor& state, at::Tensor& conv, const at::Tensor& slots,
                       const at::Tensor& pos0, const OptTensor& cu, int64_t G, int64_t form, const OptTensor& chunk_seq, const OptTensor& chunk_t0,
                       const OptTensor& seq_chunk0) {
  tdb::SsdArgs a = {};
  a.is_f32 = act_f32(z, "z");
  TORCH_CHECK(z.dim() == 2 && z.stride(1) == 1, "ssd: z [T, ld]");
  TORCH_CHECK(state.dim() == 4 && conv.dim() == 3, "ssd: state [slots, H, dk, dv], conv [slots, taps, channels]");
  a.T = z.size(0); a.ld = z.stride(0);
  a.G = G; a.H = state.size(1); a.dk = state.size(2); a.dv = state.size(3);
  a.taps = conv.size(1);
  a.dt_col = dt_col;
  const int64_t Hv = static_cast<int64_t>(a.H) * a.dv, C = Hv + 2 * G * a.dk;
  TORCH_CHECK(dt_col >= C && z.size(1) >= dt_col + a.H && conv.size(2) == C && conv.size(0) == state.size(0), "ssd: shapes of z and conv");
  TORCH_CHECK(conv_w.dim() == 2 && conv_w.size(0) == C && conv_w.size(1) == a.taps, "ssd: conv_w [channels, taps]");
  a.z = z.data_ptr();
  a.conv_w = f32(conv_w, C * a.taps, "conv_w");
  a.conv_b = f32(conv_b, C, "conv_b");
  a.a_log = f32(a_log, a.H, "a_log");
  a.dt_bias = f32(dt_bias, a.H, "dt_bias");
  a.skip = f32(skip, a.H, "skip");
  a.state = f32(state, 0, "state");
  a.conv = same(conv, z, -1, "conv");
  a.N = slots.numel();
  a.slots = i32(slots, a.N, "slots");
  a.pos0 = i64(pos0, a.N, "pos0");
  if (cu.has_value()) a.cu = i32(*cu, a.N + 1, "cu");
  c10::cuda::CUDAGuard guard(z.device());
  at::Tensor out = at::empty({a.T, Hv}, z.options());
  a.out = out.data_ptr();
  if (form == 0) {
    TORCH_CHECK(a.T == a.N, "ssd decode: one token per sequence");
    check_cuda(tdb::launch_ssd_decode(a, cur_stream()), "launch_ssd_decode");
    return out;
  }
  TORCH_CHECK(cu.has_value() && chunk_seq.has_value() && chunk_t0.has_value() && seq_chunk0.has_value(), "ssd prompt: tables missing");
  a.NC = chunk_seq->numel();
  a.chunk_seq = i32(*chunk_seq, a.NC, "chunk_seq");
  a.chunk_t0 = i32(*chunk_t0, a.NC, "chunk_t0");
  a.seq_chunk0 = i32(*seq_chunk0, a.N + 1, "seq_chunk0");
  const auto fo = z.options().dtype(at::kFloat);
  at::Tensor xbc = at::empty({a.T, C}, z.options()), gd = at::empty({2, a.T, a.H}, fo);
  a.xbc = xbc.data_ptr();
  a.dt = gd.data_ptr<float>();
  a.log_g = a.dt + a.T * a.H;
  if (form == 1) {
    check_cuda(tdb::launch_ssd_recurrent(a, cur_stream()), "launch_ssd_recurrent");
    return out;
  }
  at::Tensor inject = at::empty({static_cast<int64_t>(a.NC) * a.H, a.dk, a.dv}, fo);
  a.inject = inject.data_ptr<float>();
  check_cuda(tdb::launch_ssd_chunk(a, cur_stream()), "launch_ssd_chunk");
  return out;
}

at::Tensor gated_norm(const at::Tensor& y, const at::Tensor& gate, const at::Tensor& w, int64_t H, int64_t dv_real, int64_t parts, double eps) {
  tdb::GatedNormArgs a = {};
  a.is_f32 = act_f32(y, "y");
  TORCH_CHECK(y.dim() == 2 && y.size(1) % H == 0, "gated_norm: y [T, H dv]");
  a.T = y.size(0); a.H = H; a.dv = y.size(1) / H; a.dv_real = dv_real; a.parts = parts; a.eps = eps;
  a.y = same(y, y, -1, "y");
  TORCH_CHECK(gate.is_cuda() && gate.scalar_type() == y.scalar_type() && gate.dim() == 2 && gate.size(0) == a.T && gate.size(1) >= y.size(1) && gate.stride(1) == 1,
              "gated_norm: gate [T, >= H dv] of y's dtype");
  a.gate = gate.data_ptr();
  a.ld_gate = gate.stride(0);
  a.w = f32(w, y.size(1), "w");
  c10::cuda::CUDAGuard guard(y.device());
  at::Tensor out = at::empty_like(y);
  a.out = out.data_ptr();
  check_cuda(tdb::launch_gated_norm(a, cur_stream()), "launch_gated_norm");
  return out;
}

}  // namespace

void bind_window(py::module_& m) {
  m.def("sandwich", &sandwich);
  m.def("qkv_prep", &qkv_prep);
  m.def("window_simple", &window_simple);
  m.def("window_decode", &window_decode);
  m.def("window_prompt", &window_prompt);
  m.def("window_head_chunks", &tdb::window_head_chunks);
  m.def("ssd_forward", &ssd_forward);
  m.def("ssd_chunk_supported", &tdb::ssd_chunk_supported);
  m.def("gated_norm", &gated_norm);
}
