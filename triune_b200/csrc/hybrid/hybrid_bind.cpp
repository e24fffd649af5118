// Python bindings of the heterogeneous-layer kernels. Shapes, strides and dtypes are checked here, so that no launch
// can leave its buffers.
#include <ATen/cuda/CUDAContext.h>
#include <c10/cuda/CUDAGuard.h>
#include <torch/extension.h>

#include "hybrid.cuh"

namespace {
using torch::Tensor;
using OptT = c10::optional<Tensor>;

inline cudaStream_t cur_stream() { return at::cuda::getCurrentCUDAStream().stream(); }

// [rows, >= cols] compute matrix with contiguous rows; returns true for fp32
bool rows_of(const Tensor& t, int64_t rows, int64_t cols, const char* n) {
  TORCH_CHECK(t.is_cuda() && t.dim() == 2 && t.stride(1) == 1, n, ": 2-D CUDA matrix with contiguous rows expected");
  TORCH_CHECK(t.size(0) >= rows && t.size(1) >= cols, n, ": [", t.size(0), ", ", t.size(1), "] is smaller than [", rows, ", ", cols, "]");
  TORCH_CHECK(t.scalar_type() == at::kFloat || t.scalar_type() == at::kBFloat16, n, ": fp32 or bf16 expected");
  return t.scalar_type() == at::kFloat;
}
const float* f32v(const Tensor& t, int64_t n, const char* name) {
  TORCH_CHECK(t.is_cuda() && t.scalar_type() == at::kFloat && t.is_contiguous() && t.numel() >= n, name, ": contiguous CUDA fp32 of ", n, " expected");
  return t.data_ptr<float>();
}
const float* f32o(const OptT& t, int64_t n, const char* name) {
  return t.has_value() && t->defined() ? f32v(*t, n, name) : nullptr;
}
const double* f64v(const Tensor& t, int64_t n, const char* name) {
  TORCH_CHECK(t.is_cuda() && t.scalar_type() == at::kDouble && t.is_contiguous() && t.numel() >= n, name, ": contiguous CUDA fp64 of ", n, " expected");
  return t.data_ptr<double>();
}
tb::Pos pos_of(int64_t host, const OptT& dev) {
  tb::Pos p{host, nullptr};
  if (dev.has_value() && dev->defined()) {
    TORCH_CHECK(dev->is_cuda() && dev->scalar_type() == at::kLong && dev->numel() >= 1, "position: CUDA int64 expected");
    p.dev = reinterpret_cast<const long long*>(dev->data_ptr<int64_t>());
  } else {
    TORCH_CHECK(host >= 0, "position must not be negative");
  }
  return p;
}

int* status_of(const OptT& status) {
  if (!status.has_value() || !status->defined()) return nullptr;
  TORCH_CHECK(status->is_cuda() && status->scalar_type() == at::kInt && status->numel() >= 1, "status: CUDA int32 expected");
  return status->data_ptr<int>();
}

Tensor embed_rows(const Tensor& table, const Tensor& ids) {
  TORCH_CHECK(table.is_contiguous(), "table must be contiguous");
  const bool f32 = rows_of(table, 0, 0, "table");
  TORCH_CHECK(ids.is_cuda() && ids.scalar_type() == at::kLong && ids.is_contiguous(), "ids: contiguous CUDA int64 expected");
  c10::cuda::CUDAGuard guard(table.device());
  Tensor out = torch::empty({ids.numel(), table.size(1)}, table.options().dtype(at::kFloat));
  tb::launch_embed_rows(table.data_ptr(), f32, reinterpret_cast<const long long*>(ids.data_ptr<int64_t>()), out.data_ptr<float>(),
                        (int)ids.numel(), (int)table.size(1), (int)table.size(0), cur_stream());
  return out;
}

Tensor norm_rows(const Tensor& x, const Tensor& w, double eps, int64_t kind, bool f32) {
  TORCH_CHECK(x.is_cuda() && x.dim() == 2 && x.scalar_type() == at::kFloat && x.is_contiguous(), "x: contiguous CUDA fp32 rows expected");
  c10::cuda::CUDAGuard guard(x.device());
  Tensor y = torch::empty_like(x, x.options().dtype(f32 ? at::kFloat : at::kBFloat16));
  tb::launch_norm_rows(x.data_ptr<float>(), f32v(w, x.size(1), "w"), y.data_ptr(), f32, (int)x.size(0), (int)x.size(1), (float)eps,
                       (int)kind, cur_stream());
  return y;
}

tb::GluArgs glu_args(int64_t act, const OptT& bias, int64_t n, double limit, double alpha) {
  TORCH_CHECK(act != tb::HA_CLAMPED || limit > 0, "the clamped activation needs a positive limit");
  return tb::GluArgs{(int)act, (float)limit, (float)alpha, f32o(bias, n, "bias")};
}

Tensor glu_rows(const Tensor& gu, int64_t F, int64_t act, const OptT& bias, double limit, double alpha) {
  const bool f32 = rows_of(gu, 0, 2 * F, "gate_up");
  c10::cuda::CUDAGuard guard(gu.device());
  Tensor out = torch::empty({gu.size(0), F}, gu.options());
  tb::launch_glu_rows(gu.data_ptr(), gu.stride(0), out.data_ptr(), F, f32, (int)gu.size(0), (int)F, glu_args(act, bias, 2 * F, limit, alpha),
                      cur_stream());
  return out;
}

const long long* ids_of(const Tensor& ids, int64_t n) {
  TORCH_CHECK(ids.is_cuda() && ids.scalar_type() == at::kLong && ids.is_contiguous() && ids.numel() >= n, "ids: contiguous CUDA int64 expected");
  return reinterpret_cast<const long long*>(ids.data_ptr<int64_t>());
}

Tensor side_rows(const Tensor& gate, const Tensor& table, const Tensor& ids, int64_t col0, int64_t act) {
  const int64_t rows = gate.size(0), dim = gate.size(1);
  const bool f32 = rows_of(gate, rows, dim, "gate");
  TORCH_CHECK(rows_of(table, 0, col0 + dim, "table") == f32, "side_rows: one dtype expected");
  c10::cuda::CUDAGuard guard(gate.device());
  Tensor out = torch::empty({rows, dim}, gate.options());
  tb::launch_side_rows(gate.data_ptr(), gate.stride(0), table.data_ptr(), table.stride(0), ids_of(ids, rows), (int)table.size(0), (int)col0,
                       out.data_ptr(), f32, (int)rows, (int)dim, (int)act, cur_stream());
  return out;
}

void add_norm(Tensor& x, const Tensor& y, const OptT& bias, const Tensor& post_w, double post_eps, int64_t post_kind, const OptT& out,
              const OptT& pre_w, double pre_eps, int64_t pre_kind) {
  TORCH_CHECK(x.is_cuda() && x.dim() == 2 && x.scalar_type() == at::kFloat && x.is_contiguous(), "x: contiguous CUDA fp32 rows expected");
  const int64_t rows = x.size(0), W = x.size(1);
  tb::AddNormArgs a{};
  a.x = x.data_ptr<float>();
  a.y_f32 = rows_of(y, rows, W, "y");
  a.y = y.data_ptr(); a.ldy = y.stride(0);
  a.bias = f32o(bias, W, "bias");
  a.post_w = f32v(post_w, W, "post_w");
  a.pre_w = f32o(pre_w, W, "pre_w");
  a.out_f32 = true;
  if (out.has_value() && out->defined()) {
    a.out_f32 = rows_of(*out, rows, W, "out");
    TORCH_CHECK(out->is_contiguous(), "out: contiguous rows expected");
    a.out = out->data_ptr();
  }
  a.rows = (int)rows; a.W = (int)W;
  a.post_kind = (int)post_kind; a.pre_kind = (int)pre_kind;
  a.post_eps = (float)post_eps; a.pre_eps = (float)pre_eps;
  c10::cuda::CUDAGuard guard(x.device());
  tb::launch_add_norm(a, cur_stream());
}

Tensor rotation_rows(const Tensor& freqs, double amplitude, int64_t T, int64_t pos, const OptT& pos_dev) {
  const int64_t n = freqs.numel();
  c10::cuda::CUDAGuard guard(freqs.device());
  Tensor out = torch::empty({T, 2 * n}, freqs.options().dtype(at::kFloat));
  tb::launch_rotation_rows(f64v(freqs, n, "freqs"), (int)n, (float)amplitude, out.data_ptr<float>(), (int)T, pos_of(pos, pos_dev), cur_stream());
  return out;
}

void gated_norm(const Tensor& y, const Tensor& gate, const OptT& w, Tensor& out, int64_t inner, int64_t groups, double eps,
                int64_t order, double scale) {
  const int64_t rows = y.size(0);
  const bool f32 = rows_of(y, rows, inner, "y");
  TORCH_CHECK(rows_of(gate, rows, inner, "gate") == f32 && rows_of(out, rows, inner, "out") == f32, "gated_norm: one dtype expected");
  TORCH_CHECK(groups > 0 && inner % groups == 0, "gated_norm: parts must divide the width");
  const int64_t part = inner / groups;
  const bool weighted = w.has_value() && w->defined();
  TORCH_CHECK(!weighted || w->numel() == inner || w->numel() == part, "gated_norm: one weight per channel or per position of a part");
  c10::cuda::CUDAGuard guard(y.device());
  tb::launch_gated_norm(y.data_ptr(), y.stride(0), gate.data_ptr(), gate.stride(0), f32o(w, 0, "w"), weighted ? (int)w->numel() : (int)part,
                        out.data_ptr(), out.stride(0), f32, (int)rows, (int)inner, (int)groups, (float)eps, (int)order, (float)scale,
                        cur_stream());
}

Tensor causal_conv(const Tensor& u, const Tensor& w, const OptT& bias, const Tensor& ring_in, Tensor& ring_out, int64_t B, int64_t T,
                   int64_t pos, const OptT& pos_dev) {
  TORCH_CHECK(w.dim() == 2, "w: [channels, taps] expected");
  const int64_t C = w.size(0), taps = w.size(1);
  const bool f32 = rows_of(u, B * T, C, "u");
  TORCH_CHECK(ring_in.numel() == B * taps * C && ring_out.numel() == B * taps * C, "ring: [B, taps, C] expected");
  c10::cuda::CUDAGuard guard(u.device());
  Tensor out = torch::empty({B * T, (C + 7) / 8 * 8}, u.options());
  tb::launch_causal_conv(u.data_ptr(), u.stride(0), f32v(w, C * taps, "w"), f32o(bias, C, "bias"), f32v(ring_in, 0, "ring_in"),
                         const_cast<float*>(f32v(ring_out, 0, "ring_out")), out.data_ptr(), out.stride(0), f32, (int)B, (int)T, (int)C,
                         (int)taps, pos_of(pos, pos_dev), cur_stream());
  return out;
}

// q, k, v, a, b: column views of row matrices; state [B, H, Dk, Dv] fp32 in place
void fill_recurrent(tb::RecurrentArgs& r, const Tensor& q, const Tensor& k, const Tensor& v, const Tensor& a, const OptT& b,
                    const Tensor& A_log, const Tensor& dt_bias, const OptT& D, Tensor& state, Tensor& out, int64_t B, int64_t T,
                    int64_t KG, int64_t kind, double unit_eps) {
  TORCH_CHECK(state.dim() == 4 && state.is_cuda() && state.scalar_type() == at::kFloat && state.is_contiguous() && state.size(0) == B,
              "state: contiguous CUDA fp32 [B, H, Dk, Dv] expected");
  const int64_t H = state.size(1), Dk = state.size(2), Dv = state.size(3), rows = B * T;
  TORCH_CHECK(KG > 0 && H % KG == 0, "heads must be a multiple of the key groups");
  r.f32 = rows_of(q, rows, KG * Dk, "q");
  TORCH_CHECK(rows_of(k, rows, KG * Dk, "k") == r.f32 && rows_of(v, rows, H * Dv, "v") == r.f32 && rows_of(a, rows, H, "a") == r.f32 &&
                  rows_of(out, rows, H * Dv, "out") == r.f32,
              "recurrent: one dtype expected");
  r.q = q.data_ptr(); r.k = k.data_ptr(); r.v = v.data_ptr(); r.a = a.data_ptr(); r.b = nullptr;
  r.ldq = q.stride(0); r.ldk = k.stride(0); r.ldv = v.stride(0); r.lda = a.stride(0); r.ldb = 0;
  if (kind == tb::RK_DELTA) {
    TORCH_CHECK(b.has_value() && b->defined() && rows_of(*b, rows, H, "b") == r.f32, "delta: b is needed");
    r.b = b->data_ptr();
    r.ldb = b->stride(0);
    r.D = nullptr;
  } else {
    TORCH_CHECK(D.has_value() && D->defined(), "mamba2: D is needed");
    r.D = f32v(*D, H, "D");
  }
  r.A_log = f32v(A_log, H, "A_log");
  r.dt_bias = f32v(dt_bias, H, "dt_bias");
  r.state = state.data_ptr<float>();
  r.out = out.data_ptr();
  r.ldo = out.stride(0);
  r.B = (int)B; r.T = (int)T; r.H = (int)H; r.KG = (int)KG; r.Dk = (int)Dk; r.Dv = (int)Dv;
  r.rows = T;
  r.kind = (int)kind;
  r.unit_eps = (float)unit_eps;
}

void recurrent(const Tensor& q, const Tensor& k, const Tensor& v, const Tensor& a, const OptT& b, const Tensor& A_log,
               const Tensor& dt_bias, const OptT& D, Tensor& state, Tensor& out, int64_t B, int64_t T, int64_t KG, int64_t kind,
               double unit_eps, bool chunked, const OptT& status) {
  tb::RecurrentArgs r{};
  fill_recurrent(r, q, k, v, a, b, A_log, dt_bias, D, state, out, B, T, KG, kind, unit_eps);
  c10::cuda::CUDAGuard guard(q.device());
  if (!chunked || !tb::chunk_scan_supported(r)) {
    tb::launch_recurrent(r, cur_stream());
    return;
  }
  // prompts longer than the scratch budget go in parts: the state carries over
  constexpr int64_t budget = 1024ll << 20;
  tb::RecurrentArgs part = r;
  int64_t per = (T + 63) / 64 * 64;
  auto scratch_of = [](const tb::RecurrentArgs& x) { return tb::ssd_tc_supported(x) ? tb::ssd_tc_scratch(x) : tb::chunk_scan_scratch(x); };
  while (per > 4096 && (part.T = (int)std::min(per, T), scratch_of(part)) > budget) per = (per / 2 + 127) / 128 * 128;
  int* st = status_of(status);
  Tensor scratch;
  for (int64_t t = 0; t < T; t += per) {
    part.T = (int)std::min(per, T - t);
    auto at = [&](const void* p, int64_t ld) { return static_cast<const char*>(p) + t * ld * 2; };
    part.q = at(r.q, r.ldq); part.k = at(r.k, r.ldk); part.v = at(r.v, r.ldv); part.a = at(r.a, r.lda);
    if (r.b != nullptr) part.b = at(r.b, r.ldb);
    part.out = const_cast<char*>(at(r.out, r.ldo));
    if (!tb::chunk_scan_supported(part)) {  // a short rest
      tb::launch_recurrent(part, cur_stream());
      continue;
    }
    const int64_t need = scratch_of(part);
    if (!scratch.defined() || scratch.numel() < need) scratch = torch::empty({need}, q.options().dtype(at::kByte));
    if (tb::ssd_tc_supported(part)) tb::launch_ssd_tc(part, scratch.data_ptr(), st, cur_stream());
    else tb::launch_chunk_scan(part, scratch.data_ptr(), cur_stream());
  }
}

// q, k, v: column views of row matrices; rot [T, 2 n]; state [B, H, Dk, Dv] fp32 in place
void retention(const Tensor& q, const Tensor& k, const Tensor& v, const Tensor& rot, const Tensor& decay, Tensor& state, Tensor& out, int64_t B,
               int64_t T, bool chunked, const OptT& status) {
  TORCH_CHECK(state.dim() == 4 && state.is_cuda() && state.scalar_type() == at::kFloat && state.is_contiguous() && state.size(0) == B,
              "state: contiguous CUDA fp32 [B, H, Dk, Dv] expected");
  const int64_t H = state.size(1), Dk = state.size(2), Dv = state.size(3), rows = B * T;
  tb::RecurrentArgs r{};
  r.f32 = rows_of(q, rows, H * Dk, "q");
  TORCH_CHECK(rows_of(k, rows, H * Dk, "k") == r.f32 && rows_of(v, rows, H * Dv, "v") == r.f32 && rows_of(out, rows, H * Dv, "out") == r.f32,
              "retention: one dtype expected");
  TORCH_CHECK(rot.dim() == 2 && rot.size(0) == T && rot.size(1) <= Dk && rot.size(1) % 2 == 0, "retention: rotation rows");
  r.q = q.data_ptr(); r.k = k.data_ptr(); r.v = v.data_ptr();
  r.ldq = q.stride(0); r.ldk = k.stride(0); r.ldv = v.stride(0);
  r.state = state.data_ptr<float>();
  r.out = out.data_ptr(); r.ldo = out.stride(0);
  r.B = (int)B; r.T = (int)T; r.H = r.KG = (int)H; r.Dk = (int)Dk; r.Dv = (int)Dv;
  r.rows = T;
  r.kind = tb::RK_RETENTION;
  r.rot = f32v(rot, T * rot.size(1), "rotation rows");
  r.rot_dims = (int)rot.size(1);
  r.decay = f64v(decay, H, "decay");
  c10::cuda::CUDAGuard guard(q.device());
  if (!chunked || !tb::retention_tc_supported(r)) {
    tb::launch_recurrent(r, cur_stream());
    return;
  }
  // prompts longer than the scratch budget go in parts: the state carries over
  constexpr int64_t budget = 1024ll << 20;
  tb::RecurrentArgs part = r;
  int64_t per = (T + 127) / 128 * 128;
  while (per > 2048 && (part.T = (int)std::min(per, T), tb::retention_tc_scratch(part)) > budget) per = (per / 2 + 127) / 128 * 128;
  Tensor scratch;
  for (int64_t t = 0; t < T; t += per) {
    part.T = (int)std::min(per, T - t);
    auto at = [&](const void* p, int64_t ld) { return static_cast<const char*>(p) + t * ld * 2; };
    part.q = at(r.q, r.ldq); part.k = at(r.k, r.ldk); part.v = at(r.v, r.ldv);
    part.out = const_cast<char*>(at(r.out, r.ldo));
    part.rot = r.rot + t * r.rot_dims;
    if (!tb::retention_tc_supported(part)) {  // a short rest
      tb::launch_recurrent(part, cur_stream());
      continue;
    }
    const int64_t need = tb::retention_tc_scratch(part);
    if (!scratch.defined() || scratch.numel() < need) scratch = torch::empty({need}, q.options().dtype(at::kByte));
    tb::launch_retention_tc(part, scratch.data_ptr(), status_of(status), cur_stream());
  }
}

bool cache_of(const Tensor& c, int64_t B, int64_t G, int64_t d, const char* n) {
  TORCH_CHECK(c.is_cuda() && c.dim() == 4 && c.is_contiguous() && c.size(0) == B && c.size(1) == G && c.size(3) >= d && c.size(3) % 8 == 0,
              n, ": contiguous CUDA [B, groups, capacity, padded head] expected");
  TORCH_CHECK(c.scalar_type() == at::kFloat || c.scalar_type() == at::kBFloat16, n, ": fp32 or bf16 expected");
  return c.scalar_type() == at::kFloat;
}

Tensor attn_prep(const Tensor& proj, int64_t col_q, int64_t col_k, int64_t col_v, const OptT& q_w, const OptT& k_w, double eps,
                 const Tensor& freqs, Tensor& kc, Tensor& vc, int64_t B, int64_t T, int64_t H, int64_t D, int64_t E, int64_t pos,
                 const OptT& pos_dev) {
  const int64_t G = kc.size(1);
  const bool f32 = rows_of(proj, B * T, std::max(col_q + H * D, std::max(col_k + G * D, col_v + G * E)), "proj");
  TORCH_CHECK(cache_of(kc, B, G, D, "k cache") == f32 && cache_of(vc, B, G, E, "v cache") == f32, "attn_prep: one dtype expected");
  TORCH_CHECK(kc.size(2) == vc.size(2) && 2 * freqs.numel() <= D && H % G == 0, "attn_prep: shapes");
  if (!(pos_dev.has_value() && pos_dev->defined())) TORCH_CHECK(pos + T <= kc.size(2), "attn_prep: the cache is too small");
  c10::cuda::CUDAGuard guard(proj.device());
  Tensor q = torch::empty({B, H, T, kc.size(3)}, proj.options());
  tb::AttnPrepArgs a{};
  a.proj = proj.data_ptr(); a.ld = proj.stride(0);
  a.col_q = (int)col_q; a.col_k = (int)col_k; a.col_v = (int)col_v;
  a.q_w = f32o(q_w, D, "q_w"); a.k_w = f32o(k_w, D, "k_w");
  a.eps = (float)eps;
  a.rot_dims = (int)(2 * freqs.numel());
  a.freqs = f64v(freqs, 0, "freqs");
  a.q = q.data_ptr(); a.kc = kc.data_ptr(); a.vc = vc.data_ptr();
  a.B = (int)B; a.T = (int)T; a.H = (int)H; a.G = (int)G; a.D = (int)D; a.E = (int)E;
  a.cap = (int)kc.size(2); a.pitch_k = (int)kc.size(3); a.pitch_v = (int)vc.size(3);
  a.pos = pos_of(pos, pos_dev);
  a.f32 = f32;
  tb::launch_attn_prep(a, cur_stream());
  return q;
}

tb::AttnArgs attn_args(const Tensor& q, const Tensor& kc, const Tensor& vc, const OptT& sink, Tensor& out, int64_t D, int64_t E,
                       double scale, double out_scale, int64_t pos, const OptT& pos_dev) {
  TORCH_CHECK(q.is_cuda() && q.dim() == 4 && q.is_contiguous(), "q: contiguous CUDA [B, H, T, padded head] expected");
  tb::AttnArgs a{};
  a.B = (int)q.size(0); a.H = (int)q.size(1); a.T = (int)q.size(2);
  a.G = (int)kc.size(1); a.D = (int)D; a.E = (int)E;
  a.f32 = cache_of(kc, a.B, a.G, D, "k cache");
  TORCH_CHECK(cache_of(vc, a.B, a.G, E, "v cache") == a.f32 && (q.scalar_type() == at::kFloat) == a.f32 && q.size(3) == kc.size(3) &&
                  vc.size(2) == kc.size(2) && a.H % a.G == 0,
              "attention: shapes or dtypes differ");
  TORCH_CHECK(rows_of(out, (int64_t)a.B * a.T, (int64_t)a.H * E, "out") == a.f32, "attention: one dtype expected");
  if (!(pos_dev.has_value() && pos_dev->defined())) TORCH_CHECK(pos + a.T <= kc.size(2), "attention: the cache is too small");
  auto operand = [](const Tensor& t) { return tb::AttnOperand{t.data_ptr(), t.stride(2), t.stride(1), t.stride(0)}; };
  a.q = operand(q); a.k = operand(kc); a.v = operand(vc);
  a.sink = f32o(sink, a.H, "sink");
  a.out = out.data_ptr(); a.ldo = out.stride(0);
  a.rows = (int)kc.size(2);
  a.scale = (float)scale; a.out_scale = (float)out_scale;
  a.pos = pos_of(pos, pos_dev);
  return a;
}

void attn_simple(const Tensor& q, const Tensor& kc, const Tensor& vc, const OptT& sink, Tensor& out, int64_t D, int64_t E, double scale,
                 double out_scale, int64_t pos, const OptT& pos_dev) {
  tb::AttnArgs a = attn_args(q, kc, vc, sink, out, D, E, scale, out_scale, pos, pos_dev);
  c10::cuda::CUDAGuard guard(q.device());
  tb::launch_attn_simple(a, cur_stream());
}

// the tensor-core kernel where it takes the shape, else the fp32 CUDA-core kernel
void attention(const Tensor& q, const Tensor& kc, const Tensor& vc, const OptT& sink, Tensor& out, int64_t D, int64_t E, double scale,
               double out_scale, int64_t pos, const OptT& pos_dev, const OptT& status) {
  tb::AttnArgs a = attn_args(q, kc, vc, sink, out, D, E, scale, out_scale, pos, pos_dev);
  c10::cuda::CUDAGuard guard(q.device());
  int* st = status_of(status);
  if (tb::attn_tc_supported(a)) tb::launch_attn_tc(a, st, cur_stream());
  else tb::launch_attn_simple(a, cur_stream());
}

// Query heads of [Dp | Rp] columns of proj, cache [B, 1, capacity, rank_p + Rp]
void check_latent(const Tensor& proj, int64_t rows, int64_t col_q, int64_t H, int64_t Dp, int64_t Rp, int64_t col_c, const OptT& norm_w,
                  const Tensor& cache, int64_t B, int64_t rank, int64_t rank_p, int64_t R) {
  rows_of(proj, rows, std::max(col_q + H * (Dp + Rp), col_c + rank_p + Rp), "proj");
  cache_of(cache, B, 1, rank_p + Rp, "latent cache");
  TORCH_CHECK(cache.size(3) == rank_p + Rp && rank > 0 && rank <= rank_p && R >= 0 && R <= Rp && R % 2 == 0 && Dp % 8 == 0 && Rp % 8 == 0 &&
                  rank_p % 8 == 0 && col_q >= 0,
              "latent attention: shapes");
  if (col_c >= 0) TORCH_CHECK(norm_w.has_value() && norm_w->defined(), "latent attention: own latents need their norm");
}

void latent_prep(Tensor& proj, int64_t col_q, int64_t H, int64_t Dp, int64_t Rp, int64_t col_c, const OptT& norm_w, double eps, Tensor& cache,
                 int64_t rank, int64_t rank_p, int64_t R, const Tensor& rot, int64_t B, int64_t T, int64_t pos, const OptT& pos_dev) {
  check_latent(proj, B * T, col_q, H, Dp, Rp, col_c, norm_w, cache, B, rank, rank_p, R);
  tb::LatentPrepArgs a{};
  a.f32 = proj.scalar_type() == at::kFloat;
  TORCH_CHECK((cache.scalar_type() == at::kFloat) == a.f32, "latent_prep: one dtype expected");
  TORCH_CHECK(rot.dim() == 2 && rot.size(0) == T && rot.size(1) == R, "latent_prep: rotation rows");
  if (!(pos_dev.has_value() && pos_dev->defined())) TORCH_CHECK(pos + T <= cache.size(2), "latent_prep: the cache is too small");
  a.proj = proj.data_ptr(); a.ld = proj.stride(0);
  a.col_q = (int)col_q; a.H = (int)H; a.Dp = (int)Dp; a.Rp = (int)Rp; a.col_c = (int)col_c;
  a.norm_w = f32o(norm_w, rank, "norm_w");
  a.eps = (float)eps;
  a.cache = cache.data_ptr(); a.cap = (int)cache.size(2);
  a.rank = (int)rank; a.rank_p = (int)rank_p; a.R = (int)R;
  a.rot = f32v(rot, T * R, "rotation rows");
  a.B = (int)B; a.T = (int)T;
  a.pos = pos_of(pos, pos_dev);
  c10::cuda::CUDAGuard guard(proj.device());
  tb::launch_latent_prep(a, cur_stream());
}

// Heads g0 .. g0 + Hn - 1 of a layer, whose keys and values are expanded in kv [B, n, Hn (Dp + Ep)].
void latent_attention(const Tensor& proj, int64_t col_q, int64_t col_g, const Tensor& cache, const Tensor& kv, const OptT& sink, Tensor& out,
                      int64_t g0, int64_t Hn, int64_t B, int64_t T, int64_t Dp, int64_t Rp, int64_t rank_p, int64_t D, int64_t R, int64_t E,
                      double scale, double out_scale, int64_t pos, const OptT& pos_dev, const OptT& status) {
  const int64_t Ep = (E + 7) / 8 * 8;
  check_latent(proj, B * T, col_q, g0 + Hn, Dp, Rp, -1, c10::nullopt, cache, B, rank_p, rank_p, R);
  TORCH_CHECK(kv.is_cuda() && kv.dim() == 3 && kv.size(0) == B && kv.is_contiguous() && kv.size(2) == Hn * (Dp + Ep) && D <= Dp,
              "latent_attention: expanded keys and values [B, n, heads * (key + value)] expected");
  TORCH_CHECK(kv.scalar_type() == proj.scalar_type() && cache.scalar_type() == proj.scalar_type() && out.scalar_type() == proj.scalar_type(),
              "latent_attention: one dtype expected");
  const int64_t n = kv.size(1), size = kv.element_size();
  TORCH_CHECK(n <= cache.size(2), "latent_attention: more keys than cached rows");
  const bool on_device = pos_dev.has_value() && pos_dev->defined();
  TORCH_CHECK(on_device ? n == cache.size(2) : pos + T <= n, "latent_attention: ", n, " keys for ", T, " tokens after ", pos);
  rows_of(out, B * T, (g0 + Hn) * E, "out");
  TORCH_CHECK(col_g < 0 || col_g + g0 + Hn <= proj.size(1), "latent_attention: gate columns");
  auto at = [&](const Tensor& t, int64_t off) { return static_cast<char*>(t.data_ptr()) + off * size; };
  const int64_t ld = proj.stride(0), head = Dp + Rp;
  tb::AttnArgs a{};
  a.q = {at(proj, col_q + g0 * head), ld, head, T * ld};
  a.q2 = {at(proj, col_q + g0 * head + Dp), ld, head, T * ld};
  a.k = {kv.data_ptr(), kv.stride(1), Dp + Ep, kv.stride(0)};
  a.v = {at(kv, Dp), kv.stride(1), Dp + Ep, kv.stride(0)};
  a.k2 = {at(cache, rank_p), cache.stride(2), 0, cache.stride(0)};
  a.sink = f32o(sink, g0 + Hn, "sink");
  if (a.sink != nullptr) a.sink += g0;
  if (col_g >= 0) a.gate = at(proj, col_g + g0);
  a.ldg = ld;
  a.out = at(out, g0 * E); a.ldo = out.stride(0);
  a.B = (int)B; a.T = (int)T; a.H = a.G = (int)Hn; a.D = (int)D; a.E = (int)E; a.R = (int)R;
  a.rows = (int)n;
  a.scale = (float)scale; a.out_scale = (float)out_scale;
  a.pos = pos_of(pos, pos_dev);
  a.f32 = proj.scalar_type() == at::kFloat;
  c10::cuda::CUDAGuard guard(proj.device());
  if (tb::attn_tc_supported(a)) tb::launch_attn_tc(a, status_of(status), cur_stream());
  else tb::launch_attn_simple(a, cur_stream());
}

void latent_step(const Tensor& proj, int64_t col_q, int64_t col_g, int64_t col_c, const OptT& norm_w, double eps, Tensor& cache, const Tensor& up,
                 const Tensor& freqs, double amplitude, const OptT& sink, Tensor& qa, Tensor& part, Tensor& out, int64_t rank, int64_t D,
                 int64_t R, int64_t E, double scale, double out_scale, int64_t pos, const OptT& pos_dev) {
  const int64_t B = proj.size(0), Dp = (D + 7) / 8 * 8, Ep = (E + 7) / 8 * 8, Rp = (R + 7) / 8 * 8;
  TORCH_CHECK(up.is_cuda() && up.dim() == 3 && up.is_contiguous() && up.size(1) == Dp + Ep, "latent_step: expansion [H, key + value, latent] expected");
  const int64_t H = up.size(0), rank_p = up.size(2);
  TORCH_CHECK(rows_of(proj, B, 0, "proj"), "latent_step: fp32 projection rows expected");
  check_latent(proj, B, col_q, H, Dp, Rp, col_c, norm_w, cache, B, rank, rank_p, R);
  TORCH_CHECK(cache.scalar_type() == up.scalar_type() && 2 * freqs.numel() == R && (col_g < 0 || col_g + H <= proj.size(1)), "latent_step: shapes");
  if (!(pos_dev.has_value() && pos_dev->defined())) TORCH_CHECK(pos < cache.size(2), "latent_step: the cache is full");
  tb::LatentStepArgs a{};
  a.proj = proj.data_ptr<float>(); a.ld = proj.stride(0);
  a.col_q = (int)col_q; a.col_g = (int)col_g; a.col_c = (int)col_c;
  a.H = (int)H; a.D = (int)D; a.Dp = (int)Dp; a.R = (int)R; a.Rp = (int)Rp; a.E = (int)E; a.Ep = (int)Ep; a.rank = (int)rank; a.rank_p = (int)rank_p;
  a.norm_w = f32o(norm_w, rank, "norm_w");
  a.eps = (float)eps;
  a.cache = cache.data_ptr(); a.up = up.data_ptr();
  a.f32 = up.scalar_type() == at::kFloat;
  a.cap = (int)cache.size(2);
  a.freqs = f64v(freqs, R / 2, "freqs");
  a.amplitude = (float)amplitude;
  a.sink = f32o(sink, H, "sink");
  a.qa = const_cast<float*>(f32v(qa, B * H * (rank_p + Rp), "qa"));
  TORCH_CHECK(part.dim() == 4 && part.size(0) == B && part.size(1) == H && part.size(2) >= 1 && part.size(2) <= 128, "latent_step: split results");
  a.splits = (int)part.size(2);
  a.part = const_cast<float*>(f32v(part, B * H * a.splits * tb::step_part_stride((int)rank_p), "part"));
  TORCH_CHECK(rows_of(out, B, H * E, "out"), "latent_step: fp32 output expected");
  a.out = out.data_ptr<float>(); a.ldo = out.stride(0);
  a.scale = (float)scale; a.out_scale = (float)out_scale;
  a.B = (int)B;
  a.pos = pos_of(pos, pos_dev);
  c10::cuda::CUDAGuard guard(proj.device());
  tb::launch_latent_step(a, cur_stream());
}

// segments: dicts with x [B, n], kind, and what the kind needs
void gemv(const std::vector<py::dict>& segs, const Tensor& W, Tensor& y, int64_t epilogue, int64_t act, const OptT& bias, double limit,
          double alpha, const OptT& table, const OptT& ids, int64_t col0) {
  TORCH_CHECK(segs.size() >= 1 && segs.size() <= 2, "gemv: one or two input segments");
  tb::GemvArgs g{};
  g.nseg = (int)segs.size();
  g.B = (int)y.size(0);
  g.N = (int)y.size(1);
  TORCH_CHECK(y.is_cuda() && y.dim() == 2 && y.scalar_type() == at::kFloat && y.stride(1) == 1, "y: CUDA fp32 rows expected");
  std::vector<Tensor> keep;
  for (size_t i = 0; i < segs.size(); ++i) {
    const py::dict& d = segs[i];
    tb::GemvSegment& s = g.seg[i];
    Tensor x = d["x"].cast<Tensor>();
    TORCH_CHECK(rows_of(x, g.B, 0, "x"), "gemv: fp32 input rows expected");
    s.x = x.data_ptr<float>(); s.ld = x.stride(0); s.n = (int)x.size(1);
    s.kind = d["kind"].cast<int>();
    s.scale = d.contains("scale") ? d["scale"].cast<float>() : 1.f;
    s.groups = 1; s.w_period = s.n;
    if (s.kind != 0) {
      s.norm_kind = d["norm"].cast<int>();
      s.eps = d["eps"].cast<float>();
      const bool weighted = !d["w"].is_none();
      TORCH_CHECK(weighted || s.kind != 1, "gemv: norm weight");
      if (weighted) {
        Tensor w = d["w"].cast<Tensor>();
        s.w = f32v(w, w.numel(), "w");
        s.w_period = (int)w.numel();
      }
      if (s.kind == 2) {
        s.groups = d["groups"].cast<int>();
        TORCH_CHECK(s.groups > 0 && s.n % s.groups == 0, "gemv: gated norm parts");
        if (!weighted) s.w_period = s.n / s.groups;
        TORCH_CHECK(s.w_period == s.n || s.w_period == s.n / s.groups, "gemv: gated norm weight");
        Tensor gate = d["gate"].cast<Tensor>();
        TORCH_CHECK(rows_of(gate, g.B, s.n, "gate"), "gemv: fp32 gate rows expected");
        s.gate = gate.data_ptr<float>(); s.ldg = gate.stride(0);
      } else {
        TORCH_CHECK(s.w_period == s.n, "gemv: norm weight");
      }
      if (s.kind == 3) {
        TORCH_CHECK(i == 0 && segs.size() == 1, "gemv: a sum is the only segment");
        Tensor add = d["y"].cast<Tensor>();
        TORCH_CHECK(rows_of(add, g.B, s.n, "y"), "gemv: fp32 rows to add expected");
        s.y = add.data_ptr<float>(); s.ldy = add.stride(0);
        if (!d["bias"].is_none()) s.y_bias = f32v(d["bias"].cast<Tensor>(), s.n, "bias");
        s.post_w = f32v(d["post_w"].cast<Tensor>(), s.n, "post_w");
        s.post_kind = d["post_norm"].cast<int>();
        s.post_eps = d["post_eps"].cast<float>();
        if (!d["x_out"].is_none()) {
          Tensor xo = d["x_out"].cast<Tensor>();
          s.x_out = const_cast<float*>(f32v(xo, (int64_t)g.B * s.n, "x_out"));
          TORCH_CHECK(s.x_out != s.x, "gemv: the sum goes to rows of its own");
        }
      }
    }
    g.K += s.n;
  }
  g.f32 = rows_of(W, epilogue == 2 ? 2 * g.N : g.N, g.K, "W");
  TORCH_CHECK(W.size(1) == g.K, "gemv: W has ", W.size(1), " columns, the input ", g.K);
  g.W = W.data_ptr(); g.ldw = W.stride(0);
  g.y = y.data_ptr<float>(); g.ldy = y.stride(0);
  g.epilogue = (int)epilogue;
  g.glu = glu_args(act, bias, epilogue == 2 ? 2 * g.N : g.N, limit, alpha);
  if (epilogue == 3) {
    TORCH_CHECK(table.has_value() && ids.has_value(), "gemv: the side epilogue needs a table and token ids");
    TORCH_CHECK(rows_of(*table, 0, col0 + g.N, "table") == g.f32 && col0 >= 0, "gemv: the table has W's dtype");
    g.table = table->data_ptr(); g.ldt = table->stride(0);
    g.ids = ids_of(*ids, g.B);
    g.V = (int)table->size(0); g.col0 = (int)col0;
  }
  c10::cuda::CUDAGuard guard(W.device());
  tb::launch_gemv(g, cur_stream());
}

tb::StepRecurrent step_recurrent(const py::dict& d, const Tensor& proj, int64_t B) {
  tb::StepRecurrent r{};
  Tensor state = d["state"].cast<Tensor>(), out = d["out"].cast<Tensor>();
  TORCH_CHECK(state.dim() == 4 && state.size(0) == B, "step: state");
  r.H = (int)state.size(1); r.Dk = (int)state.size(2); r.Dv = (int)state.size(3);
  r.kind = d["kind"].cast<int>();
  r.proj = proj.data_ptr<float>(); r.ld = proj.stride(0);
  r.state = const_cast<float*>(f32v(state, 0, "state"));
  TORCH_CHECK(rows_of(out, B, (int64_t)r.H * r.Dv, "out"), "step: fp32 output expected");
  r.out = out.data_ptr<float>(); r.ldo = out.stride(0);
  if (r.kind == tb::RK_RETENTION) {
    r.KG = r.H;
    r.col_q = d["col_q"].cast<int>(); r.col_k = d["col_k"].cast<int>(); r.col_v = d["col_v"].cast<int>();
    TORCH_CHECK(r.col_q + r.H * r.Dk <= proj.size(1) && r.col_k + r.H * r.Dk <= proj.size(1) && r.col_v + r.H * r.Dv <= proj.size(1),
                "step: columns outside the projection");
    Tensor freqs = d["freqs"].cast<Tensor>();
    r.rot_dims = (int)(2 * freqs.numel());
    TORCH_CHECK(r.rot_dims <= r.Dk, "step: rotated dimensions");
    r.freqs = f64v(freqs, 0, "freqs");
    r.decay = f64v(d["decay"].cast<Tensor>(), r.H, "decay");
    r.amplitude = d["amplitude"].cast<float>();
    return r;
  }
  Tensor ring = d["ring"].cast<Tensor>(), cw = d["conv_w"].cast<Tensor>();
  r.KG = d["key_groups"].cast<int>();
  r.C = (int)cw.size(0); r.taps = (int)cw.size(1);
  r.col_u = d["col_u"].cast<int>(); r.col_a = d["col_a"].cast<int>(); r.col_b = d["col_b"].cast<int>();
  r.off_q = d["off_q"].cast<int>(); r.off_k = d["off_k"].cast<int>(); r.off_v = d["off_v"].cast<int>();
  TORCH_CHECK(r.KG > 0 && r.H % r.KG == 0 && r.off_q + r.KG * r.Dk <= r.C && r.off_k + r.KG * r.Dk <= r.C && r.off_v + r.H * r.Dv <= r.C &&
                  r.col_u + r.C <= proj.size(1) && r.col_a + r.H <= proj.size(1) && (r.kind != tb::RK_DELTA || r.col_b + r.H <= proj.size(1)),
              "step: columns outside the projection");
  r.conv_w = f32v(cw, (int64_t)r.C * r.taps, "conv_w");
  if (d.contains("conv_b") && !d["conv_b"].is_none()) r.conv_b = f32v(d["conv_b"].cast<Tensor>(), r.C, "conv_b");
  r.ring = const_cast<float*>(f32v(ring, B * r.taps * r.C, "ring"));
  r.A_log = f32v(d["A_log"].cast<Tensor>(), r.H, "A_log");
  r.dt_bias = f32v(d["dt_bias"].cast<Tensor>(), r.H, "dt_bias");
  if (r.kind == tb::RK_MAMBA2) r.D = f32v(d["D"].cast<Tensor>(), r.H, "D");
  r.unit_eps = d["unit_eps"].cast<float>();
  return r;
}

tb::StepAttention step_attention(const py::dict& d, const Tensor& proj, int64_t B, int64_t pos, bool host_pos) {
  tb::StepAttention a{};
  Tensor kc = d["k"].cast<Tensor>(), vc = d["v"].cast<Tensor>(), part = d["part"].cast<Tensor>(), cnt = d["counters"].cast<Tensor>(),
         out = d["out"].cast<Tensor>(), fr = d["freqs"].cast<Tensor>();
  a.H = d["heads"].cast<int>(); a.D = d["dim"].cast<int>(); a.E = d["vdim"].cast<int>();
  a.G = (int)kc.size(1);
  a.cache_f32 = cache_of(kc, B, a.G, a.D, "k cache");
  TORCH_CHECK(cache_of(vc, B, a.G, a.E, "v cache") == a.cache_f32 && vc.size(2) == kc.size(2) && a.H % a.G == 0, "step: caches differ");
  if (host_pos) TORCH_CHECK(pos < kc.size(2), "step: the cache is full");
  a.proj = proj.data_ptr<float>(); a.ld = proj.stride(0);
  a.col_q = d["col_q"].cast<int>(); a.col_k = d["col_k"].cast<int>(); a.col_v = d["col_v"].cast<int>();
  TORCH_CHECK(a.col_q + a.H * a.D <= proj.size(1) && a.col_k + a.G * a.D <= proj.size(1) && a.col_v + a.G * a.E <= proj.size(1),
              "step: columns outside the projection");
  if (!d["q_w"].is_none()) a.q_w = f32v(d["q_w"].cast<Tensor>(), a.D, "q_w");
  if (!d["k_w"].is_none()) a.k_w = f32v(d["k_w"].cast<Tensor>(), a.D, "k_w");
  a.eps = d["eps"].cast<float>();
  a.rot_dims = (int)(2 * fr.numel());
  TORCH_CHECK(a.rot_dims <= a.D, "step: rotated dimensions");
  a.freqs = f64v(fr, 0, "freqs");
  if (!d["sink"].is_none()) a.sink = f32v(d["sink"].cast<Tensor>(), a.H, "sink");
  a.kc = kc.data_ptr(); a.vc = vc.data_ptr();
  a.cap = (int)kc.size(2); a.pitch_k = (int)kc.size(3); a.pitch_v = (int)vc.size(3);
  const int rep = a.H / a.G, rm = tb::step_head_chunk(rep);
  a.splits = d["splits"].cast<int>();
  TORCH_CHECK(a.splits >= 1 && a.splits <= 64, "step: 1 to 64 splits");
  a.part = const_cast<float*>(f32v(part, B * a.H * a.splits * tb::step_part_stride(a.E), "part"));
  TORCH_CHECK(cnt.is_cuda() && cnt.scalar_type() == at::kInt && cnt.is_contiguous() && cnt.numel() >= B * a.G * ((rep + rm - 1) / rm), "step: counters");
  a.counters = cnt.data_ptr<int>();
  TORCH_CHECK(rows_of(out, B, (int64_t)a.H * a.E, "out"), "step: fp32 output expected");
  a.out = out.data_ptr<float>(); a.ldo = out.stride(0);
  a.scale = d["scale"].cast<float>(); a.out_scale = d["out_scale"].cast<float>();
  return a;
}

void mixer_step(const Tensor& proj, const c10::optional<py::dict>& rec, const c10::optional<py::dict>& att, int64_t pos, const OptT& pos_dev) {
  TORCH_CHECK(rows_of(proj, 0, 0, "proj"), "step: fp32 projection rows expected");
  const int64_t B = proj.size(0);
  tb::StepArgs s{};
  s.B = (int)B;
  s.pos = pos_of(pos, pos_dev);
  s.has_rec = rec.has_value();
  s.has_att = att.has_value();
  if (s.has_rec) s.rec = step_recurrent(*rec, proj, B);
  if (s.has_att) s.att = step_attention(*att, proj, B, pos, s.pos.dev == nullptr);
  c10::cuda::CUDAGuard guard(proj.device());
  tb::launch_mixer_step(s, cur_stream());
}

}  // namespace

void register_hybrid(pybind11::module& m) {
  m.def("hybrid_embed_rows", &embed_rows);
  m.def("hybrid_norm_rows", &norm_rows);
  m.def("hybrid_glu_rows", &glu_rows);
  m.def("hybrid_side_rows", &side_rows);
  m.def("hybrid_add_norm", &add_norm);
  m.def("hybrid_rotation_rows", &rotation_rows);
  m.def("hybrid_retention", &retention);
  m.def("hybrid_latent_prep", &latent_prep);
  m.def("hybrid_latent_attention", &latent_attention);
  m.def("hybrid_latent_step", &latent_step);
  m.def("hybrid_latent_step_splits", &tb::latent_step_splits);
  m.def("hybrid_gated_norm", &gated_norm);
  m.def("hybrid_causal_conv", &causal_conv);
  m.def("hybrid_recurrent", &recurrent, pybind11::arg("q"), pybind11::arg("k"), pybind11::arg("v"), pybind11::arg("a"), pybind11::arg("b"),
        pybind11::arg("A_log"), pybind11::arg("dt_bias"), pybind11::arg("D"), pybind11::arg("state"), pybind11::arg("out"), pybind11::arg("B"),
        pybind11::arg("T"), pybind11::arg("key_groups"), pybind11::arg("kind"), pybind11::arg("unit_eps"), pybind11::arg("chunked") = true,
        pybind11::arg("status") = pybind11::none());
  m.def("hybrid_attn_prep", &attn_prep);
  m.def("hybrid_attn_simple", &attn_simple);
  m.def("hybrid_attention", &attention);
  m.def("hybrid_gemv", &gemv);
  m.def("hybrid_mixer_step", &mixer_step);
  m.def("hybrid_step_head_chunk", &tb::step_head_chunk);
  m.def("hybrid_step_part_stride", &tb::step_part_stride);
}
