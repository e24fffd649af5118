// Python bindings of the tcgen05 GEMM family; part of the full extension and of the serving subset.
#include <ATen/cuda/CUDAContext.h>
#include <c10/cuda/CUDAGuard.h>
#include <torch/extension.h>

#include "tc_gemm.cuh"

namespace {

using torch::Tensor;

inline cudaStream_t cur_stream() { return at::cuda::getCurrentCUDAStream().stream(); }
inline const __nv_bfloat16* bf(const Tensor& t) { return reinterpret_cast<const __nv_bfloat16*>(t.data_ptr()); }
inline __nv_bfloat16* bfm(Tensor& t) { return reinterpret_cast<__nv_bfloat16*>(t.data_ptr()); }
inline const __nv_bfloat16* bf_opt(const c10::optional<Tensor>& t) {
  return t.has_value() && t->defined() ? reinterpret_cast<const __nv_bfloat16*>(t->data_ptr()) : nullptr;
}

void check_bf16_cuda(const Tensor& t, const char* name) {
  TORCH_CHECK(t.is_cuda(), name, " must be a CUDA tensor");
  TORCH_CHECK(t.scalar_type() == at::kBFloat16, name, " must be bfloat16");
  // every kernel reads and writes bf16 data in 16-byte vectors: a misaligned base would fault on the device
  TORCH_CHECK((reinterpret_cast<uintptr_t>(t.data_ptr()) & 15) == 0, name, " must start on a 16-byte boundary");
}

// C[b] = alpha * op(A[b]) * op(B[b])^T with the fused epilogue. a: [batch?, M, K] (or [batch?, K, M] when
// a_mn_major), b: [batch?, N, K] (or [batch?, K, N] when b_mn_major). Inner dims must be contiguous.
void tc_gemm(const Tensor& a, const Tensor& b, Tensor& c, bool a_mn_major, bool b_mn_major, int64_t mode, int64_t flags,
             double alpha, const c10::optional<Tensor>& bias, const c10::optional<Tensor>& aux_in,
             const c10::optional<Tensor>& aux_out, const c10::optional<Tensor>& row_scale,
             const c10::optional<Tensor>& tile_group, const c10::optional<Tensor>& group_offsets,
             const c10::optional<Tensor>& status, double beta, const c10::optional<Tensor>& k_runs) {
  check_bf16_cuda(a, "a");
  check_bf16_cuda(b, "b");
  TORCH_CHECK(c.is_cuda(), "c must be CUDA");
  TORCH_CHECK(a.stride(-1) == 1 && b.stride(-1) == 1 && c.stride(-1) == 1, "inner dims must be contiguous");
  c10::cuda::CUDAGuard guard(a.device());
  tb::GemmArgs g{};
  g.A = bf(a);
  g.B = bf(b);
  g.C = c.data_ptr();
  g.a_mn_major = a_mn_major;
  g.b_mn_major = b_mn_major;
  g.mode = (int)mode;
  g.flags = (int)flags;
  if (c.scalar_type() == at::kFloat) g.flags |= tb::GF_OUT_F32;
  else TORCH_CHECK(c.scalar_type() == at::kBFloat16, "c must be bf16 or fp32");
  g.alpha = (float)alpha;
  g.beta = (float)beta;
  const int ad = a.dim(), bd = b.dim(), cd = c.dim();
  TORCH_CHECK(ad >= 2 && bd >= 2 && cd >= 2, "operands must be at least 2-D");
  g.lda = a.stride(-2);
  g.ldb = b.stride(-2);
  g.ldc = c.stride(-2);
  g.strideA = ad == 3 ? a.stride(0) : 0;
  g.strideB = bd == 3 ? b.stride(0) : 0;
  g.strideC = cd == 3 ? c.stride(0) : 0;
  g.batch = cd == 3 ? (int)c.size(0) : 1;
  g.M = (int)c.size(-2);
  g.N = (int)c.size(-1);
  if (mode == tb::GEMM_GROUPED_K) {
    g.K = (int)a.size(-2);  // total rows being reduced over
    TORCH_CHECK(a.size(-2) == b.size(-2), "grouped-K operands must share the row dimension");
    TORCH_CHECK(a.size(-1) == g.M && b.size(-1) == g.N, "grouped-K: c[g] is [a.cols, b.cols]");
  } else {
    g.K = (int)(a_mn_major ? a.size(-2) : a.size(-1));
    const int64_t kb = b_mn_major ? b.size(-2) : b.size(-1);
    TORCH_CHECK(kb == g.K, "reduction dims differ: ", g.K, " vs ", kb);
    const int64_t am = a_mn_major ? a.size(-1) : a.size(-2);
    const int64_t bn = b_mn_major ? b.size(-1) : b.size(-2);
    TORCH_CHECK(am == g.M, "a rows (", am, ") != c rows (", g.M, ")");
    TORCH_CHECK(bn == g.N, "b rows (", bn, ") != c cols (", g.N, ")");
  }
  if (mode == tb::GEMM_GROUPED_M) {
    TORCH_CHECK(bd == 3, "grouped-M: b must be [groups, N, K]");
    g.batch = (int)b.size(0);
    g.strideB = b.stride(0);
  }
  if (bias.has_value() && bias->defined()) {
    check_bf16_cuda(*bias, "bias");
    g.bias = bf(*bias);
    g.bias_stride = bias->dim() == 2 ? bias->stride(0) : 0;
  }
  if (aux_in.has_value() && aux_in->defined()) {
    check_bf16_cuda(*aux_in, "aux_in");
    TORCH_CHECK(aux_in->stride(-2) == g.ldc, "aux_in must share c's layout");
    g.aux_in = bf(*aux_in);
  }
  if (aux_out.has_value() && aux_out->defined()) {
    check_bf16_cuda(*aux_out, "aux_out");
    TORCH_CHECK(aux_out->stride(-2) == g.ldc, "aux_out must share c's layout");
    g.aux_out = reinterpret_cast<__nv_bfloat16*>(aux_out->data_ptr());
  }
  if (row_scale.has_value() && row_scale->defined()) {
    TORCH_CHECK(row_scale->scalar_type() == at::kFloat && row_scale->is_contiguous(), "row_scale must be fp32");
    g.row_scale = row_scale->data_ptr<float>();
  }
  if (tile_group.has_value() && tile_group->defined()) {
    TORCH_CHECK(tile_group->scalar_type() == at::kInt, "tile_group must be int32");
    g.tile_group = tile_group->data_ptr<int>();
  }
  if (group_offsets.has_value() && group_offsets->defined()) {
    TORCH_CHECK(group_offsets->scalar_type() == at::kInt, "group_offsets must be int32");
    g.group_offsets = group_offsets->data_ptr<int>();
  }
  if (status.has_value() && status->defined()) {
    TORCH_CHECK(status->scalar_type() == at::kInt, "status must be int32");
    g.status = status->data_ptr<int>();
  }
  if (k_runs.has_value() && k_runs->defined()) {
    TORCH_CHECK(mode == tb::GEMM_GROUPED_K && g.group_offsets != nullptr, "k_runs belongs to the grouped-K mode");
    TORCH_CHECK(k_runs->is_cuda() && k_runs->scalar_type() == at::kInt && k_runs->is_contiguous() && k_runs->dim() == 2 &&
                    k_runs->size(1) == 2,
                "k_runs must be a contiguous CUDA int32 tensor [runs, 2]");
    g.k_runs = k_runs->data_ptr<int>();
  }
  tb::launch_tc_gemm(g, cur_stream());
}

// SwiGLU over the fused gate/up weight inside the GEMM: h [M, H] = silu(x Wg^T) * (x Wu^T) with w13 = [Wg ; Wu]
// ([2H, K]); gu (optional, [M, 2H]) receives both pre-activations for the backward pass. act: 0 silu, 1 relu, 2 clamped
// (see GemmArgs::glu_act); bias: fp32 [2H] or none (forward only, as the last two activations are).
void tc_gemm_swiglu(const Tensor& x, const Tensor& w13, Tensor& h, const c10::optional<Tensor>& gu, int64_t act,
                    const c10::optional<Tensor>& bias, double limit, double alpha) {
  check_bf16_cuda(x, "x");
  check_bf16_cuda(w13, "w13");
  check_bf16_cuda(h, "h");
  TORCH_CHECK(x.dim() == 2 && w13.dim() == 2 && h.dim() == 2 && x.stride(1) == 1 && w13.stride(1) == 1 && h.stride(1) == 1,
              "tc_gemm_swiglu: 2-D operands with contiguous rows");
  const int64_t M = x.size(0), K = x.size(1), H = h.size(1);
  TORCH_CHECK(w13.size(0) == 2 * H && w13.size(1) == K && h.size(0) == M, "tc_gemm_swiglu: shapes");
  c10::cuda::CUDAGuard guard(x.device());
  tb::GemmArgs g{};
  g.A = bf(x); g.B = bf(w13); g.C = h.data_ptr();
  g.M = (int)M; g.N = (int)H; g.K = (int)K;
  g.lda = x.stride(0); g.ldb = w13.stride(0); g.ldc = h.stride(0);
  g.batch = 1; g.mode = tb::GEMM_DENSE; g.flags = tb::GF_SWIGLU; g.alpha = 1.0f; g.n_split = (int)H;
  TORCH_CHECK(act >= 0 && act <= 2 && (act != 2 || limit > 0), "tc_gemm_swiglu: activation");
  g.glu_act = (int)act;
  g.glu_limit = (float)limit;
  g.glu_alpha = (float)alpha;
  if (bias.has_value() && bias->defined()) {
    TORCH_CHECK(bias->is_cuda() && bias->scalar_type() == at::kFloat && bias->is_contiguous() && bias->numel() == 2 * H &&
                    (reinterpret_cast<uintptr_t>(bias->data_ptr()) & 15) == 0,
                "tc_gemm_swiglu: bias [2H] fp32");
    g.glu_bias = bias->data_ptr<float>();
  }
  if (gu.has_value() && gu->defined()) {
    check_bf16_cuda(*gu, "gu");
    TORCH_CHECK(gu->dim() == 2 && gu->is_contiguous() && gu->size(0) == M && gu->size(1) == 2 * H, "gu must be [M, 2H] contiguous");
    g.aux_out = reinterpret_cast<__nv_bfloat16*>(gu->data_ptr());
  }
  tb::launch_tc_gemm(g, cur_stream());
}

// Backward of the SwiGLU epilogue inside the GEMM that forms d(hidden): dgu [M, 2H] = (d gate | d up) from
// dh = dy op(w) ([M, H], never written) and the saved pre-activations gu [M, 2H]. w is [H, K] (K-major) or, with
// w_mn_major, stored [K, H] (the FFN's down projection as it is stored).
void tc_gemm_dswiglu(const Tensor& dy, const Tensor& w, bool w_mn_major, const Tensor& gu, Tensor& dgu) {
  check_bf16_cuda(dy, "dy");
  check_bf16_cuda(w, "w");
  check_bf16_cuda(gu, "gu");
  check_bf16_cuda(dgu, "dgu");
  TORCH_CHECK(dy.dim() == 2 && w.dim() == 2 && dy.stride(1) == 1 && w.stride(1) == 1, "tc_gemm_dswiglu: 2-D operands");
  const int64_t M = dy.size(0), K = dy.size(1);
  const int64_t H = w_mn_major ? w.size(1) : w.size(0);
  TORCH_CHECK((w_mn_major ? w.size(0) : w.size(1)) == K, "tc_gemm_dswiglu: reduction dims differ");
  TORCH_CHECK(gu.is_contiguous() && dgu.is_contiguous() && gu.size(0) == M && gu.size(1) == 2 * H && dgu.sizes() == gu.sizes(),
              "gu and dgu must be [M, 2H] contiguous");
  c10::cuda::CUDAGuard guard(dy.device());
  tb::GemmArgs g{};
  g.A = bf(dy); g.B = bf(w); g.C = dgu.data_ptr();
  g.M = (int)M; g.N = (int)H; g.K = (int)K;
  g.lda = dy.stride(0); g.ldb = w.stride(0); g.ldc = dgu.stride(0);
  g.b_mn_major = w_mn_major;
  g.batch = 1; g.mode = tb::GEMM_DENSE; g.flags = tb::GF_DSWIGLU; g.alpha = 1.0f; g.n_split = (int)H;
  g.aux_in = bf(gu);
  tb::launch_tc_gemm(g, cur_stream());
}

}  // namespace

void register_gemm(pybind11::module& m) {
  m.def("tc_gemm", &tc_gemm);
  m.def("tc_gemm_debug_buffer", [](const c10::optional<Tensor>& t) {
    const bool on = t.has_value() && t->defined();
    TORCH_CHECK(!on || (t->is_cuda() && t->scalar_type() == at::kLong && t->is_contiguous() && t->numel() >= 16),
                "tc_gemm_debug_buffer: a contiguous CUDA int64 tensor with at least 16 entries, or None");
    tb::tc_gemm_set_debug_buffer(on ? (long long*)t->data_ptr<int64_t>() : nullptr);
  });
  m.def("tc_gemm_pair_launches", []() { return (int64_t)tb::tc_gemm_pair_launch_count(); });
  m.def("tc_gemm_swiglu", &tc_gemm_swiglu, pybind11::arg("x"), pybind11::arg("w13"), pybind11::arg("h"), pybind11::arg("gu"), pybind11::arg("act") = 0,
        pybind11::arg("bias") = pybind11::none(), pybind11::arg("limit") = 0.0, pybind11::arg("alpha") = 0.0);
  m.def("tc_gemm_dswiglu", &tc_gemm_dswiglu);
}
