// Bindings of the kernels every engine model uses: dense GEMM, few-row products, sampling. Part of `_C` and of `_hybrid`.
#include "binding_helpers.h"
#include "launchers.h"

namespace {

using namespace mb_bind;

void gemm(const at::Tensor& a, const at::Tensor& b, at::Tensor& c, bool a_mn, bool b_mn, bool accumulate,
          int64_t block_n, const c10::optional<at::Tensor>& status, const std::vector<int64_t>& dest,
          const c10::optional<at::Tensor>& sig_ctrl, const std::vector<int64_t>& sig_flags, int64_t sig_me) {
  check_bf16_2d(a, "a");
  check_bf16_2d(b, "b");
  TORCH_CHECK(c.dim() == 2, "c must be 2-D");
  const c10::cuda::CUDAGuard guard(a.device());
  mb::GemmProblem p{};
  p.mode = mb::GEMM_DENSE;
  p.M = a_mn ? a.size(1) : a.size(0);
  p.K = a_mn ? a.size(0) : a.size(1);
  p.N = b_mn ? b.size(1) : b.size(0);
  const int64_t kb = b_mn ? b.size(0) : b.size(1);
  TORCH_CHECK(kb == p.K, "contraction extents differ: ", p.K, " vs ", kb);
  TORCH_CHECK(c.size(0) == p.M && c.size(1) == p.N, "output shape must be [", p.M, ", ", p.N, "]");
  p.a = operand(a, a_mn);
  p.b = operand(b, b_mn);
  fill_out(p, c);
  p.ldc = c.stride(0);
  p.accumulate = accumulate;
  p.status = status_ptr(status);
  p.block_n = static_cast<int>(block_n);
  if (!dest.empty()) {  // replicated output: each destination receives the tile at the offset it has in c
    TORCH_CHECK(dest.size() <= 8, "at most 8 destinations");
    p.n_dest = static_cast<int>(dest.size());
    for (size_t i = 0; i < dest.size(); ++i) p.dest[i] = reinterpret_cast<void*>(dest[i]);
    if (sig_ctrl.has_value()) {
      TORCH_CHECK(sig_ctrl->scalar_type() == at::kLong && sig_ctrl->numel() >= 6 && sig_flags.size() <= 8, "bad signal arguments");
      p.sig_ctrl = reinterpret_cast<unsigned long long*>(sig_ctrl->data_ptr<int64_t>());
      for (size_t i = 0; i < sig_flags.size(); ++i) p.sig_flags[i] = reinterpret_cast<unsigned long long*>(sig_flags[i]);
      p.sig_nranks = static_cast<int>(sig_flags.size());
      p.sig_me = static_cast<int>(sig_me);
    }
  }
  TORCH_CHECK(mb::gemm_bf16_launch(p, cur_stream()) == 0, "gemm: ", mb::gemm_last_error());
}

// logits [B, V] (bf16/fp32) -> (token int32 [B], logprob fp32 [B]); per-row parameters are optional tensors.
void sample_rows(const at::Tensor& logits, const c10::optional<at::Tensor>& temperature,
                 const c10::optional<at::Tensor>& top_k, const c10::optional<at::Tensor>& top_p,
                 const c10::optional<at::Tensor>& seeds, const c10::optional<at::Tensor>& step, at::Tensor& out_token,
                 at::Tensor& out_logprob) {
  TORCH_CHECK(logits.is_cuda() && logits.dim() == 2 && logits.stride(1) == 1, "logits must be 2-D with contiguous rows");
  const bool fp32 = logits.scalar_type() == at::kFloat;
  TORCH_CHECK(fp32 || logits.scalar_type() == at::kBFloat16, "logits must be bf16 or fp32");
  CHECK_I32(out_token); CHECK_F32(out_logprob);
  if (seeds.has_value()) TORCH_CHECK(seeds->scalar_type() == at::kLong && seeds->is_cuda(), "seeds must be int64 CUDA");
  const c10::cuda::CUDAGuard guard(logits.device());
  mb::sample_rows(logits.data_ptr(), fp32, logits.size(0), logits.size(1), logits.stride(0), opt_ptr<float>(temperature),
                  opt_ptr<int>(top_k), opt_ptr<float>(top_p),
                  reinterpret_cast<const unsigned long long*>(opt_ptr<int64_t>(seeds)), opt_ptr<int>(step),
                  out_token.data_ptr<int>(), out_logprob.data_ptr<float>(), cur_stream());
}

void small_gemv(const at::Tensor& x, const c10::optional<at::Tensor>& norm_w, double eps, const at::Tensor& W,
                const c10::optional<at::Tensor>& residual, at::Tensor& out, const c10::optional<at::Tensor>& status) {
  CHECK_BF16(x); CHECK_BF16(W);
  const int T = x.size(0), K = x.size(1), N = W.size(0);
  TORCH_CHECK(T >= 1 && T <= 64 && W.size(1) == K && K % 32 == 0 && N % 16 == 0, "small_gemv: need 1 <= T <= 64, K % 32 == 0, N % 16 == 0");
  TORCH_CHECK(T <= 8 || !norm_w.has_value(), "small_gemv: the folded RMSNorm is available for at most 8 rows");
  TORCH_CHECK(out.is_cuda() && out.is_contiguous() && out.size(0) == T && out.size(1) == N, "small_gemv: bad output shape");
  const bool f32 = out.scalar_type() == at::kFloat;
  TORCH_CHECK(f32 || out.scalar_type() == at::kBFloat16, "small_gemv: output must be fp32 or bf16");
  if (norm_w.has_value()) CHECK_BF16((*norm_w));
  if (residual.has_value()) { CHECK_BF16((*residual)); TORCH_CHECK(residual->numel() == out.numel(), "small_gemv: residual shape"); }
  const c10::cuda::CUDAGuard guard(x.device());
  mb::small_gemv(x.data_ptr(), T, norm_w.has_value() ? norm_w->data_ptr() : nullptr, eps, W.data_ptr(), N, K,
                 residual.has_value() ? residual->data_ptr() : nullptr, out.data_ptr(), f32,
                 status.has_value() ? status->data_ptr<int>() : nullptr, cur_stream());
}

}  // namespace

void register_serving(pybind11::module_& m) {
  namespace py = pybind11;
  m.def("gemm", &gemm, "bf16 tcgen05 GEMM: c (+)= a . b^T with selectable operand majors", py::arg("a"), py::arg("b"),
        py::arg("c"), py::arg("a_mn"), py::arg("b_mn"), py::arg("accumulate"), py::arg("block_n"), py::arg("status"),
        py::arg("dest") = std::vector<int64_t>(), py::arg("sig_ctrl") = py::none(),
        py::arg("sig_flags") = std::vector<int64_t>(), py::arg("sig_me") = 0);
  m.def("sample_rows", &sample_rows);
  m.def("small_gemv", &small_gemv);
}
