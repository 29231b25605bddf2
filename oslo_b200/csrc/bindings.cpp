// torch.ops.oslo_b200.*: argument checking, allocation and stream plumbing around the C launchers.
#include <ATen/cuda/CUDAContext.h>
#include <c10/cuda/CUDAGuard.h>
#include <torch/library.h>
#include <torch/torch.h>

#include <atomic>
#include <mutex>
#include <unordered_map>

#include "oslo_kernels.h"

namespace {

using at::Tensor;
using c10::optional;

int dt_code(const Tensor& t) {
  switch (t.scalar_type()) {
    case at::kBFloat16: return OSLO_DT_BF16;
    case at::kHalf: return OSLO_DT_FP16;
    case at::kFloat: return OSLO_DT_FP32;
    default: TORCH_CHECK(false, "oslo_b200: unsupported dtype ", t.scalar_type());
  }
}
void check_rc(int rc, const char* what) {
  TORCH_CHECK(rc == 0, "oslo_b200::", what, " failed with code ", rc,
              rc > 0 ? std::string(" (") + cudaGetErrorString(static_cast<cudaError_t>(rc)) + ")" : std::string());
}
std::atomic<int64_t> g_launches{0};
// every binding passes through here once per kernel it enqueues
cudaStream_t cur_stream(int kernels = 1) {
  g_launches.fetch_add(kernels, std::memory_order_relaxed);
  return at::cuda::getCurrentCUDAStream().stream();
}
int64_t launch_count() { return g_launches.load(std::memory_order_relaxed); }
// SMs that the persistent GEMM kernels leave free (their grids are sized for `SM count - reserved`). A pipeline stage
// keeps point-to-point transfers in flight that wait for the neighbouring stage while holding an SM each; with a
// statically scheduled persistent grid every SM taken away would delay that SM's whole share of the tiles to the end
// of the kernel. Process-wide; every rank of a tensor-parallel group must use the same value (the fused GEMM +
// collective kernels need the same grid on every rank).
std::atomic<int> g_reserved_sms{0};
int64_t set_reserved_sms(int64_t n) {
  const int prev = g_reserved_sms.exchange(static_cast<int>(n < 0 ? 0 : n));
  return prev;
}
int64_t reserved_sms() { return g_reserved_sms.load(); }
const void* ptr_or_null(const optional<Tensor>& t) { return t.has_value() && t->defined() ? t->data_ptr() : nullptr; }

struct DevState {
  Tensor err;
  int sms = 0;
};
DevState& dev_state(int dev) {
  static std::mutex mu;
  static std::unordered_map<int, DevState> states;
  std::lock_guard<std::mutex> g(mu);
  auto it = states.find(dev);
  if (it == states.end()) {
    DevState s;
    s.err = at::zeros({1}, at::TensorOptions().dtype(at::kInt).device(at::kCUDA, dev));
    s.sms = at::cuda::getDeviceProperties(dev)->multiProcessorCount;
    it = states.emplace(dev, std::move(s)).first;
  }
  return it->second;
}

// SM count the persistent kernels may fill: all of them minus the reserved ones, an even number of at least 2
int usable_sms(const DevState& st) {
  int n = st.sms - g_reserved_sms.load(std::memory_order_relaxed);
  if (n < 2) n = 2;
  return n & ~1;
}

// The word that kernels set when a bounded wait runs out (0 = no error). Reading it synchronises.
Tensor error_word(const Tensor& like) { return dev_state(like.get_device()).err; }

void check_2d_operand(const Tensor& t, const char* name) {
  TORCH_CHECK(t.is_cuda() && t.dim() == 2, name, " must be a 2-D CUDA tensor");
  TORCH_CHECK(t.stride(1) == 1 && t.stride(0) % 8 == 0 && t.stride(0) >= t.size(1), name,
              " needs a contiguous last dim and a row stride that is a multiple of 8 elements");
  TORCH_CHECK(reinterpret_cast<uintptr_t>(t.data_ptr()) % 16 == 0, name, " must be 16-byte aligned");
}

// D[M,N] = alpha * A x B^T-style product with fused epilogue; see gemm_sm100.cu for the operand layouts.
Tensor gemm(const Tensor& a, const Tensor& b, int64_t a_mn, int64_t b_mn, const optional<Tensor>& bias,
            const optional<Tensor>& aux, const optional<Tensor>& out, const optional<Tensor>& aux_out, int64_t flags,
            double alpha) {
  check_2d_operand(a, "a");
  check_2d_operand(b, "b");
  TORCH_CHECK(a.scalar_type() == b.scalar_type(), "a and b must share a dtype");
  TORCH_CHECK(a.scalar_type() == at::kBFloat16 || a.scalar_type() == at::kHalf, "gemm inputs must be bf16 or fp16");
  c10::cuda::CUDAGuard guard(a.device());
  const int64_t M = a_mn ? a.size(1) : a.size(0), K = a_mn ? a.size(0) : a.size(1);
  const int64_t N = b_mn ? b.size(1) : b.size(0), Kb = b_mn ? b.size(0) : b.size(1);
  TORCH_CHECK(K == Kb, "contraction sizes differ: ", K, " vs ", Kb);
  int fl = static_cast<int>(flags) & ~GEMM_FLAG_FP16;
  if (a.scalar_type() == at::kHalf) fl |= GEMM_FLAG_FP16;
  const bool out_f32 = fl & GEMM_FLAG_OUT_FP32;
  Tensor d;
  if (out.has_value() && out->defined()) {
    d = *out;
    TORCH_CHECK(d.is_cuda() && d.dim() == 2 && d.size(0) == M && d.size(1) == N && d.stride(1) == 1, "bad out");
    TORCH_CHECK(d.scalar_type() == (out_f32 ? at::kFloat : a.scalar_type()), "out dtype does not match flags");
  } else {
    TORCH_CHECK(!(fl & GEMM_FLAG_ACCUMULATE), "accumulate needs an out tensor");
    d = at::empty({M, N}, a.options().dtype(out_f32 ? at::kFloat : a.scalar_type()));
  }
  if (M == 0 || N == 0) return d;
  // the epilogue moves 32 columns of a row in 16-byte pieces
  const auto rows16 = [&](const Tensor& t) {
    return N < 32 || (t.stride(0) * t.element_size() % 16 == 0 && reinterpret_cast<uintptr_t>(t.data_ptr()) % 16 == 0);
  };
  TORCH_CHECK(rows16(d), "gemm: rows of a result with 32 or more columns must start at 16-byte boundaries");
  if (fl & GEMM_FLAG_BIAS) {
    TORCH_CHECK(bias.has_value() && bias->numel() == N && bias->scalar_type() == a.scalar_type() && bias->is_contiguous(),
                "bias must be a contiguous [N] tensor of the input dtype");
  }
  int ld_aux = 0, ld_aux_out = 0;
  if (fl & (GEMM_FLAG_DGELU | GEMM_FLAG_RESIDUAL)) {
    TORCH_CHECK(!((fl & GEMM_FLAG_DGELU) && (fl & GEMM_FLAG_RESIDUAL)), "dgelu and residual share the aux operand");
    TORCH_CHECK(aux.has_value() && aux->dim() == 2 && aux->size(0) == M && aux->size(1) == N && aux->stride(1) == 1, "bad aux");
    const auto want = (fl & GEMM_FLAG_RESIDUAL) ? d.scalar_type() : a.scalar_type();
    TORCH_CHECK(aux->scalar_type() == want, "aux dtype mismatch");
    TORCH_CHECK(rows16(*aux), "gemm: rows of aux must start at 16-byte boundaries");
    ld_aux = static_cast<int>(aux->stride(0));
  }
  if (fl & GEMM_FLAG_SAVE_PREACT) {
    TORCH_CHECK(aux_out.has_value() && aux_out->dim() == 2 && aux_out->size(0) == M && aux_out->size(1) == N &&
                    aux_out->stride(1) == 1 && aux_out->scalar_type() == a.scalar_type() && rows16(*aux_out), "bad aux_out");
    ld_aux_out = static_cast<int>(aux_out->stride(0));
  }
  auto& st = dev_state(a.get_device());
  const int rc = oslo_gemm_16bit(a.data_ptr(), b.data_ptr(), d.data_ptr(), static_cast<int>(M), static_cast<int>(N),
                                 static_cast<int>(K), static_cast<int>(a.stride(0)), static_cast<int>(b.stride(0)),
                                 static_cast<int>(d.stride(0)), static_cast<int>(a_mn), static_cast<int>(b_mn),
                                 ptr_or_null(bias), ptr_or_null(aux), ld_aux,
                                 const_cast<void*>(ptr_or_null(aux_out)), ld_aux_out, fl, static_cast<float>(alpha),
                                 st.err.data_ptr<int>(), usable_sms(st), cur_stream());
  check_rc(rc, "gemm");
  return d;
}

// LM-head projection whose epilogue does the cross-entropy work; the logits a @ b^T + bias are never stored.
//   forward  (lse undefined): returns (rowmax, sumexp, target logit), fp32 [M] each
//   backward (lse, scale given): returns ((softmax - onehot) * scale) [M, N] in the input dtype, written into `out`
//   when given
std::tuple<Tensor, Tensor, Tensor> gemm_ce_stats(const Tensor& a, const Tensor& b, int64_t b_mn, const optional<Tensor>& bias,
                                                 const Tensor& labels, int64_t vocab_start) {
  check_2d_operand(a, "a");
  check_2d_operand(b, "b");
  TORCH_CHECK(a.scalar_type() == b.scalar_type() && (a.scalar_type() == at::kBFloat16 || a.scalar_type() == at::kHalf),
              "gemm_ce inputs must both be bf16 or fp16");
  const int64_t M = a.size(0), K = a.size(1), N = b_mn ? b.size(1) : b.size(0);
  TORCH_CHECK((b_mn ? b.size(0) : b.size(1)) == K, "contraction sizes differ");
  TORCH_CHECK(labels.is_cuda() && labels.scalar_type() == at::kLong && labels.numel() == M && labels.is_contiguous(), "bad labels");
  const bool has_bias = bias.has_value() && bias->defined();
  if (has_bias) TORCH_CHECK(bias->numel() == N && bias->scalar_type() == a.scalar_type() && bias->is_contiguous(), "bad bias");
  c10::cuda::CUDAGuard guard(a.device());
  auto f32 = a.options().dtype(at::kFloat);
  Tensor mx = at::empty({M}, f32), se = at::empty({M}, f32), tg = at::empty({M}, f32);
  if (M == 0) return {mx, se, tg};
  const int64_t blocks = (N + GEMM_CE_BLOCK - 1) / GEMM_CE_BLOCK;
  Tensor stats = at::empty({blocks, M, 3}, f32);
  auto& st = dev_state(a.get_device());
  check_rc(oslo_gemm_ce_16bit(a.data_ptr(), b.data_ptr(), static_cast<int>(M), static_cast<int>(N), static_cast<int>(K),
                              static_cast<int>(a.stride(0)), static_cast<int>(b.stride(0)), static_cast<int>(b_mn),
                              has_bias ? bias->data_ptr() : nullptr,
                              reinterpret_cast<const long long*>(labels.data_ptr<int64_t>()), vocab_start, 0,
                              stats.data_ptr<float>(), nullptr, nullptr, nullptr, 0, a.scalar_type() == at::kHalf ? 1 : 0,
                              st.err.data_ptr<int>(), usable_sms(st), cur_stream()), "gemm_ce_stats");
  check_rc(oslo_ce_reduce_stats(stats.data_ptr<float>(), mx.data_ptr<float>(), se.data_ptr<float>(), tg.data_ptr<float>(),
                                static_cast<int>(M), static_cast<int>(blocks), cur_stream()), "ce_reduce_stats");
  return {mx, se, tg};
}
Tensor gemm_ce_grad(const Tensor& a, const Tensor& b, int64_t b_mn, const optional<Tensor>& bias, const Tensor& labels,
                    int64_t vocab_start, const Tensor& lse, const Tensor& scale) {
  check_2d_operand(a, "a");
  check_2d_operand(b, "b");
  TORCH_CHECK(a.scalar_type() == b.scalar_type() && (a.scalar_type() == at::kBFloat16 || a.scalar_type() == at::kHalf),
              "gemm_ce inputs must both be bf16 or fp16");
  const int64_t M = a.size(0), K = a.size(1), N = b_mn ? b.size(1) : b.size(0);
  TORCH_CHECK((b_mn ? b.size(0) : b.size(1)) == K, "contraction sizes differ");
  TORCH_CHECK(labels.is_cuda() && labels.scalar_type() == at::kLong && labels.numel() == M && labels.is_contiguous(), "bad labels");
  TORCH_CHECK(lse.scalar_type() == at::kFloat && lse.numel() == M && lse.is_contiguous() &&
              scale.scalar_type() == at::kFloat && scale.numel() == M && scale.is_contiguous(), "lse / scale must be fp32 [M]");
  const bool has_bias = bias.has_value() && bias->defined();
  if (has_bias) TORCH_CHECK(bias->numel() == N && bias->scalar_type() == a.scalar_type() && bias->is_contiguous(), "bad bias");
  c10::cuda::CUDAGuard guard(a.device());
  Tensor d = at::empty({M, N}, a.options());
  if (M == 0) return d;
  auto& st = dev_state(a.get_device());
  check_rc(oslo_gemm_ce_16bit(a.data_ptr(), b.data_ptr(), static_cast<int>(M), static_cast<int>(N), static_cast<int>(K),
                              static_cast<int>(a.stride(0)), static_cast<int>(b.stride(0)), static_cast<int>(b_mn),
                              has_bias ? bias->data_ptr() : nullptr,
                              reinterpret_cast<const long long*>(labels.data_ptr<int64_t>()), vocab_start, 1, nullptr,
                              lse.data_ptr<float>(), scale.data_ptr<float>(), d.data_ptr(), static_cast<int>(d.stride(0)),
                              a.scalar_type() == at::kHalf ? 1 : 0, st.err.data_ptr<int>(), usable_sms(st), cur_stream()),
           "gemm_ce_grad");
  return d;
}

// y = act(a @ b^T + bias) for few rows (decode steps): split-K GEMM into fp32 planes, then one finalisation
// kernel that sums them in a fixed order. Falls back to the ordinary GEMM when splitting the k range gains nothing.
// `gelu_from`: -1 = no activation, c >= 0 = tanh-GeLU on output columns >= c (0 = all of them), which lets one GEMM
// serve several layers that share an input when only the last of them is followed by the activation.
Tensor gemm_small_m(const Tensor& a, const Tensor& b, int64_t b_mn, const optional<Tensor>& bias, int64_t gelu_from) {
  check_2d_operand(a, "a");
  check_2d_operand(b, "b");
  TORCH_CHECK(a.scalar_type() == b.scalar_type(), "a and b must share a dtype");
  TORCH_CHECK(a.scalar_type() == at::kBFloat16 || a.scalar_type() == at::kHalf, "gemm inputs must be bf16 or fp16");
  c10::cuda::CUDAGuard guard(a.device());
  const int64_t M = a.size(0), K = a.size(1);
  const int64_t N = b_mn ? b.size(1) : b.size(0), Kb = b_mn ? b.size(0) : b.size(1);
  TORCH_CHECK(K == Kb, "contraction sizes differ: ", K, " vs ", Kb);
  auto& st = dev_state(a.get_device());
  const int split = std::max(1, oslo_gemm_split_k_for(static_cast<int>(M), static_cast<int>(N), static_cast<int>(K), usable_sms(st)));
  const bool has_bias = bias.has_value() && bias->defined();
  if (has_bias)
    TORCH_CHECK(bias->numel() == N && bias->scalar_type() == a.scalar_type() && bias->is_contiguous(), "bad bias");
  if (split <= 1 && gelu_from <= 0) {
    const int64_t fl = (has_bias ? GEMM_FLAG_BIAS : 0) | (gelu_from == 0 ? GEMM_FLAG_GELU : 0) | (gelu_from == OSLO_ACT_RELU2 ? GEMM_FLAG_RELU2 : 0);
    return gemm(a, b, 0, b_mn, bias, optional<Tensor>(), optional<Tensor>(), optional<Tensor>(), fl, 1.0);
  }
  Tensor ws = at::empty({split, M, N}, a.options().dtype(at::kFloat));
  check_rc(oslo_gemm_splitk_16bit(a.data_ptr(), b.data_ptr(), ws.data_ptr<float>(), static_cast<int>(M),
                                  static_cast<int>(N), static_cast<int>(K), static_cast<int>(a.stride(0)),
                                  static_cast<int>(b.stride(0)), static_cast<int>(N), 0, static_cast<int>(b_mn),
                                  a.scalar_type() == at::kHalf ? 1 : 0, split, st.err.data_ptr<int>(), usable_sms(st),
                                  cur_stream()), "gemm_splitk");
  Tensor y = at::empty({M, N}, a.options());
  check_rc(oslo_splitk_finalize(ws.data_ptr<float>(), has_bias ? bias->data_ptr() : nullptr, y.data_ptr(), M,
                                static_cast<int>(N), split, static_cast<int>(gelu_from), dt_code(a), cur_stream()), "splitk_finalize");
  return y;
}

std::tuple<Tensor, Tensor, Tensor> layernorm_fwd(const Tensor& x, const Tensor& w, const optional<Tensor>& b, double eps) {
  TORCH_CHECK(x.is_cuda() && x.is_contiguous() && w.is_contiguous(), "layernorm: contiguous CUDA tensors required");
  c10::cuda::CUDAGuard guard(x.device());
  const int64_t cols = x.size(-1), rows = x.numel() / std::max<int64_t>(cols, 1);
  Tensor y = at::empty_like(x);
  Tensor mean = at::empty({rows}, x.options().dtype(at::kFloat));
  Tensor rstd = at::empty({rows}, x.options().dtype(at::kFloat));
  check_rc(oslo_layernorm_fwd(x.data_ptr(), w.data_ptr(), ptr_or_null(b), y.data_ptr(), mean.data_ptr<float>(),
                              rstd.data_ptr<float>(), static_cast<int>(rows), static_cast<int>(cols),
                              static_cast<float>(eps), dt_code(x), cur_stream()), "layernorm_fwd");
  return {y, mean, rstd};
}

std::tuple<Tensor, Tensor, Tensor> layernorm_bwd(const Tensor& dy, const Tensor& x, const Tensor& w, const Tensor& mean,
                                                  const Tensor& rstd) {
  TORCH_CHECK(dy.is_contiguous() && x.is_contiguous(), "layernorm_bwd: contiguous tensors required");
  c10::cuda::CUDAGuard guard(x.device());
  const int64_t cols = x.size(-1), rows = x.numel() / std::max<int64_t>(cols, 1);
  const int parts = static_cast<int>(std::min<int64_t>(rows, 2 * dev_state(x.get_device()).sms));
  Tensor dx = at::empty_like(x);
  Tensor dw = at::empty_like(w), db = at::empty_like(w);
  Tensor part = at::empty({2, std::max(parts, 1), cols}, x.options().dtype(at::kFloat));
  check_rc(oslo_layernorm_bwd(dy.data_ptr(), x.data_ptr(), w.data_ptr(), mean.data_ptr<float>(), rstd.data_ptr<float>(),
                              dx.data_ptr(), part[0].data_ptr<float>(), part[1].data_ptr<float>(), dw.data_ptr(),
                              db.data_ptr(), static_cast<int>(rows), static_cast<int>(cols), parts, dt_code(x),
                              cur_stream(2)), "layernorm_bwd");
  return {dx, dw, db};
}

Tensor bias_gelu_fwd(const Tensor& x, const optional<Tensor>& bias) {
  TORCH_CHECK(x.is_cuda() && x.is_contiguous(), "bias_gelu: contiguous CUDA tensor required");
  c10::cuda::CUDAGuard guard(x.device());
  Tensor y = at::empty_like(x);
  const int64_t cols = x.size(-1);
  check_rc(oslo_bias_gelu_fwd(x.data_ptr(), ptr_or_null(bias), y.data_ptr(), x.numel() / std::max<int64_t>(cols, 1),
                              static_cast<int>(cols), dt_code(x), cur_stream()), "bias_gelu_fwd");
  return y;
}
Tensor bias_gelu_bwd(const Tensor& dy, const Tensor& x, const optional<Tensor>& bias) {
  TORCH_CHECK(dy.is_contiguous() && x.is_contiguous(), "bias_gelu_bwd: contiguous tensors required");
  c10::cuda::CUDAGuard guard(x.device());
  Tensor dx = at::empty_like(x);
  const int64_t cols = x.size(-1);
  check_rc(oslo_bias_gelu_bwd(dy.data_ptr(), x.data_ptr(), ptr_or_null(bias), dx.data_ptr(),
                              x.numel() / std::max<int64_t>(cols, 1), static_cast<int>(cols), dt_code(x), cur_stream()),
           "bias_gelu_bwd");
  return dx;
}

Tensor bias_dropout_residual(const Tensor& x, const optional<Tensor>& bias, const optional<Tensor>& residual, double p,
                             int64_t seed, int64_t mode) {
  TORCH_CHECK(x.is_cuda() && x.is_contiguous(), "bias_dropout_residual: contiguous CUDA tensor required");
  c10::cuda::CUDAGuard guard(x.device());
  Tensor y = at::empty_like(x);
  const int64_t cols = x.size(-1);
  check_rc(oslo_bias_dropout_residual(x.data_ptr(), ptr_or_null(bias), ptr_or_null(residual), y.data_ptr(),
                                      x.numel() / std::max<int64_t>(cols, 1), static_cast<int>(cols),
                                      static_cast<float>(p), static_cast<unsigned long long>(seed),
                                      static_cast<int>(mode), dt_code(x), cur_stream()), "bias_dropout_residual");
  return y;
}

Tensor colsum(const Tensor& x) {
  TORCH_CHECK(x.is_cuda() && x.dim() == 2 && x.is_contiguous(), "colsum: contiguous 2-D CUDA tensor required");
  c10::cuda::CUDAGuard guard(x.device());
  const int rows = static_cast<int>(x.size(0)), cols = static_cast<int>(x.size(1));
  const int parts = std::max(1, std::min(rows, 64));
  Tensor part = at::empty({parts, cols}, x.options().dtype(at::kFloat));
  Tensor out = at::zeros({cols}, x.options().dtype(at::kFloat));
  check_rc(oslo_colsum(x.data_ptr(), part.data_ptr<float>(), out.data_ptr<float>(), rows, cols, parts, dt_code(x),
                       cur_stream(2)), "colsum");
  return out;
}

Tensor rotary(const Tensor& x, const Tensor& positions, int64_t rotary_dim, double base, bool inverse) {
  TORCH_CHECK(x.is_cuda() && x.dim() == 4 && x.is_contiguous(), "rotary: contiguous [B,S,H,D] CUDA tensor required");
  TORCH_CHECK(positions.scalar_type() == at::kLong && positions.is_contiguous() &&
                  positions.numel() == x.size(0) * x.size(1), "rotary: positions must be int64 [B,S]");
  c10::cuda::CUDAGuard guard(x.device());
  Tensor y = at::empty_like(x);
  check_rc(oslo_rotary(x.data_ptr(), y.data_ptr(), reinterpret_cast<const long long*>(positions.data_ptr<int64_t>()),
                       static_cast<int>(x.size(0)), static_cast<int>(x.size(1)), static_cast<int>(x.size(2)),
                       static_cast<int>(x.size(3)), static_cast<int>(rotary_dim), static_cast<float>(base),
                       inverse ? 1 : 0, dt_code(x), cur_stream()), "rotary");
  return y;
}

// in place: only the first rotary_dim dims of every head are read and written. x is any contiguous tensor whose
// memory is [tokens, heads, head_dim] (e.g. the [B, S, heads * head_dim] output of a projection)
Tensor rotary_(Tensor x, const Tensor& positions, int64_t heads, int64_t head_dim, int64_t rotary_dim, double base,
               bool inverse) {
  TORCH_CHECK(x.is_cuda() && x.is_contiguous(), "rotary_: contiguous CUDA tensor required");
  TORCH_CHECK(positions.scalar_type() == at::kLong && positions.is_contiguous() &&
                  positions.numel() * heads * head_dim == x.numel(), "rotary_: positions must be int64 [tokens]");
  c10::cuda::CUDAGuard guard(x.device());
  check_rc(oslo_rotary_inplace(x.data_ptr(), reinterpret_cast<const long long*>(positions.data_ptr<int64_t>()), 1,
                               static_cast<int>(positions.numel()), static_cast<int>(heads), static_cast<int>(head_dim),
                               static_cast<int>(rotary_dim), static_cast<float>(base), inverse ? 1 : 0, dt_code(x),
                               cur_stream()), "rotary_");
  return x;
}

Tensor causal_softmax_fwd(const Tensor& x, double scale) {
  TORCH_CHECK(x.is_cuda() && x.dim() == 3 && x.is_contiguous(), "causal_softmax: contiguous [batches,sq,sk] required");
  c10::cuda::CUDAGuard guard(x.device());
  Tensor y = at::empty_like(x);
  check_rc(oslo_causal_softmax_fwd(x.data_ptr(), y.data_ptr(), static_cast<int>(x.size(0)), static_cast<int>(x.size(1)),
                                   static_cast<int>(x.size(2)), static_cast<float>(scale), dt_code(x), cur_stream()),
           "causal_softmax_fwd");
  return y;
}
Tensor masked_softmax_fwd(const Tensor& x, const Tensor& mask, double scale) {
  TORCH_CHECK(x.is_cuda() && x.dim() == 4 && x.is_contiguous(), "masked_softmax: contiguous [b,h,sq,sk] required");
  TORCH_CHECK(mask.scalar_type() == at::kByte && mask.is_contiguous() && mask.dim() == 4 && mask.size(1) == 1 &&
                  mask.size(2) == x.size(2) && mask.size(3) == x.size(3) &&
                  (mask.size(0) == 1 || mask.size(0) == x.size(0)), "mask must be uint8 [1|b,1,sq,sk]");
  c10::cuda::CUDAGuard guard(x.device());
  Tensor y = at::empty_like(x);
  check_rc(oslo_masked_softmax_fwd(x.data_ptr(), mask.data_ptr<uint8_t>(), y.data_ptr(), static_cast<int>(x.size(0)),
                                   static_cast<int>(x.size(1)), static_cast<int>(x.size(2)), static_cast<int>(x.size(3)),
                                   static_cast<int>(mask.size(0)), static_cast<float>(scale), dt_code(x), cur_stream()),
           "masked_softmax_fwd");
  return y;
}
Tensor softmax_bwd(const Tensor& y, const Tensor& dy, double scale) {
  TORCH_CHECK(y.is_contiguous() && dy.is_contiguous(), "softmax_bwd: contiguous tensors required");
  c10::cuda::CUDAGuard guard(y.device());
  Tensor dx = at::empty_like(y);
  const int64_t cols = y.size(-1);
  check_rc(oslo_softmax_bwd(y.data_ptr(), dy.data_ptr(), dx.data_ptr(), y.numel() / std::max<int64_t>(cols, 1),
                            static_cast<int>(cols), static_cast<float>(scale), dt_code(y), cur_stream()), "softmax_bwd");
  return dx;
}

std::tuple<Tensor, Tensor, Tensor> ce_stats(const Tensor& logits, const Tensor& labels, int64_t vocab_start) {
  TORCH_CHECK(logits.is_cuda() && logits.dim() == 2 && logits.stride(1) == 1, "ce_stats: [rows, cols] logits required");
  TORCH_CHECK(labels.scalar_type() == at::kLong && labels.is_contiguous() && labels.numel() == logits.size(0), "bad labels");
  c10::cuda::CUDAGuard guard(logits.device());
  const auto fo = logits.options().dtype(at::kFloat);
  Tensor mx = at::empty({logits.size(0)}, fo), se = at::empty({logits.size(0)}, fo), tg = at::empty({logits.size(0)}, fo);
  check_rc(oslo_ce_stats(logits.data_ptr(), reinterpret_cast<const long long*>(labels.data_ptr<int64_t>()),
                         mx.data_ptr<float>(), se.data_ptr<float>(), tg.data_ptr<float>(), static_cast<int>(logits.size(0)),
                         static_cast<int>(logits.size(1)), static_cast<int>(logits.stride(0)), vocab_start,
                         dt_code(logits), cur_stream()), "ce_stats");
  return {mx, se, tg};
}
Tensor ce_grad_(Tensor logits, const Tensor& labels, int64_t vocab_start, const Tensor& lse, const Tensor& scale) {
  TORCH_CHECK(logits.is_cuda() && logits.dim() == 2 && logits.stride(1) == 1, "ce_grad_: [rows, cols] logits required");
  TORCH_CHECK(lse.scalar_type() == at::kFloat && scale.scalar_type() == at::kFloat && lse.is_contiguous() &&
                  scale.is_contiguous() && labels.is_contiguous(), "ce_grad_: fp32 contiguous lse/scale required");
  c10::cuda::CUDAGuard guard(logits.device());
  check_rc(oslo_ce_grad(logits.data_ptr(), reinterpret_cast<const long long*>(labels.data_ptr<int64_t>()),
                        lse.data_ptr<float>(), scale.data_ptr<float>(), static_cast<int>(logits.size(0)),
                        static_cast<int>(logits.size(1)), static_cast<int>(logits.stride(0)), vocab_start,
                        dt_code(logits), cur_stream()), "ce_grad");
  return logits;
}

void adam_step(Tensor p, const Tensor& g, Tensor m, Tensor v, const optional<Tensor>& p_lp, double lr, double beta1,
               double beta2, double eps, double wd, int64_t step, double grad_scale, const optional<Tensor>& inv_scale) {
  TORCH_CHECK(p.is_cuda() && p.scalar_type() == at::kFloat && m.scalar_type() == at::kFloat && v.scalar_type() == at::kFloat,
              "adam: fp32 master/moment buffers required");
  TORCH_CHECK(p.is_contiguous() && g.is_contiguous() && m.is_contiguous() && v.is_contiguous() &&
                  g.numel() == p.numel() && m.numel() == p.numel() && v.numel() == p.numel(), "adam: size mismatch");
  c10::cuda::CUDAGuard guard(p.device());
  int lp_dt = OSLO_DT_BF16;
  if (p_lp.has_value() && p_lp->defined()) {
    TORCH_CHECK(p_lp->is_contiguous() && p_lp->numel() == p.numel(), "adam: low-precision copy size mismatch");
    lp_dt = dt_code(*p_lp);
    TORCH_CHECK(lp_dt != OSLO_DT_FP32, "adam: low-precision copy must be 16-bit");
  }
  const float bc1 = 1.f - static_cast<float>(std::pow(beta1, static_cast<double>(step)));
  const float bc2 = 1.f - static_cast<float>(std::pow(beta2, static_cast<double>(step)));
  const float* inv = inv_scale.has_value() && inv_scale->defined() ? inv_scale->data_ptr<float>() : nullptr;
  check_rc(oslo_adam(p.data_ptr<float>(), g.data_ptr(), m.data_ptr<float>(), v.data_ptr<float>(),
                     const_cast<void*>(ptr_or_null(p_lp)), p.numel(), static_cast<float>(lr), static_cast<float>(beta1),
                     static_cast<float>(beta2), static_cast<float>(eps), static_cast<float>(wd), bc1, bc2,
                     static_cast<float>(grad_scale), inv, dt_code(g), lp_dt, cur_stream()), "adam");
}

Tensor sumsq(const Tensor& x) {
  TORCH_CHECK(x.is_cuda() && x.is_contiguous(), "sumsq: contiguous CUDA tensor required");
  c10::cuda::CUDAGuard guard(x.device());
  Tensor out = at::zeros({1}, x.options().dtype(at::kFloat));
  check_rc(oslo_sumsq(x.data_ptr(), out.data_ptr<float>(), x.numel(), dt_code(x), cur_stream()), "sumsq");
  return out;
}

Tensor ngram_ban_(const Tensor& tokens, Tensor lprobs, int64_t n) {
  TORCH_CHECK(tokens.is_cuda() && tokens.scalar_type() == at::kLong && tokens.dim() == 2 && tokens.is_contiguous(), "bad tokens");
  TORCH_CHECK(lprobs.is_cuda() && lprobs.scalar_type() == at::kFloat && lprobs.dim() == 2 && lprobs.is_contiguous() &&
                  lprobs.size(0) == tokens.size(0), "lprobs must be fp32 [rows, vocab]");
  c10::cuda::CUDAGuard guard(lprobs.device());
  check_rc(oslo_ngram_ban(reinterpret_cast<const long long*>(tokens.data_ptr<int64_t>()), lprobs.data_ptr<float>(),
                          static_cast<int>(tokens.size(0)), static_cast<int>(tokens.size(1)),
                          static_cast<int>(lprobs.size(1)), static_cast<int>(n),
                          dev_state(lprobs.get_device()).err.data_ptr<int>(), cur_stream()), "ngram_ban");
  return lprobs;
}

void check_attn_operand(const Tensor& t, const char* name) {
  TORCH_CHECK(t.is_cuda() && t.dim() == 4 && t.stride(3) == 1, name, " must be [B,H,S,D] with contiguous D");
  TORCH_CHECK(t.stride(0) % 8 == 0 && t.stride(1) % 8 == 0 && t.stride(2) % 8 == 0 &&
                  reinterpret_cast<uintptr_t>(t.data_ptr()) % 16 == 0, name, " needs 16-byte aligned rows");
}

// impl 0 = mma.sync kernel (attention.cu), 1 = tcgen05/TMEM kernel (attention_sm100.cu)
std::tuple<Tensor, Tensor> flash_fwd(const Tensor& q, const Tensor& k, const Tensor& v, double scale, bool causal,
                                     int64_t window, const optional<Tensor>& kpm, int64_t impl) {
  check_attn_operand(q, "q"); check_attn_operand(k, "k"); check_attn_operand(v, "v");
  c10::cuda::CUDAGuard guard(q.device());
  const int B = q.size(0), H = q.size(1), Sq = q.size(2), D = q.size(3), Sk = k.size(2);
  // output laid out [B, S, H, D] in memory and returned as a [B, H, S, D] view, so merging heads is free
  Tensor o = at::empty({B, Sq, H, D}, q.options()).permute({0, 2, 1, 3});
  Tensor lse = at::empty({B, H, Sq}, q.options().dtype(at::kFloat));
  const uint8_t* mp = nullptr;
  if (kpm.has_value() && kpm->defined()) {
    TORCH_CHECK(kpm->scalar_type() == at::kByte && kpm->is_contiguous() && kpm->size(0) == B && kpm->size(1) == Sk, "bad key padding mask");
    mp = kpm->data_ptr<uint8_t>();
  }
  if (impl == 1) {
    check_rc(oslo_flash_fwd_sm100(q.data_ptr(), k.data_ptr(), v.data_ptr(), o.data_ptr(), lse.data_ptr<float>(), mp, B, H,
                                  Sq, Sk, D, q.stride(0), q.stride(1), q.stride(2), k.stride(0), k.stride(1), k.stride(2),
                                  v.stride(0), v.stride(1), v.stride(2), o.stride(0), o.stride(1), o.stride(2),
                                  static_cast<float>(scale), causal ? 1 : 0, static_cast<int>(window), dt_code(q),
                                  dev_state(q.get_device()).err.data_ptr<int>(), cur_stream()), "flash_fwd_sm100");
    return {o, lse};
  }
  check_rc(oslo_flash_fwd(q.data_ptr(), k.data_ptr(), v.data_ptr(), o.data_ptr(), lse.data_ptr<float>(), mp, B, H, Sq, Sk,
                          D, q.stride(0), q.stride(1), q.stride(2), k.stride(0), k.stride(1), k.stride(2), v.stride(0),
                          v.stride(1), v.stride(2), o.stride(0), o.stride(1), o.stride(2), static_cast<float>(scale),
                          causal ? 1 : 0, static_cast<int>(window), dt_code(q), cur_stream()), "flash_fwd");
  return {o, lse};
}

std::tuple<Tensor, Tensor, Tensor> flash_bwd(const Tensor& dout, const Tensor& q, const Tensor& k, const Tensor& v,
                                             const Tensor& o, const Tensor& lse, double scale, bool causal,
                                             int64_t window, const optional<Tensor>& kpm, int64_t impl) {
  check_attn_operand(q, "q"); check_attn_operand(k, "k"); check_attn_operand(v, "v");
  check_attn_operand(o, "o"); check_attn_operand(dout, "dout");
  c10::cuda::CUDAGuard guard(q.device());
  const int B = q.size(0), H = q.size(1), Sq = q.size(2), D = q.size(3), Sk = k.size(2);
  Tensor dq = at::empty_strided(q.sizes(), q.strides(), q.options());
  Tensor dk = at::empty_strided(k.sizes(), k.strides(), k.options());
  Tensor dv = at::empty_strided(v.sizes(), v.strides(), v.options());
  Tensor delta = at::empty({B, H, Sq}, q.options().dtype(at::kFloat));
  const uint8_t* mp = (kpm.has_value() && kpm->defined()) ? kpm->data_ptr<uint8_t>() : nullptr;
  if (impl == 1) {
    check_rc(oslo_flash_bwd_sm100(q.data_ptr(), k.data_ptr(), v.data_ptr(), o.data_ptr(), dout.data_ptr(),
                                  lse.data_ptr<float>(), delta.data_ptr<float>(), dq.data_ptr(), dk.data_ptr(),
                                  dv.data_ptr(), mp, B, H, Sq, Sk, D, q.stride(0), q.stride(1), q.stride(2), k.stride(0),
                                  k.stride(1), k.stride(2), v.stride(0), v.stride(1), v.stride(2), o.stride(0),
                                  o.stride(1), o.stride(2), dout.stride(0), dout.stride(1), dout.stride(2),
                                  static_cast<float>(scale), causal ? 1 : 0, static_cast<int>(window), dt_code(q),
                                  dev_state(q.get_device()).err.data_ptr<int>(), cur_stream(4)), "flash_bwd_sm100");
    return {dq, dk, dv};
  }
  check_rc(oslo_flash_bwd(q.data_ptr(), k.data_ptr(), v.data_ptr(), o.data_ptr(), dout.data_ptr(), lse.data_ptr<float>(),
                          delta.data_ptr<float>(), nullptr, dq.data_ptr(), dk.data_ptr(), dv.data_ptr(), mp, B, H, Sq, Sk,
                          D, q.stride(0), q.stride(1), q.stride(2), k.stride(0), k.stride(1), k.stride(2), v.stride(0),
                          v.stride(1), v.stride(2), o.stride(0), o.stride(1), o.stride(2), dout.stride(0),
                          dout.stride(1), dout.stride(2), static_cast<float>(scale), causal ? 1 : 0,
                          static_cast<int>(window), dt_code(q), cur_stream(D > 128 ? 4 : 3)), "flash_bwd");
  return {dq, dk, dv};
}

Tensor decode_attn(const Tensor& q, const Tensor& kc, const Tensor& vc, const Tensor& lengths, double scale,
                   int64_t window) {
  TORCH_CHECK(q.is_cuda() && q.dim() == 3 && q.is_contiguous(), "decode_attn: q must be contiguous [B,H,D]");
  TORCH_CHECK(kc.dim() == 4 && kc.is_contiguous() && vc.is_contiguous(), "decode_attn: caches must be contiguous [B,H,T,D]");
  TORCH_CHECK(lengths.scalar_type() == at::kInt && lengths.is_contiguous() && lengths.numel() == q.size(0), "bad lengths");
  c10::cuda::CUDAGuard guard(q.device());
  const int B = q.size(0), H = q.size(1), D = q.size(2), T = kc.size(2);
  const int sms = dev_state(q.get_device()).sms;
  int splits = std::max(1, std::min(32, (2 * sms) / std::max(1, B * H)));
  splits = std::min(splits, std::max(1, T / 32));   // at least one 8-key batch per warp and slice
  Tensor ws = at::empty({B, H, splits, D + 2}, q.options().dtype(at::kFloat));
  Tensor o = at::empty_like(q);
  check_rc(oslo_decode_attn(q.data_ptr(), kc.data_ptr(), vc.data_ptr(), o.data_ptr(), lengths.data_ptr<int>(),
                            ws.data_ptr<float>(), B, H, T, D, splits, static_cast<float>(scale),
                            static_cast<int>(window), dt_code(q), dev_state(q.get_device()).err.data_ptr<int>(),
                            cur_stream(2)), "decode_attn");
  return o;
}

// GEMM fused with a collective over the symmetric buffer of a tensor-parallel group (fused_comm_gemm.cu).
// mode 1: all-reduce, the summed [M,N] is left in the staging matrix at data_off (returned view is built in
// Python); mode 2: reduce-scatter into `out` [M/world, N]; mode 3: all-gather of `a` shards, product into `out`.
int64_t gemm_comm(const Tensor& a, const Tensor& b, int64_t a_mn, int64_t b_mn, const optional<Tensor>& bias,
               const optional<Tensor>& aux, const optional<Tensor>& aux_out, const optional<Tensor>& out, int64_t flags,
               double alpha, int64_t M,
               int64_t N, int64_t K, int64_t peer_bufs_dev, int64_t own_buf, int64_t mc_base, int64_t data_off,
               int64_t flag_off, int64_t flag_bytes, int64_t rank, int64_t world, int64_t epoch, int64_t done_base,
               int64_t mode, bool use_multimem, const optional<Tensor>& trace) {
  check_2d_operand(a, "a");
  check_2d_operand(b, "b");
  TORCH_CHECK(a.scalar_type() == b.scalar_type() && (a.scalar_type() == at::kBFloat16 || a.scalar_type() == at::kHalf),
              "gemm_comm inputs must both be bf16 or fp16");
  c10::cuda::CUDAGuard guard(a.device());
  int fl = static_cast<int>(flags) & ~GEMM_FLAG_FP16;
  if (a.scalar_type() == at::kHalf) fl |= GEMM_FLAG_FP16;
  void* out_ptr = nullptr;
  int ld_out = 0;
  if (mode != 1) {
    TORCH_CHECK(out.has_value() && out->is_cuda() && out->dim() == 2 && out->stride(1) == 1 &&
                    out->scalar_type() == a.scalar_type(), "gemm_comm: bad out");
    TORCH_CHECK(out->size(1) == N && out->size(0) == (mode == 2 ? M / world : M), "gemm_comm: out shape");
    out_ptr = out->data_ptr();
    ld_out = static_cast<int>(out->stride(0));
  }
  int ld_aux_out = 0;
  if (fl & GEMM_FLAG_SAVE_PREACT) {
    TORCH_CHECK(mode == 3 && aux_out.has_value() && aux_out->size(0) == M && aux_out->size(1) == N &&
                    aux_out->stride(1) == 1, "gemm_comm: bad aux_out");
    ld_aux_out = static_cast<int>(aux_out->stride(0));
  }
  if (fl & GEMM_FLAG_BIAS) TORCH_CHECK(bias.has_value() && bias->numel() == N && bias->is_contiguous(), "bad bias");
  int ld_aux = 0;
  if (fl & GEMM_FLAG_RESIDUAL) {
    TORCH_CHECK(mode != 3 && aux.has_value() && aux->dim() == 2 && aux->size(0) == M && aux->size(1) == N &&
                    aux->stride(1) == 1 && aux->scalar_type() == a.scalar_type(), "gemm_comm: bad partial-sum operand");
    ld_aux = static_cast<int>(aux->stride(0));
  }
  auto& st = dev_state(a.get_device());
  // tile shape must be the same on every rank: decide from the problem size only
  const int wide = (N >= 256 && ((M + 127) / 128) * ((N + 255) / 256) >= usable_sms(st) / 2) ? 1 : 0;
  const int rc = oslo_gemm_comm_16bit(
      a.data_ptr(), b.data_ptr(), static_cast<int>(M), static_cast<int>(N), static_cast<int>(K),
      static_cast<int>(a.stride(0)), static_cast<int>(b.stride(0)), static_cast<int>(a_mn), static_cast<int>(b_mn),
      ptr_or_null(bias), (fl & GEMM_FLAG_RESIDUAL) ? aux->data_ptr() : nullptr, ld_aux,
      const_cast<void*>(ptr_or_null(aux_out)), ld_aux_out, fl, static_cast<float>(alpha),
      reinterpret_cast<void* const*>(peer_bufs_dev), reinterpret_cast<void*>(own_buf), reinterpret_cast<void*>(mc_base),
      data_off, flag_off, flag_bytes, static_cast<int>(rank), static_cast<int>(world), static_cast<unsigned>(epoch),
      static_cast<unsigned>(done_base), static_cast<int>(mode), use_multimem ? 1 : 0, out_ptr, ld_out, wide,
      trace.has_value() && trace->defined() ? reinterpret_cast<unsigned long long*>(trace->data_ptr<int64_t>()) : nullptr,
      st.err.data_ptr<int>(), usable_sms(st), cur_stream());
  check_rc(rc, "gemm_comm");
  // how far this call advances the slot's completion counter (the caller keeps the running total)
  const int64_t bn = wide ? 256 : 128;
  return mode == 1 ? ((M + 127) / 128) * ((N + bn - 1) / bn) * 4 : 0;
}

// In-place all-reduce of a symmetric buffer. ptr tables are device arrays of `world` addresses.
void allreduce_symm(int64_t peer_ptrs_dev, int64_t mc_ptr, int64_t signal_ptrs_dev, Tensor out, int64_t numel,
                    int64_t rank, int64_t world, bool use_multimem) {
  c10::cuda::CUDAGuard guard(out.device());
  auto& st = dev_state(out.get_device());
  check_rc(oslo_allreduce_symm(reinterpret_cast<void* const*>(peer_ptrs_dev), reinterpret_cast<void*>(mc_ptr),
                               reinterpret_cast<uint32_t* const*>(signal_ptrs_dev), out.data_ptr(), numel,
                               static_cast<int>(rank), static_cast<int>(world), dt_code(out), use_multimem ? 1 : 0,
                               st.err.data_ptr<int>(), cur_stream()), "allreduce_symm");
}

// (max, sum exp, label logit) per row combined over the ranks of a tensor-parallel group, in place
void ce_combine(Tensor mx, Tensor se, Tensor tg, int64_t peer_ptrs_dev, int64_t signal_ptrs_dev, Tensor counters,
                int64_t cap, int64_t rank, int64_t world) {
  TORCH_CHECK(mx.is_cuda() && mx.scalar_type() == at::kFloat && mx.is_contiguous() && se.is_contiguous() &&
                  tg.is_contiguous() && se.scalar_type() == at::kFloat && tg.scalar_type() == at::kFloat &&
                  se.numel() == mx.numel() && tg.numel() == mx.numel(), "ce_combine: fp32 contiguous vectors of one length");
  c10::cuda::CUDAGuard guard(mx.device());
  auto& st = dev_state(mx.get_device());
  check_rc(oslo_ce_combine(mx.data_ptr<float>(), se.data_ptr<float>(), tg.data_ptr<float>(), mx.data_ptr<float>(),
                           se.data_ptr<float>(), tg.data_ptr<float>(), reinterpret_cast<void* const*>(peer_ptrs_dev),
                           reinterpret_cast<uint32_t* const*>(signal_ptrs_dev),
                           reinterpret_cast<uint32_t*>(counters.data_ptr<int>()), static_cast<int>(mx.numel()),
                           static_cast<int>(cap), static_cast<int>(rank), static_cast<int>(world),
                           st.err.data_ptr<int>(), cur_stream()), "ce_combine");
}

// One bucket of the data-parallel gradient reduce-scatter / parameter all-gather on a symmetric flat buffer.
// `like` names the device and (reduce-scatter) the 16-bit dtype; the buffer itself is given by its address tables.
void dp_reduce_scatter(const Tensor& like, int64_t peer_ptrs_dev, int64_t mc_ptr, int64_t signal_ptrs_dev, int64_t lo,
                       int64_t hi, int64_t shard, int64_t rank, int64_t world, bool use_multimem) {
  c10::cuda::CUDAGuard guard(like.device());
  auto& st = dev_state(like.get_device());
  check_rc(oslo_dp_reduce_scatter(reinterpret_cast<void* const*>(peer_ptrs_dev), reinterpret_cast<void*>(mc_ptr),
                                  reinterpret_cast<uint32_t* const*>(signal_ptrs_dev), lo, hi, shard,
                                  static_cast<int>(rank), static_cast<int>(world), dt_code(like), use_multimem ? 1 : 0,
                                  st.err.data_ptr<int>(), cur_stream()), "dp_reduce_scatter");
}
void dp_all_gather(const Tensor& like, int64_t peer_ptrs_dev, int64_t mc_ptr, int64_t signal_ptrs_dev, int64_t lo,
                   int64_t hi, int64_t shard, int64_t rank, int64_t world, bool use_multimem) {
  c10::cuda::CUDAGuard guard(like.device());
  auto& st = dev_state(like.get_device());
  check_rc(oslo_dp_all_gather(reinterpret_cast<void* const*>(peer_ptrs_dev), reinterpret_cast<void*>(mc_ptr),
                              reinterpret_cast<uint32_t* const*>(signal_ptrs_dev), lo, hi, shard, static_cast<int>(rank),
                              static_cast<int>(world), use_multimem ? 1 : 0, st.err.data_ptr<int>(), cur_stream()),
           "dp_all_gather");
}

// y [M, N] = act([x1 | x2] @ w^T + bias) for M <= 4 rows; w [N, K1 + K2]; x1 / x2 are 2-D with contiguous last dims
Tensor gemv_rows(const Tensor& x1, const optional<Tensor>& x2, const Tensor& w, const optional<Tensor>& bias,
                 int64_t gelu_from, const optional<Tensor>& res) {
  check_2d_operand(x1, "x1");
  check_2d_operand(w, "w");
  const bool two = x2.has_value() && x2->defined();
  if (two) check_2d_operand(*x2, "x2");
  const int64_t M = x1.size(0), K1 = x1.size(1), K2 = two ? x2->size(1) : 0, N = w.size(0);
  TORCH_CHECK(w.size(1) == K1 + K2 && (!two || x2->size(0) == M), "gemv_rows: shapes do not match");
  TORCH_CHECK(x1.scalar_type() == w.scalar_type() && (!two || x2->scalar_type() == w.scalar_type()), "gemv_rows: dtypes differ");
  const bool has_bias = bias.has_value() && bias->defined();
  if (has_bias) TORCH_CHECK(bias->numel() == N && bias->scalar_type() == w.scalar_type() && bias->is_contiguous(), "bad bias");
  const bool has_res = res.has_value() && res->defined();
  if (has_res)
    TORCH_CHECK(res->dim() == 2 && res->size(0) == M && res->size(1) == N && res->stride(1) == 1 &&
                    res->scalar_type() == w.scalar_type(), "bad residual");
  c10::cuda::CUDAGuard guard(x1.device());
  Tensor y = at::empty({M, N}, x1.options());
  auto& st = dev_state(x1.get_device());
  check_rc(oslo_gemv_rows(x1.data_ptr(), static_cast<int>(x1.stride(0)), static_cast<int>(K1),
                          two ? x2->data_ptr() : nullptr, two ? static_cast<int>(x2->stride(0)) : 0, static_cast<int>(K2),
                          w.data_ptr(), static_cast<int>(w.stride(0)), has_bias ? bias->data_ptr() : nullptr,
                          has_res ? res->data_ptr() : nullptr, has_res ? static_cast<int>(res->stride(0)) : 0, y.data_ptr(),
                          static_cast<int>(N), static_cast<int>(M), static_cast<int>(N), static_cast<int>(gelu_from),
                          dt_code(x1), usable_sms(st), cur_stream()), "gemv_rows");
  return y;
}

// GPT-J rotary on q, k ([B, H*D] row slices) + append of k, v to the static cache at the device-side position
Tensor rotary_append(const Tensor& q, const Tensor& k, const Tensor& v, Tensor kc, Tensor vc, const Tensor& lengths,
                     const Tensor& write_index, int64_t rotary_dim, double base) {
  TORCH_CHECK(q.is_cuda() && q.dim() == 2 && k.dim() == 2 && v.dim() == 2 && q.stride(1) == 1 && k.stride(1) == 1 &&
                  v.stride(1) == 1, "rotary_append: q, k, v must be [B, H*D] with contiguous last dim");
  TORCH_CHECK(kc.dim() == 4 && kc.is_contiguous() && vc.is_contiguous() && kc.sizes() == vc.sizes(), "bad cache");
  TORCH_CHECK(lengths.scalar_type() == at::kInt && write_index.scalar_type() == at::kLong, "bad position tensors");
  const int64_t B = kc.size(0), H = kc.size(1), T = kc.size(2), D = kc.size(3);
  TORCH_CHECK(q.size(0) == B && q.size(1) == H * D && k.size(1) == H * D && v.size(1) == H * D, "shape mismatch");
  c10::cuda::CUDAGuard guard(q.device());
  Tensor q_out = at::empty({B, H, D}, q.options());
  check_rc(oslo_rotary_append(q.data_ptr(), k.data_ptr(), v.data_ptr(), q.stride(0), k.stride(0), v.stride(0),
                              q_out.data_ptr(), kc.data_ptr(), vc.data_ptr(), lengths.data_ptr<int>(),
                              reinterpret_cast<const long long*>(write_index.data_ptr<int64_t>()), static_cast<int>(B),
                              static_cast<int>(H), static_cast<int>(D), static_cast<int>(T), static_cast<int>(rotary_dim),
                              static_cast<float>(base), dt_code(q), dev_state(q.get_device()).err.data_ptr<int>(),
                              cur_stream()), "rotary_append");
  return q_out;
}

// Vocab-parallel embedding: ids int64 [tokens], weight = this rank's [hi - lo, H] shard; returns [tokens, H]
Tensor vocab_embed(const Tensor& ids, const Tensor& weight, int64_t lo, int64_t hi, int64_t peer_ptrs_dev,
                   int64_t mc_ptr, int64_t signal_ptrs_dev, Tensor counters, int64_t half_bytes, int64_t rank,
                   int64_t world, bool use_multimem) {
  TORCH_CHECK(ids.is_cuda() && ids.scalar_type() == at::kLong && ids.is_contiguous(), "vocab_embed: ids must be contiguous int64");
  TORCH_CHECK(weight.is_cuda() && weight.dim() == 2 && weight.is_contiguous() && weight.size(0) == hi - lo, "vocab_embed: bad weight shard");
  TORCH_CHECK(counters.is_cuda() && counters.scalar_type() == at::kInt && counters.numel() >= 64, "vocab_embed: bad counters");
  c10::cuda::CUDAGuard guard(ids.device());
  const int64_t tokens = ids.numel(), H = weight.size(1);
  Tensor out = at::empty({tokens, H}, weight.options());
  auto& st = dev_state(ids.get_device());
  check_rc(oslo_vocab_embed(reinterpret_cast<const long long*>(ids.data_ptr<int64_t>()), weight.data_ptr(), out.data_ptr(),
                            reinterpret_cast<void* const*>(peer_ptrs_dev), reinterpret_cast<void*>(mc_ptr),
                            reinterpret_cast<uint32_t* const*>(signal_ptrs_dev),
                            reinterpret_cast<uint32_t*>(counters.data_ptr<int>()), tokens, static_cast<int>(H), lo, hi,
                            half_bytes, static_cast<int>(rank), static_cast<int>(world), dt_code(weight),
                            use_multimem ? 1 : 0, st.err.data_ptr<int>(), usable_sms(st), cur_stream()), "vocab_embed");
  return out;
}

// Wait (bounded by limit_ms, at most 1000) until flag[0] >= target; returns the nanoseconds spent. A wait that runs
// out leaves ERR_WAIT_PEER in the device error word, exactly like the waits inside the communication kernels.
Tensor wait_probe(const Tensor& flag, int64_t target, double limit_ms) {
  TORCH_CHECK(flag.is_cuda() && flag.scalar_type() == at::kInt && flag.numel() >= 1, "wait_probe: int32 CUDA flag");
  c10::cuda::CUDAGuard guard(flag.device());
  Tensor waited = at::zeros({1}, flag.options().dtype(at::kLong));
  auto& st = dev_state(flag.get_device());
  check_rc(oslo_wait_probe(reinterpret_cast<const uint32_t*>(flag.data_ptr<int>()), static_cast<uint32_t>(target),
                           static_cast<unsigned long long>(limit_ms * 1e6), st.err.data_ptr<int>(),
                           reinterpret_cast<unsigned long long*>(waited.data_ptr<int64_t>()), cur_stream()), "wait_probe");
  return waited;
}

// In-place one-kernel all-reduce of a small tensor through two alternating staging halves of a symmetric buffer.
void allreduce_oneshot(Tensor x, int64_t peer_ptrs_dev, int64_t mc_ptr, int64_t signal_ptrs_dev, Tensor counters,
                       int64_t stage_off, int64_t half_bytes, int64_t rank, int64_t world, bool use_multimem) {
  TORCH_CHECK(x.is_cuda() && x.is_contiguous() && counters.is_cuda() && counters.scalar_type() == at::kInt &&
                  counters.numel() >= 64, "allreduce_oneshot: bad arguments");
  c10::cuda::CUDAGuard guard(x.device());
  auto& st = dev_state(x.get_device());
  check_rc(oslo_allreduce_oneshot(x.data_ptr(), x.data_ptr(), reinterpret_cast<void* const*>(peer_ptrs_dev),
                                  reinterpret_cast<void*>(mc_ptr), reinterpret_cast<uint32_t* const*>(signal_ptrs_dev),
                                  reinterpret_cast<uint32_t*>(counters.data_ptr<int>()), x.numel(), stage_off, half_bytes,
                                  static_cast<int>(rank), static_cast<int>(world), dt_code(x), use_multimem ? 1 : 0,
                                  st.err.data_ptr<int>(), cur_stream()), "allreduce_oneshot");
}


// ---------------------------------------------------------------------- RMS norms, residual join, gated MLP
void check_rows(const Tensor& t, const char* name) {
  TORCH_CHECK(t.is_cuda() && t.dim() == 2 && t.stride(1) == 1 && t.stride(0) >= t.size(1), name,
              " must be a 2-D CUDA tensor with a contiguous last dim");
}
const uint8_t* keep_ptr(const optional<Tensor>& keep, int64_t rows, int64_t cols, int64_t& ld) {
  ld = 0;
  if (!keep.has_value() || !keep->defined()) return nullptr;
  TORCH_CHECK(keep->is_cuda() && keep->scalar_type() == at::kByte && keep->dim() == 2 && keep->size(0) == rows &&
                  keep->size(1) >= cols && keep->stride(1) == 1, "keep must be uint8 [rows, positions]");
  ld = keep->stride(0);
  return keep->data_ptr<uint8_t>();
}

Tensor rms_norm(const Tensor& x, const Tensor& w, double eps, double offset) {
  check_rows(x, "x");
  TORCH_CHECK(w.is_cuda() && w.is_contiguous() && (w.numel() == x.size(1) || w.numel() == 1), "rms_norm: weight size");
  TORCH_CHECK(x.scalar_type() == w.scalar_type() || x.scalar_type() == at::kFloat, "rms_norm: x is fp32 or has the weight's type");
  c10::cuda::CUDAGuard guard(x.device());
  Tensor out = at::empty({x.size(0), x.size(1)}, w.options());
  check_rc(oslo_rms_norm(x.data_ptr(), x.stride(0), x.scalar_type() == at::kFloat, w.data_ptr(), w.numel() != x.size(1), out.data_ptr(),
                         out.stride(0), x.size(0), static_cast<int>(x.size(1)), static_cast<float>(eps), static_cast<float>(offset), dt_code(w),
                         cur_stream()), "rms_norm");
  return out;
}

std::tuple<Tensor, Tensor> residual_join(const Tensor& x, const Tensor& y, const optional<Tensor>& slots,
                                         const optional<Tensor>& slot_weights, const Tensor& gate, const Tensor& gate_bias,
                                         const Tensor& w_post, const optional<Tensor>& w_next, double eps) {
  check_rows(x, "x"); check_rows(y, "y"); check_rows(gate, "gate");
  const int64_t rows = x.size(0), cols = x.size(1);
  TORCH_CHECK(x.scalar_type() == at::kFloat && x.is_contiguous(), "residual_join: the residual stream is contiguous fp32");
  TORCH_CHECK(y.size(1) == cols && gate.size(0) == rows && gate.size(1) == cols && gate_bias.numel() == cols &&
                  w_post.numel() == cols, "residual_join: sizes");
  TORCH_CHECK(y.scalar_type() == w_post.scalar_type() && gate.scalar_type() == y.scalar_type() &&
                  gate_bias.scalar_type() == y.scalar_type(), "residual_join: dtypes");
  int top = 1;
  const float* sw = nullptr;
  const int* sl = nullptr;
  if (slot_weights.has_value() && slot_weights->defined()) {
    TORCH_CHECK(slot_weights->is_contiguous() && slot_weights->scalar_type() == at::kFloat && slot_weights->size(0) == rows, "slot weights");
    top = static_cast<int>(slot_weights->size(1));
    sw = slot_weights->data_ptr<float>();
    if (slots.has_value() && slots->defined()) {
      TORCH_CHECK(slots->is_contiguous() && slots->scalar_type() == at::kInt && slots->numel() == rows * top, "slots");
      sl = slots->data_ptr<int>();
    } else {
      TORCH_CHECK(y.size(0) == rows * top, "residual_join: one row of y per (token, choice)");
    }
  } else {
    TORCH_CHECK(y.size(0) == rows, "residual_join: rows of y");
  }
  const bool next = w_next.has_value() && w_next->defined();
  if (next) TORCH_CHECK(w_next->numel() == cols && w_next->scalar_type() == w_post.scalar_type(), "residual_join: next weight");
  c10::cuda::CUDAGuard guard(x.device());
  Tensor xo = at::empty_like(x);
  Tensor h = at::empty({next ? rows : 0, cols}, y.options());
  check_rc(oslo_residual_join(x.data_ptr<float>(), y.data_ptr(), y.stride(0), sl, sw, top, gate.data_ptr(), gate.stride(0),
                              gate_bias.data_ptr(), w_post.data_ptr(), ptr_or_null(w_next), xo.data_ptr<float>(),
                              next ? h.data_ptr() : nullptr, rows, static_cast<int>(cols), static_cast<float>(eps), dt_code(y),
                              cur_stream()), "residual_join");
  return {xo, h};
}

Tensor silu_mul(const Tensor& gate, const Tensor& up) {
  check_rows(gate, "gate"); check_rows(up, "up");
  TORCH_CHECK(gate.sizes() == up.sizes() && gate.scalar_type() == up.scalar_type(), "silu_mul: operands differ");
  c10::cuda::CUDAGuard guard(gate.device());
  Tensor out = at::empty({gate.size(0), gate.size(1)}, gate.options());
  check_rc(oslo_silu_mul(gate.data_ptr(), gate.stride(0), up.data_ptr(), up.stride(0), out.data_ptr(), gate.size(0),
                         static_cast<int>(gate.size(1)), dt_code(gate), cur_stream()), "silu_mul");
  return out;
}

Tensor clamped_glu(const Tensor& gate, const Tensor& up, double limit, double alpha) {
  check_rows(gate, "gate"); check_rows(up, "up");
  TORCH_CHECK(gate.sizes() == up.sizes() && gate.scalar_type() == up.scalar_type(), "clamped_glu: operands differ");
  c10::cuda::CUDAGuard guard(gate.device());
  Tensor out = at::empty({gate.size(0), gate.size(1)}, gate.options());
  check_rc(oslo_clamped_glu(gate.data_ptr(), gate.stride(0), up.data_ptr(), up.stride(0), out.data_ptr(), gate.size(0),
                            static_cast<int>(gate.size(1)), static_cast<float>(limit), static_cast<float>(alpha), dt_code(gate),
                            cur_stream()), "clamped_glu");
  return out;
}

// up to three results join the stream; h1 / h2: the sum normed with w1 / w2 (empty without them)
void check_state(const Tensor& state, int64_t n);
using OptList = c10::List<optional<Tensor>>;

// up to three branches y[i] with weights w[i] (normed[i] or elementwise), the sums of top[i] rows slots[i] where top[i] > 0; two norms of
// the sum, or a copy of it; for single tokens also the convolution of the first norm (conv_w, prev). See oslo_kernels.h
std::tuple<Tensor, Tensor, Tensor, Tensor> branch_join(const Tensor& x, at::TensorList y, const OptList& w, at::ArrayRef<double> factor,
                                                       at::IntArrayRef normed, const OptList& slots, at::IntArrayRef top, double mult,
                                                       double eps, const optional<Tensor>& w1, const optional<Tensor>& w2, bool copy,
                                                       const optional<Tensor>& conv_w, optional<Tensor> prev,
                                                       const optional<Tensor>& keep) {
  check_rows(x, "x");
  const int64_t rows = x.size(0), cols = x.size(1), n = y.size();
  TORCH_CHECK(x.scalar_type() == at::kFloat && x.is_contiguous(), "branch_join: the residual stream is contiguous fp32");
  TORCH_CHECK(n >= 1 && n <= 3 && w.size() == static_cast<size_t>(n) && slots.size() == static_cast<size_t>(n) && static_cast<int64_t>(factor.size()) == n &&
                  static_cast<int64_t>(normed.size()) == n && static_cast<int64_t>(top.size()) == n, "branch_join: one to three branches");
  const auto type = y[0].scalar_type();
  OsloBranchJoin a{};
  a.x = x.data_ptr<float>();
  a.n = static_cast<int>(n);
  const auto has = [](const optional<Tensor>& t) { return t.has_value() && t->defined(); };
  const auto vec_ok = [&](const optional<Tensor>& v, bool one) {
    return !has(v) || (v->is_cuda() && v->is_contiguous() && (v->numel() == cols || (one && v->numel() == 1)) && v->scalar_type() == type);
  };
  for (int64_t i = 0; i < n; ++i) {
    const optional<Tensor> wi = w.get(i), si = slots.get(i);
    check_rows(y[i], "y");
    TORCH_CHECK(y[i].size(1) == cols && y[i].scalar_type() == type && vec_ok(wi, false) && top[i] >= 0, "branch_join: branch");
    TORCH_CHECK(top[i] == 0 ? y[i].size(0) == rows : (has(si) || y[i].size(0) == rows * top[i]), "branch_join: rows of a branch");
    if (top[i] > 0 && has(si)) {
      TORCH_CHECK(si->is_cuda() && si->is_contiguous() && si->scalar_type() == at::kInt && si->numel() == rows * top[i], "branch_join: slots");
      a.slots[i] = si->data_ptr<int>();
    }
    a.y[i] = y[i].data_ptr(); a.ldy[i] = y[i].stride(0); a.w[i] = ptr_or_null(wi); a.normed[i] = normed[i] != 0;
    a.top[i] = static_cast<int>(top[i]); a.factor[i] = static_cast<float>(factor[i]);
  }
  TORCH_CHECK(vec_ok(w1, true) && vec_ok(w2, true) && (has(w1) || !has(w2)) && !(copy && has(w1)), "branch_join: norm weights");
  a.mult = static_cast<float>(mult); a.eps = static_cast<float>(eps);
  a.w1 = ptr_or_null(w1); a.w2 = ptr_or_null(w2); a.copy = copy;
  a.one1 = has(w1) && w1->numel() != cols; a.one2 = has(w2) && w2->numel() != cols;
  if (has(conv_w)) {
    TORCH_CHECK(conv_w->dim() == 2 && conv_w->is_contiguous() && conv_w->size(0) == cols && conv_w->scalar_type() == type && has(w1), "branch_join: convolution");
    a.conv_w = conv_w->data_ptr();
    a.taps = static_cast<int>(conv_w->size(1));
    if (has(prev) && a.taps > 1) {
      check_state(*prev, rows * (a.taps - 1) * cols);
      a.prev = prev->data_ptr<float>();
    }
    int64_t ld_keep = 0;
    a.keep = keep_ptr(keep, rows, 1, ld_keep);
    a.ld_keep = ld_keep;
  }
  c10::cuda::CUDAGuard guard(x.device());
  const auto out = y[0].options();
  Tensor xo = at::empty_like(x);
  Tensor h1 = at::empty({has(w1) || copy ? rows : 0, cols}, out), h2 = at::empty({has(w2) ? rows : 0, cols}, out);
  Tensor co = at::empty({has(conv_w) ? rows : 0, cols}, out);
  a.x_out = xo.data_ptr<float>();
  a.h1 = has(w1) || copy ? h1.data_ptr() : nullptr;
  a.h2 = has(w2) ? h2.data_ptr() : nullptr;
  a.conv_out = has(conv_w) ? co.data_ptr() : nullptr;
  check_rc(oslo_branch_join(&a, rows, static_cast<int>(cols), dt_code(y[0]), cur_stream()), "branch_join");
  return {xo, h1, h2, co};
}

// gelu_tanh(z) times the tokens' columns `first` and on of table [vocab, *]
Tensor token_gate(const Tensor& z, const Tensor& ids, const Tensor& table, int64_t first) {
  check_rows(z, "z");
  TORCH_CHECK(ids.is_cuda() && ids.dim() == 1 && ids.scalar_type() == at::kLong && ids.size(0) == z.size(0), "token_gate: ids");
  TORCH_CHECK(table.dim() == 2 && table.stride(1) == 1 && table.scalar_type() == z.scalar_type() && first >= 0 &&
                  first + z.size(1) <= table.size(1), "token_gate: table");
  c10::cuda::CUDAGuard guard(z.device());
  Tensor out = at::empty({z.size(0), z.size(1)}, z.options());
  check_rc(oslo_token_gate(z.data_ptr(), z.stride(0), reinterpret_cast<const long long*>(ids.data_ptr<int64_t>()), ids.stride(0), table.data_ptr(),
                           table.stride(0), table.size(0), static_cast<int>(first), out.data_ptr(), z.size(0),
                           static_cast<int>(z.size(1)), dt_code(z), dev_state(z.get_device()).err.data_ptr<int>(), cur_stream()),
           "token_gate");
  return out;
}

Tensor gated_rms_norm(const Tensor& o, const Tensor& w, const Tensor& gate, double eps, int64_t group, int64_t act,
                      const optional<Tensor>& z, const optional<Tensor>& m) {
  check_rows(o, "o"); check_rows(gate, "gate");
  TORCH_CHECK(o.scalar_type() == at::kFloat && o.is_contiguous() && w.is_contiguous() && w.numel() == o.size(1) &&
                  gate.size(0) == o.size(0) && gate.size(1) == o.size(1) && gate.scalar_type() == w.scalar_type() && group > 0 &&
                  o.size(1) % group == 0, "gated_rms_norm: operands");
  for (const optional<Tensor>* t : {&z, &m})
    TORCH_CHECK(!ptr_or_null(*t) || ((*t)->is_contiguous() && (*t)->scalar_type() == at::kFloat && (*t)->numel() == o.size(0) * (o.size(1) / group)),
                "gated_rms_norm: normalizer");
  c10::cuda::CUDAGuard guard(o.device());
  Tensor out = at::empty({o.size(0), o.size(1)}, w.options());
  check_rc(oslo_gated_rms_norm(o.data_ptr<float>(), w.data_ptr(), gate.data_ptr(), gate.stride(0), out.data_ptr(),
                               static_cast<const float*>(ptr_or_null(z)), static_cast<const float*>(ptr_or_null(m)), o.size(0),
                               static_cast<int>(o.size(1)), static_cast<int>(group), static_cast<float>(eps), static_cast<int>(act),
                               dt_code(w), cur_stream()), "gated_rms_norm");
  return out;
}

// residual streams take a sublayer's result (y, ...; none: they stay) and the next sublayer's input is read from them
std::tuple<Tensor, Tensor> hyper_join(const Tensor& x, const optional<Tensor>& y, const optional<Tensor>& slots,
                                      const optional<Tensor>& weights, const optional<Tensor>& choice, int64_t experts,
                                      const optional<Tensor>& own, const optional<Tensor>& shared, const optional<Tensor>& gate,
                                      const optional<Tensor>& w_out, const optional<Tensor>& mix, const optional<Tensor>& w_in,
                                      const Tensor& w_norm, double eps, double scale) {
  TORCH_CHECK(x.is_cuda() && x.dim() == 3 && x.stride(2) == 1 && x.scalar_type() == at::kFloat, "hyper_join: streams are fp32 [rows, streams, cols]");
  const int64_t rows = x.size(0), n = x.size(1), cols = x.size(2);
  auto has = [](const optional<Tensor>& t) { return t.has_value() && t->defined(); };
  auto param = [&](const optional<Tensor>& t, int64_t numel, const char* what) {
    TORCH_CHECK(!has(t) || (t->is_contiguous() && t->numel() == numel && t->scalar_type() == w_norm.scalar_type()), what);
  };
  auto matrix = [&](const optional<Tensor>& t, int64_t width, const char* what) {
    if (has(t)) {
      check_rows(*t, what);
      TORCH_CHECK(t->size(0) == rows && t->size(1) == width && t->scalar_type() == w_norm.scalar_type(), what);
    }
  };
  TORCH_CHECK(w_norm.is_contiguous() && w_norm.numel() == cols, "hyper_join: norm weight");
  param(w_in, n, "hyper_join: w_in"); param(w_out, n, "hyper_join: w_out"); param(mix, n * n, "hyper_join: mix");
  matrix(shared, cols, "hyper_join: shared"); matrix(own, cols, "hyper_join: own rows"); matrix(gate, 1, "hyper_join: gate");
  TORCH_CHECK(has(shared) == has(gate) && (!has(choice) || has(own)), "hyper_join: operands that belong together");
  int top = 0;
  if (has(y)) {
    check_rows(*y, "y");
    TORCH_CHECK(has(w_out) && has(mix) && y->size(1) == cols && y->scalar_type() == w_norm.scalar_type(), "hyper_join: result");
    if (has(weights)) {
      TORCH_CHECK(weights->is_contiguous() && weights->scalar_type() == at::kFloat && weights->dim() == 2 && weights->size(0) == rows, "hyper_join: weights");
      top = static_cast<int>(weights->size(1));
      for (const optional<Tensor>* t : {&slots, &choice})
        TORCH_CHECK(!has(*t) || ((*t)->is_contiguous() && (*t)->scalar_type() == at::kInt && (*t)->numel() == rows * top), "hyper_join: slots / choices");
      TORCH_CHECK(has(slots) || y->size(0) == rows * top, "hyper_join: one row of y per (token, choice)");
    } else {
      TORCH_CHECK(y->size(0) == rows, "hyper_join: rows of y");
    }
  }
  c10::cuda::CUDAGuard guard(x.device());
  Tensor xo = at::empty({has(y) ? rows : 0, n, cols}, x.options());
  Tensor h = at::empty({rows, cols}, w_norm.options());
  const bool experts_rows = has(y) && has(weights);
  check_rc(oslo_hyper_join(x.data_ptr<float>(), x.stride(0), x.stride(1), ptr_or_null(y), has(y) ? y->stride(0) : 0,
                           experts_rows && has(slots) ? slots->data_ptr<int>() : nullptr, experts_rows ? weights->data_ptr<float>() : nullptr,
                           top, experts_rows && has(choice) ? choice->data_ptr<int>() : nullptr, static_cast<int>(experts),
                           ptr_or_null(own), has(own) ? own->stride(0) : 0, ptr_or_null(shared), has(shared) ? shared->stride(0) : 0,
                           ptr_or_null(gate), has(gate) ? gate->stride(0) : 0, ptr_or_null(w_out), ptr_or_null(mix), ptr_or_null(w_in),
                           w_norm.data_ptr(), has(y) ? xo.data_ptr<float>() : nullptr, h.data_ptr(), rows, static_cast<int>(n),
                           static_cast<int>(cols), static_cast<float>(eps), static_cast<float>(scale), dt_code(w_norm), cur_stream()),
           "hyper_join");
  return {xo, h};
}

// x [P, M <= 4, K] (rows of a part contiguous in K), w [P, N, K] -> [P, M, N]
Tensor gemv_stacked(const Tensor& x, const Tensor& w) {
  TORCH_CHECK(x.is_cuda() && x.dim() == 3 && w.dim() == 3 && x.stride(2) == 1 && w.is_contiguous() && x.size(0) == w.size(0) &&
                  x.size(2) == w.size(2) && x.scalar_type() == w.scalar_type(), "gemv_stacked: operands");
  c10::cuda::CUDAGuard guard(x.device());
  Tensor out = at::empty({x.size(0), x.size(1), w.size(1)}, x.options());
  check_rc(oslo_gemv_stacked(x.data_ptr(), static_cast<int>(x.stride(1)), x.stride(0), w.data_ptr(), static_cast<int>(w.size(2)),
                             w.size(1) * w.size(2), out.data_ptr(), static_cast<int>(x.size(0)), static_cast<int>(x.size(1)),
                             static_cast<int>(w.size(1)), static_cast<int>(w.size(2)), dt_code(x), dev_state(x.get_device()).sms,
                             cur_stream()), "gemv_stacked");
  return out;
}

// ---------------------------------------------------------------------- linear recurrences
void check_recurrence(const Tensor& q, const Tensor& f, const Tensor& v, const Tensor& f_bias, const Tensor& lower, int64_t heads,
                      int64_t dim, int64_t vdim) {
  check_rows(q, "q"); check_rows(f, "f"); check_rows(v, "v");
  TORCH_CHECK(q.size(1) == heads * dim && f.size(1) == heads * dim && v.size(1) == heads * vdim && f.size(0) == q.size(0) &&
                  v.size(0) == q.size(0), "recurrence: projection sizes");
  TORCH_CHECK(f_bias.is_contiguous() && lower.is_contiguous() && f_bias.numel() == heads * dim && lower.numel() == heads * dim,
              "recurrence: gate bias / lower bound sizes");
  TORCH_CHECK(f.scalar_type() == q.scalar_type() && v.scalar_type() == q.scalar_type() && f_bias.scalar_type() == q.scalar_type() &&
                  lower.scalar_type() == q.scalar_type(), "recurrence: dtypes");
}

struct RecurrenceRule {
  int rule = 0;
  const Tensor *f_bias = nullptr, *lower = nullptr, *z = nullptr, *head_decay = nullptr;
};

Tensor run_recurrence(const RecurrenceRule& r, const Tensor& q, const Tensor& f, const Tensor& v, const optional<Tensor>& keep,
                      const optional<Tensor>& state, int64_t batch, int64_t heads, int64_t dim, int64_t vdim, int64_t chunks) {
  TORCH_CHECK(batch > 0 && q.size(0) % batch == 0, "recurrence: rows are not batch x positions");
  const int64_t S = q.size(0) / batch;
  int64_t ld_keep = 0;
  const uint8_t* kp = keep_ptr(keep, batch, S, ld_keep);
  float* st = nullptr;
  if (state.has_value() && state->defined()) {
    TORCH_CHECK(state->is_contiguous() && state->scalar_type() == at::kFloat && state->numel() == batch * heads * dim * vdim, "recurrence: state");
    st = state->data_ptr<float>();
  }
  c10::cuda::CUDAGuard guard(q.device());
  const int sms = dev_state(q.get_device()).sms;
  int nch = chunks > 0 ? static_cast<int>(chunks)
                       : oslo_recurrence_chunks(r.rule, static_cast<int>(batch), static_cast<int>(S), static_cast<int>(heads),
                                                static_cast<int>(dim), static_cast<int>(vdim), sms);
  const auto f32 = q.options().dtype(at::kFloat);
  Tensor out = at::empty({batch, S, heads, vdim}, f32);
  Tensor ws, decay;
  if (nch > 1) {
    ws = at::empty({batch, nch, heads, dim, vdim}, f32);
    decay = at::empty({batch, nch, heads, dim}, f32);
  }
  check_rc(oslo_recurrence(r.rule, q.data_ptr(), q.stride(0), f.data_ptr(), f.stride(0), v.data_ptr(), v.stride(0),
                           r.f_bias ? r.f_bias->data_ptr() : nullptr, r.lower ? r.lower->data_ptr() : nullptr,
                           r.z ? r.z->data_ptr<float>() : nullptr, r.z ? r.z->stride(0) : 0,
                           r.head_decay ? r.head_decay->data_ptr<float>() : nullptr, kp, ld_keep, st, out.data_ptr<float>(),
                           nch > 1 ? ws.data_ptr<float>() : nullptr, nch > 1 ? decay.data_ptr<float>() : nullptr, nch,
                           static_cast<int>(batch), static_cast<int>(S), static_cast<int>(heads), static_cast<int>(dim),
                           static_cast<int>(vdim), dt_code(q), cur_stream(nch > 1 ? 3 : 1)), "recurrence");
  return out;
}

Tensor recurrence(const Tensor& q, const Tensor& f, const Tensor& v, const Tensor& f_bias, const Tensor& lower,
                  const optional<Tensor>& keep, const optional<Tensor>& state, int64_t batch, int64_t heads, int64_t dim,
                  int64_t vdim, int64_t chunks) {
  check_recurrence(q, f, v, f_bias, lower, heads, dim, vdim);
  RecurrenceRule r;
  r.f_bias = &f_bias; r.lower = &lower;
  return run_recurrence(r, q, f, v, keep, state, batch, heads, dim, vdim, chunks);
}

void check_qkv_rows(const Tensor& q, const Tensor& k, const Tensor& v, int64_t heads, int64_t dim, int64_t vdim) {
  check_rows(q, "q"); check_rows(k, "k"); check_rows(v, "v");
  TORCH_CHECK(q.size(1) == heads * dim && k.sizes() == q.sizes() && v.size(1) == heads * vdim && v.size(0) == q.size(0) &&
                  k.scalar_type() == q.scalar_type() && v.scalar_type() == q.scalar_type(), "recurrence: projections");
}
void check_head_decay(const Tensor& decay, int64_t heads) {
  TORCH_CHECK(decay.is_cuda() && decay.is_contiguous() && decay.scalar_type() == at::kFloat && decay.numel() == heads, "head decays: fp32 [heads]");
}

Tensor decayed_recurrence(const Tensor& q, const Tensor& k, const Tensor& v, const Tensor& decay, const optional<Tensor>& keep,
                          const optional<Tensor>& state, int64_t batch, int64_t heads, int64_t dim, int64_t vdim, int64_t chunks) {
  check_qkv_rows(q, k, v, heads, dim, vdim);
  check_head_decay(decay, heads);
  RecurrenceRule r;
  r.rule = 1; r.head_decay = &decay;
  return run_recurrence(r, q, k, v, keep, state, batch, heads, dim, vdim, chunks);
}

void check_channels(const Tensor& t, int64_t n, const Tensor& like, const char* what) {
  TORCH_CHECK(t.is_cuda() && t.is_contiguous() && t.numel() == n && t.scalar_type() == like.scalar_type(), what);
}

Tensor bonus_recurrence(const Tensor& q, const Tensor& k, const Tensor& v, const Tensor& z, const Tensor& w0, const Tensor& u,
                        const optional<Tensor>& keep, const optional<Tensor>& state, int64_t batch, int64_t heads, int64_t dim,
                        int64_t vdim, int64_t chunks) {
  check_qkv_rows(q, k, v, heads, dim, vdim);
  check_rows(z, "z");
  TORCH_CHECK(z.scalar_type() == at::kFloat && z.sizes() == q.sizes(), "bonus_recurrence: decay logits are fp32 [rows, heads * dim]");
  check_channels(w0, heads * dim, q, "bonus_recurrence: w0");
  check_channels(u, heads * dim, q, "bonus_recurrence: u");
  RecurrenceRule r;
  r.rule = 2; r.f_bias = &w0; r.lower = &u; r.z = &z;
  return run_recurrence(r, q, k, v, keep, state, batch, heads, dim, vdim, chunks);
}

void check_state(const Tensor& state, int64_t n);

// z fp32 [B * S, 2 heads] -> read, write, start [B, heads, S], running maximum [B * S, heads]
std::tuple<Tensor, Tensor, Tensor, Tensor> memory_gates(const Tensor& z, const Tensor& bias, double cap, const optional<Tensor>& keep,
                                                        optional<Tensor> top, int64_t batch) {
  check_rows(z, "z");
  const int64_t H = z.size(1) / 2;
  TORCH_CHECK(batch > 0 && z.size(0) % batch == 0 && z.size(1) % 2 == 0 && z.scalar_type() == at::kFloat && bias.is_contiguous() &&
                  bias.numel() == 2 * H && cap > 0.0, "memory_gates: operands");
  const int64_t S = z.size(0) / batch;
  const bool has = top.has_value() && top->defined();
  if (has) check_state(*top, batch * H);
  int64_t ld_keep = 0;
  const uint8_t* kp = keep_ptr(keep, batch, S, ld_keep);
  c10::cuda::CUDAGuard guard(z.device());
  Tensor rd = at::empty({batch, H, S}, z.options()), wr = at::empty({batch, H, S}, z.options()), st = at::empty({batch, H, S}, z.options());
  Tensor m = at::empty({batch * S, H}, z.options());
  check_rc(oslo_memory_gates(z.data_ptr<float>(), z.stride(0), bias.data_ptr(), static_cast<float>(cap), kp, ld_keep,
                             has ? top->data_ptr<float>() : nullptr, rd.data_ptr<float>(), wr.data_ptr<float>(), st.data_ptr<float>(),
                             m.data_ptr<float>(), static_cast<int>(batch), static_cast<int>(S), static_cast<int>(H), dt_code(bias),
                             cur_stream()), "memory_gates");
  return {rd, wr, st, m};
}

// S^T q [B * S, heads * vdim] and n . q [B * S, heads], fp32
std::tuple<Tensor, Tensor> memory_recurrence(const Tensor& q, const Tensor& k, const Tensor& v, const Tensor& read, const Tensor& write,
                                             const Tensor& start, double q_scale, const optional<Tensor>& keep, optional<Tensor> state,
                                             int64_t batch, int64_t heads, int64_t dim, int64_t vdim, int64_t chunks) {
  check_qkv_rows(q, k, v, heads, dim, vdim);
  TORCH_CHECK(batch > 0 && q.size(0) % batch == 0, "memory_recurrence: rows are not batch x positions");
  const int64_t S = q.size(0) / batch, lds = (vdim + 1 + 3) / 4 * 4;
  for (const Tensor* t : {&read, &write, &start})
    TORCH_CHECK(t->is_cuda() && t->is_contiguous() && t->scalar_type() == at::kFloat && t->numel() == batch * heads * S, "memory_recurrence: gates");
  const bool has = state.has_value() && state->defined();
  if (has) check_state(*state, batch * heads * dim * lds);
  int64_t ld_keep = 0;
  const uint8_t* kp = keep_ptr(keep, batch, S, ld_keep);
  c10::cuda::CUDAGuard guard(q.device());
  const int nch = chunks > 0 ? static_cast<int>(chunks)
                             : oslo_recurrence_chunks(3, static_cast<int>(batch), static_cast<int>(S), static_cast<int>(heads),
                                                      static_cast<int>(dim), static_cast<int>(vdim), dev_state(q.get_device()).sms);
  const auto f32 = q.options().dtype(at::kFloat);
  Tensor out = at::empty({q.size(0), heads * vdim}, f32), norm = at::empty({q.size(0), heads}, f32);
  Tensor ws, decay;
  if (nch > 1) {
    ws = at::empty({batch, nch, heads, dim, lds}, f32);
    decay = at::empty({batch, nch, heads, dim}, f32);
  }
  check_rc(oslo_memory_recurrence(q.data_ptr(), q.stride(0), k.data_ptr(), k.stride(0), v.data_ptr(), v.stride(0),
                                  read.data_ptr<float>(), write.data_ptr<float>(), start.data_ptr<float>(), static_cast<float>(q_scale),
                                  kp, ld_keep, has ? state->data_ptr<float>() : nullptr, out.data_ptr<float>(), norm.data_ptr<float>(),
                                  nch > 1 ? ws.data_ptr<float>() : nullptr, nch > 1 ? decay.data_ptr<float>() : nullptr, nch,
                                  static_cast<int>(batch), static_cast<int>(S), static_cast<int>(heads), static_cast<int>(dim),
                                  static_cast<int>(vdim), dt_code(q), cur_stream(nch > 1 ? 3 : 1)), "memory_recurrence");
  return {out, norm};
}

Tensor memory_step(const Tensor& q, const Tensor& k, const Tensor& v, const Tensor& x, const Tensor& w, const Tensor& bias, double cap,
                   const Tensor& gate, const Tensor& norm_w, const optional<Tensor>& keep, Tensor state, Tensor top, double q_scale,
                   double eps, int64_t heads, int64_t dim, int64_t vdim) {
  check_qkv_rows(q, k, v, heads, dim, vdim);
  check_rows(x, "x"); check_rows(gate, "gate");
  const int64_t B = q.size(0);
  check_state(state, B * heads * dim * ((vdim + 1 + 3) / 4 * 4));
  check_state(top, B * heads);
  for (const Tensor* t : {&x, &w, &bias, &gate, &norm_w}) TORCH_CHECK(t->scalar_type() == q.scalar_type(), "memory_step: dtypes");
  TORCH_CHECK(x.size(0) == B && w.is_contiguous() && w.dim() == 2 && w.size(0) == 2 * heads && w.size(1) == x.size(1) && bias.is_contiguous() &&
                  bias.numel() == 2 * heads && gate.size(0) == B && gate.size(1) == heads * vdim && norm_w.is_contiguous() &&
                  norm_w.numel() == heads * vdim && cap > 0.0, "memory_step: operands");
  int64_t ld_keep = 0;
  const uint8_t* kp = keep_ptr(keep, B, 1, ld_keep);
  c10::cuda::CUDAGuard guard(q.device());
  Tensor out = at::empty({B, heads * vdim}, q.options());
  check_rc(oslo_memory_step(q.data_ptr(), q.stride(0), k.data_ptr(), k.stride(0), v.data_ptr(), v.stride(0), x.data_ptr(), x.stride(0),
                            static_cast<int>(x.size(1)), w.data_ptr(), bias.data_ptr(), static_cast<float>(cap), gate.data_ptr(),
                            gate.stride(0), norm_w.data_ptr(), kp, ld_keep, state.data_ptr<float>(), top.data_ptr<float>(), out.data_ptr(),
                            static_cast<float>(q_scale), static_cast<float>(eps), static_cast<int>(B), static_cast<int>(heads),
                            static_cast<int>(dim), static_cast<int>(vdim), dev_state(q.get_device()).sms, dt_code(q), cur_stream()),
           "memory_step");
  return out;
}

void check_state(const Tensor& state, int64_t n) {
  TORCH_CHECK(state.is_cuda() && state.is_contiguous() && state.scalar_type() == at::kFloat && state.numel() == n, "state: contiguous fp32 of the right size");
}

Tensor decayed_step(const Tensor& q, const Tensor& k, const Tensor& v, const Tensor& decay, const optional<Tensor>& keep, Tensor state,
                    int64_t heads, int64_t dim, int64_t vdim) {
  check_qkv_rows(q, k, v, heads, dim, vdim);
  check_head_decay(decay, heads);
  const int64_t B = q.size(0);
  check_state(state, B * heads * dim * vdim);
  int64_t ld_keep = 0;
  const uint8_t* kp = keep_ptr(keep, B, 1, ld_keep);
  c10::cuda::CUDAGuard guard(q.device());
  Tensor out = at::empty({B, heads * vdim}, q.options().dtype(at::kFloat));
  check_rc(oslo_decayed_step(q.data_ptr(), q.stride(0), k.data_ptr(), k.stride(0), v.data_ptr(), v.stride(0), decay.data_ptr<float>(),
                             kp, ld_keep, state.data_ptr<float>(), out.data_ptr<float>(), static_cast<int>(B),
                             static_cast<int>(heads), static_cast<int>(dim), static_cast<int>(vdim),
                             dev_state(q.get_device()).sms, dt_code(q), cur_stream()), "decayed_step");
  return out;
}

Tensor bonus_step(const Tensor& r, const Tensor& k, const Tensor& v, const Tensor& t, const Tensor& w2, const Tensor& w0, const Tensor& u,
                  const Tensor& norm_w, const Tensor& gate, const optional<Tensor>& keep, Tensor state, double eps, int64_t heads,
                  int64_t dim, int64_t vdim) {
  check_qkv_rows(r, k, v, heads, dim, vdim);
  check_rows(t, "t"); check_rows(gate, "gate");
  const int64_t B = r.size(0);
  check_state(state, B * heads * dim * vdim);
  check_channels(w0, heads * dim, r, "bonus_step: w0");
  check_channels(u, heads * dim, r, "bonus_step: u");
  check_channels(norm_w, heads * vdim, r, "bonus_step: norm weight");
  check_channels(w2, heads * dim * t.size(1), r, "bonus_step: w2");
  TORCH_CHECK(t.size(0) == B && gate.size(0) == B && gate.size(1) == heads * vdim && t.scalar_type() == r.scalar_type() &&
                  gate.scalar_type() == r.scalar_type(), "bonus_step: operands");
  int64_t ld_keep = 0;
  const uint8_t* kp = keep_ptr(keep, B, 1, ld_keep);
  c10::cuda::CUDAGuard guard(r.device());
  Tensor out = at::empty({B, heads * vdim}, r.options());
  check_rc(oslo_bonus_step(r.data_ptr(), r.stride(0), k.data_ptr(), k.stride(0), v.data_ptr(), v.stride(0), t.data_ptr(), t.stride(0),
                           w2.data_ptr(), static_cast<int>(t.size(1)), w0.data_ptr(), u.data_ptr(), norm_w.data_ptr(),
                           gate.data_ptr(), gate.stride(0), kp, ld_keep, state.data_ptr<float>(), out.data_ptr(),
                           static_cast<float>(eps), static_cast<int>(B), static_cast<int>(heads), static_cast<int>(dim),
                           static_cast<int>(vdim), dev_state(r.get_device()).sms, dt_code(r), cur_stream()), "bonus_step");
  return out;
}

Tensor recurrence_step(const Tensor& q, const Tensor& f, const Tensor& v, const Tensor& f_bias, const Tensor& lower,
                       const Tensor& norm_w, const optional<Tensor>& keep, Tensor state, double eps, int64_t heads, int64_t dim,
                       int64_t vdim) {
  check_recurrence(q, f, v, f_bias, lower, heads, dim, vdim);
  const int64_t B = q.size(0);
  TORCH_CHECK(state.is_contiguous() && state.scalar_type() == at::kFloat && state.numel() == B * heads * dim * vdim, "recurrence_step: state");
  TORCH_CHECK(norm_w.is_contiguous() && norm_w.numel() == vdim && norm_w.scalar_type() == q.scalar_type(), "recurrence_step: norm weight");
  int64_t ld_keep = 0;
  const uint8_t* kp = keep_ptr(keep, B, 1, ld_keep);
  c10::cuda::CUDAGuard guard(q.device());
  Tensor out = at::empty({B, heads * vdim}, q.options());
  check_rc(oslo_recurrence_step(q.data_ptr(), q.stride(0), f.data_ptr(), f.stride(0), v.data_ptr(), v.stride(0),
                                f_bias.data_ptr(), lower.data_ptr(), norm_w.data_ptr(), kp, ld_keep, state.data_ptr<float>(), out.data_ptr(),
                                static_cast<float>(eps), static_cast<int>(B), static_cast<int>(heads), static_cast<int>(dim),
                                static_cast<int>(vdim), dev_state(q.get_device()).sms, dt_code(q), cur_stream()), "recurrence_step");
  return out;
}

// ---------------------------------------------------------------------- latent attention
Tensor sink_gate(const Tensor& o, const Tensor& lse, const Tensor& sink, const Tensor& gate, int64_t vdim) {
  // o is [B, H, S, D] (any strides, contiguous D), of which the first vdim columns count
  TORCH_CHECK(o.is_cuda() && o.dim() == 4 && o.stride(3) == 1 && o.size(3) >= vdim, "sink_gate: o");
  const int64_t B = o.size(0), H = o.size(1), S = o.size(2);
  check_rows(gate, "gate");
  TORCH_CHECK(lse.is_contiguous() && lse.scalar_type() == at::kFloat && lse.numel() == B * H * S && sink.numel() == H &&
                  gate.size(0) == B * S && gate.size(1) == H && gate.scalar_type() == o.scalar_type() &&
                  sink.scalar_type() == o.scalar_type(), "sink_gate: operands");
  c10::cuda::CUDAGuard guard(o.device());
  Tensor out = at::empty({B * S, H * vdim}, o.options());
  check_rc(oslo_sink_gate(o.data_ptr(), o.stride(0), o.stride(2), o.stride(1), lse.data_ptr<float>(), sink.data_ptr(),
                          gate.data_ptr(), gate.stride(0), out.data_ptr(), static_cast<int>(B), static_cast<int>(S),
                          static_cast<int>(H), static_cast<int>(vdim), dt_code(o), cur_stream()), "sink_gate");
  return out;
}

// the output gate: none, one column per head or one per output column; returns whether it is the latter
bool check_gate(const optional<Tensor>& gate, int64_t rows, int64_t heads, int64_t vdim, const Tensor& like, const char* what) {
  if (!(gate.has_value() && gate->defined())) return false;
  check_rows(*gate, what);
  TORCH_CHECK(gate->size(0) == rows && (gate->size(1) == heads || gate->size(1) == heads * vdim) && gate->scalar_type() == like.scalar_type(), what);
  return gate->size(1) != heads;
}
const void* sink_ptr(const optional<Tensor>& sink, int64_t heads, const Tensor& like, const char* what) {
  if (!(sink.has_value() && sink->defined())) return nullptr;
  TORCH_CHECK(sink->is_contiguous() && sink->numel() == heads && sink->scalar_type() == like.scalar_type(), what);
  return sink->data_ptr();
}
const int* lead_ptr(const optional<Tensor>& lead, int64_t B) {
  if (!(lead.has_value() && lead->defined())) return nullptr;
  TORCH_CHECK(lead->is_cuda() && lead->is_contiguous() && lead->scalar_type() == at::kInt && lead->numel() == B, "lead: int32 [batch]");
  return lead->data_ptr<int>();
}

// q [B, H, Sq, dim], k [B, G, Sk, dim], v [B, G, Sk, vdim] (any strides that TMA takes, contiguous last dim) -> [B * Sq, H * vdim];
// q2 [B, H, Sq, rot], k2 [B, Sk, rot]: a part of queries and keys whose keys all heads share
Tensor flash_sink_fwd(const Tensor& q, const Tensor& k, const Tensor& v, const optional<Tensor>& kpm, const optional<Tensor>& sink,
                      const optional<Tensor>& gate, double scale, double softcap, int64_t window, int64_t keep_first,
                      const optional<Tensor>& lead, const optional<Tensor>& q2, const optional<Tensor>& k2) {
  TORCH_CHECK(q.is_cuda() && q.dim() == 4 && k.dim() == 4 && v.dim() == 4 && q.stride(3) == 1 && k.stride(3) == 1 && v.stride(3) == 1 &&
                  k.size(3) == q.size(3) && k.size(0) == q.size(0) && v.size(0) == q.size(0) && v.size(1) == k.size(1) &&
                  v.size(2) == k.size(2) && q.size(1) % k.size(1) == 0 && k.size(2) >= q.size(2), "flash_sink_fwd: q, k, v");
  const int64_t B = q.size(0), H = q.size(1), G = k.size(1), Sq = q.size(2), Sk = k.size(2), dim = q.size(3), vdim = v.size(3);
  TORCH_CHECK(k.scalar_type() == q.scalar_type() && v.scalar_type() == q.scalar_type(), "flash_sink_fwd: operands");
  const void* sp = sink_ptr(sink, H, q, "flash_sink_fwd: sink");
  const bool wide = check_gate(gate, B * Sq, H, vdim, q, "flash_sink_fwd: gate");
  const bool gated = gate.has_value() && gate->defined(), parts = q2.has_value() && q2->defined();
  TORCH_CHECK(window >= 0 && keep_first >= 0 && parts == (k2.has_value() && k2->defined()), "flash_sink_fwd: window / second parts");
  if (parts)
    TORCH_CHECK(q2->dim() == 4 && k2->dim() == 3 && q2->stride(3) == 1 && k2->stride(2) == 1 && q2->size(0) == B && q2->size(1) == H &&
                    q2->size(2) == Sq && k2->size(0) == B && k2->size(1) == Sk && k2->size(2) == q2->size(3) &&
                    q2->scalar_type() == q.scalar_type() && k2->scalar_type() == q.scalar_type(), "flash_sink_fwd: second parts");
  const uint8_t* kp = nullptr;
  if (kpm.has_value() && kpm->defined()) {
    TORCH_CHECK(kpm->is_contiguous() && kpm->scalar_type() == at::kByte && kpm->numel() == B * Sk, "flash_sink_fwd: mask");
    kp = kpm->data_ptr<uint8_t>();
  }
  c10::cuda::CUDAGuard guard(q.device());
  Tensor out = at::empty({B * Sq, H * vdim}, q.options());
  check_rc(oslo_flash_sink_fwd_sm100(q.data_ptr(), k.data_ptr(), v.data_ptr(), out.data_ptr(), kp, sp,
                                     ptr_or_null(gate), gated ? gate->stride(0) : 0, static_cast<int>(B), static_cast<int>(H),
                                     static_cast<int>(G), static_cast<int>(Sq), static_cast<int>(Sk), static_cast<int>(dim),
                                     static_cast<int>(vdim), q.stride(0), q.stride(1), q.stride(2), k.stride(0), k.stride(1),
                                     k.stride(2), v.stride(0), v.stride(1), v.stride(2), Sq * H * vdim, vdim, H * vdim,
                                     static_cast<float>(scale), static_cast<float>(softcap), static_cast<int>(window),
                                     static_cast<int>(keep_first), lead_ptr(lead, B), wide ? 1 : 0, ptr_or_null(q2),
                                     parts ? q2->stride(0) : 0, parts ? q2->stride(1) : 0, parts ? q2->stride(2) : 0, ptr_or_null(k2),
                                     parts ? k2->stride(0) : 0, parts ? k2->stride(1) : 0, parts ? static_cast<int>(q2->size(3)) : 0,
                                     dt_code(q), dev_state(q.get_device()).err.data_ptr<int>(), cur_stream()), "flash_sink_fwd");
  return out;
}

// q [B, H, Sq, dim], k [B, 1, Sk, dim] (one key head of any width for all), v [B, G, Sk, vdim] -> [B * Sq, H * vdim]
Tensor flash_wide_fwd(const Tensor& q, const Tensor& k, const Tensor& v, const optional<Tensor>& kpm, const optional<Tensor>& sink,
                      const optional<Tensor>& gate, double scale, int64_t window, int64_t keep_first, const optional<Tensor>& lead) {
  TORCH_CHECK(q.is_cuda() && q.dim() == 4 && k.dim() == 4 && v.dim() == 4 && q.stride(3) == 1 && k.stride(3) == 1 && v.stride(3) == 1 &&
                  k.size(1) == 1 && k.size(3) == q.size(3) && k.size(0) == q.size(0) && v.size(0) == q.size(0) && v.size(2) == k.size(2) &&
                  q.size(1) % v.size(1) == 0 && k.size(2) >= q.size(2), "flash_wide_fwd: q, k, v");
  const int64_t B = q.size(0), H = q.size(1), G = v.size(1), Sq = q.size(2), Sk = k.size(2), dim = q.size(3), vdim = v.size(3);
  TORCH_CHECK(k.scalar_type() == q.scalar_type() && v.scalar_type() == q.scalar_type() && window >= 0 && keep_first >= 0, "flash_wide_fwd: operands");
  const void* sp = sink_ptr(sink, H, q, "flash_wide_fwd: sink");
  const bool wide = check_gate(gate, B * Sq, H, vdim, q, "flash_wide_fwd: gate");
  const bool gated = gate.has_value() && gate->defined();
  const uint8_t* kp = nullptr;
  if (kpm.has_value() && kpm->defined()) {
    TORCH_CHECK(kpm->is_contiguous() && kpm->scalar_type() == at::kByte && kpm->numel() == B * Sk, "flash_wide_fwd: mask");
    kp = kpm->data_ptr<uint8_t>();
  }
  c10::cuda::CUDAGuard guard(q.device());
  Tensor out = at::empty({B * Sq, H * vdim}, q.options());
  check_rc(oslo_flash_wide_fwd_sm100(q.data_ptr(), k.data_ptr(), v.data_ptr(), out.data_ptr(), kp, sp, ptr_or_null(gate),
                                     gated ? gate->stride(0) : 0, wide ? 1 : 0, static_cast<int>(B), static_cast<int>(H),
                                     static_cast<int>(G), static_cast<int>(Sq), static_cast<int>(Sk), static_cast<int>(dim),
                                     static_cast<int>(vdim), q.stride(0), q.stride(1), q.stride(2), k.stride(0), k.stride(2),
                                     v.stride(0), v.stride(1), v.stride(2), Sq * H * vdim, vdim, H * vdim, static_cast<float>(scale),
                                     static_cast<int>(window), static_cast<int>(keep_first), lead_ptr(lead, B), dt_code(q),
                                     dev_state(q.get_device()).err.data_ptr<int>(), cur_stream()), "flash_wide_fwd");
  return out;
}

Tensor sink_attention(const Tensor& q, const Tensor& k, const Tensor& v, const optional<Tensor>& keep, const optional<Tensor>& sink,
                      const optional<Tensor>& gate, double scale, double softcap, int64_t window, int64_t keep_first,
                      const optional<Tensor>& lead) {
  // [B, S, heads, D] views with contiguous D
  TORCH_CHECK(q.is_cuda() && q.dim() == 4 && k.dim() == 4 && v.dim() == 4 && q.stride(3) == 1 && k.stride(3) == 1 && v.stride(3) == 1,
              "sink_attention: q, k, v must be [B, S, H, D] with a contiguous last dim");
  const int64_t B = q.size(0), Sq = q.size(1), H = q.size(2), G = v.size(2), KG = k.size(2), D = q.size(3), Sk = k.size(1), Dv = v.size(3);
  TORCH_CHECK(k.size(0) == B && v.size(0) == B && G > 0 && KG > 0 && H % G == 0 && H % KG == 0 && v.size(1) == Sk && k.size(3) == D && Sk >= Sq,
              "sink_attention: sizes");
  TORCH_CHECK(k.scalar_type() == q.scalar_type() && v.scalar_type() == q.scalar_type() && window >= 0 && keep_first >= 0,
              "sink_attention: operands");
  const void* sp = sink_ptr(sink, H, q, "sink_attention: sink");
  const bool wide = check_gate(gate, B * Sq, H, Dv, q, "sink_attention: gate");
  const bool gated = gate.has_value() && gate->defined();
  int64_t ld_keep = 0;
  const uint8_t* kp = keep_ptr(keep, B, Sk, ld_keep);
  c10::cuda::CUDAGuard guard(q.device());
  Tensor out = at::empty({B * Sq, H * Dv}, q.options());
  check_rc(oslo_sink_attention(q.data_ptr(), q.stride(0), q.stride(1), q.stride(2), k.data_ptr(), k.stride(0), k.stride(1),
                               k.stride(2), v.data_ptr(), v.stride(0), v.stride(1), v.stride(2), kp, ld_keep, sp,
                               ptr_or_null(gate), gated ? gate->stride(0) : 0, out.data_ptr(), static_cast<int>(B),
                               static_cast<int>(H), static_cast<int>(G), static_cast<int>(KG), static_cast<int>(Sq), static_cast<int>(Sk),
                               static_cast<int>(D), static_cast<int>(Dv), static_cast<float>(scale), static_cast<float>(softcap),
                               static_cast<int>(window), static_cast<int>(keep_first), lead_ptr(lead, B), wide ? 1 : 0,
                               dt_code(q), cur_stream()), "sink_attention");
  return out;
}

// ---------------------------------------------------------------------- grouped-query attention
Tensor qkv_prep(const Tensor& q, const Tensor& k, const Tensor& v, const optional<Tensor>& wq, const optional<Tensor>& wk, double eps, const Tensor& positions,
                const Tensor& freq, Tensor kc, Tensor vc, const Tensor& lengths) {
  check_rows(q, "q"); check_rows(k, "k"); check_rows(v, "v");
  TORCH_CHECK(kc.dim() == 4 && vc.dim() == 4 && kc.is_contiguous() && vc.is_contiguous() && vc.size(0) == kc.size(0) &&
                  vc.size(1) == kc.size(1) && vc.size(2) == kc.size(2), "qkv_prep: caches");
  const int64_t B = kc.size(0), G = kc.size(1), T = kc.size(2), dim = kc.size(3), vdim = vc.size(3);
  TORCH_CHECK(q.size(0) % B == 0 && q.size(1) % dim == 0 && k.size(0) == q.size(0) && v.size(0) == q.size(0) && k.size(1) == G * dim &&
                  v.size(1) == G * vdim, "qkv_prep: projections");
  const int64_t S = q.size(0) / B, H = q.size(1) / dim;
  for (const Tensor* t : {&k, &v, static_cast<const Tensor*>(&kc), static_cast<const Tensor*>(&vc)})
    TORCH_CHECK(t->scalar_type() == q.scalar_type(), "qkv_prep: dtypes");
  if (ptr_or_null(wq)) check_channels(*wq, dim, q, "qkv_prep: query norm weight");
  if (ptr_or_null(wk)) check_channels(*wk, dim, q, "qkv_prep: key norm weight");
  TORCH_CHECK(positions.is_cuda() && positions.dim() == 2 && positions.size(0) == B && positions.size(1) == S && positions.scalar_type() == at::kLong, "qkv_prep: positions");
  TORCH_CHECK(freq.is_cuda() && freq.is_contiguous() && freq.scalar_type() == at::kFloat && 2 * freq.numel() <= dim, "qkv_prep: frequencies");
  TORCH_CHECK(lengths.scalar_type() == at::kInt && lengths.is_contiguous() && lengths.numel() == B, "qkv_prep: lengths");
  c10::cuda::CUDAGuard guard(q.device());
  Tensor out = at::empty({B, S, H, dim}, q.options());
  check_rc(oslo_qkv_prep(q.data_ptr(), q.stride(0), k.data_ptr(), k.stride(0), v.data_ptr(), v.stride(0), ptr_or_null(wq), ptr_or_null(wk),
                         static_cast<float>(eps), reinterpret_cast<const long long*>(positions.data_ptr<int64_t>()), positions.stride(0),
                         positions.stride(1), freq.numel() ? freq.data_ptr<float>() : nullptr, static_cast<int>(freq.numel()),
                         out.data_ptr(), kc.data_ptr(), vc.data_ptr(), lengths.data_ptr<int>(), static_cast<int>(B),
                         static_cast<int>(S), static_cast<int>(H), static_cast<int>(G), static_cast<int>(dim),
                         static_cast<int>(vdim), static_cast<int>(T), dt_code(q), dev_state(q.get_device()).err.data_ptr<int>(),
                         cur_stream()), "qkv_prep");
  return out;
}

// caches kc [B, G, T, dim], vc [B, G, T, vdim] of any strides with contiguous heads; talk [H, H]: the queries of mixed scores, [B, S, H, G * dim]
Tensor head_prep(const Tensor& q, const Tensor& k, const Tensor& v, const optional<Tensor>& wq, const optional<Tensor>& wk, double eps,
                 const Tensor& positions, const Tensor& freq, bool halves, double amplitude, const optional<Tensor>& talk, Tensor kc,
                 Tensor vc, const Tensor& lengths) {
  check_rows(q, "q"); check_rows(k, "k"); check_rows(v, "v");
  TORCH_CHECK(kc.is_cuda() && kc.dim() == 4 && vc.dim() == 4 && kc.stride(3) == 1 && vc.stride(3) == 1 && vc.size(0) == kc.size(0) &&
                  vc.size(1) == kc.size(1) && vc.size(2) == kc.size(2), "head_prep: caches");
  const int64_t B = kc.size(0), G = kc.size(1), T = kc.size(2), dim = kc.size(3), vdim = vc.size(3);
  TORCH_CHECK(q.size(0) % B == 0 && q.size(1) % dim == 0 && k.size(0) == q.size(0) && v.size(0) == q.size(0) && k.size(1) == G * dim &&
                  v.size(1) == G * vdim, "head_prep: projections");
  const int64_t S = q.size(0) / B, H = q.size(1) / dim;
  for (const Tensor* t : {&k, &v, static_cast<const Tensor*>(&kc), static_cast<const Tensor*>(&vc)})
    TORCH_CHECK(t->scalar_type() == q.scalar_type(), "head_prep: dtypes");
  if (ptr_or_null(wq)) check_channels(*wq, dim, q, "head_prep: query norm weight");
  if (ptr_or_null(wk)) check_channels(*wk, dim, q, "head_prep: key norm weight");
  const bool mixed = talk.has_value() && talk->defined();
  if (mixed) check_channels(*talk, H * H, q, "head_prep: mix of the heads");
  TORCH_CHECK(positions.is_cuda() && positions.dim() == 2 && positions.size(0) == B && positions.size(1) == S && positions.scalar_type() == at::kLong, "head_prep: positions");
  TORCH_CHECK(freq.is_cuda() && freq.is_contiguous() && freq.scalar_type() == at::kFloat && 2 * freq.numel() <= dim, "head_prep: frequencies");
  TORCH_CHECK(lengths.scalar_type() == at::kInt && lengths.is_contiguous() && lengths.numel() == B, "head_prep: lengths");
  c10::cuda::CUDAGuard guard(q.device());
  auto& st = dev_state(q.get_device());
  Tensor out = at::empty({B, S, H, mixed ? G * dim : dim}, q.options());
  check_rc(oslo_head_prep(q.data_ptr(), q.stride(0), k.data_ptr(), k.stride(0), v.data_ptr(), v.stride(0), ptr_or_null(wq), ptr_or_null(wk),
                          static_cast<float>(eps), reinterpret_cast<const long long*>(positions.data_ptr<int64_t>()), positions.stride(0),
                          positions.stride(1), freq.numel() ? freq.data_ptr<float>() : nullptr, static_cast<int>(freq.numel()),
                          halves ? 1 : 0, static_cast<float>(amplitude), ptr_or_null(talk), out.data_ptr(), kc.data_ptr(), kc.stride(0),
                          kc.stride(1), kc.stride(2), vc.data_ptr(), vc.stride(0), vc.stride(1), vc.stride(2), lengths.data_ptr<int>(),
                          static_cast<int>(B), static_cast<int>(S), static_cast<int>(H), static_cast<int>(G), static_cast<int>(dim),
                          static_cast<int>(vdim), static_cast<int>(T), st.sms, dt_code(q), st.err.data_ptr<int>(), cur_stream()), "head_prep");
  return out;
}

// whether grouped_decode has a kernel for wide keys of these sizes
bool wide_decode_fits(const Tensor& like, int64_t heads, int64_t value_heads, int64_t dim, int64_t vdim) {
  return oslo_wide_decode_fits(static_cast<int>(heads), static_cast<int>(value_heads), static_cast<int>(dim), static_cast<int>(vdim), dt_code(like)) != 0;
}

// value_heads > 1: kc [B, 1, T, dim] (wide keys), vc [B, 1, T, value_heads * vdim]; query heads read value heads in equal groups
Tensor grouped_decode(const Tensor& q, const Tensor& kc, const Tensor& vc, const Tensor& lengths, const optional<Tensor>& keep,
                      const optional<Tensor>& sink, double scale, double softcap, const optional<Tensor>& gate, int64_t window,
                      int64_t keep_first, const optional<Tensor>& lead, int64_t value_heads) {
  TORCH_CHECK(q.is_cuda() && q.dim() == 3 && q.is_contiguous() && kc.dim() == 4 && vc.dim() == 4 && kc.is_contiguous() && vc.is_contiguous() &&
                  vc.size(0) == kc.size(0) && vc.size(1) == kc.size(1) && vc.size(2) == kc.size(2) && kc.size(0) == q.size(0) &&
                  kc.size(3) == q.size(2) && q.size(1) % kc.size(1) == 0, "grouped_decode: q [B, H, dim], caches [B, G, T, *]");
  const int64_t B = q.size(0), H = q.size(1), G = kc.size(1), T = kc.size(2), row = vc.size(3);
  TORCH_CHECK(value_heads >= 1 && (value_heads == 1 || (G == 1 && H % value_heads == 0 && row % value_heads == 0)), "grouped_decode: value heads");
  const int64_t vdim = row / value_heads;
  TORCH_CHECK(kc.scalar_type() == q.scalar_type() && vc.scalar_type() == q.scalar_type() && window >= 0 && keep_first >= 0, "grouped_decode: operands");
  const void* sp = sink_ptr(sink, H, q, "grouped_decode: sink");
  const bool wide = check_gate(gate, B, H, vdim, q, "grouped_decode: gate");
  const bool gated = gate.has_value() && gate->defined();
  TORCH_CHECK(lengths.scalar_type() == at::kInt && lengths.is_contiguous() && lengths.numel() == B, "grouped_decode: lengths");
  int64_t ld_keep = 0;
  const uint8_t* kp = keep_ptr(keep, B, 0, ld_keep);
  c10::cuda::CUDAGuard guard(q.device());
  auto& st = dev_state(q.get_device());
  const int64_t most = window > 0 ? std::min(T, window + keep_first) : T;     // keys a query can see
  const int splits = oslo_grouped_splits(static_cast<int>(B), static_cast<int>(H), static_cast<int>(G), static_cast<int>(value_heads),
                                         static_cast<int>(most), static_cast<int>(q.size(2)), static_cast<int>(row), dt_code(q), st.sms);
  const auto f32 = q.options().dtype(at::kFloat);
  Tensor ws = at::empty({B, H, splits, (vdim + 3) / 4 * 4}, f32);
  Tensor stat = at::empty({B, H, splits, 2}, f32);
  Tensor out = at::empty({B, H * vdim}, q.options());
  check_rc(oslo_grouped_decode(q.data_ptr(), kc.data_ptr(), vc.data_ptr(), lengths.data_ptr<int>(), kp, ld_keep,
                               kp ? static_cast<int>(keep->size(1)) : 0, sp, ptr_or_null(gate), gated ? gate->stride(0) : 0, wide ? 1 : 0,
                               static_cast<int>(window), static_cast<int>(keep_first), lead_ptr(lead, B), ws.data_ptr<float>(),
                               stat.data_ptr<float>(), out.data_ptr(), static_cast<int>(B), static_cast<int>(H), static_cast<int>(G),
                               static_cast<int>(value_heads), static_cast<int>(q.size(2)), static_cast<int>(row), static_cast<int>(T), splits,
                               static_cast<float>(scale), static_cast<float>(softcap), dt_code(q), st.err.data_ptr<int>(),
                               cur_stream(2)), "grouped_decode");
  return out;
}

// ---------------------------------------------------------------------- token shift, convolution, selective scan
float* carried_ptr(const optional<Tensor>& t, int64_t n) {
  if (!(t.has_value() && t->defined())) return nullptr;
  check_state(*t, n);
  return t->data_ptr<float>();
}

Tensor token_shift(const Tensor& h, const Tensor& mu, int64_t batch, const optional<Tensor>& keep, optional<Tensor> prev) {
  check_rows(h, "h");
  TORCH_CHECK(batch > 0 && h.size(0) % batch == 0 && mu.dim() == 2 && mu.is_contiguous() && mu.size(1) == h.size(1) &&
                  mu.scalar_type() == h.scalar_type(), "token_shift: operands");
  const int64_t S = h.size(0) / batch, width = h.size(1), P = mu.size(0);
  int64_t ld_keep = 0;
  const uint8_t* kp = keep_ptr(keep, batch, S, ld_keep);
  c10::cuda::CUDAGuard guard(h.device());
  Tensor out = at::empty({P, h.size(0), width}, h.options());
  check_rc(oslo_token_shift(h.data_ptr(), h.stride(0), mu.data_ptr(), kp, ld_keep, carried_ptr(prev, batch * width), out.data_ptr(),
                            static_cast<int>(batch), static_cast<int>(S), static_cast<int>(width), static_cast<int>(P), dt_code(h),
                            cur_stream()), "token_shift");
  return out;
}

Tensor causal_conv(const Tensor& x, const Tensor& w, const optional<Tensor>& bias, int64_t batch, const optional<Tensor>& keep,
                   optional<Tensor> prev, bool silu, bool residual) {
  check_rows(x, "x");
  const int64_t C = x.size(1);
  TORCH_CHECK(batch > 0 && x.size(0) % batch == 0 && w.dim() == 2 && w.is_contiguous() && w.size(0) == C && w.scalar_type() == x.scalar_type() &&
                  !(silu && residual), "causal_conv: operands");
  if (ptr_or_null(bias)) check_channels(*bias, C, x, "causal_conv: bias");
  const int64_t S = x.size(0) / batch, taps = w.size(1);
  int64_t ld_keep = 0;
  const uint8_t* kp = keep_ptr(keep, batch, S, ld_keep);
  c10::cuda::CUDAGuard guard(x.device());
  Tensor out = at::empty({x.size(0), C}, x.options());
  check_rc(oslo_causal_conv(x.data_ptr(), x.stride(0), w.data_ptr(), ptr_or_null(bias), kp, ld_keep,
                            taps > 1 ? carried_ptr(prev, batch * (taps - 1) * C) : nullptr, out.data_ptr(), static_cast<int>(batch),
                            static_cast<int>(S), static_cast<int>(C), static_cast<int>(taps), silu ? 1 : 0, residual ? 1 : 0,
                            dt_code(x), cur_stream()), "causal_conv");
  return out;
}

void check_scan(const Tensor& x, const Tensor& dt_bias, const Tensor& a_log, const Tensor& b, const Tensor& c, const Tensor& d, const Tensor& z) {
  check_rows(x, "x"); check_rows(b, "b"); check_rows(c, "c"); check_rows(z, "z");
  const int64_t C = x.size(1);
  TORCH_CHECK(a_log.dim() == 2 && a_log.size(0) == C, "selective_scan: a_log is [channels, states]");
  const int64_t N = a_log.size(1);
  check_channels(a_log, C * N, x, "selective_scan: a_log");
  check_channels(dt_bias, C, x, "selective_scan: dt bias");
  check_channels(d, C, x, "selective_scan: d");
  TORCH_CHECK(z.sizes() == x.sizes() && b.size(0) == x.size(0) && c.size(0) == x.size(0) && b.size(1) == N && c.size(1) == N &&
                  z.scalar_type() == x.scalar_type() && b.scalar_type() == x.scalar_type() && c.scalar_type() == x.scalar_type(),
              "selective_scan: operands");
}

Tensor selective_scan(const Tensor& x, const Tensor& dt, const Tensor& dt_bias, const Tensor& a_log, const Tensor& b, const Tensor& c,
                      const Tensor& d, const Tensor& z, int64_t batch, const optional<Tensor>& keep, optional<Tensor> state,
                      int64_t chunks) {
  check_scan(x, dt_bias, a_log, b, c, d, z);
  check_rows(dt, "dt");
  TORCH_CHECK(batch > 0 && x.size(0) % batch == 0 && dt.sizes() == x.sizes() && dt.scalar_type() == at::kFloat, "selective_scan: dt is fp32 [rows, channels]");
  const int64_t S = x.size(0) / batch, C = x.size(1), N = a_log.size(1);
  int64_t ld_keep = 0;
  const uint8_t* kp = keep_ptr(keep, batch, S, ld_keep);
  c10::cuda::CUDAGuard guard(x.device());
  const int nch = chunks > 0 ? static_cast<int>(chunks)
                             : oslo_scan_chunks(static_cast<int>(batch), static_cast<int>(S), static_cast<int>(C),
                                                static_cast<int>(N), dev_state(x.get_device()).sms);
  const auto f32 = x.options().dtype(at::kFloat);
  Tensor out = at::empty({x.size(0), C}, x.options());
  Tensor ws, steps;
  if (nch > 1) {
    ws = at::empty({batch, nch, C, N}, f32);
    steps = at::empty({batch, nch, C}, f32);
  }
  check_rc(oslo_selective_scan(x.data_ptr(), x.stride(0), dt.data_ptr<float>(), dt.stride(0), dt_bias.data_ptr(), a_log.data_ptr(),
                               b.data_ptr(), b.stride(0), c.data_ptr(), c.stride(0), d.data_ptr(), z.data_ptr(), z.stride(0), kp,
                               ld_keep, carried_ptr(state, batch * C * N), out.data_ptr(), nch > 1 ? ws.data_ptr<float>() : nullptr,
                               nch > 1 ? steps.data_ptr<float>() : nullptr, nch, static_cast<int>(batch), static_cast<int>(S),
                               static_cast<int>(C), static_cast<int>(N), dev_state(x.get_device()).sms, dt_code(x),
                               cur_stream(nch > 1 ? 3 : 1)), "selective_scan");
  return out;
}

Tensor scan_step(const Tensor& x, const Tensor& dt, const Tensor& w_dt, const Tensor& dt_bias, const Tensor& a_log, const Tensor& b,
                 const Tensor& c, const Tensor& d, const Tensor& z, const optional<Tensor>& keep, Tensor state) {
  check_scan(x, dt_bias, a_log, b, c, d, z);
  check_rows(dt, "dt");
  const int64_t B = x.size(0), C = x.size(1), N = a_log.size(1);
  TORCH_CHECK(dt.size(0) == B && dt.scalar_type() == x.scalar_type(), "scan_step: dt");
  check_channels(w_dt, C * dt.size(1), x, "scan_step: step projection");
  check_state(state, B * C * N);
  int64_t ld_keep = 0;
  const uint8_t* kp = keep_ptr(keep, B, 1, ld_keep);
  c10::cuda::CUDAGuard guard(x.device());
  Tensor out = at::empty({B, C}, x.options());
  check_rc(oslo_scan_step(x.data_ptr(), x.stride(0), dt.data_ptr(), dt.stride(0), w_dt.data_ptr(), static_cast<int>(dt.size(1)),
                          dt_bias.data_ptr(), a_log.data_ptr(), b.data_ptr(), b.stride(0), c.data_ptr(), c.stride(0), d.data_ptr(),
                          z.data_ptr(), z.stride(0), kp, ld_keep, state.data_ptr<float>(), out.data_ptr(), static_cast<int>(B),
                          static_cast<int>(C), static_cast<int>(N), dt_code(x), cur_stream()), "scan_step");
  return out;
}

// positions int64 [B, S] and frequencies fp32 [rot / 2] of a rotation (rot 0: none are needed)
struct Turn {
  const long long* pos = nullptr;
  int64_t sb = 0, ss = 0;
  const float* freq = nullptr;
  Turn(const optional<Tensor>& positions, const optional<Tensor>& freqs, int64_t B, int64_t S, int64_t rot) {
    if (rot == 0) return;
    TORCH_CHECK(positions.has_value() && positions->defined() && freqs.has_value() && freqs->defined() && positions->is_cuda() &&
                    positions->dim() == 2 && positions->size(0) == B && positions->size(1) == S && positions->scalar_type() == at::kLong &&
                    freqs->is_cuda() && freqs->is_contiguous() && freqs->scalar_type() == at::kFloat && 2 * freqs->numel() == rot,
                "rotation: positions int64 [batch, S], frequencies fp32 [dims / 2]");
    pos = reinterpret_cast<const long long*>(positions->data_ptr<int64_t>());
    sb = positions->stride(0);
    ss = positions->stride(1);
    freq = freqs->data_ptr<float>();
  }
};

// rows b * S + t; the columns of ckv after wkv's are rotated and cached behind the latent. Returns the normed query latents and
// (rows) the normed key-value latents
std::tuple<Tensor, Tensor> latent_prep(const Tensor& cq, const Tensor& wq, const optional<Tensor>& ckv, const optional<Tensor>& wkv,
                                       optional<Tensor> cache, const Tensor& lengths, double eps, const optional<Tensor>& positions,
                                       const optional<Tensor>& freq, bool rows) {
  check_rows(cq, "cq");
  TORCH_CHECK(wq.is_contiguous() && wq.numel() == cq.size(1) && wq.scalar_type() == cq.scalar_type(), "latent_prep: query norm weight");
  const int64_t n = cq.size(0), B = lengths.numel();
  TORCH_CHECK(lengths.scalar_type() == at::kInt && lengths.is_contiguous() && B > 0 && n % B == 0, "latent_prep: lengths");
  const int64_t S = n / B;
  const bool kv = ckv.has_value() && ckv->defined();
  int64_t R = 0, W = 0, T = 0;
  if (kv) {
    check_rows(*ckv, "ckv");
    TORCH_CHECK(wkv.has_value() && wkv->defined() && wkv->is_contiguous() && cache.has_value() && cache->dim() == 3 && cache->is_contiguous(),
                "latent_prep: key-value operands");
    R = wkv->numel();
    W = ckv->size(1);
    TORCH_CHECK(W >= R && cache->size(0) == B && cache->size(2) == W && ckv->size(0) == n && cache->scalar_type() == cq.scalar_type() &&
                    ckv->scalar_type() == cq.scalar_type() && wkv->scalar_type() == cq.scalar_type(), "latent_prep: key-value sizes");
    T = cache->size(1);
  }
  const Turn turn(positions, freq, B, S, W - R);
  c10::cuda::CUDAGuard guard(cq.device());
  Tensor out = at::empty({n, cq.size(1)}, cq.options());
  Tensor c = at::empty({kv && rows ? n : 0, R}, cq.options());
  check_rc(oslo_latent_prep(cq.data_ptr(), cq.stride(0), wq.data_ptr(), static_cast<int>(cq.size(1)), out.data_ptr(),
                            ptr_or_null(ckv), kv ? ckv->stride(0) : 0, ptr_or_null(wkv), static_cast<int>(R),
                            kv ? cache->data_ptr() : nullptr, lengths.data_ptr<int>(), static_cast<int>(T),
                            static_cast<float>(eps), static_cast<int>(B), static_cast<int>(S), static_cast<int>(W - R), turn.pos, turn.sb,
                            turn.ss, turn.freq, kv && rows ? c.data_ptr() : nullptr, dt_code(cq),
                            dev_state(cq.get_device()).err.data_ptr<int>(), cur_stream()), "latent_prep");
  return {out, c};
}

// q [B, S, heads, dim + rot] contiguous: the last rot dims of every head are rotated in place (halves paired)
Tensor rotate_halves_(Tensor q, const Tensor& positions, const Tensor& freq) {
  TORCH_CHECK(q.is_cuda() && q.dim() == 4 && q.is_contiguous() && 2 * freq.numel() <= q.size(3), "rotate_halves_: q [B, S, heads, dim]");
  const int64_t rot = 2 * freq.numel();
  const Turn turn(positions, freq, q.size(0), q.size(1), rot);
  c10::cuda::CUDAGuard guard(q.device());
  check_rc(oslo_rotate_halves(q.data_ptr(), turn.pos, turn.sb, turn.ss, turn.freq, static_cast<int>(q.size(0)), static_cast<int>(q.size(1)),
                              static_cast<int>(q.size(2)), static_cast<int>(q.size(3) - rot), static_cast<int>(rot), dt_code(q),
                              cur_stream()), "rotate_halves_");
  return q;
}

Tensor latent_decode(const Tensor& q, const Tensor& w_uk, const Tensor& w_uv, const Tensor& cache, const Tensor& lengths,
                     const optional<Tensor>& keep, const optional<Tensor>& sink, const Tensor& gate, double scale, int64_t heads,
                     const optional<Tensor>& positions, const optional<Tensor>& freq) {
  check_rows(q, "q"); check_rows(w_uk, "w_uk"); check_rows(w_uv, "w_uv");
  TORCH_CHECK(cache.dim() == 3 && cache.is_contiguous(), "latent_decode: cache must be contiguous [B, T, rank + rotated]");
  const int64_t B = q.size(0), R = w_uk.size(1), rot = cache.size(2) - R, T = cache.size(1);
  TORCH_CHECK(rot >= 0 && q.size(1) % heads == 0 && w_uk.size(0) == q.size(1) - heads * rot && w_uv.size(0) % heads == 0 &&
                  w_uv.size(1) == R && cache.size(0) == B, "latent_decode: sizes");
  TORCH_CHECK(w_uk.scalar_type() == q.scalar_type() && w_uv.scalar_type() == q.scalar_type() && cache.scalar_type() == q.scalar_type(),
              "latent_decode: dtypes");
  TORCH_CHECK(lengths.scalar_type() == at::kInt && lengths.is_contiguous() && lengths.numel() == B, "latent_decode: lengths");
  int64_t ld_keep = 0;
  const uint8_t* kp = keep_ptr(keep, B, 0, ld_keep);
  const int64_t dim = q.size(1) / heads - rot, vdim = w_uv.size(0) / heads;
  const void* sp = sink_ptr(sink, heads, q, "latent_decode: sink");
  const bool wide = check_gate(gate, B, heads, vdim, q, "latent_decode: gate");
  const Turn turn(positions, freq, B, 1, rot);
  c10::cuda::CUDAGuard guard(q.device());
  auto& st = dev_state(q.get_device());
  const int splits = oslo_latent_splits(static_cast<int>(B), static_cast<int>(heads), static_cast<int>(T), st.sms);
  const auto f32 = q.options().dtype(at::kFloat);
  Tensor qa = at::empty({B, heads, R + rot}, f32);
  Tensor ws = at::empty({B, heads, splits, (R + 3) / 4 * 4}, f32);
  Tensor stat = at::empty({B, heads, splits, 2}, f32);
  Tensor out = at::empty({B, heads * vdim}, q.options());
  check_rc(oslo_latent_decode(q.data_ptr(), q.stride(0), w_uk.data_ptr(), w_uk.stride(0), w_uv.data_ptr(), w_uv.stride(0),
                              cache.data_ptr(), lengths.data_ptr<int>(), kp, ld_keep, kp ? static_cast<int>(keep->size(1)) : 0,
                              sp, gate.data_ptr(), gate.stride(0), qa.data_ptr<float>(), ws.data_ptr<float>(),
                              stat.data_ptr<float>(), out.data_ptr(), static_cast<int>(B), static_cast<int>(heads), static_cast<int>(dim),
                              static_cast<int>(vdim), static_cast<int>(R), static_cast<int>(rot), turn.pos, turn.sb, turn.freq,
                              wide ? 1 : 0, static_cast<int>(T), splits, static_cast<float>(scale), st.sms, dt_code(q),
                              st.err.data_ptr<int>(), cur_stream(3)), "latent_decode");
  return out;
}

// ---------------------------------------------------------------------- mixture of experts
std::tuple<Tensor, Tensor> moe_route(const Tensor& h, const Tensor& w, const optional<Tensor>& bias, const optional<Tensor>& logits,
                                     int64_t top, int64_t scored) {
  check_rows(h, "h");
  TORCH_CHECK(w.dim() == 2 && w.is_contiguous() && w.size(1) == h.size(1) && w.scalar_type() == h.scalar_type() && scored >= 0 && scored <= 2,
              "moe_route: router");
  if (ptr_or_null(bias)) check_channels(*bias, w.size(0), h, "moe_route: bias");
  const int64_t n = h.size(0), E = w.size(0);
  const float* lg = nullptr;
  int64_t ldl = 0;
  if (logits.has_value() && logits->defined()) {
    check_rows(*logits, "logits");
    TORCH_CHECK(logits->scalar_type() == at::kFloat && logits->size(0) == n && logits->size(1) == E, "moe_route: logits");
    lg = logits->data_ptr<float>();
    ldl = logits->stride(0);
  }
  c10::cuda::CUDAGuard guard(h.device());
  Tensor idx = at::empty({n, top}, h.options().dtype(at::kInt));
  Tensor wgt = at::empty({n, top}, h.options().dtype(at::kFloat));
  check_rc(oslo_moe_route(h.data_ptr(), h.stride(0), w.data_ptr(), ptr_or_null(bias), lg, ldl, idx.data_ptr<int>(), wgt.data_ptr<float>(),
                          n, static_cast<int>(E), static_cast<int>(h.size(1)), static_cast<int>(top), static_cast<int>(scored), dt_code(h),
                          cur_stream()), "moe_route");
  return {idx, wgt};
}

// (slots [n, top], rows sorted by expert, expert of every 128-row tile, tiles in use)
// scale [pairs] (fp32, or none) multiplies the rows
const float* pair_scale(const optional<Tensor>& scale, int64_t pairs) {
  if (!(scale.has_value() && scale->defined())) return nullptr;
  TORCH_CHECK(scale->is_cuda() && scale->is_contiguous() && scale->scalar_type() == at::kFloat && scale->numel() == pairs, "weights of (token, choice) pairs");
  return scale->data_ptr<float>();
}
std::tuple<Tensor, Tensor, Tensor, Tensor> moe_plan(const Tensor& h, const Tensor& idx, int64_t experts, const optional<Tensor>& scale) {
  check_rows(h, "h");
  TORCH_CHECK(idx.is_contiguous() && idx.scalar_type() == at::kInt && idx.dim() == 2 && idx.size(0) == h.size(0), "moe_plan: idx");
  const int64_t pairs = idx.numel(), K = h.size(1);
  const int64_t tiles = (pairs + 127) / 128 + std::min<int64_t>(experts, pairs);   // every expert rounds up by at most one tile
  c10::cuda::CUDAGuard guard(h.device());
  const auto i32 = h.options().dtype(at::kInt);
  Tensor cursor = at::empty({experts}, i32), tg = at::empty({tiles}, i32), nt = at::empty({1}, i32);
  Tensor slots = at::empty({idx.size(0), idx.size(1)}, i32);
  Tensor rows = at::empty({tiles * 128, K}, h.options());
  check_rc(oslo_moe_plan(h.data_ptr(), h.stride(0), idx.data_ptr<int>(), cursor.data_ptr<int>(), tg.data_ptr<int>(),
                         nt.data_ptr<int>(), slots.data_ptr<int>(), rows.data_ptr(), pair_scale(scale, pairs), pairs, static_cast<int>(experts),
                         static_cast<int>(K), static_cast<int>(idx.size(1)), static_cast<int>(tiles), dt_code(h), cur_stream(2)),
           "moe_plan");
  return {slots, rows, tg, nt};
}

// unit(rows . w[expert of the tile]^T): [slots, N], or [slots, N / 2] for units 2 and 3 (silu(gate) * up of column pairs, its clamped
// form); tcgen05 for 16-bit types with K % 8 == 0 and 16-byte result rows
Tensor moe_grouped(const Tensor& rows, const Tensor& w, const Tensor& tile_group, const Tensor& n_tiles, int64_t unit, double limit,
                   double alpha) {
  TORCH_CHECK(rows.is_cuda() && rows.dim() == 2 && rows.is_contiguous() && w.dim() == 3 && w.is_contiguous() &&
                  w.size(2) == rows.size(1) && w.scalar_type() == rows.scalar_type(), "moe_grouped: operands");
  TORCH_CHECK(tile_group.scalar_type() == at::kInt && tile_group.numel() * 128 == rows.size(0) && n_tiles.scalar_type() == at::kInt,
              "moe_grouped: plan");
  const int64_t N = w.size(1), K = w.size(2), cols = unit >= 2 ? N / 2 : N;
  TORCH_CHECK(unit >= 0 && unit <= 3 && (unit < 2 || N % 2 == 0), "moe_grouped: unit");
  c10::cuda::CUDAGuard guard(rows.device());
  auto& st = dev_state(rows.get_device());
  Tensor out = at::empty({rows.size(0), cols}, rows.options());
  if (rows.scalar_type() != at::kFloat && K % 8 == 0 && cols % 8 == 0 && reinterpret_cast<uintptr_t>(w.data_ptr()) % 16 == 0) {
    const int fl = (unit == 1 ? GEMM_FLAG_RELU2 : 0) | (unit >= 2 ? GEMM_FLAG_GLU : 0) | (rows.scalar_type() == at::kHalf ? GEMM_FLAG_FP16 : 0);
    check_rc(oslo_gemm_grouped(rows.data_ptr(), w.data_ptr(), out.data_ptr(), static_cast<int>(rows.size(0)), static_cast<int>(N),
                               static_cast<int>(K), static_cast<int>(w.size(0)), tile_group.data_ptr<int>(),
                               n_tiles.data_ptr<int>(), fl, unit == 3 ? 1 : 0, static_cast<float>(limit), static_cast<float>(alpha),
                               st.err.data_ptr<int>(), usable_sms(st), cur_stream()), "gemm_grouped");
  } else {
    check_rc(oslo_moe_grouped(rows.data_ptr(), w.data_ptr(), out.data_ptr(), tile_group.data_ptr<int>(), n_tiles.data_ptr<int>(),
                              static_cast<int>(tile_group.numel()), static_cast<int>(N), static_cast<int>(K), static_cast<int>(unit),
                              static_cast<float>(limit), static_cast<float>(alpha), dt_code(rows), cur_stream()), "moe_grouped");
  }
  return out;
}

// one row of the result per (row, choice): unit(w[idx] . x[row]); x has one row per `per_row` entries of idx; rows of entries that are
// no expert (>= w.size(0)) are not written; scale [pairs] (or none) multiplies the rows of x
Tensor moe_few(const Tensor& x, const Tensor& idx, const Tensor& w, int64_t per_row, int64_t unit, double limit, double alpha,
               const optional<Tensor>& scale) {
  check_rows(x, "x");
  TORCH_CHECK(w.dim() == 3 && w.is_contiguous() && w.size(2) == x.size(1) && w.scalar_type() == x.scalar_type(), "moe_few: weights");
  TORCH_CHECK(idx.is_contiguous() && idx.scalar_type() == at::kInt && idx.numel() == x.size(0) * per_row, "moe_few: idx");
  TORCH_CHECK(unit >= 0 && unit <= 3 && (unit < 2 || w.size(1) % 2 == 0), "moe_few: unit");
  c10::cuda::CUDAGuard guard(x.device());
  Tensor out = at::empty({idx.numel(), unit >= 2 ? w.size(1) / 2 : w.size(1)}, x.options());
  check_rc(oslo_moe_few(x.data_ptr(), x.stride(0), idx.data_ptr<int>(), w.data_ptr(), out.data_ptr(), static_cast<int>(idx.numel()),
                        static_cast<int>(per_row), static_cast<int>(w.size(1)), static_cast<int>(w.size(2)), static_cast<int>(unit),
                        static_cast<float>(limit), static_cast<float>(alpha), pair_scale(scale, idx.numel()), static_cast<int>(w.size(0)),
                        dt_code(x), cur_stream()), "moe_few");
  return out;
}

}  // namespace

// Schemas. Kernels that take tensors are registered for the CUDA dispatch key (below), which leaves the Meta /
// fake-tensor slot free for the shape implementations that oslo_b200/ops/fake_impls.py registers from Python.
TORCH_LIBRARY(oslo_b200, m) {
  m.def("error_word(Tensor like) -> Tensor");
  m.def("launch_count() -> int", &launch_count);
  m.def("set_reserved_sms(int n) -> int", &set_reserved_sms);
  m.def("reserved_sms() -> int", &reserved_sms);
  m.def("gemm(Tensor a, Tensor b, int a_mn, int b_mn, Tensor? bias, Tensor? aux, Tensor(a!)? out, Tensor(b!)? aux_out, int flags, float alpha) -> Tensor");
  m.def("gemm_ce_stats(Tensor a, Tensor b, int b_mn, Tensor? bias, Tensor labels, int vocab_start) -> (Tensor, Tensor, Tensor)");
  m.def("gemm_ce_grad(Tensor a, Tensor b, int b_mn, Tensor? bias, Tensor labels, int vocab_start, Tensor lse, Tensor scale) -> Tensor");
  m.def("gemm_small_m(Tensor a, Tensor b, int b_mn, Tensor? bias, int gelu_from) -> Tensor");
  m.def("layernorm_fwd(Tensor x, Tensor w, Tensor? b, float eps) -> (Tensor, Tensor, Tensor)");
  m.def("layernorm_bwd(Tensor dy, Tensor x, Tensor w, Tensor mean, Tensor rstd) -> (Tensor, Tensor, Tensor)");
  m.def("bias_gelu_fwd(Tensor x, Tensor? bias) -> Tensor");
  m.def("bias_gelu_bwd(Tensor dy, Tensor x, Tensor? bias) -> Tensor");
  m.def("bias_dropout_residual(Tensor x, Tensor? bias, Tensor? residual, float p, int seed, int mode) -> Tensor");
  m.def("colsum(Tensor x) -> Tensor");
  m.def("rotary(Tensor x, Tensor positions, int rotary_dim, float base, bool inverse) -> Tensor");
  m.def("rotary_(Tensor(a!) x, Tensor positions, int heads, int head_dim, int rotary_dim, float base, bool inverse) -> Tensor(a!)");
  m.def("causal_softmax_fwd(Tensor x, float scale) -> Tensor");
  m.def("masked_softmax_fwd(Tensor x, Tensor mask, float scale) -> Tensor");
  m.def("softmax_bwd(Tensor y, Tensor dy, float scale) -> Tensor");
  m.def("ce_stats(Tensor logits, Tensor labels, int vocab_start) -> (Tensor, Tensor, Tensor)");
  m.def("ce_grad_(Tensor(a!) logits, Tensor labels, int vocab_start, Tensor lse, Tensor scale) -> Tensor(a!)");
  m.def("adam_step(Tensor(a!) p, Tensor g, Tensor(b!) m, Tensor(c!) v, Tensor(d!)? p_lp, float lr, float beta1, float beta2, float eps, float wd, int step, float grad_scale, Tensor? inv_scale) -> ()");
  m.def("sumsq(Tensor x) -> Tensor");
  m.def("ngram_ban_(Tensor tokens, Tensor(a!) lprobs, int n) -> Tensor(a!)");
  m.def("flash_fwd(Tensor q, Tensor k, Tensor v, float scale, bool causal, int window, Tensor? kpm, int impl=1) -> (Tensor, Tensor)");
  m.def("flash_bwd(Tensor dout, Tensor q, Tensor k, Tensor v, Tensor o, Tensor lse, float scale, bool causal, int window, Tensor? kpm, int impl=1) -> (Tensor, Tensor, Tensor)");
  m.def("decode_attn(Tensor q, Tensor kc, Tensor vc, Tensor lengths, float scale, int window) -> Tensor");
  m.def("gemm_comm(Tensor a, Tensor b, int a_mn, int b_mn, Tensor? bias, Tensor? aux, Tensor(a!)? aux_out, Tensor(b!)? out, int flags, float alpha, int M, int N, int K, int peer_bufs_dev, int own_buf, int mc_base, int data_off, int flag_off, int flag_bytes, int rank, int world, int epoch, int done_base, int mode, bool use_multimem, Tensor(c!)? trace) -> int");
  m.def("gemv_rows(Tensor x1, Tensor? x2, Tensor w, Tensor? bias, int gelu_from, Tensor? res=None) -> Tensor");
  m.def("rotary_append(Tensor q, Tensor k, Tensor v, Tensor(a!) kc, Tensor(b!) vc, Tensor lengths, Tensor write_index, int rotary_dim, float base) -> Tensor");
  m.def("vocab_embed(Tensor ids, Tensor weight, int lo, int hi, int peer_ptrs_dev, int mc_ptr, int signal_ptrs_dev, Tensor(a!) counters, int half_bytes, int rank, int world, bool use_multimem) -> Tensor");
  m.def("wait_probe(Tensor flag, int target, float limit_ms) -> Tensor");
  m.def("allreduce_oneshot(Tensor(a!) x, int peer_ptrs_dev, int mc_ptr, int signal_ptrs_dev, Tensor(b!) counters, int stage_off, int half_bytes, int rank, int world, bool use_multimem) -> ()");
  m.def("ce_combine(Tensor(a!) mx, Tensor(b!) se, Tensor(c!) tg, int peer_ptrs_dev, int signal_ptrs_dev, Tensor(d!) counters, int cap, int rank, int world) -> ()");
  m.def("dp_reduce_scatter(Tensor like, int peer_ptrs_dev, int mc_ptr, int signal_ptrs_dev, int lo, int hi, int shard, int rank, int world, bool use_multimem) -> ()");
  m.def("dp_all_gather(Tensor like, int peer_ptrs_dev, int mc_ptr, int signal_ptrs_dev, int lo, int hi, int shard, int rank, int world, bool use_multimem) -> ()");
  m.def("allreduce_symm(int peer_ptrs_dev, int mc_ptr, int signal_ptrs_dev, Tensor(a!) out, int numel, int rank, int world, bool use_multimem) -> ()");
  m.def("rms_norm(Tensor x, Tensor w, float eps, float offset) -> Tensor");
  m.def("residual_join(Tensor x, Tensor y, Tensor? slots, Tensor? slot_weights, Tensor gate, Tensor gate_bias, Tensor w_post, Tensor? w_next, float eps) -> (Tensor, Tensor)");
  m.def("silu_mul(Tensor gate, Tensor up) -> Tensor");
  m.def("recurrence(Tensor q, Tensor f, Tensor v, Tensor f_bias, Tensor lower, Tensor? keep, Tensor(a!)? state, int batch, int heads, int dim, int vdim, int chunks=0) -> Tensor");
  m.def("recurrence_step(Tensor q, Tensor f, Tensor v, Tensor f_bias, Tensor lower, Tensor norm_w, Tensor? keep, Tensor(a!) state, float eps, int heads, int dim, int vdim) -> Tensor");
  m.def("sink_gate(Tensor o, Tensor lse, Tensor sink, Tensor gate, int vdim) -> Tensor");
  m.def("flash_sink_fwd(Tensor q, Tensor k, Tensor v, Tensor? kpm, Tensor? sink, Tensor? gate, float scale, float softcap, int window=0, int keep_first=0, Tensor? lead=None, Tensor? q2=None, Tensor? k2=None) -> Tensor");
  m.def("sink_attention(Tensor q, Tensor k, Tensor v, Tensor? keep, Tensor? sink, Tensor? gate, float scale, float softcap, int window=0, int keep_first=0, Tensor? lead=None) -> Tensor");
  m.def("latent_prep(Tensor cq, Tensor wq, Tensor? ckv, Tensor? wkv, Tensor(a!)? cache, Tensor lengths, float eps, Tensor? positions=None, Tensor? freq=None, bool rows=False) -> (Tensor, Tensor)");
  m.def("rotate_halves_(Tensor(a!) q, Tensor positions, Tensor freq) -> Tensor(a!)");
  m.def("latent_decode(Tensor q, Tensor w_uk, Tensor w_uv, Tensor cache, Tensor lengths, Tensor? keep, Tensor? sink, Tensor gate, float scale, int heads, Tensor? positions=None, Tensor? freq=None) -> Tensor");
  m.def("moe_route(Tensor h, Tensor w, Tensor? bias, Tensor? logits, int top, int scored=0) -> (Tensor, Tensor)");
  m.def("moe_plan(Tensor h, Tensor idx, int experts, Tensor? scale=None) -> (Tensor, Tensor, Tensor, Tensor)");
  m.def("moe_grouped(Tensor rows, Tensor w, Tensor tile_group, Tensor n_tiles, int unit, float limit=0., float alpha=1.) -> Tensor");
  m.def("moe_few(Tensor x, Tensor idx, Tensor w, int per_row, int unit, float limit=0., float alpha=1., Tensor? scale=None) -> Tensor");
  m.def("clamped_glu(Tensor gate, Tensor up, float limit, float alpha) -> Tensor");
  m.def("branch_join(Tensor x, Tensor[] y, Tensor?[] w, float[] factor, int[] normed, Tensor?[] slots, int[] top, float mult, float eps, Tensor? w1, Tensor? w2, bool copy=False, Tensor? conv_w=None, Tensor(a!)? prev=None, Tensor? keep=None) -> (Tensor, Tensor, Tensor, Tensor)");
  m.def("gated_rms_norm(Tensor o, Tensor w, Tensor gate, float eps, int group, int act, Tensor? z=None, Tensor? m=None) -> Tensor");
  m.def("hyper_join(Tensor x, Tensor? y, Tensor? slots, Tensor? weights, Tensor? choice, int experts, Tensor? own, Tensor? shared, Tensor? gate, Tensor? w_out, Tensor? mix, Tensor? w_in, Tensor w_norm, float eps, float scale) -> (Tensor, Tensor)");
  m.def("memory_gates(Tensor z, Tensor bias, float cap, Tensor? keep, Tensor(a!)? top, int batch) -> (Tensor, Tensor, Tensor, Tensor)");
  m.def("memory_recurrence(Tensor q, Tensor k, Tensor v, Tensor read, Tensor write, Tensor start, float q_scale, Tensor? keep, Tensor(a!)? state, int batch, int heads, int dim, int vdim, int chunks=0) -> (Tensor, Tensor)");
  m.def("memory_step(Tensor q, Tensor k, Tensor v, Tensor x, Tensor w, Tensor bias, float cap, Tensor gate, Tensor norm_w, Tensor? keep, Tensor(a!) state, Tensor(b!) top, float q_scale, float eps, int heads, int dim, int vdim) -> Tensor");
  m.def("gemv_stacked(Tensor x, Tensor w) -> Tensor");
  m.def("decayed_recurrence(Tensor q, Tensor k, Tensor v, Tensor decay, Tensor? keep, Tensor(a!)? state, int batch, int heads, int dim, int vdim, int chunks=0) -> Tensor");
  m.def("bonus_recurrence(Tensor q, Tensor k, Tensor v, Tensor z, Tensor w0, Tensor u, Tensor? keep, Tensor(a!)? state, int batch, int heads, int dim, int vdim, int chunks=0) -> Tensor");
  m.def("decayed_step(Tensor q, Tensor k, Tensor v, Tensor decay, Tensor? keep, Tensor(a!) state, int heads, int dim, int vdim) -> Tensor");
  m.def("bonus_step(Tensor r, Tensor k, Tensor v, Tensor t, Tensor w2, Tensor w0, Tensor u, Tensor norm_w, Tensor gate, Tensor? keep, Tensor(a!) state, float eps, int heads, int dim, int vdim) -> Tensor");
  m.def("qkv_prep(Tensor q, Tensor k, Tensor v, Tensor? wq, Tensor? wk, float eps, Tensor positions, Tensor freq, Tensor(a!) kc, Tensor(b!) vc, Tensor lengths) -> Tensor");
  m.def("head_prep(Tensor q, Tensor k, Tensor v, Tensor? wq, Tensor? wk, float eps, Tensor positions, Tensor freq, bool halves, float amplitude, Tensor? talk, Tensor(a!) kc, Tensor(b!) vc, Tensor lengths) -> Tensor");
  m.def("wide_decode_fits(Tensor like, int heads, int value_heads, int dim, int vdim) -> bool");
  m.def("flash_wide_fwd(Tensor q, Tensor k, Tensor v, Tensor? kpm, Tensor? sink, Tensor? gate, float scale, int window=0, int keep_first=0, Tensor? lead=None) -> Tensor");
  m.def("token_gate(Tensor z, Tensor ids, Tensor table, int first) -> Tensor");
  m.def("grouped_decode(Tensor q, Tensor kc, Tensor vc, Tensor lengths, Tensor? keep, Tensor? sink, float scale, float softcap, Tensor? gate=None, int window=0, int keep_first=0, Tensor? lead=None, int value_heads=1) -> Tensor");
  m.def("token_shift(Tensor h, Tensor mu, int batch, Tensor? keep, Tensor(a!)? prev) -> Tensor");
  m.def("causal_conv(Tensor x, Tensor w, Tensor? bias, int batch, Tensor? keep, Tensor(a!)? prev, bool silu=False, bool residual=False) -> Tensor");
  m.def("selective_scan(Tensor x, Tensor dt, Tensor dt_bias, Tensor a_log, Tensor b, Tensor c, Tensor d, Tensor z, int batch, Tensor? keep, Tensor(a!)? state, int chunks=0) -> Tensor");
  m.def("scan_step(Tensor x, Tensor dt, Tensor w_dt, Tensor dt_bias, Tensor a_log, Tensor b, Tensor c, Tensor d, Tensor z, Tensor? keep, Tensor(a!) state) -> Tensor");
}

TORCH_LIBRARY_IMPL(oslo_b200, CUDA, m) {
  m.impl("error_word", &error_word);
  m.impl("gemm", &gemm);
  m.impl("gemm_small_m", &gemm_small_m);
  m.impl("gemm_ce_stats", &gemm_ce_stats);
  m.impl("gemm_ce_grad", &gemm_ce_grad);
  m.impl("layernorm_fwd", &layernorm_fwd);
  m.impl("layernorm_bwd", &layernorm_bwd);
  m.impl("bias_gelu_fwd", &bias_gelu_fwd);
  m.impl("bias_gelu_bwd", &bias_gelu_bwd);
  m.impl("bias_dropout_residual", &bias_dropout_residual);
  m.impl("colsum", &colsum);
  m.impl("rotary", &rotary);
  m.impl("rotary_", &rotary_);
  m.impl("causal_softmax_fwd", &causal_softmax_fwd);
  m.impl("masked_softmax_fwd", &masked_softmax_fwd);
  m.impl("softmax_bwd", &softmax_bwd);
  m.impl("ce_stats", &ce_stats);
  m.impl("ce_grad_", &ce_grad_);
  m.impl("adam_step", &adam_step);
  m.impl("sumsq", &sumsq);
  m.impl("ngram_ban_", &ngram_ban_);
  m.impl("flash_fwd", &flash_fwd);
  m.impl("flash_bwd", &flash_bwd);
  m.impl("decode_attn", &decode_attn);
  m.impl("gemm_comm", &gemm_comm);
  m.impl("gemv_rows", &gemv_rows);
  m.impl("rotary_append", &rotary_append);
  m.impl("vocab_embed", &vocab_embed);
  m.impl("wait_probe", &wait_probe);
  m.impl("allreduce_oneshot", &allreduce_oneshot);
  m.impl("allreduce_symm", &allreduce_symm);
  m.impl("ce_combine", &ce_combine);
  m.impl("dp_reduce_scatter", &dp_reduce_scatter);
  m.impl("dp_all_gather", &dp_all_gather);
  m.impl("rms_norm", &rms_norm);
  m.impl("residual_join", &residual_join);
  m.impl("silu_mul", &silu_mul);
  m.impl("recurrence", &recurrence);
  m.impl("recurrence_step", &recurrence_step);
  m.impl("sink_gate", &sink_gate);
  m.impl("flash_sink_fwd", &flash_sink_fwd);
  m.impl("sink_attention", &sink_attention);
  m.impl("latent_prep", &latent_prep);
  m.impl("rotate_halves_", &rotate_halves_);
  m.impl("hyper_join", &hyper_join);
  m.impl("memory_gates", &memory_gates);
  m.impl("memory_recurrence", &memory_recurrence);
  m.impl("memory_step", &memory_step);
  m.impl("latent_decode", &latent_decode);
  m.impl("moe_route", &moe_route);
  m.impl("moe_plan", &moe_plan);
  m.impl("moe_grouped", &moe_grouped);
  m.impl("moe_few", &moe_few);
  m.impl("clamped_glu", &clamped_glu);
  m.impl("branch_join", &branch_join);
  m.impl("gated_rms_norm", &gated_rms_norm);
  m.impl("gemv_stacked", &gemv_stacked);
  m.impl("decayed_recurrence", &decayed_recurrence);
  m.impl("bonus_recurrence", &bonus_recurrence);
  m.impl("decayed_step", &decayed_step);
  m.impl("bonus_step", &bonus_step);
  m.impl("qkv_prep", &qkv_prep);
  m.impl("head_prep", &head_prep);
  m.impl("wide_decode_fits", &wide_decode_fits);
  m.impl("flash_wide_fwd", &flash_wide_fwd);
  m.impl("token_gate", &token_gate);
  m.impl("grouped_decode", &grouped_decode);
  m.impl("token_shift", &token_shift);
  m.impl("causal_conv", &causal_conv);
  m.impl("selective_scan", &selective_scan);
  m.impl("scan_step", &scan_step);
}
