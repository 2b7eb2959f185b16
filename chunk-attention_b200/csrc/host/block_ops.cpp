// chunk_attn_c.ops, second part: the block kernels of decoders with an fp32 residual stream and recurrent mixers.  They
// check and unwrap the tensors and call the C ABI on torch's current stream.
#include <c10/cuda/CUDAGuard.h>
#include <c10/cuda/CUDAStream.h>
#include <pybind11/pybind11.h>
#include <pybind11/stl.h>
#include <torch/extension.h>

#include <stdexcept>

#include "../../../include/chunk_attn_b200.h"
#include "spans.h"

namespace py = pybind11;

namespace ca_host {
namespace {

using torch::Tensor;

int dtype_code(const Tensor& t, const char* what) {
    if (t.scalar_type() == torch::kFloat16) return CA_DTYPE_F16;
    if (t.scalar_type() == torch::kFloat32) return CA_DTYPE_F32;
    if (t.scalar_type() == torch::kBFloat16) return CA_DTYPE_BF16;
    throw std::runtime_error(std::string(what) + ": fp16, bf16 and fp32 tensors only");
}
void need(bool ok, const char* msg) {
    if (!ok) throw std::runtime_error(msg);
}
void check_rc(int rc, const char* what) {
    if (rc != CA_OK) throw std::runtime_error(std::string(what) + ": " + ca_last_error());
}
void* stream_of(const Tensor& t) { return c10::cuda::getCurrentCUDAStream(t.device().index()).stream(); }
bool f32_vec(const Tensor& t, int64_t n) {
    return t.is_cuda() && t.scalar_type() == torch::kFloat32 && t.is_contiguous() && t.numel() == n;
}
// rows of a 2-d tensor whose columns are contiguous
bool rows_of(const Tensor& t, int64_t rows, int64_t width) {
    return t.is_cuda() && t.dim() == 2 && t.size(0) == rows && t.size(1) == width && (t.stride(1) == 1 || width == 1);
}
bool state_ok(const Tensor& s, const SpanBatch& sp, int64_t per_slot) {
    return s.is_cuda() && s.scalar_type() == torch::kFloat32 && s.is_contiguous() && s.dim() >= 1 && s.size(0) > sp.max_slot() &&
           s.numel() == s.size(0) * per_slot;
}

py::tuple token_shift(Tensor x, Tensor mu, Tensor state, const SpanBatch& sp, py::object dtype) {
    const int64_t T = sp.n_tokens(), W = x.size(-1);
    need(rows_of(x, T, W) && x.is_contiguous() && x.scalar_type() == torch::kFloat32, "token_shift: x must be contiguous fp32 [n_tokens, width] on a CUDA device (there is no CPU path)");
    need(f32_vec(mu, W) && state_ok(state, sp, W), "token_shift: mu must be fp32 [width], state fp32 [slots, width]");
    c10::cuda::CUDAGuard guard(x.device());
    const auto opt = x.options().dtype(torch::python::detail::py_object_to_dtype(dtype));
    Tensor plain = torch::empty({T, W}, opt), shifted = torch::empty({T, W}, opt);
    check_rc(ca_token_shift(x.data_ptr<float>(), mu.data_ptr<float>(), state.data_ptr<float>(), plain.data_ptr(), shifted.data_ptr(),
                            sp.view(), (int)W, dtype_code(plain, "token_shift"), stream_of(x)),
             "token_shift");
    return py::make_tuple(plain, shifted);
}

// x (fp32, in place) += rms_norm(r * sigmoid(gate + bias)) * weight.  Returns (x rounded, shifted or None).
py::tuple gated_norm_add(Tensor x, Tensor r, Tensor gate, Tensor bias, Tensor weight, double eps, bool want_plain,
                         c10::optional<Tensor> next_mu, c10::optional<Tensor> next_state, c10::optional<const SpanBatch*> sp) {
    const int64_t T = x.size(0), W = x.size(-1);
    need(rows_of(x, T, W) && x.is_contiguous() && x.scalar_type() == torch::kFloat32, "gated_norm_add: x must be contiguous fp32 [n_tokens, width] on a CUDA device (there is no CPU path)");
    need(rows_of(r, T, W) && rows_of(gate, T, W) && gate.scalar_type() == r.scalar_type(), "gated_norm_add: r and gate must be [n_tokens, width] of one dtype");
    need(f32_vec(bias, W) && f32_vec(weight, W), "gated_norm_add: bias and weight must be fp32 [width]");
    c10::cuda::CUDAGuard guard(x.device());
    const bool fuse = next_mu.has_value();
    need(!fuse || (next_state.has_value() && sp.has_value() && *sp && f32_vec(*next_mu, W) && state_ok(*next_state, **sp, W)),
         "gated_norm_add: the fused token shift needs spans, fp32 mu [width] and state [slots, width]");
    Tensor plain, shifted;
    if (want_plain) plain = torch::empty({T, W}, r.options());
    if (fuse) shifted = torch::empty({T, W}, r.options());
    check_rc(ca_gated_norm_add(x.data_ptr<float>(), r.data_ptr(), r.stride(0), gate.data_ptr(), gate.stride(0), bias.data_ptr<float>(),
                               weight.data_ptr<float>(), (float)eps, want_plain ? plain.data_ptr() : nullptr,
                               fuse ? next_mu->data_ptr<float>() : nullptr, fuse ? next_state->data_ptr<float>() : nullptr,
                               fuse ? shifted.data_ptr() : nullptr, fuse ? (*sp)->view() : nullptr, T, (int)W,
                               dtype_code(r, "gated_norm_add"), stream_of(x)),
             "gated_norm_add");
    return py::make_tuple(want_plain ? py::cast(plain) : py::none(), fuse ? py::cast(shifted) : py::none());
}

Tensor norm_rows(Tensor x, Tensor weight, double eps, py::object dtype, c10::optional<Tensor> rows, c10::optional<Tensor> gate) {
    const int64_t W = x.size(-1), T = rows.has_value() ? rows->numel() : x.size(0);
    need(rows_of(x, x.size(0), W) && f32_vec(weight, W), "norm_rows: x must be [rows, width] on a CUDA device, weight fp32 [width]");
    need(!rows.has_value() || (rows->is_cuda() && rows->scalar_type() == torch::kInt32 && rows->is_contiguous()), "norm_rows: rows must be int32");
    c10::cuda::CUDAGuard guard(x.device());
    Tensor out = torch::empty({T, W}, x.options().dtype(torch::python::detail::py_object_to_dtype(dtype)));
    need(x.scalar_type() == torch::kFloat32 || x.scalar_type() == out.scalar_type(), "norm_rows: x must be fp32 or of the output's dtype");
    need(!gate.has_value() || (rows_of(*gate, T, W) && gate->scalar_type() == out.scalar_type()), "norm_rows: gate must be [rows, width] of the output's dtype");
    check_rc(ca_norm_rows(out.data_ptr(), x.data_ptr(), x.scalar_type() == torch::kFloat32, x.stride(0),
                          rows.has_value() ? rows->data_ptr<int32_t>() : nullptr, weight.data_ptr<float>(),
                          gate.has_value() ? gate->data_ptr() : nullptr, gate.has_value() ? gate->stride(0) : 0, (float)eps, T, (int)W,
                          dtype_code(out, "norm_rows"), stream_of(x)),
             "norm_rows");
    return out;
}

// fp32 rows of the embedding table for a batch's tokens, times scale, and with want_plain the same rounded; a token outside
// the table raises before anything runs
py::object embed_rows(Tensor table, const SpanBatch& sp, double scale, bool want_plain) {
    need(table.is_cuda() && table.dim() == 2 && table.is_contiguous() && table.device() == sp.device(), "embed_rows: a contiguous [vocab, width] table on the spans' CUDA device is required");
    need(sp.min_token() >= 0 && sp.max_token() < table.size(0), "embed_rows: a token id lies outside the vocabulary");
    c10::cuda::CUDAGuard guard(table.device());
    Tensor x = torch::empty({sp.n_tokens(), table.size(1)}, table.options().dtype(torch::kFloat32)), plain;
    if (want_plain) plain = torch::empty({sp.n_tokens(), table.size(1)}, table.options());
    check_rc(ca_embed_rows(x.data_ptr<float>(), want_plain ? plain.data_ptr() : nullptr, table.data_ptr(), sp.tokens.data_ptr<int32_t>(),
                           (float)scale, sp.n_tokens(), (int)table.size(1), dtype_code(table, "embed_rows"), stream_of(table)),
             "embed_rows");
    if (!want_plain) return py::cast(x);
    return py::make_tuple(x, plain);
}

// x (fp32, in place) = rms_norm(alpha * x + r + bias) * weight.  Returns x rounded to r's type, or x itself in fp32.
Tensor scaled_norm(Tensor x, Tensor r, double alpha, Tensor weight, double eps, c10::optional<Tensor> bias) {
    const int64_t T = x.size(0), W = x.size(-1);
    need(rows_of(x, T, W) && x.is_contiguous() && x.scalar_type() == torch::kFloat32, "scaled_norm: x must be contiguous fp32 [n_tokens, width] on a CUDA device (there is no CPU path)");
    need(rows_of(r, T, W) && f32_vec(weight, W) && (!bias.has_value() || f32_vec(*bias, W)), "scaled_norm: r must be [n_tokens, width], weight and bias fp32 [width]");
    c10::cuda::CUDAGuard guard(x.device());
    const bool rounded = r.scalar_type() != torch::kFloat32;
    Tensor plain = rounded ? torch::empty({T, W}, r.options()) : x;
    check_rc(ca_scaled_norm(x.data_ptr<float>(), r.data_ptr(), r.stride(0), bias.has_value() ? bias->data_ptr<float>() : nullptr, (float)alpha,
                            weight.data_ptr<float>(), (float)eps, rounded ? plain.data_ptr() : nullptr, T, (int)W, dtype_code(r, "scaled_norm"),
                            stream_of(x)),
             "scaled_norm");
    return plain;
}

Tensor clamped_glu(Tensor x, Tensor bias, double limit, double slope) {
    const int64_t T = x.size(0), F = x.size(-1) / 2;
    need(rows_of(x, T, 2 * F) && f32_vec(bias, 2 * F), "clamped_glu: [rows, gate | up] on a CUDA device and an fp32 bias [gate | up] are required");
    c10::cuda::CUDAGuard guard(x.device());
    Tensor out = torch::empty({T, F}, x.options());
    check_rc(ca_clamped_glu(out.data_ptr(), x.data_ptr(), x.stride(0), bias.data_ptr<float>(), (float)limit, (float)slope, T, (int)F,
                            dtype_code(x, "clamped_glu"), stream_of(x)),
             "clamped_glu");
    return out;
}

Tensor softcap(Tensor z, double cap) {
    need(z.is_cuda() && z.scalar_type() == torch::kFloat32 && z.is_contiguous(), "softcap: a contiguous fp32 tensor on a CUDA device is required");
    c10::cuda::CUDAGuard guard(z.device());
    check_rc(ca_softcap(z.data_ptr<float>(), (float)cap, z.numel(), stream_of(z)), "softcap");
    return z;
}

Tensor gelu_tanh(Tensor x) {
    need(rows_of(x, x.size(0), x.size(-1)), "gelu_tanh: [rows, width] on a CUDA device is required");
    c10::cuda::CUDAGuard guard(x.device());
    Tensor out = torch::empty({x.size(0), x.size(1)}, x.options());
    check_rc(ca_gelu_tanh(out.data_ptr(), x.data_ptr(), x.stride(0), x.size(0), (int)x.size(1), dtype_code(x, "gelu_tanh"), stream_of(x)), "gelu_tanh");
    return out;
}

Tensor conv_silu(Tensor x, Tensor taps, Tensor bias, Tensor state, const SpanBatch& sp) {
    const int64_t T = sp.n_tokens(), C = x.size(-1);
    need(rows_of(x, T, C), "conv_silu: x must be [n_tokens, channels] on a CUDA device (there is no CPU path)");
    const int64_t K = taps.size(-1);
    need(f32_vec(taps, C * K) && f32_vec(bias, C) && state_ok(state, sp, (K - 1) * C), "conv_silu: taps must be fp32 [channels, taps], bias fp32 [channels], state fp32 [slots, taps - 1, channels]");
    c10::cuda::CUDAGuard guard(x.device());
    Tensor out = torch::empty({T, C}, x.options());
    // a filter of one tap has no state; the kernel still wants an address
    check_rc(ca_conv_silu(out.data_ptr(), x.data_ptr(), x.stride(0), taps.data_ptr<float>(), bias.data_ptr<float>(),
                          K > 1 ? state.data_ptr<float>() : bias.data_ptr<float>(), sp.view(), (int)C, (int)K, dtype_code(x, "conv_silu"), stream_of(x)),
             "conv_silu");
    return out;
}

Tensor selective_scan(Tensor x, Tensor z, Tensor dt, Tensor dt_bias, Tensor A, Tensor bc, Tensor D, Tensor state, const SpanBatch& sp) {
    const int64_t T = sp.n_tokens(), C = x.size(-1), N = A.size(-1);
    need(rows_of(x, T, C) && x.is_contiguous() && rows_of(z, T, C) && z.scalar_type() == x.scalar_type(), "selective_scan: x and z must be [n_tokens, channels] on a CUDA device (there is no CPU path)");
    need(rows_of(dt, T, C) && dt.is_contiguous() && dt.scalar_type() == torch::kFloat32, "selective_scan: dt must be fp32 [n_tokens, channels]");
    need(rows_of(bc, T, 2 * N) && bc.scalar_type() == torch::kFloat32, "selective_scan: bc must be fp32 [n_tokens, 2 states]");
    need(f32_vec(A, C * N) && f32_vec(D, C) && f32_vec(dt_bias, C) && state_ok(state, sp, C * N), "selective_scan: A fp32 [channels, states], D and dt_bias fp32 [channels], state fp32 [slots, channels, states]");
    c10::cuda::CUDAGuard guard(x.device());
    Tensor y = torch::empty({T, C}, x.options());
    const int64_t n = ca_scan_scratch_floats(sp.view(), (int)C, (int)N);
    Tensor scratch;
    if (n > 0) scratch = torch::empty({n}, x.options().dtype(torch::kFloat32));
    check_rc(ca_selective_scan(y.data_ptr(), x.data_ptr(), z.data_ptr(), z.stride(0), dt.data_ptr<float>(), dt_bias.data_ptr<float>(),
                               A.data_ptr<float>(), bc.data_ptr<float>(), bc.stride(0), D.data_ptr<float>(), state.data_ptr<float>(),
                               n > 0 ? scratch.data_ptr<float>() : nullptr, sp.view(), (int)C, (int)N, dtype_code(x, "selective_scan"), stream_of(x)),
             "selective_scan");
    return y;
}

Tensor decay_attention(Tensor qkv, Tensor decay, int64_t d_key, int64_t d_value, Tensor state, const SpanBatch& sp) {
    const int64_t T = sp.n_tokens(), H = decay.numel();
    need(qkv.is_cuda() && qkv.dim() == 2 && qkv.size(0) == T && qkv.stride(1) == 1 && qkv.size(1) >= H * (2 * d_key + d_value), "decay_attention: qkv must be [n_tokens, q | k | v heads] on a CUDA device (there is no CPU path)");
    need(f32_vec(decay, H) && state_ok(state, sp, H * d_key * d_value), "decay_attention: decay fp32 [heads], state fp32 [slots, heads, d_key, d_value]");
    c10::cuda::CUDAGuard guard(qkv.device());
    Tensor out = torch::empty({T, H * d_value}, qkv.options());
    const int64_t n = ca_decay_scratch_floats(sp.view(), (int)H, (int)d_key, (int)d_value, dtype_code(qkv, "decay_attention"));
    Tensor scratch;
    if (n > 0) scratch = torch::empty({n}, qkv.options().dtype(torch::kFloat32));
    check_rc(ca_decay_attention(out.data_ptr(), qkv.data_ptr(), qkv.stride(0), decay.data_ptr<float>(), state.data_ptr<float>(),
                                n > 0 ? scratch.data_ptr<float>() : nullptr, sp.view(),
                                (int)H, (int)d_key, (int)d_value, dtype_code(qkv, "decay_attention"), stream_of(qkv)),
             "decay_attention");
    return out;
}

}  // namespace

void init_block_ops(py::module& m, py::module& ops) {
    py::class_<SpanBatch, std::shared_ptr<SpanBatch>>(m, "SpanBatch", py::module_local())
      .def(py::init([](const std::vector<std::vector<int>>& tokens, const std::vector<int>& starts, const std::vector<int>& slots,
                       py::object device, int work_len) {
               return std::make_shared<SpanBatch>(tokens, starts, slots, torch::python::detail::py_object_to_device(device), work_len);
           }),
           py::arg("tokens"), py::arg("starts"), py::arg("slots"), py::arg("device"), py::arg("work_len") = 64)
      .def_property_readonly("n_entries", &SpanBatch::n_entries)
      .def_property_readonly("n_tokens", &SpanBatch::n_tokens)
      .def_property_readonly("single", &SpanBatch::single)
      .def_readonly("tokens", &SpanBatch::tokens)
      .def_readonly("positions", &SpanBatch::positions)
      .def_readonly("entry_of", &SpanBatch::entry_of)
      .def_readonly("last", &SpanBatch::last);
    ops.def("token_shift", &token_shift, py::arg("x"), py::arg("mu"), py::arg("state"), py::arg("spans"), py::arg("dtype"),
            "(x rounded, x mixed with the previous token's) of an fp32 stream");
    ops.def("gated_norm_add", &gated_norm_add, py::arg("x"), py::arg("r"), py::arg("gate"), py::arg("bias"), py::arg("weight"), py::arg("eps"),
            py::arg("want_plain") = true, py::arg("next_mu") = py::none(), py::arg("next_state") = py::none(), py::arg("spans") = py::none(),
            "x += rms_norm(r * sigmoid(gate + bias)) * weight on an fp32 stream, in place");
    ops.def("norm_rows", &norm_rows, py::arg("x"), py::arg("weight"), py::arg("eps"), py::arg("dtype"), py::arg("rows") = py::none(),
            py::arg("gate") = py::none(), "RMS norm of (selected) rows, optionally times sigmoid(gate)");
    ops.def("embed_rows", &embed_rows, py::arg("table"), py::arg("spans"), py::arg("scale") = 1.0, py::arg("want_plain") = false,
            "fp32 embedding rows of a batch's tokens, times scale; with want_plain also rounded");
    ops.def("scaled_norm", &scaled_norm, py::arg("x"), py::arg("r"), py::arg("alpha"), py::arg("weight"), py::arg("eps"), py::arg("bias") = py::none(),
            "x = rms_norm(alpha x + r + bias) * weight on an fp32 stream, in place; returns it rounded to r's type");
    ops.def("clamped_glu", &clamped_glu, py::arg("x"), py::arg("bias"), py::arg("limit"), py::arg("slope") = 1.702,
            "gated linear unit of clamped halves: g sigmoid(slope g) (u + 1)");
    ops.def("softcap", &softcap, py::arg("z"), py::arg("cap"), "cap * tanh(z / cap) in place");
    ops.def("gelu_tanh", &gelu_tanh, py::arg("x"), "tanh form of GELU");
    ops.def("conv_silu", &conv_silu, py::arg("x"), py::arg("taps"), py::arg("bias"), py::arg("state"), py::arg("spans"),
            "causal depthwise convolution + SiLU over spans");
    ops.def("selective_scan", &selective_scan, py::arg("x"), py::arg("z"), py::arg("dt"), py::arg("dt_bias"), py::arg("A"), py::arg("bc"),
            py::arg("D"), py::arg("state"), py::arg("spans"), "selective scan over spans, gated by silu(z)");
    ops.def("block_status", [](py::object device) {
                const torch::Device d = torch::python::detail::py_object_to_device(device);
                c10::cuda::CUDAGuard guard(d);
                int32_t st = 0;
                check_rc(ca_block_status(&st, c10::cuda::getCurrentCUDAStream(d.index()).stream()), "block_status");
                return st;
            }, py::arg("device"), "0, or 1 when a bounded wait inside a block kernel has run out");
    ops.def("decay_attention", &decay_attention, py::arg("qkv"), py::arg("decay"), py::arg("d_key"), py::arg("d_value"), py::arg("state"),
            py::arg("spans"), "linear attention with a per-head decay over spans");
}

}  // namespace ca_host
