// Python bindings of the listed-layer kernels (launchers_layers.h).
#include "bindings_layers.h"

#include <ATen/cuda/CUDAContext.h>
#include <c10/cuda/CUDAGuard.h>
#include <pybind11/stl.h>

#include "launchers.h"
#include "launchers_layers.h"

namespace {

using torch::Tensor;
using OptTensor = c10::optional<torch::Tensor>;

inline cudaStream_t cur_stream() { return at::cuda::getCurrentCUDAStream(); }
inline bool is_f32(const Tensor& t, const char* name) {
  TORCH_CHECK(t.is_cuda() && (t.scalar_type() == torch::kFloat32 || t.scalar_type() == torch::kBFloat16), name, ": fp32 or bf16 CUDA tensor");
  return t.scalar_type() == torch::kFloat32;
}
inline void same_type(const Tensor& t, bool fp32, const char* name) {
  TORCH_CHECK(t.is_cuda() && t.scalar_type() == (fp32 ? torch::kFloat32 : torch::kBFloat16), name, ": dtype of the activations expected");
}
inline void check_f32(const Tensor& t, const char* name) { TORCH_CHECK(t.is_cuda() && t.scalar_type() == torch::kFloat32, name, ": fp32"); }
inline void check_i32(const Tensor& t, const char* name) { TORCH_CHECK(t.is_cuda() && t.scalar_type() == torch::kInt32, name, ": int32"); }
inline void rows2d(const Tensor& t, const char* name) { TORCH_CHECK(t.dim() == 2 && t.stride(1) == 1, name, ": 2-D, inner stride 1"); }
inline int* iptr(const OptTensor& t) { return t.has_value() && t->defined() ? t->data_ptr<int>() : nullptr; }
inline bool given(const OptTensor& t) { return t.has_value() && t->defined(); }
inline bool aligned16(const Tensor& t) { return (reinterpret_cast<uintptr_t>(t.data_ptr()) & 15) == 0; }

agrpo::DytArgs norm_args(const std::vector<Tensor>& n, bool fp32, int64_t W, const char* name) {
  TORCH_CHECK(n.size() == 3, name, ": (w, b, alpha)");
  for (const Tensor& t : n) same_type(t, fp32, name);
  TORCH_CHECK(n[0].numel() == W && n[1].numel() == W && n[2].numel() == 1 && n[0].is_contiguous() && n[1].is_contiguous() && aligned16(n[0]) &&
              aligned16(n[1]), name, ": w, b [width] contiguous and aligned, alpha one value");
  return agrpo::DytArgs{n[0].data_ptr(), n[1].data_ptr(), n[2].data_ptr()};
}

void embed_dyt(const Tensor& ids, const Tensor& table, double scale, Tensor& x, Tensor& h, const std::vector<Tensor>& norm) {
  const bool f = is_f32(table, "table");
  check_i32(ids, "ids"); check_f32(x, "x"); same_type(h, f, "h");
  const int64_t T = ids.numel(), W = table.size(1);
  TORCH_CHECK(table.is_contiguous() && x.is_contiguous() && h.is_contiguous() && W % 8 == 0 && aligned16(table), "embed_dyt layout");
  TORCH_CHECK(x.size(0) >= T && h.size(0) >= T && x.size(1) == W && h.size(1) == W, "embed_dyt: shapes");
  const c10::cuda::CUDAGuard guard(table.device());
  agrpo::launch_embed_dyt(f, ids.data_ptr<int>(), table.data_ptr(), (float)scale, x.data_ptr<float>(), h.data_ptr(),
                          norm_args(norm, f, W, "embed_dyt norm"), (int)T, (int)W, (int)table.size(0), cur_stream());
}

agrpo::ShortConvArgs conv_args(const Tensor& u, const Tensor& w, Tensor& ring, const OptTensor& rows, const OptTensor& seq_lens,
                               const Tensor& block_tables, Tensor& q_out, Tensor& k_cache, const OptTensor& status) {
  const bool f = is_f32(u, "u");
  same_type(w, f, "conv w"); same_type(ring, f, "ring"); same_type(q_out, f, "q_out"); same_type(k_cache, f, "k_cache");
  rows2d(u, "u"); check_i32(block_tables, "block_tables");
  TORCH_CHECK(k_cache.dim() == 4 && k_cache.is_contiguous() && k_cache.size(3) % 8 == 0, "short_conv: cache [blocks, G, bs, D]");
  agrpo::ShortConvArgs a{};
  a.D = (int)k_cache.size(3);
  a.k_cols = (int)(k_cache.size(1) * k_cache.size(3));
  a.q_cols = (int)q_out.size(1);
  const int64_t C = a.q_cols + a.k_cols, T = u.size(0);
  TORCH_CHECK(w.dim() == 2 && w.size(1) == C && w.is_contiguous() && aligned16(w), "short_conv: w [taps, q + k channels]");
  TORCH_CHECK(ring.dim() == 3 && ring.size(2) == C && ring.size(1) >= w.size(0) && ring.stride(2) == 1 &&
              ring.stride(1) == C && ring.stride(0) % 8 == 0 && aligned16(ring),
              "short_conv: ring [slots, >= taps, channels]");
  TORCH_CHECK(u.size(1) >= C && u.stride(0) % 8 == 0 && aligned16(u) && q_out.is_contiguous() && q_out.size(0) >= T && aligned16(q_out), "short_conv: u / q_out");
  TORCH_CHECK(block_tables.dim() == 2 && block_tables.is_contiguous(), "short_conv: tables");
  if (given(rows)) { check_i32(*rows, "rows"); TORCH_CHECK(rows->is_contiguous() && rows->numel() >= 4 * T, "short_conv: rows [T, 4]"); }
  else { TORCH_CHECK(given(seq_lens), "short_conv: rows or seq_lens"); check_i32(*seq_lens, "seq_lens");
         TORCH_CHECK(seq_lens->numel() >= T && block_tables.size(0) >= T && ring.size(0) >= T, "short_conv: decode rows"); }
  a.u = u.data_ptr(); a.ldu = u.stride(0);
  a.w = w.data_ptr(); a.taps = (int)w.size(0);
  a.ring = ring.data_ptr(); a.ring_len = (int)ring.size(1); a.ring_pitch = ring.stride(0);
  a.rows = iptr(rows); a.seq_lens = iptr(seq_lens);
  a.block_tables = block_tables.data_ptr<int>(); a.max_blocks = (int)block_tables.size(1);
  a.q_out = q_out.data_ptr(); a.k_cache = k_cache.data_ptr();
  a.block_size = (int)k_cache.size(2); a.num_cache_blocks = (int)k_cache.size(0);
  a.T = (int)T;
  a.status = iptr(status);
  return a;
}

void short_conv(const Tensor& u, const Tensor& w, Tensor& ring, const OptTensor& rows, const OptTensor& ring_rows, const OptTensor& seq_lens,
                const Tensor& block_tables, Tensor& q_out, Tensor& k_cache, const OptTensor& status) {
  const agrpo::ShortConvArgs a = conv_args(u, w, ring, rows, seq_lens, block_tables, q_out, k_cache, status);
  const bool f = u.scalar_type() == torch::kFloat32;
  if (given(rows)) { TORCH_CHECK(given(ring_rows) && ring_rows->is_contiguous(), "short_conv: ring_rows with rows"); check_i32(*ring_rows, "ring_rows"); }
  const c10::cuda::CUDAGuard guard(u.device());
  if (!given(rows)) return agrpo::launch_short_conv_decode(f, a, cur_stream());
  agrpo::launch_short_conv(f, a, cur_stream());
  agrpo::launch_short_conv_ring(f, a, ring_rows->data_ptr<int>(), (int)ring_rows->numel(), cur_stream());
}

agrpo::WindowAttnArgs attn_args(const OptTensor& q, const Tensor& k_cache, const OptTensor& rows, const OptTensor& seq_lens,
                                const Tensor& block_tables, const Tensor& bias, const Tensor& qscale, const OptTensor& talk,
                                const OptTensor& gate, int64_t window, Tensor& out, const OptTensor& status) {
  const bool f = is_f32(k_cache, "k_cache");
  same_type(out, f, "out");
  check_i32(block_tables, "block_tables"); check_f32(bias, "bias"); check_f32(qscale, "qscale");
  TORCH_CHECK(k_cache.dim() == 4 && k_cache.is_contiguous() && k_cache.size(3) % 8 == 0 && aligned16(k_cache), "attn: cache [blocks, G, bs, D]");
  TORCH_CHECK(bias.dim() == 2 && bias.is_contiguous() && qscale.is_contiguous(), "attn: bias [H, distances]");
  agrpo::WindowAttnArgs a{};
  a.H = (int)bias.size(0); a.G = (int)k_cache.size(1); a.D = (int)k_cache.size(3);
  TORCH_CHECK(a.H % a.G == 0, "attn: key heads must divide query heads");
  rows2d(out, "out");
  a.T = (int)out.size(0);
  TORCH_CHECK(out.size(1) == (int64_t)a.H * a.D && out.stride(0) % 8 == 0 && aligned16(out), "attn: out [T, H * D]");
  if (given(q)) {
    same_type(*q, f, "q"); rows2d(*q, "q");
    TORCH_CHECK(q->size(1) == out.size(1) && q->size(0) >= a.T && q->stride(0) % 8 == 0 && aligned16(*q), "attn: q [T, H * D]");
    a.q = q->data_ptr(); a.ldq = q->stride(0);
  }
  if (given(talk)) { same_type(*talk, f, "talk"); TORCH_CHECK(talk->numel() == (int64_t)a.H * a.H && talk->is_contiguous(), "attn: talk [H, H]"); a.talk = talk->data_ptr(); }
  if (given(gate)) { same_type(*gate, f, "gate"); rows2d(*gate, "gate");
                     TORCH_CHECK(gate->size(1) == out.size(1) && gate->size(0) >= a.T && gate->stride(0) % 8 == 0 && aligned16(*gate), "attn: gate [T, H * D]");
                     a.gate = gate->data_ptr(); a.ldg = gate->stride(0); }
  TORCH_CHECK(window >= 1 && bias.size(1) >= std::min<int64_t>(window, qscale.numel()), "attn: bias table shorter than the window");
  TORCH_CHECK(block_tables.dim() == 2 && block_tables.is_contiguous(), "attn: tables");
  if (given(rows)) { check_i32(*rows, "rows"); TORCH_CHECK(rows->is_contiguous() && rows->numel() >= 4 * a.T, "attn: rows [T, 4]"); }
  if (given(seq_lens)) { check_i32(*seq_lens, "seq_lens"); TORCH_CHECK(seq_lens->numel() >= a.T && block_tables.size(0) >= a.T, "attn: decode rows"); }
  a.k_cache = k_cache.data_ptr();
  a.rows = iptr(rows); a.seq_lens = iptr(seq_lens);
  a.block_tables = block_tables.data_ptr<int>(); a.max_blocks = (int)block_tables.size(1);
  a.bias = bias.data_ptr<float>(); a.bias_len = (int)bias.size(1);
  a.qscale = qscale.data_ptr<float>(); a.qscale_len = (int)qscale.numel();
  a.window = (int)window;
  a.out = out.data_ptr(); a.ldo = out.stride(0);
  a.block_size = (int)k_cache.size(2); a.num_cache_blocks = (int)k_cache.size(0);
  a.status = iptr(status);
  return a;
}

void window_attn(const Tensor& q, const Tensor& k_cache, const OptTensor& rows, const OptTensor& seq_lens, const Tensor& block_tables,
                 const Tensor& bias, const Tensor& qscale, const OptTensor& talk, const OptTensor& gate, int64_t window, Tensor& out,
                 const OptTensor& status) {
  TORCH_CHECK(given(rows) || given(seq_lens), "window_attn: rows or seq_lens");
  const agrpo::WindowAttnArgs a = attn_args(q, k_cache, rows, seq_lens, block_tables, bias, qscale, talk, gate, window, out, status);
  const c10::cuda::CUDAGuard guard(k_cache.device());
  agrpo::launch_window_attn(k_cache.scalar_type() == torch::kFloat32, a, cur_stream());
}

// Tensor-core form for prompts; false (nothing launched) when the shape is not served.
bool talk_attn_prefill(const Tensor& q, const Tensor& k_cache, const Tensor& tiles, const Tensor& pages, Tensor& keys, const Tensor& block_tables, const Tensor& bias,
                       const Tensor& qscale, const OptTensor& talk, const OptTensor& gate, int64_t window, Tensor& acc, Tensor& out,
                       const OptTensor& status) {
  if (k_cache.scalar_type() != torch::kBFloat16 || k_cache.size(2) != 16) return false;
  check_i32(tiles, "tiles");
  TORCH_CHECK(tiles.dim() == 2 && tiles.size(1) == 4 && tiles.is_contiguous() && aligned16(tiles), "talk_attn_prefill: tiles [n, 4]");
  check_i32(pages, "pages"); same_type(keys, false, "keys");
  TORCH_CHECK(pages.dim() == 2 && pages.size(1) == 2 && pages.is_contiguous() && (reinterpret_cast<uintptr_t>(pages.data_ptr()) & 7) == 0, "talk_attn_prefill: pages [n, 2]");
  TORCH_CHECK(keys.is_contiguous() && aligned16(keys) && keys.numel() >= pages.size(0) * 16 * k_cache.size(1) * k_cache.size(3),
              "talk_attn_prefill: keys [16 pages, G * D]");
  const agrpo::WindowAttnArgs a = attn_args(q, k_cache, OptTensor(), OptTensor(), block_tables, bias, qscale, talk, gate, window, out, status);
  same_type(acc, false, "acc");
  TORCH_CHECK(acc.is_contiguous() && acc.numel() >= (int64_t)a.T * a.H * a.G * a.D && aligned16(acc), "talk_attn_prefill: acc [T, H, G, D]");
  const c10::cuda::CUDAGuard guard(k_cache.device());
  return agrpo::launch_talk_attn_prefill(a, tiles.data_ptr<int>(), (int)tiles.size(0), pages.data_ptr<int>(), (int)pages.size(0),
                                         keys.data_ptr(), acc.data_ptr(), cur_stream());
}

// Decode step of a mixer after its fused projection u = [q | k | gate]: convolution, attention, mixing, gate, state update.
void talk_attn_decode(const Tensor& u, const Tensor& conv_w, Tensor& ring, Tensor& k_cache, const Tensor& seq_lens, const Tensor& block_tables,
                      const Tensor& bias, const Tensor& qscale, const OptTensor& talk, const OptTensor& gate, int64_t window, Tensor& out,
                      int64_t splits, Tensor& part_o, Tensor& part_ml, Tensor& tickets, const OptTensor& status) {
  TORCH_CHECK(k_cache.scalar_type() == torch::kBFloat16, "talk_attn_decode: bf16");
  agrpo::TalkDecodeArgs d{};
  d.at = attn_args(OptTensor(), k_cache, OptTensor(), seq_lens, block_tables, bias, qscale, talk, gate, window, out, status);
  const int64_t C = (int64_t)(d.at.H + d.at.G) * d.at.D, B = d.at.T;
  same_type(u, false, "u"); same_type(conv_w, false, "conv_w"); same_type(ring, false, "ring"); rows2d(u, "u");
  check_f32(part_o, "part_o"); check_f32(part_ml, "part_ml"); check_i32(tickets, "tickets");
  TORCH_CHECK(u.size(0) >= B && u.size(1) >= C && u.stride(0) % 8 == 0 && aligned16(u), "talk_attn_decode: u");
  TORCH_CHECK(conv_w.dim() == 2 && conv_w.size(1) == C && conv_w.is_contiguous() && aligned16(conv_w), "talk_attn_decode: conv_w [taps, q + k channels]");
  TORCH_CHECK(ring.dim() == 3 && ring.size(0) >= B && ring.size(1) == conv_w.size(0) && ring.size(2) == C && ring.stride(2) == 1 &&
              ring.stride(1) == C && ring.stride(0) % 8 == 0 && aligned16(ring), "talk_attn_decode: ring [slots, taps, channels]");
  TORCH_CHECK(splits >= 1 && splits <= 8, "talk_attn_decode: 1 to 8 splits");
  TORCH_CHECK(splits == 1 || (part_o.numel() >= B * splits * d.at.H * d.at.G * d.at.D && part_ml.numel() >= B * splits * d.at.H * 2 &&
              tickets.numel() >= B), "talk_attn_decode: scratch");
  d.u = u.data_ptr(); d.ldu = u.stride(0);
  d.conv_w = conv_w.data_ptr(); d.taps = (int)conv_w.size(0);
  d.ring = ring.data_ptr(); d.ring_len = (int)ring.size(1); d.ring_pitch = ring.stride(0);
  d.k_cache = k_cache.data_ptr();
  d.splits = (int)splits;
  d.part_o = part_o.data_ptr<float>(); d.part_ml = part_ml.data_ptr<float>(); d.tickets = tickets.data_ptr<int>();
  const c10::cuda::CUDAGuard guard(k_cache.device());
  agrpo::launch_talk_attn_decode(d, cur_stream());
}

// D = A . B^T + the sublayer tail; fp32 operands run the true-fp32 kernel
void gemm_dyt(const Tensor& a, const Tensor& b, Tensor& x, const std::vector<Tensor>& n1, const std::vector<Tensor>& n2, Tensor& h,
              const OptTensor& status, int64_t num_sms) {
  const bool f = is_f32(a, "a");
  same_type(b, f, "b"); same_type(h, f, "h"); check_f32(x, "x");
  rows2d(a, "a"); rows2d(b, "b"); rows2d(x, "x"); rows2d(h, "h");
  const int64_t M = a.size(0), K = a.size(1), N = b.size(0);
  TORCH_CHECK(b.size(1) == K && x.size(0) >= M && h.size(0) >= M && x.size(1) == N && h.size(1) == N && N % 8 == 0, "gemm_dyt: shapes");
  TORCH_CHECK(a.stride(0) % 8 == 0 && b.stride(0) % 8 == 0 && x.stride(0) % 8 == 0 && h.stride(0) % 8 == 0 && aligned16(a) && aligned16(b) &&
              aligned16(x) && aligned16(h), "gemm_dyt: pitches / alignment");
  const auto d1 = norm_args(n1, f, N, "gemm_dyt n1"), d2 = norm_args(n2, f, N, "gemm_dyt n2");
  const c10::cuda::CUDAGuard guard(a.device());
  if (f)
    agrpo::launch_gemm_dyt_f32(a.data_ptr<float>(), a.stride(0), b.data_ptr<float>(), b.stride(0), (int)M, (int)N, (int)K, x.data_ptr<float>(),
                               x.stride(0), h.data_ptr<float>(), h.stride(0), d1, d2, cur_stream());
  else
    agrpo::launch_gemm_dyt_bf16(a.data_ptr(), a.stride(0), b.data_ptr(), b.stride(0), (int)M, (int)N, (int)K, x.data_ptr<float>(), x.stride(0),
                                h.data_ptr(), h.stride(0), d1, d2, iptr(status),
                                num_sms > 0 ? (int)num_sms : at::cuda::getCurrentDeviceProperties()->multiProcessorCount, cur_stream());
}

void gemm_f32(const Tensor& a, const Tensor& b, Tensor& d, bool relu2, double softcap, bool accumulate) {
  check_f32(a, "a"); check_f32(b, "b"); check_f32(d, "d");
  rows2d(a, "a"); rows2d(b, "b"); rows2d(d, "d");
  TORCH_CHECK(a.size(1) == b.size(1) && d.size(0) == a.size(0) && d.size(1) == b.size(0), "gemm_f32: shapes");
  const c10::cuda::CUDAGuard guard(a.device());
  agrpo::launch_gemm_f32(a.data_ptr<float>(), a.stride(0), b.data_ptr<float>(), b.stride(0), d.data_ptr<float>(), d.stride(0), (int)a.size(0),
                         (int)b.size(0), (int)a.size(1), cur_stream(), agrpo::GemmF32Post{relu2 ? 1 : 0, (float)softcap, accumulate ? 1 : 0});
}
void gemm_swiglu_f32(const Tensor& a, const Tensor& b, Tensor& d) {
  check_f32(a, "a"); check_f32(b, "b"); check_f32(d, "d");
  rows2d(a, "a"); rows2d(b, "b"); rows2d(d, "d");
  TORCH_CHECK(a.size(1) == b.size(1) && d.size(0) == a.size(0) && b.size(0) == 2 * d.size(1), "gemm_swiglu_f32: shapes");
  const c10::cuda::CUDAGuard guard(a.device());
  agrpo::launch_gemm_swiglu_f32(a.data_ptr<float>(), a.stride(0), b.data_ptr<float>(), b.stride(0), d.data_ptr<float>(), d.stride(0),
                                (int)a.size(0), (int)d.size(1), (int)a.size(1), cur_stream());
}

void sample_logits(const Tensor& logits, double temperature, const Tensor& seeds, Tensor& tokens, const OptTensor& logprobs) {
  check_f32(logits, "logits"); rows2d(logits, "logits"); check_i32(tokens, "tokens");
  const int64_t R = logits.size(0);
  TORCH_CHECK(seeds.is_cuda() && seeds.scalar_type() == torch::kInt64 && seeds.numel() >= R && tokens.numel() >= R, "sample_logits: seeds / tokens");
  if (given(logprobs)) { check_f32(*logprobs, "logprobs"); TORCH_CHECK(logprobs->numel() >= R, "sample_logits: logprobs"); }
  const c10::cuda::CUDAGuard guard(logits.device());
  agrpo::launch_sample_logits(logits.data_ptr<float>(), logits.stride(0), (int)R, (int)logits.size(1), (float)temperature,
                              reinterpret_cast<const unsigned long long*>(seeds.data_ptr<int64_t>()), tokens.data_ptr<int>(),
                              given(logprobs) ? logprobs->data_ptr<float>() : nullptr, cur_stream());
}

}  // namespace

void bind_layer_ops(pybind11::module_& m) {
  namespace py = pybind11;
  using NoGil = py::call_guard<py::gil_scoped_release>;
  m.def("embed_dyt", &embed_dyt, NoGil());
  m.def("short_conv", &short_conv, py::arg("u"), py::arg("w"), py::arg("ring"), py::arg("rows"), py::arg("ring_rows"), py::arg("seq_lens"),
        py::arg("block_tables"), py::arg("q_out"), py::arg("k_cache"), py::arg("status"), NoGil());
  m.def("window_attn", &window_attn, py::arg("q"), py::arg("k_cache"), py::arg("rows"), py::arg("seq_lens"), py::arg("block_tables"),
        py::arg("bias"), py::arg("qscale"), py::arg("talk"), py::arg("gate"), py::arg("window"), py::arg("out"), py::arg("status"), NoGil());
  m.def("talk_attn_prefill", &talk_attn_prefill, py::arg("q"), py::arg("k_cache"), py::arg("tiles"), py::arg("pages"), py::arg("keys"), py::arg("block_tables"), py::arg("bias"),
        py::arg("qscale"), py::arg("talk"), py::arg("gate"), py::arg("window"), py::arg("acc"), py::arg("out"), py::arg("status"), NoGil());
  m.def("talk_attn_decode", &talk_attn_decode, py::arg("u"), py::arg("conv_w"), py::arg("ring"), py::arg("k_cache"), py::arg("seq_lens"),
        py::arg("block_tables"), py::arg("bias"), py::arg("qscale"), py::arg("talk"), py::arg("gate"), py::arg("window"), py::arg("out"),
        py::arg("splits"), py::arg("part_o"), py::arg("part_ml"), py::arg("tickets"), py::arg("status"), NoGil());
  m.def("talk_decode_ctas_per_sm", &agrpo::talk_decode_ctas_per_sm);
  m.def("gemm_dyt", &gemm_dyt, py::arg("a"), py::arg("b"), py::arg("x"), py::arg("n1"), py::arg("n2"), py::arg("h"), py::arg("status"),
        py::arg("num_sms") = 0, NoGil());
  m.def("gemm_f32", &gemm_f32, py::arg("a"), py::arg("b"), py::arg("d"), py::arg("relu2") = false, py::arg("softcap") = 0.0,
        py::arg("accumulate") = false, NoGil());
  m.def("gemm_swiglu_f32", &gemm_swiglu_f32, NoGil());
  m.def("sample_logits", &sample_logits, py::arg("logits"), py::arg("temperature"), py::arg("seeds"), py::arg("tokens"),
        py::arg("logprobs") = py::none(), NoGil());
}
