// Python bindings of the hybrid attention / scan kernels (launchers_hybrid.h).
#include "bindings_layers.h"

#include <ATen/cuda/CUDAContext.h>
#include <c10/cuda/CUDAGuard.h>
#include <pybind11/stl.h>

#include "launchers.h"
#include "launchers_hybrid.h"

namespace {

using torch::Tensor;
using OptTensor = c10::optional<torch::Tensor>;

inline cudaStream_t cur_stream() { return at::cuda::getCurrentCUDAStream(); }
inline int sms() { return at::cuda::getCurrentDeviceProperties()->multiProcessorCount; }
inline bool is_f32(const Tensor& t, const char* name) {
  TORCH_CHECK(t.is_cuda() && (t.scalar_type() == torch::kFloat32 || t.scalar_type() == torch::kBFloat16), name, ": fp32 or bf16 CUDA tensor");
  return t.scalar_type() == torch::kFloat32;
}
inline void same_type(const Tensor& t, bool fp32, const char* name) {
  TORCH_CHECK(t.is_cuda() && t.scalar_type() == (fp32 ? torch::kFloat32 : torch::kBFloat16), name, ": dtype of the activations expected");
}
inline void check_f32(const Tensor& t, const char* name) { TORCH_CHECK(t.is_cuda() && t.scalar_type() == torch::kFloat32, name, ": fp32"); }
inline void check_i32(const Tensor& t, const char* name) { TORCH_CHECK(t.is_cuda() && t.scalar_type() == torch::kInt32, name, ": int32"); }
inline void check_i64(const Tensor& t, const char* name) { TORCH_CHECK(t.is_cuda() && t.scalar_type() == torch::kInt64, name, ": int64"); }
inline bool given(const OptTensor& t) { return t.has_value() && t->defined(); }
inline int* iptr(const OptTensor& t) { return given(t) ? t->data_ptr<int>() : nullptr; }
inline bool aligned16(const Tensor& t) { return (reinterpret_cast<uintptr_t>(t.data_ptr()) & 15) == 0; }
// 2-D matrix with contiguous rows whose starts are aligned for vector accesses
inline void mat(const Tensor& t, const char* name) {
  TORCH_CHECK(t.dim() == 2 && t.stride(1) == 1 && t.stride(0) % 8 == 0 && aligned16(t), name, ": 2-D, contiguous aligned rows");
}
inline long long* fixed(const OptTensor& t, int64_t n, const char* name) {
  if (!given(t)) return nullptr;
  check_i64(*t, name);
  TORCH_CHECK(t->is_contiguous() && t->numel() >= n, name, ": one entry per row");
  return reinterpret_cast<long long*>(t->data_ptr<int64_t>());
}

agrpo::NormOut norm_out(const OptTensor& h, const OptTensor& w, bool fp32, int64_t rows, int64_t W, const char* name) {
  agrpo::NormOut o{nullptr, 0, nullptr};
  if (!given(h)) return o;
  same_type(*h, fp32, name);
  mat(*h, name);
  TORCH_CHECK(h->size(0) >= rows && h->size(1) == W, name, ": [rows, width]");
  o.h = h->data_ptr();
  o.ld = h->stride(0);
  if (given(w)) {
    same_type(*w, fp32, name);
    TORCH_CHECK(w->numel() == W && w->is_contiguous() && aligned16(*w), name, ": norm weight [width]");
    o.w = w->data_ptr();
  }
  return o;
}

void embed_norm(const Tensor& ids, const Tensor& table, double scale, Tensor& x, const OptTensor& copy, const OptTensor& h1, const OptTensor& w1,
                const OptTensor& h2, const OptTensor& w2, const OptTensor& ss) {
  const bool f = is_f32(table, "table");
  check_i32(ids, "ids"); check_f32(x, "x"); mat(x, "x"); mat(table, "table");
  const int64_t T = ids.numel(), W = table.size(1);
  TORCH_CHECK(table.is_contiguous() && x.is_contiguous() && x.size(0) >= T && x.size(1) == W && W % 8 == 0, "embed_norm: shapes");
  agrpo::EmbedArgs a{};
  a.ids = ids.data_ptr<int>(); a.table = table.data_ptr(); a.scale = (float)scale; a.x = x.data_ptr<float>();
  const agrpo::NormOut c = norm_out(copy, OptTensor(), f, T, W, "embed_norm copy");
  a.copy = c.h; a.ld_copy = c.ld;
  a.out[0] = norm_out(h1, w1, f, T, W, "embed_norm h1");
  a.out[1] = norm_out(h2, w2, f, T, W, "embed_norm h2");
  if (given(ss)) {
    check_i64(*ss, "ss");
    TORCH_CHECK(ss->dim() == 2 && ss->is_contiguous() && ss->size(1) >= T, "embed_norm: ss [stats, rows]");
    a.ss = reinterpret_cast<long long*>(ss->data_ptr<int64_t>());
    a.n_stats = (int)ss->size(0); a.ss_pitch = ss->size(1);
  }
  a.T = (int)T; a.W = (int)W; a.V = (int)table.size(0);
  const c10::cuda::CUDAGuard guard(table.device());
  agrpo::launch_embed_norm(f, a, cur_stream());
}

void rms_rows(const Tensor& x, double eps, int64_t width, Tensor& h1, const OptTensor& w1, const OptTensor& h2, const OptTensor& w2) {
  check_f32(x, "x"); mat(x, "x");
  const bool f = is_f32(h1, "h1");
  const int64_t T = x.size(0), W = x.size(1);
  TORCH_CHECK(W % 8 == 0 && width >= 1 && width <= W, "rms_rows: width");
  const agrpo::NormOut out[2] = {norm_out(h1, w1, f, T, W, "rms_rows h1"), norm_out(h2, w2, f, T, W, "rms_rows h2")};
  const c10::cuda::CUDAGuard guard(x.device());
  agrpo::launch_rms_rows(f, x.data_ptr<float>(), x.stride(0), out, (float)eps, (int)width, (int)T, (int)W, cur_stream());
}

void softcap_rows(Tensor& z, double cap) {
  check_f32(z, "z");
  TORCH_CHECK(z.dim() == 2 && z.stride(1) == 1, "softcap_rows: 2-D");
  const c10::cuda::CUDAGuard guard(z.device());
  agrpo::launch_softcap_rows(z.data_ptr<float>(), z.stride(0), (int)z.size(0), (int)z.size(1), (float)cap, cur_stream());
}

void conv_silu(const Tensor& u, const Tensor& w, const Tensor& bias, Tensor& ring, const OptTensor& rows, const OptTensor& ring_rows,
               const OptTensor& seq_lens, Tensor& out, const OptTensor& status) {
  const bool f = is_f32(u, "u");
  same_type(w, f, "conv w"); same_type(bias, f, "conv bias"); same_type(ring, f, "ring"); same_type(out, f, "out");
  mat(u, "u"); mat(out, "out");
  agrpo::ShortConvArgs a{};
  const int64_t C = out.size(1), T = u.size(0);
  TORCH_CHECK(C % 8 == 0 && u.size(1) >= C && out.is_contiguous() && out.size(0) >= T, "conv_silu: u / out");
  TORCH_CHECK(w.dim() == 2 && w.size(1) == C && w.is_contiguous() && aligned16(w) && bias.numel() == C && bias.is_contiguous() && aligned16(bias), "conv_silu: w, bias");
  TORCH_CHECK(ring.dim() == 3 && ring.size(2) == C && ring.size(1) >= w.size(0) && ring.stride(2) == 1 && ring.stride(1) == C && ring.stride(0) % 8 == 0 && aligned16(ring),
              "conv_silu: ring [slots, >= taps, channels]");
  if (given(rows)) {
    check_i32(*rows, "rows");
    TORCH_CHECK(rows->is_contiguous() && rows->numel() >= 4 * T && given(ring_rows) && ring_rows->is_contiguous(), "conv_silu: rows [T, 4] with ring_rows");
    check_i32(*ring_rows, "ring_rows");
  } else {
    TORCH_CHECK(given(seq_lens), "conv_silu: rows or seq_lens");
    check_i32(*seq_lens, "seq_lens");
    TORCH_CHECK(seq_lens->numel() >= T && ring.size(0) >= T, "conv_silu: decode rows");
  }
  a.u = u.data_ptr(); a.ldu = u.stride(0);
  a.w = w.data_ptr(); a.taps = (int)w.size(0);
  a.ring = ring.data_ptr(); a.ring_len = (int)ring.size(1); a.ring_pitch = ring.stride(0);
  a.rows = iptr(rows); a.seq_lens = iptr(seq_lens);
  a.q_out = out.data_ptr(); a.q_cols = (int)C; a.k_cols = 0; a.D = 8;
  a.T = (int)T; a.status = iptr(status);
  a.bias = bias.data_ptr(); a.silu = 1;
  const c10::cuda::CUDAGuard guard(u.device());
  if (!given(rows)) return agrpo::launch_short_conv_decode(f, a, cur_stream());
  agrpo::launch_short_conv(f, a, cur_stream());
  agrpo::launch_short_conv_ring(f, a, ring_rows->data_ptr<int>(), (int)ring_rows->numel(), cur_stream());
}

agrpo::QkRopeArgs qk_args(const Tensor& u, const Tensor& qn, const Tensor& kn, double eps, int64_t dim, const Tensor& cos_t, const Tensor& sin_t,
                          const OptTensor& ss_q, const OptTensor& ss_k, const OptTensor& rows, const OptTensor& seq_lens, const Tensor& tables,
                          Tensor& k_cache, Tensor& v_cache, const OptTensor& status) {
  const bool f = is_f32(u, "u");
  same_type(qn, f, "q norm"); same_type(kn, f, "k norm"); same_type(k_cache, f, "k_cache"); same_type(v_cache, f, "v_cache");
  mat(u, "u"); check_f32(cos_t, "cos"); check_f32(sin_t, "sin"); check_i32(tables, "block_tables");
  TORCH_CHECK(k_cache.dim() == 4 && v_cache.dim() == 4 && k_cache.is_contiguous() && v_cache.is_contiguous() && k_cache.size(3) % 8 == 0 &&
              v_cache.size(3) % 8 == 0 && aligned16(k_cache) && aligned16(v_cache), "qk: caches [blocks, G, bs, D]");
  TORCH_CHECK(k_cache.size(0) == v_cache.size(0) && k_cache.size(1) == v_cache.size(1) && k_cache.size(2) == v_cache.size(2), "qk: caches agree");
  agrpo::QkRopeArgs a{};
  a.G = (int)k_cache.size(1); a.D = (int)k_cache.size(3); a.E = (int)v_cache.size(3);
  TORCH_CHECK(qn.numel() % a.D == 0 && kn.numel() == (int64_t)a.G * a.D && qn.is_contiguous() && kn.is_contiguous() && aligned16(qn) && aligned16(kn), "qk: norm weights");
  a.H = (int)(qn.numel() / a.D);
  const int64_t T = u.size(0);
  TORCH_CHECK(u.size(1) >= (int64_t)(a.H + a.G) * a.D + (int64_t)a.G * a.E && dim >= 1 && dim <= a.D, "qk: u [T, q | k | v]");
  TORCH_CHECK(cos_t.dim() == 2 && cos_t.is_contiguous() && sin_t.is_contiguous() && sin_t.sizes() == cos_t.sizes() && 2 * cos_t.size(1) <= dim, "qk: tables [positions, rot / 2]");
  TORCH_CHECK(tables.dim() == 2 && tables.is_contiguous(), "qk: block tables");
  if (given(rows)) { check_i32(*rows, "rows"); TORCH_CHECK(rows->is_contiguous() && rows->numel() >= 4 * T, "qk: rows [T, 4]"); }
  else { TORCH_CHECK(given(seq_lens), "qk: rows or seq_lens"); }
  if (given(seq_lens)) { check_i32(*seq_lens, "seq_lens"); TORCH_CHECK(given(rows) || (seq_lens->numel() >= T && tables.size(0) >= T), "qk: decode rows"); }
  TORCH_CHECK(given(ss_q) == given(ss_k), "qk: both sums or none");
  a.u = u.data_ptr(); a.ldu = u.stride(0);
  a.q_norm = qn.data_ptr(); a.k_norm = kn.data_ptr(); a.eps = (float)eps;
  a.ss_q = fixed(ss_q, T, "ss_q"); a.ss_k = fixed(ss_k, T, "ss_k");
  a.cos_t = cos_t.data_ptr<float>(); a.sin_t = sin_t.data_ptr<float>(); a.max_pos = (int)cos_t.size(0);
  a.rows = iptr(rows); a.seq_lens = given(rows) ? nullptr : iptr(seq_lens);
  a.block_tables = tables.data_ptr<int>(); a.max_blocks = (int)tables.size(1);
  a.k_cache = k_cache.data_ptr(); a.v_cache = v_cache.data_ptr();
  a.dim = (int)dim; a.rot = (int)(2 * cos_t.size(1));
  a.block_size = (int)k_cache.size(2); a.num_cache_blocks = (int)k_cache.size(0);
  a.T = (int)T; a.status = iptr(status);
  return a;
}

void qk_norm_rope(Tensor& u, const Tensor& qn, const Tensor& kn, double eps, int64_t dim, const Tensor& cos_t, const Tensor& sin_t, const OptTensor& ss_q,
                  const OptTensor& ss_k, const OptTensor& rows, const OptTensor& seq_lens, const Tensor& tables, Tensor& k_cache, Tensor& v_cache,
                  const OptTensor& status) {
  const agrpo::QkRopeArgs a = qk_args(u, qn, kn, eps, dim, cos_t, sin_t, ss_q, ss_k, rows, seq_lens, tables, k_cache, v_cache, status);
  const c10::cuda::CUDAGuard guard(u.device());
  agrpo::launch_qk_norm_rope(u.scalar_type() == torch::kFloat32, a, cur_stream());
}

agrpo::ChunkAttnArgs chunk_args(const OptTensor& q, const Tensor& k_cache, const Tensor& v_cache, const OptTensor& rows, const OptTensor& seq_lens,
                                const Tensor& tables, double scale, double softcap, int64_t chunk, Tensor& out, const OptTensor& status) {
  const bool f = is_f32(k_cache, "k_cache");
  same_type(v_cache, f, "v_cache"); same_type(out, f, "out"); check_i32(tables, "block_tables"); mat(out, "out");
  TORCH_CHECK(k_cache.dim() == 4 && v_cache.dim() == 4 && k_cache.is_contiguous() && v_cache.is_contiguous() && k_cache.size(3) % 8 == 0 &&
              v_cache.size(3) % 8 == 0 && aligned16(k_cache) && aligned16(v_cache) && k_cache.size(0) == v_cache.size(0) &&
              k_cache.size(1) == v_cache.size(1) && k_cache.size(2) == v_cache.size(2), "chunk_attn: caches [blocks, G, bs, D]");
  agrpo::ChunkAttnArgs a{};
  a.G = (int)k_cache.size(1); a.D = (int)k_cache.size(3); a.E = (int)v_cache.size(3);
  TORCH_CHECK(out.size(1) % a.E == 0 && (out.size(1) / a.E) % a.G == 0, "chunk_attn: out [T, H * E]");
  a.H = (int)(out.size(1) / a.E);
  a.T = (int)out.size(0);
  if (given(q)) {
    same_type(*q, f, "q"); mat(*q, "q");
    TORCH_CHECK(q->size(1) >= (int64_t)a.H * a.D && q->size(0) >= a.T, "chunk_attn: q [T, >= H * D]");
    a.q = q->data_ptr(); a.ldq = q->stride(0);
  }
  TORCH_CHECK(chunk >= 1 && softcap >= 0, "chunk_attn: chunk / cap");
  TORCH_CHECK(tables.dim() == 2 && tables.is_contiguous(), "chunk_attn: tables");
  if (given(rows)) { check_i32(*rows, "rows"); TORCH_CHECK(rows->is_contiguous() && rows->numel() >= 4 * a.T, "chunk_attn: rows [T, 4]"); }
  else if (given(seq_lens)) { check_i32(*seq_lens, "seq_lens"); TORCH_CHECK(seq_lens->numel() >= a.T && tables.size(0) >= a.T, "chunk_attn: decode rows"); }
  a.k_cache = k_cache.data_ptr(); a.v_cache = v_cache.data_ptr();
  a.rows = iptr(rows); a.seq_lens = iptr(seq_lens);
  a.block_tables = tables.data_ptr<int>(); a.max_blocks = (int)tables.size(1);
  a.scale = (float)scale; a.softcap = (float)softcap;
  a.chunk = (int)std::min<int64_t>(chunk, 1 << 30);
  a.out = out.data_ptr(); a.ldo = out.stride(0);
  a.block_size = (int)k_cache.size(2); a.num_cache_blocks = (int)k_cache.size(0);
  a.status = iptr(status);
  return a;
}

void chunk_attn(const Tensor& q, const Tensor& k_cache, const Tensor& v_cache, const OptTensor& rows, const OptTensor& seq_lens, const Tensor& tables,
                double scale, double softcap, int64_t chunk, Tensor& out, const OptTensor& status) {
  TORCH_CHECK(given(rows) || given(seq_lens), "chunk_attn: rows or seq_lens");
  const agrpo::ChunkAttnArgs a = chunk_args(q, k_cache, v_cache, rows, seq_lens, tables, scale, softcap, chunk, out, status);
  const c10::cuda::CUDAGuard guard(q.device());
  agrpo::launch_chunk_attn(q.scalar_type() == torch::kFloat32, a, cur_stream());
}

// Tensor-core form for prompts; false (nothing launched) when the shape is not served.
bool chunk_attn_prefill(const Tensor& q, const Tensor& k_cache, const Tensor& v_cache, const Tensor& tiles, const Tensor& pages, Tensor& keys,
                        Tensor& values, const Tensor& tables, double scale, double softcap, int64_t chunk, Tensor& out, const OptTensor& status) {
  if (k_cache.scalar_type() != torch::kBFloat16 || k_cache.size(2) != 16) return false;
  check_i32(tiles, "tiles"); check_i32(pages, "pages"); same_type(keys, false, "keys"); same_type(values, false, "values");
  TORCH_CHECK(tiles.dim() == 2 && tiles.size(1) == 4 && tiles.is_contiguous() && aligned16(tiles), "chunk_attn_prefill: tiles [n, 4]");
  TORCH_CHECK(pages.dim() == 2 && pages.size(1) == 2 && pages.is_contiguous() && (reinterpret_cast<uintptr_t>(pages.data_ptr()) & 7) == 0, "chunk_attn_prefill: pages [n, 2]");
  const int64_t n = pages.size(0) * 16 * k_cache.size(1);
  TORCH_CHECK(keys.is_contiguous() && values.is_contiguous() && aligned16(keys) && aligned16(values) && keys.numel() >= n * k_cache.size(3) &&
              values.numel() >= n * v_cache.size(3), "chunk_attn_prefill: keys, values [16 pages, G * D]");
  const agrpo::ChunkAttnArgs a = chunk_args(q, k_cache, v_cache, OptTensor(), OptTensor(), tables, scale, softcap, chunk, out, status);
  const c10::cuda::CUDAGuard guard(q.device());
  return agrpo::launch_chunk_attn_prefill(a, (int)q.size(1), tiles.data_ptr<int>(), (int)tiles.size(0), pages.data_ptr<int>(), (int)pages.size(0),
                                          keys.data_ptr(), values.data_ptr(), cur_stream());
}

// Decode step of the mixer after its projection u = [q | k | v]: norms, rotation, cache write, attention.
void chunk_attn_decode(const Tensor& u, const Tensor& qn, const Tensor& kn, double eps, int64_t dim, const Tensor& cos_t, const Tensor& sin_t,
                       const Tensor& ss_q, const Tensor& ss_k, const Tensor& seq_lens, const Tensor& tables, Tensor& k_cache, Tensor& v_cache,
                       double scale, double softcap, int64_t chunk, Tensor& out, int64_t splits, Tensor& part_o, Tensor& part_ml, Tensor& tickets,
                       const OptTensor& status) {
  TORCH_CHECK(k_cache.scalar_type() == torch::kBFloat16 && k_cache.size(2) == 16, "chunk_attn_decode: bf16, pages of 16");
  agrpo::ChunkDecodeArgs d{};
  d.qk = qk_args(u, qn, kn, eps, dim, cos_t, sin_t, ss_q, ss_k, OptTensor(), seq_lens, tables, k_cache, v_cache, status);
  d.at = chunk_args(OptTensor(), k_cache, v_cache, OptTensor(), seq_lens, tables, scale, softcap, chunk, out, status);
  TORCH_CHECK(d.at.H == d.qk.H && d.at.T <= d.qk.T, "chunk_attn_decode: out [B, H * E]");
  TORCH_CHECK(agrpo::chunk_decode_serves(d.at.H, d.at.G, d.at.D, d.at.E), "chunk_attn_decode: head sizes 64 or 128");
  TORCH_CHECK(splits >= 1 && splits <= 8, "chunk_attn_decode: 1 to 8 splits");
  check_f32(part_o, "part_o"); check_f32(part_ml, "part_ml"); check_i32(tickets, "tickets");
  const int64_t n = (int64_t)d.at.T * d.at.H;
  TORCH_CHECK(splits == 1 || (part_o.numel() >= n * splits * d.at.E && part_ml.numel() >= n * splits * 2 && tickets.numel() >= n), "chunk_attn_decode: scratch");
  d.splits = (int)splits;
  d.part_o = part_o.data_ptr<float>(); d.part_ml = part_ml.data_ptr<float>(); d.tickets = tickets.data_ptr<int>();
  const c10::cuda::CUDAGuard guard(u.device());
  agrpo::launch_chunk_attn_decode(d, cur_stream());
}

agrpo::ScanArgs scan_args(const Tensor& xc, const Tensor& r, const Tensor& z, const Tensor& wdt, int64_t rank, const Tensor& dt_b, const Tensor& a_,
                          const Tensor& d_, Tensor& state, const OptTensor& segs, const OptTensor& seq_lens, Tensor& out) {
  const bool f = is_f32(xc, "xc");
  same_type(z, f, "z"); same_type(wdt, f, "wdt"); same_type(out, f, "out");
  check_f32(r, "r"); check_f32(dt_b, "dt_b"); check_f32(a_, "a"); check_f32(d_, "d"); check_f32(state, "state");
  mat(xc, "xc"); mat(r, "r"); mat(z, "z"); mat(wdt, "wdt"); mat(out, "out");
  agrpo::ScanArgs a{};
  a.T = (int)xc.size(0); a.C = (int)xc.size(1); a.N = (int)a_.size(1); a.rank = (int)rank;
  TORCH_CHECK(a_.dim() == 2 && a_.is_contiguous() && a_.size(0) == a.C && dt_b.numel() == a.C && d_.numel() == a.C && wdt.size(0) == a.C, "scan: channels");
  TORCH_CHECK(z.size(0) >= a.T && z.size(1) >= a.C && out.size(0) >= a.T && out.size(1) >= a.C && r.size(0) >= a.T, "scan: rows");
  TORCH_CHECK(state.dim() == 3 && state.size(1) == a.C && state.size(2) == a.N && state.stride(2) == 1 && state.stride(1) == a.N, "scan: state [slots, C, N]");
  if (given(segs)) { check_i32(*segs, "segs"); TORCH_CHECK(segs->dim() == 2 && segs->size(1) == 4 && segs->is_contiguous() && aligned16(*segs), "scan: segs [n, 4]");
                     a.segs = segs->data_ptr<int>(); a.n_segs = (int)segs->size(0); }
  else { TORCH_CHECK(given(seq_lens), "scan: segs or seq_lens"); check_i32(*seq_lens, "seq_lens");
         TORCH_CHECK(seq_lens->numel() >= a.T && state.size(0) >= a.T, "scan: decode rows"); a.seq_lens = seq_lens->data_ptr<int>(); }
  a.xc = xc.data_ptr(); a.ldx = xc.stride(0);
  a.r = r.data_ptr<float>(); a.ldr = r.stride(0);
  a.z = z.data_ptr(); a.ldz = z.stride(0);
  a.wdt = wdt.data_ptr(); a.ldw = wdt.stride(0);
  a.dt_b = dt_b.data_ptr<float>(); a.a = a_.data_ptr<float>(); a.d = d_.data_ptr<float>();
  a.state = state.data_ptr<float>(); a.state_pitch = state.stride(0);
  a.out = out.data_ptr(); a.ldo = out.stride(0);
  return a;
}

void selective_scan_plain(const Tensor& xc, const Tensor& r, const Tensor& z, const Tensor& wdt, int64_t rank, const Tensor& dt_b, const Tensor& a_,
                          const Tensor& d_, Tensor& state, const OptTensor& segs, const OptTensor& seq_lens, Tensor& out) {
  const agrpo::ScanArgs a = scan_args(xc, r, z, wdt, rank, dt_b, a_, d_, state, segs, seq_lens, out);
  TORCH_CHECK(r.size(1) >= rank + 2 * a.N && wdt.size(1) >= rank, "scan: r [T, rank | B | C]");
  const c10::cuda::CUDAGuard guard(xc.device());
  agrpo::launch_selective_scan_plain(xc.scalar_type() == torch::kFloat32, a, cur_stream());
}

// Packed form (bf16): step-size code by itself, r = B and C by quarters; A in log2 units and the state have
// 4 * scan_states_per_lane(N) entries per channel.
void selective_scan(const Tensor& xc, const Tensor& code, const Tensor& r, const Tensor& z, const Tensor& wdt, int64_t rank, const Tensor& dt_b,
                    const Tensor& a_, const Tensor& d_, Tensor& state, const OptTensor& segs, const OptTensor& seq_lens, Tensor& out) {
  TORCH_CHECK(xc.scalar_type() == torch::kBFloat16, "selective_scan: bf16");
  agrpo::ScanArgs a = scan_args(xc, r, z, wdt, rank, dt_b, a_, d_, state, segs, seq_lens, out);
  same_type(code, false, "code"); mat(code, "code");
  const int64_t rank_p = (rank + 15) / 16 * 16;
  TORCH_CHECK(4 * agrpo::scan_states_per_lane(a.N) == a.N && agrpo::selective_scan_serves(a.N, a.rank), "selective_scan: states");
  TORCH_CHECK(code.size(0) >= a.T && code.size(1) == rank_p && code.stride(0) == agrpo::scan_code_pitch(a.rank) && r.size(1) == 2 * a.N && r.is_contiguous() && wdt.size(1) >= rank_p && a.C % 32 == 0 &&
              state.stride(0) % 4 == 0 && aligned16(state) && aligned16(a_), "selective_scan: packed layout");
  a.code = code.data_ptr(); a.ldcode = code.stride(0);
  const c10::cuda::CUDAGuard guard(xc.device());
  TORCH_CHECK(agrpo::launch_selective_scan(a, cur_stream()), "selective_scan: shape not served");
}

void gemm_split_store(const Tensor& a_, const Tensor& w, Tensor& d16, Tensor& d32, const OptTensor& status) {
  same_type(a_, false, "a"); same_type(w, false, "w"); same_type(d16, false, "d16"); check_f32(d32, "d32");
  mat(a_, "a"); mat(w, "w"); mat(d16, "d16"); mat(d32, "d32");
  agrpo::SplitStoreArgs a{};
  a.M = (int)a_.size(0); a.K = (int)w.size(1); a.n1 = (int)d16.size(1); a.n2 = (int)d32.size(1);
  TORCH_CHECK(a_.size(1) == a.K && a.K % 8 == 0 && a.n1 % 8 == 0 && a.n2 % 8 == 0 && w.size(0) == a.n1 + a.n2 && d16.size(0) >= a.M && d32.size(0) >= a.M,
              "gemm_split_store: shapes");
  a.a = a_.data_ptr(); a.lda = a_.stride(0); a.w = w.data_ptr(); a.ldw = w.stride(0);
  a.d16 = d16.data_ptr(); a.ld16 = d16.stride(0); a.d32 = d32.data_ptr<float>(); a.ld32 = d32.stride(0);
  a.status = iptr(status);
  const c10::cuda::CUDAGuard guard(a_.device());
  agrpo::launch_gemm_split_store(a, sms(), cur_stream());
}

void gemm_parallel_proj(const Tensor& h, const Tensor& w, Tensor& u, const OptTensor& act, const OptTensor& ss_in, int64_t width, double eps,
                        const OptTensor& ss_q, const OptTensor& ss_k, int64_t q_end, int64_t k_end, const OptTensor& status) {
  same_type(h, false, "h"); same_type(w, false, "w"); same_type(u, false, "u");
  mat(h, "h"); mat(w, "w"); mat(u, "u");
  agrpo::ParallelProjArgs a{};
  a.M = (int)h.size(0); a.K = (int)w.size(1); a.n1 = (int)u.size(1); a.n2 = (int)w.size(0) - a.n1;
  a.a2 = a.K;
  TORCH_CHECK(a.K % 8 == 0 && a.n1 % 8 == 0 && a.n2 >= 0 && a.n2 % 8 == 0 && u.size(0) >= a.M && h.size(1) >= (a.n2 > 0 ? 2 : 1) * (int64_t)a.K, "parallel_proj: shapes");
  TORCH_CHECK((a.n2 > 0) == given(act), "parallel_proj: act goes with further rows of w");
  if (given(act)) {
    same_type(*act, false, "act"); mat(*act, "act");
    TORCH_CHECK(act->size(0) >= a.M && act->size(1) == a.n2, "parallel_proj: act [M, n2]");
    a.act = act->data_ptr(); a.ldact = act->stride(0);
  }
  TORCH_CHECK(given(ss_q) == given(ss_k) && q_end % 8 == 0 && k_end % 8 == 0 && 0 <= q_end && q_end <= k_end && k_end <= a.n1, "parallel_proj: statistics");
  a.h = h.data_ptr(); a.lda = h.stride(0); a.w = w.data_ptr(); a.ldw = w.stride(0);
  a.u = u.data_ptr(); a.ldu = u.stride(0);
  a.ss_in = fixed(ss_in, a.M, "ss_in"); a.width = (int)width; a.eps = (float)eps;
  a.ss_q = fixed(ss_q, a.M, "ss_q"); a.ss_k = fixed(ss_k, a.M, "ss_k"); a.q_end = (int)q_end; a.k_end = (int)k_end;
  a.status = iptr(status);
  const c10::cuda::CUDAGuard guard(h.device());
  agrpo::launch_gemm_parallel_proj(a, sms(), cur_stream());
}

void gemm_residual(const Tensor& a_, const Tensor& w, Tensor& x, bool accumulate, const OptTensor& h1, const OptTensor& w1, const OptTensor& h2,
                   const OptTensor& w2, const OptTensor& ss, const OptTensor& status) {
  same_type(a_, false, "a"); same_type(w, false, "w"); check_f32(x, "x");
  mat(a_, "a"); mat(w, "w"); mat(x, "x");
  agrpo::ResidualArgs a{};
  a.M = (int)a_.size(0); a.N = (int)w.size(0); a.K = (int)w.size(1);
  TORCH_CHECK(a_.size(1) == a.K && a.K % 8 == 0 && a.N % 8 == 0 && x.size(0) >= a.M && x.size(1) == a.N, "residual: shapes");
  a.a = a_.data_ptr(); a.lda = a_.stride(0); a.w = w.data_ptr(); a.ldw = w.stride(0);
  a.x = x.data_ptr<float>(); a.ldx = x.stride(0); a.accumulate = accumulate ? 1 : 0;
  a.out[0] = norm_out(h1, w1, false, a.M, a.N, "residual h1");
  a.out[1] = norm_out(h2, w2, false, a.M, a.N, "residual h2");
  a.ss = fixed(ss, a.M, "ss"); a.status = iptr(status);
  const c10::cuda::CUDAGuard guard(a_.device());
  agrpo::launch_gemm_residual(a, sms(), cur_stream());
}

}  // namespace

void bind_hybrid_ops(pybind11::module_& m) {
  namespace py = pybind11;
  using NoGil = py::call_guard<py::gil_scoped_release>;
  m.def("embed_norm", &embed_norm, py::arg("ids"), py::arg("table"), py::arg("scale"), py::arg("x"), py::arg("copy"), py::arg("h1"), py::arg("w1"),
        py::arg("h2"), py::arg("w2"), py::arg("ss"), NoGil());
  m.def("rms_rows", &rms_rows, py::arg("x"), py::arg("eps"), py::arg("width"), py::arg("h1"), py::arg("w1"), py::arg("h2") = py::none(),
        py::arg("w2") = py::none(), NoGil());
  m.def("softcap_rows", &softcap_rows, NoGil());
  m.def("conv_silu", &conv_silu, py::arg("u"), py::arg("w"), py::arg("bias"), py::arg("ring"), py::arg("rows"), py::arg("ring_rows"),
        py::arg("seq_lens"), py::arg("out"), py::arg("status"), NoGil());
  m.def("qk_norm_rope", &qk_norm_rope, py::arg("u"), py::arg("q_norm"), py::arg("k_norm"), py::arg("eps"), py::arg("dim"), py::arg("cos"), py::arg("sin"),
        py::arg("ss_q"), py::arg("ss_k"), py::arg("rows"), py::arg("seq_lens"), py::arg("block_tables"), py::arg("k_cache"), py::arg("v_cache"),
        py::arg("status"), NoGil());
  m.def("chunk_attn", &chunk_attn, py::arg("q"), py::arg("k_cache"), py::arg("v_cache"), py::arg("rows"), py::arg("seq_lens"), py::arg("block_tables"),
        py::arg("scale"), py::arg("softcap"), py::arg("chunk"), py::arg("out"), py::arg("status"), NoGil());
  m.def("chunk_attn_prefill", &chunk_attn_prefill, py::arg("q"), py::arg("k_cache"), py::arg("v_cache"), py::arg("tiles"), py::arg("pages"), py::arg("keys"),
        py::arg("values"), py::arg("block_tables"), py::arg("scale"), py::arg("softcap"), py::arg("chunk"), py::arg("out"), py::arg("status"), NoGil());
  m.def("chunk_attn_decode", &chunk_attn_decode, py::arg("u"), py::arg("q_norm"), py::arg("k_norm"), py::arg("eps"), py::arg("dim"), py::arg("cos"),
        py::arg("sin"), py::arg("ss_q"), py::arg("ss_k"), py::arg("seq_lens"), py::arg("block_tables"), py::arg("k_cache"), py::arg("v_cache"),
        py::arg("scale"), py::arg("softcap"), py::arg("chunk"), py::arg("out"), py::arg("splits"), py::arg("part_o"), py::arg("part_ml"),
        py::arg("tickets"), py::arg("status"), NoGil());
  m.def("chunk_decode_serves", &agrpo::chunk_decode_serves);
  m.def("scan_states_per_lane", &agrpo::scan_states_per_lane);
  m.def("scan_code_pitch", &agrpo::scan_code_pitch);
  m.def("selective_scan_serves", &agrpo::selective_scan_serves);
  m.def("selective_scan_plain", &selective_scan_plain, py::arg("xc"), py::arg("r"), py::arg("z"), py::arg("wdt"), py::arg("rank"), py::arg("dt_b"),
        py::arg("a"), py::arg("d"), py::arg("state"), py::arg("segs"), py::arg("seq_lens"), py::arg("out"), NoGil());
  m.def("gemm_split_store", &gemm_split_store, py::arg("a"), py::arg("w"), py::arg("d16"), py::arg("d32"), py::arg("status"), NoGil());
  m.def("selective_scan", &selective_scan, py::arg("xc"), py::arg("code"), py::arg("r"), py::arg("z"), py::arg("wdt"), py::arg("rank"), py::arg("dt_b"), py::arg("a"),
        py::arg("d"), py::arg("state"), py::arg("segs"), py::arg("seq_lens"), py::arg("out"), NoGil());
  m.def("gemm_parallel_proj", &gemm_parallel_proj, py::arg("h"), py::arg("w"), py::arg("u"), py::arg("act"), py::arg("ss_in"), py::arg("width"),
        py::arg("eps"), py::arg("ss_q"), py::arg("ss_k"), py::arg("q_end"), py::arg("k_end"), py::arg("status"), NoGil());
  m.def("gemm_residual", &gemm_residual, py::arg("a"), py::arg("w"), py::arg("x"), py::arg("accumulate"), py::arg("h1"), py::arg("w1"), py::arg("h2"),
        py::arg("w2"), py::arg("ss"), py::arg("status"), NoGil());
}
