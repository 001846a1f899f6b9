// Python binding of the kernels that serve layer-list models (kernels/hybrid_api.h), a module of its
// own (mythos_b200._H) so that serving such a model needs a fraction of the library's sources compiled.
#include "binding_sampler.h"
#include "kernels/api.h"
#include "kernels/host_util.h"
#include "kernels/hybrid_api.h"

namespace {

bool is_f32(const Tensor& t, const char* name) {
  TORCH_CHECK(t.is_cuda(), name, " must be a CUDA tensor");
  TORCH_CHECK(t.scalar_type() == BF16 || t.scalar_type() == F32, name, " must be bf16 or fp32");
  return t.scalar_type() == F32;
}
// 2-D activations with unit inner stride, of the given type.
void chk_rows(const Tensor& t, bool f32, int64_t rows, int64_t cols, const char* name) {
  chk(t, f32 ? F32 : BF16, name);
  TORCH_CHECK(t.dim() == 2 && t.stride(1) == 1 && t.size(0) >= rows && t.size(1) >= cols, name,
              ": expected at least [", rows, ", ", cols, "]");
}
const float* fptr(const OptTensor& t, int64_t n, const char* name) {
  if (!t.has_value()) return nullptr;
  chk_c(*t, F32, name);
  TORCH_CHECK(t->numel() >= n, name, ": expected ", n, " values");
  return t->data_ptr<float>();
}
const float* fptr(const Tensor& t, int64_t n, const char* name) { return fptr(OptTensor(t), n, name); }

// batch = (cu_q, kv_lens, slots, row_seq, pos)
mb::RaggedBatch ragged(const std::vector<Tensor>& batch) {
  TORCH_CHECK(batch.size() == 5, "ragged batch: cu_q, kv_lens, slots, row_seq, pos");
  for (const auto& t : batch) chk_c(t, I32, "ragged batch");
  const int64_t n = batch[1].numel(), rows = batch[4].numel();
  TORCH_CHECK(batch[0].numel() == n + 1 && batch[2].numel() == n && batch[3].numel() == rows, "ragged batch: sizes");
  return mb::RaggedBatch{batch[0].data_ptr<int>(), batch[1].data_ptr<int>(), batch[2].data_ptr<int>(),
                         batch[3].data_ptr<int>(), batch[4].data_ptr<int>(), (int)n, (int)rows};
}

// Short causal convolution of one layer's channels, built once per layer: w [taps, channels] (last row: the current
// token's), state [slots, taps - 1, channels].
struct Conv {
  int channels = 0, taps = 0;
  bool residual = false;
  Tensor w;
  OptTensor bias, state;

  void validate() const {
    TORCH_CHECK(channels > 0 && taps > 0 && taps <= 64, "convolution: sizes");
    fptr(w, (int64_t)taps * channels, "convolution: w");
    fptr(bias, channels, "convolution: bias");
    TORCH_CHECK(taps == 1 || state.has_value(), "convolution: more than one tap needs a state");
    if (taps > 1) fptr(state, state->size(0) * (taps - 1) * channels, "convolution: state");
  }
  mb::ShortConv raw() const {
    return mb::ShortConv{channels, taps, residual, w.data_ptr<float>(), fptr(bias, channels, "bias"),
                         taps > 1 ? const_cast<float*>(fptr(state, 0, "state")) : nullptr};
  }
  // x: [rows, >= off + channels], columns from off on
  void run(const Tensor& x, int64_t off, const std::vector<Tensor>& batch, bool one_token, Tensor& y) const {
    const auto rb = ragged(batch);
    const bool f32 = is_f32(y, "y");
    chk_rows(x, f32, rb.rows, off + channels, "x");
    chk_rows(y, f32, rb.rows, channels, "y");
    TORCH_CHECK(y.stride(0) == y.size(1), "convolution: y must be contiguous");
    c10::cuda::CUDAGuard guard(y.device());
    mb::short_conv(f32, raw(), static_cast<const char*>(x.data_ptr()) + off * (f32 ? 4 : 2), x.stride(0), rb, one_token, y.data_ptr(),
                   y.stride(0), cur_stream());
  }
  // The same inside a kernel that writes the convolution's input, one token per sequence.
  mb::ConvTail tail(const std::vector<Tensor>& batch, Tensor& out, bool f32, int64_t rows) const {
    const auto rb = ragged(batch);
    chk_rows(out, f32, rows, channels, "convolution output");
    TORCH_CHECK(rb.rows == rows && rb.n_seq == rows && residual && !bias.has_value(), "convolution tail: one token per sequence");
    return mb::ConvTail{raw(), rb.slots, rb.kv_lens, out.data_ptr(), out.stride(0)};
  }
};
using ConvArg = std::optional<std::tuple<Conv, std::vector<Tensor>, Tensor>>;     // convolution, batch, output
mb::ConvTail conv_tail(const ConvArg& a, bool f32, int64_t rows) {
  if (!a.has_value()) return mb::ConvTail{};
  Tensor out = std::get<2>(*a);
  return std::get<0>(*a).tail(std::get<1>(*a), out, f32, rows);
}

void embed_pos_norm(const Tensor& ids, const Tensor& pos, const Tensor& embed, const OptTensor& pos_table, double scale,
                    const OptTensor& gamma, Tensor& x, Tensor& h, double eps, const OptTensor& gamma0, const ConvArg& conv) {
  const bool f32 = is_f32(h, "h");
  const int64_t rows = ids.numel(), dim = embed.size(1);
  chk_c(ids, I32, "ids");
  chk_c(pos, I32, "pos");
  chk_c(embed, f32 ? F32 : BF16, "embed");
  chk_c(x, F32, "x");
  chk_rows(h, f32, rows, dim, "h");
  TORCH_CHECK(pos.numel() == rows && x.numel() == rows * dim, "embed_pos_norm: sizes");
  if (pos_table.has_value()) {
    chk_c(*pos_table, f32 ? F32 : BF16, "pos_table");
    TORCH_CHECK(pos_table->size(1) == dim, "pos_table width");
  }
  c10::cuda::CUDAGuard guard(h.device());
  mb::embed_pos_norm(f32, ids.data_ptr<int>(), pos.data_ptr<int>(), embed.data_ptr(), cptr(pos_table),
                     (int)embed.size(0), pos_table.has_value() ? (int)pos_table->size(0) : 1, (float)scale,
                     fptr(gamma0, dim, "gamma0"), fptr(gamma, dim, "gamma"), x.data_ptr<float>(), h.data_ptr(), h.stride(0),
                     (int)rows, (int)dim, (float)eps, conv_tail(conv, f32, rows), cur_stream());
}

// x += mult * (y + bias); h = rms(x) * w_next, with conv also h + conv(h).
void residual_norm(const Tensor& y, const OptTensor& bias, double mult, Tensor& x, const Tensor& w_next, Tensor& h, double eps,
                   const ConvArg& conv) {
  const bool f32 = is_f32(h, "h");
  chk_c(x, F32, "x");
  const int64_t rows = x.size(0), dim = x.size(1);
  chk_rows(y, f32, rows, dim, "y");
  chk_rows(h, f32, rows, dim, "h");
  c10::cuda::CUDAGuard guard(h.device());
  mb::residual_norm(f32, y.data_ptr(), y.stride(0), fptr(bias, dim, "bias"), (float)mult, x.data_ptr<float>(),
                    fptr(w_next, dim, "w_next"), h.data_ptr(), h.stride(0), (int)rows, (int)dim, (float)eps,
                    conv_tail(conv, f32, rows), cur_stream());
}

// out[:, :width] from y + bias; the rest of out's columns are zeroed.
void poly_norm(const Tensor& y, const OptTensor& bias, const Tensor& abce, int64_t width, Tensor& out, double eps) {
  const bool f32 = is_f32(out, "out");
  const int64_t rows = out.size(0);
  chk_rows(y, f32, rows, width, "y");
  chk_rows(out, f32, rows, width, "out");
  c10::cuda::CUDAGuard guard(out.device());
  mb::poly_norm(f32, y.data_ptr(), y.stride(0), fptr(bias, width, "bias"), fptr(abce, 4, "abce"), out.data_ptr(), out.stride(0),
                (int)rows, (int)width, (int)out.size(1), (float)eps, cur_stream());
}

void sandwich_norm(const Tensor& y1, const OptTensor& y2, const OptTensor& w1, const OptTensor& w2, const Tensor& w_post,
                   Tensor& x, const OptTensor& w_next, Tensor& h, double eps, double mult) {
  const bool f32 = is_f32(h, "h");
  chk_c(x, F32, "x");
  const int64_t rows = x.size(0), dim = x.size(1);
  chk_rows(y1, f32, rows, dim, "y1");
  chk_rows(h, f32, rows, dim, "h");
  if (y2.has_value()) {
    chk_rows(*y2, f32, rows, dim, "y2");
    TORCH_CHECK(y2->stride(0) == y1.stride(0), "sandwich_norm: y1 and y2 need the same row stride");
  }
  c10::cuda::CUDAGuard guard(h.device());
  const mb::SublayerOut y{y1.data_ptr(), cptr(y2), y1.stride(0), fptr(w1, dim, "w1"), fptr(w2, dim, "w2"), nullptr, nullptr, 0};
  mb::sandwich_norm(f32, y, fptr(w_post, dim, "w_post"), (float)mult, x.data_ptr<float>(), fptr(w_next, dim, "w_next"),
                    h.data_ptr(), h.stride(0), (int)rows, (int)dim, (float)eps, cur_stream());
}

// The same with the weighted sum of a token's experts as the sublayer's output: y [pairs, dim], row and weight [rows, top];
// shared [rows, dim] (may be null) is added.
void expert_norm(const Tensor& y, const OptTensor& shared, const Tensor& row, const Tensor& weight, const Tensor& w_post, Tensor& x,
                 const OptTensor& w_next, Tensor& h, double eps, double mult) {
  const bool f32 = is_f32(h, "h");
  chk_c(x, F32, "x");
  const int64_t rows = x.size(0), dim = x.size(1), top = row.size(1);
  chk_c(row, I32, "row");
  chk_c(weight, F32, "weight");
  TORCH_CHECK(row.dim() == 2 && row.size(0) == rows && weight.sizes() == row.sizes(), "expert_norm: row / weight");
  chk_rows(y, f32, rows * top, dim, "y");
  chk_rows(h, f32, rows, dim, "h");
  if (shared.has_value()) {
    chk_rows(*shared, f32, rows, dim, "shared");
    TORCH_CHECK(shared->stride(0) == y.stride(0), "expert_norm: y and shared need the same row stride");
  }
  c10::cuda::CUDAGuard guard(h.device());
  const mb::SublayerOut s{y.data_ptr(), cptr(shared), y.stride(0), nullptr, nullptr, row.data_ptr<int>(), weight.data_ptr<float>(),
                          (int)top};
  mb::sandwich_norm(f32, s, fptr(w_post, dim, "w_post"), (float)mult, x.data_ptr<float>(), fptr(w_next, dim, "w_next"),
                    h.data_ptr(), h.stride(0), (int)rows, (int)dim, (float)eps, cur_stream());
}

struct Pages {
  const int* table;
  int stride, page_size, kv_heads, dk, dv;
};
Pages pages(const Tensor& table, const Tensor& k_cache, const Tensor& v_cache, bool f32, int n_seq) {
  chk_c(table, I32, "block_table");
  chk_c(k_cache, f32 ? F32 : BF16, "k_cache");
  chk_c(v_cache, f32 ? F32 : BF16, "v_cache");
  TORCH_CHECK(table.dim() == 2 && table.size(0) >= n_seq, "block_table: one row per sequence of the batch");
  TORCH_CHECK(k_cache.dim() == 4 && v_cache.dim() == 4 && k_cache.size(0) == v_cache.size(0) &&
                  k_cache.size(1) == v_cache.size(1) && k_cache.size(2) == v_cache.size(2),
              "caches: [pages, page_size, kv_heads, width]");
  return Pages{table.data_ptr<int>(), (int)table.size(1), (int)k_cache.size(1), (int)k_cache.size(2),
               (int)k_cache.size(3), (int)v_cache.size(3)};
}

// Softmax attention over the pages of one layer: sizes, offsets in the projection and parameters, built once per layer.
// Head widths are the stored ones (dk, dv); norm_dim, the true key width, counts where heads are normalised.
struct Attention {
  mb::HeadPrep p{};
  float scale = 1.f, out_scale = 1.f;
  int window = 0;
  bool gate_channels = false;
  OptTensor q_bias, k_bias, v_bias, q_gamma, k_gamma, turns, sink;

  mb::AttnExtras extras(const OptTensor& gate, bool f32, int64_t rows) const {
    mb::AttnExtras ex;
    if (gate.has_value()) {
      chk_rows(*gate, f32, rows, gate_channels ? (int64_t)p.heads * p.dv : p.heads, "gate");
      ex.gate = gate->data_ptr();
      ex.ld_gate = gate->stride(0);
      ex.gate_channels = gate_channels;
    }
    ex.sink = fptr(sink, p.heads, "sink");
    ex.window = window;
    ex.out_scale = out_scale;
    return ex;
  }
  Pages layer_pages(const Tensor& table, const Tensor& k_cache, const Tensor& v_cache, bool f32, int n_seq) const {
    const Pages pg = pages(table, k_cache, v_cache, f32, n_seq);
    TORCH_CHECK(pg.kv_heads == p.kv_heads && pg.dk == p.dk && pg.dv == p.dv, "attention: the pages have other heads");
    return pg;
  }
  void check_q(const Tensor& q, bool f32, int64_t rows) const {
    chk_c(q, f32 ? F32 : BF16, "q");
    TORCH_CHECK(q.dim() == 3 && q.size(0) == rows && q.size(1) == p.heads && q.size(2) == p.dk, "q: [rows, heads, dk]");
  }
  void prep(const Tensor& proj, const std::vector<Tensor>& batch, const Tensor& table, Tensor& q, Tensor& k_cache, Tensor& v_cache) const {
    const bool f32 = is_f32(q, "q");
    const auto rb = ragged(batch);
    const Pages pg = layer_pages(table, k_cache, v_cache, f32, rb.n_seq);
    check_q(q, f32, rb.rows);
    int cols = p.q_off + p.heads * p.dk;
    if (p.k_off >= 0) cols = std::max({cols, p.k_off + p.kv_heads * p.dk, p.v_off + p.kv_heads * p.dv});
    chk_rows(proj, f32, rb.rows, cols, "proj");
    c10::cuda::CUDAGuard guard(q.device());
    mb::attn_prep(f32, proj.data_ptr(), proj.stride(0), p, rb, pg.table, pg.stride, pg.page_size, q.data_ptr(), k_cache.data_ptr(),
                  v_cache.data_ptr(), cur_stream());
  }
  // Any widths, scalar arithmetic in 32-bit.
  void any(const Tensor& q, const Tensor& k_cache, const Tensor& v_cache, const std::vector<Tensor>& batch, const Tensor& table,
           const OptTensor& gate, Tensor& o) const {
    const bool f32 = is_f32(q, "q");
    const auto rb = ragged(batch);
    const Pages pg = layer_pages(table, k_cache, v_cache, f32, rb.n_seq);
    check_q(q, f32, rb.rows);
    chk_rows(o, f32, rb.rows, (int64_t)p.heads * p.dv, "o");
    c10::cuda::CUDAGuard guard(q.device());
    mb::paged_attn_any(f32, q.data_ptr(), k_cache.data_ptr(), v_cache.data_ptr(), rb, pg.table, pg.stride, pg.page_size,
                       extras(gate, f32, rb.rows), o.data_ptr(), o.stride(0), p.heads, p.kv_heads, p.dk, p.dv, scale, cur_stream());
  }
  bool tensor_ok(int64_t page_size) const { return page_size == 16 && p.dk % 8 == 0 && p.dv % 8 == 0 && p.dk <= 128 && p.dv <= 128; }
  // Tensor cores: prompts and portions.
  void prefill(const Tensor& q, const Tensor& k_cache, const Tensor& v_cache, const std::vector<Tensor>& batch, const Tensor& table,
               const OptTensor& gate, Tensor& o, int64_t max_q, const OptTensor& status) const {
    const auto rb = ragged(batch);
    const Pages pg = layer_pages(table, k_cache, v_cache, false, rb.n_seq);
    check_q(q, false, rb.rows);
    TORCH_CHECK(tensor_ok(pg.page_size), "attention prefill: widths / page size");
    chk_rows(o, false, rb.rows, (int64_t)p.heads * p.dv, "o");
    c10::cuda::CUDAGuard guard(q.device());
    mb::flash_attn_paged_prefill(q.data_ptr(), q.stride(0), k_cache.data_ptr(), v_cache.data_ptr(), (int)k_cache.size(0), pg.table,
                                 pg.stride, rb.cu_q, rb.kv_lens, o.data_ptr(), o.stride(0), rb.n_seq, rb.rows, (int)max_q, p.heads,
                                 p.kv_heads, p.dk, p.dv, extras(gate, false, rb.rows), scale, status_ptr(status), cur_stream());
  }
  // One token per sequence, split over the context.
  void decode(const Tensor& q, const Tensor& k_cache, const Tensor& v_cache, const std::vector<Tensor>& batch, const Tensor& table,
              const OptTensor& gate, Tensor& o, Tensor& scratch, Tensor& counters, int64_t splits, const OptTensor& status) const {
    const auto rb = ragged(batch);
    const Pages pg = layer_pages(table, k_cache, v_cache, false, rb.n_seq);
    check_q(q, false, rb.rows);
    TORCH_CHECK(tensor_ok(pg.page_size) && rb.rows == rb.n_seq, "attention decode: widths / page size / one token per sequence");
    chk_rows(o, false, rb.rows, (int64_t)p.heads * p.dv, "o");
    chk_c(scratch, F32, "scratch");
    chk_c(counters, I32, "counters");
    TORCH_CHECK(scratch.numel() >= decode_scratch(rb.rows, splits) &&
                    counters.numel() >= (int64_t)rb.rows * p.kv_heads * ((p.heads / p.kv_heads + 7) / 8), "attention decode: scratch");
    c10::cuda::CUDAGuard guard(q.device());
    mb::paged_attn_decode(q.data_ptr(), k_cache.data_ptr(), v_cache.data_ptr(), pg.table, rb.kv_lens, o.data_ptr(),
                          scratch.data_ptr<float>(), counters.data_ptr<int>(), rb.n_seq, p.heads, p.kv_heads, p.dk, 16, pg.stride,
                          (int)k_cache.size(0), (int)splits, scale, status_ptr(status), cur_stream(), q.stride(0), p.dv,
                          extras(gate, false, rb.rows), o.stride(0));
  }
  int64_t decode_scratch(int64_t rows, int64_t splits) const { return rows * p.heads * splits * ((p.dv + 63) / 64 * 64 + 2); }
};

// Gated activation (kind, limit, alpha); see GateAct.
using Act = std::tuple<int64_t, double, double>;
mb::GateAct gate(const Act& a) { return mb::GateAct{(int)std::get<0>(a), (float)std::get<1>(a), (float)std::get<2>(a)}; }

// Few-token GEMM: out = alpha * x w^T, or with f > 0 act(x w[:f]^T, x w[f_off : f_off + f]^T), or with mul
// gelu_tanh(x w^T) * mul[ids, :], or with cap > 0 the soft-capped product.
void gemm_decode(const Tensor& x, const Tensor& w, Tensor& out, int64_t f, int64_t f_off, double alpha,
                 const OptTensor& status, const Act& act, const OptTensor& mul, const OptTensor& ids, double cap) {
  chk(x, BF16, "x");
  chk(w, BF16, "w");
  const bool of32 = is_f32(out, "out");
  TORCH_CHECK(x.dim() == 2 && w.dim() == 2 && out.dim() == 2 && x.stride(1) == 1 && w.stride(1) == 1 && out.stride(1) == 1 &&
                  x.size(1) == w.size(1), "gemm_decode: operands");
  const int64_t n = f > 0 ? f : w.size(0);
  TORCH_CHECK(out.size(0) == x.size(0) && out.size(1) >= n && (f == 0 || f_off + f <= w.size(0)), "gemm_decode: shapes");
  mb::GemmTail tail{f > 0 ? (int)f_off : 0, gate(act), nullptr, nullptr, 0, 0, (float)cap, nullptr, 0, 0};
  if (mul.has_value()) {
    TORCH_CHECK(ids.has_value() && mul->dim() == 2 && mul->stride(1) == 1 && mul->size(1) >= n, "gemm_decode: mul");
    chk(*mul, BF16, "mul");
    chk_c(*ids, I32, "ids");
    TORCH_CHECK(ids->numel() == x.size(0), "gemm_decode: one id per row");
    tail.mul = mul->data_ptr();
    tail.mul_ids = ids->data_ptr<int>();
    tail.ld_mul = mul->stride(0);
    tail.vocab = (int)mul->size(0);
  }
  c10::cuda::CUDAGuard guard(x.device());
  mb::gemm_decode(x.data_ptr(), x.stride(0), w.data_ptr(), w.stride(0), out.data_ptr(), of32, out.stride(0),
                  (int)x.size(0), (int)n, (int)x.size(1), (float)alpha, tail, mb::GemmGroup{}, status_ptr(status), cur_stream());
}

// out[:, b] = x[:, b] w[b]^T for every b: x [rows, b, K], w [b, N, K], out [rows, b, N], inner strides 1. With gate
// [rows, b * N] times its sigmoid.
void gemm_heads(const Tensor& x, const Tensor& w, Tensor& out, const OptTensor& status, const OptTensor& gate) {
  const bool f32 = is_f32(x, "x");
  for (const Tensor* t : {&x, &w, (const Tensor*)&out}) {
    chk(*t, f32 ? F32 : BF16, "gemm_heads operand");
    TORCH_CHECK(t->dim() == 3 && t->stride(2) == 1, "gemm_heads: 3-D operands with unit inner stride");
  }
  const int64_t rows = x.size(0), b = x.size(1), K = x.size(2), N = w.size(1);
  TORCH_CHECK(w.size(0) == b && w.size(2) == K && out.size(0) == rows && out.size(1) == b && out.size(2) == N, "gemm_heads: shapes");
  if (rows == 0) return;
  mb::GemmTail tail{};
  if (gate.has_value()) {
    chk_rows(*gate, f32, rows, b * N, "gate");
    TORCH_CHECK(out.stride(1) == N, "gemm_heads: a gated output has its products side by side");
    tail.gate = gate->data_ptr();
    tail.ld_gate = gate->stride(0);
    tail.gate_batch = N;
  }
  c10::cuda::CUDAGuard guard(x.device());
  if (f32) {
    mb::gemm_f32(x.data_ptr<float>(), x.stride(0), w.data_ptr<float>(), w.stride(1), out.data_ptr<float>(), out.stride(0), (int)rows,
                 (int)N, (int)K, 1.f, cur_stream(), (int)b, x.stride(1), w.stride(0), out.stride(1));
    if (gate.has_value())
      mb::sigmoid_mul(true, out.data_ptr(), out.stride(0), gate->data_ptr(), gate->stride(0), (int)rows, (int)(b * N), cur_stream());
  } else {
    mb::gemm_decode(x.data_ptr(), x.stride(0), w.data_ptr(), w.stride(1), out.data_ptr(), false, out.stride(0), (int)rows, (int)N,
                    (int)K, 1.f, tail, mb::GemmGroup{(int)b, x.stride(1), w.stride(0), out.stride(1), nullptr, 0},
                    status_ptr(status), cur_stream());
  }
}

mb::TileList tile_list(const Tensor& tiles, const Tensor& count) {
  chk_c(tiles, I32, "tiles");
  chk_c(count, I32, "tile count");
  TORCH_CHECK(tiles.dim() == 2 && tiles.size(1) == 3 && tiles.size(0) > 0 && count.numel() == 1, "tile list");
  return mb::TileList{tiles.data_ptr<int>(), count.data_ptr<int>(), (int)tiles.size(0)};
}

// Row segments that meet a matrix each: out rows = x rows times w[matrix]^T (w [matrices, rows, K]), tiles of tile_rows
// rows. f > 0: act of the halves (bf16; fp32 operands take the plain product only). 128-row tiles run the prompt-sized
// kernel, smaller ones the few-token kernel, fp32 operands the fp32 kernel (64-row tiles).
void gemm_tiles(const Tensor& x, const Tensor& w, Tensor& out, const Tensor& tiles, const Tensor& count, int64_t tile_rows,
                int64_t f, int64_t f_off, const Act& act, const OptTensor& status) {
  const bool f32 = is_f32(x, "x");
  chk(w, f32 ? F32 : BF16, "w");
  chk(out, f32 ? F32 : BF16, "out");
  TORCH_CHECK(x.dim() == 2 && x.stride(1) == 1 && w.dim() == 3 && w.stride(2) == 1 && x.size(1) == w.size(2) && out.dim() == 2 &&
                  out.stride(1) == 1 && out.size(0) == x.size(0), "gemm_tiles: operands");
  const int64_t n = f > 0 ? f : w.size(1);
  TORCH_CHECK(out.size(1) >= n && (f == 0 || f_off + f <= w.size(1)), "gemm_tiles: shapes");
  const mb::TileList list = tile_list(tiles, count);
  const mb::GemmTail tail{f > 0 ? (int)f_off : 0, gate(act), nullptr, nullptr, 0, 0, 0.f, nullptr, 0, 0};
  c10::cuda::CUDAGuard guard(x.device());
  if (f32) {
    TORCH_CHECK(f == 0 && tile_rows == 64, "gemm_tiles: fp32 takes 64-row tiles and no tail");
    mb::gemm_f32(x.data_ptr<float>(), x.stride(0), w.data_ptr<float>(), w.stride(1), out.data_ptr<float>(), out.stride(0),
                 (int)x.size(0), (int)n, (int)x.size(1), 1.f, cur_stream(), 1, 0, w.stride(0), 0, &list);
  } else if (tile_rows == 128) {
    mb::gemm_segments(x.data_ptr(), x.stride(0), w.data_ptr(), w.stride(1), w.stride(0), (int)w.size(0), out.data_ptr(),
                      out.stride(0), (int)x.size(0), (int)n, (int)x.size(1), tail, list, status_ptr(status), cur_stream());
  } else {
    mb::gemm_decode(x.data_ptr(), x.stride(0), w.data_ptr(), w.stride(1), out.data_ptr(), false, out.stride(0), (int)x.size(0),
                    (int)n, (int)x.size(1), 1.f, tail,
                    mb::GemmGroup{(int)w.size(0), 0, w.stride(0), 0, &list, (int)tile_rows}, status_ptr(status), cur_stream());
  }
}

// ---- routed experts: spec = (experts, top, groups, keep), rule = (sigmoid, group_best, normalise, scale)
using Router = std::tuple<int64_t, int64_t, int64_t, int64_t>;
using RouterRule = std::tuple<int64_t, int64_t, int64_t, double>;
struct Routing {
  mb::RouterSpec s;
  mb::RouterBuffers b;
};
// idx, weight, slot [rows, top]; state: counts [experts + 1] (zeroed once); plan: offset [experts] | tile count
Routing routing(const Router& r, const Tensor& idx, const Tensor& weight, const Tensor& slot, const Tensor& counts, const Tensor& offset,
                const Tensor& tiles, const Tensor& count) {
  for (const Tensor* t : {&idx, &slot, &counts, &offset}) chk_c(*t, I32, "routing buffer");
  chk_c(weight, F32, "weight");
  const mb::TileList l = tile_list(tiles, count);
  Routing out{{(int)std::get<0>(r), (int)std::get<1>(r), (int)std::get<2>(r), (int)std::get<3>(r), 0, 1, 0, 1.f}, {}};
  TORCH_CHECK(idx.dim() == 2 && idx.size(1) == out.s.top && slot.sizes() == idx.sizes() && weight.sizes() == idx.sizes() &&
                  counts.numel() > out.s.experts && offset.numel() >= out.s.experts, "routing buffers");
  out.b = {idx.data_ptr<int>(), weight.data_ptr<float>(), slot.data_ptr<int>(), counts.data_ptr<int>(), offset.data_ptr<int>(),
           const_cast<int*>(l.tiles), const_cast<int*>(l.count), l.max_tiles};
  return out;
}
void expert_select(const Tensor& logits, const OptTensor& correction, const Router& r, int64_t tile_rows, Tensor& idx, Tensor& weight,
                   Tensor& slot, Tensor& counts, Tensor& offset, Tensor& tiles, Tensor& count, const RouterRule& rule) {
  Routing rt = routing(r, idx, weight, slot, counts, offset, tiles, count);
  rt.s.sigmoid = (int)std::get<0>(rule);
  rt.s.group_best = (int)std::get<1>(rule);
  rt.s.normalise = (int)std::get<2>(rule);
  rt.s.scale = (float)std::get<3>(rule);
  const int64_t rows = idx.size(0);
  chk_rows(logits, true, rows, rt.s.experts, "logits");
  TORCH_CHECK(tile_rows > 0 && tiles.size(0) >= std::min<int64_t>(rows * rt.s.top, rt.s.experts + rows * rt.s.top / tile_rows),
              "expert_select: tile list too short");
  c10::cuda::CUDAGuard guard(logits.device());
  mb::expert_select(logits.data_ptr<float>(), logits.stride(0), fptr(correction, rt.s.experts, "correction"), rt.s, rt.b,
                    (int)tile_rows, (int)rows, cur_stream());
}
void expert_gather(const Tensor& h, const Router& r, const Tensor& idx, const Tensor& weight, const Tensor& slot, const Tensor& counts,
                   const Tensor& offset, const Tensor& tiles, const Tensor& count, Tensor& out, Tensor& row) {
  const Routing rt = routing(r, idx, weight, slot, counts, offset, tiles, count);
  const bool f32 = is_f32(h, "h");
  const int64_t rows = idx.size(0), es = f32 ? 4 : 2;
  chk_rows(h, f32, rows, 1, "h");
  chk_c(out, f32 ? F32 : BF16, "out");
  chk_c(row, I32, "row");
  TORCH_CHECK(out.dim() == 2 && out.size(0) >= rows * rt.s.top && out.size(1) <= h.size(1) && row.numel() == rows * rt.s.top,
              "expert_gather: shapes");
  c10::cuda::CUDAGuard guard(h.device());
  mb::expert_gather(h.data_ptr(), h.stride(0) * es, rt.s, rt.b, out.data_ptr(), row.data_ptr<int>(), out.size(1) * es, (int)rows,
                    cur_stream());
}

void gelu_mul(Tensor& y, const Tensor& table, const Tensor& ids) {
  const bool f32 = is_f32(y, "y");
  chk_rows(y, f32, y.size(0), y.size(1), "y");
  chk_c(ids, I32, "ids");
  TORCH_CHECK(ids.numel() == y.size(0), "gelu_mul: one id per row");
  chk(table, f32 ? F32 : BF16, "table");
  TORCH_CHECK(table.dim() == 2 && table.stride(1) == 1, "gelu_mul: table");
  c10::cuda::CUDAGuard guard(y.device());
  mb::gelu_mul(f32, y.data_ptr(), y.stride(0), table.data_ptr(), table.stride(0), ids.data_ptr<int>(), (int)table.size(0),
               (int)y.size(0), (int)std::min(y.size(1), table.size(1)), cur_stream());
}

// ---- latent attention of one layer: sizes, offsets in the projection and parameters, built once per layer
struct Latent {
  mb::LatentSpec s{};
  int qr_off = 0, c_off = 0, kr_off = 0, low_off = -1, low_rank = 0;   // c_off < 0: another layer's latents
  float scale = 1.f, eps = 1e-6f;
  OptTensor gamma, sink, low_gamma;
  Tensor turns;

  mb::LatentPages pages(const Tensor& table, const Tensor& cache, bool f32, int64_t n_seq) const {
    chk_c(table, I32, "block_table");
    chk_c(cache, f32 ? F32 : BF16, "cache");
    TORCH_CHECK(table.dim() == 2 && table.size(0) >= n_seq, "block_table: one row per sequence of the batch");
    TORCH_CHECK(cache.dim() == 4 && cache.size(2) == 1 && cache.size(3) == s.row(), "cache: [pages, page_size, 1, latent row]");
    return mb::LatentPages{cache.data_ptr(), table.data_ptr<int>(), (int)table.size(1), (int)cache.size(1), (int)cache.size(0)};
  }
  // What of a projection is prepared: latents (and what queries are a map of), rotated query columns, or both.
  void prep(Tensor& proj, const std::vector<Tensor>& batch, const Tensor& table, const Tensor& cache, bool latents, bool queries) const {
    const auto rb = ragged(batch);
    const bool f32 = is_f32(proj, "proj"), own = latents && c_off >= 0, low = latents && low_off >= 0;
    int cols = 0;
    if (queries) cols = qr_off + s.heads * s.rot_p;
    if (own) cols = std::max({cols, c_off + s.rank_p, kr_off + s.rot_p});
    if (low) cols = std::max(cols, low_off + (low_rank + 7) / 8 * 8);
    if (cols == 0) return;
    chk_rows(proj, f32, rb.rows, cols, "proj");
    const mb::LatentPrep p{low ? low_off : -1, low_rank, queries ? qr_off : -1, own ? c_off : -1, own ? kr_off : -1,
                           fptr(low_gamma, low_rank, "low_gamma"), fptr(gamma, s.rank, "gamma"), turns.data_ptr<double>()};
    c10::cuda::CUDAGuard guard(proj.device());
    mb::latent_prep(f32, proj.data_ptr(), proj.stride(0), p, s, rb, pages(table, cache, f32, rb.n_seq), eps, cur_stream());
  }
  void gather(const Tensor& table, const Tensor& cache, const Tensor& cu_k, const Tensor& first, int64_t max_kv, Tensor& out) const {
    chk_c(out, BF16, "out");
    chk_c(cu_k, I32, "cu_k");
    TORCH_CHECK(out.dim() == 2 && out.size(1) == s.row(), "gather: out");
    const int n_seq = (int)cu_k.numel() - 1;
    chk_c(first, I32, "first");
    TORCH_CHECK(first.numel() == n_seq, "gather: first");
    c10::cuda::CUDAGuard guard(out.device());
    mb::latent_gather(s, pages(table, cache, false, n_seq), cu_k.data_ptr<int>(), first.data_ptr<int>(), n_seq, (int)max_kv,
                      out.data_ptr(), cur_stream());
  }
  mb::LatentQuery query(const Tensor& q_lat, const Tensor& proj, const Tensor& row_seq, const Tensor& pos, const Tensor& o,
                        bool f32) const {
    const int64_t rows = q_lat.size(0);
    for (const Tensor* t : {&q_lat, &o}) {
      chk_c(*t, f32 ? F32 : BF16, "q_lat / o");
      TORCH_CHECK(t->dim() == 3 && t->size(0) == rows && t->size(1) == s.heads && t->size(2) == s.rank_p, "q_lat / o: [rows, heads, rank]");
    }
    chk_rows(proj, f32, rows, qr_off + s.heads * s.rot_p, "proj");
    chk_c(row_seq, I32, "row_seq");
    chk_c(pos, I32, "pos");
    TORCH_CHECK(row_seq.numel() == rows && pos.numel() == rows, "row_seq / pos");
    return mb::LatentQuery{q_lat.data_ptr(), static_cast<const char*>(proj.data_ptr()) + (int64_t)qr_off * (f32 ? 4 : 2), proj.stride(0),
                           row_seq.data_ptr<int>(), pos.data_ptr<int>(), (int)rows};
  }
  void attn_any(const Tensor& q_lat, const Tensor& proj, const Tensor& row_seq, const Tensor& pos, const Tensor& table,
                const Tensor& cache, Tensor& o) const {
    const bool f32 = is_f32(q_lat, "q_lat");
    const auto q = query(q_lat, proj, row_seq, pos, o, f32);
    c10::cuda::CUDAGuard guard(o.device());
    mb::latent_attn_any(f32, q, s, pages(table, cache, f32, 0), fptr(sink, s.heads, "sink"), o.data_ptr(), scale, cur_stream());
  }
  bool decode_ok(int64_t page_size) const { return mb::latent_decode_ok(s, (int)page_size); }
  void attn_decode(const Tensor& q_lat, const Tensor& proj, const Tensor& row_seq, const Tensor& pos, const Tensor& table,
                   const Tensor& cache, Tensor& o, Tensor& scratch, int64_t splits, const OptTensor& status) const {
    const auto q = query(q_lat, proj, row_seq, pos, o, false);
    chk_c(scratch, F32, "scratch");
    TORCH_CHECK(splits == 1 || scratch.numel() >= (int64_t)q.rows * s.heads * splits * (s.rank_p + 4), "attn_decode: scratch");
    c10::cuda::CUDAGuard guard(o.device());
    mb::latent_attn_decode(q, s, pages(table, cache, false, 0), fptr(sink, s.heads, "sink"), o.data_ptr(), scratch.data_ptr<float>(),
                           (int)splits, scale, status_ptr(status), cur_stream());
  }
  bool prefill_ok(int64_t dim_p, int64_t vdim_p) const { return mb::flash_attn_ragged_ok((int)dim_p, s.rot_p, (int)vdim_p); }
  // q, kv: [rows, heads, width] views (unrotated queries; expanded keys and values), latents [keys, row], key_lens keys of every
  // sequence, o [rows, heads, vdim], gate [rows, heads * vdim] or null
  void attn_prefill(const Tensor& q, const Tensor& proj, const Tensor& k, const Tensor& v, const Tensor& latents,
                    const std::vector<Tensor>& batch, const Tensor& cu_k, const Tensor& key_lens, int64_t max_q, int64_t min_q,
                    const OptTensor& gate, Tensor& o, const OptTensor& status) const {
    const auto rb = ragged(batch);
    for (const Tensor* t : {&q, &k, &v, (const Tensor*)&o}) {
      chk(*t, BF16, "attn_prefill operand");
      TORCH_CHECK(t->dim() == 3 && t->size(1) == s.heads && t->stride(2) == 1 && t->stride(1) == t->size(2), "attn_prefill: [rows, heads, width]");
    }
    chk_rows(proj, false, rb.rows, qr_off + s.heads * s.rot_p, "proj");
    chk_c(latents, BF16, "latents");
    chk_c(cu_k, I32, "cu_k");
    chk_c(key_lens, I32, "key_lens");
    TORCH_CHECK(key_lens.numel() == rb.n_seq, "attn_prefill: key_lens");
    TORCH_CHECK(q.size(0) == rb.rows && o.size(0) == rb.rows && k.size(0) == v.size(0) && k.stride(0) == v.stride(0) &&
                    q.size(2) == k.size(2) && v.size(2) == o.size(2) && proj.stride(0) == q.stride(0) && latents.size(0) == k.size(0) &&
                    latents.size(1) == s.row() && cu_k.numel() == rb.n_seq + 1, "attn_prefill: shapes");
    mb::RaggedAttn a{};
    a.q = q.data_ptr();
    a.q_rot = static_cast<const char*>(proj.data_ptr()) + (int64_t)qr_off * 2;
    a.k = k.data_ptr();
    a.k_rot = static_cast<const char*>(latents.data_ptr()) + (int64_t)s.rank_p * 2;
    a.v = v.data_ptr();
    a.o = o.data_ptr();
    a.ldq = q.stride(0);
    a.ldkv = k.stride(0);
    a.ldk_rot = latents.stride(0);
    a.ldo = o.stride(0);
    a.cu_q = rb.cu_q;
    a.cu_k = cu_k.data_ptr<int>();
    a.key_lens = key_lens.data_ptr<int>();
    a.sink = fptr(sink, s.heads, "sink");
    if (gate.has_value()) {
      chk_rows(*gate, false, rb.rows, s.heads * o.size(2), "gate");
      a.gate = gate->data_ptr();
      a.ld_gate = gate->stride(0);
    }
    a.window = s.window;
    a.batch = rb.n_seq;
    a.total_q = rb.rows;
    a.total_k = (int)k.size(0);
    a.max_q = (int)max_q;
    a.min_q = (int)min_q;
    a.heads = s.heads;
    a.dim = (int)q.size(2);
    a.rot = s.rot_p;
    a.vdim = (int)v.size(2);
    a.scale = scale;
    c10::cuda::CUDAGuard guard(o.device());
    mb::flash_attn_ragged(a, status_ptr(status), cur_stream());
  }
};

// h = silu(x w[:f]^T) * (x w[f:2f]^T) in the GEMM's epilogue (prompt-sized batches, f a multiple of 128).
void gemm_swiglu(const Tensor& x, const Tensor& w, Tensor& h, const OptTensor& status) {
  chk(x, BF16, "x");
  chk(w, BF16, "w");
  chk(h, BF16, "h");
  TORCH_CHECK(x.dim() == 2 && w.dim() == 2 && h.dim() == 2 && x.stride(1) == 1 && w.stride(1) == 1 && h.stride(1) == 1 &&
                  x.size(1) == w.size(1) && h.size(0) == x.size(0) && h.size(1) * 2 == w.size(0), "gemm_swiglu: shapes");
  c10::cuda::CUDAGuard guard(x.device());
  mb::gemm_swiglu_fwd(x.data_ptr(), x.stride(0), w.data_ptr(), w.stride(0), nullptr, 0, h.data_ptr(), h.stride(0),
                      (int)x.size(0), (int)h.size(1), (int)x.size(1), status_ptr(status), cur_stream());
}

// out = alpha * a b^T; bf16 operands run the tcgen05 GEMM (bf16 or fp32 output), fp32 operands the fp32 kernel.
void gemm_nt(const Tensor& a, const Tensor& b, Tensor& out, double alpha, const OptTensor& status) {
  const bool f32 = is_f32(a, "a");
  chk(b, f32 ? F32 : BF16, "b");
  TORCH_CHECK(a.dim() == 2 && b.dim() == 2 && out.dim() == 2 && a.stride(1) == 1 && b.stride(1) == 1 && out.stride(1) == 1,
              "gemm_nt: 2-D operands with unit inner stride");
  TORCH_CHECK(a.size(1) == b.size(1) && out.size(0) == a.size(0) && out.size(1) == b.size(0), "gemm_nt: shapes");
  c10::cuda::CUDAGuard guard(a.device());
  if (f32) {
    chk(out, F32, "out");
    mb::gemm_f32(a.data_ptr<float>(), a.stride(0), b.data_ptr<float>(), b.stride(0), out.data_ptr<float>(), out.stride(0),
                 (int)a.size(0), (int)b.size(0), (int)a.size(1), (float)alpha, cur_stream());
  } else {
    const bool of32 = is_f32(out, "out");
    mb::gemm_bf16(a.data_ptr(), a.stride(0), false, b.data_ptr(), b.stride(0), false, out.data_ptr(), out.stride(0),
                  (int)a.size(0), (int)b.size(0), (int)a.size(1), of32 ? mb::EPI_F32 : mb::EPI_BF16, (float)alpha,
                  status_ptr(status), cur_stream());
  }
}

void gate_pair(const Tensor& gu, int64_t f, int64_t f_off, const Act& act, Tensor& h) {
  const bool f32 = is_f32(h, "h");
  chk_rows(h, f32, h.size(0), f, "h");
  chk_rows(gu, f32, h.size(0), f_off + f, "gu");
  TORCH_CHECK(h.stride(0) == h.size(1), "gate_pair: h must be contiguous");
  c10::cuda::CUDAGuard guard(h.device());
  mb::gate_pair(f32, gu.data_ptr(), gu.stride(0), (int)f, (int)f_off, gate(act), h.data_ptr(), h.stride(0), (int)h.size(0),
                cur_stream());
}

// The recurrence of one layer with its parameters and state, built once per layer.
struct Recurrent {
  mb::RecurrentSpec s{};
  int q_off = 0, k_off = 0, v_off = 0, b_off = 0;
  OptTensor z_bias, a_log, conv_w, conv_state, gamma, a2, g2;
  Tensor state;

  int channels() const { return 2 * s.kv_heads * s.dim + s.heads * s.vdim; }
  void validate() const {
    chk_c(state, F32, "state");
    TORCH_CHECK(state.dim() == 4 && state.size(1) == s.heads && state.size(2) == s.vdim && state.size(3) == s.dim,
                "state: [slots, heads, vdim, dim]");
    TORCH_CHECK(z_bias.has_value(), "recurrent: z_bias");
    fptr(z_bias, (int64_t)s.heads * s.dim, "z_bias");
    TORCH_CHECK(s.decay_kind == 0 || a_log.has_value(), "recurrent: a_log");
    fptr(a_log, s.heads, "a_log");
    if (s.taps > 0) {
      TORCH_CHECK(conv_w.has_value(), "recurrent: conv_w");
      fptr(conv_w, (int64_t)channels() * s.taps, "conv_w");
      if (s.taps > 1) {
        TORCH_CHECK(conv_state.has_value(), "recurrent: conv_state");
        fptr(conv_state, state.size(0) * (s.taps - 1) * channels(), "conv_state");
      }
    }
  }
  mb::RecurrentInputs inputs(const Tensor& proj, const OptTensor& z, int64_t rows) {
    const bool f32 = is_f32(proj, "proj");
    const int64_t cq = (int64_t)s.kv_heads * s.dim, cv = (int64_t)s.heads * s.vdim;
    chk_rows(proj, f32, rows, std::max({q_off + cq, k_off + cq, v_off + cv, (int64_t)(s.delta ? b_off + s.heads : 0)}),
             "proj");
    mb::RecurrentInputs in{};
    in.proj = proj.data_ptr();
    in.ld = proj.stride(0);
    in.q_off = q_off;
    in.k_off = k_off;
    in.v_off = v_off;
    in.b_off = b_off;
    if (z.has_value()) {
      chk_rows(*z, true, rows, (int64_t)s.heads * s.dim, "z");
      in.z = z->data_ptr<float>();
      in.ldz = z->stride(0);
    }
    in.z_bias = z_bias->data_ptr<float>();
    in.a_log = fptr(a_log, s.heads, "a_log");
    in.conv_w = fptr(conv_w, 0, "conv_w");
    in.conv_state = const_cast<float*>(fptr(conv_state, 0, "conv_state"));
    in.state = state.data_ptr<float>();
    return in;
  }
  // o [rows, heads, vdim] fp32; the recurrence state and the convolution state advance.
  void scan_seq(const Tensor& proj, const Tensor& z, const std::vector<Tensor>& batch, Tensor& scratch, Tensor& o) {
    const auto rb = ragged(batch);
    const int64_t need = (int64_t)rb.rows * (2 * s.kv_heads * s.dim + s.heads * (s.vdim + s.dim + 1));
    chk_c(scratch, F32, "scratch");
    chk_c(o, F32, "o");
    TORCH_CHECK(scratch.numel() >= need && o.numel() >= (int64_t)rb.rows * s.heads * s.vdim, "scan_seq: buffers");
    const auto in = inputs(proj, z, rb.rows);
    c10::cuda::CUDAGuard guard(proj.device());
    const bool f32 = is_f32(proj, "proj");
    mb::recurrent_scan_seq(f32, s, in, rb, scratch.data_ptr<float>(), o.data_ptr<float>(), cur_stream());
    mb::conv_state_update(f32, s, in, rb, cur_stream());
  }
  bool chunked_ok() const { return mb::recurrent_chunked_ok(s); }
  int64_t chunked_scratch(int64_t rows, int64_t n_seq) const {
    return mb::recurrent_chunked_scratch(s, (int)rows, (int)n_seq);
  }
  void scan_chunked(const Tensor& proj, const Tensor& z, const std::vector<Tensor>& batch, Tensor& scratch, Tensor& o,
                    const OptTensor& status) {
    const auto rb = ragged(batch);
    chk(proj, BF16, "proj");
    chk_c(scratch, U8, "scratch");
    chk_c(o, F32, "o");
    TORCH_CHECK(scratch.numel() >= chunked_scratch(rb.rows, rb.n_seq) &&
                    o.numel() >= (int64_t)rb.rows * s.heads * s.vdim, "scan_chunked: buffers");
    const auto in = inputs(proj, z, rb.rows);
    c10::cuda::CUDAGuard guard(proj.device());
    mb::recurrent_scan_chunked(s, in, rb, scratch.data_ptr(), o.data_ptr<float>(), status_ptr(status), cur_stream());
    mb::conv_state_update(false, s, in, rb, cur_stream());
  }
  // One token per sequence in one launch; z / gate null: computed from the columns a_off / g_off of proj.
  void decode(const Tensor& proj, const OptTensor& z, const OptTensor& gate, int64_t a_off, int64_t g_off,
              const std::vector<Tensor>& batch, Tensor& out) {
    const auto rb = ragged(batch);
    const bool f32 = is_f32(out, "out");
    const int64_t cv = (int64_t)s.heads * s.vdim;
    chk_rows(out, f32, rb.rows, cv, "out");
    TORCH_CHECK(out.stride(0) == out.size(1), "decode: out must be contiguous");
    auto map = [&](const OptTensor& w, int64_t off, int64_t outputs, const char* name) {
      mb::DecodeLowRank m{};
      if (!w.has_value()) return m;
      chk_c(*w, f32 ? F32 : BF16, name);
      TORCH_CHECK(w->dim() == 2 && w->size(0) == outputs && off + w->size(1) <= proj.size(1), name);
      m.w = w->data_ptr();
      m.ld = w->stride(0);
      m.off = (int)off;
      m.rank = (int)w->size(1);
      return m;
    };
    const auto ma = z.has_value() ? mb::DecodeLowRank{} : map(a2, a_off, (int64_t)s.heads * s.dim, "a2");
    const auto mg = gate.has_value() ? mb::DecodeLowRank{} : map(g2, g_off, cv, "g2");
    if (gate.has_value()) chk_rows(*gate, f32, rb.rows, cv, "gate");
    const auto in = inputs(proj, z, rb.rows);
    c10::cuda::CUDAGuard guard(out.device());
    mb::recurrent_decode(f32, s, in, rb, ma, mg, fptr(gamma, s.vdim, "gamma"), cptr(gate),
                         gate.has_value() ? gate->stride(0) : 0, out.data_ptr(), out.stride(0), cur_stream());
  }
  void norm_gate(const Tensor& o, const Tensor& gate, Tensor& out) {
    const bool f32 = is_f32(out, "out");
    const int64_t rows = out.size(0), cv = (int64_t)s.heads * s.vdim;
    chk_c(o, F32, "o");
    TORCH_CHECK(o.numel() >= rows * cv, "norm_gate: o");
    chk_rows(out, f32, rows, cv, "out");
    chk_rows(gate, f32, rows, cv, "gate");
    TORCH_CHECK(out.stride(0) == out.size(1), "norm_gate: out must be contiguous");
    c10::cuda::CUDAGuard guard(out.device());
    mb::head_norm_gate(f32, s, o.data_ptr<float>(), fptr(gamma, s.vdim, "gamma"), gate.data_ptr(), gate.stride(0),
                       out.data_ptr(), out.stride(0), (int)rows, cur_stream());
  }
};

// The selective scan of one layer with its parameters and state, built once per layer.
struct Selective {
  mb::SelectiveSpec s{};
  int z_off = 0, b_off = 0, c_off = 0;
  Tensor a, d, dt_b, state, w_dt;

  void validate() const {
    const int64_t sp = mb::selective_padded_state(s.state);
    TORCH_CHECK(s.inner > 0 && s.state > 0 && s.rank > 0, "selective: sizes");
    chk_c(state, F32, "state");
    TORCH_CHECK(state.dim() == 3 && state.size(1) == s.inner && state.size(2) == sp, "state: [slots, inner, padded state]");
    for (const Tensor* t : {&d, &dt_b}) fptr(*t, s.inner, "selective: channel parameters");
    fptr(a, s.inner * sp, "a");
    is_f32(w_dt, "w_dt");
    TORCH_CHECK(w_dt.dim() == 2 && w_dt.size(0) == s.inner && w_dt.stride(1) == 1 && w_dt.size(1) >= (s.rank + 7) / 8 * 8, "w_dt");
  }
  mb::SelectiveInputs inputs(const Tensor& proj, bool f32, int64_t rows) const {
    chk_rows(proj, f32, rows, z_off + s.inner, "proj");
    mb::SelectiveInputs in{};
    in.proj = proj.data_ptr();
    in.ld = proj.stride(0);
    in.z_off = z_off;
    in.a = a.data_ptr<float>();
    in.d = d.data_ptr<float>();
    in.dt_bias = dt_b.data_ptr<float>();
    in.state = state.data_ptr<float>();
    in.b_off = b_off;
    in.c_off = c_off;
    return in;
  }
  mb::SelectiveInputs inputs(const Tensor& proj, const Tensor& x, const Tensor& low, bool f32, int64_t rows) const {
    mb::SelectiveInputs in = inputs(proj, f32, rows);
    chk_rows(x, f32, rows, s.inner, "x");
    chk_rows(low, f32, rows, std::max({std::max(b_off, c_off) + (s.state + 7) / 8 * 8, (s.rank + 7) / 8 * 8}), "low");
    in.x = x.data_ptr();
    in.ld_x = x.stride(0);
    in.low = low.data_ptr();
    in.ld_low = low.stride(0);
    return in;
  }
  int64_t scratch_floats(int64_t n_seq, int64_t rows, int64_t max_q) const {
    return mb::selective_scratch(s, (int)n_seq, (int)rows, (int)max_q);
  }
  void scan(const Tensor& proj, const Tensor& x, const Tensor& low, const Tensor& dt, const std::vector<Tensor>& batch, int64_t max_q,
            Tensor& scratch, Tensor& out, const OptTensor& status) const {
    const auto rb = ragged(batch);
    const bool f32 = is_f32(out, "out");
    chk_rows(out, f32, rb.rows, s.inner, "out");
    chk_rows(dt, true, rb.rows, s.inner, "dt");
    chk_c(scratch, F32, "scratch");
    TORCH_CHECK(scratch.numel() >= scratch_floats(rb.n_seq, rb.rows, max_q), "scan: scratch");
    c10::cuda::CUDAGuard guard(out.device());
    mb::selective_scan(f32, s, inputs(proj, x, low, f32, rb.rows), rb, (int)max_q, dt.data_ptr<float>(), dt.stride(0),
                       scratch.data_ptr<float>(), out.data_ptr(), out.stride(0), status_ptr(status), cur_stream());
  }
  // One token per sequence; dt null: computed from the first columns of low.
  void step(const Tensor& proj, const Tensor& x, const Tensor& low, const OptTensor& dt, const std::vector<Tensor>& batch,
            Tensor& out) const {
    const auto rb = ragged(batch);
    const bool f32 = is_f32(out, "out");
    chk_rows(out, f32, rb.rows, s.inner, "out");
    if (dt.has_value()) chk_rows(*dt, true, rb.rows, s.inner, "dt");
    TORCH_CHECK(is_f32(w_dt, "w_dt") == f32, "step: w_dt and the activations differ in type");
    c10::cuda::CUDAGuard guard(out.device());
    mb::selective_step(f32, s, inputs(proj, x, low, f32, rb.rows), rb, dt.has_value() ? dt->data_ptr<float>() : nullptr,
                       dt.has_value() ? dt->stride(0) : 0, w_dt.data_ptr(), w_dt.stride(0), out.data_ptr(), out.stride(0), cur_stream());
  }
};

void soft_cap(Tensor& y, double cap) {
  chk_rows(y, true, y.size(0), y.size(1), "y");
  c10::cuda::CUDAGuard guard(y.device());
  mb::soft_cap(y.data_ptr<float>(), y.stride(0), (int)y.size(0), (int)y.size(1), (float)cap, cur_stream());
}

}  // namespace

PYBIND11_MODULE(TORCH_EXTENSION_NAME, m) {
  m.doc() = "sm_100a kernels of layer-list models";
  namespace py = pybind11;
  py::class_<Conv>(m, "Conv")
      .def(py::init([](int64_t channels, bool residual, const Tensor& w, const OptTensor& bias, const OptTensor& state) {
             Conv c;
             TORCH_CHECK(w.dim() == 2 && w.size(1) == channels, "convolution: w [taps, channels]");
             c.channels = (int)channels;
             c.taps = (int)w.size(0);
             c.residual = residual;
             c.w = w;
             c.bias = bias;
             c.state = state;
             c.validate();
             return c;
           }),
           py::arg("channels"), py::arg("residual"), py::arg("w"), py::arg("bias") = OptTensor(), py::arg("state") = OptTensor())
      .def("run", &Conv::run);
  m.def("embed_pos_norm", &embed_pos_norm, py::arg("ids"), py::arg("pos"), py::arg("embed"), py::arg("pos_table"), py::arg("scale"),
        py::arg("gamma"), py::arg("x"), py::arg("h"), py::arg("eps"), py::arg("gamma0") = OptTensor(), py::arg("conv") = ConvArg());
  m.def("residual_norm", &residual_norm, py::arg("y"), py::arg("bias"), py::arg("mult"), py::arg("x"), py::arg("w_next"), py::arg("h"),
        py::arg("eps"), py::arg("conv") = ConvArg());
  m.def("poly_norm", &poly_norm);
  m.def("sandwich_norm", &sandwich_norm, py::arg("y1"), py::arg("y2"), py::arg("w1"), py::arg("w2"), py::arg("w_post"), py::arg("x"),
        py::arg("w_next"), py::arg("h"), py::arg("eps"), py::arg("mult") = 1.0);
  m.def("expert_norm", &expert_norm, py::arg("y"), py::arg("shared"), py::arg("row"), py::arg("weight"), py::arg("w_post"), py::arg("x"),
        py::arg("w_next"), py::arg("h"), py::arg("eps"), py::arg("mult") = 1.0);
  m.def("gemm_decode", &gemm_decode, py::arg("x"), py::arg("w"), py::arg("out"), py::arg("f"), py::arg("f_off"), py::arg("alpha"),
        py::arg("status"), py::arg("act") = Act(0, 0.0, 0.0), py::arg("mul") = OptTensor(), py::arg("ids") = OptTensor(),
        py::arg("cap") = 0.0);
  m.def("gemm_heads", &gemm_heads, py::arg("x"), py::arg("w"), py::arg("out"), py::arg("status"), py::arg("gate") = OptTensor());
  m.def("gemm_tiles", &gemm_tiles);
  m.def("expert_select", &expert_select, py::arg("logits"), py::arg("correction"), py::arg("spec"), py::arg("tile_rows"), py::arg("idx"),
        py::arg("weight"), py::arg("slot"), py::arg("counts"), py::arg("offset"), py::arg("tiles"), py::arg("count"),
        py::arg("rule") = RouterRule(0, 1, 0, 1.0));
  m.def("soft_cap", &soft_cap);
  m.def("selective_padded_state", [](int64_t state) { return mb::selective_padded_state((int)state); });
  m.def("expert_gather", &expert_gather);
  m.def("gelu_mul", &gelu_mul);
  m.def("gate_pair", &gate_pair);
  m.def("gemm_swiglu", &gemm_swiglu);
  m.def("gemm_nt", &gemm_nt);
  m.def("sample_tokens", &sample_tokens);
  pybind11::class_<Recurrent>(m, "Recurrent")
      .def(pybind11::init([](pybind11::dict spec, pybind11::dict tensors) {
        Recurrent r;
        auto geti = [&](const char* k, int d) { return spec.contains(k) ? spec[k].cast<int>() : d; };
        auto getf = [&](const char* k, float d) { return spec.contains(k) ? spec[k].cast<float>() : d; };
        auto gett = [&](const char* k) -> OptTensor {
          if (!tensors.contains(k)) return c10::nullopt;
          return tensors[k].cast<Tensor>();
        };
        r.s.heads = geti("heads", 0);
        r.s.kv_heads = geti("kv_heads", r.s.heads);
        r.s.dim = geti("dim", 0);
        r.s.vdim = geti("vdim", 0);
        r.s.taps = geti("taps", 0);
        r.s.delta = geti("delta", 0);
        r.s.unit_norm = geti("unit_norm", 0);
        r.s.decay_kind = geti("decay_kind", 0);
        r.s.gate_kind = geti("gate_kind", 0);
        r.s.q_scale = getf("q_scale", 1.f);
        r.s.inv_tau = getf("inv_tau", 1.f);
        r.s.eps = getf("eps", 1e-6f);
        r.q_off = geti("q_off", 0);
        r.k_off = geti("k_off", 0);
        r.v_off = geti("v_off", 0);
        r.b_off = geti("b_off", 0);
        r.z_bias = gett("z_bias");
        r.a_log = gett("a_log");
        r.conv_w = gett("conv_w");
        r.conv_state = gett("conv_state");
        r.gamma = gett("gamma");
        r.a2 = gett("a2");
        r.g2 = gett("g2");
        r.state = tensors["state"].cast<Tensor>();
        r.validate();
        return r;
      }))
      .def("scan_seq", &Recurrent::scan_seq)
      .def("chunked_ok", &Recurrent::chunked_ok)
      .def("chunked_scratch", &Recurrent::chunked_scratch)
      .def("scan_chunked", &Recurrent::scan_chunked)
      .def("decode", &Recurrent::decode)
      .def("norm_gate", &Recurrent::norm_gate);
  py::class_<Latent>(m, "Latent")
      .def(py::init([](py::dict d, const OptTensor& gamma, const Tensor& turns, const OptTensor& sink, const OptTensor& low_gamma) {
        Latent l;
        auto geti = [&](const char* k) { return d[k].cast<int>(); };
        l.s = mb::LatentSpec{geti("heads"), geti("rank"), geti("rot"), geti("rank_p"), geti("rot_p"),
                             d.contains("window") ? geti("window") : 0, d.contains("rot_amp") ? d["rot_amp"].cast<float>() : 1.f};
        TORCH_CHECK(l.s.window >= 0, "latent: window");
        if (d.contains("low_off")) {
          l.low_off = geti("low_off");
          l.low_rank = geti("low_rank");
          TORCH_CHECK(l.low_off >= 0 && l.low_off % 8 == 0 && l.low_rank > 0 && low_gamma.has_value(), "latent: low-rank queries");
        }
        TORCH_CHECK(l.s.heads > 0 && l.s.rank > 0 && l.s.rot > 0 && l.s.rank_p >= l.s.rank && l.s.rot_p >= l.s.rot &&
                        l.s.rank_p % 8 == 0 && l.s.rot_p % 8 == 0, "latent: sizes");
        l.qr_off = geti("qr_off");
        l.c_off = d.contains("c_off") ? geti("c_off") : -1;
        if (l.c_off >= 0) {
          l.kr_off = geti("kr_off");
          TORCH_CHECK(l.kr_off >= 0 && (l.c_off | l.kr_off) % 8 == 0 && gamma.has_value(), "latent: offsets");
        }
        TORCH_CHECK(l.qr_off >= 0 && l.qr_off % 8 == 0, "latent: offsets");
        l.scale = d["scale"].cast<float>();
        l.eps = d["eps"].cast<float>();
        fptr(gamma, l.s.rank, "gamma");
        fptr(sink, l.s.heads, "sink");
        chk_c(turns, torch::kFloat64, "turns");
        TORCH_CHECK(turns.numel() >= l.s.rot / 2, "latent: turns");
        fptr(low_gamma, l.low_rank, "low_gamma");
        l.gamma = gamma;
        l.turns = turns;
        l.sink = sink;
        l.low_gamma = low_gamma;
        return l;
      }), py::arg("spec"), py::arg("gamma"), py::arg("turns"), py::arg("sink"), py::arg("low_gamma") = OptTensor())
      .def("prep", &Latent::prep, py::arg("proj"), py::arg("batch"), py::arg("table"), py::arg("cache"), py::arg("latents") = true,
           py::arg("queries") = true)
      .def("gather", &Latent::gather)
      .def("attn_any", &Latent::attn_any)
      .def("decode_ok", &Latent::decode_ok)
      .def("attn_decode", &Latent::attn_decode)
      .def("prefill_ok", &Latent::prefill_ok)
      .def("attn_prefill", &Latent::attn_prefill);
  py::class_<Attention>(m, "Attention")
      .def(py::init([](py::dict spec, py::dict tensors) {
        Attention t;
        auto geti = [&](const char* k, int v) { return spec.contains(k) ? spec[k].cast<int>() : v; };
        auto getf = [&](const char* k, float v) { return spec.contains(k) ? spec[k].cast<float>() : v; };
        auto gett = [&](const char* k) -> OptTensor {
          if (!tensors.contains(k)) return c10::nullopt;
          return tensors[k].cast<Tensor>();
        };
        t.p.heads = geti("heads", 0);
        t.p.kv_heads = geti("kv_heads", t.p.heads);
        t.p.dk = geti("dk", 0);
        t.p.dv = geti("dv", 0);
        TORCH_CHECK(t.p.heads > 0 && t.p.kv_heads > 0 && t.p.heads % t.p.kv_heads == 0 && t.p.dk > 0 && t.p.dv > 0, "attention: sizes");
        t.p.q_off = geti("q_off", 0);
        t.p.k_off = geti("k_off", -1);
        t.p.v_off = geti("v_off", 0);
        t.p.norm_dim = geti("norm_dim", 0);
        t.p.rot = geti("rot", 0);
        t.p.pairs = geti("pairs", 0) != 0;
        t.p.rot_amp = getf("rot_amp", 1.f);
        t.p.temp_coef = getf("temp_coef", 0.f);
        t.p.temp_every = getf("temp_every", 1.f);
        t.p.eps = getf("eps", 1e-6f);
        t.scale = getf("scale", 1.f);
        t.out_scale = getf("out_scale", 1.f);
        t.window = geti("window", 0);
        t.gate_channels = geti("gate_channels", 0) != 0;
        t.q_bias = gett("q_bias");
        t.k_bias = gett("k_bias");
        t.v_bias = gett("v_bias");
        t.q_gamma = gett("q_gamma");
        t.k_gamma = gett("k_gamma");
        t.turns = gett("turns");
        t.sink = gett("sink");
        TORCH_CHECK(t.window >= 0 && t.p.norm_dim >= 0 && t.p.norm_dim <= t.p.dk && t.p.rot >= 0 && t.p.rot <= t.p.dk && t.p.rot % 2 == 0,
                    "attention: window / norm / rotation");
        t.p.q_bias = fptr(t.q_bias, (int64_t)t.p.heads * t.p.dk, "q_bias");
        t.p.k_bias = fptr(t.k_bias, (int64_t)t.p.kv_heads * t.p.dk, "k_bias");
        t.p.v_bias = fptr(t.v_bias, (int64_t)t.p.kv_heads * t.p.dv, "v_bias");
        t.p.q_gamma = fptr(t.q_gamma, t.p.dk, "q_gamma");
        t.p.k_gamma = fptr(t.k_gamma, t.p.dk, "k_gamma");
        fptr(t.sink, t.p.heads, "sink");
        if (t.p.rot > 0) {
          TORCH_CHECK(t.turns.has_value(), "attention: turns");
          chk_c(*t.turns, torch::kFloat64, "turns");
          TORCH_CHECK(t.turns->numel() >= t.p.rot / 2, "attention: turns");
          t.p.turns = t.turns->data_ptr<double>();
        }
        return t;
      }))
      .def("prep", &Attention::prep)
      .def("any", &Attention::any)
      .def("tensor_ok", &Attention::tensor_ok)
      .def("prefill", &Attention::prefill)
      .def("decode", &Attention::decode)
      .def("decode_scratch", &Attention::decode_scratch);
  py::class_<Selective>(m, "Selective")
      .def(py::init([](py::dict spec, py::dict tensors) {
        Selective t;
        auto geti = [&](const char* k) { return spec[k].cast<int>(); };
        auto gett = [&](const char* k) { return tensors[k].cast<Tensor>(); };
        t.s = mb::SelectiveSpec{geti("inner"), geti("state"), geti("rank"), spec["out_scale"].cast<float>()};
        t.z_off = geti("z_off");
        t.b_off = geti("b_off");
        t.c_off = geti("c_off");
        t.a = gett("a");
        t.d = gett("d");
        t.dt_b = gett("dt_b");
        t.state = gett("state");
        t.w_dt = gett("w_dt");
        t.validate();
        return t;
      }))
      .def("scratch_floats", &Selective::scratch_floats)
      .def("scan", &Selective::scan)
      .def("step", &Selective::step);
  m.def("launch_count", []() { return (int64_t)mb::launch_counter().load(); });
}
