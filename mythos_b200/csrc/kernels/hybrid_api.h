// Launch API of the kernels behind layer-list ("hybrid") models: gated linear attention and gated
// delta-rule recurrences, selective scans, attention with unequal key / value widths, windows, sinks and output
// gates, attention over a cached latent, routed experts, RMSNorms around sublayers on a 32-bit residual stream, and the
// GEMMs those models need beside gemm.cu.
// Same conventions as api.h (raw pointers, asynchronous on `stream`, exceptions on bad arguments).
// `f32` selects the activation type: false = bf16 (serving), true = 32-bit floats throughout.
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

namespace mb {

struct AttnExtras;   // api.h

// A ragged batch of new tokens: sequence b owns rows cu_q[b] .. cu_q[b+1]; kv_lens[b] counts its
// tokens including the new ones; slots[b] is its state slot; row_seq[t] = b; pos[t] = position.
struct RaggedBatch {
  const int *cu_q, *kv_lens, *slots, *row_seq, *pos;
  int n_seq, rows;
};

// ---- short causal convolution per channel (short_conv.cu): y = silu(conv(x) + bias), or residual: x + conv(x) + bias
struct ShortConv {
  int channels, taps;
  bool residual;
  const float *w, *bias;            // [taps, channels] (last row: the current token's), [channels] or null
  float* state;                     // [slots][taps - 1][channels] last inputs of every sequence
};
// A ragged batch; columns [channels, ldy) are zeroed and the state advances. one_token: row b belongs to sequence b.
void short_conv(bool f32, const ShortConv& s, const void* x, long long ldx, const RaggedBatch& rb, bool one_token, void* y,
                long long ldy, cudaStream_t stream);

// Where a kernel that writes a normalised row h of one token per sequence also writes h + conv(h): c.taps 0: nowhere.
struct ConvTail {
  ShortConv c;
  const int *slots, *kv_lens;
  void* out;
  long long ld;
};

// x[t] = embed[id] * scale + pos_table[pos] (fp32 stream; the table may be null), with gamma0 normalised,
// h[t] = rmsnorm(x[t]) * gamma, or x[t] with gamma null.
void embed_pos_norm(bool f32, const int* ids, const int* pos, const void* embed, const void* pos_table, int vocab,
                    int max_pos, float scale, const float* gamma0, const float* gamma, float* x, void* h, long long ldh,
                    int rows, int dim, float eps, const ConvTail& conv, cudaStream_t stream);

// x += mult * (y + bias) (bias may be null);  h = rms(x) * w_next.
void residual_norm(bool f32, const void* y, long long ldy, const float* bias, float mult, float* x, const float* w_next, void* h,
                   long long ldh, int rows, int dim, float eps, const ConvTail& conv, cudaStream_t stream);

// out = a N(z) + b N(z^2) + c N(z^3) + e with z = y + bias and abce = {a, b, c, e}, N dividing a row by its root mean
// square over the `width` columns; columns [width, ldo) of out are zeroed.
void poly_norm(bool f32, const void* y, long long ldy, const float* bias, const float* abce, void* out, long long ldo, int rows,
               int width, int padded, float eps, cudaStream_t stream);

// y[t, n] *= sigmoid(gate[t, n])
void sigmoid_mul(bool f32, void* y, long long ldy, const void* gate, long long ld_gate, int rows, int width, cudaStream_t stream);

// Output of a sublayer: y1 alone; (rms(y1) * w1 + rms(y2) * w2) / 2; or the sum over j < top of
// weight[t, j] * y1[row[t, j]] (routed experts), plus y2[t] if there is one (their shared expert).
struct SublayerOut {
  const void *y1, *y2;
  long long ld;
  const float *w1, *w2;
  const int* row;
  const float* weight;
  int top;
};
// x += mult * rms(y) * w_post;  h = rms(x) * w_next, or x with w_next null.
void sandwich_norm(bool f32, const SublayerOut& y, const float* w_post, float mult, float* x, const float* w_next, void* h,
                   long long ldh, int rows, int dim, float eps, cudaStream_t stream);

// How projected heads become queries, keys and values: bias, RMS norm of every q and k head, rotation, query
// temperature. q [rows, heads, dk] is written out, k and v go to their pages; v may be the same columns as k (it is neither
// normalised nor rotated). dk and dv are the stored widths;
// columns past a head's true width are zero in the projection and stay zero.
struct HeadPrep {
  int heads, kv_heads, dk, dv;
  int q_off, k_off, v_off;          // columns of the projection; k_off < 0: queries only
  const float *q_bias, *k_bias, *v_bias;      // [heads * dk], [kv_heads * dk], [kv_heads * dv], or null
  int norm_dim;                     // columns the norm averages over; 0: no norm
  const float *q_gamma, *k_gamma;   // [dk] norm weights, or null
  const double* turns;              // revolutions per position of the pair (i, i + rot / 2), or (2i, 2i + 1) with pairs
  int rot;                          // rotated columns (0: none)
  bool pairs;
  float rot_amp;                    // factor of cosines and sines
  float temp_coef, temp_every;      // queries times 1 + coef ln(floor((pos + 1) / every) + 1); coef 0: none
  float eps;
};
void attn_prep(bool f32, const void* proj, long long ld, const HeadPrep& p, const RaggedBatch& rb, const int* block_table,
               int table_stride, int page_size, void* q_out, void* k_cache, void* v_cache, cudaStream_t stream);

// Causal attention of every new token over its sequence's pages, any widths, 32-bit arithmetic. The gate of `ex` is in
// the activation type. block_table row b belongs to sequence b of the batch.
void paged_attn_any(bool f32, const void* q, const void* k_cache, const void* v_cache, const RaggedBatch& rb,
                    const int* block_table, int table_stride, int page_size, const AttnExtras& ex, void* o, long long ldo,
                    int heads, int kv_heads, int dk, int dv, float scale, cudaStream_t stream);

// Segments of rows that meet a weight matrix each: tiles[i] = (matrix, first row, rows), *count of them.
struct TileList {
  const int *tiles, *count;
  int max_tiles;
};

// C[M, N] = alpha * A[M, K] B[N, K]^T, all fp32, no reduced-precision mode. batch > 1: that many products, the
// operands of each `*_batch` elements further. With `list` (64-row tiles) row segments meet the matrix they name.
void gemm_f32(const float* A, long long lda, const float* B, long long ldb, float* C, long long ldc, int M, int N,
              int K, float alpha, cudaStream_t stream, int batch = 1, long long a_batch = 0, long long b_batch = 0,
              long long c_batch = 0, const TileList* list = nullptr);

// Gated feed-forward activations: what a gate value g does to its up value u.
struct GateAct {
  int kind;                 // 0: silu(g) u   1: relu(g) u   2: g' sigmoid(alpha g') (u' + 1) with g' = min(g, limit),
  float limit, alpha;       //    u' = u clamped to [-limit, limit]
};
// What a few-token GEMM does with the products of a row: nothing; a gated activation of two halves of W;
// gelu_tanh(y) * mul[mul_ids[t] * ld_mul + n]; a soft cap; or y * sigmoid(gate[t * ld_gate + n]), in product b of a batch
// + b * gate_batch.
struct GemmTail {
  int f_off;                // > 0: W holds a gate matrix in rows [0, N) and an up matrix from row f_off
  GateAct act;
  const void* mul;
  const int* mul_ids;
  long long ld_mul;
  int vocab;                // rows of mul
  float cap;                // > 0: y <- cap tanh(y / cap)
  const void* gate;
  long long ld_gate, gate_batch;
};
// Several products in one launch: `batch` of them side by side (x, W and out advance by *_batch elements), or with
// `list` (tile rows = mt: 16, 32, 64 or 128) rows grouped by matrix, W advancing by w_batch elements.
struct GemmGroup {
  int batch;
  long long x_batch, w_batch, out_batch;
  const TileList* list;
  int mt;
};
// y = alpha * x W^T for a few tokens (bf16 in, bf16 or fp32 out), reduction split over a cluster.
void gemm_decode(const void* x, long long ldx, const void* W, long long ldw, void* out, bool out_f32, long long ldo, int M,
                 int N, int K, float alpha, const GemmTail& tail, const GemmGroup& group, int* status, cudaStream_t stream);

// The same products for prompt-sized row segments: persistent 128-token x 256-weight-row tiles (128 of each half with
// a gated tail), bf16 out. `list` has 128-row tiles; total_rows: rows of x.
void gemm_segments(const void* x, long long ldx, const void* W, long long ldw, long long w_batch, int matrices, void* out,
                   long long ldo, int total_rows, int N, int K, const GemmTail& tail, const TileList& list, int* status,
                   cudaStream_t stream);

// h = act(gu[:, :f], gu[:, f_off : f_off + f])
void gate_pair(bool f32, const void* gu, long long ldg, int f, int f_off, const GateAct& act, void* h, long long ldh, int rows,
               cudaStream_t stream);
// y[t, n] = gelu_tanh(y[t, n]) * table[ids[t] * ld_table + n], n < width
void gelu_mul(bool f32, void* y, long long ldy, const void* table, long long ld_table, const int* ids, int vocab, int rows,
              int width, cudaStream_t stream);

// y[t, n] = cap * tanh(y[t, n] / cap) in place, n < width
void soft_cap(float* y, long long ldy, int rows, int width, float cap, cudaStream_t stream);

// ---- routed experts (expert_route.cu)
struct RouterSpec {
  int experts, top, groups, keep;
  int sigmoid;              // scores: 0 softmax over all experts, 1 sigmoid of each logit
  int group_best;           // a group counts the sum of its 1 or 2 largest choice scores
  int normalise;            // 1: the chosen scores are divided by their sum (+ 1e-20) and multiplied by scale
  float scale;
};
struct RouterBuffers {
  int* idx;                 // [rows, top] chosen expert
  float* weight;            // [rows, top] its score, normalised if the router says so
  int* slot;                // [rows, top] place within the expert's segment
  int* counts;              // [experts + 1], zero before the first launch and left zero by every launch
  int* offset;              // [experts] first row of the segment
  int *tiles, *tile_count;  // tile list for `tile_rows` rows a tile
  int max_tiles;
};
// Scores of fp32 logits, choice by score + correction (may be null) within the best groups, row segments per expert.
void expert_select(const float* logits, long long ldz, const float* correction, const RouterSpec& s, const RouterBuffers& b,
                   int tile_rows, int rows, cudaStream_t stream);
// Rows of h (row_bytes each, a multiple of 16) into their segments; row[t, j] = where (t, j) went.
void expert_gather(const void* h, long long ldh_bytes, const RouterSpec& s, const RouterBuffers& b, void* out, int* row,
                   long long row_bytes, int rows, cudaStream_t stream);

// ---- attention over a cached latent (latent.cu): a page row holds [latent | rotated key part], each padded to a
// multiple of 8 values with zeros; all heads read the same rows.
struct LatentSpec {
  int heads, rank, rot, rank_p, rot_p;   // widths and their padded forms
  int window;                            // keys a query sees, its own included (0: all earlier ones)
  float rot_amp;                         // factor of cosines and sines
  __host__ __device__ int row() const { return rank_p + rot_p; }
};
struct LatentPages {
  void* cache;              // [pages, page_size, row]
  const int* table;
  int stride, page_size, pages;
};
// Columns of a projection, each part left out with a negative offset: vectors that queries are a map of (low_off: RMS
// norm over low_rank columns in place), the queries' rotated columns (qr_off: rotated in place), latent (c_off: RMS norm) and
// rotated key part (kr_off: rotation), which go to the pages. Columns 2i and 2i + 1 are a pair, turns[i] its revolutions
// per position.
struct LatentPrep {
  int low_off, low_rank, qr_off, c_off, kr_off;
  const float *low_gamma, *gamma;
  const double* turns;
};
void latent_prep(bool f32, void* proj, long long ld, const LatentPrep& p, const LatentSpec& s, const RaggedBatch& rb,
                 const LatentPages& pg, float eps, cudaStream_t stream);
// Latent rows of the sequences' pages, packed: sequence b, from its token first[b] on, at rows cu_k[b] .. cu_k[b + 1] of out.
void latent_gather(const LatentSpec& s, const LatentPages& pg, const int* cu_k, const int* first, int n_seq, int max_kv, void* out,
                   cudaStream_t stream);
// Queries of single tokens: q_lat [rows, heads, rank_p] (unrotated part taken into the latent's space) and the rotated
// part at qr + t * ld_qr + h * rot_p; token t sees positions up to pos[t] of sequence row_seq[t].
struct LatentQuery {
  const void* q_lat;
  const void* qr;
  long long ld_qr;
  const int *row_seq, *pos;
  int rows;
};
// out [rows, heads, rank_p]: softmax-weighted latents, with exp(sink[h]) in the denominator (sink may be null).
void latent_attn_any(bool f32, const LatentQuery& q, const LatentSpec& s, const LatentPages& pg, const float* sink, void* out,
                     float scale, cudaStream_t stream);
bool latent_decode_ok(const LatentSpec& s, int page_size);
// scratch: rows * heads * splits * (rank_p + 4) floats (none with one split).
void latent_attn_decode(const LatentQuery& q, const LatentSpec& s, const LatentPages& pg, const float* sink, void* out,
                        float* scratch, int splits, float scale, int* status, cudaStream_t stream);

// ---- recurrences: S <- diag(g) S ; u = beta (v - S^T k) or u = v ; S <- S + k u^T ; o = S^T q
// State layout: [slot][head][vdim][dim] fp32 (a row of S^T is contiguous).
struct RecurrentSpec {
  int heads, kv_heads, dim, vdim;   // kv_heads: heads of q and k (a divisor of heads)
  int taps;                         // short convolution on q, k, v (0: none)
  int delta;                        // 1: delta rule (u = beta (v - S^T k)), 0: u = v
  int unit_norm;                    // 1: q and k are made unit vectors
  int decay_kind;                   // 0: sigmoid(z)^(1/tau); 1: exp(-exp(a_log_h) softplus(z))
  int gate_kind;                    // output gate: 0 silu, 1 sigmoid
  float q_scale, inv_tau, eps;
};
struct RecurrentInputs {
  const void* proj;                 // [rows, ld]: q | k | v (| beta) columns at the offsets below
  long long ld;
  int q_off, k_off, v_off, b_off;
  const float* z;                   // [rows, heads * dim] decay pre-activations without bias
  long long ldz;
  const float* z_bias;              // [heads * dim]
  const float* a_log;               // [heads] (decay_kind 1)
  const float* conv_w;              // [channels q | k | v, taps]
  float* conv_state;                // [slots][taps - 1][channels]
  float* state;                     // [slots][heads][vdim][dim]
};
// Token-by-token form (any dim / vdim): q, k, v, log decay and beta in 32-bit, then the scan. Scratch
// floats per row: 2 * kv_heads * dim + heads * (vdim + dim + 1).
void recurrent_scan_seq(bool f32, const RecurrentSpec& s, const RecurrentInputs& in, const RaggedBatch& rb,
                        float* scratch, float* o, cudaStream_t stream);
// Chunked form on tensor cores (bf16 projections, dim <= 128): same result, for prompts and portions.
bool recurrent_chunked_ok(const RecurrentSpec& s);
long long recurrent_chunked_scratch(const RecurrentSpec& s, int rows, int n_seq);   // bytes
void recurrent_scan_chunked(const RecurrentSpec& s, const RecurrentInputs& in, const RaggedBatch& rb, void* scratch,
                            float* o, int* status, cudaStream_t stream);
// One token per sequence (row b belongs to sequence b), everything in one launch: short convolution and its
// state, norms, decay, state update, read-out, head norm and output gate -> out [rows, ldo]. The decay
// pre-activations come from in.z, or are computed here from a1 (proj columns) and a2 [heads * dim, ld_a2];
// the gate comes from `gate`, or from g1 and g2 [heads * vdim, ld_g2].
struct DecodeLowRank {
  const void* w;        // [outputs, ld]
  long long ld;
  int off, rank;        // columns of proj that hold the inner product
};
void recurrent_decode(bool f32, const RecurrentSpec& s, const RecurrentInputs& in, const RaggedBatch& rb,
                      const DecodeLowRank& a, const DecodeLowRank& g, const float* gamma, const void* gate,
                      long long ld_gate, void* out, long long ldo, cudaStream_t stream);
// Shift the new inputs into the convolution state (after every reader of the old state has run).
void conv_state_update(bool f32, const RecurrentSpec& s, const RecurrentInputs& in, const RaggedBatch& rb,
                       cudaStream_t stream);
// ---- selective scan (selective_scan.cu), per channel c and state value n:
// S[c, n] <- exp(dt_c A[c, n]) S[c, n] + dt_c x_c B_n;  out_c = (sum_n S[c, n] C_n + D_c x_c) silu(z_c) out_scale
// with x = silu(short convolution of the projection's x columns + bias) and dt = softplus(pre-activation + bias).
struct SelectiveSpec {
  int inner, state, rank;           // channels, state values per channel, width of the map to dt
  float out_scale;
};
int selective_padded_state(int state);   // state values per channel as stored
struct SelectiveInputs {
  const void* proj;                 // [rows, ld]: z columns at the offset below
  long long ld;
  int z_off;
  const float* a;                   // [inner, padded state]: A log2(e), zero in the padding
  const float *d, *dt_bias;         // [inner]
  float* state;                     // [slots][inner][padded state]
  const void* low;                  // [rows, ld_low]: x's maps, dt columns from 0, B and C columns at the offsets below
  long long ld_low;
  int b_off, c_off;
  const void* x;                    // [rows, ld_x] the convolved channels
  long long ld_x;
};
// Prompts and portions; dt [rows, ld_dt]: pre-activations without bias. Long portions are cut into chunks that run side
// by side: a first kernel forms every chunk's own state and summed step sizes, the second starts each chunk from
// the states before it. Scratch: selective_scratch floats.
long long selective_scratch(const SelectiveSpec& s, int n_seq, int rows, int max_q);
void selective_scan(bool f32, const SelectiveSpec& s, const SelectiveInputs& in, const RaggedBatch& rb, int max_q,
                    const float* dt, long long ld_dt, float* scratch, void* out, long long ldo, int* status, cudaStream_t stream);
// One token per sequence. The pre-activations come from dt, or from the dt columns of `low` and w_dt [inner, ld_w].
void selective_step(bool f32, const SelectiveSpec& s, const SelectiveInputs& in, const RaggedBatch& rb, const float* dt,
                    long long ld_dt, const void* w_dt, long long ld_w, void* out, long long ldo, cudaStream_t stream);

// out = rms_over_vdim(o) * gamma * act(gate)
void head_norm_gate(bool f32, const RecurrentSpec& s, const float* o, const float* gamma, const void* gate,
                    long long ld_gate, void* out, long long ldo, int rows, cudaStream_t stream);

}  // namespace mb
