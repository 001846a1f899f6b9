// Launch API of the kernels behind layer-list ("hybrid") models: gated linear attention and gated
// delta-rule recurrences, attention with unequal key / value widths and per-head output gates,
// sandwich RMSNorms on a 32-bit residual stream, and the GEMMs those models need beside gemm.cu.
// Same conventions as api.h (raw pointers, asynchronous on `stream`, exceptions on bad arguments).
// `f32` selects the activation type: false = bf16 (serving), true = 32-bit floats throughout.
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

namespace mb {

// A ragged batch of new tokens: sequence b owns rows cu_q[b] .. cu_q[b+1]; kv_lens[b] counts its
// tokens including the new ones; slots[b] is its state slot; row_seq[t] = b; pos[t] = position.
struct RaggedBatch {
  const int *cu_q, *kv_lens, *slots, *row_seq, *pos;
  int n_seq, rows;
};

// x[t] = embed[id] * scale + pos_table[pos] (fp32 stream), h[t] = rmsnorm(x[t]) * gamma.
void embed_pos_norm(bool f32, const int* ids, const int* pos, const void* embed, const void* pos_table, int vocab,
                    int max_pos, float scale, const float* gamma, float* x, void* h, long long ldh, int rows, int dim,
                    float eps, cudaStream_t stream);

// y = y1, or with y2: (rms(y1) * w1 + rms(y2) * w2) / 2.  x += rms(y) * w_post;  h = rms(x) * w_next.
void sandwich_norm(bool f32, const void* y1, const void* y2, long long ldy, const float* w1, const float* w2,
                   const float* w_post, float* x, const float* w_next, void* h, long long ldh, int rows, int dim,
                   float eps, cudaStream_t stream);

// Per-head RMSNorm of q and k, q written out, k and v stored into their pages (key width dk, value width dv).
void qk_norm_append(bool f32, const void* proj, long long ld, int q_off, int k_off, int v_off, const float* q_gamma,
                    const float* k_gamma, const RaggedBatch& rb, const int* block_table, int table_stride,
                    int page_size, void* q_out, void* k_cache, void* v_cache, int heads, int kv_heads, int dk, int dv,
                    float eps, cudaStream_t stream);

// Causal attention of every new token over its sequence's pages, any widths, 32-bit arithmetic.
// gate (may be null): logits [rows, heads] with row stride ld_gate; head h is multiplied by sigmoid(gate[t, h]).
// block_table row b belongs to sequence b of the batch.
void paged_attn_any(bool f32, const void* q, const void* k_cache, const void* v_cache, const RaggedBatch& rb,
                    const int* block_table, int table_stride, int page_size, const void* gate, long long ld_gate,
                    void* o, long long ldo, int heads, int kv_heads, int dk, int dv, float scale, cudaStream_t stream);

// C[M, N] = alpha * A[M, K] B[N, K]^T, all fp32, no reduced-precision mode.
void gemm_f32(const float* A, long long lda, const float* B, long long ldb, float* C, long long ldc, int M, int N,
              int K, float alpha, cudaStream_t stream);

// y = alpha * x W^T for a few tokens (bf16 in, bf16 or fp32 out), reduction split over a cluster. f_off > 0: W holds
// a gate matrix in rows [0, N) and an up matrix from row f_off; y = silu(gate) * up.
void gemm_decode(const void* x, long long ldx, const void* W, long long ldw, void* out, bool out_f32, long long ldo, int M,
                 int N, int K, int f_off, float alpha, int* status, cudaStream_t stream);

// h = silu(gu[:, :f]) * gu[:, f_off : f_off + f]
void silu_gate(bool f32, const void* gu, long long ldg, int f, int f_off, void* h, long long ldh, int rows,
               cudaStream_t stream);

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
// out = rms_over_vdim(o) * gamma * act(gate)
void head_norm_gate(bool f32, const RecurrentSpec& s, const float* o, const float* gamma, const void* gate,
                    long long ld_gate, void* out, long long ldo, int rows, cudaStream_t stream);

}  // namespace mb
