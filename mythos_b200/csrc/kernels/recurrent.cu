// Linear recurrences with a decay per key channel: gated linear attention and the gated delta rule.
//
//   S <- diag(g_t) S;   u_t = v_t                        (gated linear attention)
//                       u_t = beta_t (v_t - S^T k_t)     (delta rule)
//   S <- S + k_t u_t^T; o_t = S^T q_t
//
// This file holds the token-by-token form, which works for every width and in both activation types
// (it is what 32-bit engines and unusual widths use), and the steps around it: projections to 32-bit
// q / k / v / log decay / beta (short convolution, silu, unit norms, decays), the convolution state,
// and the per-head output norm with its gate. The columns of S belong to value channels and are
// independent, so a warp owns a few of them (rows of S^T, lanes across the key channels).
#include "common.cuh"
#include "hybrid_api.h"
#include "hybrid_dev.cuh"
#include "host_util.h"

namespace mb {
namespace {

struct PrepOut {
  float *q, *k, *v, *lg, *beta;   // [rows, G, dim] x 2, [rows, H, vdim], [rows, H, dim], [rows, H]
};

// Input of channel c (within the concatenated q | k | v channels) j tokens before local token i.
template <typename T>
__device__ __forceinline__ float conv_tap(const T* __restrict__ col, long long ld, long long row, int i, int j,
                                          const float* __restrict__ st, int channels, int taps, int c) {
  if (i - j >= 0) return ldf(col + (row - j) * ld);
  return st ? st[(long long)(taps - 1 + i - j) * channels + c] : 0.f;
}

template <typename T>
__device__ __forceinline__ float conv_silu(const RecurrentSpec& s, const RecurrentInputs& in, const T* proj, long long row,
                                           int i, const float* st, int channels, int c, int col) {
  if (s.taps <= 0) return ldf(proj + row * in.ld + col);
  float a = 0.f;
  const float* w = in.conv_w + (long long)c * s.taps;
  for (int j = 0; j < s.taps; ++j)
    a = fmaf(w[s.taps - 1 - j], conv_tap(proj + col, in.ld, row, i, j, st, channels, s.taps, c), a);
  return silu_f(a);
}

// One CTA per token.
template <typename T>
__global__ void __launch_bounds__(256)
recurrent_prep_kernel(RecurrentSpec s, RecurrentInputs in, RaggedBatch rb, PrepOut out) {
  extern __shared__ float sm[];   // q then k of the token, after convolution
  const long long row = blockIdx.x;
  const int b = rb.row_seq[row];
  const int i = (int)row - rb.cu_q[b];
  const int base = rb.kv_lens[b] - (rb.cu_q[b + 1] - rb.cu_q[b]);
  const int cq = s.kv_heads * s.dim, cv = s.heads * s.vdim, channels = 2 * cq + cv;
  const T* proj = static_cast<const T*>(in.proj);
  const float* st = (base > 0 && s.taps > 1) ? in.conv_state + (long long)rb.slots[b] * (s.taps - 1) * channels : nullptr;
  for (int c = threadIdx.x; c < 2 * cq; c += blockDim.x) {
    const int col = c < cq ? in.q_off + c : in.k_off + c - cq;
    sm[c] = conv_silu(s, in, proj, row, i, st, channels, c, col);
  }
  for (int c = threadIdx.x; c < cv; c += blockDim.x)
    out.v[row * cv + c] = conv_silu(s, in, proj, row, i, st, channels, 2 * cq + c, in.v_off + c);
  for (int c = threadIdx.x; c < s.heads * s.dim; c += blockDim.x) {
    const float z = in.z[row * in.ldz + c] + in.z_bias[c];
    out.lg[row * s.heads * s.dim + c] =
        s.decay_kind == 1 ? -expf(in.a_log[c / s.dim]) * softplus_f(z) : -softplus_f(-z) * s.inv_tau;
  }
  if (s.delta)
    for (int h = threadIdx.x; h < s.heads; h += blockDim.x)
      out.beta[row * s.heads + h] = sigmoid_f(ldf(proj + row * in.ld + in.b_off + h));
  __syncthreads();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
  for (int g = warp; g < 2 * s.kv_heads; g += nw) {
    const float* x = sm + g * s.dim;
    float r = 1.f;
    if (s.unit_norm) {
      float ss = 0.f;
      for (int c = lane; c < s.dim; c += 32) ss += x[c] * x[c];
      r = 1.f / sqrtf(warp_sum(ss) + 1e-6f);
    }
    const bool is_q = g < s.kv_heads;
    if (is_q) r *= s.q_scale;
    float* dst = is_q ? out.q + row * cq + g * s.dim : out.k + row * cq + (g - s.kv_heads) * s.dim;
    for (int c = lane; c < s.dim; c += 32) dst[c] = x[c] * r;
  }
}

// grid (sequence, head, value block); a warp owns R rows of S^T in registers, lane l holds key channels
// l, l + 32, ...
constexpr int RS_WARPS = 4, RS_R = 4;
template <int NI>
__global__ void __launch_bounds__(RS_WARPS * 32)
recurrent_scan_seq_kernel(RecurrentSpec s, RaggedBatch rb, PrepOut in, float* __restrict__ state, float* __restrict__ o) {
  const int b = blockIdx.x, h = blockIdx.y;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int v0 = (blockIdx.z * RS_WARPS + warp) * RS_R;
  if (v0 >= s.vdim) return;
  const int r0 = rb.cu_q[b], r1 = rb.cu_q[b + 1];
  if (r0 >= r1) return;
  const bool fresh = rb.kv_lens[b] == r1 - r0;
  const int g = h / (s.heads / s.kv_heads);
  float* stp = state + (((long long)rb.slots[b] * s.heads + h) * s.vdim + v0) * s.dim;
  float S[RS_R][NI];
#pragma unroll
  for (int r = 0; r < RS_R; ++r)
#pragma unroll
    for (int n = 0; n < NI; ++n) {
      const int c = lane + 32 * n;
      S[r][n] = (!fresh && c < s.dim && v0 + r < s.vdim) ? stp[(long long)r * s.dim + c] : 0.f;
    }
  for (long long t = r0; t < r1; ++t) {
    float q[NI], k[NI], d[NI];
#pragma unroll
    for (int n = 0; n < NI; ++n) {
      const int c = lane + 32 * n;
      const bool ok = c < s.dim;
      q[n] = ok ? in.q[(t * s.kv_heads + g) * s.dim + c] : 0.f;
      k[n] = ok ? in.k[(t * s.kv_heads + g) * s.dim + c] : 0.f;
      d[n] = ok ? expf(in.lg[(t * s.heads + h) * s.dim + c]) : 0.f;
    }
    float u[RS_R];
#pragma unroll
    for (int r = 0; r < RS_R; ++r) {
      u[r] = v0 + r < s.vdim ? in.v[(t * s.heads + h) * s.vdim + v0 + r] : 0.f;
#pragma unroll
      for (int n = 0; n < NI; ++n) S[r][n] *= d[n];
    }
    if (s.delta) {
      const float beta = in.beta[t * s.heads + h];
#pragma unroll
      for (int r = 0; r < RS_R; ++r) {
        float a = 0.f;
#pragma unroll
        for (int n = 0; n < NI; ++n) a = fmaf(S[r][n], k[n], a);
        u[r] = beta * (u[r] - warp_sum(a));
      }
    }
#pragma unroll
    for (int r = 0; r < RS_R; ++r) {
      float a = 0.f;
#pragma unroll
      for (int n = 0; n < NI; ++n) {
        S[r][n] = fmaf(k[n], u[r], S[r][n]);
        a = fmaf(S[r][n], q[n], a);
      }
      a = warp_sum(a);
      if (lane == 0 && v0 + r < s.vdim) o[(t * s.heads + h) * s.vdim + v0 + r] = a;
    }
  }
#pragma unroll
  for (int r = 0; r < RS_R; ++r)
#pragma unroll
    for (int n = 0; n < NI; ++n) {
      const int c = lane + 32 * n;
      if (c < s.dim && v0 + r < s.vdim) stp[(long long)r * s.dim + c] = S[r][n];
    }
}

// One thread per (sequence, channel): the last taps - 1 inputs of the sequence become the state.
template <typename T>
__global__ void conv_state_kernel(RecurrentSpec s, RecurrentInputs in, RaggedBatch rb) {
  const int cq = s.kv_heads * s.dim, channels = 2 * cq + s.heads * s.vdim;
  const int c = blockIdx.x * blockDim.x + threadIdx.x, b = blockIdx.y;
  if (c >= channels) return;
  const int r0 = rb.cu_q[b], len = rb.cu_q[b + 1] - r0, n = s.taps - 1;
  if (len <= 0) return;
  const bool fresh = rb.kv_lens[b] == len;
  const int col = c < cq ? in.q_off + c : (c < 2 * cq ? in.k_off + c - cq : in.v_off + c - 2 * cq);
  float* st = in.conv_state + (long long)rb.slots[b] * n * channels + c;
  const T* proj = static_cast<const T*>(in.proj) + col;
  // entry j holds the input of token len - n + j; an entry moves down, never up, so in-place order is safe
  for (int j = 0; j < n; ++j) {
    const int i = len - n + j;
    float v;
    if (i >= 0) v = ldf(proj + (long long)(r0 + i) * in.ld);
    else v = fresh ? 0.f : st[(long long)(n + i) * channels];
    st[(long long)j * channels] = v;
  }
}

template <typename T>
__device__ __forceinline__ void ld4(const T* p, float (&f)[4]) {
  if constexpr (sizeof(T) == 4) {
    const float4 v = *reinterpret_cast<const float4*>(p);
    f[0] = v.x; f[1] = v.y; f[2] = v.z; f[3] = v.w;
  } else {
    const uint2 v = *reinterpret_cast<const uint2*>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&v.x));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&v.y));
    f[0] = a.x; f[1] = a.y; f[2] = b.x; f[3] = b.y;
  }
}
template <typename T>
__device__ __forceinline__ void st4(T* p, const float (&f)[4]) {
  if constexpr (sizeof(T) == 4) {
    *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]);
  } else {
    const __nv_bfloat162 a = __floats2bfloat162_rn(f[0], f[1]), b = __floats2bfloat162_rn(f[2], f[3]);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
  }
}

// The same for value widths up to 128 that are multiples of 4: four channels per lane, one pass.
template <typename T>
__global__ void __launch_bounds__(256)
head_norm_gate4_kernel(RecurrentSpec s, const float* __restrict__ o, const float* __restrict__ gamma,
                       const T* __restrict__ gate, long long ld_gate, T* __restrict__ out, long long ldo, long long rows) {
  const int lane = threadIdx.x & 31, nw = (int)(gridDim.x * (blockDim.x >> 5));
  const bool on = lane * 4 < s.vdim;
  float g[4] = {};
  if (on) ld4(gamma + lane * 4, g);
  const long long total = rows * s.heads;
  for (long long w = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5); w < total; w += nw) {
    const long long t = w / s.heads;
    const int h = (int)(w % s.heads);
    float x[4] = {}, z[4] = {};
    if (on) {
      ld4(o + w * s.vdim + lane * 4, x);
      ld4(gate + t * ld_gate + h * s.vdim + lane * 4, z);
    }
    const float r = 1.f / sqrtf(warp_sum(x[0] * x[0] + x[1] * x[1] + x[2] * x[2] + x[3] * x[3]) / (float)s.vdim + s.eps);
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const float e = __fdividef(1.f, 1.f + __expf(-z[j]));
      x[j] *= r * g[j] * (s.gate_kind == 1 ? e : z[j] * e);
    }
    if (on) st4(out + t * ldo + h * s.vdim + lane * 4, x);
  }
}

// One warp per (token, head).
template <typename T>
__global__ void head_norm_gate_kernel(RecurrentSpec s, const float* __restrict__ o, const float* __restrict__ gamma,
                                      const T* __restrict__ gate, long long ld_gate, T* __restrict__ out, long long ldo,
                                      long long rows) {
  const int lane = threadIdx.x & 31;
  const long long w = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (w >= rows * s.heads) return;
  const long long t = w / s.heads;
  const int h = (int)(w % s.heads);
  const float* x = o + w * s.vdim;
  float ss = 0.f;
  for (int i = lane; i < s.vdim; i += 32) ss += x[i] * x[i];
  const float r = 1.f / sqrtf(warp_sum(ss) / (float)s.vdim + s.eps);
  const T* gp = gate + t * ld_gate + h * s.vdim;
  T* op = out + t * ldo + h * s.vdim;
  for (int i = lane; i < s.vdim; i += 32) {
    const float z = ldf(gp + i);
    stf(op + i, x[i] * r * gamma[i] * (s.gate_kind == 1 ? sigmoid_f(z) : silu_f(z)));
  }
  if (h == s.heads - 1)
    for (long long i = (long long)s.heads * s.vdim + lane; i < ldo; i += 32) stf(out + t * ldo + i, 0.f);
}

// sum_r x[r] w[r] of one output channel, x in shared memory (fp32), w a row in the activation type.
template <typename T>
__device__ __forceinline__ float low_rank_dot(const float* x, const T* w, int rank) {
  float a = 0.f;
  int i = 0;
  if constexpr (sizeof(T) == 2) {
    for (; i + 8 <= rank; i += 8) {
      float f[8];
      unpack8(ldg8(w, i), f);
#pragma unroll
      for (int j = 0; j < 8; ++j) a = fmaf(f[j], x[i + j], a);
    }
  }
  for (; i < rank; ++i) a = fmaf(ldf(w + i), x[i], a);
  return a;
}

// grid (head, sequence), RD_THREADS threads; one token per sequence.
constexpr int RD_THREADS = 256, RD_R = 4;
template <typename T, int NI>
__global__ void __launch_bounds__(RD_THREADS)
recurrent_decode_kernel(RecurrentSpec s, RecurrentInputs in, RaggedBatch rb, DecodeLowRank a, DecodeLowRank g2,
                        const float* __restrict__ gamma, const T* __restrict__ gate, long long ld_gate,
                        T* __restrict__ out, long long ldo, bool own_conv) {
  extern __shared__ float sm[];   // q, k, decay [dim]; v, o [vdim]; inner products of the two low-rank maps
  __shared__ float red[32];
  const int h = blockIdx.x, b = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  constexpr int NW = RD_THREADS / 32;
  const long long row = b;
  const int slot = rb.slots[b];
  const bool fresh = rb.kv_lens[b] <= 1;
  float *q = sm, *k = q + s.dim, *d = k + s.dim, *v = d + s.dim, *o = v + s.vdim, *xa = o + s.vdim, *xg = xa + a.rank;
  const int g = h / (s.heads / s.kv_heads), cq = s.kv_heads * s.dim, channels = 2 * cq + s.heads * s.vdim;
  const T* proj = static_cast<const T*>(in.proj) + row * in.ld;
  // the state rows of the warp's first group are on their way while q, k, v and the decays are prepared,
  // those of every next group while the one before is worked on
  float* st = in.state + ((long long)slot * s.heads + h) * s.vdim * s.dim;
  float nextS[RD_R][NI];
  auto fetch = [&](int v0) {
#pragma unroll
    for (int r = 0; r < RD_R; ++r)
#pragma unroll
      for (int n = 0; n < NI; ++n) {
        const int c = lane + 32 * n;
        nextS[r][n] = (!fresh && c < s.dim && v0 + r < s.vdim) ? st[(long long)(v0 + r) * s.dim + c] : 0.f;
      }
  };
  fetch(warp * RD_R);
  for (int c = tid; c < 2 * s.dim + s.vdim; c += RD_THREADS) {
    int ch, col;
    if (c < s.dim) { ch = g * s.dim + c; col = in.q_off + ch; }
    else if (c < 2 * s.dim) { ch = cq + g * s.dim + c - s.dim; col = in.k_off + ch - cq; }
    else { ch = 2 * cq + h * s.vdim + c - 2 * s.dim; col = in.v_off + ch - 2 * cq; }
    float y = ldf(proj + col);
    if (s.taps > 0) {
      const float* w = in.conv_w + (long long)ch * s.taps;
      float acc = w[s.taps - 1] * y, x = y;
      if (s.taps > 1) {
        float* st = in.conv_state + (long long)slot * (s.taps - 1) * channels + ch;
        if (s.taps == 4) {                            // all loads before the stores
          float old[3];
#pragma unroll
          for (int j = 0; j < 3; ++j) old[j] = fresh ? 0.f : st[(long long)j * channels];
#pragma unroll
          for (int j = 0; j < 3; ++j) acc = fmaf(w[j], old[j], acc);
          if (own_conv) {
            st[0] = old[1];
            st[channels] = old[2];
            st[2ll * channels] = x;
          }
        } else {
          float nxt = x;                              // newest first: entry j moves to j - 1
          for (int j = s.taps - 2; j >= 0; --j) {
            const float old = fresh ? 0.f : st[(long long)j * channels];
            acc = fmaf(w[j], old, acc);
            if (own_conv) st[(long long)j * channels] = nxt;
            nxt = old;
          }
        }
      }
      y = silu_f(acc);
    }
    sm[c < 2 * s.dim ? c : c + s.dim] = y;            // q | k, then past the decay: v
  }
  if (!in.z)
    for (int i = tid; i < a.rank; i += RD_THREADS) xa[i] = ldf(proj + a.off + i);
  if (!gate)
    for (int i = tid; i < g2.rank; i += RD_THREADS) xg[i] = ldf(proj + g2.off + i);
  __syncthreads();
  for (int c = tid; c < s.dim; c += RD_THREADS) {
    const int ch = h * s.dim + c;
    const float z = in.z_bias[ch] + (in.z ? in.z[row * in.ldz + ch]
                                          : low_rank_dot(xa, static_cast<const T*>(a.w) + ch * a.ld, a.rank));
    d[c] = expf(s.decay_kind == 1 ? -expf(in.a_log[h]) * softplus_f(z) : -softplus_f(-z) * s.inv_tau);
  }
  if (warp >= NW - 2) {                               // unit norms on the last two warps
    float* x = warp == NW - 2 ? q : k;
    float r = 1.f;
    if (s.unit_norm) {
      float ss = 0.f;
      for (int c = lane; c < s.dim; c += 32) ss += x[c] * x[c];
      r = 1.f / sqrtf(warp_sum(ss) + 1e-6f);
    }
    if (warp == NW - 2) r *= s.q_scale;
    for (int c = lane; c < s.dim; c += 32) x[c] *= r;
  }
  const float beta = s.delta ? sigmoid_f(ldf(proj + in.b_off + h)) : 1.f;
  __syncthreads();
  float qr[NI], kr[NI], dr[NI];
#pragma unroll
  for (int n = 0; n < NI; ++n) {
    const int c = lane + 32 * n;
    const bool ok = c < s.dim;
    qr[n] = ok ? q[c] : 0.f;
    kr[n] = ok ? k[c] : 0.f;
    dr[n] = ok ? d[c] : 0.f;
  }
  for (int v0 = warp * RD_R; v0 < s.vdim; v0 += NW * RD_R) {
    float S[RD_R][NI];
#pragma unroll
    for (int r = 0; r < RD_R; ++r)
#pragma unroll
      for (int n = 0; n < NI; ++n) S[r][n] = nextS[r][n];
    if (v0 + NW * RD_R < s.vdim) fetch(v0 + NW * RD_R);
    float u[RD_R];
#pragma unroll
    for (int r = 0; r < RD_R; ++r) {
      float acc = 0.f;
#pragma unroll
      for (int n = 0; n < NI; ++n) {
        S[r][n] *= dr[n];
        acc = fmaf(S[r][n], kr[n], acc);
      }
      u[r] = v0 + r < s.vdim ? v[v0 + r] : 0.f;
      if (s.delta) u[r] = beta * (u[r] - warp_sum(acc));
    }
#pragma unroll
    for (int r = 0; r < RD_R; ++r) {
      float acc = 0.f;
#pragma unroll
      for (int n = 0; n < NI; ++n) {
        S[r][n] = fmaf(kr[n], u[r], S[r][n]);
        acc = fmaf(S[r][n], qr[n], acc);
      }
      acc = warp_sum(acc);
      if (lane == 0 && v0 + r < s.vdim) o[v0 + r] = acc;
    }
#pragma unroll
    for (int r = 0; r < RD_R; ++r)
#pragma unroll
      for (int n = 0; n < NI; ++n) {
        const int c = lane + 32 * n;
        if (c < s.dim && v0 + r < s.vdim) st[(long long)(v0 + r) * s.dim + c] = S[r][n];
      }
  }
  __syncthreads();
  float ss = 0.f;
  for (int i = tid; i < s.vdim; i += RD_THREADS) ss += o[i] * o[i];
  ss = block_sum(ss, red);
  const float r = 1.f / sqrtf(ss / (float)s.vdim + s.eps);
  for (int i = tid; i < s.vdim; i += RD_THREADS) {
    const int ch = h * s.vdim + i;
    const float z = gate ? ldf(gate + row * ld_gate + ch)
                         : low_rank_dot(xg, static_cast<const T*>(g2.w) + ch * g2.ld, g2.rank);
    stf(out + row * ldo + ch, o[i] * r * gamma[i] * (s.gate_kind == 1 ? sigmoid_f(z) : silu_f(z)));
  }
  if (h == s.heads - 1)
    for (long long i = (long long)s.heads * s.vdim + tid; i < ldo; i += RD_THREADS) stf(out + row * ldo + i, 0.f);
}

PrepOut carve(const RecurrentSpec& s, float* p, long long rows) {
  PrepOut o;
  o.q = p;
  o.k = o.q + rows * s.kv_heads * s.dim;
  o.v = o.k + rows * s.kv_heads * s.dim;
  o.lg = o.v + rows * s.heads * s.vdim;
  o.beta = o.lg + rows * s.heads * s.dim;
  return o;
}

void check_spec(const RecurrentSpec& s) {
  MB_REQUIRE(s.heads > 0 && s.kv_heads > 0 && s.heads % s.kv_heads == 0, "recurrent: heads must be a multiple of kv_heads");
  MB_REQUIRE(s.dim > 0 && s.dim <= 256 && s.vdim > 0, "recurrent: key width up to 256");
  MB_REQUIRE(s.taps >= 0 && s.taps <= 64, "recurrent: convolution taps out of range");
}

}  // namespace

void recurrent_scan_seq(bool f32, const RecurrentSpec& s, const RecurrentInputs& in, const RaggedBatch& rb,
                        float* scratch, float* o, cudaStream_t stream) {
  check_spec(s);
  if (rb.rows == 0) return;
  const PrepOut p = carve(s, scratch, rb.rows);
  const int smem = 2 * s.kv_heads * s.dim * 4;
  MB_REQUIRE(smem <= 200 * 1024, "recurrent: q / k of one token exceed shared memory");
  if (smem > 48 * 1024) {
    if (f32) MB_CUDA_CHECK(cudaFuncSetAttribute(recurrent_prep_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
    else MB_CUDA_CHECK(cudaFuncSetAttribute(recurrent_prep_kernel<__nv_bfloat16>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
  }
  if (f32) recurrent_prep_kernel<float><<<rb.rows, 256, smem, stream>>>(s, in, rb, p);
  else recurrent_prep_kernel<__nv_bfloat16><<<rb.rows, 256, smem, stream>>>(s, in, rb, p);
  const dim3 grid(rb.n_seq, s.heads, (s.vdim + RS_WARPS * RS_R - 1) / (RS_WARPS * RS_R));
  if (s.dim <= 32) recurrent_scan_seq_kernel<1><<<grid, RS_WARPS * 32, 0, stream>>>(s, rb, p, in.state, o);
  else if (s.dim <= 64) recurrent_scan_seq_kernel<2><<<grid, RS_WARPS * 32, 0, stream>>>(s, rb, p, in.state, o);
  else if (s.dim <= 128) recurrent_scan_seq_kernel<4><<<grid, RS_WARPS * 32, 0, stream>>>(s, rb, p, in.state, o);
  else recurrent_scan_seq_kernel<8><<<grid, RS_WARPS * 32, 0, stream>>>(s, rb, p, in.state, o);
  count_launch(2);
  check_launch();
}

void recurrent_decode(bool f32, const RecurrentSpec& s, const RecurrentInputs& in, const RaggedBatch& rb,
                      const DecodeLowRank& a, const DecodeLowRank& g, const float* gamma, const void* gate,
                      long long ld_gate, void* out, long long ldo, cudaStream_t stream) {
  check_spec(s);
  MB_REQUIRE(in.z || a.w, "recurrent_decode: decay pre-activations or their low-rank map");
  MB_REQUIRE(gate || g.w, "recurrent_decode: output gate or its low-rank map");
  MB_REQUIRE((!a.w || a.ld % 8 == 0) && (!g.w || g.ld % 8 == 0), "recurrent_decode: low-rank maps need 16-byte rows");
  if (rb.n_seq == 0) return;
  MB_REQUIRE(rb.rows == rb.n_seq, "recurrent_decode: one token per sequence");
  const bool own_conv = s.heads == s.kv_heads;      // otherwise several heads read one channel's convolution state
  const int smem = (3 * s.dim + 2 * s.vdim + (in.z ? 0 : a.rank) + (gate ? 0 : g.rank)) * 4;
  MB_REQUIRE(smem <= 48 * 1024, "recurrent_decode: head too wide");
  DecodeLowRank aa = a, gg = g;
  if (in.z) aa.rank = 0;
  if (gate) gg.rank = 0;
  const dim3 grid(s.heads, rb.n_seq);
#define MB_RD(T, NI)                                                                                              \
  recurrent_decode_kernel<T, NI><<<grid, RD_THREADS, smem, stream>>>(s, in, rb, aa, gg, gamma, (const T*)gate, ld_gate, \
                                                                     (T*)out, ldo, own_conv)
  if (f32) {
    if (s.dim <= 32) MB_RD(float, 1); else if (s.dim <= 64) MB_RD(float, 2); else if (s.dim <= 128) MB_RD(float, 4);
    else MB_RD(float, 8);
  } else {
    if (s.dim <= 32) MB_RD(__nv_bfloat16, 1); else if (s.dim <= 64) MB_RD(__nv_bfloat16, 2);
    else if (s.dim <= 128) MB_RD(__nv_bfloat16, 4); else MB_RD(__nv_bfloat16, 8);
  }
#undef MB_RD
  count_launch();
  check_launch();
  if (!own_conv) conv_state_update(f32, s, in, rb, stream);
}

void conv_state_update(bool f32, const RecurrentSpec& s, const RecurrentInputs& in, const RaggedBatch& rb,
                       cudaStream_t stream) {
  if (s.taps <= 1 || rb.n_seq == 0) return;
  const int channels = 2 * s.kv_heads * s.dim + s.heads * s.vdim;
  const dim3 grid((channels + 255) / 256, rb.n_seq);
  if (f32) conv_state_kernel<float><<<grid, 256, 0, stream>>>(s, in, rb);
  else conv_state_kernel<__nv_bfloat16><<<grid, 256, 0, stream>>>(s, in, rb);
  count_launch();
  check_launch();
}

void head_norm_gate(bool f32, const RecurrentSpec& s, const float* o, const float* gamma, const void* gate,
                    long long ld_gate, void* out, long long ldo, int rows, cudaStream_t stream) {
  if (rows == 0) return;
  const int grid = ceil_div((long long)rows * s.heads, 8);
  if (!f32 && s.vdim <= 128 && s.vdim % 4 == 0 && ld_gate % 4 == 0 && ldo == (long long)s.heads * s.vdim &&
      (reinterpret_cast<uintptr_t>(gate) & 7) == 0) {
    const int cap = sm_count() * 16;
    head_norm_gate4_kernel<__nv_bfloat16><<<grid < cap ? grid : cap, 256, 0, stream>>>(
        s, o, gamma, (const __nv_bfloat16*)gate, ld_gate, (__nv_bfloat16*)out, ldo, rows);
    count_launch();
    check_launch();
    return;
  }
  if (f32)
    head_norm_gate_kernel<float><<<grid, 256, 0, stream>>>(s, o, gamma, (const float*)gate, ld_gate, (float*)out, ldo, rows);
  else
    head_norm_gate_kernel<__nv_bfloat16><<<grid, 256, 0, stream>>>(s, o, gamma, (const __nv_bfloat16*)gate, ld_gate,
                                                                   (__nv_bfloat16*)out, ldo, rows);
  count_launch();
  check_launch();
}

}  // namespace mb
