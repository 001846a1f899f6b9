// Chunked form of the linear recurrences (recurrent.cu has the token-by-token form and the definitions).
//
// A portion of a sequence is cut into chunks of 16 tokens. With b_t the running sum of log decays inside
// a chunk (per key channel) and S_0 the state before it,
//
//   S_0^T-part of a read-out   q~_t = q_t e^{b_t},      of a write-back  k~_t = k_t e^{b_t}
//   P[t, s] = sum_c q_t k_s e^{b_t - b_s} (s <= t),     A[t, s] = sum_c k_t k_s e^{b_t - b_s} (s < t)
//   delta rule: (I + diag(beta) A) U = diag(beta) (V - K~ S_0), so U = T (V - K~ S_0) with
//               T = (I + diag(beta) A)^{-1} diag(beta);     gated linear attention: U = V
//   O = Q~ S_0 + P U,     S_16 = diag(e^{b_16}) S_0 + K-^T U,   K-_s = k_s e^{b_16 - b_s}
//
// Everything but S_0 is local to a chunk: chunk_prep computes it for all chunks at once (one CTA per
// chunk and head) and leaves one contiguous record per chunk. chunk_scan walks the chunks of a sequence
// in order; a warp owns 16 value channels, holds its rows of S^T in fp32 registers and does the products
// with warp-level MMAs. Operands are split into a bf16 head and a bf16 tail (three products), which keeps
// the recurrence at 32-bit accuracy although the tensor cores take 16-bit operands: the state, the
// decays, the unit norms and the chunk matrices never see a plain bf16 rounding.
//
// No exponent above is positive. P and A are formed as (q e^{b_t}) (k e^{-b_s}), whose second factor grows
// with the decay inside the chunk: a channel that decays by more than e^-60 in one chunk sends the chunk to
// a pairwise evaluation instead.
#include "common.cuh"
#include "hybrid_api.h"
#include "hybrid_dev.cuh"
#include "host_util.h"
#include "tc.cuh"

#include <type_traits>

namespace mb {
namespace {

constexpr int CK = 16;            // tokens per chunk
constexpr int CS_WARPS = 4;       // scan warps per CTA
constexpr int CS_V = 16 * CS_WARPS;
// threads and resident CTAs per SM of chunk_prep by key width
__host__ __device__ constexpr int cp_threads(int dp) { return dp == 128 ? 256 : 128; }
__host__ __device__ constexpr int cp_blocks(int dp) { return dp == 128 ? 4 : 8; }

__device__ __forceinline__ void mma_bf16(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, "
               "{%0, %1, %2, %3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ldm_x4(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ldm_x4_t(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
// (x0, x1) -> bf16 pair and the bf16 pair of what it left over
__device__ __forceinline__ void split2(float x0, float x1, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16x2(x0, x1);
  const float h0 = __uint_as_float(hi << 16), h1 = __uint_as_float(hi & 0xFFFF0000u);
  lo = pack_bf16x2(x0 - h0, x1 - h1);
}

// Record of one (chunk, head). Rows of the [16][DP] matrices hold their 16-byte units in the order
// unit ^ (row & mask), so that ldmatrix reads without bank conflicts.
template <int DP, bool DELTA>
struct Rec {
  static constexpr int MAT = CK * DP * 2;
  static constexpr int Q_HI = 0, Q_LO = MAT, B_HI = 2 * MAT, B_LO = 3 * MAT;      // q~, K-
  static constexpr int K_HI = 4 * MAT, K_LO = 5 * MAT;                            // k~ (delta)
  static constexpr int P_HI = (DELTA ? 6 : 4) * MAT, P_LO = P_HI + 512;
  static constexpr int T_HI = P_LO + 512, T_LO = T_HI + 512;                      // delta
  static constexpr int DEC = DELTA ? T_LO + 512 : P_LO + 512;
  static constexpr int BYTES = DEC + DP * 4;
  static constexpr int V_BLOCK = CK * CS_V * 4;                                   // fp32 [16][64], one per 64 channels
};
template <int DP>
__device__ __forceinline__ int unit_off(int row, int unit) {   // byte offset inside a [16][DP] matrix
  constexpr int mask = DP >= 64 ? 7 : 3;
  const int x = DP >= 64 ? (row & 7) : ((row >> 1) & 3);
  return row * (DP * 2) + ((unit ^ (x & mask)) << 4);
}

// First chunk slot of sequence b: an upper bound that needs no prefix sum (ceil(n / 16) chunks always
// fit between the floors).
__device__ __forceinline__ int chunk_base(const int* cu_q, int b) { return cu_q[b] / CK + b; }

using T = __nv_bfloat16;   // projections (32-bit engines use the token-by-token form)

// Activation of the short convolution. The projections are bf16 and the convolution need not be better, so
// the fast exponential and divide will do here (unlike in the decays).
__device__ __forceinline__ float conv_act(float y) { return __fdividef(y, 1.f + __expf(-y)); }
// log(1 + e^x), small arguments of the logarithm from its series
__device__ __forceinline__ float softplus_fast(float x) {
  const float e = __expf(-fabsf(x));
  const float l = e < 0.015625f ? e * (1.f + e * (-0.5f + e * (1.f / 3.f))) : logf(1.f + e);
  return fmaxf(x, 0.f) + l;
}

// Input of a channel at local token i < 0: the convolution state, or 0 at a sequence's start.
__device__ __forceinline__ float conv_past(const float* st, int i, int taps, int channels) {
  return st && i + taps - 1 >= 0 ? st[(long long)(taps - 1 + i) * channels] : 0.f;
}

// W adjacent channels (2 when every offset is even, else 1) of the chunk's 16 tokens through the short
// convolution; `put(t, y)` takes the result. col: the channel's column of the projection; ch: its index.
template <int W, bool FULL, class Put>
__device__ __forceinline__ void conv_column(const RecurrentSpec& s, const RecurrentInputs& in, const T* __restrict__ col, int q0,
                                            int i0, int n, const float* __restrict__ st, int channels, int ch, Put put) {
  const T* p = col + (long long)(q0 + i0) * in.ld;
  float x[CK][W];
#pragma unroll
  for (int t = 0; t < CK; ++t) {
    if constexpr (W == 2) {
      float2 f = make_float2(0.f, 0.f);
      if (FULL || t < n) f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p + t * in.ld));
      x[t][0] = f.x;
      x[t][1] = f.y;
    } else {
      x[t][0] = FULL || t < n ? __bfloat162float(p[t * in.ld]) : 0.f;
    }
  }
  if (s.taps == 0) {
#pragma unroll
    for (int t = 0; t < CK; ++t) put(t, x[t]);
    return;
  }
  auto before = [&](int i, int w) {        // input i of the portion
    return i >= 0 ? __bfloat162float(col[(long long)(q0 + i) * in.ld + w]) : conv_past(st ? st + w : nullptr, i, s.taps, channels);
  };
  if (s.taps == 4) {
    float w4[4][W], h1[W], h2[W], h3[W];
#pragma unroll
    for (int w = 0; w < W; ++w) {
      h3[w] = before(i0 - 3, w);
      h2[w] = before(i0 - 2, w);
      h1[w] = before(i0 - 1, w);
#pragma unroll
      for (int j = 0; j < 4; ++j) w4[j][w] = in.conv_w[(long long)(ch + w) * 4 + j];
    }
#pragma unroll
    for (int t = 0; t < CK; ++t) {
      float y[W];
#pragma unroll
      for (int w = 0; w < W; ++w) {
        const float a = fmaf(w4[0][w], h3[w], fmaf(w4[1][w], h2[w], fmaf(w4[2][w], h1[w], w4[3][w] * x[t][w])));
        y[w] = FULL || t < n ? conv_act(a) : 0.f;
        h3[w] = h2[w];
        h2[w] = h1[w];
        h1[w] = x[t][w];
      }
      put(t, y);
    }
  } else {
    for (int t = 0; t < CK; ++t) {         // any number of taps: inputs are read again
      float y[W] = {};
      if (t < n) {
        for (int w = 0; w < W; ++w) {
          for (int j = 0; j < s.taps; ++j)
            y[w] = fmaf(in.conv_w[(long long)(ch + w) * s.taps + s.taps - 1 - j], before(i0 + t - j, w), y[w]);
          y[w] = conv_act(y[w]);
        }
      }
      put(t, y);
    }
  }
}

template <int DP, bool DELTA>
struct PrepSmem {
  using R = Rec<DP, DELTA>;
  static constexpr int LD = DP + 8;                        // fp32 rows
  static constexpr int F32 = 3 * CK * LD * 4;              // q, k, running log decay
  static constexpr int KHAT = R::BYTES;                    // k e^{-b}, head and tail, behind the record image
  static constexpr int IMG = KHAT + 2 * R::MAT;
  static constexpr int OFF_MISC = IMG > F32 ? IMG : F32;   // the record image replaces the fp32 rows
  // norms [32], beta [16], e^{-b_16} [DP], P / A [512], blocks of the inverse [256]
  static constexpr int BYTES = OFF_MISC + (48 + DP + 512 + 256) * 4;
};

// One CTA per (chunk, head).
template <int DP, bool DELTA>
__global__ void __launch_bounds__(cp_threads(DP), cp_blocks(DP))
chunk_prep_kernel(RecurrentSpec s, RecurrentInputs in, RaggedBatch rb, uint8_t* __restrict__ records,
                  float* __restrict__ vbuf, int vblocks) {
  using R = Rec<DP, DELTA>;
  using PS = PrepSmem<DP, DELTA>;
  constexpr int LD = PS::LD, CP_THREADS = cp_threads(DP);
  extern __shared__ __align__(128) uint8_t psm[];
  float* sq = reinterpret_cast<float*>(psm);     // [16][LD]
  float* sk = sq + CK * LD;
  float* sb = sk + CK * LD;
  float* s_norm = reinterpret_cast<float*>(psm + PS::OFF_MISC);   // [32] scales of the q and k rows
  float* sbeta = s_norm + 32;
  float* s_inv = sbeta + CK;                     // [DP] e^{-b_16}
  float* sP = s_inv + DP;                        // [16][16], pairwise form only
  float* sA = sP + 256;                          // A, then diag(beta) A
  float* sD = sA + 256;                          // inverses of the two diagonal 8 x 8 blocks, two products [8][8] each
  const int slot = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  int b = 0;
  {
    int lo = 0, hi = rb.n_seq - 1;
    while (lo < hi) {
      const int mid = (lo + hi + 1) >> 1;
      if (chunk_base(rb.cu_q, mid) <= slot) lo = mid; else hi = mid - 1;
    }
    b = lo;
  }
  const int q0 = rb.cu_q[b], len = rb.cu_q[b + 1] - q0;
  const int i0 = (slot - chunk_base(rb.cu_q, b)) * CK;     // first local token of the chunk
  if (i0 >= len) return;
  const int n = min(CK, len - i0);
  const long long r0 = q0 + i0;                            // its row
  const bool has_state = rb.kv_lens[b] > len;
  const int g = h / (s.heads / s.kv_heads);
  const int cq = s.kv_heads * s.dim, channels = 2 * cq + s.heads * s.vdim;
  const T* proj = static_cast<const T*>(in.proj);
  const float* st = (has_state && s.taps > 1) ? in.conv_state + (long long)rb.slots[b] * (s.taps - 1) * channels : nullptr;
  // ---- q, k, v: short convolution + silu
  float* vrow = vbuf + ((long long)slot * s.heads + h) * vblocks * (CK * CS_V);
  auto columns = [&](auto wide, auto full) {
    constexpr int W = decltype(wide)::value;
    constexpr bool FULL = decltype(full)::value;
    const int tasks = (2 * s.dim + s.vdim) / W;
    for (int i = tid; i < tasks; i += CP_THREADS) {
      const int c = i * W;
      if (c < 2 * s.dim) {
        const bool is_q = c < s.dim;
        const int cc = is_q ? c : c - s.dim, at = g * s.dim + cc;
        const int ch = is_q ? at : cq + at;
        float* dst = (is_q ? sq : sk) + cc;
        conv_column<W, FULL>(s, in, proj + (is_q ? in.q_off : in.k_off) + at, q0, i0, n, st ? st + ch : nullptr, channels, ch,
                       [&](int t, const float (&y)[W]) {
                         if constexpr (W == 2) *reinterpret_cast<float2*>(dst + t * LD) = make_float2(y[0], y[1]);
                         else dst[t * LD] = y[0];
                       });
      } else {
        const int v = c - 2 * s.dim, at = h * s.vdim + v, ch = 2 * cq + at;
        float* dst = vrow + (v / CS_V) * (CK * CS_V);
        conv_column<W, FULL>(s, in, proj + in.v_off + at, q0, i0, n, st ? st + ch : nullptr, channels, ch,
                       [&](int t, const float (&y)[W]) {
                         float* d = dst + t * CS_V + ((v % CS_V) ^ (((t >> 1) & 3) << 3));
                         if constexpr (W == 2) *reinterpret_cast<float2*>(d) = make_float2(y[0], y[1]);
                         else *d = y[0];
                       });
      }
    }
  };
  if (((s.dim | s.vdim | (int)in.ld) & 1) != 0) columns(std::integral_constant<int, 1>{}, std::false_type{});
  else if (n == CK) columns(std::integral_constant<int, 2>{}, std::true_type{});
  else columns(std::integral_constant<int, 2>{}, std::false_type{});
  for (int v = s.vdim + tid; v < vblocks * CS_V; v += CP_THREADS)
    for (int t = 0; t < CK; ++t) vrow[(v / CS_V) * (CK * CS_V) + t * CS_V + ((v % CS_V) ^ (((t >> 1) & 3) << 3))] = 0.f;
  // ---- log decays and their running sum; channels past dim are empty
  float range = 0.f;
  for (int c = tid; c < DP; c += CP_THREADS) {
    float run = 0.f;
    if (c < s.dim) {
      const float bias = in.z_bias[h * s.dim + c];
      const float ea = DELTA ? -expf(in.a_log[h]) : -s.inv_tau;
      const float* zp = in.z + r0 * in.ldz + h * s.dim + c;
      float z[CK];
#pragma unroll
      for (int t = 0; t < CK; ++t) z[t] = t < n ? zp[t * in.ldz] : 0.f;
#pragma unroll
      for (int t = 0; t < CK; ++t) {
        if (t < n) run = fmaf(ea, softplus_fast(DELTA ? z[t] + bias : -(z[t] + bias)), run);
        sb[t * LD + c] = run;
      }
    } else {
#pragma unroll
      for (int t = 0; t < CK; ++t) { sb[t * LD + c] = 0.f; sq[t * LD + c] = 0.f; sk[t * LD + c] = 0.f; }
    }
    s_inv[c] = __expf(-run);
    range = fmaxf(range, -run);
  }
  if (DELTA && tid < CK) sbeta[tid] = tid < n ? sigmoid_f(ldf(proj + (r0 + tid) * in.ld + in.b_off + h)) : 0.f;
  const bool pairwise = __syncthreads_or(!(range <= 60.f)) != 0;
  // ---- unit norms (as one scale per row) and the query scale
  for (int j = warp; j < 2 * CK; j += CP_THREADS / 32) {
    const float* x = (j < CK ? sq : sk) + (j & (CK - 1)) * LD;
    float r = 1.f;
    if (s.unit_norm) {
      float ss = 0.f;
#pragma unroll
      for (int c = lane; c < DP; c += 32) ss = fmaf(x[c], x[c], ss);
      r = 1.f / sqrtf(warp_sum(ss) + 1e-6f);
    }
    if (lane == 0) s_norm[j] = j < CK ? r * s.q_scale : r;
  }
  __syncthreads();
  if (pairwise) {
    for (int i = tid; i < CK * CK; i += CP_THREADS) {
      const int t = i / CK, c = i % CK;
      float p = 0.f, a = 0.f;
      if (c <= t)
        for (int k = 0; k < s.dim; ++k) {
          const float w = sk[c * LD + k] * __expf(sb[t * LD + k] - sb[c * LD + k]);
          p = fmaf(sq[t * LD + k], w, p);
          a = fmaf(sk[t * LD + k], w, a);
        }
      sP[i] = p * s_norm[t] * s_norm[CK + c];
      sA[i] = DELTA && c < t ? a * s_norm[CK + t] * s_norm[CK + c] : 0.f;
    }
  }
  // ---- decayed operands: a thread takes units of 8 channels of one token through registers, because the
  // record image takes the place of the fp32 rows
  constexpr int UPR = DP / 8, UNITS = (CK * UPR + CP_THREADS - 1) / CP_THREADS;
  const int u = tid % UPR;
  float qv[UNITS][8], kv[UNITS][8], bv[UNITS][8], be[8];
#pragma unroll
  for (int m = 0; m < UNITS; ++m) {
    const int t = (tid + m * CP_THREADS) / UPR;
    if (t < CK) {
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const float4 q4 = *reinterpret_cast<const float4*>(sq + t * LD + u * 8 + 4 * e);
        const float4 k4 = *reinterpret_cast<const float4*>(sk + t * LD + u * 8 + 4 * e);
        const float4 b4 = *reinterpret_cast<const float4*>(sb + t * LD + u * 8 + 4 * e);
        qv[m][4 * e] = q4.x; qv[m][4 * e + 1] = q4.y; qv[m][4 * e + 2] = q4.z; qv[m][4 * e + 3] = q4.w;
        kv[m][4 * e] = k4.x; kv[m][4 * e + 1] = k4.y; kv[m][4 * e + 2] = k4.z; kv[m][4 * e + 3] = k4.w;
        bv[m][4 * e] = b4.x; bv[m][4 * e + 1] = b4.y; bv[m][4 * e + 2] = b4.z; bv[m][4 * e + 3] = b4.w;
      }
    }
  }
#pragma unroll
  for (int e = 0; e < 8; ++e) be[e] = sb[(CK - 1) * LD + u * 8 + e];
  __syncthreads();
#pragma unroll
  for (int m = 0; m < UNITS; ++m) {
    const int t = (tid + m * CP_THREADS) / UPR;
    if (t < CK) {
      const float nq = s_norm[t], nk = s_norm[CK + t];
      uint32_t qh[4], ql[4], kh[4], kl[4], bh[4], bl[4], gh[4], gl[4];
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        float q2[2], k2[2], b2[2], g2[2];
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int i = 2 * j + e;
          const float d = __expf(bv[m][i]), k0 = kv[m][i] * nk;
          q2[e] = qv[m][i] * nq * d;
          k2[e] = k0 * d;
          b2[e] = k0 * __expf(be[i] - bv[m][i]);
          g2[e] = b2[e] * s_inv[u * 8 + i];
        }
        split2(q2[0], q2[1], qh[j], ql[j]);
        if (DELTA) split2(k2[0], k2[1], kh[j], kl[j]);
        split2(b2[0], b2[1], bh[j], bl[j]);
        split2(g2[0], g2[1], gh[j], gl[j]);
      }
      const int o = unit_off<DP>(t, u);
      *reinterpret_cast<uint4*>(psm + R::Q_HI + o) = make_uint4(qh[0], qh[1], qh[2], qh[3]);
      *reinterpret_cast<uint4*>(psm + R::Q_LO + o) = make_uint4(ql[0], ql[1], ql[2], ql[3]);
      *reinterpret_cast<uint4*>(psm + R::B_HI + o) = make_uint4(bh[0], bh[1], bh[2], bh[3]);
      *reinterpret_cast<uint4*>(psm + R::B_LO + o) = make_uint4(bl[0], bl[1], bl[2], bl[3]);
      *reinterpret_cast<uint4*>(psm + PS::KHAT + o) = make_uint4(gh[0], gh[1], gh[2], gh[3]);
      *reinterpret_cast<uint4*>(psm + PS::KHAT + R::MAT + o) = make_uint4(gl[0], gl[1], gl[2], gl[3]);
      if constexpr (DELTA) {
        *reinterpret_cast<uint4*>(psm + R::K_HI + o) = make_uint4(kh[0], kh[1], kh[2], kh[3]);
        *reinterpret_cast<uint4*>(psm + R::K_LO + o) = make_uint4(kl[0], kl[1], kl[2], kl[3]);
      }
    }
  }
  if (tid < UPR)
#pragma unroll
    for (int e = 0; e < 8; ++e) reinterpret_cast<float*>(psm + R::DEC)[u * 8 + e] = __expf(be[e]);
  __syncthreads();
  // ---- warp 0: P = tril(q~ k^^T); warp 1: A = tril(k~ k^^T, -1) and T
  if (warp < (DELTA ? 2 : 1)) {
    const int r = lane >> 2, tq = lane & 3;
    const int x_hi = warp == 0 ? R::Q_HI : (DELTA ? R::K_HI : 0), x_lo = warp == 0 ? R::Q_LO : (DELTA ? R::K_LO : 0);
    float* dst = warp == 0 ? sP : sA;
    float acc[3][2][4] = {};
    if (!pairwise) {
      const int n_row = (lane & 7) + ((lane >> 4) << 3), n_unit = (lane >> 3) & 1;      // B fragments (row = token)
      const int a_row = (lane & 7) + (((lane >> 3) & 1) << 3), a_unit = lane >> 4;      // A fragments
      const uint32_t base = smem_u32(psm);
#pragma unroll
      for (int ks = 0; ks < DP / 16; ++ks) {
        uint32_t xh[4], xl[4], bh[4], bl[4];
        const int bo = unit_off<DP>(n_row, 2 * ks + n_unit), ao = unit_off<DP>(a_row, 2 * ks + a_unit);
        ldm_x4(base + PS::KHAT + bo, bh);
        ldm_x4(base + PS::KHAT + R::MAT + bo, bl);
        ldm_x4(base + x_hi + ao, xh);
        ldm_x4(base + x_lo + ao, xl);
#pragma unroll
        for (int nt = 0; nt < 2; ++nt) {
          mma_bf16(acc[0][nt], xh, bh[2 * nt], bh[2 * nt + 1]);
          mma_bf16(acc[1][nt], xh, bl[2 * nt], bl[2 * nt + 1]);
          mma_bf16(acc[2][nt], xl, bh[2 * nt], bh[2 * nt + 1]);
        }
      }
    }
#pragma unroll
    for (int nt = 0; nt < 2; ++nt)
#pragma unroll
      for (int e = 0; e < 4; e += 2) {
        const int t = r + 4 * e, c = nt * 8 + 2 * tq;
        float v[2];
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          const float y = pairwise ? dst[t * CK + c + i] : acc[0][nt][e + i] + (acc[1][nt][e + i] + acc[2][nt][e + i]);
          // past the diagonal the factors may be out of range: select, do not multiply
          v[i] = (warp == 0 ? c + i <= t : c + i < t) ? y : 0.f;
        }
        if (warp == 0) {
          uint32_t hi, lo;
          split2(v[0], v[1], hi, lo);
          *reinterpret_cast<uint32_t*>(psm + R::P_HI + (t * CK + c) * 2) = hi;
          *reinterpret_cast<uint32_t*>(psm + R::P_LO + (t * CK + c) * 2) = lo;
        } else {
          *reinterpret_cast<float2*>(sA + t * CK + c) = make_float2(sbeta[t] * v[0], sbeta[t] * v[1]);
        }
      }
    __syncwarp();
    // T = (I + N)^-1 diag(beta), N = diag(beta) A: the two diagonal 8 x 8 blocks by forward substitution (a lane
    // per column), the block below them as -D22 N21 D11
    if constexpr (DELTA) {
      if (warp == 1) {
        if (lane < CK) {
          const int j = lane & 7;
          const float* nb = sA + (lane & 8) * (CK + 1);
          float x[8];
#pragma unroll
          for (int t = 0; t < 8; ++t) {
            float y = 0.f;
#pragma unroll
            for (int c = 0; c < t; ++c) y = fmaf(nb[t * CK + c], x[c], y);
            x[t] = t == j ? 1.f : (t > j ? -y : 0.f);
            sD[(lane & 8) * 8 + t * 8 + j] = x[t];
          }
        }
        __syncwarp();
        float m[2] = {};
#pragma unroll
        for (int c = 0; c < 8; ++c) {
          const float d = sD[c * 8 + (lane & 7)];
          m[0] = fmaf(sA[(8 + (lane >> 3)) * CK + c], d, m[0]);
          m[1] = fmaf(sA[(12 + (lane >> 3)) * CK + c], d, m[1]);
        }
        sD[128 + lane] = m[0];
        sD[160 + lane] = m[1];
        __syncwarp();
        m[0] = m[1] = 0.f;
#pragma unroll
        for (int c = 0; c < 8; ++c) {
          const float d = sD[128 + c * 8 + (lane & 7)];
          m[0] = fmaf(-sD[64 + (lane >> 3) * 8 + c], d, m[0]);
          m[1] = fmaf(-sD[96 + (lane >> 3) * 8 + c], d, m[1]);
        }
        sD[192 + lane] = m[0];
        sD[224 + lane] = m[1];
        __syncwarp();
        const int t = lane >> 1, half = lane & 1;      // 8 columns of a row per lane
        const float* row = t < 8 ? sD + t * 8 : (half ? sD + 64 + (t - 8) * 8 : sD + 192 + (t - 8) * 8);
        uint32_t hi[4], lo[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const bool zero = t < 8 && half;
          split2(zero ? 0.f : row[2 * i] * sbeta[half * 8 + 2 * i], zero ? 0.f : row[2 * i + 1] * sbeta[half * 8 + 2 * i + 1], hi[i],
                 lo[i]);
        }
        *reinterpret_cast<uint4*>(psm + R::T_HI + t * 32 + half * 16) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
        *reinterpret_cast<uint4*>(psm + R::T_LO + t * 32 + half * 16) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
      }
    }
  }
  fence_proxy_async_smem();
  __syncthreads();
  if (tid == 0) {
    asm volatile("cp.async.bulk.global.shared::cta.bulk_group [%0], [%1], %2;"
                 ::"l"(records + ((long long)slot * s.heads + h) * R::BYTES), "r"(smem_u32(psm)), "r"((uint32_t)R::BYTES) : "memory");
    tma_store_commit();
    tma_store_wait_read0();          // shared memory has been read; the grid's end covers the rest
  }
}

// grid (64-channel value block, head, sequence), 4 independent warps of 16 value channels.
constexpr int CS_STAGES = 3;
template <int DP, bool DELTA>
struct ScanSmem {
  using R = Rec<DP, DELTA>;
  static constexpr int STAGE = R::BYTES + R::V_BLOCK;
  static constexpr int OFF_BAR = CS_STAGES * STAGE;
  static constexpr int BYTES = OFF_BAR + 2 * CS_STAGES * 8 + 16;
};

__device__ __forceinline__ void bulk_load(void* dst, const void* src, uint32_t bytes, uint64_t* bar) {
  asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];"
               ::"r"(smem_u32(dst)), "l"(src), "r"(bytes), "r"(smem_u32(bar)) : "memory");
}

template <int DP, bool DELTA>
__global__ void __launch_bounds__(CS_WARPS * 32)
chunk_scan_kernel(RecurrentSpec s, RaggedBatch rb, const uint8_t* __restrict__ records, const float* __restrict__ vbuf,
                  int vblocks, float* __restrict__ state, float* __restrict__ o, int* status) {
  using R = Rec<DP, DELTA>;
  using SM = ScanSmem<DP, DELTA>;
  constexpr int KS = DP / 16;
  extern __shared__ __align__(128) uint8_t smem[];
  uint64_t* full = reinterpret_cast<uint64_t*>(smem + SM::OFF_BAR);
  uint64_t* empty = full + CS_STAGES;
  volatile int* abort_flag = reinterpret_cast<volatile int*>(empty + CS_STAGES);
  const int vb = blockIdx.x, h = blockIdx.y, b = blockIdx.z;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, r = lane >> 2, tq = lane & 3;
  const int q0 = rb.cu_q[b], len = rb.cu_q[b + 1] - q0;
  if (len <= 0) return;
  const int chunks = (len + CK - 1) / CK;
  const long long slot0 = chunk_base(rb.cu_q, b);
  if (threadIdx.x == 0) {
    for (int i = 0; i < CS_STAGES; ++i) {
      mbar_init(&full[i], 1);
      mbar_init(&empty[i], CS_WARPS);
    }
    *abort_flag = 0;
    fence_mbar_init();
  }
  __syncthreads();
  auto issue = [&](int c) {
    const int st = c % CS_STAGES;
    const long long rec = (slot0 + c) * s.heads + h;
    uint8_t* dst = smem + st * SM::STAGE;
    mbar_arrive_expect_tx(&full[st], R::BYTES + R::V_BLOCK);
    bulk_load(dst, records + rec * R::BYTES, R::BYTES, &full[st]);
    bulk_load(dst + R::BYTES, vbuf + (rec * vblocks + vb) * (CK * CS_V), R::V_BLOCK, &full[st]);
  };
  if (threadIdx.x == 0)
    for (int c = 0; c < CS_STAGES && c < chunks; ++c) issue(c);

  // this warp's rows of S^T: tile n holds key channels 8 n + 2 tq, + 1 of value channels v, v + 8
  const int v = vb * CS_V + warp * 16 + r;
  float* st0 = state + (((long long)rb.slots[b] * s.heads + h) * s.vdim + v) * s.dim;
  float* st1 = st0 + 8ll * s.dim;
  const bool fresh = rb.kv_lens[b] == len, ok0 = v < s.vdim, ok1 = v + 8 < s.vdim;
  float S[2 * KS][4];
#pragma unroll
  for (int n = 0; n < 2 * KS; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int c = n * 8 + 2 * tq + (e & 1);
      const bool ok = !fresh && c < s.dim && (e < 2 ? ok0 : ok1);
      S[n][e] = ok ? (e < 2 ? st0 : st1)[c] : 0.f;
    }
  // ldmatrix row / unit of this lane: plain (row = token) and transposed forms
  const int n_row = (lane & 7) + ((lane >> 4) << 3), n_unit = (lane >> 3) & 1;
  const int t_row = (lane & 7) + (((lane >> 3) & 1) << 3), t_unit = lane >> 4;
  bool ok = true;
  for (int c = 0; c < chunks; ++c) {
    const int stg = c % CS_STAGES;
    const uint32_t ph = (c / CS_STAGES) & 1;
    ok = mbar_wait(&full[stg], ph, abort_flag, status, 80);
    ok = __all_sync(0xffffffffu, ok);
    if (!ok) break;
    const uint8_t* rec = smem + stg * SM::STAGE;
    const uint32_t ra = smem_u32(rec);
    const float* sv = reinterpret_cast<const float*>(rec + R::BYTES);
    // The chain from one chunk to the next is S -> W -> U -> S; O hangs off it. So the products of W go
    // first and those of O fill the waits on U. The three parts of a split product have accumulators of
    // their own: a chain of dependent MMAs is then as short as the number of k-steps.
    uint32_t ah[KS][4], al[KS][4];
#pragma unroll
    for (int j = 0; j < KS; ++j) {
      split2(S[2 * j][0], S[2 * j][1], ah[j][0], al[j][0]);
      split2(S[2 * j][2], S[2 * j][3], ah[j][1], al[j][1]);
      split2(S[2 * j + 1][0], S[2 * j + 1][1], ah[j][2], al[j][2]);
      split2(S[2 * j + 1][2], S[2 * j + 1][3], ah[j][3], al[j][3]);
    }
    auto read_out = [&](int hi_off, int lo_off, float (&acc)[3][2][4]) {   // S^T x^T, x = q~ or k~
#pragma unroll
      for (int j = 0; j < KS; ++j) {
        uint32_t bh[4], bl[4];
        const int off = unit_off<DP>(n_row, 2 * j + n_unit);
        ldm_x4(ra + hi_off + off, bh);
        ldm_x4(ra + lo_off + off, bl);
#pragma unroll
        for (int nt = 0; nt < 2; ++nt) {
          mma_bf16(acc[0][nt], ah[j], bh[2 * nt], bh[2 * nt + 1]);
          mma_bf16(acc[1][nt], ah[j], bl[2 * nt], bl[2 * nt + 1]);
          mma_bf16(acc[2][nt], al[j], bh[2 * nt], bh[2 * nt + 1]);
        }
      }
    };
    // ---- U^T (16 channels x 16 tokens) as accumulator fragments
    float U[2][4];
#pragma unroll
    for (int nt = 0; nt < 2; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int t = nt * 8 + 2 * tq + (e & 1), col = warp * 16 + r + 8 * (e >> 1);
        U[nt][e] = sv[t * CS_V + (col ^ (((t >> 1) & 3) << 3))];
      }
    uint32_t uh[4], ul[4];
    auto split_u = [&]() {
      split2(U[0][0], U[0][1], uh[0], ul[0]);
      split2(U[0][2], U[0][3], uh[1], ul[1]);
      split2(U[1][0], U[1][1], uh[2], ul[2]);
      split2(U[1][2], U[1][3], uh[3], ul[3]);
    };
    float Oa[3][2][4] = {};
    if constexpr (DELTA) {
      float Wa[3][2][4] = {};
      read_out(R::K_HI, R::K_LO, Wa);
#pragma unroll
      for (int nt = 0; nt < 2; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) U[nt][e] -= Wa[0][nt][e] + (Wa[1][nt][e] + Wa[2][nt][e]);
      split_u();
      uint32_t th[4], tl[4];
      ldm_x4(ra + R::T_HI + n_row * 32 + n_unit * 16, th);
      ldm_x4(ra + R::T_LO + n_row * 32 + n_unit * 16, tl);
      float Ua[3][2][4] = {};
#pragma unroll
      for (int nt = 0; nt < 2; ++nt) {
        mma_bf16(Ua[0][nt], uh, th[2 * nt], th[2 * nt + 1]);
        mma_bf16(Ua[1][nt], uh, tl[2 * nt], tl[2 * nt + 1]);
        mma_bf16(Ua[2][nt], ul, th[2 * nt], th[2 * nt + 1]);
      }
      read_out(R::Q_HI, R::Q_LO, Oa);
#pragma unroll
      for (int nt = 0; nt < 2; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) U[nt][e] = Ua[0][nt][e] + (Ua[1][nt][e] + Ua[2][nt][e]);
    } else {
      read_out(R::Q_HI, R::Q_LO, Oa);
    }
    split_u();
    float O[2][4];
#pragma unroll
    for (int nt = 0; nt < 2; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) O[nt][e] = Oa[0][nt][e] + (Oa[1][nt][e] + Oa[2][nt][e]);
    // ---- S^T = S^T diag(e^b) + U^T K-
    const float* dec = reinterpret_cast<const float*>(rec + R::DEC);
#pragma unroll
    for (int j = 0; j < KS; ++j) {
      uint32_t bh[4], bl[4];
      const int off = unit_off<DP>(t_row, 2 * j + t_unit);
      ldm_x4_t(ra + R::B_HI + off, bh);
      ldm_x4_t(ra + R::B_LO + off, bl);
#pragma unroll
      for (int nt = 0; nt < 2; ++nt) {
        float (&acc)[4] = S[2 * j + nt];
        const float2 d = *reinterpret_cast<const float2*>(dec + (2 * j + nt) * 8 + 2 * tq);
        acc[0] *= d.x;
        acc[1] *= d.y;
        acc[2] *= d.x;
        acc[3] *= d.y;
        mma_bf16(acc, uh, bh[2 * nt], bh[2 * nt + 1]);
        mma_bf16(acc, uh, bl[2 * nt], bl[2 * nt + 1]);
        if (DELTA) mma_bf16(acc, ul, bh[2 * nt], bh[2 * nt + 1]);   // without the delta rule U = V is exact in bf16
      }
    }
    // ---- O^T += U^T P^T
    {
      uint32_t phh[4], pll[4];
      ldm_x4(ra + R::P_HI + n_row * 32 + n_unit * 16, phh);
      ldm_x4(ra + R::P_LO + n_row * 32 + n_unit * 16, pll);
#pragma unroll
      for (int nt = 0; nt < 2; ++nt) {
        mma_bf16(O[nt], uh, phh[2 * nt], phh[2 * nt + 1]);
        mma_bf16(O[nt], uh, pll[2 * nt], pll[2 * nt + 1]);
        if (DELTA) mma_bf16(O[nt], ul, phh[2 * nt], phh[2 * nt + 1]);
      }
    }
    // ---- the warp is done with the stage; thread 0 refills it once all warps are
    __syncwarp();
    if (lane == 0) mbar_arrive(&empty[stg]);
#pragma unroll
    for (int nt = 0; nt < 2; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int t = c * CK + nt * 8 + 2 * tq + (e & 1);
        if (t < len && (e < 2 ? ok0 : ok1))
          o[((long long)(q0 + t) * s.heads + h) * s.vdim + v + 8 * (e >> 1)] = O[nt][e];
      }
    if (threadIdx.x == 0 && c + CS_STAGES < chunks) {
      if (mbar_wait(&empty[stg], ph, abort_flag, status, 81)) issue(c + CS_STAGES);
    }
    __syncwarp();
  }
  if (ok) {
#pragma unroll
    for (int n = 0; n < 2 * KS; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int c = n * 8 + 2 * tq + (e & 1);
        if (c < s.dim && (e < 2 ? ok0 : ok1)) (e < 2 ? st0 : st1)[c] = S[n][e];
      }
  }
  __syncthreads();
  if (*abort_flag) {     // let copies in flight land before the CTA's shared memory goes away
    const long long t0 = clock64();
    while (clock64() - t0 < 10000000LL) {}
  }
}

template <int DP, bool DELTA>
void launch_chunked(const RecurrentSpec& s, const RecurrentInputs& in, const RaggedBatch& rb, uint8_t* records,
                    float* vbuf, float* o, int* status, cudaStream_t stream) {
  using SM = ScanSmem<DP, DELTA>;
  const int vblocks = (s.vdim + CS_V - 1) / CS_V;
  const int slots = rb.rows / CK + rb.n_seq;
  using PS = PrepSmem<DP, DELTA>;
  static bool configured = false;
  if (!configured) {
    MB_CUDA_CHECK(cudaFuncSetAttribute(chunk_scan_kernel<DP, DELTA>, cudaFuncAttributeMaxDynamicSharedMemorySize, SM::BYTES));
    MB_CUDA_CHECK(cudaFuncSetAttribute(chunk_prep_kernel<DP, DELTA>, cudaFuncAttributeMaxDynamicSharedMemorySize, PS::BYTES));
    configured = true;
  }
  chunk_prep_kernel<DP, DELTA><<<dim3(slots, s.heads), cp_threads(DP), PS::BYTES, stream>>>(s, in, rb, records, vbuf, vblocks);
  check_launch();
  chunk_scan_kernel<DP, DELTA><<<dim3(vblocks, s.heads, rb.n_seq), CS_WARPS * 32, SM::BYTES, stream>>>(
      s, rb, records, vbuf, vblocks, in.state, o, status);
  count_launch(2);
  check_launch();
}

long long record_bytes(const RecurrentSpec& s) {
  const int dp = s.dim <= 32 ? 32 : (s.dim <= 64 ? 64 : 128);
  if (s.delta) return dp == 32 ? Rec<32, true>::BYTES : (dp == 64 ? Rec<64, true>::BYTES : Rec<128, true>::BYTES);
  return dp == 32 ? Rec<32, false>::BYTES : (dp == 64 ? Rec<64, false>::BYTES : Rec<128, false>::BYTES);
}

}  // namespace

bool recurrent_chunked_ok(const RecurrentSpec& s) {
  return s.dim <= 128 && (s.delta ? s.decay_kind == 1 : s.decay_kind == 0 && s.taps == 0);
}

long long recurrent_chunked_scratch(const RecurrentSpec& s, int rows, int n_seq) {
  const long long recs = ((long long)rows / CK + n_seq) * s.heads;
  return recs * (record_bytes(s) + (long long)((s.vdim + CS_V - 1) / CS_V) * CK * CS_V * 4);
}

void recurrent_scan_chunked(const RecurrentSpec& s, const RecurrentInputs& in, const RaggedBatch& rb,
                            void* scratch, float* o, int* status, cudaStream_t stream) {
  MB_REQUIRE(recurrent_chunked_ok(s), "recurrent_scan_chunked: key width up to 128; the delta rule with its own decay, "
                                      "or gated linear attention without a convolution");
  MB_REQUIRE((reinterpret_cast<uintptr_t>(scratch) & 15) == 0, "recurrent_scan_chunked: scratch must be 16-byte aligned");
  if (rb.rows == 0) return;
  uint8_t* rec = static_cast<uint8_t*>(scratch);
  float* vbuf = reinterpret_cast<float*>(rec + ((long long)rb.rows / CK + rb.n_seq) * s.heads * record_bytes(s));
  if (s.delta) {
    if (s.dim <= 32) launch_chunked<32, true>(s, in, rb, rec, vbuf, o, status, stream);
    else if (s.dim <= 64) launch_chunked<64, true>(s, in, rb, rec, vbuf, o, status, stream);
    else launch_chunked<128, true>(s, in, rb, rec, vbuf, o, status, stream);
  } else {
    if (s.dim <= 32) launch_chunked<32, false>(s, in, rb, rec, vbuf, o, status, stream);
    else if (s.dim <= 64) launch_chunked<64, false>(s, in, rb, rec, vbuf, o, status, stream);
    else launch_chunked<128, false>(s, in, rb, rec, vbuf, o, status, stream);
  }
}

}  // namespace mb
