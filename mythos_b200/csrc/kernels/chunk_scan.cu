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
// No exponent above is positive. P and A are formed as (q e^{b_t - m}) (k e^{m - b_s}) around the middle
// m of the chunk's decay, where the factors stay in range; a channel that decays by more than e^-80
// inside one chunk sends the chunk to a pairwise evaluation instead.
#include "common.cuh"
#include "hybrid_api.h"
#include "hybrid_dev.cuh"
#include "host_util.h"
#include "tc.cuh"

namespace mb {
namespace {

constexpr int CK = 16;            // tokens per chunk
constexpr int CS_WARPS = 4;       // scan warps per CTA
constexpr int CS_V = 16 * CS_WARPS;
constexpr int CP_THREADS = 128;

__device__ __forceinline__ void mma_bf16(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, "
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

__device__ __forceinline__ float raw_tap(const T* col, long long ld, long long r0, int i, const float* st, int channels,
                                         int taps, int n) {
  // input at local token i (i < 0: the convolution state, i >= n: past the end)
  if (i >= n) return 0.f;
  if (i >= 0) return ldf(col + (r0 + i) * ld);
  return st ? st[(long long)(taps - 1 + i) * channels] : 0.f;
}

template <int DP, bool DELTA>
__global__ void __launch_bounds__(CP_THREADS)
chunk_prep_kernel(RecurrentSpec s, RecurrentInputs in, RaggedBatch rb, uint8_t* __restrict__ records,
                  float* __restrict__ vbuf, int vblocks) {
  using R = Rec<DP, DELTA>;
  constexpr int LD = DP + 1;
  extern __shared__ float sm[];
  float* sq = sm;                     // [16][LD]
  float* sk = sq + CK * LD;
  float* sb = sk + CK * LD;           // running log decay
  float* sP = sb + CK * LD;           // [16][16]
  float* sA = sP + 256;
  float* sbeta = sA + 256;            // [16]
  float* part = sbeta + CK;           // [warps][2][256] partial P and A
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
  // ---- q, k, v: short convolution + silu, channel by channel
  const int tasks = 2 * s.dim + s.vdim;
  float* vrow = vbuf + ((long long)slot * s.heads + h) * vblocks * (CK * CS_V);
  for (int c = tid; c < tasks; c += CP_THREADS) {
    int ch, col;                                           // channel within q | k | v, column of the projection
    if (c < s.dim) { ch = g * s.dim + c; col = in.q_off + ch; }
    else if (c < 2 * s.dim) { ch = cq + g * s.dim + c - s.dim; col = in.k_off + ch - cq; }
    else { ch = 2 * cq + h * s.vdim + c - 2 * s.dim; col = in.v_off + ch - 2 * cq; }
    const T* p = proj + col;
    float y[CK];
    if (s.taps > 0) {
      const float* st = (has_state && s.taps > 1)
                            ? in.conv_state + (long long)rb.slots[b] * (s.taps - 1) * channels + ch : nullptr;
      const float* w = in.conv_w + (long long)ch * s.taps;
#pragma unroll
      for (int t = 0; t < CK; ++t) y[t] = 0.f;
      // input i of the portion feeds outputs i .. i + taps - 1
      if (s.taps == 4) {
        float x[CK + 3];
#pragma unroll
        for (int j = 0; j < CK + 3; ++j) x[j] = raw_tap(p, in.ld, q0, i0 + j - 3, st, channels, 4, len);
        const float w0 = w[0], w1 = w[1], w2 = w[2], w3 = w[3];
#pragma unroll
        for (int t = 0; t < CK; ++t) y[t] = fmaf(w0, x[t], fmaf(w1, x[t + 1], fmaf(w2, x[t + 2], w3 * x[t + 3])));
      } else {
        for (int j = 0; j < s.taps; ++j) {
          const float wj = w[s.taps - 1 - j];
#pragma unroll
          for (int t = 0; t < CK; ++t) y[t] = fmaf(wj, raw_tap(p, in.ld, q0, i0 + t - j, st, channels, s.taps, len), y[t]);
        }
      }
#pragma unroll
      for (int t = 0; t < CK; ++t) y[t] = silu_f(y[t]);
    } else {
#pragma unroll
      for (int t = 0; t < CK; ++t) y[t] = t < n ? ldf(p + (r0 + t) * in.ld) : 0.f;
    }
    if (c < 2 * s.dim) {
      float* dst = c < s.dim ? sq + c : sk + c - s.dim;
#pragma unroll
      for (int t = 0; t < CK; ++t) dst[t * LD] = t < n ? y[t] : 0.f;
    } else {
      const int v = c - 2 * s.dim;
      float* dst = vrow + (v / CS_V) * (CK * CS_V);
#pragma unroll
      for (int t = 0; t < CK; ++t) dst[t * CS_V + ((v % CS_V) ^ (((t >> 1) & 3) << 3))] = t < n ? y[t] : 0.f;
    }
  }
  for (int v = s.vdim + tid; v < vblocks * CS_V; v += CP_THREADS)
#pragma unroll
    for (int t = 0; t < CK; ++t) vrow[(v / CS_V) * (CK * CS_V) + t * CS_V + ((v % CS_V) ^ (((t >> 1) & 3) << 3))] = 0.f;
  // ---- log decays and their running sum; channels past dim are empty
  float range = 0.f;
  for (int c = tid; c < DP; c += CP_THREADS) {
    float run = 0.f;
    if (c < s.dim) {
      const float bias = in.z_bias[h * s.dim + c];
      const float ea = DELTA ? expf(in.a_log[h]) : 0.f;
      float z[CK];
#pragma unroll
      for (int t = 0; t < CK; ++t) z[t] = t < n ? in.z[(r0 + t) * in.ldz + h * s.dim + c] : 0.f;
#pragma unroll
      for (int t = 0; t < CK; ++t) {
        if (t < n) run += DELTA ? -ea * softplus_f(z[t] + bias) : -softplus_f(-(z[t] + bias)) * s.inv_tau;
        sb[t * LD + c] = run;
      }
    } else {
#pragma unroll
      for (int t = 0; t < CK; ++t) { sb[t * LD + c] = 0.f; sq[t * LD + c] = 0.f; sk[t * LD + c] = 0.f; }
    }
    range = fmaxf(range, -run);
  }
  if (DELTA && tid < CK) sbeta[tid] = tid < n ? sigmoid_f(ldf(proj + (r0 + tid) * in.ld + in.b_off + h)) : 0.f;
  const bool pairwise = __syncthreads_or(!(range <= 80.f)) != 0;
  // ---- unit norms
  for (int j = warp; j < 2 * CK; j += CP_THREADS / 32) {
    float* x = (j < CK ? sq : sk) + (j & (CK - 1)) * LD;
    float r = 1.f;
    if (s.unit_norm) {
      float ss = 0.f;
      for (int c = lane; c < s.dim; c += 32) ss += x[c] * x[c];
      r = 1.f / sqrtf(warp_sum(ss) + 1e-6f);
    }
    if (j < CK) r *= s.q_scale;
    for (int c = lane; c < s.dim; c += 32) x[c] *= r;
  }
  for (int i = tid; i < 512; i += CP_THREADS) sP[i] = 0.f;   // P and A (the pairwise form leaves their upper triangles)
  __syncthreads();
  // ---- decayed operands of the scan
  uint8_t* rec = records + ((long long)slot * s.heads + h) * R::BYTES;
  for (int i = tid; i < CK * (DP / 8); i += CP_THREADS) {
    const int t = i / (DP / 8), u = i % (DP / 8);
    uint32_t qh[4], ql[4], kh[4], kl[4], bh[4], bl[4];
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      float qv[2], kv[2], bv[2];
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int c = u * 8 + 2 * j + e;
        const float bt = sb[t * LD + c], d = __expf(bt);
        qv[e] = sq[t * LD + c] * d;
        if (DELTA) kv[e] = sk[t * LD + c] * d;
        bv[e] = sk[t * LD + c] * __expf(sb[(CK - 1) * LD + c] - bt);
      }
      split2(qv[0], qv[1], qh[j], ql[j]);
      if (DELTA) split2(kv[0], kv[1], kh[j], kl[j]);
      split2(bv[0], bv[1], bh[j], bl[j]);
    }
    const int o = unit_off<DP>(t, u);
    *reinterpret_cast<uint4*>(rec + R::Q_HI + o) = make_uint4(qh[0], qh[1], qh[2], qh[3]);
    *reinterpret_cast<uint4*>(rec + R::Q_LO + o) = make_uint4(ql[0], ql[1], ql[2], ql[3]);
    *reinterpret_cast<uint4*>(rec + R::B_HI + o) = make_uint4(bh[0], bh[1], bh[2], bh[3]);
    *reinterpret_cast<uint4*>(rec + R::B_LO + o) = make_uint4(bl[0], bl[1], bl[2], bl[3]);
    if (DELTA) {
      *reinterpret_cast<uint4*>(rec + R::K_HI + o) = make_uint4(kh[0], kh[1], kh[2], kh[3]);
      *reinterpret_cast<uint4*>(rec + R::K_LO + o) = make_uint4(kl[0], kl[1], kl[2], kl[3]);
    }
  }
  for (int c = tid; c < DP; c += CP_THREADS) reinterpret_cast<float*>(rec + R::DEC)[c] = __expf(sb[(CK - 1) * LD + c]);
  // ---- P and A
  if (!pairwise) {
    const int r = lane >> 2, tq = lane & 3;
    float p[2][4] = {}, a[2][4] = {};
    for (int ks = warp; ks < DP / 16; ks += CP_THREADS / 32) {
      uint32_t qh[4], ql[4], kh[4], kl[4], bh[2][2], bl[2][2];
#pragma unroll
      for (int f = 0; f < 4; ++f) {       // A fragments: rows r, r + 8; columns 2 tq (+ 8)
        const int t = r + 8 * (f & 1), c = ks * 16 + 2 * tq + 8 * (f >> 1);
        const float d0 = __expf(sb[t * LD + c] - 0.5f * sb[(CK - 1) * LD + c]);
        const float d1 = __expf(sb[t * LD + c + 1] - 0.5f * sb[(CK - 1) * LD + c + 1]);
        split2(sq[t * LD + c] * d0, sq[t * LD + c + 1] * d1, qh[f], ql[f]);
        if (DELTA) split2(sk[t * LD + c] * d0, sk[t * LD + c + 1] * d1, kh[f], kl[f]);
      }
#pragma unroll
      for (int nt = 0; nt < 2; ++nt)
#pragma unroll
        for (int f = 0; f < 2; ++f) {     // B fragments: k = 2 tq (+ 8), n = r
          const int t = nt * 8 + r, c = ks * 16 + 2 * tq + 8 * f;
          const float d0 = __expf(0.5f * sb[(CK - 1) * LD + c] - sb[t * LD + c]);
          const float d1 = __expf(0.5f * sb[(CK - 1) * LD + c + 1] - sb[t * LD + c + 1]);
          split2(sk[t * LD + c] * d0, sk[t * LD + c + 1] * d1, bh[nt][f], bl[nt][f]);
        }
#pragma unroll
      for (int nt = 0; nt < 2; ++nt) {
        mma_bf16(p[nt], qh, bh[nt][0], bh[nt][1]);
        mma_bf16(p[nt], qh, bl[nt][0], bl[nt][1]);
        mma_bf16(p[nt], ql, bh[nt][0], bh[nt][1]);
        if (DELTA) {
          mma_bf16(a[nt], kh, bh[nt][0], bh[nt][1]);
          mma_bf16(a[nt], kh, bl[nt][0], bl[nt][1]);
          mma_bf16(a[nt], kl, bh[nt][0], bh[nt][1]);
        }
      }
    }
#pragma unroll
    for (int nt = 0; nt < 2; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int t = r + 8 * (e >> 1), c = nt * 8 + 2 * tq + (e & 1);
        part[warp * 512 + t * CK + c] = c <= t ? p[nt][e] : 0.f;     // above the diagonal: may be out of range
        part[warp * 512 + 256 + t * CK + c] = DELTA && c < t ? a[nt][e] : 0.f;
      }
    __syncthreads();
    for (int i = tid; i < 512; i += CP_THREADS)
      sP[i] = (part[i] + part[512 + i]) + (part[1024 + i] + part[1536 + i]);
  } else {
    for (int i = tid; i < CK * CK; i += CP_THREADS) {
      const int t = i / CK, c = i % CK;
      if (c > t) continue;
      float p = 0.f, a = 0.f;
      for (int k = 0; k < s.dim; ++k) {
        const float w = sk[c * LD + k] * __expf(sb[t * LD + k] - sb[c * LD + k]);
        p = fmaf(sq[t * LD + k], w, p);
        a = fmaf(sk[t * LD + k], w, a);
      }
      sP[i] = p;
      if (DELTA && c < t) sA[i] = a;
    }
  }
  __syncthreads();
  // ---- T = (I + diag(beta) A)^-1 diag(beta): lane j solves column j by forward substitution
  if (DELTA && warp == 0 && lane < CK) {
    float x[CK];
#pragma unroll
    for (int t = 0; t < CK; ++t) {
      float y = 0.f;
#pragma unroll
      for (int c = 0; c < t; ++c) y = fmaf(sA[t * CK + c], x[c], y);
      x[t] = t == lane ? 1.f : (t > lane ? -sbeta[t] * y : 0.f);
    }
    const float beta = sbeta[lane];
#pragma unroll
    for (int t = 0; t < CK; ++t) {
      const float v = x[t] * beta;
      const __nv_bfloat16 hi = __float2bfloat16(v);
      reinterpret_cast<__nv_bfloat16*>(rec + R::T_HI)[t * CK + lane] = hi;
      reinterpret_cast<__nv_bfloat16*>(rec + R::T_LO)[t * CK + lane] = __float2bfloat16(v - __bfloat162float(hi));
    }
  }
  for (int i = tid - 32; i >= 0 && i < CK * CK; i += CP_THREADS - 32) {
    const float v = sP[i];
    const __nv_bfloat16 hi = __float2bfloat16(v);
    reinterpret_cast<__nv_bfloat16*>(rec + R::P_HI)[i] = hi;
    reinterpret_cast<__nv_bfloat16*>(rec + R::P_LO)[i] = __float2bfloat16(v - __bfloat162float(hi));
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
    float O[2][4] = {}, W[2][4] = {};
    // ---- read the old state: O^T = S^T q~^T, W^T = S^T k~^T
#pragma unroll
    for (int j = 0; j < KS; ++j) {
      uint32_t ah[4], al[4], bh[4], bl[4];
      split2(S[2 * j][0], S[2 * j][1], ah[0], al[0]);
      split2(S[2 * j][2], S[2 * j][3], ah[1], al[1]);
      split2(S[2 * j + 1][0], S[2 * j + 1][1], ah[2], al[2]);
      split2(S[2 * j + 1][2], S[2 * j + 1][3], ah[3], al[3]);
      const int off = unit_off<DP>(n_row, 2 * j + n_unit);
      ldm_x4(ra + R::Q_HI + off, bh);
      ldm_x4(ra + R::Q_LO + off, bl);
#pragma unroll
      for (int nt = 0; nt < 2; ++nt) {
        mma_bf16(O[nt], ah, bh[2 * nt], bh[2 * nt + 1]);
        mma_bf16(O[nt], ah, bl[2 * nt], bl[2 * nt + 1]);
        mma_bf16(O[nt], al, bh[2 * nt], bh[2 * nt + 1]);
      }
      if (DELTA) {
        ldm_x4(ra + R::K_HI + off, bh);
        ldm_x4(ra + R::K_LO + off, bl);
#pragma unroll
        for (int nt = 0; nt < 2; ++nt) {
          mma_bf16(W[nt], ah, bh[2 * nt], bh[2 * nt + 1]);
          mma_bf16(W[nt], ah, bl[2 * nt], bl[2 * nt + 1]);
          mma_bf16(W[nt], al, bh[2 * nt], bh[2 * nt + 1]);
        }
      }
    }
    // ---- U^T (16 channels x 16 tokens) as accumulator fragments
    float U[2][4];
#pragma unroll
    for (int nt = 0; nt < 2; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int t = nt * 8 + 2 * tq + (e & 1), col = warp * 16 + r + 8 * (e >> 1);
        U[nt][e] = sv[t * CS_V + (col ^ (((t >> 1) & 3) << 3))] - (DELTA ? W[nt][e] : 0.f);
      }
    uint32_t uh[4], ul[4];
    split2(U[0][0], U[0][1], uh[0], ul[0]);
    split2(U[0][2], U[0][3], uh[1], ul[1]);
    split2(U[1][0], U[1][1], uh[2], ul[2]);
    split2(U[1][2], U[1][3], uh[3], ul[3]);
    if (DELTA) {
      uint32_t th[4], tl[4];
      ldm_x4(ra + R::T_HI + n_row * 32 + n_unit * 16, th);
      ldm_x4(ra + R::T_LO + n_row * 32 + n_unit * 16, tl);
#pragma unroll
      for (int nt = 0; nt < 2; ++nt) {
        U[nt][0] = U[nt][1] = U[nt][2] = U[nt][3] = 0.f;
        mma_bf16(U[nt], uh, th[2 * nt], th[2 * nt + 1]);
        mma_bf16(U[nt], uh, tl[2 * nt], tl[2 * nt + 1]);
        mma_bf16(U[nt], ul, th[2 * nt], th[2 * nt + 1]);
      }
      split2(U[0][0], U[0][1], uh[0], ul[0]);
      split2(U[0][2], U[0][3], uh[1], ul[1]);
      split2(U[1][0], U[1][1], uh[2], ul[2]);
      split2(U[1][2], U[1][3], uh[3], ul[3]);
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
        mma_bf16(O[nt], ul, phh[2 * nt], phh[2 * nt + 1]);
      }
    }
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
        mma_bf16(acc, ul, bh[2 * nt], bh[2 * nt + 1]);
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
  const int prep_smem = (3 * CK * (DP + 1) + 512 + CK + 2048) * 4;
  static bool configured = false;
  if (!configured) {
    MB_CUDA_CHECK(cudaFuncSetAttribute(chunk_scan_kernel<DP, DELTA>, cudaFuncAttributeMaxDynamicSharedMemorySize, SM::BYTES));
    configured = true;
  }
  chunk_prep_kernel<DP, DELTA><<<dim3(slots, s.heads), CP_THREADS, prep_smem, stream>>>(s, in, rb, records, vbuf, vblocks);
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

bool recurrent_chunked_ok(const RecurrentSpec& s) { return s.dim <= 128; }

long long recurrent_chunked_scratch(const RecurrentSpec& s, int rows, int n_seq) {
  const long long recs = ((long long)rows / CK + n_seq) * s.heads;
  return recs * (record_bytes(s) + (long long)((s.vdim + CS_V - 1) / CS_V) * CK * CS_V * 4);
}

void recurrent_scan_chunked(const RecurrentSpec& s, const RecurrentInputs& in, const RaggedBatch& rb,
                            void* scratch, float* o, int* status, cudaStream_t stream) {
  MB_REQUIRE(recurrent_chunked_ok(s), "recurrent_scan_chunked: key width up to 128");
  MB_REQUIRE((s.delta != 0) == (s.decay_kind == 1), "recurrent_scan_chunked: decay kind and rule come in pairs");
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
