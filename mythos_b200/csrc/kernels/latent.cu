// Attention over a cached latent (hybrid_api.h): every token stores one normalised latent row and one
// rotated key part, shared by all heads.
//
//   latent_prep         norms of latents and of what queries are a map of, rotation of neighbouring columns, append to the pages
//   latent_gather       latent rows of whole sequences, packed (keys and values of prompts are expanded from
//                       them by one GEMM, and the attention kernel of attention_fwd.cu takes over)
//   latent_attn_any     any widths, fp32 arithmetic, one warp per (token, head)
//   latent_attn_decode  single tokens: 16 heads share every cached row that is read; the row serves as key
//                       and, its latent columns, as value. Split over the context,
//                       the splits' states merged by a second kernel.
//
// In the single-token forms the queries have been taken into the latent's space beforehand
// (q_lat = W_uk^T q) and the output leaves it afterwards (W_uv), so nothing per head is cached.
#include "common.cuh"
#include "host_util.h"
#include "hybrid_api.h"
#include "hybrid_dev.cuh"
#include "tc.cuh"

namespace mb {
namespace {

// 16 bytes of a row as floats.
template <typename T>
struct Vec16 {
  static constexpr int N = 16 / (int)sizeof(T);
  float v[N];
  __device__ __forceinline__ void load(const T* p) {
    const uint4 raw = *reinterpret_cast<const uint4*>(p);
    const T* e = reinterpret_cast<const T*>(&raw);
#pragma unroll
    for (int i = 0; i < N; ++i) v[i] = ldf(e + i);
  }
  __device__ __forceinline__ void store(T* p) const {
    uint4 raw;
    T* e = reinterpret_cast<T*>(&raw);
#pragma unroll
    for (int i = 0; i < N; ++i) stf(e + i, v[i]);
    *reinterpret_cast<uint4*>(p) = raw;
  }
  // Pairs (2i, 2i + 1) turned by the (cos, sin) entries cs[0 ..]
  __device__ __forceinline__ void rotate(const float2* cs) {
#pragma unroll
    for (int i = 0; i < N / 2; ++i) {
      const float u = v[2 * i], w = v[2 * i + 1];
      v[2 * i] = u * cs[i].x - w * cs[i].y;
      v[2 * i + 1] = w * cs[i].x + u * cs[i].y;
    }
  }
};

// Normalises `width` columns of a row by a warp (zeros up to padded): out = x / rms * gamma.
template <typename T>
__device__ __forceinline__ void lp_norm(const T* src, T* dst, int width, int padded, const float* gamma, float eps, int lane) {
  constexpr int N = Vec16<T>::N, KEEP = 4;       // vectors that stay in registers
  uint4 raw[KEEP];
  float ss = 0.f;
#pragma unroll
  for (int k = 0; k < KEEP; ++k) {
    const int i = (lane + 32 * k) * N;
    if (i < padded) raw[k] = *reinterpret_cast<const uint4*>(src + i);
  }
#pragma unroll
  for (int k = 0; k < KEEP; ++k) {
    const int i = (lane + 32 * k) * N;
    if (i < padded) {
      Vec16<T> x;
      x.load(reinterpret_cast<const T*>(&raw[k]));
#pragma unroll
      for (int j = 0; j < N; ++j) ss = fmaf(x.v[j], x.v[j], ss);
    }
  }
  for (int i = (lane + 32 * KEEP) * N; i < padded; i += 32 * N) {
    Vec16<T> x;
    x.load(src + i);
#pragma unroll
    for (int j = 0; j < N; ++j) ss = fmaf(x.v[j], x.v[j], ss);
  }
  const float r = 1.f / sqrtf(warp_sum(ss) / (float)width + eps);
  auto put = [&](Vec16<T>& x, int i) {
    if (i + N <= width) {
#pragma unroll
      for (int j = 0; j < N; j += 4) {
        const float4 g = *reinterpret_cast<const float4*>(gamma + i + j);
        x.v[j] *= r * g.x;
        x.v[j + 1] *= r * g.y;
        x.v[j + 2] *= r * g.z;
        x.v[j + 3] *= r * g.w;
      }
    } else {
#pragma unroll
      for (int j = 0; j < N; ++j) x.v[j] *= i + j < width ? r * gamma[i + j] : 0.f;
    }
    x.store(dst + i);
  };
#pragma unroll
  for (int k = 0; k < KEEP; ++k) {
    const int i = (lane + 32 * k) * N;
    if (i < padded) {
      Vec16<T> x;
      x.load(reinterpret_cast<const T*>(&raw[k]));
      put(x, i);
    }
  }
  for (int i = (lane + 32 * KEEP) * N; i < padded; i += 32 * N) {
    Vec16<T> x;
    x.load(src + i);
    put(x, i);
  }
}

// One warp per token. Angles: position x revolutions, reduced to a fraction of a turn in double precision. Padded
// columns of the projection are zero, and so are those of a page row. ROWS: norms and page rows (else queries only).
constexpr int LP_WARPS = 4;
template <typename T, bool ROWS>
__global__ void __launch_bounds__(LP_WARPS * 32)
latent_prep_kernel(T* __restrict__ proj, long long ld, LatentPrep p, LatentSpec s, RaggedBatch rb, LatentPages pg, float eps) {
  constexpr int N = Vec16<T>::N;
  extern __shared__ float2 cs_all[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int t = blockIdx.x * LP_WARPS + warp;
  if (t >= rb.rows) return;
  float2* cs = cs_all + warp * (s.rot_p / 2);
  const int pos = rb.pos[t];
  T* row = proj + (long long)t * ld;
  if constexpr (ROWS) {
    if (p.low_off >= 0) lp_norm(row + p.low_off, row + p.low_off, p.low_rank, (p.low_rank + 7) / 8 * 8, p.low_gamma, eps, lane);
    if (p.qr_off < 0 && p.c_off < 0) return;
  }
  for (int i = lane; i < s.rot_p / 2; i += 32) {
    float sn = 0.f, co = 1.f;
    if (i < s.rot / 2) {
      const double a = pos * p.turns[i];
      sincospif(2.f * (float)(a - rint(a)), &sn, &co);
    }
    cs[i] = make_float2(s.rot_amp * co, s.rot_amp * sn);
  }
  __syncwarp();                              // cs is complete
  if (ROWS && p.c_off >= 0) {
    const int page = pg.table[(long long)rb.row_seq[t] * pg.stride + pos / pg.page_size];
    if (page >= 0) {
      T* dst = static_cast<T*>(pg.cache) + ((long long)page * pg.page_size + pos % pg.page_size) * s.row();
      lp_norm(row + p.c_off, dst, s.rank, s.rank_p, p.gamma, eps, lane);
      for (int i = lane * N; i < s.rot_p; i += 32 * N) {
        Vec16<T> x;
        x.load(row + p.kr_off + i);
        x.rotate(cs + i / 2);
        x.store(dst + s.rank_p + i);
      }
    }
  }
  if (p.qr_off < 0) return;
  const int per = s.rot_p / N;               // vectors per head
#pragma unroll 4
  for (int j = lane; j < s.heads * per; j += 32) {
    Vec16<T> x;
    T* q = row + p.qr_off + j * N;
    x.load(q);
    x.rotate(cs + (j % per) * (N / 2));
    x.store(q);
  }
}

// grid (token blocks, sequences); 16-byte units.
__global__ void __launch_bounds__(256)
latent_gather_kernel(LatentPages pg, const int* __restrict__ cu_k, const int* __restrict__ first, uint4* __restrict__ out, int units) {
  const int b = blockIdx.y, lo = cu_k[b], n = cu_k[b + 1] - lo, skip = first[b];
  const int* table = pg.table + (long long)b * pg.stride;
  const uint4* cache = static_cast<const uint4*>(pg.cache);
  const long long total = (long long)n * units;
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
    const int r = (int)(i / units), t = skip + r, c = (int)(i % units);
    const int page = max(table[t / pg.page_size], 0);
    out[((long long)lo + r) * units + c] = cache[((long long)page * pg.page_size + t % pg.page_size) * units + c];
  }
}

constexpr int LA_WARPS = 4;
template <typename T, int ND>   // ND * 32 >= rank
__global__ void __launch_bounds__(LA_WARPS * 32)
latent_attn_any_kernel(LatentQuery q, LatentSpec s, LatentPages pg, const float* __restrict__ sink, T* __restrict__ out,
                       float scale) {
  extern __shared__ float sq_all[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, W = s.row();
  const long long w = (long long)blockIdx.x * LA_WARPS + warp;
  if (w >= (long long)q.rows * s.heads) return;
  const int t = q.rows - 1 - (int)(w / s.heads), h = (int)(w % s.heads);   // longest contexts first
  float* sq = sq_all + warp * W;
  const T* ql = static_cast<const T*>(q.q_lat) + ((long long)t * s.heads + h) * s.rank_p;
  const T* qr = static_cast<const T*>(q.qr) + t * q.ld_qr + h * s.rot_p;
  for (int i = lane; i < s.rank_p; i += 32) sq[i] = i < s.rank ? ldf(ql + i) * scale : 0.f;
  for (int i = lane; i < s.rot_p; i += 32) sq[s.rank_p + i] = i < s.rot ? ldf(qr + i) * scale : 0.f;
  __syncwarp();
  const int* bt = pg.table + (long long)q.row_seq[t] * pg.stride;
  const T* cache = static_cast<const T*>(pg.cache);
  const int n = q.pos[t] + 1, first = s.window > 0 ? max(0, n - s.window) : 0;
  float m = sink ? sink[h] : -INFINITY, l = sink ? 1.f : 0.f, acc[ND];         // the sink is a key without value
#pragma unroll
  for (int j = 0; j < ND; ++j) acc[j] = 0.f;
  for (int j0 = first; j0 < n; j0 += 32) {
    const int key = j0 + lane;
    float sc = -INFINITY;
    long long tok = 0;
    if (key < n) {
      tok = ((long long)bt[key / pg.page_size] * pg.page_size + key % pg.page_size) * W;
      sc = 0.f;
      for (int i = 0; i < W; ++i) sc = fmaf(sq[i], ldf(cache + tok + i), sc);
    }
    const float mn = fmaxf(m, warp_max(sc));
    const float a = expf(m - mn), p = expf(sc - mn);
    l = l * a + warp_sum(p);
    m = mn;
#pragma unroll
    for (int j = 0; j < ND; ++j) acc[j] *= a;
    const int cnt = min(32, n - j0);
    for (int jj = 0; jj < cnt; ++jj) {
      const float pj = __shfl_sync(0xffffffffu, p, jj);
      const T* vp = cache + __shfl_sync(0xffffffffu, tok, jj);
#pragma unroll
      for (int j = 0; j < ND; ++j) {
        const int d = lane + 32 * j;
        if (d < s.rank) acc[j] = fmaf(pj, ldf(vp + d), acc[j]);
      }
    }
  }
  T* o = out + ((long long)t * s.heads + h) * s.rank_p;
#pragma unroll
  for (int j = 0; j < ND; ++j) {
    const int d = lane + 32 * j;
    if (d < s.rank_p) stf(o + d, d < s.rank ? acc[j] / l : 0.f);
  }
}

// ---------------------------------------------------------------------------------------------
// Single tokens on tensor cores. grid (rows, groups of 16 heads, splits), 8 warps. Tiles of 64 cached
// tokens (four pages) come through a TMA ring as 64-column chunks in the 128-byte-swizzled layout.
//   scores:  warp = (16-token quarter, half of the columns); the halves meet in shared memory
//   softmax: 16 threads per head row
//   values:  warp = NT 8-column tiles of the latent
constexpr int LD_THREADS = 256;
constexpr int LD_TOK = 64;
constexpr int LD_CHUNK = LD_TOK * 128;       // bytes: 64 tokens x 64 columns
constexpr int LD_MAX_STAGES = 4;
constexpr int LD_SLD = LD_TOK + 4;           // row stride of the score partials
constexpr int LD_MAX_SPLITS = 64;

struct LdLayout {
  int chunks, stages, off_q, off_s, off_p, off_w, bytes;
};
__host__ __device__ inline LdLayout ld_layout(int row) {
  LdLayout l;
  l.chunks = (row + 63) / 64;
  const int fixed = l.chunks * 16 * 128 + 2 * 16 * LD_SLD * 4 + 16 * 128 + 64 + 1024;
  l.stages = (220 * 1024 - fixed) / (l.chunks * LD_CHUNK);
  if (l.stages > LD_MAX_STAGES) l.stages = LD_MAX_STAGES;
  l.off_q = l.stages * l.chunks * LD_CHUNK;
  l.off_p = l.off_q + l.chunks * 16 * 128;
  l.off_s = l.off_p + 16 * 128;
  l.off_w = l.off_s + 2 * 16 * LD_SLD * 4;
  l.bytes = l.off_w + 64 + 1024;
  return l;
}

__device__ __forceinline__ void ld_matrix4(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ld_matrix4_trans(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ld_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, "
               "{%0, %1, %2, %3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

template <int NT>
__global__ void __launch_bounds__(LD_THREADS, 1)
latent_decode_kernel(const __grid_constant__ CUtensorMap tm_c, LatentQuery q, LatentSpec s, LatentPages pg,
                     const float* __restrict__ sink, __nv_bfloat16* __restrict__ out, float* __restrict__ scratch,
                     int splits, float scale_log2, int* status) {
  extern __shared__ uint8_t smem_raw[];
  __shared__ uint64_t full[LD_MAX_STAGES];
  __shared__ int abort_word;
  volatile int* abort_flag = &abort_word;
  uint8_t* smem = smem_raw + ((1024u - (smem_u32(smem_raw) & 1023u)) & 1023u);
  const LdLayout L = ld_layout(s.row());
  float* s_part = reinterpret_cast<float*>(smem + L.off_s);
  float* s_alpha = reinterpret_cast<float*>(smem + L.off_w);        // [16]
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int b = blockIdx.x, h0 = blockIdx.y * 16, G = min(16, s.heads - h0), split = blockIdx.z;
  if (threadIdx.x == 0) {
    *abort_flag = 0;
    for (int i = 0; i < L.stages; ++i) mbar_init(&full[i], 1);
    fence_mbar_init();
  }
  __syncthreads();
  const int ctx = q.pos[b] + 1;
  const int lo = s.window > 0 ? max(0, ctx - s.window) : 0;         // first visible token
  const int first = lo / LD_TOK, n_tiles = (ctx + LD_TOK - 1) / LD_TOK, per = (n_tiles - first + splits - 1) / splits;
  const int j0 = first + split * per, j1 = min(n_tiles, j0 + per);
  const int* bt = pg.table + (long long)q.row_seq[b] * pg.stride;
  auto issue = [&](int j) {                                         // warp 0: tile j0 + j
    const int st = j % L.stages;
    uint8_t* dst = smem + st * L.chunks * LD_CHUNK;
    if (lane == 0) mbar_arrive_expect_tx(&full[st], (uint32_t)(L.chunks * LD_CHUNK));
    __syncwarp();
    for (int i = lane; i < 4 * L.chunks; i += 32) {
      const int p = i & 3, c = i >> 2, lp = (j0 + j) * 4 + p;
      // a page past the context is masked below; page 0 keeps the transaction count fixed
      const int page = lp * 16 < ctx ? max(bt[lp], 0) : 0;
      tma_load_2d(dst + c * LD_CHUNK + p * 2048, &tm_c, &full[st], c * 64, page * 16);
    }
  };
  const int mine = max(0, j1 - j0);
  if (warp == 0)
    for (int j = 0; j < L.stages && j < mine; ++j) issue(j);
  // queries: [16 heads][chunks] swizzled like the cache; rows past the last head are zero
  for (int i = threadIdx.x; i < 16 * L.chunks * 8; i += LD_THREADS) {
    const int h = i / (L.chunks * 8), u = i % (L.chunks * 8), col = u * 8;
    uint4 v = make_uint4(0u, 0u, 0u, 0u);
    if (h < G && col < s.row()) {
      const __nv_bfloat16* src = col < s.rank_p
          ? static_cast<const __nv_bfloat16*>(q.q_lat) + ((long long)b * s.heads + h0 + h) * s.rank_p + col
          : static_cast<const __nv_bfloat16*>(q.qr) + b * q.ld_qr + (h0 + h) * s.rot_p + (col - s.rank_p);
      v = *reinterpret_cast<const uint4*>(src);
    }
    *reinterpret_cast<uint4*>(smem + L.off_q + (u >> 3) * 2048 + sw128_offset(h, u & 7)) = v;
  }
  __syncthreads();

  const uint32_t q_addr = smem_u32(smem + L.off_q), p_addr = smem_u32(smem + L.off_p), kv_addr = smem_u32(smem);
  const int tq = warp & 3, kh = warp >> 2;                          // scores: token quarter, half of the columns
  const int a_row = (lane & 7) + ((lane >> 3) & 1) * 8, a_unit = lane >> 4;
  const int k_tok = tq * 16 + ((lane >> 4) << 3) + (lane & 7), k_unit = (lane >> 3) & 1;
  const int v_tok = ((lane >> 3) & 1) * 8 + (lane & 7), v_unit = lane >> 4;
  const int srow = threadIdx.x >> 4, slane = threadIdx.x & 15;      // softmax: head row, 4 tokens
  const int cols = L.chunks * 64, col0 = warp * NT * 8;
  float o[NT][4];
#pragma unroll
  for (int n = 0; n < NT; ++n) o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.f;
  float m_run = -INFINITY, l_run = 0.f;
  bool ok = true;
  for (int j = 0; j < mine; ++j) {
    const int st = j % L.stages;
    ok = mbar_wait(&full[st], (j / L.stages) & 1, abort_flag, status, 110);
    if (!__syncthreads_and(ok)) { ok = false; break; }
    const uint32_t tile = kv_addr + st * L.chunks * LD_CHUNK;
    // ---- scores: two independent chains of products
    float sc[2][2][4];
#pragma unroll
    for (int i = 0; i < 8; ++i) sc[i >> 2][(i >> 1) & 1][(i & 1) * 2] = sc[i >> 2][(i >> 1) & 1][(i & 1) * 2 + 1] = 0.f;
    const int half = L.chunks * 2;                                  // 16-column steps per half
#pragma unroll 2
    for (int k0 = kh * half; k0 < (kh + 1) * half; k0 += 2) {
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int c = (k0 + e) >> 2, u = ((k0 + e) & 3) << 1;
        uint32_t qa[4], kb[4];
        ld_matrix4(q_addr + c * 2048 + sw128_offset(a_row, u + a_unit), qa);
        ld_matrix4(tile + c * LD_CHUNK + sw128_offset(k_tok, u + k_unit), kb);
        ld_mma(sc[e][0], qa, kb[0], kb[1]);
        ld_mma(sc[e][1], qa, kb[2], kb[3]);
      }
    }
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      float* dst = s_part + (kh * 16 + (lane >> 2)) * LD_SLD + tq * 16 + i * 8 + 2 * (lane & 3);
      *reinterpret_cast<float2*>(dst) = make_float2(sc[0][i][0] + sc[1][i][0], sc[0][i][1] + sc[1][i][1]);
      *reinterpret_cast<float2*>(dst + 8 * LD_SLD) = make_float2(sc[0][i][2] + sc[1][i][2], sc[0][i][3] + sc[1][i][3]);
    }
    __syncthreads();
    // ---- softmax of the tile
    {
      const float4 x = *reinterpret_cast<const float4*>(s_part + srow * LD_SLD + slane * 4);
      const float4 y = *reinterpret_cast<const float4*>(s_part + (16 + srow) * LD_SLD + slane * 4);
      float v[4] = {x.x + y.x, x.y + y.y, x.z + y.z, x.w + y.w};
      const int tok = (j0 + j) * LD_TOK + slane * 4;
      float mx = -INFINITY;
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        v[i] = tok + i < ctx && tok + i >= lo ? v[i] * scale_log2 : -INFINITY;
        mx = fmaxf(mx, v[i]);
      }
#pragma unroll
      for (int d = 8; d > 0; d >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, d));
      const float m_new = fmaxf(m_run, mx);                         // finite: every tile holds a visible token
      const float alpha = exp2f(m_run - m_new);
      float sum = 0.f;
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        v[i] = exp2f(v[i] - m_new);
        sum += v[i];
      }
      l_run = l_run * alpha + sum;
      m_run = m_new;
      *reinterpret_cast<uint2*>(smem + L.off_p + sw128_offset(srow, slane >> 1) + (slane & 1) * 8) =
          make_uint2(pack_bf16x2(v[0], v[1]), pack_bf16x2(v[2], v[3]));
      if (slane == 0) s_alpha[srow] = alpha;
    }
    __syncthreads();
    // ---- values
    const float al0 = s_alpha[lane >> 2], al1 = s_alpha[(lane >> 2) + 8];
#pragma unroll
    for (int n = 0; n < NT; ++n) {
      o[n][0] *= al0;
      o[n][1] *= al0;
      o[n][2] *= al1;
      o[n][3] *= al1;
    }
#pragma unroll
    for (int ks = 0; ks < 4; ++ks) {
      uint32_t pa[4];
      ld_matrix4(p_addr + sw128_offset(a_row, ks * 2 + a_unit), pa);
#pragma unroll
      for (int n = 0; n < NT; n += 2) {
        const int col = col0 + n * 8;
        if (col < cols) {
          uint32_t vb[4];
          ld_matrix4_trans(tile + (col >> 6) * LD_CHUNK + sw128_offset(ks * 16 + v_tok, ((col & 63) >> 3) + v_unit), vb);
          ld_mma(o[n], pa, vb[0], vb[1]);
          ld_mma(o[n + 1], pa, vb[2], vb[3]);
        }
      }
    }
    __syncthreads();                                                // tile, partials and P are free again
    if (warp == 0 && j + L.stages < mine) issue(j + L.stages);
  }

  if (!ok) {                                    // copies in flight land in this CTA's memory: give them time
    const long long t0 = clock64();
    while (clock64() - t0 < 10000000LL) {}
    __syncthreads();
  }
#pragma unroll
  for (int d = 8; d > 0; d >>= 1) l_run += __shfl_xor_sync(0xffffffffu, l_run, d);
  const int r0 = lane >> 2;
  if (splits == 1) {                            // nothing to merge: the sink, then the quotient
    if (slane == 0) {
      const float sk = sink && srow < G ? sink[h0 + srow] * 1.4426950408889634f : -INFINITY, M = fmaxf(m_run, sk);
      const float w = exp2f(m_run - M);
      s_alpha[srow] = w / (w * l_run + exp2f(sk - M));
    }
    __syncthreads();
    const float w0 = s_alpha[r0], w1 = s_alpha[r0 + 8];
    __nv_bfloat16* dst = out + ((long long)b * s.heads + h0) * s.rank_p;
#pragma unroll
    for (int n = 0; n < NT; ++n) {
      const int col = col0 + n * 8 + 2 * (lane & 3);
      if (col < s.rank_p) {
        if (r0 < G) *reinterpret_cast<uint32_t*>(dst + r0 * s.rank_p + col) = pack_bf16x2(o[n][0] * w0, o[n][1] * w0);
        if (r0 + 8 < G) *reinterpret_cast<uint32_t*>(dst + (r0 + 8) * s.rank_p + col) = pack_bf16x2(o[n][2] * w1, o[n][3] * w1);
      }
    }
    return;
  }
  // this split's state: the weighted latents, then maximum and sum
  const int stride = s.rank_p + 4;
  float* part = scratch + (((long long)b * s.heads + h0) * splits + split) * stride;     // head h: + h * splits * stride
  if (slane == 0 && srow < G)
    *reinterpret_cast<float2*>(part + (long long)srow * splits * stride + s.rank_p) = make_float2(ok ? m_run : -INFINITY, l_run);
#pragma unroll
  for (int n = 0; n < NT; ++n) {
    const int col = col0 + n * 8 + 2 * (lane & 3);
    if (col < s.rank_p) {
      if (r0 < G) *reinterpret_cast<float2*>(part + (long long)r0 * splits * stride + col) = make_float2(o[n][0], o[n][1]);
      if (r0 + 8 < G)
        *reinterpret_cast<float2*>(part + (long long)(r0 + 8) * splits * stride + col) = make_float2(o[n][2], o[n][3]);
    }
  }
}

// One CTA per (token, head): the splits' states and the sink into one result.
__global__ void __launch_bounds__(128)
latent_merge_kernel(const float* __restrict__ scratch, const float* __restrict__ sink, __nv_bfloat16* __restrict__ out, int heads,
                    int rank_p, int splits) {
  __shared__ float s_w[LD_MAX_SPLITS], s_sum;
  const int stride = rank_p + 4;
  const float* base = scratch + (long long)blockIdx.x * splits * stride;
  if (threadIdx.x < 32) {
    const int lane = threadIdx.x;
    float2 ml[2];
    const float sk = sink ? sink[blockIdx.x % heads] * 1.4426950408889634f : -INFINITY;
    float M = sk;
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int k = lane + 32 * i;
      ml[i] = k < splits ? *reinterpret_cast<const float2*>(base + (long long)k * stride + rank_p) : make_float2(-INFINITY, 0.f);
      M = fmaxf(M, ml[i].x);
    }
    M = warp_max(M);
    float sum = 0.f;
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const float w = exp2f(ml[i].x - M);
      s_w[lane + 32 * i] = w;
      if (w > 0.f) sum += w * ml[i].y;
    }
    sum = warp_sum(sum) + exp2f(sk - M);
    if (lane == 0) s_sum = 1.f / sum;
  }
  __syncthreads();
  const float inv = s_sum;
  for (int d = threadIdx.x * 4; d < rank_p; d += 512) {
    float4 y = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 8
    for (int k = 0; k < splits; ++k) {
      const float4 v = *reinterpret_cast<const float4*>(base + (long long)k * stride + d);
      const float w = s_w[k];
      if (w > 0.f) {                            // an empty split's numbers are never used
        y.x = fmaf(w, v.x, y.x);
        y.y = fmaf(w, v.y, y.y);
        y.z = fmaf(w, v.z, y.z);
        y.w = fmaf(w, v.w, y.w);
      }
    }
    *reinterpret_cast<uint2*>(out + (long long)blockIdx.x * rank_p + d) =
        make_uint2(pack_bf16x2(y.x * inv, y.y * inv), pack_bf16x2(y.z * inv, y.w * inv));
  }
}

}  // namespace

void latent_prep(bool f32, void* proj, long long ld, const LatentPrep& p, const LatentSpec& s, const RaggedBatch& rb,
                 const LatentPages& pg, float eps, cudaStream_t stream) {
  MB_REQUIRE(s.rot > 0 && s.rot % 2 == 0 && s.rot <= 2048, "latent_prep: rotated width");
  for (int off : {p.low_off, p.qr_off, p.c_off, p.kr_off}) MB_REQUIRE(off < 0 || off % 8 == 0, "latent_prep: columns in units of 8");
  MB_REQUIRE(ld % 8 == 0 && (p.c_off < 0 || (p.kr_off >= 0 && p.gamma)) && (p.low_off < 0 || (p.low_gamma && p.low_rank > 0)) &&
                 ((reinterpret_cast<uintptr_t>(proj) | reinterpret_cast<uintptr_t>(p.gamma) | reinterpret_cast<uintptr_t>(p.low_gamma)) & 15) == 0,
             "latent_prep: arguments");
  if (rb.rows == 0) return;
  const int smem = LP_WARPS * (s.rot_p / 2) * (int)sizeof(float2), grid = (rb.rows + LP_WARPS - 1) / LP_WARPS;
  const bool rows = p.low_off >= 0 || p.c_off >= 0;
#define MB_LP(T, ROWS) latent_prep_kernel<T, ROWS><<<grid, LP_WARPS * 32, smem, stream>>>((T*)proj, ld, p, s, rb, pg, eps)
  if (f32) { if (rows) MB_LP(float, true); else MB_LP(float, false); }
  else     { if (rows) MB_LP(__nv_bfloat16, true); else MB_LP(__nv_bfloat16, false); }
#undef MB_LP
  count_launch();
  check_launch();
}

void latent_gather(const LatentSpec& s, const LatentPages& pg, const int* cu_k, const int* first, int n_seq, int max_kv, void* out,
                   cudaStream_t stream) {
  if (n_seq == 0 || max_kv == 0) return;
  const int units = s.row() / 8;
  const long long want = ((long long)max_kv * units + 1023) / 1024;
  const dim3 grid((unsigned)(want < 2048 ? want : 2048), n_seq);
  latent_gather_kernel<<<grid, 256, 0, stream>>>(pg, cu_k, first, (uint4*)out, units);
  count_launch();
  check_launch();
}

void latent_attn_any(bool f32, const LatentQuery& q, const LatentSpec& s, const LatentPages& pg, const float* sink, void* out,
                     float scale, cudaStream_t stream) {
  MB_REQUIRE(s.rank_p <= 1024 && s.row() <= 3000, "latent_attn_any: latents up to 1024 wide");
  if (q.rows == 0) return;
  const int grid = ceil_div((long long)q.rows * s.heads, LA_WARPS), smem = LA_WARPS * s.row() * 4;
#define MB_LA(T, ND) latent_attn_any_kernel<T, ND><<<grid, LA_WARPS * 32, smem, stream>>>(q, s, pg, sink, (T*)out, scale)
#define MB_LAT(T)                                                                                                   \
  do {                                                                                                              \
    if (s.rank_p <= 64) MB_LA(T, 2); else if (s.rank_p <= 128) MB_LA(T, 4); else if (s.rank_p <= 256) MB_LA(T, 8);  \
    else if (s.rank_p <= 512) MB_LA(T, 16); else MB_LA(T, 32);                                                      \
  } while (0)
  if (f32) MB_LAT(float); else MB_LAT(__nv_bfloat16);
#undef MB_LAT
#undef MB_LA
  count_launch();
  check_launch();
}

bool latent_decode_ok(const LatentSpec& s, int page_size) {
  return page_size == 16 && s.rank_p <= 512 && ld_layout(s.row()).stages >= 2;
}

void latent_attn_decode(const LatentQuery& q, const LatentSpec& s, const LatentPages& pg, const float* sink, void* out,
                        float* scratch, int splits, float scale, int* status, cudaStream_t stream) {
  MB_REQUIRE(latent_decode_ok(s, pg.page_size), "latent_attn_decode: widths or page size");
  MB_REQUIRE(splits >= 1 && splits <= LD_MAX_SPLITS && q.ld_qr % 8 == 0, "latent_attn_decode: splits / stride");
  if (q.rows == 0) return;
  uint64_t dims[2] = {(uint64_t)s.row(), (uint64_t)pg.pages * 16}, strides[1] = {(uint64_t)s.row() * 2};
  uint32_t box[2] = {64, 16};
  const CUtensorMap tc = make_tensor_map(pg.cache, TmaDType::BF16, 2, dims, strides, box, true);
  const int smem = ld_layout(s.row()).bytes;
  const dim3 grid(q.rows, (s.heads + 15) / 16, splits);
  auto go = [&](auto kern) {
    MB_CUDA_CHECK(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
    kern<<<grid, LD_THREADS, smem, stream>>>(tc, q, s, pg, sink, (__nv_bfloat16*)out, scratch, splits,
                                             scale * 1.4426950408889634f, status);
  };
  if (s.rank_p <= 128) go(latent_decode_kernel<2>);
  else if (s.rank_p <= 256) go(latent_decode_kernel<4>);
  else go(latent_decode_kernel<8>);
  count_launch();
  check_launch();
  if (splits > 1) {
    latent_merge_kernel<<<q.rows * s.heads, 128, 0, stream>>>(scratch, sink, (__nv_bfloat16*)out, s.heads, s.rank_p, splits);
    count_launch();
    check_launch();
  }
}

}  // namespace mb
