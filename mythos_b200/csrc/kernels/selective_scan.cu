// Selective scan (hybrid_api.h): a diagonal recurrence per channel whose step size, input map and read-out map
// depend on the token.
//
//   selective_scan  prompts and portions: a thread owns NR state values of a channel in registers and walks the
//                   tokens of a chunk; tiles of inputs pass through shared memory by TMA, B and C of a token are read
//                   by all channels.
//                   Chunks of a long portion run side by side: kernel 1 forms each chunk's state from zero and the sum
//                   of its step sizes (the decay over a chunk is exp(A sum dt)), kernel 2 composes the states before
//                   a chunk, walks it again and reads out.
//   selective_step  one token per sequence: the same update on the stored state, for few sequences with the map to
//                   the step sizes inside.
//
// The short convolution in front of it is short_conv.cu.
//
// Step sizes, decays, states and the read-out are fp32 in both activation types. A is stored times log2(e), so a
// decay is one exp2.
#include <type_traits>

#include "common.cuh"
#include "host_util.h"
#include "hybrid_api.h"
#include "hybrid_dev.cuh"
#include "tc.cuh"

namespace mb {
namespace {

constexpr int SS_THREADS = 128;
constexpr int SS_TILE = 16;            // tokens of a tile (fewer for wide states)
constexpr int SS_BLOCKS = 4;           // blocks of a scan that fit into an SM
constexpr int SS_STAGES = 3;           // tiles in flight
constexpr int SS_GROUP = 4;            // tokens handled together
constexpr int SS_TILE_VALUES = 2048;   // at most this many values of B (and of C) in a tile
constexpr int SS_CHUNK = 64;           // shortest chunk

// A channel's state values lie on `lanes` neighbouring threads, nr on each.
struct StateMap {
  int nr, lanes;
};
StateMap state_map(int state) {
  StateMap m{0, 1};
  while ((state + m.lanes - 1) / m.lanes > 16) m.lanes *= 2;
  m.nr = ((state + m.lanes - 1) / m.lanes + 3) / 4 * 4;
  return m;
}

// ln(1 + e) for 0 <= e <= 1 as 2 artanh(e / (2 + e)), series in t^2 <= 1/9.
__device__ __forceinline__ float log1p_unit(float e) {
  const float t = e * fast_rcp(2.f + e), t2 = t * t;
  float p = fmaf(t2, 1.f / 15.f, 1.f / 13.f);
  p = fmaf(p, t2, 1.f / 11.f);
  p = fmaf(p, t2, 1.f / 9.f);
  p = fmaf(p, t2, 1.f / 7.f);
  p = fmaf(p, t2, 1.f / 5.f);
  p = fmaf(p, t2, 1.f / 3.f);
  p = fmaf(p, t2, 1.f);
  return 2.f * t * p;
}
__device__ __forceinline__ float softplus_fast(float z) { return fmaxf(z, 0.f) + log1p_unit(fast_exp2(-1.4426950408889634f * fabsf(z))); }
// 2^x for x <= 0 by its Taylor series about the nearest integer, the last step one rounding: a decay just below one is
// off by half a unit in the last place either way, so thousands of them in a row do not drift.
__device__ __forceinline__ float exp2_series(float x) {
  x = fmaxf(x, -126.f);
  const float i = rintf(x), f = x - i;
  float p = fmaf(f, 1.5252734e-5f, 1.5403530e-4f);       // ln(2)^k / k!, k = 7 .. 1
  p = fmaf(p, f, 1.3333558e-3f);
  p = fmaf(p, f, 9.6181291e-3f);
  p = fmaf(p, f, 5.5504109e-2f);
  p = fmaf(p, f, 2.4022651e-1f);
  p = fmaf(p, f, 6.9314718e-1f);
  p = fmaf(p, f, 1.f);
  return x <= -126.f ? 0.f : p * __int_as_float(((int)i + 127) << 23);
}
// Decays, step sizes and gates: with 32-bit activations as exactly as 32-bit arithmetic goes, with 16-bit ones by the
// special-function unit (relative error about 2^-22).
template <typename T>
__device__ __forceinline__ float decay_t(float x) {
  if constexpr (sizeof(T) == 2) return fast_exp2(x);
  else return exp2_series(x);
}
template <typename T>
__device__ __forceinline__ float softplus_t(float z) {
  if constexpr (sizeof(T) == 2) return softplus_fast(z);
  else return softplus_f(z);
}
// ---------------------------------------------------------------------------------------------
// Scratch of a chunked scan: the state every sequence starts from, and per chunk its own state (from zero) and the sum
// of its step sizes.
struct ChunkScratch {
  float *init, *ends, *sums;       // [n_seq][inner][state], [n_seq][chunks][inner][state], [n_seq][chunks][inner]
};

// State update of one token on packed pairs of state values; the read-out is formed when Y.
template <typename T, int NR, bool Y>
__device__ __forceinline__ float advance(uint64_t (&S)[NR / 2], const uint64_t (&a)[NR / 2], float dt, float x, const float* sB,
                                         const float* sC) {
  const uint64_t dt2 = f32x2(dt, dt), dx2 = f32x2(dt * x, dt * x);
  uint64_t y[2] = {0ull, 0ull};
#pragma unroll
  for (int i = 0; i < NR / 4; ++i) {
    const ulonglong2 B = reinterpret_cast<const ulonglong2*>(sB)[i];
    ulonglong2 C{};
    if constexpr (Y) C = reinterpret_cast<const ulonglong2*>(sC)[i];
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      const int n = 2 * i + j;
      float e0, e1;
      f32x2_unpack(mul_f32x2(dt2, a[n]), e0, e1);
      S[n] = fma_f32x2(f32x2(decay_t<T>(e0), decay_t<T>(e1)), S[n], mul_f32x2(dx2, j ? B.y : B.x));
      if constexpr (Y) y[j] = fma_f32x2(S[n], j ? C.y : C.x, y[j]);
    }
  }
  if constexpr (!Y) return 0.f;
  float y0, y1;
  f32x2_unpack(add_f32x2(y[0], y[1]), y0, y1);
  return y0 + y1;
}
template <int NR>
__device__ __forceinline__ void load_pairs(const float* p, uint64_t (&v)[NR / 2]) {
#pragma unroll
  for (int i = 0; i < NR / 4; ++i) {
    const ulonglong2 t = reinterpret_cast<const ulonglong2*>(p)[i];
    v[2 * i] = t.x;
    v[2 * i + 1] = t.y;
  }
}
template <int NR>
__device__ __forceinline__ void store_pairs(float* p, const uint64_t (&v)[NR / 2]) {
#pragma unroll
  for (int i = 0; i < NR / 4; ++i) reinterpret_cast<ulonglong2*>(p)[i] = make_ulonglong2(v[2 * i], v[2 * i + 1]);
}

// Inputs of a tile of tokens in shared memory: [token][channel of the block] x, z (T) and pre-activations, and
// [token][row] B and C as they lie in memory (T). SS_STAGES of them form a ring.
template <typename T>
struct TileLayout {
  int tokens, channels, row;       // row: state values of B (and of C) per token, a whole number of 16-byte units
  static __host__ __device__ int up(int n) { return (n + 127) / 128 * 128; }
  __host__ __device__ int x() const { return 0; }
  __host__ __device__ int z() const { return up(tokens * channels * (int)sizeof(T)); }
  __host__ __device__ int dt() const { return 2 * z(); }
  __host__ __device__ int b() const { return dt() + up(tokens * channels * 4); }
  __host__ __device__ int c() const { return b() + up(tokens * row * (int)sizeof(T)); }
  __host__ __device__ int bytes() const { return c() + up(tokens * row * (int)sizeof(T)); }
  // bytes of a tile's copies
  __host__ __device__ int loaded(bool out) const {
    return tokens * ((out ? 2 : 1) * (channels + row) * (int)sizeof(T) + channels * 4);
  }
};
struct TileMaps {
  CUtensorMap x, z, dt, b, c, out;
};

// Quotients of small numbers by one that is not a constant (exact below 2^22).
struct Quotient {
  float inv;
  __device__ __forceinline__ explicit Quotient(int d) : inv(1.f / (float)d) {}
  __device__ __forceinline__ int operator()(int i) const { return (int)(((float)i + 0.5f) * inv); }
};
// n rows of `cols` values: dst (row stride dst_ld) <- src (row stride ld)
template <typename E>
__device__ __forceinline__ void copy_rows(E* dst, long long dst_ld, const E* src, long long ld, int n, int cols) {
  const Quotient by(cols);
  for (int i = threadIdx.x; i < n * cols; i += SS_THREADS) {
    const int r = by(i), c = i - r * cols;
    dst[r * dst_ld + c] = src[r * ld + c];
  }
}

// grid (channel blocks, chunks, sequences). OUT: read out and store; else form the chunk's summary. tma: tiles arrive
// and leave by TMA (rows of whole 16-byte units), else by plain copies. LANES: threads per channel (0: `lanes_`).
template <typename T, int NR, bool OUT, int LANES>
__global__ void __launch_bounds__(SS_THREADS, SS_BLOCKS)
selective_scan_kernel(const __grid_constant__ SelectiveSpec s, const __grid_constant__ SelectiveInputs in,
                      const __grid_constant__ RaggedBatch rb, int lanes_, int chunk, int chunks, const float* __restrict__ dt,
                      long long ld_dt, ChunkScratch sc, T* __restrict__ out, long long ldo, TileLayout<T> lay, bool tma,
                      const __grid_constant__ TileMaps maps, int* status) {
  extern __shared__ uint8_t smem_raw[];
  __shared__ uint64_t full[SS_STAGES];
  __shared__ int abort_word;
  volatile int* abort_flag = &abort_word;
  uint8_t* smem = smem_raw + ((128u - (smem_u32(smem_raw) & 127u)) & 127u);
  const int lanes = LANES > 0 ? LANES : lanes_, channels = SS_THREADS / lanes;
  const int b = blockIdx.z, k = blockIdx.y;
  const int row0 = rb.cu_q[b], len = rb.cu_q[b + 1] - row0, t0 = k * chunk;
  if (t0 >= len) return;
  const int t1 = min(len, t0 + chunk), state_p = NR * lanes;
  const bool last = t1 == len;
  if (!OUT && last) return;                        // nothing starts from the last chunk's state
  const int cl = threadIdx.x / lanes, sub = threadIdx.x % lanes, c0 = blockIdx.x * channels;
  const bool live = c0 + cl < s.inner;
  const int ch = live ? c0 + cl : s.inner - 1, width = min(channels, s.inner - c0);
  const int tile = lay.tokens, tiles = (t1 - t0 + tile - 1) / tile;
  if (threadIdx.x == 0) {
    for (int i = 0; i < SS_STAGES; ++i) mbar_init(&full[i], 1);
    *abort_flag = 0;
    fence_mbar_init();
  }
  __syncthreads();
  auto fetch = [&](int i) {                        // by TMA: one thread
    const int st = i % SS_STAGES, row = row0 + t0 + i * tile;
    uint8_t* buf = smem + st * lay.bytes();
    mbar_arrive_expect_tx(&full[st], (uint32_t)lay.loaded(OUT));
    tma_load_2d(buf + lay.x(), &maps.x, &full[st], c0, row);
    tma_load_2d(buf + lay.dt(), &maps.dt, &full[st], c0, row);
    tma_load_2d(buf + lay.b(), &maps.b, &full[st], 0, row);
    if constexpr (OUT) {
      tma_load_2d(buf + lay.z(), &maps.z, &full[st], c0, row);
      tma_load_2d(buf + lay.c(), &maps.c, &full[st], 0, row);
    }
  };
  if (tma && threadIdx.x == 0)
    for (int i = 0; i < SS_STAGES - 1 && i < tiles; ++i) fetch(i);
  const bool fresh = rb.kv_lens[b] == len;
  float* slot = in.state + ((long long)rb.slots[b] * s.inner + ch) * state_p + sub * NR;
  uint64_t a[NR / 2], S[NR / 2];                   // pairs of state values
  load_pairs<NR>(in.a + (long long)ch * state_p + sub * NR, a);
  if (OUT && (k > 0 || !last)) {                   // several chunks: the slot may already hold the final state
    load_pairs<NR>(sc.init + ((long long)b * s.inner + ch) * state_p + sub * NR, S);
    for (int i = 0; i < k; ++i) {
      const long long at = ((long long)b * chunks + i) * s.inner + ch;
      const float sum = sc.sums[at];
      uint64_t e[NR / 2];
      load_pairs<NR>(sc.ends + at * state_p + sub * NR, e);
#pragma unroll
      for (int n = 0; n < NR / 2; ++n) {
        float d0, d1;
        f32x2_unpack(mul_f32x2(f32x2(sum, sum), a[n]), d0, d1);
        S[n] = fma_f32x2(f32x2(decay_t<T>(d0), decay_t<T>(d1)), S[n], e[n]);
      }
    }
  } else {
#pragma unroll
    for (int n = 0; n < NR / 2; ++n) S[n] = 0ull;
    if ((OUT || k == 0) && !fresh) load_pairs<NR>(slot, S);
    if (!OUT && k == 0) {
      if (live) store_pairs<NR>(sc.init + ((long long)b * s.inner + ch) * state_p + sub * NR, S);
#pragma unroll
      for (int n = 0; n < NR / 2; ++n) S[n] = 0ull;
    }
  }
  const float bias = in.dt_bias[ch], D = OUT ? in.d[ch] : 0.f, scale = s.out_scale;
  // B, then C, of the tile in fp32, zeros in the padding
  float* sB = reinterpret_cast<float*>(smem + (tma ? SS_STAGES : 1) * lay.bytes());
  float* sC = sB + tile * state_p;
  float total = 0.f;
  for (int i = 0; i < tiles; ++i) {
    const int tt = t0 + i * tile, n = min(tile, t1 - tt), st = tma ? i % SS_STAGES : 0;
    uint8_t* buf = smem + st * lay.bytes();
    if (tma) {
      const bool ok = mbar_wait(&full[st], (i / SS_STAGES) & 1, abort_flag, status, 110);
      if (!__syncthreads_and(ok)) break;           // also: nobody reads B and C of the tile before any more
    } else {
      __syncthreads();
      const long long row = row0 + tt;
      copy_rows((T*)(buf + lay.x()), channels, static_cast<const T*>(in.x) + row * in.ld_x + c0, in.ld_x, n, width);
      copy_rows((float*)(buf + lay.dt()), channels, dt + row * ld_dt + c0, ld_dt, n, width);
      copy_rows((T*)(buf + lay.b()), lay.row, static_cast<const T*>(in.low) + row * in.ld_low + in.b_off, in.ld_low, n, s.state);
      if constexpr (OUT) {
        copy_rows((T*)(buf + lay.z()), channels, static_cast<const T*>(in.proj) + row * in.ld + in.z_off + c0, in.ld, n, width);
        copy_rows((T*)(buf + lay.c()), lay.row, static_cast<const T*>(in.low) + row * in.ld_low + in.c_off, in.ld_low, n, s.state);
      }
      __syncthreads();
    }
    const Quotient by_state(state_p);
    for (int j = threadIdx.x; j < n * state_p; j += SS_THREADS) {
      const int u = by_state(j), v = j - u * state_p;
      sB[j] = v < s.state ? ldf((const T*)(buf + lay.b()) + u * lay.row + v) : 0.f;
      if constexpr (OUT) sC[j] = v < s.state ? ldf((const T*)(buf + lay.c()) + u * lay.row + v) : 0.f;
    }
    __syncthreads();
    T* sx = (T*)(buf + lay.x()) + cl;
    const T* sz = (const T*)(buf + lay.z()) + cl;
    const float* sd = (const float*)(buf + lay.dt()) + cl;
    const float *pB = sB + sub * NR, *pC = sC + sub * NR;
    // G tokens at a time: their step sizes and gates overlap, and no store lies between their state updates
    auto run = [&](auto group, int u0) {
      constexpr int G = decltype(group)::value;
      float x[G], d[G], y[G];
#pragma unroll
      for (int g = 0; g < G; ++g) {
        x[g] = ldf(sx + (u0 + g) * channels);
        d[g] = softplus_t<T>(sd[(u0 + g) * channels] + bias);
        if constexpr (!OUT) total += d[g];
      }
#pragma unroll
      for (int g = 0; g < G; ++g) y[g] = advance<T, NR, OUT>(S, a, d[g], x[g], pB + (u0 + g) * state_p, pC + (u0 + g) * state_p);
      if constexpr (OUT) {
        for (int o = 1; o < lanes; o <<= 1)
#pragma unroll
          for (int g = 0; g < G; ++g) y[g] += __shfl_xor_sync(0xffffffffu, y[g], o);
#pragma unroll
        for (int g = 0; g < G; ++g) y[g] = fmaf(D, x[g], y[g]) * scale * silu_t<T>(ldf(sz + (u0 + g) * channels));
        if (sub == 0) {                            // the output takes x's place
#pragma unroll
          for (int g = 0; g < G; ++g) stf(sx + (u0 + g) * channels, y[g]);
        }
      }
    };
    int u = 0;
    for (; u + SS_GROUP <= n; u += SS_GROUP) run(std::integral_constant<int, SS_GROUP>{}, u);
    for (; u < n; ++u) run(std::integral_constant<int, 1>{}, u);
    if (OUT && tma) fence_proxy_async_smem();
    __syncthreads();
    if (tma && threadIdx.x == 0) {
      // the tile before has long been read by its store: its place takes the tile after the next
      if constexpr (OUT) tma_store_wait_read0();
      if (i + SS_STAGES - 1 < tiles) fetch(i + SS_STAGES - 1);
      if (OUT && n == tile) {
        tma_store_2d(&maps.out, buf + lay.x(), c0, row0 + tt);
        tma_store_commit();
      }
    }
    if (OUT && !(tma && n == tile))
      copy_rows(out + (long long)(row0 + tt) * ldo + c0, ldo, (const T*)(buf + lay.x()), channels, n, width);
  }
  if (tma && *abort_flag) {        // copies in flight land in this CTA's memory: give them time
    const long long c = clock64();
    while (clock64() - c < 10000000LL) {}
    return;
  }
  if (OUT && tma && threadIdx.x == 0) tma_store_wait_read0();
  if (!live) return;
  if constexpr (OUT) {
    if (last) store_pairs<NR>(slot, S);
  } else {
    const long long at = ((long long)b * chunks + k) * s.inner + ch;
    store_pairs<NR>(sc.ends + at * state_p + sub * NR, S);
    if (sub == 0) sc.sums[at] = total;
  }
}

// grid (channel blocks, sequences), one token each.
template <typename T, int NR>
__global__ void __launch_bounds__(SS_THREADS)
selective_step_kernel(SelectiveSpec s, SelectiveInputs in, RaggedBatch rb, int lanes, const float* __restrict__ dt,
                      long long ld_dt, const T* __restrict__ w_dt, long long ld_w, T* __restrict__ out, long long ldo) {
  extern __shared__ __align__(16) float sm[];
  const int b = blockIdx.y, state_p = NR * lanes;
  const int idx = blockIdx.x * SS_THREADS + threadIdx.x, sub = idx % lanes;
  const bool live = idx / lanes < s.inner;
  const int ch = live ? idx / lanes : s.inner - 1;
  float* slot = in.state + ((long long)rb.slots[b] * s.inner + ch) * state_p + sub * NR;
  uint64_t a[NR / 2], S[NR / 2];
#pragma unroll
  for (int n = 0; n < NR / 2; ++n) S[n] = 0ull;
  if (rb.kv_lens[b] > 1) load_pairs<NR>(slot, S);
  load_pairs<NR>(in.a + (long long)ch * state_p + sub * NR, a);
  const T* low = static_cast<const T*>(in.low) + b * in.ld_low;
  float *sB = sm, *sC = sm + state_p, *sR = sC + state_p;
  for (int v = threadIdx.x; v < state_p; v += SS_THREADS) {
    sB[v] = v < s.state ? ldf(low + in.b_off + v) : 0.f;
    sC[v] = v < s.state ? ldf(low + in.c_off + v) : 0.f;
  }
  const int rank_p = (s.rank + 7) / 8 * 8;         // columns past the rank are zero on both sides
  if (!dt)
    for (int v = threadIdx.x; v < rank_p; v += SS_THREADS) sR[v] = ldf(low + v);
  __syncthreads();
  const float x = ldf(static_cast<const T*>(in.x) + b * in.ld_x + ch);
  const float z = ldf(static_cast<const T*>(in.proj) + b * in.ld + in.z_off + ch);
  float pre;
  if (dt) {
    pre = dt[b * ld_dt + ch];
  } else {
    pre = 0.f;
    for (int i = sub * 8; i < rank_p; i += 8 * lanes) {
      float w[8];
      load_v<8>(w_dt + (long long)ch * ld_w + i, w);
#pragma unroll
      for (int j = 0; j < 8; ++j) pre = fmaf(w[j], sR[i + j], pre);
    }
    for (int o = 1; o < lanes; o <<= 1) pre += __shfl_xor_sync(0xffffffffu, pre, o);
  }
  const float d = softplus_t<T>(pre + in.dt_bias[ch]);
  float y = advance<T, NR, true>(S, a, d, x, sB + sub * NR, sC + sub * NR);
  for (int o = 1; o < lanes; o <<= 1) y += __shfl_xor_sync(0xffffffffu, y, o);
  if (!live) return;
  store_pairs<NR>(slot, S);
  if (sub == 0) stf(out + b * ldo + ch, fmaf(in.d[ch], x, y) * silu_t<T>(z) * s.out_scale);
}

void check_spec(const SelectiveSpec& s) {
  MB_REQUIRE(s.inner > 0 && s.rank > 0, "selective scan: sizes");
  MB_REQUIRE(s.state > 0 && s.state <= 512, "selective scan: at most 512 state values per channel");
}

// Chunks of the longest portion. Chunks cost a second pass, so a portion is cut only where its blocks leave SMs idle, and
// then into enough of them to fill every SM (measured: 4 blocks on an SM run twice as fast as one).
struct ChunkPlan {
  int chunk, chunks;
};
ChunkPlan plan_chunks(const SelectiveSpec& s, int rows, int max_q) {
  const StateMap m = state_map(s.state);
  if (max_q <= 0) return ChunkPlan{1, 1};
  const long long blocks = ((long long)s.inner * m.lanes + SS_THREADS - 1) / SS_THREADS * ((rows + max_q - 1) / max_q);
  long long chunks = blocks * 5 >= sm_count() * 4ll ? 1 : 6ll * sm_count() / blocks;
  const long long most = (max_q + SS_CHUNK - 1) / SS_CHUNK;
  if (chunks > most) chunks = most;
  if (chunks > 64) chunks = 64;
  if (chunks < 2) return ChunkPlan{max_q, 1};
  const int chunk = (int)((max_q + chunks - 1) / chunks);
  return ChunkPlan{chunk, (max_q + chunk - 1) / chunk};
}

}  // namespace

int selective_padded_state(int state) {
  const StateMap m = state_map(state);
  return m.nr * m.lanes;
}

long long selective_scratch(const SelectiveSpec& s, int n_seq, int rows, int max_q) {
  const ChunkPlan p = plan_chunks(s, rows, max_q);
  if (p.chunks <= 1) return 0;
  const long long state = (long long)s.inner * selective_padded_state(s.state);
  return n_seq * (state + p.chunks * (state + s.inner));
}

#define MB_SS_NR(GO)                                                        \
  if (m.nr == 4) GO(4); else if (m.nr == 8) GO(8); else if (m.nr == 12) GO(12); else GO(16)

void selective_scan(bool f32, const SelectiveSpec& s, const SelectiveInputs& in, const RaggedBatch& rb, int max_q,
                    const float* dt, long long ld_dt, float* scratch, void* out, long long ldo, int* status,
                    cudaStream_t stream) {
  check_spec(s);
  if (rb.rows == 0) return;
  MB_REQUIRE(max_q > 0 && rb.n_seq <= 65535, "selective_scan: batch");
  const StateMap m = state_map(s.state);
  const ChunkPlan p = plan_chunks(s, rb.rows, max_q);
  const int state_p = m.nr * m.lanes;
  const long long state = (long long)s.inner * state_p;
  ChunkScratch sc{scratch, scratch + rb.n_seq * state, scratch + rb.n_seq * state * (1 + p.chunks)};
  const dim3 grid((int)(((long long)s.inner * m.lanes + SS_THREADS - 1) / SS_THREADS), p.chunks, rb.n_seq);
  const int per = SS_TILE_VALUES / state_p, tile = per < SS_TILE ? per : SS_TILE;
  const int channels = SS_THREADS / m.lanes, es = f32 ? 4 : 2, unit = 16 / es;
  auto whole = [&](const void* p, long long ld, int off) {       // rows of 16-byte units
    return ((reinterpret_cast<uintptr_t>(p) + (uintptr_t)off * es) & 15) == 0 && ld % unit == 0;
  };
  const int row = (s.state + unit - 1) / unit * unit;
  const bool tma = channels % unit == 0 && channels % 4 == 0 && row <= 256 && whole(in.x, in.ld_x, 0) && whole(in.proj, in.ld, in.z_off) &&
                   whole(in.low, in.ld_low, in.b_off) && whole(in.low, in.ld_low, in.c_off) && whole(out, ldo, 0) &&
                   ld_dt % 4 == 0 && (reinterpret_cast<uintptr_t>(dt) & 15) == 0;
  TileMaps maps{};
  if (tma) {
    auto map = [&](const void* p, long long ld, int off, int cols, int box_cols, int size) {
      uint64_t dims[2] = {(uint64_t)cols, (uint64_t)rb.rows}, strides[1] = {(uint64_t)ld * size};
      uint32_t box[2] = {(uint32_t)box_cols, (uint32_t)tile};
      return make_tensor_map((const char*)p + (long long)off * size, size == 4 ? TmaDType::F32 : TmaDType::BF16, 2, dims, strides, box,
                             false);
    };
    maps.x = map(in.x, in.ld_x, 0, s.inner, channels, es);
    maps.z = map(in.proj, in.ld, in.z_off, s.inner, channels, es);
    maps.dt = map(dt, ld_dt, 0, s.inner, channels, 4);
    maps.b = map(in.low, in.ld_low, in.b_off, s.state, row, es);
    maps.c = map(in.low, in.ld_low, in.c_off, s.state, row, es);
    maps.out = map(out, ldo, 0, s.inner, channels, es);
  }
  auto go = [&](auto kernel, auto layout, auto* o) {
    layout.tokens = tile;
    layout.channels = channels;
    layout.row = row;
    const int smem = (tma ? SS_STAGES : 1) * layout.bytes() + 2 * tile * state_p * 4 + 128;
    MB_CUDA_CHECK(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
    kernel<<<grid, SS_THREADS, smem, stream>>>(s, in, rb, m.lanes, p.chunk, p.chunks, dt, ld_dt, sc, o, ldo, layout, tma, maps, status);
  };
#define MB_SS_L(T, NR, L)                                                                         \
  do {                                                                                            \
    if (p.chunks > 1) go(selective_scan_kernel<T, NR, false, L>, TileLayout<T>{}, (T*)out);       \
    go(selective_scan_kernel<T, NR, true, L>, TileLayout<T>{}, (T*)out);                          \
  } while (0)
#define MB_SS(T, NR) do { if (m.lanes == 1) MB_SS_L(T, NR, 1); else MB_SS_L(T, NR, 0); } while (0)
#define MB_SS_BF(NR) MB_SS(__nv_bfloat16, NR)
#define MB_SS_F(NR) MB_SS(float, NR)
  if (f32) { MB_SS_NR(MB_SS_F); } else { MB_SS_NR(MB_SS_BF); }
#undef MB_SS_F
#undef MB_SS_BF
#undef MB_SS
#undef MB_SS_L
  count_launch(p.chunks > 1 ? 2 : 1);
  check_launch();
}

void selective_step(bool f32, const SelectiveSpec& s, const SelectiveInputs& in, const RaggedBatch& rb, const float* dt,
                    long long ld_dt, const void* w_dt, long long ld_w, void* out, long long ldo, cudaStream_t stream) {
  check_spec(s);
  if (rb.n_seq == 0) return;
  MB_REQUIRE(rb.rows == rb.n_seq, "selective_step: one token per sequence");
  MB_REQUIRE(dt || (w_dt && ld_w % 8 == 0 && (reinterpret_cast<uintptr_t>(w_dt) & 15) == 0), "selective_step: step sizes or their map");
  const StateMap m = state_map(s.state);
  const int rank_p = (s.rank + 7) / 8 * 8, smem = (2 * m.nr * m.lanes + (dt ? 0 : rank_p)) * 4;
  MB_REQUIRE(smem <= 48 * 1024, "selective_step: map to the step sizes too wide");
  const dim3 grid((int)(((long long)s.inner * m.lanes + SS_THREADS - 1) / SS_THREADS), rb.n_seq);
#define MB_ST(T, NR)                                                                                            \
  selective_step_kernel<T, NR><<<grid, SS_THREADS, smem, stream>>>(s, in, rb, m.lanes, dt, ld_dt, (const T*)w_dt, ld_w, \
                                                                   (T*)out, ldo)
#define MB_ST_F(NR) MB_ST(float, NR)
#define MB_ST_BF(NR) MB_ST(__nv_bfloat16, NR)
  if (f32) { MB_SS_NR(MB_ST_F); } else { MB_SS_NR(MB_ST_BF); }
#undef MB_ST_F
#undef MB_ST_BF
#undef MB_ST
  count_launch();
  check_launch();
}
#undef MB_SS_NR

}  // namespace mb
