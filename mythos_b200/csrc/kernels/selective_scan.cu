// Selective scan (hybrid_api.h): a diagonal recurrence per channel whose step size, input map and read-out map
// depend on the token.
//
//   selective_conv  short causal convolution + silu of the channels, and its state
//   selective_scan  prompts and portions: a thread owns NR state values of a channel in registers and walks the
//                   tokens of a chunk; B and C of a tile of tokens lie in shared memory and are read by all channels.
//                   Chunks of a long portion run side by side: kernel 1 forms each chunk's state from zero and the sum
//                   of its step sizes (the decay over a chunk is exp(A sum dt)), kernel 2 composes the states before
//                   a chunk, walks it again and reads out.
//   selective_step  one token per sequence: the same update on the stored state, for few sequences with the map to
//                   the step sizes inside.
//
// Step sizes, decays, states and the read-out are fp32 in both activation types. A is stored times log2(e), so a
// decay is one exp2.
#include "common.cuh"
#include "host_util.h"
#include "hybrid_api.h"
#include "hybrid_dev.cuh"
#include "tc.cuh"

namespace mb {
namespace {

constexpr int SS_THREADS = 128;
constexpr int SS_GROUP = 4;            // tokens whose inputs are loaded together
constexpr int SS_TILE = 32;            // tokens whose B and C are staged together (fewer for wide states)
constexpr int SS_TILE_VALUES = 4096;   // at most this many values of B (and of C) in shared memory
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
  const float t = __fdividef(e, 2.f + e), t2 = t * t;
  float p = fmaf(t2, 1.f / 15.f, 1.f / 13.f);
  p = fmaf(p, t2, 1.f / 11.f);
  p = fmaf(p, t2, 1.f / 9.f);
  p = fmaf(p, t2, 1.f / 7.f);
  p = fmaf(p, t2, 1.f / 5.f);
  p = fmaf(p, t2, 1.f / 3.f);
  p = fmaf(p, t2, 1.f);
  return 2.f * t * p;
}
__device__ __forceinline__ float softplus_fast(float z) { return fmaxf(z, 0.f) + log1p_unit(expf(-fabsf(z))); }

template <int V>
__device__ __forceinline__ void load_v(const float* p, float (&f)[V]) {
  if constexpr (V % 4 == 0) {
#pragma unroll
    for (int i = 0; i < V / 4; ++i) {
      const float4 t = reinterpret_cast<const float4*>(p)[i];
      f[4 * i] = t.x; f[4 * i + 1] = t.y; f[4 * i + 2] = t.z; f[4 * i + 3] = t.w;
    }
  } else {
#pragma unroll
    for (int i = 0; i < V; ++i) f[i] = p[i];
  }
}
template <int V>
__device__ __forceinline__ void load_v(const __nv_bfloat16* p, float (&f)[V]) {
  if constexpr (V == 8) {
    unpack8(*reinterpret_cast<const bf16x8*>(p), f);
  } else {
#pragma unroll
    for (int i = 0; i < V; ++i) f[i] = __bfloat162float(p[i]);
  }
}
template <int V>
__device__ __forceinline__ void store_v(float* p, const float (&f)[V]) {
  if constexpr (V % 4 == 0) {
#pragma unroll
    for (int i = 0; i < V / 4; ++i) reinterpret_cast<float4*>(p)[i] = make_float4(f[4 * i], f[4 * i + 1], f[4 * i + 2], f[4 * i + 3]);
  } else {
#pragma unroll
    for (int i = 0; i < V; ++i) p[i] = f[i];
  }
}
template <int V>
__device__ __forceinline__ void store_v(__nv_bfloat16* p, const float (&f)[V]) {
  if constexpr (V == 8) {
    *reinterpret_cast<bf16x8*>(p) = pack8(f);
  } else {
#pragma unroll
    for (int i = 0; i < V; ++i) p[i] = __float2bfloat16(f[i]);
  }
}

// ---------------------------------------------------------------------------------------------
// V channels and SC_ROWS neighbouring rows per thread, so that a row's input is read about twice and not once per tap.
// TAPS: number of taps, weights held in registers (0: any number, weights read from the cache).
constexpr int SC_ROWS = 4;
template <typename T, int V, int TAPS>
__global__ void __launch_bounds__(256)
selective_conv_kernel(SelectiveSpec s, SelectiveInputs in, RaggedBatch rb, T* __restrict__ x, long long ldx) {
  const long long c = ((long long)blockIdx.x * blockDim.x + threadIdx.x) * V;
  const int r0 = blockIdx.y * SC_ROWS, n = min(SC_ROWS, rb.rows - r0), taps = TAPS > 0 ? TAPS : s.taps;
  if (c >= ldx) return;
  if (c >= s.inner) {                              // padding (V = 1)
    for (int r = 0; r < n; ++r) stf(x + (r0 + r) * ldx + c, 0.f);
    return;
  }
  float acc[SC_ROWS][V], wr[TAPS > 0 ? TAPS : 1][V];
  if constexpr (TAPS > 0) {
#pragma unroll
    for (int j = 0; j < TAPS; ++j) load_v<V>(in.conv_w + (long long)j * s.inner + c, wr[j]);
  }
  int lo[SC_ROWS];
#pragma unroll
  for (int r = 0; r < SC_ROWS; ++r) {
    lo[r] = r < n ? rb.cu_q[rb.row_seq[r0 + r]] : 0x7fffffff;
    load_v<V>(in.conv_b + c, acc[r]);
  }
  const T* col = static_cast<const T*>(in.proj) + in.x_off + c;
  auto add = [&](int j, const float (&v)[V], float (&a)[V]) {   // input v, j tokens before the current one
    if constexpr (TAPS > 0) {
#pragma unroll
      for (int k = 0; k < TAPS; ++k)
        if (k == j)
#pragma unroll
          for (int i = 0; i < V; ++i) a[i] = fmaf(wr[TAPS - 1 - k][i], v[i], a[i]);
    } else {
      float w[V];
      load_v<V>(in.conv_w + (long long)(taps - 1 - j) * s.inner + c, w);
#pragma unroll
      for (int i = 0; i < V; ++i) a[i] = fmaf(w[i], v[i], a[i]);
    }
  };
  auto source = [&](int k) {                       // row r0 - (taps - 1) + k
    const int src = r0 - (taps - 1) + k;
    if (src < 0 || src >= r0 + n) return;
    float v[V];
    load_v<V>(col + src * in.ld, v);
#pragma unroll
    for (int r = 0; r < SC_ROWS; ++r) {
      const int j = r + taps - 1 - k;
      if (j >= 0 && j < taps && src >= lo[r]) add(j, v, acc[r]);
    }
  };
  if constexpr (TAPS > 0) {
#pragma unroll
    for (int k = 0; k < TAPS - 1 + SC_ROWS; ++k) source(k);
  } else {
    for (int k = 0; k < taps - 1 + SC_ROWS; ++k) source(k);
  }
#pragma unroll
  for (int r = 0; r < SC_ROWS; ++r) {
    if (r >= n) break;
    const int i = r0 + r - lo[r];
    if (i < taps - 1) {                            // inputs before this portion: from the state, zeros before the start
      const int b = rb.row_seq[r0 + r];
      if (rb.kv_lens[b] > rb.cu_q[b + 1] - lo[r]) {
        const float* st = in.conv_state + (long long)rb.slots[b] * (taps - 1) * s.inner + c;
        for (int j = i + 1; j < taps; ++j) {
          float v[V];
          load_v<V>(st + (long long)(taps - 1 + i - j) * s.inner, v);
          add(j, v, acc[r]);
        }
      }
    }
#pragma unroll
    for (int q = 0; q < V; ++q) acc[r][q] = silu_f(acc[r][q]);
    store_v<V>(x + (r0 + r) * ldx + c, acc[r]);
  }
}

// One thread per (sequence, channel): the last taps - 1 inputs of the sequence become the state.
template <typename T>
__global__ void selective_conv_state_kernel(SelectiveSpec s, SelectiveInputs in, RaggedBatch rb) {
  const int c = blockIdx.x * blockDim.x + threadIdx.x, b = blockIdx.y;
  if (c >= s.inner) return;
  const int r0 = rb.cu_q[b], len = rb.cu_q[b + 1] - r0, n = s.taps - 1;
  if (len <= 0) return;
  const bool fresh = rb.kv_lens[b] == len;
  float* st = in.conv_state + (long long)rb.slots[b] * n * s.inner + c;
  const T* col = static_cast<const T*>(in.proj) + in.x_off + c;
  // entry j holds the input of token len - n + j; an entry moves down, never up, so in-place order is safe
  for (int j = 0; j < n; ++j) {
    const int i = len - n + j;
    float v;
    if (i >= 0) v = ldf(col + (long long)(r0 + i) * in.ld);
    else v = fresh ? 0.f : st[(long long)(n + i) * s.inner];
    st[(long long)j * s.inner] = v;
  }
}

// One token per sequence: convolution and its state in one pass, one channel per thread.
template <typename T>
__global__ void __launch_bounds__(256)
selective_conv_step_kernel(SelectiveSpec s, SelectiveInputs in, RaggedBatch rb, T* __restrict__ x, long long ldx) {
  const int c = blockIdx.x * blockDim.x + threadIdx.x, b = blockIdx.y;
  if (c >= ldx) return;
  if (c >= s.inner) {
    stf(x + b * ldx + c, 0.f);
    return;
  }
  const bool fresh = rb.kv_lens[b] <= 1;
  const float cur = ldf(static_cast<const T*>(in.proj) + b * in.ld + in.x_off + c);
  float acc = fmaf(in.conv_w[(long long)(s.taps - 1) * s.inner + c], cur, in.conv_b[c]);
  float* st = in.conv_state + (long long)rb.slots[b] * (s.taps - 1) * s.inner + c;
  const float* w = in.conv_w + c;
  if (s.taps == 4) {                               // all loads before the stores
    float old[3];
#pragma unroll
    for (int j = 0; j < 3; ++j) old[j] = fresh ? 0.f : st[(long long)j * s.inner];
#pragma unroll
    for (int j = 0; j < 3; ++j) acc = fmaf(w[(long long)j * s.inner], old[j], acc);
    st[0] = old[1];
    st[s.inner] = old[2];
    st[2ll * s.inner] = cur;
  } else {
    float nxt = cur;                               // newest first: entry j moves to j - 1
    for (int j = s.taps - 2; j >= 0; --j) {
      const float old = fresh ? 0.f : st[(long long)j * s.inner];
      acc = fmaf(w[(long long)j * s.inner], old, acc);
      st[(long long)j * s.inner] = nxt;
      nxt = old;
    }
  }
  stf(x + b * ldx + c, silu_f(acc));
}

// ---------------------------------------------------------------------------------------------
// Scratch of a chunked scan: the state every sequence starts from, and per chunk its own state (from zero) and the sum
// of its step sizes.
struct ChunkScratch {
  float *init, *ends, *sums;       // [n_seq][inner][state], [n_seq][chunks][inner][state], [n_seq][chunks][inner]
};

// State update of one token; the read-out is formed when Y.
template <int NR, bool Y>
__device__ __forceinline__ float advance(float (&S)[NR], const float (&a)[NR], float dt, float x, const float* sB, const float* sC) {
  const float dx = dt * x;
  float y[2] = {0.f, 0.f};
#pragma unroll
  for (int i = 0; i < NR / 4; ++i) {
    const float4 B = reinterpret_cast<const float4*>(sB)[i];
    const float bv[4] = {B.x, B.y, B.z, B.w};
    float cv[4];
    if constexpr (Y) {
      const float4 C = reinterpret_cast<const float4*>(sC)[i];
      cv[0] = C.x; cv[1] = C.y; cv[2] = C.z; cv[3] = C.w;
    }
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = 4 * i + j;
      S[n] = fmaf(fast_exp2(dt * a[n]), S[n], dx * bv[j]);
      if constexpr (Y) y[j & 1] = fmaf(S[n], cv[j], y[j & 1]);
    }
  }
  return y[0] + y[1];
}

// grid (channel blocks, chunks, sequences). OUT: read out and store; else form the chunk's summary.
template <typename T, int NR, bool OUT>
__global__ void __launch_bounds__(SS_THREADS)
selective_scan_kernel(SelectiveSpec s, SelectiveInputs in, RaggedBatch rb, int lanes, int chunk, int chunks,
                      const float* __restrict__ dt, long long ld_dt, ChunkScratch sc, T* __restrict__ out, long long ldo) {
  extern __shared__ __align__(16) float sm[];
  const int b = blockIdx.z, k = blockIdx.y;
  const int row0 = rb.cu_q[b], len = rb.cu_q[b + 1] - row0, t0 = k * chunk;
  if (t0 >= len) return;
  const int t1 = min(len, t0 + chunk), state_p = NR * lanes;
  const bool last = t1 == len;
  if (!OUT && last) return;                        // nothing starts from the last chunk's state
  const int idx = blockIdx.x * SS_THREADS + threadIdx.x, sub = idx % lanes;
  const bool live = idx / lanes < s.inner;
  const int ch = live ? idx / lanes : s.inner - 1;
  const bool fresh = rb.kv_lens[b] == len;
  float* slot = in.state + ((long long)rb.slots[b] * s.inner + ch) * state_p + sub * NR;
  float a[NR], S[NR];
  load_v<NR>(in.a + (long long)ch * state_p + sub * NR, a);
  if (OUT && (k > 0 || !last)) {                   // several chunks: the slot may already hold the final state
    load_v<NR>(sc.init + ((long long)b * s.inner + ch) * state_p + sub * NR, S);
    for (int i = 0; i < k; ++i) {
      const long long at = ((long long)b * chunks + i) * s.inner + ch;
      const float sum = sc.sums[at];
      float e[NR];
      load_v<NR>(sc.ends + at * state_p + sub * NR, e);
#pragma unroll
      for (int n = 0; n < NR; ++n) S[n] = fmaf(fast_exp2(sum * a[n]), S[n], e[n]);
    }
  } else {
#pragma unroll
    for (int n = 0; n < NR; ++n) S[n] = 0.f;
    if ((OUT || k == 0) && !fresh) load_v<NR>(slot, S);
    if (!OUT && k == 0) {
      if (live) store_v<NR>(sc.init + ((long long)b * s.inner + ch) * state_p + sub * NR, S);
#pragma unroll
      for (int n = 0; n < NR; ++n) S[n] = 0.f;
    }
  }
  const float bias = in.dt_bias[ch], D = OUT ? in.d[ch] : 0.f;
  const T* xp = static_cast<const T*>(in.x) + (long long)row0 * in.ld_x + ch;
  const T* zp = static_cast<const T*>(in.proj) + (long long)row0 * in.ld + in.z_off + ch;
  const float* dp = dt + (long long)row0 * ld_dt + ch;
  const T* low = static_cast<const T*>(in.low) + (long long)row0 * in.ld_low;
  const int tile = min(SS_TILE, SS_TILE_VALUES / state_p / SS_GROUP * SS_GROUP);
  float *sB = sm, *sC = sm + tile * state_p;
  float total = 0.f;
  float nx[SS_GROUP], nd[SS_GROUP], nz[SS_GROUP];  // inputs of the next group
  auto fetch = [&](int t) {
#pragma unroll
    for (int u = 0; u < SS_GROUP; ++u) {
      const bool on = t + u < t1;
      nx[u] = on ? ldf(xp + (long long)(t + u) * in.ld_x) : 0.f;
      nd[u] = on ? dp[(long long)(t + u) * ld_dt] : 0.f;
      if constexpr (OUT) nz[u] = on ? ldf(zp + (long long)(t + u) * in.ld) : 0.f;
    }
  };
  fetch(t0);
  for (int tt = t0; tt < t1; tt += tile) {
    const int n = min(tile, t1 - tt);
    __syncthreads();
    for (int i = threadIdx.x; i < n * state_p; i += SS_THREADS) {
      const int u = i / state_p, v = i % state_p;
      const T* row = low + (long long)(tt + u) * in.ld_low;
      sB[i] = v < s.state ? ldf(row + in.b_off + v) : 0.f;
      if constexpr (OUT) sC[i] = v < s.state ? ldf(row + in.c_off + v) : 0.f;
    }
    __syncthreads();
    for (int g = 0; g < n; g += SS_GROUP) {
      float x[SS_GROUP], d[SS_GROUP], z[SS_GROUP];
#pragma unroll
      for (int u = 0; u < SS_GROUP; ++u) {
        x[u] = nx[u];
        d[u] = softplus_fast(nd[u] + bias);
        if constexpr (OUT) z[u] = nz[u];
      }
      fetch(tt + g + SS_GROUP);
#pragma unroll
      for (int u = 0; u < SS_GROUP; ++u) {
        if (g + u >= n) break;                     // the same for the whole block
        const int at = (g + u) * state_p + sub * NR;
        float y = advance<NR, OUT>(S, a, d[u], x[u], sB + at, sC + at);
        if constexpr (OUT) {
          for (int o = 1; o < lanes; o <<= 1) y += __shfl_xor_sync(0xffffffffu, y, o);
          if (live && sub == 0)
            stf(out + (long long)(row0 + tt + g + u) * ldo + ch,
                fmaf(D, x[u], y) * __fdividef(z[u], 1.f + __expf(-z[u])) * s.out_scale);
        } else {
          total += d[u];
        }
      }
    }
  }
  if (!live) return;
  if constexpr (OUT) {
    if (last) store_v<NR>(slot, S);
  } else {
    const long long at = ((long long)b * chunks + k) * s.inner + ch;
    store_v<NR>(sc.ends + at * state_p + sub * NR, S);
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
  float a[NR], S[NR];
#pragma unroll
  for (int n = 0; n < NR; ++n) S[n] = 0.f;
  if (rb.kv_lens[b] > 1) load_v<NR>(slot, S);
  load_v<NR>(in.a + (long long)ch * state_p + sub * NR, a);
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
  const float d = softplus_fast(pre + in.dt_bias[ch]);
  float y = advance<NR, true>(S, a, d, x, sB + sub * NR, sC + sub * NR);
  for (int o = 1; o < lanes; o <<= 1) y += __shfl_xor_sync(0xffffffffu, y, o);
  if (!live) return;
  store_v<NR>(slot, S);
  if (sub == 0) stf(out + b * ldo + ch, fmaf(in.d[ch], x, y) * __fdividef(z, 1.f + __expf(-z)) * s.out_scale);
}

void check_spec(const SelectiveSpec& s) {
  MB_REQUIRE(s.inner > 0 && s.rank > 0 && s.taps > 0 && s.taps <= 64, "selective scan: sizes");
  MB_REQUIRE(s.state > 0 && s.state <= 512, "selective scan: at most 512 state values per channel");
}

// Chunks of the longest portion: enough blocks for the machine, unless a single pass already gives half of them.
struct ChunkPlan {
  int chunk, chunks;
};
ChunkPlan plan_chunks(const SelectiveSpec& s, int n_seq, int max_q) {
  const StateMap m = state_map(s.state);
  const long long blocks = ((long long)s.inner * m.lanes + SS_THREADS - 1) / SS_THREADS * n_seq;
  long long chunks = 6ll * sm_count() / (blocks > 0 ? blocks : 1);
  const long long most = (max_q + SS_CHUNK - 1) / SS_CHUNK;
  if (chunks > most) chunks = most;
  if (chunks > 64) chunks = 64;
  if (chunks < 2) return ChunkPlan{max_q > 0 ? max_q : 1, 1};
  const int chunk = (int)((max_q + chunks - 1) / chunks);
  return ChunkPlan{chunk, (max_q + chunk - 1) / chunk};
}

}  // namespace

int selective_padded_state(int state) {
  const StateMap m = state_map(state);
  return m.nr * m.lanes;
}

void selective_conv(bool f32, const SelectiveSpec& s, const SelectiveInputs& in, const RaggedBatch& rb, bool one_token,
                    void* x, long long ldx, cudaStream_t stream) {
  check_spec(s);
  MB_REQUIRE(ldx >= s.inner, "selective_conv: output width");
  if (rb.rows == 0) return;
  if (one_token) {
    MB_REQUIRE(rb.rows == rb.n_seq, "selective_conv: one token per sequence");
    const dim3 grid((int)((ldx + 255) / 256), rb.n_seq);
    if (f32) selective_conv_step_kernel<float><<<grid, 256, 0, stream>>>(s, in, rb, (float*)x, ldx);
    else selective_conv_step_kernel<__nv_bfloat16><<<grid, 256, 0, stream>>>(s, in, rb, (__nv_bfloat16*)x, ldx);
    count_launch();
    check_launch();
    return;
  }
  const int es = f32 ? 4 : 2, V = 16 / es;
  const bool vec = s.inner % V == 0 && ldx == s.inner && in.ld % V == 0 && in.x_off % V == 0 &&
                   ((reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(in.proj)) & 15) == 0;
  const int units = (int)(vec ? ldx / V : ldx), threads = units >= 256 ? 256 : (units + 31) / 32 * 32;
  const dim3 grid((units + threads - 1) / threads, (rb.rows + SC_ROWS - 1) / SC_ROWS);
  MB_REQUIRE(grid.y <= 65535, "selective_conv: too many rows in one batch");
#define MB_SC(T, V, TAPS) selective_conv_kernel<T, V, TAPS><<<grid, threads, 0, stream>>>(s, in, rb, (T*)x, ldx)
  if (f32) {
    if (vec && s.taps == 4) MB_SC(float, 4, 4); else if (vec) MB_SC(float, 4, 0); else MB_SC(float, 1, 0);
  } else {
    if (vec && s.taps == 4) MB_SC(__nv_bfloat16, 8, 4); else if (vec) MB_SC(__nv_bfloat16, 8, 0); else MB_SC(__nv_bfloat16, 1, 0);
  }
#undef MB_SC
  count_launch();
  check_launch();
  if (s.taps > 1) {
    const dim3 sgrid((s.inner + 255) / 256, rb.n_seq);
    if (f32) selective_conv_state_kernel<float><<<sgrid, 256, 0, stream>>>(s, in, rb);
    else selective_conv_state_kernel<__nv_bfloat16><<<sgrid, 256, 0, stream>>>(s, in, rb);
    count_launch();
    check_launch();
  }
}

long long selective_scratch(const SelectiveSpec& s, int n_seq, int max_q) {
  const ChunkPlan p = plan_chunks(s, n_seq, max_q);
  if (p.chunks <= 1) return 0;
  const long long state = (long long)s.inner * selective_padded_state(s.state);
  return n_seq * (state + p.chunks * (state + s.inner));
}

#define MB_SS_NR(GO)                                                        \
  if (m.nr == 4) GO(4); else if (m.nr == 8) GO(8); else if (m.nr == 12) GO(12); else GO(16)

void selective_scan(bool f32, const SelectiveSpec& s, const SelectiveInputs& in, const RaggedBatch& rb, int max_q,
                    const float* dt, long long ld_dt, float* scratch, void* out, long long ldo, cudaStream_t stream) {
  check_spec(s);
  if (rb.rows == 0) return;
  MB_REQUIRE(max_q > 0 && rb.n_seq <= 65535, "selective_scan: batch");
  const StateMap m = state_map(s.state);
  const ChunkPlan p = plan_chunks(s, rb.n_seq, max_q);
  const int state_p = m.nr * m.lanes;
  const long long state = (long long)s.inner * state_p;
  ChunkScratch sc{scratch, scratch + rb.n_seq * state, scratch + rb.n_seq * state * (1 + p.chunks)};
  const dim3 grid((int)(((long long)s.inner * m.lanes + SS_THREADS - 1) / SS_THREADS), p.chunks, rb.n_seq);
  const int per = SS_TILE_VALUES / state_p / SS_GROUP * SS_GROUP, tile = per < SS_TILE ? per : SS_TILE;
  const int smem = 2 * tile * state_p * 4;
#define MB_SS(T, NR, OUT)                                                                                           \
  selective_scan_kernel<T, NR, OUT><<<grid, SS_THREADS, smem, stream>>>(s, in, rb, m.lanes, p.chunk, p.chunks, dt, ld_dt, sc, \
                                                                        (T*)out, ldo)
#define MB_SS_BF(NR) do { if (p.chunks > 1) MB_SS(__nv_bfloat16, NR, false); MB_SS(__nv_bfloat16, NR, true); } while (0)
#define MB_SS_F(NR) do { if (p.chunks > 1) MB_SS(float, NR, false); MB_SS(float, NR, true); } while (0)
  if (f32) { MB_SS_NR(MB_SS_F); } else { MB_SS_NR(MB_SS_BF); }
#undef MB_SS_F
#undef MB_SS_BF
#undef MB_SS
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
