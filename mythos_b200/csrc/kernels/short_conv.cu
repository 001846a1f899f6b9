// Short causal convolution per channel over a ragged batch (hybrid_api.h): with a bias and silu, or added to its own input.
// The last taps - 1 inputs of a sequence are its state, 32-bit, one slot per sequence.
#include "common.cuh"
#include "host_util.h"
#include "hybrid_api.h"
#include "hybrid_dev.cuh"

namespace mb {
namespace {

// V channels of SC_ROWS neighbouring rows per thread; the rows' inputs pass through registers (TAPS > 0), so each is read
// once. TAPS: number of taps, 0: any number, read from the cache.
constexpr int SC_ROWS = 16, SC_STEP = 4;
template <typename T, int V, int TAPS, bool RES>
__global__ void __launch_bounds__(256)
short_conv_kernel(ShortConv s, const T* __restrict__ x, long long ldx, RaggedBatch rb, T* __restrict__ y, long long ldy) {
  __shared__ int s_index[SC_ROWS];                 // row within its sequence's portion
  __shared__ long long s_state[SC_ROWS];           // its sequence's convolution state, -1: it has no earlier tokens
  const long long c = ((long long)blockIdx.x * blockDim.x + threadIdx.x) * V;
  const int r0 = blockIdx.y * SC_ROWS, n = min(SC_ROWS, rb.rows - r0), taps = TAPS > 0 ? TAPS : s.taps;
  if (threadIdx.x < n) {
    const int b = rb.row_seq[r0 + threadIdx.x], lo = rb.cu_q[b];
    s_index[threadIdx.x] = r0 + threadIdx.x - lo;
    s_state[threadIdx.x] = rb.kv_lens[b] > rb.cu_q[b + 1] - lo ? (long long)rb.slots[b] * (taps - 1) * s.channels : -1;
  }
  __syncthreads();
  if (c >= ldy) return;
  if (c >= s.channels) {                           // padding (V = 1)
    for (int r = 0; r < n; ++r) stf(y + (r0 + r) * ldy + c, 0.f);
    return;
  }
  const T* col = x + (long long)r0 * ldx + c;
  T* dst = y + (long long)r0 * ldy + c;
  const float* w = s.w + c;
  float bias[V];
#pragma unroll
  for (int i = 0; i < V; ++i) bias[i] = 0.f;
  if (s.bias) load_v<V>(s.bias + c, bias);
  // inputs j tokens before row r that lie before its portion: from the state, zeros before the start
  auto early = [&](int r, int j, float (&v)[V]) {
    const long long st = s_state[r];
    if (st >= 0) {
      load_v<V>(s.state + st + (long long)(taps - 1 + s_index[r] - j) * s.channels + c, v);
    } else {
#pragma unroll
      for (int i = 0; i < V; ++i) v[i] = 0.f;
    }
  };
  if constexpr (TAPS > 0) {
    float wr[TAPS][V], h[TAPS - 1 + SC_STEP][V];   // h: inputs from row r - (TAPS - 1) on
#pragma unroll
    for (int j = 0; j < TAPS; ++j) load_v<V>(w + (long long)j * s.channels, wr[j]);
#pragma unroll
    for (int j = 0; j < TAPS - 1; ++j) {
      if (r0 - (TAPS - 1) + j >= 0) {
        load_v<V>(col + (long long)(j - (TAPS - 1)) * ldx, h[j]);
      } else {
#pragma unroll
        for (int i = 0; i < V; ++i) h[j][i] = 0.f;
      }
    }
#pragma unroll 1
    for (int r = 0; r < n; r += SC_STEP) {
#pragma unroll
      for (int u = 0; u < SC_STEP; ++u)
        if (r + u < n) load_v<V>(col + (long long)(r + u) * ldx, h[TAPS - 1 + u]);
#pragma unroll
      for (int u = 0; u < SC_STEP; ++u) {
        if (r + u >= n) break;
        const int i0 = s_index[r + u];
        float acc[V];
#pragma unroll
        for (int i = 0; i < V; ++i) acc[i] = fmaf(wr[TAPS - 1][i], h[TAPS - 1 + u][i], bias[i]);
#pragma unroll
        for (int j = 1; j < TAPS; ++j) {
          if (j <= i0) {                           // the same for the whole block
#pragma unroll
            for (int i = 0; i < V; ++i) acc[i] = fmaf(wr[TAPS - 1 - j][i], h[TAPS - 1 + u - j][i], acc[i]);
          } else {
            float v[V];
            early(r + u, j, v);
#pragma unroll
            for (int i = 0; i < V; ++i) acc[i] = fmaf(wr[TAPS - 1 - j][i], v[i], acc[i]);
          }
        }
#pragma unroll
        for (int i = 0; i < V; ++i) acc[i] = RES ? acc[i] + h[TAPS - 1 + u][i] : silu_t<T>(acc[i]);
        store_v<V>(dst + (long long)(r + u) * ldy, acc);
      }
#pragma unroll
      for (int j = 0; j < TAPS - 1; ++j)
#pragma unroll
        for (int i = 0; i < V; ++i) h[j][i] = h[j + SC_STEP][i];
    }
  } else {
    for (int r = 0; r < n; ++r) {
      float acc[V], own[V];
#pragma unroll
      for (int i = 0; i < V; ++i) acc[i] = bias[i];
      if constexpr (RES) load_v<V>(col + (long long)r * ldx, own);
      for (int j = 0; j < taps; ++j) {
        float v[V], wj[V];
        if (j <= s_index[r]) load_v<V>(col + (long long)(r - j) * ldx, v);
        else early(r, j, v);
        load_v<V>(w + (long long)(taps - 1 - j) * s.channels, wj);
#pragma unroll
        for (int i = 0; i < V; ++i) acc[i] = fmaf(wj[i], v[i], acc[i]);
      }
#pragma unroll
      for (int i = 0; i < V; ++i) acc[i] = RES ? acc[i] + own[i] : silu_t<T>(acc[i]);
      store_v<V>(dst + (long long)r * ldy, acc);
    }
  }
}

// One thread per (sequence, channel): the last taps - 1 inputs of the sequence become the state.
template <typename T>
__global__ void short_conv_state_kernel(ShortConv s, const T* __restrict__ x, long long ldx, RaggedBatch rb) {
  const int c = blockIdx.x * blockDim.x + threadIdx.x, b = blockIdx.y;
  if (c >= s.channels) return;
  const int r0 = rb.cu_q[b], len = rb.cu_q[b + 1] - r0, n = s.taps - 1;
  if (len <= 0) return;
  const bool fresh = rb.kv_lens[b] == len;
  float* st = s.state + (long long)rb.slots[b] * n * s.channels + c;
  const T* col = x + c;
  // entry j holds the input of token len - n + j; an entry moves down, never up, so in-place order is safe
  for (int j = 0; j < n; ++j) {
    const int i = len - n + j;
    float v;
    if (i >= 0) v = ldf(col + (long long)(r0 + i) * ldx);
    else v = fresh ? 0.f : st[(long long)(n + i) * s.channels];
    st[(long long)j * s.channels] = v;
  }
}

// One token per sequence: convolution and its state in one pass, one channel per thread.
template <typename T>
__global__ void __launch_bounds__(256)
short_conv_step_kernel(ShortConv s, const T* __restrict__ x, long long ldx, RaggedBatch rb, T* __restrict__ y, long long ldy) {
  const int c = blockIdx.x * blockDim.x + threadIdx.x, b = blockIdx.y;
  if (c >= ldy) return;
  if (c >= s.channels) {
    stf(y + b * ldy + c, 0.f);
    return;
  }
  const bool fresh = rb.kv_lens[b] <= 1;
  const float cur = ldf(x + b * ldx + c);
  float acc = conv_step(s, s.state ? s.state + (long long)rb.slots[b] * (s.taps - 1) * s.channels : nullptr, fresh, c, cur);
  if (s.bias) acc += s.bias[c];
  stf(y + b * ldy + c, s.residual ? acc + cur : silu_f(acc));
}

}  // namespace

void short_conv(bool f32, const ShortConv& s, const void* x, long long ldx, const RaggedBatch& rb, bool one_token, void* y,
                long long ldy, cudaStream_t stream) {
  MB_REQUIRE(s.channels > 0 && s.taps > 0 && s.taps <= 64 && ldx >= s.channels && ldy >= s.channels, "short_conv: sizes");
  MB_REQUIRE(s.taps == 1 || s.state, "short_conv: more than one tap needs a state");
  if (rb.rows == 0) return;
  if (one_token) {
    MB_REQUIRE(rb.rows == rb.n_seq, "short_conv: one token per sequence");
    const dim3 grid((int)((ldy + 255) / 256), rb.n_seq);
    if (f32) short_conv_step_kernel<float><<<grid, 256, 0, stream>>>(s, (const float*)x, ldx, rb, (float*)y, ldy);
    else short_conv_step_kernel<__nv_bfloat16><<<grid, 256, 0, stream>>>(s, (const __nv_bfloat16*)x, ldx, rb, (__nv_bfloat16*)y, ldy);
    count_launch();
    check_launch();
    return;
  }
  const int V = 4;
  const bool vec = s.channels % V == 0 && ldy == s.channels && ldx % V == 0 &&
                   ((reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(y)) & 15) == 0;
  const int units = (int)(vec ? ldy / V : ldy), threads = units >= 128 ? 128 : (units + 31) / 32 * 32;
  const dim3 grid((units + threads - 1) / threads, (rb.rows + SC_ROWS - 1) / SC_ROWS);
  MB_REQUIRE(grid.y <= 65535 && rb.n_seq <= 65535, "short_conv: too many rows in one batch");
#define MB_SC(T, V, TAPS)                                                                                            \
  do {                                                                                                               \
    if (s.residual) short_conv_kernel<T, V, TAPS, true><<<grid, threads, 0, stream>>>(s, (const T*)x, ldx, rb, (T*)y, ldy); \
    else short_conv_kernel<T, V, TAPS, false><<<grid, threads, 0, stream>>>(s, (const T*)x, ldx, rb, (T*)y, ldy);    \
  } while (0)
  if (f32) {
    if (vec && s.taps == 4) MB_SC(float, 4, 4); else if (vec) MB_SC(float, 4, 0); else MB_SC(float, 1, 0);
  } else {
    if (vec && s.taps == 4) MB_SC(__nv_bfloat16, 4, 4); else if (vec) MB_SC(__nv_bfloat16, 4, 0); else MB_SC(__nv_bfloat16, 1, 0);
  }
#undef MB_SC
  count_launch();
  check_launch();
  if (s.taps > 1) {
    const dim3 sgrid((s.channels + 255) / 256, rb.n_seq);
    if (f32) short_conv_state_kernel<float><<<sgrid, 256, 0, stream>>>(s, (const float*)x, ldx, rb);
    else short_conv_state_kernel<__nv_bfloat16><<<sgrid, 256, 0, stream>>>(s, (const __nv_bfloat16*)x, ldx, rb);
    count_launch();
    check_launch();
  }
}

}  // namespace mb
