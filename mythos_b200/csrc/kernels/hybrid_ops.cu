// Pointwise, normalisation and any-shape kernels of the layer-list models (hybrid_api.h).
//
// The residual stream is fp32. A sublayer's output is normalised before it is added ("sandwich"
// norms), and the next sublayer reads the sum (through a norm of its own, or as it is), so one kernel
// does post-norm, residual add and pre-norm of a row; for two mixers side by side it also normalises and
// averages the two, and for routed experts it forms the weighted sum of their outputs.
#include "api.h"
#include "common.cuh"
#include "hybrid_api.h"
#include "hybrid_dev.cuh"
#include "host_util.h"

namespace mb {
namespace {

constexpr int SN_THREADS = 256;

__device__ __forceinline__ float2 block_sum2(float2 v, float2* scratch) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = (blockDim.x + 31) >> 5;
  v.x = warp_sum(v.x);
  v.y = warp_sum(v.y);
  __syncthreads();
  if (lane == 0) scratch[warp] = v;
  __syncthreads();
  float2 t = (lane < nw) ? scratch[lane] : make_float2(0.f, 0.f);
  t.x = warp_sum(t.x);
  t.y = warp_sum(t.y);
  return t;
}

// Four values per step when the row allows it (V = 4), else one.
template <int V>
__device__ __forceinline__ void ldv(const float* p, float (&f)[V]) {
  if constexpr (V == 4) {
    const float4 t = *reinterpret_cast<const float4*>(p);
    f[0] = t.x; f[1] = t.y; f[2] = t.z; f[3] = t.w;
  } else {
    f[0] = *p;
  }
}
template <int V>
__device__ __forceinline__ void ldv(const __nv_bfloat16* p, float (&f)[V]) {
  if constexpr (V == 4) {
    const uint2 t = *reinterpret_cast<const uint2*>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&t.x));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&t.y));
    f[0] = a.x; f[1] = a.y; f[2] = b.x; f[3] = b.y;
  } else {
    f[0] = __bfloat162float(*p);
  }
}
// What type T keeps of a value.
template <typename T>
__device__ __forceinline__ float kept(float v) {
  if constexpr (sizeof(T) == 2) return __bfloat162float(__float2bfloat16(v));
  else return v;
}
template <int V>
__device__ __forceinline__ void stv(float* p, const float (&f)[V]) {
  if constexpr (V == 4) *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]);
  else *p = f[0];
}
template <int V>
__device__ __forceinline__ void stv(__nv_bfloat16* p, const float (&f)[V]) {
  if constexpr (V == 4) {
    __nv_bfloat162 a = __floats2bfloat162_rn(f[0], f[1]), b = __floats2bfloat162_rn(f[2], f[3]);
    uint2 t;
    t.x = *reinterpret_cast<uint32_t*>(&a);
    t.y = *reinterpret_cast<uint32_t*>(&b);
    *reinterpret_cast<uint2*>(p) = t;
  } else {
    *p = __float2bfloat16(f[0]);
  }
}

// The state and weights that row t's convolution will want, on their way to L2 while the row is reduced.
__device__ __forceinline__ void prefetch_tail(const ConvTail& cv, int dim, long long t) {
  if (cv.c.taps <= 1) return;
  const float* state = cv.c.state + (long long)cv.slots[t] * (cv.c.taps - 1) * dim;
  const int n = (cv.c.taps - 1) * dim;
  for (int i = threadIdx.x * 32; i < n; i += SN_THREADS * 32) {
    asm volatile("prefetch.global.L2 [%0];" ::"l"(state + i));
    asm volatile("prefetch.global.L2 [%0];" ::"l"(cv.c.w + i));
  }
}

// h = rms(row) * gamma (or the row itself) for a row held in shared memory; columns [dim, ldh) are zeroed (GEMM padding).
// With a convolution tail, row t being the new token of sequence t, also h + conv(h) of what the activation type keeps of h.
template <typename T, int V, bool CONV>
__device__ __forceinline__ void write_normed(const float* row, float ss, const float* gamma, T* h, long long ldh,
                                             int dim, float eps, const ConvTail& cv, long long t) {
  const float r = 1.f / sqrtf(ss / (float)dim + eps);
  const int taps = CONV ? cv.c.taps : 0;
  T* out = taps > 0 ? static_cast<T*>(cv.out) + t * cv.ld : nullptr;
  float* state = taps > 1 ? cv.c.state + (long long)cv.slots[t] * (taps - 1) * dim : nullptr;
  const bool fresh = taps > 0 && cv.kv_lens[t] <= 1;
  for (int i = threadIdx.x * V; i < dim; i += SN_THREADS * V) {
    float x[V], g[V];
    if (CONV && V == 4 && taps == 4) {                 // all loads first
      float w[4][V], old[3][V];
#pragma unroll
      for (int j = 0; j < 4; ++j) ldv<V>(cv.c.w + (long long)j * dim + i, w[j]);
#pragma unroll
      for (int j = 0; j < 3; ++j) ldv<V>(state + (long long)j * dim + i, old[j]);
      ldv<V>(row + i, x);
      ldv<V>(gamma + i, g);
#pragma unroll
      for (int j = 0; j < V; ++j) {
        x[j] = kept<T>(x[j] * r * g[j]);
#pragma unroll
        for (int k = 0; k < 3; ++k) old[k][j] = fresh ? 0.f : old[k][j];
        float y = fmaf(w[3][j], x[j], x[j]);
#pragma unroll
        for (int k = 0; k < 3; ++k) y = fmaf(w[k][j], old[k][j], y);
        g[j] = y;
      }
      stv<V>(h + i, x);
      stv<V>(out + i, g);
      stv<V>(state + i, old[1]);
      stv<V>(state + dim + i, old[2]);
      stv<V>(state + 2ll * dim + i, x);
      continue;
    }
    ldv<V>(row + i, x);
    if (gamma) {
      ldv<V>(gamma + i, g);
#pragma unroll
      for (int j = 0; j < V; ++j) x[j] *= r * g[j];
    }
    stv<V>(h + i, x);
    if (CONV) {
#pragma unroll
      for (int j = 0; j < V; ++j) {
        const float cur = kept<T>(x[j]);
        stf(out + i + j, cur + conv_step(cv.c, state, fresh, i + j, cur));
      }
    }
  }
  for (int i = dim + threadIdx.x; i < ldh; i += SN_THREADS) stf(h + i, 0.f);
  if (taps > 0)
    for (int i = dim + threadIdx.x; i < cv.ld; i += SN_THREADS) stf(out + i, 0.f);
}

template <typename T, int V, bool CONV>
__global__ void __launch_bounds__(SN_THREADS)
embed_pos_norm_kernel(const int* __restrict__ ids, const int* __restrict__ pos, const T* __restrict__ embed,
                      const T* __restrict__ pos_table, int vocab, int max_pos, float scale,
                      const float* __restrict__ gamma0, const float* __restrict__ gamma, float* __restrict__ x,
                      T* __restrict__ h, long long ldh, int dim, float eps, const __grid_constant__ ConvTail cv) {
  extern __shared__ __align__(16) float row[];
  __shared__ float scratch[32];
  const long long t = blockIdx.x;
  if constexpr (CONV) prefetch_tail(cv, dim, t);
  int id = ids[t];
  id = id < 0 ? 0 : (id >= vocab ? vocab - 1 : id);
  int p = pos[t];
  p = p < 0 ? 0 : (p >= max_pos ? max_pos - 1 : p);
  float ss = 0.f;
  for (int i = threadIdx.x * V; i < dim; i += SN_THREADS * V) {
    float e[V], q[V], y[V];
    ldv<V>(embed + (long long)id * dim + i, e);
#pragma unroll
    for (int j = 0; j < V; ++j) q[j] = 0.f;
    if (pos_table) ldv<V>(pos_table + (long long)p * dim + i, q);
#pragma unroll
    for (int j = 0; j < V; ++j) {
      y[j] = fmaf(e[j], scale, q[j]);
      ss += y[j] * y[j];
    }
    stv<V>(row + i, y);
    if (!gamma0) stv<V>(x + t * dim + i, y);
  }
  ss = block_sum(ss, scratch);
  if (gamma0) {                                        // the stream starts from the normalised row
    const float r = 1.f / sqrtf(ss / (float)dim + eps);
    ss = 0.f;
    for (int i = threadIdx.x * V; i < dim; i += SN_THREADS * V) {
      float y[V], g[V];
      ldv<V>(row + i, y);
      ldv<V>(gamma0 + i, g);
#pragma unroll
      for (int j = 0; j < V; ++j) {
        y[j] *= r * g[j];
        ss += y[j] * y[j];
      }
      stv<V>(row + i, y);
      stv<V>(x + t * dim + i, y);
    }
    ss = block_sum(ss, scratch);
  }
  write_normed<T, V, CONV>(row, ss, gamma, h + t * ldh, ldh, dim, eps, cv, t);
}

template <typename T, int V, bool CONV>
__global__ void __launch_bounds__(SN_THREADS)
residual_norm_kernel(const T* __restrict__ y, long long ldy, const float* __restrict__ bias, float mult, float* __restrict__ x,
                     const float* __restrict__ w_next, T* __restrict__ h, long long ldh, int dim, float eps,
                     const __grid_constant__ ConvTail cv) {
  extern __shared__ __align__(16) float row[];
  __shared__ float scratch[32];
  const long long t = blockIdx.x;
  if constexpr (CONV) prefetch_tail(cv, dim, t);
  float sx = 0.f;
  for (int i = threadIdx.x * V; i < dim; i += SN_THREADS * V) {
    float a[V], b[V], xv[V];
    ldv<V>(y + t * ldy + i, a);
    ldv<V>(x + t * dim + i, xv);
    if (bias) {
      ldv<V>(bias + i, b);
#pragma unroll
      for (int j = 0; j < V; ++j) a[j] += b[j];
    }
#pragma unroll
    for (int j = 0; j < V; ++j) {
      xv[j] = fmaf(mult, a[j], xv[j]);
      sx += xv[j] * xv[j];
    }
    stv<V>(x + t * dim + i, xv);
    stv<V>(row + i, xv);
  }
  sx = block_sum(sx, scratch);
  write_normed<T, V, CONV>(row, sx, w_next, h + t * ldh, ldh, dim, eps, cv, t);
}

template <int V>
__device__ __forceinline__ void load_bias(const float* bias, int i, float (&b)[V]) {
  if constexpr (V == 8) {
    float lo[4], hi[4];
    load_v<4>(bias + i, lo);
    load_v<4>(bias + i + 4, hi);
#pragma unroll
    for (int j = 0; j < 4; ++j) { b[j] = lo[j]; b[4 + j] = hi[j]; }
  } else {
    load_v<V>(bias + i, b);
  }
}
template <int V>
__device__ __forceinline__ void add_powers(const float (&z)[V], float3& s) {
#pragma unroll
  for (int j = 0; j < V; ++j) {
    const float q = z[j] * z[j], q2 = q * q;
    s.x += q;
    s.y += q2;
    s.z = fmaf(q2, q, s.z);
  }
}
// Factors of z, z^2 and z^3 from a block's sums of squares.
__device__ __forceinline__ float3 power_factors(float3 s, float (*part)[16], const float4& abce, float width, float eps) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
  s = make_float3(warp_sum(s.x), warp_sum(s.y), warp_sum(s.z));
  if (lane == 0) {
    part[0][warp] = s.x;
    part[1][warp] = s.y;
    part[2][warp] = s.z;
  }
  __syncthreads();
  s.x = warp_sum(lane < nw ? part[0][lane] : 0.f);
  s.y = warp_sum(lane < nw ? part[1][lane] : 0.f);
  s.z = warp_sum(lane < nw ? part[2][lane] : 0.f);
  return make_float3(abce.x / sqrtf(s.x / width + eps), abce.y / sqrtf(s.y / width + eps), abce.z / sqrtf(s.z / width + eps));
}
template <typename T, int V>
__device__ __forceinline__ void store_poly(T* out, float (&z)[V], const float3& f, float e) {
#pragma unroll
  for (int j = 0; j < V; ++j) z[j] = fmaf(fmaf(fmaf(f.z, z[j], f.y), z[j], f.x), z[j], e);
  if constexpr (V == 8) *reinterpret_cast<bf16x8*>(out) = pack8(z);
  else stv<V>(out, z);
}

// One block per row; a thread holds NV vectors of V values (16 bytes).
template <typename T, int V, int NV>
__global__ void __launch_bounds__(512)
poly_norm_kernel(const T* __restrict__ y, long long ldy, const float* __restrict__ bias, const float* __restrict__ abce_p,
                 T* __restrict__ out, long long ldo, int width, int padded, float eps) {
  __shared__ float part[3][16];
  const int step = blockDim.x * V, c = threadIdx.x * V;
  y += blockIdx.x * ldy;
  out += blockIdx.x * ldo;
  uint4 raw[NV];
#pragma unroll
  for (int k = 0; k < NV; ++k)
    if (c + k * step < width) raw[k] = *reinterpret_cast<const uint4*>(y + c + k * step);
  const float4 abce = make_float4(abce_p[0], abce_p[1], abce_p[2], abce_p[3]);
  float z[NV][V];
  float3 s = make_float3(0.f, 0.f, 0.f);
#pragma unroll
  for (int k = 0; k < NV; ++k) {
    const int i = c + k * step;
    if (i >= width) continue;
    load_v<V>(reinterpret_cast<const T*>(&raw[k]), z[k]);
    if (bias) {
      float b[V];
      load_bias<V>(bias, i, b);
#pragma unroll
      for (int j = 0; j < V; ++j) z[k][j] += b[j];
    }
    add_powers<V>(z[k], s);
  }
  const float3 f = power_factors(s, part, abce, (float)width, eps);
#pragma unroll
  for (int k = 0; k < NV; ++k) {
    const int i = c + k * step;
    if (i < width) store_poly<T, V>(out + i, z[k], f, abce.w);
  }
  for (int i = width + threadIdx.x; i < padded; i += blockDim.x) stf(out + i, 0.f);
}

// Any width and alignment, one block per row, the row is read twice.
template <typename T>
__global__ void __launch_bounds__(256)
poly_norm_any_kernel(const T* __restrict__ y, long long ldy, const float* __restrict__ bias, const float* __restrict__ abce_p,
                     T* __restrict__ out, long long ldo, int width, int padded, float eps) {
  __shared__ float part[3][16];
  const float4 abce = make_float4(abce_p[0], abce_p[1], abce_p[2], abce_p[3]);
  y += blockIdx.x * ldy;
  out += blockIdx.x * ldo;
  float3 s = make_float3(0.f, 0.f, 0.f);
  for (int i = threadIdx.x; i < width; i += blockDim.x) {
    const float z[1] = {ldf(y + i) + (bias ? bias[i] : 0.f)};
    add_powers<1>(z, s);
  }
  const float3 f = power_factors(s, part, abce, (float)width, eps);
  for (int i = threadIdx.x; i < padded; i += blockDim.x) {
    float z[1] = {0.f};
    if (i < width) {
      z[0] = ldf(y + i) + (bias ? bias[i] : 0.f);
      store_poly<T, 1>(out + i, z, f, abce.w);
    } else {
      stf(out + i, 0.f);
    }
  }
}

enum { SUB_ONE, SUB_TWO, SUB_EXPERTS };
constexpr int SN_MAX_TOP = 32;

template <typename T, int V, int SRC>
__global__ void __launch_bounds__(SN_THREADS)
sandwich_norm_kernel(SublayerOut src, const float* __restrict__ w_post, float mult, float* __restrict__ x,
                     const float* __restrict__ w_next, T* __restrict__ h, long long ldh, int dim, float eps) {
  extern __shared__ __align__(16) float row[];
  __shared__ float2 scratch2[32];
  __shared__ float scratch[32];
  __shared__ long long s_row[SN_MAX_TOP];
  __shared__ float s_weight[SN_MAX_TOP];
  const long long t = blockIdx.x;
  const T* y1 = static_cast<const T*>(src.y1);
  const T* y2 = static_cast<const T*>(src.y2);
  if constexpr (SRC == SUB_EXPERTS) {
    if (threadIdx.x < src.top) {
      s_row[threadIdx.x] = (long long)src.row[t * src.top + threadIdx.x] * src.ld;
      s_weight[threadIdx.x] = src.weight[t * src.top + threadIdx.x];
    }
    __syncthreads();
  } else {
    y1 += t * src.ld;
    y2 += t * src.ld;
  }
  float2 s2 = make_float2(0.f, 0.f);
  for (int i = threadIdx.x * V; i < dim; i += SN_THREADS * V) {
    float a[V];
    if constexpr (SRC == SUB_EXPERTS) {
#pragma unroll
      for (int j = 0; j < V; ++j) a[j] = 0.f;
      for (int e = 0; e < src.top; ++e) {
        float b[V];
        ldv<V>(y1 + s_row[e] + i, b);
#pragma unroll
        for (int j = 0; j < V; ++j) a[j] = fmaf(s_weight[e], b[j], a[j]);
      }
      if (y2) {
        float b[V];
        ldv<V>(y2 + t * src.ld + i, b);
#pragma unroll
        for (int j = 0; j < V; ++j) a[j] += b[j];
      }
    } else {
      ldv<V>(y1 + i, a);
    }
#pragma unroll
    for (int j = 0; j < V; ++j) s2.x += a[j] * a[j];
    if constexpr (SRC == SUB_TWO) {
      float b[V];
      ldv<V>(y2 + i, b);
#pragma unroll
      for (int j = 0; j < V; ++j) s2.y += b[j] * b[j];
    } else {
      stv<V>(row + i, a);
    }
  }
  s2 = block_sum2(s2, scratch2);
  float ss = s2.x;
  if constexpr (SRC == SUB_TWO) {
    const float ra = 0.5f / sqrtf(s2.x / (float)dim + eps), rb = 0.5f / sqrtf(s2.y / (float)dim + eps);
    ss = 0.f;
    for (int i = threadIdx.x * V; i < dim; i += SN_THREADS * V) {
      float a[V], b[V], wa[V], wb[V];
      ldv<V>(y1 + i, a);
      ldv<V>(y2 + i, b);
      ldv<V>(src.w1 + i, wa);
      ldv<V>(src.w2 + i, wb);
#pragma unroll
      for (int j = 0; j < V; ++j) {
        a[j] = a[j] * ra * wa[j] + b[j] * rb * wb[j];
        ss += a[j] * a[j];
      }
      stv<V>(row + i, a);
    }
    ss = block_sum(ss, scratch);
  }
  const float r = mult / sqrtf(ss / (float)dim + eps);
  float sx = 0.f;
  for (int i = threadIdx.x * V; i < dim; i += SN_THREADS * V) {
    float a[V], w[V], xv[V];
    ldv<V>(row + i, a);
    ldv<V>(w_post + i, w);
    ldv<V>(x + t * dim + i, xv);
#pragma unroll
    for (int j = 0; j < V; ++j) {
      xv[j] += a[j] * r * w[j];
      sx += xv[j] * xv[j];
    }
    stv<V>(x + t * dim + i, xv);
    stv<V>(row + i, xv);
  }
  if (w_next) sx = block_sum(sx, scratch);
  write_normed<T, V, false>(row, sx, w_next, h + t * ldh, ldh, dim, eps, ConvTail{}, t);
}

// Cosine and sine of a position's turn: position x revolutions, reduced to a fraction of a turn in double precision.
__device__ __forceinline__ float2 turn(int pos, double revolutions, float amp) {
  const double a = pos * revolutions;
  float sn, co;
  sincospif(2.f * (float)(a - rint(a)), &sn, &co);
  return make_float2(amp * co, amp * sn);
}
__device__ __forceinline__ float query_factor(const HeadPrep& p, int pos) {
  return p.temp_coef == 0.f ? 1.f : 1.f + p.temp_coef * logf(floorf((float)(pos + 1) / p.temp_every) + 1.f);
}

// One warp per (token, head slot): slots [0, H) are q, [H, H + G) k, [H + G, H + 2 G) v.
template <typename T>
__global__ void attn_prep_kernel(const T* __restrict__ proj, long long ld, HeadPrep p, RaggedBatch rb,
                                 const int* __restrict__ block_table, int table_stride, int page_size, T* __restrict__ q_out,
                                 T* __restrict__ k_cache, T* __restrict__ v_cache) {
  const int lane = threadIdx.x & 31;
  const int slots = p.heads + (p.k_off < 0 ? 0 : 2 * p.kv_heads);
  const long long w = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (w >= (long long)rb.rows * slots) return;
  const int t = (int)(w / slots), hs = (int)(w % slots), pos = rb.pos[t];
  const bool is_q = hs < p.heads, is_v = hs >= p.heads + p.kv_heads;
  const int j = is_q ? hs : (is_v ? hs - p.heads - p.kv_heads : hs - p.heads), width = is_v ? p.dv : p.dk;
  const T* src = proj + (long long)t * ld + (is_q ? p.q_off : (is_v ? p.v_off : p.k_off)) + j * width;
  const float* bias = is_q ? p.q_bias : (is_v ? p.v_bias : p.k_bias);
  if (bias) bias += j * width;
  T* dst;
  if (is_q) {
    dst = q_out + ((long long)t * p.heads + j) * width;
  } else {
    const int page = block_table[(long long)rb.row_seq[t] * table_stride + pos / page_size];
    if (page < 0) return;
    dst = (is_v ? v_cache : k_cache) + (((long long)page * page_size + pos % page_size) * p.kv_heads + j) * width;
  }
  auto raw = [&](int i) { return ldf(src + i) + (bias ? bias[i] : 0.f); };
  if (is_v) {
    for (int i = lane; i < width; i += 32) stf(dst + i, raw(i));
    return;
  }
  float r = 1.f;
  if (p.norm_dim > 0) {
    float ss = 0.f;
    for (int i = lane; i < width; i += 32) {
      const float v = raw(i);
      ss += v * v;
    }
    r = 1.f / sqrtf(warp_sum(ss) / (float)p.norm_dim + p.eps);
  }
  const float* gamma = is_q ? p.q_gamma : p.k_gamma;
  auto normed = [&](int i) { return raw(i) * r * (gamma ? gamma[i] : 1.f); };
  const float f = is_q ? query_factor(p, pos) : 1.f;
  const int half = p.rot / 2;
  for (int i = lane; i < width; i += 32) {
    float x = normed(i);
    if (i < p.rot) {
      const float2 cs = turn(pos, p.turns[p.pairs ? i >> 1 : (i < half ? i : i - half)], p.rot_amp);
      const bool first = p.pairs ? (i & 1) == 0 : i < half;
      const int by = p.pairs ? 1 : half;
      x = first ? x * cs.x - normed(i + by) * cs.y : x * cs.x + normed(i - by) * cs.y;
    }
    stf(dst + i, x * f);
  }
}

__device__ __forceinline__ void load8(const float* p, float (&f)[8]) {
  const float4 a = reinterpret_cast<const float4*>(p)[0], b = reinterpret_cast<const float4*>(p)[1];
  f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w;
  f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
}

// bf16 form for widths that are multiples of 8 up to 128: 16 lanes per (token, head slot), 16-byte accesses, `tokens`
// tokens per block. What depends on the token alone (page row, query factor, angles) is evaluated once for all heads.
constexpr int AP_THREADS = 256, AP_TOKENS = 16;
__global__ void __launch_bounds__(AP_THREADS)
attn_prep8_kernel(const __nv_bfloat16* __restrict__ proj, long long ld, const __grid_constant__ HeadPrep p,
                  const __grid_constant__ RaggedBatch rb, const int* __restrict__ block_table, int table_stride, int page_size,
                  int tokens, __nv_bfloat16* __restrict__ q_out, __nv_bfloat16* __restrict__ k_cache,
                  __nv_bfloat16* __restrict__ v_cache) {
  extern __shared__ __align__(16) float2 cs_all[];         // [tokens][rot / 2], pair 8 a + b at place b * (rot / 16) + a
  __shared__ int s_page_row[AP_TOKENS];                    // row of the pages, or -1
  __shared__ float s_factor[AP_TOKENS];
  const int l = threadIdx.x & 15, c = l * 8, slots = p.heads + (p.k_off < 0 ? 0 : 2 * p.kv_heads), half = p.rot / 2;
  const int t0 = blockIdx.x * tokens, nt = min(tokens, rb.rows - t0), total = nt * slots;
  const float per = 1.f / (float)slots;
  struct Item {                                            // one head of one token
    int tl, j, width;
    bool live, is_q, is_v;
    const __nv_bfloat16* src;
  };
  auto item = [&](int w) {
    Item it;
    it.live = w < total;
    if (!it.live) w = 0;
    it.tl = (int)(((float)w + 0.5f) * per);                // exact: w is far below 2^23
    const int hs = w - it.tl * slots;
    it.is_q = hs < p.heads;
    it.is_v = hs >= p.heads + p.kv_heads;
    it.j = it.is_q ? hs : (it.is_v ? hs - p.heads - p.kv_heads : hs - p.heads);
    it.width = it.is_v ? p.dv : p.dk;
    it.src = proj + (long long)(t0 + it.tl) * ld + (it.is_q ? p.q_off : (it.is_v ? p.v_off : p.k_off)) + it.j * it.width;
    it.live = it.live && c < it.width;
    return it;
  };
  // both halves of a warp run the same number of iterations: the shuffles need the whole warp
  const int first = (threadIdx.x >> 4) & ~1, side = (threadIdx.x >> 4) & 1;
  Item next = item(first + side);
  bf16x8 raw_next{};
  if (next.live) raw_next = ldg8(next.src, c);
  for (int i = threadIdx.x; i < nt; i += AP_THREADS) {
    const int pos = rb.pos[t0 + i];
    const int page = block_table[(long long)rb.row_seq[t0 + i] * table_stride + pos / page_size];
    s_page_row[i] = page < 0 ? -1 : page * page_size + pos % page_size;
    s_factor[i] = query_factor(p, pos);
  }
  const bool spread = !p.pairs && half % 8 == 0;           // neighbouring lanes then read neighbouring entries
  for (int i = threadIdx.x; i < nt * half; i += AP_THREADS) {
    const int tl = i / half, k = i - tl * half;
    cs_all[tl * half + (spread ? (k & 7) * (half >> 3) + (k >> 3) : k)] = turn(rb.pos[t0 + tl], p.turns[k], p.rot_amp);
  }
  __syncthreads();
  for (int w0 = first; w0 < total; w0 += AP_THREADS >> 4) {
    const Item it = next;
    const bf16x8 raw = raw_next;
    next = item(w0 + (AP_THREADS >> 4) + side);            // the next item's values are on their way meanwhile
    if (next.live) raw_next = ldg8(next.src, c);
    const float* bias = it.is_q ? p.q_bias : (it.is_v ? p.v_bias : p.k_bias);
    const float* gamma = it.is_q ? p.q_gamma : p.k_gamma;
    float f[8], ss = 0.f;
    unpack8(raw, f);
    if (bias) bias += it.j * it.width;
    if (bias && it.live) {
      float g[8];
      load8(bias + c, g);
#pragma unroll
      for (int i = 0; i < 8; ++i) f[i] += g[i];
    }
    float r = 1.f;
    if (p.norm_dim > 0) {
      if (it.live) {
#pragma unroll
        for (int i = 0; i < 8; ++i) ss = fmaf(f[i], f[i], ss);
      }
#pragma unroll
      for (int o = 8; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
      r = rsqrtf(__fdividef(ss, (float)p.norm_dim) + p.eps);
    }
    if (!it.live) continue;
    if (!it.is_v) {
      const float q = it.is_q ? r * s_factor[it.tl] : r;   // the factor commutes with the rotation
      if (gamma) {
        float g[8];
        load8(gamma + c, g);
#pragma unroll
        for (int i = 0; i < 8; ++i) f[i] *= q * g[i];
      } else {
#pragma unroll
        for (int i = 0; i < 8; ++i) f[i] *= q;
      }
      if (p.pairs) {
        const float2* cs = cs_all + it.tl * half + c / 2;
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          if (c + 2 * i < p.rot) {
            const float2 t = cs[i];
            const float u = f[2 * i], v = f[2 * i + 1];
            f[2 * i] = u * t.x - v * t.y;
            f[2 * i + 1] = v * t.x + u * t.y;
          }
        }
      } else if (c < p.rot) {
        // column i < half turns with i + half; the partner's value is read again
        const float2* cs = cs_all + it.tl * half;
        if (spread) {
          const int at = c < half ? c + half : c - half, k = (c < half ? c : at) >> 3, lanes = half >> 3;
          float g[8];
          unpack8(ldg8(it.src, at), g);
          const float sign = c < half ? -q : q;
#pragma unroll
          for (int i = 0; i < 8; ++i) {
            const float v = (g[i] + (bias ? bias[at + i] : 0.f)) * (gamma ? sign * gamma[at + i] : sign);
            const float2 t = cs[i * lanes + k];
            f[i] = f[i] * t.x + v * t.y;
          }
        } else {
#pragma unroll
          for (int i = 0; i < 8; ++i) {
            const int col = c + i;
            if (col < p.rot) {
              const int at = col < half ? col + half : col - half, k = col < half ? col : at;
              const float v = (__bfloat162float(it.src[at]) + (bias ? bias[at] : 0.f)) * (gamma ? q * gamma[at] : q);
              f[i] = f[i] * cs[k].x + (col < half ? -v : v) * cs[k].y;
            }
          }
        }
      }
    }
    const bf16x8 out = pack8(f);
    const int row = s_page_row[it.tl];
    if (it.is_q) stg8(q_out, ((long long)(t0 + it.tl) * p.heads + it.j) * it.width + c, out);
    else if (row >= 0) stg8(it.is_v ? v_cache : k_cache, ((long long)row * p.kv_heads + it.j) * it.width + c, out);
  }
}

// One warp per (token, query head). Scores of 32 keys at a time (lane = key), then the value rows with
// lane = channel: every product and the softmax are fp32 whatever the storage type.
constexpr int PA_WARPS = 4;
template <typename T, int ND>   // ND * 32 >= dv
__global__ void __launch_bounds__(PA_WARPS * 32)
paged_attn_any_kernel(const T* __restrict__ q, const T* __restrict__ k_cache, const T* __restrict__ v_cache,
                      RaggedBatch rb, const int* __restrict__ block_table, int table_stride, int page_size,
                      AttnExtras ex, T* __restrict__ o, long long ldo, int heads, int kv_heads, int dk, int dv, float scale) {
  extern __shared__ float sq_all[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const long long w = (long long)blockIdx.x * PA_WARPS + warp;
  if (w >= (long long)rb.rows * heads) return;
  // the last tokens have the longest contexts: start them first
  const int t = rb.rows - 1 - (int)(w / heads), h = (int)(w % heads);
  const int g = h / (heads / kv_heads);
  float* sq = sq_all + warp * dk;
  for (int i = lane; i < dk; i += 32) sq[i] = ldf(q + ((long long)t * heads + h) * dk + i) * scale;
  __syncwarp();
  const int* bt = block_table + (long long)rb.row_seq[t] * table_stride;
  const int n = rb.pos[t] + 1, first = ex.window > 0 ? max(0, n - ex.window) : 0;
  float m = -INFINITY, l = 0.f, acc[ND];
#pragma unroll
  for (int j = 0; j < ND; ++j) acc[j] = 0.f;
  for (int j0 = first; j0 < n; j0 += 32) {
    const int key = j0 + lane;
    float s = -INFINITY;
    long long tok = 0;
    if (key < n) {
      tok = (long long)bt[key / page_size] * page_size + key % page_size;
      const T* kp = k_cache + (tok * kv_heads + g) * dk;
      s = 0.f;
      for (int i = 0; i < dk; ++i) s = fmaf(sq[i], ldf(kp + i), s);
    }
    const float mn = fmaxf(m, warp_max(s));
    const float a = expf(m - mn), p = expf(s - mn);
    l = l * a + warp_sum(p);
    m = mn;
#pragma unroll
    for (int j = 0; j < ND; ++j) acc[j] *= a;
    const int cnt = min(32, n - j0);
    for (int jj = 0; jj < cnt; ++jj) {
      const float pj = __shfl_sync(0xffffffffu, p, jj);
      const long long tk = __shfl_sync(0xffffffffu, tok, jj);
      const T* vp = v_cache + (tk * kv_heads + g) * dv;
#pragma unroll
      for (int j = 0; j < ND; ++j) {
        const int d = lane + 32 * j;
        if (d < dv) acc[j] = fmaf(pj, ldf(vp + d), acc[j]);
      }
    }
  }
  if (ex.sink) l += expf(ex.sink[h] - m);
  float r = ex.out_scale / l;
  const T* gate = ex.gate ? static_cast<const T*>(ex.gate) + (long long)t * ex.ld_gate : nullptr;
  if (gate && !ex.gate_channels) r *= sigmoid_f(ldf(gate + h));
#pragma unroll
  for (int j = 0; j < ND; ++j) {
    const int d = lane + 32 * j;
    if (d >= dv) continue;
    float y = acc[j] * r;
    if (gate && ex.gate_channels) y *= sigmoid_f(ldf(gate + h * dv + d));
    stf(o + (long long)t * ldo + (long long)h * dv + d, y);
  }
}

// 64 x 64 tile, 16-deep steps, 4 x 4 outputs per thread. blockIdx.z: product of a batch, or entry of a tile list.
__global__ void __launch_bounds__(256)
gemm_f32_kernel(const float* __restrict__ A, long long lda, const float* __restrict__ B, long long ldb,
                float* __restrict__ C, long long ldc, int M, int N, int K, float alpha, long long a_batch,
                long long b_batch, long long c_batch, TileList list) {
  __shared__ float sa[16][68], sb[16][68];
  int m0 = blockIdx.y * 64;
  const int n0 = blockIdx.x * 64;
  if (list.tiles) {
    if ((int)blockIdx.z >= *list.count) return;
    const int* tile = list.tiles + 3 * blockIdx.z;
    m0 = 0;
    M = tile[2];
    A += tile[1] * lda;
    C += tile[1] * ldc;
    B += tile[0] * b_batch;
  } else {
    A += blockIdx.z * a_batch;
    B += blockIdx.z * b_batch;
    C += blockIdx.z * c_batch;
  }
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < K; k0 += 16) {
    for (int i = threadIdx.x; i < 64 * 16; i += 256) {
      const int r = i >> 4, c = i & 15;
      sa[c][r] = (m0 + r < M && k0 + c < K) ? A[(long long)(m0 + r) * lda + k0 + c] : 0.f;
      sb[c][r] = (n0 + r < N && k0 + c < K) ? B[(long long)(n0 + r) * ldb + k0 + c] : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < 16; ++k) {
      float a[4], b[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        a[i] = sa[k][ty * 4 + i];
        b[i] = sb[k][tx * 4 + i];
      }
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int m = m0 + ty * 4 + i, n = n0 + tx * 4 + j;
      if (m < M && n < N) C[(long long)m * ldc + n] = alpha * acc[i][j];
    }
}

template <typename T>
__global__ void gate_pair_kernel(const T* __restrict__ gu, long long ldg, int f, int f_off, GateAct act, T* __restrict__ h,
                                 long long ldh, long long rows) {
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < rows * ldh;
       i += (long long)gridDim.x * blockDim.x) {
    const long long r = i / ldh;
    const int c = (int)(i % ldh);
    stf(h + i, c < f ? gate_act(act, ldf(gu + r * ldg + c), ldf(gu + r * ldg + f_off + c)) : 0.f);
  }
}

template <typename T>
__global__ void gelu_mul_kernel(T* __restrict__ y, long long ldy, const T* __restrict__ table, long long ld_table,
                                const int* __restrict__ ids, int vocab, long long rows, int width) {
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < rows * width;
       i += (long long)gridDim.x * blockDim.x) {
    const long long r = i / width;
    const int c = (int)(i % width), id = min(max(ids[r], 0), vocab - 1);
    stf(y + r * ldy + c, gelu_tanh_f(ldf(y + r * ldy + c)) * ldf(table + id * ld_table + c));
  }
}

template <typename T>
__global__ void sigmoid_mul_kernel(T* __restrict__ y, long long ldy, const T* __restrict__ gate, long long ld_gate, long long rows,
                                   int width) {
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < rows * width;
       i += (long long)gridDim.x * blockDim.x) {
    T* p = y + i / width * ldy + i % width;
    stf(p, ldf(p) * sigmoid_f(ldf(gate + i / width * ld_gate + i % width)));
  }
}

__global__ void soft_cap_kernel(float* __restrict__ y, long long ldy, long long rows, int width, float cap) {
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < rows * width;
       i += (long long)gridDim.x * blockDim.x) {
    float* p = y + i / width * ldy + i % width;
    *p = soft_cap_f(*p, cap);
  }
}

inline int grid_for(long long n, int threads, int per_sm) {
  long long g = (n + threads - 1) / threads;
  const long long cap = (long long)sm_count() * per_sm;
  return (int)(g < cap ? g : cap);
}

template <typename T, int V>
void embed_launch(const int* ids, const int* pos, const void* embed, const void* pos_table, int vocab, int max_pos,
                  float scale, const float* gamma0, const float* gamma, float* x, void* h, long long ldh, int rows, int dim,
                  float eps, const ConvTail& conv, cudaStream_t stream) {
  auto go = [&](auto kern) {
    kern<<<rows, SN_THREADS, dim * 4, stream>>>(ids, pos, (const T*)embed, (const T*)pos_table, vocab, max_pos, scale, gamma0, gamma, x,
                                                (T*)h, ldh, dim, eps, conv);
  };
  if (conv.c.taps > 0) go(embed_pos_norm_kernel<T, V, true>);
  else go(embed_pos_norm_kernel<T, V, false>);
}
void check_tail(const ConvTail& conv, int dim) {
  MB_REQUIRE(conv.c.taps >= 0 && conv.c.taps <= 64, "convolution tail: taps");
  if (conv.c.taps == 0) return;
  MB_REQUIRE(conv.c.channels == dim && conv.ld >= dim && conv.out && conv.c.w && conv.slots && conv.kv_lens &&
                 (conv.c.taps == 1 || conv.c.state) && !conv.c.bias, "convolution tail: arguments");
  MB_REQUIRE(((reinterpret_cast<uintptr_t>(conv.c.w) | reinterpret_cast<uintptr_t>(conv.c.state) | reinterpret_cast<uintptr_t>(conv.out)) & 15) == 0 &&
                 (dim % 4 != 0 || conv.ld % 4 == 0), "convolution tail: alignment");
}
template <typename T, int V>
void sandwich_launch(const SublayerOut& y, const float* w_post, float mult, float* x, const float* w_next, void* h,
                     long long ldh, int rows, int dim, float eps, cudaStream_t stream) {
#define MB_SN(SRC) \
  sandwich_norm_kernel<T, V, SRC><<<rows, SN_THREADS, dim * 4, stream>>>(y, w_post, mult, x, w_next, (T*)h, ldh, dim, eps)
  if (y.row) MB_SN(SUB_EXPERTS);
  else if (y.y2) MB_SN(SUB_TWO);
  else MB_SN(SUB_ONE);
#undef MB_SN
}

}  // namespace

void embed_pos_norm(bool f32, const int* ids, const int* pos, const void* embed, const void* pos_table, int vocab,
                    int max_pos, float scale, const float* gamma0, const float* gamma, float* x, void* h, long long ldh,
                    int rows, int dim, float eps, const ConvTail& conv, cudaStream_t stream) {
  check_tail(conv, dim);
  MB_REQUIRE(dim > 0 && dim <= 12000 && ldh >= dim, "embed_pos_norm: row width out of range");
  if (rows == 0) return;
  const bool v4 = dim % 4 == 0 && ldh % 4 == 0;
  auto go = [&](auto fn) {
    fn(ids, pos, embed, pos_table, vocab, max_pos, scale, gamma0, gamma, x, h, ldh, rows, dim, eps, conv, stream);
  };
  if (f32) { if (v4) go(embed_launch<float, 4>); else go(embed_launch<float, 1>); }
  else     { if (v4) go(embed_launch<__nv_bfloat16, 4>); else go(embed_launch<__nv_bfloat16, 1>); }
  count_launch();
  check_launch();
}

void sandwich_norm(bool f32, const SublayerOut& y, const float* w_post, float mult, float* x, const float* w_next, void* h,
                   long long ldh, int rows, int dim, float eps, cudaStream_t stream) {
  MB_REQUIRE(dim > 0 && dim <= 12000 && ldh >= dim && y.ld >= dim, "sandwich_norm: row width out of range");
  MB_REQUIRE(y.y2 == nullptr || y.row || (y.w1 && y.w2), "sandwich_norm: two inputs need their norm weights");
  MB_REQUIRE(y.row == nullptr || (y.weight && y.top > 0 && y.top <= SN_MAX_TOP), "sandwich_norm: at most 32 experts a token");
  if (rows == 0) return;
  const bool v4 = dim % 4 == 0 && ldh % 4 == 0 && y.ld % 4 == 0;
  auto go = [&](auto fn) { fn(y, w_post, mult, x, w_next, h, ldh, rows, dim, eps, stream); };
  if (f32) { if (v4) go(sandwich_launch<float, 4>); else go(sandwich_launch<float, 1>); }
  else     { if (v4) go(sandwich_launch<__nv_bfloat16, 4>); else go(sandwich_launch<__nv_bfloat16, 1>); }
  count_launch();
  check_launch();
}

void residual_norm(bool f32, const void* y, long long ldy, const float* bias, float mult, float* x, const float* w_next, void* h,
                   long long ldh, int rows, int dim, float eps, const ConvTail& conv, cudaStream_t stream) {
  MB_REQUIRE(dim > 0 && dim <= 12000 && ldh >= dim && ldy >= dim && w_next, "residual_norm: arguments");
  check_tail(conv, dim);
  if (rows == 0) return;
  const bool v4 = dim % 4 == 0 && ldh % 4 == 0 && ldy % 4 == 0;
#define MB_RNC(T, V, CONV)                                                                                                  \
  residual_norm_kernel<T, V, CONV><<<rows, SN_THREADS, dim * 4, stream>>>((const T*)y, ldy, bias, mult, x, w_next, (T*)h, ldh, \
                                                                          dim, eps, conv)
#define MB_RN(T, V) do { if (conv.c.taps > 0) MB_RNC(T, V, true); else MB_RNC(T, V, false); } while (0)
  if (f32) { if (v4) MB_RN(float, 4); else MB_RN(float, 1); }
  else     { if (v4) MB_RN(__nv_bfloat16, 4); else MB_RN(__nv_bfloat16, 1); }
#undef MB_RN
#undef MB_RNC
  count_launch();
  check_launch();
}

void poly_norm(bool f32, const void* y, long long ldy, const float* bias, const float* abce, void* out, long long ldo, int rows,
               int width, int padded, float eps, cudaStream_t stream) {
  MB_REQUIRE(width > 0 && ldy >= width && padded >= width && ldo >= padded && abce, "poly_norm: arguments");
  if (rows == 0) return;
  const int V = f32 ? 4 : 8;
  const bool vec = width % V == 0 && ldy % V == 0 && ldo % V == 0 &&
                   ((reinterpret_cast<uintptr_t>(y) | reinterpret_cast<uintptr_t>(out) | reinterpret_cast<uintptr_t>(bias)) & 15) == 0;
  const int units = width / V;
  if (!vec || units > 4096) {
    if (f32) poly_norm_any_kernel<float><<<rows, 256, 0, stream>>>((const float*)y, ldy, bias, abce, (float*)out, ldo, width, padded, eps);
    else
      poly_norm_any_kernel<__nv_bfloat16><<<rows, 256, 0, stream>>>((const __nv_bfloat16*)y, ldy, bias, abce, (__nv_bfloat16*)out, ldo,
                                                                    width, padded, eps);
  } else {
    const int nv = units <= 384 ? 1 : (units <= 768 ? 2 : (units <= 1152 ? 3 : (units <= 1536 ? 4 : (units <= 2304 ? 6 : 8))));
    const int threads = ((units + nv - 1) / nv + 31) / 32 * 32;
#define MB_PN(T, V, NV) \
  poly_norm_kernel<T, V, NV><<<rows, threads, 0, stream>>>((const T*)y, ldy, bias, abce, (T*)out, ldo, width, padded, eps)
#define MB_PNV(T, V)                                                                                               \
  do {                                                                                                             \
    if (nv == 1) MB_PN(T, V, 1); else if (nv == 2) MB_PN(T, V, 2); else if (nv == 3) MB_PN(T, V, 3);               \
    else if (nv == 4) MB_PN(T, V, 4); else if (nv == 6) MB_PN(T, V, 6); else MB_PN(T, V, 8);                       \
  } while (0)
    if (f32) MB_PNV(float, 4); else MB_PNV(__nv_bfloat16, 8);
#undef MB_PNV
#undef MB_PN
  }
  count_launch();
  check_launch();
}

void sigmoid_mul(bool f32, void* y, long long ldy, const void* gate, long long ld_gate, int rows, int width, cudaStream_t stream) {
  MB_REQUIRE(ldy >= width && ld_gate >= width, "sigmoid_mul: strides");
  if (rows == 0 || width == 0) return;
  const int grid = grid_for((long long)rows * width, 256, 16);
  if (f32)
    sigmoid_mul_kernel<float><<<grid, 256, 0, stream>>>((float*)y, ldy, (const float*)gate, ld_gate, rows, width);
  else
    sigmoid_mul_kernel<__nv_bfloat16><<<grid, 256, 0, stream>>>((__nv_bfloat16*)y, ldy, (const __nv_bfloat16*)gate, ld_gate, rows, width);
  count_launch();
  check_launch();
}

void attn_prep(bool f32, const void* proj, long long ld, const HeadPrep& p, const RaggedBatch& rb, const int* block_table,
               int table_stride, int page_size, void* q_out, void* k_cache, void* v_cache, cudaStream_t stream) {
  MB_REQUIRE(p.rot >= 0 && p.rot % 2 == 0 && p.rot <= p.dk && (p.rot == 0 || p.turns), "attn_prep: rotated columns");
  MB_REQUIRE(p.temp_coef == 0.f || p.temp_every > 0.f, "attn_prep: query temperature");
  if (rb.rows == 0) return;
  const int slots = p.heads + (p.k_off < 0 ? 0 : 2 * p.kv_heads);
  const bool kv = p.k_off >= 0;
  if (!f32 && p.dk % 8 == 0 && p.dv % 8 == 0 && p.dk <= 128 && p.dv <= 128 &&
      ((ld | p.q_off | (kv ? p.k_off | p.v_off : 0)) & 7) == 0 && (reinterpret_cast<uintptr_t>(proj) & 15) == 0) {
    // enough head slots for a few rounds of a block's 16 groups, but no fewer blocks than SMs
    int tokens = (128 + slots - 1) / slots;
    const int most = rb.rows / (4 * sm_count());
    if (tokens > most) tokens = most;
    if (tokens > AP_TOKENS) tokens = AP_TOKENS;
    if (tokens < 1) tokens = 1;
    attn_prep8_kernel<<<(rb.rows + tokens - 1) / tokens, AP_THREADS, tokens * (p.rot / 2) * 8, stream>>>(
        (const __nv_bfloat16*)proj, ld, p, rb, block_table, table_stride, page_size, tokens, (__nv_bfloat16*)q_out,
        (__nv_bfloat16*)k_cache, (__nv_bfloat16*)v_cache);
    count_launch();
    check_launch();
    return;
  }
  const int grid = ceil_div((long long)rb.rows * slots, 8);
  if (f32)
    attn_prep_kernel<float><<<grid, 256, 0, stream>>>((const float*)proj, ld, p, rb, block_table, table_stride, page_size,
                                                      (float*)q_out, (float*)k_cache, (float*)v_cache);
  else
    attn_prep_kernel<__nv_bfloat16><<<grid, 256, 0, stream>>>((const __nv_bfloat16*)proj, ld, p, rb, block_table, table_stride,
                                                              page_size, (__nv_bfloat16*)q_out, (__nv_bfloat16*)k_cache,
                                                              (__nv_bfloat16*)v_cache);
  count_launch();
  check_launch();
}

void paged_attn_any(bool f32, const void* q, const void* k_cache, const void* v_cache, const RaggedBatch& rb,
                    const int* block_table, int table_stride, int page_size, const AttnExtras& ex, void* o, long long ldo,
                    int heads, int kv_heads, int dk, int dv, float scale, cudaStream_t stream) {
  MB_REQUIRE(heads % kv_heads == 0, "paged_attn_any: heads must be a multiple of kv_heads");
  MB_REQUIRE(dk <= 1024 && dv <= 512, "paged_attn_any: head widths up to 1024 (keys) and 512 (values)");
  if (rb.rows == 0) return;
  const int grid = ceil_div((long long)rb.rows * heads, PA_WARPS);
  const int smem = PA_WARPS * dk * 4;
#define MB_PA(T, ND)                                                                                              \
  paged_attn_any_kernel<T, ND><<<grid, PA_WARPS * 32, smem, stream>>>(                                            \
      (const T*)q, (const T*)k_cache, (const T*)v_cache, rb, block_table, table_stride, page_size, ex, (T*)o, ldo, \
      heads, kv_heads, dk, dv, scale)
  if (f32) {
    if (dv <= 64) MB_PA(float, 2); else if (dv <= 128) MB_PA(float, 4); else if (dv <= 256) MB_PA(float, 8);
    else MB_PA(float, 16);
  } else {
    if (dv <= 64) MB_PA(__nv_bfloat16, 2); else if (dv <= 128) MB_PA(__nv_bfloat16, 4);
    else if (dv <= 256) MB_PA(__nv_bfloat16, 8); else MB_PA(__nv_bfloat16, 16);
  }
#undef MB_PA
  count_launch();
  check_launch();
}

void gemm_f32(const float* A, long long lda, const float* B, long long ldb, float* C, long long ldc, int M, int N,
              int K, float alpha, cudaStream_t stream, int batch, long long a_batch, long long b_batch, long long c_batch,
              const TileList* list) {
  if (M == 0 || N == 0 || batch == 0) return;
  const dim3 grid((N + 63) / 64, list ? 1 : (M + 63) / 64, list ? list->max_tiles : batch);
  gemm_f32_kernel<<<grid, 256, 0, stream>>>(A, lda, B, ldb, C, ldc, M, N, K, alpha, a_batch, b_batch, c_batch,
                                            list ? *list : TileList{nullptr, nullptr, 0});
  count_launch();
  check_launch();
}

void gate_pair(bool f32, const void* gu, long long ldg, int f, int f_off, const GateAct& act, void* h, long long ldh, int rows,
               cudaStream_t stream) {
  if (rows == 0) return;
  const int grid = grid_for((long long)rows * ldh, 256, 16);
  if (f32)
    gate_pair_kernel<float><<<grid, 256, 0, stream>>>((const float*)gu, ldg, f, f_off, act, (float*)h, ldh, rows);
  else
    gate_pair_kernel<__nv_bfloat16><<<grid, 256, 0, stream>>>((const __nv_bfloat16*)gu, ldg, f, f_off, act,
                                                              (__nv_bfloat16*)h, ldh, rows);
  count_launch();
  check_launch();
}

void gelu_mul(bool f32, void* y, long long ldy, const void* table, long long ld_table, const int* ids, int vocab, int rows,
              int width, cudaStream_t stream) {
  if (rows == 0 || width == 0) return;
  const int grid = grid_for((long long)rows * width, 256, 16);
  if (f32)
    gelu_mul_kernel<float><<<grid, 256, 0, stream>>>((float*)y, ldy, (const float*)table, ld_table, ids, vocab, rows, width);
  else
    gelu_mul_kernel<__nv_bfloat16><<<grid, 256, 0, stream>>>((__nv_bfloat16*)y, ldy, (const __nv_bfloat16*)table, ld_table, ids,
                                                             vocab, rows, width);
  count_launch();
  check_launch();
}

void soft_cap(float* y, long long ldy, int rows, int width, float cap, cudaStream_t stream) {
  MB_REQUIRE(cap > 0.f && ldy >= width, "soft_cap: arguments");
  if (rows == 0 || width == 0) return;
  soft_cap_kernel<<<grid_for((long long)rows * width, 256, 16), 256, 0, stream>>>(y, ldy, rows, width, cap);
  count_launch();
  check_launch();
}

}  // namespace mb
