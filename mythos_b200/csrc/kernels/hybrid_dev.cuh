// Device helpers shared by the layer-list model kernels.
#pragma once
#include <cuda_bf16.h>

#include "common.cuh"
#include "hybrid_api.h"
#include "tc.cuh"

namespace mb {

__device__ __forceinline__ float ldf(const float* p) { return *p; }
__device__ __forceinline__ float ldf(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void stf(float* p, float v) { *p = v; }
__device__ __forceinline__ void stf(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }

__device__ __forceinline__ float sigmoid_f(float z) { return 1.f / (1.f + expf(-z)); }
__device__ __forceinline__ float silu_f(float z) { return z / (1.f + expf(-z)); }
__device__ __forceinline__ float softplus_f(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

__device__ __forceinline__ float gate_act(const GateAct& a, float g, float u) {
  if (a.kind == 0) return silu_f(g) * u;
  if (a.kind == 1) return fmaxf(g, 0.f) * u;
  g = fminf(g, a.limit);
  u = fminf(fmaxf(u, -a.limit), a.limit);
  return g * sigmoid_f(a.alpha * g) * (u + 1.f);
}
__device__ __forceinline__ float soft_cap_f(float y, float cap) { return cap * tanhf(y / cap); }
__device__ __forceinline__ float gelu_tanh_f(float z) {
  return 0.5f * z * (1.f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
}

__device__ __forceinline__ float fast_rcp(float x) {
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// z / (1 + e^-z)
__device__ __forceinline__ float silu_fast(float z) { return z * fast_rcp(1.f + fast_exp2(-1.4426950408889634f * z)); }

template <typename T>
__device__ __forceinline__ float silu_t(float z) {
  if constexpr (sizeof(T) == 2) return silu_fast(z);
  else return silu_f(z);
}

// V neighbouring values; V = 8 (bf16), 4 and multiples take whole vectors.
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
  } else if constexpr (V == 4) {
    const uint2 t = *reinterpret_cast<const uint2*>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&t.x));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&t.y));
    f[0] = a.x; f[1] = a.y; f[2] = b.x; f[3] = b.y;
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
  if constexpr (V == 4) {
    *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(f[0], f[1]), pack_bf16x2(f[2], f[3]));
  } else {
#pragma unroll
    for (int i = 0; i < V; ++i) p[i] = __float2bfloat16(f[i]);
  }
}

// Convolution of channel c for one new token (without bias); the state takes the token in. state: the sequence's
// [taps - 1][channels], fresh: it has no earlier tokens.
__device__ __forceinline__ float conv_step(const ShortConv& s, float* state, bool fresh, int c, float cur) {
  const float* w = s.w + c;
  float acc = w[(long long)(s.taps - 1) * s.channels] * cur;
  if (s.taps == 4) {                               // all loads before the stores
    float* st = state + c;
    float old[3];
#pragma unroll
    for (int j = 0; j < 3; ++j) old[j] = fresh ? 0.f : st[(long long)j * s.channels];
#pragma unroll
    for (int j = 0; j < 3; ++j) acc = fmaf(w[(long long)j * s.channels], old[j], acc);
    st[0] = old[1];
    st[s.channels] = old[2];
    st[2ll * s.channels] = cur;
  } else {
    float nxt = cur;                               // newest first: entry j moves to j - 1
    for (int j = s.taps - 2; j >= 0; --j) {
      float* st = state + (long long)j * s.channels + c;
      const float old = fresh ? 0.f : *st;
      acc = fmaf(w[(long long)j * s.channels], old, acc);
      *st = nxt;
      nxt = old;
    }
  }
  return acc;
}

}  // namespace mb
