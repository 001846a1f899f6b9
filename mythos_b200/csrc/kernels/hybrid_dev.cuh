// Device helpers shared by the layer-list model kernels.
#pragma once
#include <cuda_bf16.h>

#include "hybrid_api.h"

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

}  // namespace mb
