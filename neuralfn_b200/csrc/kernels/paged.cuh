// Shared by the paged kernels: 4- and 8-wide loads / stores of bf16 and fp32 rows, activations, the page size.
#pragma once
#include "nfn_kernels.h"
#include "sm100_ptx.cuh"

namespace nfn {

constexpr int NFN_PAGE = 64;   // tokens per cache page
constexpr int PAGED_COUNTER_BYTES = 64 * 1024;

// the oldest key a query sees, apart from kept first tokens
__device__ __forceinline__ int first_visible(const nfn_paged_attention_args& a, int pos) {
  if (a.chunk > 0) return pos / a.chunk * a.chunk;
  return a.window > 0 ? max(0, pos - a.window + 1) : 0;
}

template <typename T>
__device__ __forceinline__ T from_float(float v);
template <>
__device__ __forceinline__ float from_float<float>(float v) { return v; }
template <>
__device__ __forceinline__ __nv_bfloat16 from_float<__nv_bfloat16>(float v) { return __float2bfloat16(v); }
__device__ __forceinline__ float to_float(float v) { return v; }
__device__ __forceinline__ float to_float(__nv_bfloat16 v) { return __bfloat162float(v); }

__device__ __forceinline__ float4 load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 load4(const __nv_bfloat16* p) {
  const uint2 u = *reinterpret_cast<const uint2*>(p);
  const float2 a = unpack_bf16x2(u.x), b = unpack_bf16x2(u.y);
  return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void store4(float* p, const float4& v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void store4(__nv_bfloat16* p, const float4& v) {
  *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(v.x, v.y), pack_bf16x2(v.z, v.w));
}
__device__ __forceinline__ void load8(const float* p, float (&v)[8]) {
  const float4 a = load4(p), b = load4(p + 4);
  v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
}
__device__ __forceinline__ void load8(const __nv_bfloat16* p, float (&v)[8]) {
  const uint4 u = *reinterpret_cast<const uint4*>(p);
  const float2 a = unpack_bf16x2(u.x), b = unpack_bf16x2(u.y), c = unpack_bf16x2(u.z), d = unpack_bf16x2(u.w);
  v[0] = a.x; v[1] = a.y; v[2] = b.x; v[3] = b.y; v[4] = c.x; v[5] = c.y; v[6] = d.x; v[7] = d.y;
}
__device__ __forceinline__ void store8(float* p, const float (&v)[8]) {
  store4(p, make_float4(v[0], v[1], v[2], v[3]));
  store4(p + 4, make_float4(v[4], v[5], v[6], v[7]));
}
__device__ __forceinline__ void store8(__nv_bfloat16* p, const float (&v)[8]) {
  *reinterpret_cast<uint4*>(p) = make_uint4(pack_bf16x2(v[0], v[1]), pack_bf16x2(v[2], v[3]), pack_bf16x2(v[4], v[5]), pack_bf16x2(v[6], v[7]));
}
__device__ __forceinline__ uint4 pack16(const float* v) {
  return make_uint4(__float_as_uint(v[0]), __float_as_uint(v[1]), __float_as_uint(v[2]), __float_as_uint(v[3]));
}
__device__ __forceinline__ uint4 pack16(const __nv_bfloat16* v) {
  uint32_t w[4];
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    __nv_bfloat162 h;
    h.x = v[2 * i];
    h.y = v[2 * i + 1];
    w[i] = *reinterpret_cast<uint32_t*>(&h);
  }
  return make_uint4(w[0], w[1], w[2], w[3]);
}

// exact forms (the GEMM epilogues use the hardware tanh)
__device__ __forceinline__ float gelu_tanh_exact(float x) {
  return 0.5f * x * (1.f + tanhf(0.7978845608028654f * (x + 0.044715f * x * x * x)));
}
__device__ __forceinline__ float ff_act(float v, int act) {
  if (act == NFN_ACT_RELU) return fmaxf(v, 0.f);
  if (act == NFN_ACT_SILU) return v / (1.f + expf(-v));
  if (act == NFN_ACT_GELU_TANH) return gelu_tanh_exact(v);
  if (act == NFN_ACT_RELU2) return fmaxf(v, 0.f) * fmaxf(v, 0.f);
  return v;
}
// by activation type: exact in 32-bit mode; for results that are rounded to bf16 the exponential and reciprocal units (a few ulp of fp32)
template <typename T>
__device__ __forceinline__ float sigmoid_for(float v) {
  if constexpr (sizeof(T) == 4) return 1.f / (1.f + expf(-v));
  else return fast_rcp(1.f + fast_exp2(v * -1.4426950408889634f));
}
__device__ __forceinline__ float sigmoid_exact(float v) { return 1.f / (1.f + expf(-v)); }

// the product of a feed-forward's gate and up values
template <typename T>
__device__ __forceinline__ float ff_gated(float g, float u, int act, const nfn_gate_clamp& c) {
  if (act != NFN_ACT_CLAMPED) return ff_act(g, act) * u;
  g = fminf(g, c.limit);
  u = fmaxf(-c.limit, fminf(u, c.limit));
  return g * sigmoid_for<T>(c.slope * g) * (u + c.shift);
}

// the score without a key in a row's softmax: is there one, and its value
__device__ __forceinline__ bool has_sink(const nfn_paged_attention_args& a) { return a.sink || a.sinks; }
__device__ __forceinline__ float sink_score(const nfn_paged_attention_args& a, int h) {
  return a.sinks ? __bfloat162float(static_cast<const __nv_bfloat16*>(a.sinks)[h]) : 0.f;
}

}  // namespace nfn
