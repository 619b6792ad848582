// Which experts a token uses and how much each counts, by one warp: scores, choice scores with a correction, groups of experts, normalised weights.
// Shared by the routing kernels of moe.cu and moe_rows.cu.
#pragma once
#include "paged.cuh"

namespace nfn {

// element i (a run-time number) of a register array
template <int PER>
__device__ __forceinline__ float pick(const float (&v)[PER], int i) {
  float r = v[0];
#pragma unroll
  for (int k = 1; k < PER; ++k) r = i == k ? v[k] : r;
  return r;
}

// Largest value not taken yet over the warp (ties: the lower index); lane l holds entries l, l + 32, ... of which `n` exist.
template <int PER>
__device__ __forceinline__ void best_of(const float (&v)[PER], uint32_t taken, int n, int lane, float& best, int& index) {
  best = -INFINITY;
  index = 0x7fffffff;
#pragma unroll
  for (int i = 0; i < PER; ++i)
    if (lane + 32 * i < n && !((taken >> i) & 1u) && (index == 0x7fffffff || v[i] > best)) { best = v[i]; index = lane + 32 * i; }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    const float ov = __shfl_xor_sync(0xffffffffu, best, o);
    const int oi = __shfl_xor_sync(0xffffffffu, index, o);
    if (oi != 0x7fffffff && (index == 0x7fffffff || ov > best || (ov == best && oi < index))) { best = ov; index = oi; }
  }
}

// Chooses `top` of `experts` for one token with router logits z; idx and weight [top] in global memory. PER: experts per lane.
template <int PER>
__device__ __forceinline__ void choose_experts(const float* z, int experts, int top, const nfn_route_rule& rule, int lane, int* idx, float* weight) {
  float s[PER], c[PER];
  const __nv_bfloat16* corr = static_cast<const __nv_bfloat16*>(rule.correction);
  const bool by_score = corr || rule.groups > 0;           // else by the logits themselves: the same order, no ties where the sigmoid saturates
#pragma unroll
  for (int i = 0; i < PER; ++i) {
    const int e = lane + 32 * i;
    const float x = e < experts ? z[e] : 0.f;
    s[i] = sigmoid_exact(x);
    c[i] = e < experts ? (by_score ? s[i] + (corr ? __bfloat162float(corr[e]) : 0.f) : x) : -INFINITY;
  }
  if (rule.groups > 0 && rule.keep_groups < rule.groups) {
    const int n = experts / rule.groups;
    float gs[PER];
#pragma unroll
    for (int i = 0; i < PER; ++i) gs[i] = -INFINITY;
    for (int g = 0; g < rule.groups; ++g) {                // sum of the group's two largest
      float a = -INFINITY, b = -INFINITY;
#pragma unroll
      for (int i = 0; i < PER; ++i) {
        const int at = lane + 32 * i - g * n;
        if (at >= 0 && at < n) {
          b = fmaxf(b, fminf(a, c[i]));
          a = fmaxf(a, c[i]);
        }
      }
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) {
        const float oa = __shfl_xor_sync(0xffffffffu, a, o), ob = __shfl_xor_sync(0xffffffffu, b, o);
        b = fmaxf(fmaxf(b, ob), fminf(a, oa));
        a = fmaxf(a, oa);
      }
      const float sum = n > 1 ? a + b : a;
#pragma unroll
      for (int i = 0; i < PER; ++i)
        if (g == lane + 32 * i) gs[i] = sum;
    }
    uint32_t kept = 0;                                     // of this lane's groups
    for (int j = 0; j < rule.keep_groups; ++j) {
      float best;
      int g;
      best_of<PER>(gs, kept, rule.groups, lane, best, g);
      if ((g & 31) == lane) kept |= 1u << (g >> 5);
    }
#pragma unroll
    for (int i = 0; i < PER; ++i) {
      const int e = lane + 32 * i, g = e < experts ? e / n : 0;
      const uint32_t of_group = __shfl_sync(0xffffffffu, kept, g & 31);
      if (e < experts && !((of_group >> (g >> 5)) & 1u)) c[i] = -INFINITY;
    }
  }
  uint32_t taken = 0;
  float sum = 0.f, first = 0.f;
  const float scale = rule.scale == 0.f ? 1.f : rule.scale;
  for (int j = 0; j < top; ++j) {
    float best;
    int e;
    best_of<PER>(c, taken, experts, lane, best, e);
    if ((e & 31) == lane) taken |= 1u << (e >> 5);
    float w = __shfl_sync(0xffffffffu, pick<PER>(s, e >> 5), e & 31);
    if (j == 0) first = best;
    if (rule.softmax) w = expf(best - first);               // the choice went by the logits, largest first
    sum += w;
    if (lane == (j & 31)) {
      idx[j] = e;
      weight[j] = w * scale;
    }
  }
  if (rule.normalise || rule.softmax) {
    const float f = 1.f / (rule.softmax ? sum : sum + 1e-20f);
    for (int j = lane; j < top; j += 32) weight[j] *= f;   // this lane's own entries
  }
}

}  // namespace nfn
