// Mixture of experts for a handful of rows (decoding, short portions) and in 32-bit mode: one launch routes the rows and lists every
// expert's items, then each chosen expert's weights are streamed once per group of eight items - a warp per weight row, its lanes
// across the input width. Also the gate of the sorted prompt rows (the grouped GEMMs around it are in gemm_tp.cu).
//
// The routing weight multiplies the expert's input. Gate and up are linear, so it is applied to their fp32 results instead:
// act(w g) * (w u).
#include "common.h"
#include "paged.cuh"

namespace nfn {

constexpr int MR_MAX_EXPERTS = 1024, MR_GROUP = 8, MR_WARPS = 8;

// One CTA. Scores: sigmoid of the fp32 logits; the `top` largest per row (ties: the lower index).
__global__ void __launch_bounds__(1024)
moe_route_rows_kernel(const nfn_moe_rows_args p) {
  __shared__ int count[MR_MAX_EXPERTS], start[MR_MAX_EXPERTS + 1];
  const int E = p.experts, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  for (int e = threadIdx.x; e < E; e += 1024) count[e] = 0;
  __syncthreads();
  for (int r = warp; r < p.rows; r += 32) {
    const float* z = p.logits + (size_t)r * p.ld_logits;
    for (int j = 0; j < p.top; ++j) {
      // the next one in (score falling, index rising) order after the one chosen before
      float best = -INFINITY;
      int bi = 0x7fffffff;
      const int prev = j > 0 ? p.idx[(size_t)r * p.top + j - 1] : -1;
      const float pz = prev >= 0 ? z[prev] : INFINITY;
      for (int e = lane; e < E; e += 32) {
        const float v = z[e];
        const bool open = prev < 0 || v < pz || (v == pz && e > prev);
        if (open && (bi == 0x7fffffff || v > best)) { best = v; bi = e; }
      }
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) {
        const float ov = __shfl_xor_sync(0xffffffffu, best, o);
        const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
        if (oi != 0x7fffffff && (bi == 0x7fffffff || ov > best || (ov == best && oi < bi))) { best = ov; bi = oi; }
      }
      if (lane == 0) {
        bi = min(bi, E - 1);
        p.idx[(size_t)r * p.top + j] = bi;
        p.weight[(size_t)r * p.top + j] = sigmoid_exact(best);
        atomicAdd(&count[bi], 1);
      }
      __syncwarp();
    }
  }
  __syncthreads();
  if (threadIdx.x == 0) {
    int run = 0, live = 0;
    for (int e = 0; e < E; ++e) {
      start[e] = run;
      p.offsets[e] = run;
      run += count[e];
      if (count[e] > 0) p.active[live++] = e;
    }
    p.offsets[E] = run;
    p.active[E] = live;
  }
  __syncthreads();
  for (int i = threadIdx.x; i < p.rows * p.top; i += 1024) p.order[atomicAdd(&start[p.idx[i]], 1)] = i;
}

// DOWN = false: mid[item][f] = act(w G_f h) * (w U_f h), h of the item's row. DOWN = true: y[item][n] = D_n mid[item].
template <typename T, bool DOWN>
__global__ void __launch_bounds__(MR_WARPS * 32)
moe_products_kernel(const nfn_moe_rows_args p) {
  if ((int)blockIdx.y >= p.active[p.experts]) return;
  const int e = p.active[blockIdx.y], warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int n = blockIdx.x * MR_WARPS + warp, N = DOWN ? p.width : p.ff, K = DOWN ? p.ff : p.width;
  if (n >= N) return;
  const __nv_bfloat16* wa = DOWN ? static_cast<const __nv_bfloat16*>(p.w_down) + ((size_t)e * N + n) * K
                                 : static_cast<const __nv_bfloat16*>(p.w_gate_up) + ((size_t)e * 2 * N + n) * K;
  const __nv_bfloat16* wb = DOWN ? wa : wa + (size_t)N * K;
  const int i0 = p.offsets[e], i1 = p.offsets[e + 1];
  for (int g = i0; g < i1; g += MR_GROUP) {
    const int m = min(MR_GROUP, i1 - g);
    const T* src[MR_GROUP];
#pragma unroll
    for (int i = 0; i < MR_GROUP; ++i) {
      const int item = p.order[i < m ? g + i : g];
      src[i] = DOWN ? static_cast<const T*>(p.mid) + (size_t)item * p.ff : static_cast<const T*>(p.h) + (size_t)(item / p.top) * p.ld_h;
    }
    float a[MR_GROUP], b[MR_GROUP];
#pragma unroll
    for (int i = 0; i < MR_GROUP; ++i) a[i] = b[i] = 0.f;
    constexpr int U = 2;
    for (int k0 = lane * 8; k0 < K; k0 += 256 * U) {
      float va[U][8], vb[U][8];
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int k = k0 + u * 256;
        if (k < K) {
          load8(wa + k, va[u]);
          if (!DOWN) load8(wb + k, vb[u]);
        }
      }
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int k = k0 + u * 256;
        if (k >= K) break;
#pragma unroll
        for (int i = 0; i < MR_GROUP; ++i) {
          if (i >= m) break;
          float x[8];
          load8(src[i] + k, x);
#pragma unroll
          for (int c = 0; c < 8; ++c) {
            a[i] += va[u][c] * x[c];
            if (!DOWN) b[i] += vb[u][c] * x[c];
          }
        }
      }
    }
#pragma unroll
    for (int i = 0; i < MR_GROUP; ++i) {
      if (i >= m) break;
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) {
        a[i] += __shfl_xor_sync(0xffffffffu, a[i], o);
        if (!DOWN) b[i] += __shfl_xor_sync(0xffffffffu, b[i], o);
      }
      if (lane == 0) {
        const int item = p.order[g + i];
        if (DOWN) {
          static_cast<T*>(p.y)[(size_t)item * p.ld_y + n] = from_float<T>(a[i]);
        } else {
          const float w = p.weight[item];
          static_cast<T*>(p.mid)[(size_t)item * p.ff + n] = from_float<T>(ff_act(w * a[i], p.act) * (w * b[i]));
        }
      }
    }
  }
}

// Sorted prompt rows: mid = act(w g) * (w u). Rows past the plan's count stay untouched.
__global__ void __launch_bounds__(256)
moe_act_rows_kernel(const __nv_bfloat16* __restrict__ gate_up, const float* __restrict__ row_w, const int* __restrict__ plan, int ff, int act,
                    __nv_bfloat16* __restrict__ mid) {
  const int r = blockIdx.x, c = (blockIdx.y * 256 + threadIdx.x) * 8;
  if (r >= plan[1] || c >= ff) return;
  float g[8], u[8];
  load8(gate_up + (size_t)r * 2 * ff + c, g);
  load8(gate_up + (size_t)r * 2 * ff + ff + c, u);
  const float w = row_w[r];
#pragma unroll
  for (int i = 0; i < 8; ++i) g[i] = ff_act(w * g[i], act) * (w * u[i]);
  store8(mid + (size_t)r * ff + c, g);
}

template <typename T>
static int launch_moe_rows(const nfn_moe_rows_args& a, cudaStream_t st) {
  const int live = (int)min((long long)a.experts, (long long)a.rows * a.top);     // most experts that can have items
  moe_route_rows_kernel<<<1, 1024, 0, st>>>(a);
  moe_products_kernel<T, false><<<dim3(ceil_div(a.ff, MR_WARPS), live), MR_WARPS * 32, 0, st>>>(a);
  moe_products_kernel<T, true><<<dim3(ceil_div(a.width, MR_WARPS), live), MR_WARPS * 32, 0, st>>>(a);
  return launch_check("moe_rows", 3);
}

}  // namespace nfn

using namespace nfn;

extern "C" int nfn_moe_rows(const nfn_moe_rows_args* args, nfn_stream_t stream) {
  if (!args) return fail(-1, "moe_rows: null args");
  const nfn_moe_rows_args& a = *args;
  if (a.rows <= 0) return 0;
  if (a.experts < 1 || a.experts > MR_MAX_EXPERTS || a.top < 1 || a.top > a.experts) return fail(-1, "moe_rows: need 1 <= top <= experts <= 1024");
  if ((a.width | a.ff | a.ld_h) & 7) return fail(-1, "moe_rows: widths must be multiples of 8");
  if ((long long)a.rows * a.top > 0x7fffffffLL / 2) return fail(-1, "moe_rows: too many rows");
  return a.f32 ? launch_moe_rows<float>(a, static_cast<cudaStream_t>(stream)) : launch_moe_rows<__nv_bfloat16>(a, static_cast<cudaStream_t>(stream));
}

extern "C" int nfn_moe_act_rows(const void* gate_up, const float* row_w, const int* plan, int capacity_rows, int ff, int act, void* mid, nfn_stream_t stream) {
  if (capacity_rows <= 0) return 0;
  if (ff & 7) return fail(-1, "moe_act_rows: the width must be a multiple of 8");
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const __nv_bfloat16* gu = static_cast<const __nv_bfloat16*>(gate_up);
  __nv_bfloat16* out = static_cast<__nv_bfloat16*>(mid);
  moe_act_rows_kernel<<<dim3(capacity_rows, ceil_div(ff, 256 * 8)), 256, 0, st>>>(gu, row_w, plan, ff, act, out);
  return launch_check("moe_act_rows");
}
