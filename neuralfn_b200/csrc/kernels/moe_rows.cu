// Mixture of experts for a handful of rows (decoding, short portions) and in 32-bit mode: one launch routes the rows and lists every
// expert's items, then each chosen expert's weights are streamed once per group of items: on the tensor cores in bf16, a warp per
// weight row in 32-bit mode. Also the gate of the sorted prompt rows (the grouped GEMMs around it are in gemm_tp.cu).
//
// For gated experts the routing weight multiplies the input. Gate and up are linear, so it is applied to their fp32 results instead:
// act(w g) * (w u). Plain experts, act(u), leave it to the pass that sums a token's items.
#include <algorithm>

#include "common.h"
#include "moe_choice.cuh"
#include "paged.cuh"

namespace nfn {

constexpr int MR_MAX_EXPERTS = 1024, MR_GROUP = 8, MR_WARPS = 8;

// One CTA, a warp per row. PER: experts per lane (experts <= 32 PER).
template <int PER>
__global__ void __launch_bounds__(1024)
moe_route_rows_kernel(const nfn_moe_rows_args p) {
  __shared__ int count[MR_MAX_EXPERTS], start[MR_MAX_EXPERTS], warp_sum[32], warp_live[32];
  const int E = p.experts, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  count[threadIdx.x] = 0;
  __syncthreads();
  for (int r = warp; r < p.rows; r += 32) {
    int* idx = p.idx + (size_t)r * p.top;
    choose_experts<PER>(p.logits + (size_t)r * p.ld_logits, E, p.top, p.rule, lane, idx, p.weight + (size_t)r * p.top);
    for (int j = lane; j < p.top; j += 32) atomicAdd(&count[idx[j]], 1);       // this lane's own entries
  }
  __syncthreads();
  // first item of every expert, and the experts that have items
  const int e = threadIdx.x, mine = e < E ? count[e] : 0;
  int run = mine;
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const int up = __shfl_up_sync(0xffffffffu, run, o);
    if (lane >= o) run += up;
  }
  const uint32_t live = __ballot_sync(0xffffffffu, mine > 0);
  if (lane == 31) {
    warp_sum[warp] = run;
    warp_live[warp] = __popc(live);
  }
  __syncthreads();
  int base = 0, slot = 0;
  for (int w = 0; w < warp; ++w) {
    base += warp_sum[w];
    slot += warp_live[w];
  }
  if (e < E) {
    start[e] = p.offsets[e] = base + run - mine;
    if (mine > 0) p.active[slot + __popc(live & ((1u << lane) - 1u))] = e;
    if (e == E - 1) {
      p.offsets[E] = base + run;
      p.active[E] = slot + __popc(live);
    }
  }
  __syncthreads();
  for (int i = threadIdx.x; i < p.rows * p.top; i += 1024) p.order[atomicAdd(&start[p.idx[i]], 1)] = i;
}

// What a launch computes. kGateUp: mid[item][f] = act(w G_f h) * (w U_f h), h of the item's row; kDown: y[item][n] = D_n mid[item]; kUp: mid[item][f] = act(U_f h).
enum { kGateUp = 0, kDown = 1, kUp = 2 };

// 32-bit mode
template <typename T, int FORM>
__global__ void __launch_bounds__(MR_WARPS * 32)
moe_products_kernel(const nfn_moe_rows_args p) {
  constexpr bool DOWN = FORM == kDown, TWO = FORM == kGateUp;
  const bool shared = DOWN && p.shared_ff > 0 && blockIdx.y == 0;        // the expert of all rows comes first
  const int at = blockIdx.y - (DOWN && p.shared_ff > 0 ? 1 : 0);
  if (!shared && at >= p.active[p.experts]) return;
  const int e = shared ? 0 : p.active[at], warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int n = blockIdx.x * MR_WARPS + warp, N = DOWN ? p.width : p.ff, K = DOWN ? (shared ? p.shared_ff : p.ff) : p.width;
  if (n >= N) return;
  const __nv_bfloat16* wa = DOWN ? static_cast<const __nv_bfloat16*>(shared ? p.w_shared_down : p.w_down) + ((size_t)e * N + n) * K
                                 : static_cast<const __nv_bfloat16*>(p.w_gate_up) + ((size_t)e * (TWO ? 2 : 1) * N + n) * K;
  const __nv_bfloat16* wb = TWO ? wa + (size_t)N * K : wa;
  const int i0 = shared ? 0 : p.offsets[e], i1 = shared ? p.rows : p.offsets[e + 1];
  for (int g = i0; g < i1; g += MR_GROUP) {
    const int m = min(MR_GROUP, i1 - g);
    const T* src[MR_GROUP];
#pragma unroll
    for (int i = 0; i < MR_GROUP; ++i) {
      const int item = shared ? (i < m ? g + i : g) : p.order[i < m ? g + i : g];
      src[i] = DOWN ? static_cast<const T*>(shared ? p.shared_mid : p.mid) + (size_t)item * K : static_cast<const T*>(p.h) + (size_t)(item / p.top) * p.ld_h;
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
          if (TWO) load8(wb + k, vb[u]);
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
            if (TWO) b[i] += vb[u][c] * x[c];
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
        if (TWO) b[i] += __shfl_xor_sync(0xffffffffu, b[i], o);
      }
      if (lane == 0) {
        const int item = shared ? g + i : p.order[g + i];
        if (DOWN) {
          static_cast<T*>(shared ? p.y_shared : p.y)[(size_t)item * p.ld_y + n] = from_float<T>(a[i]);
        } else if (!TWO) {
          static_cast<T*>(p.mid)[(size_t)item * p.ff + n] = from_float<T>(ff_act(a[i], p.act));
        } else {
          const float w = p.weigh_output ? 1.f : p.weight[item];
          static_cast<T*>(p.mid)[(size_t)item * p.ff + n] = from_float<T>(ff_gated<T>(w * a[i], w * b[i], p.act, p.clamp));
        }
      }
    }
  }
}

// The same on the tensor cores: a CTA takes 32 weight rows (kGateUp: 16 of gate and the 16 of up beside them), its four warps a quarter
// of the contraction each. Weight rows are the 16-row operand of mma.m16n8k16, items its eight columns; the order of the contraction is
// free, so every fragment is one 16-byte load per lane. Weights are read once per 8 NT items.
constexpr int MM_WARPS = 4;

__device__ __forceinline__ uint4 mm_stream(const __nv_bfloat16* p) {
  uint4 v;
  asm volatile("ld.global.nc.L1::no_allocate.v4.u32 {%0,%1,%2,%3}, [%4];" : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w) : "l"(p));
  return v;
}
__device__ __forceinline__ void mm_mma(float (&d)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
  asm("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
      : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
      : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}

template <int FORM, int NT>
__global__ void __launch_bounds__(MM_WARPS * 32)
moe_products_mma_kernel(const nfn_moe_rows_args p) {
  constexpr bool DOWN = FORM == kDown, TWO = FORM == kGateUp;
  constexpr int TILE = TWO ? 16 : 32;
  constexpr int M = 8 * NT;                               // items at a time
  constexpr int U = NT == 4 ? 2 : 4;                      // 32-channel steps in flight
  __shared__ float part[MM_WARPS][2][16][M + 1];
  const bool shared = DOWN && p.shared_ff > 0 && blockIdx.y == 0;        // the expert of all rows comes first
  const int at = blockIdx.y - (DOWN && p.shared_ff > 0 ? 1 : 0);
  if (!shared && at >= p.active[p.experts]) return;
  const int e = shared ? 0 : p.active[at], warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, j = lane & 3;
  const int N = DOWN ? p.width : p.ff, K = DOWN ? (shared ? p.shared_ff : p.ff) : p.width;
  const int n0 = blockIdx.x * TILE;
  // rows of the two 16-row tiles
  const __nv_bfloat16* w0 = (DOWN ? static_cast<const __nv_bfloat16*>(shared ? p.w_shared_down : p.w_down) + ((size_t)e * N + n0) * K : static_cast<const __nv_bfloat16*>(p.w_gate_up) + ((size_t)e * (TWO ? 2 : 1) * N + n0) * K) +
                            (size_t)g * K + 8 * j;
  const bool two = TWO || n0 + 16 < N;
  const __nv_bfloat16* w1 = two ? w0 + (size_t)(TWO ? N : 16) * K : w0;
  const int steps = (K + 31) / 32, s0 = steps * warp / MM_WARPS, s1 = steps * (warp + 1) / MM_WARPS;
  const uint4 zero4 = make_uint4(0u, 0u, 0u, 0u);
  const int i0 = shared ? 0 : p.offsets[e], i1 = shared ? p.rows : p.offsets[e + 1];
  auto item_at = [&](int i) { return shared ? i : p.order[i]; };
  for (int i = i0; i < i1; i += M) {
    const __nv_bfloat16* src[NT];
    bool on[NT];
#pragma unroll
    for (int t = 0; t < NT; ++t) {
      on[t] = i + 8 * t + g < i1;
      const int item = item_at(on[t] ? i + 8 * t + g : i0);
      src[t] = (DOWN ? static_cast<const __nv_bfloat16*>(shared ? p.shared_mid : p.mid) + (size_t)item * K : static_cast<const __nv_bfloat16*>(p.h) + (size_t)(item / p.top) * p.ld_h) + 8 * j;
    }
    float acc[2][NT][4];
#pragma unroll
    for (int m = 0; m < 2; ++m)
#pragma unroll
      for (int t = 0; t < NT; ++t)
#pragma unroll
        for (int c = 0; c < 4; ++c) acc[m][t][c] = 0.f;
    for (int s = s0; s < s1; s += U) {
      uint4 a[U][4], b[U][NT];
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int k = (s + u) * 32;
        const bool ok = s + u < s1 && k + 8 * j < K;
        a[u][0] = ok ? mm_stream(w0 + k) : zero4;
        a[u][1] = ok ? mm_stream(w0 + (size_t)8 * K + k) : zero4;
        a[u][2] = ok ? mm_stream(w1 + k) : zero4;
        a[u][3] = ok ? mm_stream(w1 + (size_t)8 * K + k) : zero4;
#pragma unroll
        for (int t = 0; t < NT; ++t) b[u][t] = ok && on[t] ? __ldg(reinterpret_cast<const uint4*>(src[t] + k)) : zero4;
      }
#pragma unroll
      for (int u = 0; u < U; ++u)
#pragma unroll
        for (int t = 0; t < NT; ++t) {
          mm_mma(acc[0][t], a[u][0].x, a[u][1].x, a[u][0].y, a[u][1].y, b[u][t].x, b[u][t].y);
          mm_mma(acc[1][t], a[u][2].x, a[u][3].x, a[u][2].y, a[u][3].y, b[u][t].x, b[u][t].y);
          mm_mma(acc[0][t], a[u][0].z, a[u][1].z, a[u][0].w, a[u][1].w, b[u][t].z, b[u][t].w);
          mm_mma(acc[1][t], a[u][2].z, a[u][3].z, a[u][2].w, a[u][3].w, b[u][t].z, b[u][t].w);
        }
    }
#pragma unroll
    for (int m = 0; m < 2; ++m)
#pragma unroll
      for (int t = 0; t < NT; ++t)
#pragma unroll
        for (int c = 0; c < 4; ++c) part[warp][m][g + (c >> 1) * 8][8 * t + 2 * j + (c & 1)] = acc[m][t][c];
    __syncthreads();
    const int live = min(M, i1 - i);
    for (int x = threadIdx.x; x < TILE * live; x += MM_WARPS * 32) {
      const int col = x / TILE, row = x % TILE, item = item_at(i + col);
      if (n0 + row >= N) continue;
      if (!TWO) {
        float v = 0.f;
#pragma unroll
        for (int w = 0; w < MM_WARPS; ++w) v += part[w][row >> 4][row & 15][col];
        if (DOWN) static_cast<__nv_bfloat16*>(shared ? p.y_shared : p.y)[(size_t)item * p.ld_y + n0 + row] = __float2bfloat16(v);
        else static_cast<__nv_bfloat16*>(p.mid)[(size_t)item * p.ff + n0 + row] = __float2bfloat16(ff_act(v, p.act));
      } else {
        float gv = 0.f, uv = 0.f;
#pragma unroll
        for (int w = 0; w < MM_WARPS; ++w) {
          gv += part[w][0][row][col];
          uv += part[w][1][row][col];
        }
        const float f = p.weigh_output ? 1.f : p.weight[item];
        static_cast<__nv_bfloat16*>(p.mid)[(size_t)item * p.ff + n0 + row] = __float2bfloat16(ff_gated<__nv_bfloat16>(f * gv, f * uv, p.act, p.clamp));
      }
    }
    __syncthreads();
  }
}

// Sorted prompt rows: mid = act(w g) * (w u). Rows past the plan's count stay untouched.
__global__ void __launch_bounds__(256)
moe_act_rows_kernel(const __nv_bfloat16* __restrict__ gate_up, const float* __restrict__ row_w, const int* __restrict__ plan, int ff, int act,
                    nfn_gate_clamp clamp, __nv_bfloat16* __restrict__ mid) {
  const int r = blockIdx.x, c = (blockIdx.y * 256 + threadIdx.x) * 8;
  if (r >= plan[1] || c >= ff) return;
  float g[8], u[8];
  load8(gate_up + (size_t)r * 2 * ff + c, g);
  load8(gate_up + (size_t)r * 2 * ff + ff + c, u);
  const float w = row_w ? row_w[r] : 1.f;
#pragma unroll
  for (int i = 0; i < 8; ++i) g[i] = ff_gated<__nv_bfloat16>(w * g[i], w * u[i], act, clamp);
  store8(mid + (size_t)r * ff + c, g);
}

// Router logits: the warps of a CTA share the contraction of one expert's row with eight rows of h, every load of a thread on its way at once.
constexpr int RT_WARPS = 8, RT_ROWS = 8;

__global__ void __launch_bounds__(RT_WARPS * 32)
router_rows_kernel(const __nv_bfloat16* __restrict__ h, int ld_h, const __nv_bfloat16* __restrict__ w, int rows, int width, float* __restrict__ logits, int ld_logits) {
  __shared__ float part[RT_WARPS][RT_ROWS];
  const int e = blockIdx.x, r0 = blockIdx.y * RT_ROWS, live = min(RT_ROWS, rows - r0), warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  float a[RT_ROWS];
#pragma unroll
  for (int i = 0; i < RT_ROWS; ++i) a[i] = 0.f;
  for (int k = threadIdx.x * 8; k < width; k += RT_WARPS * 32 * 8) {
    uint4 x[RT_ROWS];
    const uint4 u = *reinterpret_cast<const uint4*>(w + (size_t)e * width + k);
#pragma unroll
    for (int i = 0; i < RT_ROWS; ++i)
      if (i < live) x[i] = *reinterpret_cast<const uint4*>(h + (size_t)(r0 + i) * ld_h + k);
    const uint32_t uw[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
    for (int i = 0; i < RT_ROWS; ++i) {
      if (i >= live) break;
      const uint32_t xw[4] = {x[i].x, x[i].y, x[i].z, x[i].w};
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        const float2 f = unpack_bf16x2(uw[c]), g = unpack_bf16x2(xw[c]);
        a[i] += f.x * g.x + f.y * g.y;
      }
    }
  }
#pragma unroll
  for (int i = 0; i < RT_ROWS; ++i) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) a[i] += __shfl_xor_sync(0xffffffffu, a[i], o);
    if (lane == 0) part[warp][i] = a[i];
  }
  __syncthreads();
  if (threadIdx.x < live) {
    float t = 0.f;
#pragma unroll
    for (int q = 0; q < RT_WARPS; ++q) t += part[q][threadIdx.x];
    logits[(size_t)(r0 + threadIdx.x) * ld_logits + e] = t;
  }
}

template <int NT>
static void launch_products_mma(const nfn_moe_rows_args& a, int live, cudaStream_t st) {
  if (a.plain) moe_products_mma_kernel<kUp, NT><<<dim3(ceil_div(a.ff, 32), live), MM_WARPS * 32, 0, st>>>(a);
  else moe_products_mma_kernel<kGateUp, NT><<<dim3(ceil_div(a.ff, 16), live), MM_WARPS * 32, 0, st>>>(a);
  moe_products_mma_kernel<kDown, NT><<<dim3(ceil_div(a.width, 32), live + (a.shared_ff > 0)), MM_WARPS * 32, 0, st>>>(a);
}

static int launch_moe_rows(const nfn_moe_rows_args& a, cudaStream_t st) {
  const int live = (int)std::min<long long>(a.experts, (long long)a.rows * a.top);     // most experts that can have items
  if (a.experts <= 32) moe_route_rows_kernel<1><<<1, 1024, 0, st>>>(a);
  else if (a.experts <= 64) moe_route_rows_kernel<2><<<1, 1024, 0, st>>>(a);
  else if (a.experts <= 256) moe_route_rows_kernel<8><<<1, 1024, 0, st>>>(a);
  else moe_route_rows_kernel<32><<<1, 1024, 0, st>>>(a);
  if (a.f32) {
    if (a.plain) moe_products_kernel<float, kUp><<<dim3(ceil_div(a.ff, MR_WARPS), live), MR_WARPS * 32, 0, st>>>(a);
    else moe_products_kernel<float, kGateUp><<<dim3(ceil_div(a.ff, MR_WARPS), live), MR_WARPS * 32, 0, st>>>(a);
    moe_products_kernel<float, kDown><<<dim3(ceil_div(a.width, MR_WARPS), live + (a.shared_ff > 0)), MR_WARPS * 32, 0, st>>>(a);
  } else if (a.rows <= 8) {
    launch_products_mma<1>(a, live, st);
  } else if (a.rows <= 16) {
    launch_products_mma<2>(a, live, st);
  } else {
    launch_products_mma<4>(a, live, st);
  }
  return launch_check("moe_rows", 3);
}

}  // namespace nfn

using namespace nfn;

extern "C" int nfn_moe_rows(const nfn_moe_rows_args* args, nfn_stream_t stream) {
  if (!args) return fail(-1, "moe_rows: null args");
  const nfn_moe_rows_args& a = *args;
  if (a.rows <= 0) return 0;
  if (a.experts < 1 || a.experts > MR_MAX_EXPERTS || a.top < 1 || a.top > a.experts) return fail(-1, "moe_rows: need 1 <= top <= experts <= 1024");
  if (a.rule.groups < 0 || (a.rule.groups > 0 && (a.experts % a.rule.groups || a.rule.keep_groups < 1 || (long long)a.rule.keep_groups * (a.experts / a.rule.groups) < a.top)))
    return fail(-1, "moe_rows: the kept groups must hold the chosen experts");
  if (a.shared_ff < 0 || (a.shared_ff > 0 && ((a.shared_ff & 15) || !a.shared_mid || !a.w_shared_down || !a.y_shared))) return fail(-1, "moe_rows: the shared expert lacks an operand");
  if (a.rule.softmax && (a.rule.correction || a.rule.groups > 0)) return fail(-1, "moe_rows: the softmax over chosen logits has no correction or groups");
  if (a.plain && a.act == NFN_ACT_CLAMPED) return fail(-1, "moe_rows: the clamped gate needs gated experts");
  if ((a.width | a.ff | a.ld_h) & 15) return fail(-1, "moe_rows: widths must be multiples of 16");
  if ((long long)a.rows * a.top > 0x7fffffffLL / 2) return fail(-1, "moe_rows: too many rows");
  return launch_moe_rows(a, static_cast<cudaStream_t>(stream));
}

extern "C" int nfn_router_rows(const void* h, int ld_h, const void* w, int rows, int experts, int width, float* logits, int ld_logits, nfn_stream_t stream) {
  if (rows <= 0) return 0;
  if (experts < 1 || experts > ld_logits || (width & 15) || width <= 0 || (ld_h & 7) || !h || !w || !logits) return fail(-1, "router_rows: rows padded to multiples of 16, a logit per expert");
  if (ceil_div(rows, RT_ROWS) > 65535) return fail(-1, "router_rows: too many rows for one launch");
  router_rows_kernel<<<dim3(experts, ceil_div(rows, RT_ROWS)), RT_WARPS * 32, 0, static_cast<cudaStream_t>(stream)>>>(static_cast<const __nv_bfloat16*>(h), ld_h, static_cast<const __nv_bfloat16*>(w),
                                                                                                                 rows, width, logits, ld_logits);
  return launch_check("router_rows");
}

extern "C" int nfn_moe_act_rows(const void* gate_up, const float* row_w, const int* plan, int capacity_rows, int ff, int act, const nfn_gate_clamp* clamp, void* mid,
                                nfn_stream_t stream) {
  if (capacity_rows <= 0) return 0;
  if (ff & 7) return fail(-1, "moe_act_rows: the width must be a multiple of 8");
  if (act == NFN_ACT_CLAMPED && !clamp) return fail(-1, "moe_act_rows: the clamped gate needs its limits");
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const __nv_bfloat16* gu = static_cast<const __nv_bfloat16*>(gate_up);
  __nv_bfloat16* out = static_cast<__nv_bfloat16*>(mid);
  moe_act_rows_kernel<<<dim3(capacity_rows, ceil_div(ff, 256 * 8)), 256, 0, st>>>(gu, row_w, plan, ff, act, clamp ? *clamp : nfn_gate_clamp{}, out);
  return launch_check("moe_act_rows");
}
