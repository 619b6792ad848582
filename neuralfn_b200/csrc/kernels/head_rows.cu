// Between a layer's input projection and its attention, for designs with rotary positions: per-head norm and rotation of queries and keys,
// the latent and shared key part of latent attention, cache append, the per-head products around a latent cache, and the gather of
// visible latents in front of a prompt's expansion.
//
// Angles are formed in fp32 from frequencies given as two parts (high, low): position * frequency is exact to the last bit of the sum, so a
// rotation at a far position is as good as one near the start. All arithmetic between loads and stores is fp32. Rotations may happen
// in place: every element is read and written by one thread.
#include <algorithm>

#include "common.h"
#include "paged.cuh"

namespace nfn {

constexpr int HR_THREADS = 256, HR_WARPS = HR_THREADS / 32, HR_ROWS = 16;

__device__ __forceinline__ float2 rotation(int pos, const float* freq, int i) {
  const float p = (float)pos, f = freq[2 * i], hi = p * f, lo = fmaf(p, f, -hi) + p * freq[2 * i + 1];
  float s, c;
  sincosf(hi, &s, &c);
  const float q = 1.f - 0.5f * lo * lo;
  return make_float2(c * q - s * lo, s * q + c * lo);
}

// cos and sin of every row and pair of the tile, [rows][half]
__device__ __forceinline__ void fill_rotations(float2* cs, const float* freq, int half, int pos0, int n) {
  for (int i = threadIdx.x; i < n * half; i += HR_THREADS) cs[i] = rotation(pos0 + i / half, freq, i % half);
}

// dimensions c .. c + 3 of a head: the pairs below rot_dims turn
__device__ __forceinline__ float4 rotate4(const float4& v, const float2* cs, int c, int rot_dims) {
  float4 o = v;
  if (c + 1 < rot_dims) {
    const float2 a = cs[c / 2];
    o.x = v.x * a.x - v.y * a.y;
    o.y = v.y * a.x + v.x * a.y;
  }
  if (c + 3 < rot_dims) {
    const float2 a = cs[c / 2 + 1];
    o.z = v.z * a.x - v.w * a.y;
    o.w = v.w * a.x + v.z * a.y;
  }
  return o;
}

// the same for dimensions c .. c + 7
__device__ __forceinline__ void rotate8(float (&v)[8], const float2* cs, int c, int rot_dims) {
#pragma unroll
  for (int e = 0; e < 8; e += 2)
    if (c + e + 1 < rot_dims) {
      const float2 a = cs[(c + e) / 2];
      const float x = v[e] * a.x - v[e + 1] * a.y;
      v[e + 1] = v[e + 1] * a.x + v[e] * a.y;
      v[e] = x;
    }
}

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}
__device__ __forceinline__ float squares(const float4& v) { return v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w; }

// A warp takes one query or key head for all rows of a tile, R rows in flight. NV: 128-wide pieces of a head.
template <typename T, int NV>
__global__ void __launch_bounds__(HR_THREADS)
head_rows_kernel(const nfn_head_rows_args p) {
  extern __shared__ float2 hr_cs[];
  constexpr int R = NV >= 4 ? 1 : 4 / NV;
  const nfn_row_tile t = p.tiles[blockIdx.x];
  if (t.slot < 0) return;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, half = p.rot_dims / 2;
  const int pos0 = t.e_pos0 + t.row0 - t.e_row0;
  const int item = blockIdx.y * HR_WARPS + warp;
  const bool key = item >= p.heads, on = item < p.heads + p.kv_heads;
  const int head = key ? item - p.heads : item;
  const T* in = static_cast<const T*>(p.in) + (size_t)t.row0 * p.ld_in;
  const T* src = in + (key ? p.off_k : 0) + head * p.dim_p;
  float4 v[R][NV];
  auto fetch = [&](int i0) {
#pragma unroll
    for (int i = 0; i < R; ++i)
#pragma unroll
      for (int j = 0; j < NV; ++j) {
        const int c = lane * 4 + j * 128;
        v[i][j] = on && i0 + i < t.n && c < p.dim_p ? load4(src + (size_t)(i0 + i) * p.ld_in + c) : make_float4(0.f, 0.f, 0.f, 0.f);
      }
  };
  fetch(0);                                               // on their way while the angles are formed
  fill_rotations(hr_cs, p.freq, half, pos0, t.n);
  __syncthreads();
  const size_t page = p.kv_heads > 0 ? (size_t)p.table[(size_t)t.slot * p.table_ld + pos0 / NFN_PAGE] : 0;
  const int in_page = pos0 % NFN_PAGE;
  if (on) {
    T* dst = key ? static_cast<T*>(p.k_pool) + ((page * p.kv_heads + head) * NFN_PAGE + in_page) * p.dim_p
                 : static_cast<T*>(p.q_out) + (size_t)t.row0 * p.ld_q + head * p.dim_p;
    const int ld_dst = key ? p.dim_p : p.ld_q;
    const __nv_bfloat16* weight = static_cast<const __nv_bfloat16*>(key ? p.k_norm : p.q_norm);
    float4 w[NV];
#pragma unroll
    for (int j = 0; j < NV; ++j) {
      const int c = lane * 4 + j * 128;
      w[j] = weight && c < p.dim_p ? load4(weight + c) : make_float4(1.f, 1.f, 1.f, 1.f);
    }
    for (int i0 = 0; i0 < t.n; i0 += R) {
      if (i0 > 0) fetch(i0);
#pragma unroll
      for (int i = 0; i < R; ++i) {
        if (i0 + i >= t.n) break;
        if (weight) {
          float ss = 0.f;
#pragma unroll
          for (int j = 0; j < NV; ++j) ss += squares(v[i][j]);
          const float r = 1.f / sqrtf(warp_sum(ss) / (float)p.dim + p.eps);
#pragma unroll
          for (int j = 0; j < NV; ++j) {
            v[i][j].x *= r * w[j].x; v[i][j].y *= r * w[j].y; v[i][j].z *= r * w[j].z; v[i][j].w *= r * w[j].w;
          }
        }
#pragma unroll
        for (int j = 0; j < NV; ++j) {
          const int c = lane * 4 + j * 128;
          if (c < p.dim_p) store4(dst + (size_t)(i0 + i) * ld_dst + c, rotate4(v[i][j], hr_cs + (i0 + i) * half, c, p.rot_dims));
        }
      }
    }
  }
  // values, channel-major: two neighbouring channels per thread
  const int n_v = p.kv_heads * p.vdim_p;
  struct alignas(2 * sizeof(T)) Pair { T a, b; };
  for (int ch = 2 * (blockIdx.y * HR_THREADS + threadIdx.x); ch < n_v; ch += 2 * gridDim.y * HR_THREADS) {
    const T* from = in + p.off_v + ch;
    T* dst = static_cast<T*>(p.v_pool) + (page * n_v + ch) * NFN_PAGE + in_page;
    if (t.n == HR_ROWS) {
      T buf[2][HR_ROWS];
#pragma unroll
      for (int i = 0; i < HR_ROWS; ++i) {
        const Pair f = *reinterpret_cast<const Pair*>(from + (size_t)i * p.ld_in);
        buf[0][i] = f.a;
        buf[1][i] = f.b;
      }
#pragma unroll
      for (int e = 0; e < 2; ++e)
#pragma unroll
        for (int q = 0; q < HR_ROWS * (int)sizeof(T) / 16; ++q) reinterpret_cast<uint4*>(dst + e * NFN_PAGE)[q] = pack16(&buf[e][q * (16 / sizeof(T))]);
    } else {
      for (int i = 0; i < t.n; ++i) {
        const Pair f = *reinterpret_cast<const Pair*>(from + (size_t)i * p.ld_in);
        dst[i] = f.a;
        dst[NFN_PAGE + i] = f.b;
      }
    }
  }
}

// A warp takes the rotated part of one query head over the tile's rows; the CTAs of the last column take latents and shared key parts, a row per warp.
template <typename T, int NV>
__global__ void __launch_bounds__(HR_THREADS)
latent_rows_kernel(const nfn_latent_rows_args p) {
  extern __shared__ float2 hr_cs[];
  const nfn_row_tile t = p.tiles[blockIdx.x];
  const bool of_keys = blockIdx.y == gridDim.y - 1;
  if (t.slot < 0 || (of_keys && !p.k_pool)) return;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, half = p.rot_dim / 2;
  const int pos0 = t.e_pos0 + t.row0 - t.e_row0;
  const int pitch = p.dim_p + p.rot_p, lp = p.rank_p + p.rot_p;
  const T* in = static_cast<const T*>(p.in) + (size_t)t.row0 * p.ld_in;
  if (!of_keys) {
    const int head = blockIdx.y * HR_WARPS + warp;
    const bool lat = t.row0 < p.q_row0, on = head < p.heads;    // rows of an entry are all short or all long
    const T* src = in + (on ? head : 0) * pitch;
    T* dst = lat ? static_cast<T*>(p.q_lat) + (size_t)t.row0 * p.heads * lp + (size_t)head * lp + p.rank_p
                 : static_cast<T*>(p.q_out) + (size_t)t.row0 * p.ld_q + head * pitch + p.dim_p;
    const size_t ld_dst = lat ? (size_t)p.heads * lp : (size_t)p.ld_q;
    // pieces of eight over the tile's rows, four per lane in flight: narrow rotated parts leave no lane idle
    const int pieces = p.rot_p / 8, total = on ? pieces * t.n : 0;
    float v[4][8];
    auto fetch = [&](int x0) {
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int x = x0 + 32 * e;
        if (x < total) load8(src + (size_t)(x / pieces) * p.ld_in + p.dim_p + x % pieces * 8, v[e]);
      }
    };
    fetch(lane);                                          // on their way while the angles are formed
    fill_rotations(hr_cs, p.freq, half, pos0, t.n);
    __syncthreads();
    for (int x0 = lane; x0 < total; x0 += 128) {
      if (x0 != lane) fetch(x0);
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int x = x0 + 32 * e, i = x / pieces, c = x % pieces * 8;
        if (x < total) {
          rotate8(v[e], hr_cs + i * half, c, p.rot_dim);
          store8(dst + i * ld_dst + c, v[e]);
        }
      }
    }
    if (on && !lat && p.q_out != p.in)
      for (int i = 0; i < t.n; ++i)
        for (int c = lane * 4; c < p.dim_p; c += 128) store4(dst + i * ld_dst - p.dim_p + c, load4(src + (size_t)i * p.ld_in + c));
    return;
  }
  fill_rotations(hr_cs, p.freq, half, pos0, t.n);
  __syncthreads();
  const size_t page = (size_t)p.table[(size_t)t.slot * p.table_ld + pos0 / NFN_PAGE];
  T* dst = static_cast<T*>(p.k_pool) + (page * NFN_PAGE + pos0 % NFN_PAGE) * lp;
  const T* src = in + p.off_kv;
  const __nv_bfloat16* weight = static_cast<const __nv_bfloat16*>(p.c_norm);
  for (int i = warp; i < t.n; i += HR_WARPS) {
    const T* row = src + (size_t)i * p.ld_in;
    float4 v[NV];
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < NV; ++j) {
      const int c = lane * 4 + j * 128;
      v[j] = c < p.rank_p ? load4(row + c) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
#pragma unroll
    for (int j = 0; j < NV; ++j) ss += squares(v[j]);
    for (int c = lane * 4 + NV * 128; c < p.rank_p; c += 128) ss += squares(load4(row + c));
    const float r = 1.f / sqrtf(warp_sum(ss) / (float)p.rank + p.eps);
    auto leave = [&](const float4& f, int c) {
      const float4 w = load4(weight + c);
      store4(dst + (size_t)i * lp + c, make_float4(f.x * r * w.x, f.y * r * w.y, f.z * r * w.z, f.w * r * w.w));
    };
#pragma unroll
    for (int j = 0; j < NV; ++j)
      if (lane * 4 + j * 128 < p.rank_p) leave(v[j], lane * 4 + j * 128);
    for (int c = lane * 4 + NV * 128; c < p.rank_p; c += 128) leave(load4(row + c), c);
    for (int c = lane * 4; c < p.rot_p; c += 128)
      store4(dst + (size_t)i * lp + p.rank_p + c, rotate4(load4(row + p.rank_p + c), hr_cs + i * half, c, p.rot_dim));
  }
}

// ------------------------------------------------------------------------------------------------ per-group products --
// 32-bit mode: a warp per weight row, eight rows at a time.
constexpr int GP_WARPS = 8, GP_ROWS = 8;

__global__ void __launch_bounds__(GP_WARPS * 32)
group_products_f32_kernel(const nfn_group_products_args p) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, n = blockIdx.x * GP_WARPS + warp, g = blockIdx.y, r0 = blockIdx.z * GP_ROWS;
  const bool tail = g == p.groups;
  if (n >= (tail ? p.tail_n : p.n)) return;
  const __nv_bfloat16* w = tail ? static_cast<const __nv_bfloat16*>(p.tail_w) + (size_t)n * p.k : static_cast<const __nv_bfloat16*>(p.w) + ((size_t)g * p.n + n) * p.k;
  const float* in = static_cast<const float*>(p.in) + (size_t)r0 * p.ld_in + (tail ? (size_t)p.tail_in : (size_t)g * p.in_group);
  const int live = min(GP_ROWS, p.rows - r0);
  float a[GP_ROWS];
#pragma unroll
  for (int i = 0; i < GP_ROWS; ++i) a[i] = 0.f;
  for (int k = lane * 4; k < p.k; k += 128) {
    const float4 f = load4(w + k);
#pragma unroll
    for (int i = 0; i < GP_ROWS; ++i) {
      if (i >= live) break;
      const float4 x = load4(in + (size_t)i * p.ld_in + k);
      a[i] += (f.x * x.x + f.y * x.y) + (f.z * x.z + f.w * x.w);
    }
  }
  float* out = tail ? p.tail_out + (size_t)r0 * p.ld_tail + n : static_cast<float*>(p.out) + (size_t)r0 * p.ld_out + (size_t)g * p.out_group + n;
#pragma unroll
  for (int i = 0; i < GP_ROWS; ++i) {
    if (i >= live) break;
    const float s = warp_sum(a[i]);
    if (lane != 0) continue;
    float f = 1.f;
    if (!tail && p.gate) f = sigmoid_exact(static_cast<const float*>(p.gate)[(size_t)(r0 + i) * p.ld_gate + (size_t)g * p.gate_group + n]);
    out[(size_t)i * (tail ? p.ld_tail : p.ld_out)] = tail ? s : ff_act(s, p.act) * f;
  }
}

// bf16, on the tensor cores: a CTA takes 32 weight rows of a group, its warps a quarter of the contraction each; rows are the eight columns of
// mma.m16n8k16. The order of a contraction is free, so every fragment is one 16-byte load per lane.
constexpr int GM_WARPS = 4;

__device__ __forceinline__ uint4 gm_stream(const __nv_bfloat16* p) {
  uint4 v;
  asm volatile("ld.global.nc.L1::no_allocate.v4.u32 {%0,%1,%2,%3}, [%4];" : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w) : "l"(p));
  return v;
}
__device__ __forceinline__ void gm_mma(float (&d)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
  asm("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
      : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
      : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}

template <int NT>
__global__ void __launch_bounds__(GM_WARPS * 32)
group_products_mma_kernel(const nfn_group_products_args p) {
  constexpr int M = 8 * NT, U = NT == 4 ? 1 : 2;          // rows at a time; 32-wide steps per set, two sets in flight
  __shared__ float part[GM_WARPS][32][M + 1];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gr = lane >> 2, j = lane & 3, g = blockIdx.y;
  const bool tail = g == p.groups;
  const int n0 = blockIdx.x * 32, r0 = blockIdx.z * M, N = tail ? p.tail_n : p.n;
  if (n0 >= N) return;
  const bool two = n0 + 16 < N;
  const __nv_bfloat16* w0 = (tail ? static_cast<const __nv_bfloat16*>(p.tail_w) : static_cast<const __nv_bfloat16*>(p.w) + (size_t)g * p.n * p.k) + (size_t)(n0 + gr) * p.k + 8 * j;
  const __nv_bfloat16* w1 = two ? w0 + (size_t)16 * p.k : w0;
  const uint4 zero4 = make_uint4(0u, 0u, 0u, 0u);
  const __nv_bfloat16* src[NT];
  bool on[NT];
#pragma unroll
  for (int t = 0; t < NT; ++t) {
    const int r = r0 + 8 * t + gr;
    on[t] = r < p.rows;
    src[t] = static_cast<const __nv_bfloat16*>(p.in) + (size_t)(on[t] ? r : r0) * p.ld_in + (tail ? (size_t)p.tail_in : (size_t)g * p.in_group) + 8 * j;
  }
  const int live = min(M, p.rows - r0);
  constexpr int GV = 32 * M / (GM_WARPS * 32);            // results of a thread, and their gates ahead of time
  float gate[GV];
#pragma unroll
  for (int i = 0; i < GV; ++i) {
    const int x = threadIdx.x + i * GM_WARPS * 32, col = x / 32, row = x % 32;
    gate[i] = 0.f;
    if (!tail && p.gate && col < live && n0 + row < N) gate[i] = __bfloat162float(static_cast<const __nv_bfloat16*>(p.gate)[(size_t)(r0 + col) * p.ld_gate + (size_t)g * p.gate_group + n0 + row]);
  }
  float acc[2][NT][4];
#pragma unroll
  for (int m = 0; m < 2; ++m)
#pragma unroll
    for (int t = 0; t < NT; ++t)
#pragma unroll
      for (int c = 0; c < 4; ++c) acc[m][t][c] = 0.f;
  const int steps = (p.k + 31) / 32, s0 = steps * warp / GM_WARPS, s1 = steps * (warp + 1) / GM_WARPS;
  uint4 a[2][U][4], b[2][U][NT];
  auto fetch = [&](int s, uint4 (&fa)[U][4], uint4 (&fb)[U][NT]) {
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int k = (s + u) * 32;
      const bool ok = s + u < s1 && k + 8 * j < p.k;
      fa[u][0] = ok ? gm_stream(w0 + k) : zero4;
      fa[u][1] = ok ? gm_stream(w0 + (size_t)8 * p.k + k) : zero4;
      fa[u][2] = ok ? gm_stream(w1 + k) : zero4;
      fa[u][3] = ok ? gm_stream(w1 + (size_t)8 * p.k + k) : zero4;
#pragma unroll
      for (int t = 0; t < NT; ++t) fb[u][t] = ok && on[t] ? *reinterpret_cast<const uint4*>(src[t] + k) : zero4;
    }
  };
  auto use = [&](const uint4 (&fa)[U][4], const uint4 (&fb)[U][NT]) {
#pragma unroll
    for (int u = 0; u < U; ++u)
#pragma unroll
      for (int t = 0; t < NT; ++t) {
        gm_mma(acc[0][t], fa[u][0].x, fa[u][1].x, fa[u][0].y, fa[u][1].y, fb[u][t].x, fb[u][t].y);
        gm_mma(acc[1][t], fa[u][2].x, fa[u][3].x, fa[u][2].y, fa[u][3].y, fb[u][t].x, fb[u][t].y);
        gm_mma(acc[0][t], fa[u][0].z, fa[u][1].z, fa[u][0].w, fa[u][1].w, fb[u][t].z, fb[u][t].w);
        gm_mma(acc[1][t], fa[u][2].z, fa[u][3].z, fa[u][2].w, fa[u][3].w, fb[u][t].z, fb[u][t].w);
      }
  };
  fetch(s0, a[0], b[0]);
  fetch(s0 + U, a[1], b[1]);
  for (int s = s0; s < s1; s += 2 * U) {
    use(a[0], b[0]);
    fetch(s + 2 * U, a[0], b[0]);
    use(a[1], b[1]);
    fetch(s + 3 * U, a[1], b[1]);
  }
#pragma unroll
  for (int m = 0; m < 2; ++m)
#pragma unroll
    for (int t = 0; t < NT; ++t)
#pragma unroll
      for (int c = 0; c < 4; ++c) part[warp][m * 16 + gr + (c >> 1) * 8][8 * t + 2 * j + (c & 1)] = acc[m][t][c];
  __syncthreads();
#pragma unroll
  for (int i = 0; i < GV; ++i) {
    const int x = threadIdx.x + i * GM_WARPS * 32, col = x / 32, row = x % 32;
    if (col >= live || n0 + row >= N) continue;
    float v = 0.f;
#pragma unroll
    for (int w = 0; w < GM_WARPS; ++w) v += part[w][row][col];
    if (tail) {
      p.tail_out[(size_t)(r0 + col) * p.ld_tail + n0 + row] = v;
      continue;
    }
    v = ff_act(v, p.act);
    if (p.gate) v *= sigmoid_for<__nv_bfloat16>(gate[i]);
    static_cast<__nv_bfloat16*>(p.out)[(size_t)(r0 + col) * p.ld_out + (size_t)g * p.out_group + n0 + row] = __float2bfloat16(v);
  }
}

// a quarter of a page per CTA: 16 rows of `vecs` 16-byte pieces
__global__ void __launch_bounds__(256)
latent_gather_kernel(const uint4* __restrict__ pool, int ld_pool, int vecs, const int* __restrict__ table, int table_ld, const nfn_latent_span* __restrict__ spans,
                     uint4* __restrict__ out) {
  const nfn_latent_span s = spans[blockIdx.y];
  const int page = blockIdx.x / 4, r0 = blockIdx.x % 4 * 16;
  if (s.slot < 0 || page >= s.n_pages) return;
  const uint4* src = pool + ((size_t)table[(size_t)s.slot * table_ld + s.first_page + page] * NFN_PAGE + r0) * ld_pool;
  uint4* dst = out + ((size_t)s.row0 + (size_t)page * NFN_PAGE + r0) * vecs;
#pragma unroll 4
  for (int i = threadIdx.x; i < 16 * vecs; i += 256) dst[i] = src[(size_t)(i / vecs) * ld_pool + i % vecs];
}

template <typename T>
static int launch_head_rows(const nfn_head_rows_args& a, cudaStream_t st) {
  const dim3 grid(a.n_tiles, ceil_div(a.heads + a.kv_heads, HR_WARPS));
  const size_t smem = (size_t)std::max(1, a.tile_rows * (a.rot_dims / 2)) * sizeof(float2);
  if (a.dim_p <= 128) head_rows_kernel<T, 1><<<grid, HR_THREADS, smem, st>>>(a);
  else if (a.dim_p <= 256) head_rows_kernel<T, 2><<<grid, HR_THREADS, smem, st>>>(a);
  else head_rows_kernel<T, 4><<<grid, HR_THREADS, smem, st>>>(a);
  return launch_check("head_rows");
}

template <typename T>
static int launch_latent_rows(const nfn_latent_rows_args& a, cudaStream_t st) {
  const dim3 grid(a.n_tiles, ceil_div(a.heads, HR_WARPS) + 1);
  const size_t smem = (size_t)std::max(1, a.tile_rows * (a.rot_dim / 2)) * sizeof(float2);
  latent_rows_kernel<T, 4><<<grid, HR_THREADS, smem, st>>>(a);
  return launch_check("latent_rows");
}

}  // namespace nfn

using namespace nfn;

extern "C" int nfn_head_rows(const nfn_head_rows_args* args, nfn_stream_t stream) {
  if (!args) return fail(-1, "head_rows: null args");
  const nfn_head_rows_args& a = *args;
  if (a.n_tiles <= 0) return 0;
  if ((a.ld_in | a.off_k | a.off_v | a.dim_p | a.vdim_p | a.ld_q) & 7) return fail(-1, "head_rows: widths and offsets must be multiples of 8");
  if (a.heads <= 0 || a.kv_heads < 0 || a.dim <= 0 || a.dim > a.dim_p || a.dim_p > 512) return fail(-1, "head_rows: heads of at most 512 dimensions");
  if ((a.rot_dims & 1) || a.rot_dims < 0 || a.rot_dims > a.dim || (a.rot_dims > 0 && !a.freq)) return fail(-1, "head_rows: an even number of rotated dimensions, with their frequencies");
  if (a.tile_rows < 1 || a.tile_rows > HR_ROWS) return fail(-1, "head_rows: tiles hold 1 to 16 rows");
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  return a.f32 ? launch_head_rows<float>(a, st) : launch_head_rows<__nv_bfloat16>(a, st);
}

extern "C" int nfn_latent_rows(const nfn_latent_rows_args* args, nfn_stream_t stream) {
  if (!args) return fail(-1, "latent_rows: null args");
  const nfn_latent_rows_args& a = *args;
  if (a.n_tiles <= 0) return 0;
  if ((a.ld_in | a.off_kv | a.dim_p | a.rot_p | a.rank_p | a.ld_q) & 7) return fail(-1, "latent_rows: widths and offsets must be multiples of 8");
  if ((a.rot_dim & 1) || a.rot_dim <= 0 || a.rot_dim > a.rot_p || !a.freq) return fail(-1, "latent_rows: an even number of rotated dimensions, with their frequencies");
  if (a.k_pool && (!a.c_norm || a.rank <= 0 || a.rank > a.rank_p)) return fail(-1, "latent_rows: the latent needs its norm");
  if (a.q_row0 > 0 && !a.q_lat) return fail(-1, "latent_rows: short rows need their query buffer");
  if (a.tile_rows < 1 || a.tile_rows > HR_ROWS || (size_t)a.tile_rows * (a.rot_dim / 2) * sizeof(float2) > 48 * 1024) return fail(-1, "latent_rows: tiles hold 1 to 16 rows of at most 768 rotated dimensions");
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  return a.f32 ? launch_latent_rows<float>(a, st) : launch_latent_rows<__nv_bfloat16>(a, st);
}

extern "C" int nfn_group_products(const nfn_group_products_args* args, nfn_stream_t stream) {
  if (!args) return fail(-1, "group_products: null args");
  const nfn_group_products_args& a = *args;
  if (a.rows <= 0) return 0;
  if (a.groups <= 0 || a.groups > 65535 || ((a.n | a.k) & 15) || a.n <= 0 || a.k <= 0 || ((a.ld_in | a.in_group) & 7)) return fail(-1, "group_products: sizes must be multiples of 16");
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (ceil_div(a.rows, 8) > 65535) return fail(-1, "group_products: too many rows in one launch");
  if (a.tail_n < 0 || (a.tail_n > 0 && (!a.tail_w || !a.tail_out || (a.tail_in & 7)))) return fail(-1, "group_products: the tail product lacks an operand");
  const int n = std::max(a.n, a.tail_n), g = a.groups + (a.tail_n > 0 ? 1 : 0);
  if (a.f32) group_products_f32_kernel<<<dim3(ceil_div(n, GP_WARPS), g, ceil_div(a.rows, GP_ROWS)), GP_WARPS * 32, 0, st>>>(a);
  else if (a.rows <= 8) group_products_mma_kernel<1><<<dim3(ceil_div(n, 32), g, 1), GM_WARPS * 32, 0, st>>>(a);
  else if (a.rows <= 16) group_products_mma_kernel<2><<<dim3(ceil_div(n, 32), g, 1), GM_WARPS * 32, 0, st>>>(a);
  else group_products_mma_kernel<4><<<dim3(ceil_div(n, 32), g, ceil_div(a.rows, 32)), GM_WARPS * 32, 0, st>>>(a);
  return launch_check("group_products");
}

extern "C" int nfn_latent_gather(int f32, const void* pool, int ld_pool, int cols, const int* table, int table_ld, const nfn_latent_span* spans, int n_spans,
                                 int max_pages, void* out, nfn_stream_t stream) {
  if (n_spans <= 0 || max_pages <= 0) return 0;
  const int per = f32 ? 4 : 8;
  if (ld_pool % per || cols % per || n_spans > 65535) return fail(-1, "latent_gather: rows of 16-byte pieces, at most 65535 spans");
  latent_gather_kernel<<<dim3(4 * max_pages, n_spans), 256, 0, static_cast<cudaStream_t>(stream)>>>(static_cast<const uint4*>(pool), ld_pool / per, cols / per, table, table_ld,
                                                                                                 spans, static_cast<uint4*>(out));
  return launch_check("latent_gather");
}
