// Row-wise kernels of the layer-list engine: embedding / residual / norm rows, the step between a layer's input projection and
// its attention (short convolutions with their per-sequence history, query temperature, cache append, feed-forward gate), the
// per-layer token input's gate, a 32-bit matrix product, and the plain paged attention (any size, bf16 or fp32) that the
// tensor-core kernels of paged_decode.cu / paged_prefill.cu are checked against and fall back to.
//
// The kernels work on the rows of a step: consecutive tokens of several sequences, described by small device arrays, so prompt
// portions and single tokens of different sequences share every launch.
#include "common.h"
#include "paged.cuh"

namespace nfn {

// ------------------------------------------------------------------------------------------------ rows --
// One CTA per row; the row waits in shared memory between the passes.
constexpr int ROW_THREADS = 256;

__device__ __forceinline__ float block_sum(float v, float* red) {
#pragma unroll
  for (int s = 16; s > 0; s >>= 1) v += __shfl_xor_sync(0xffffffffu, v, s);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float t = 0.f;
#pragma unroll
  for (int i = 0; i < ROW_THREADS / 32; ++i) t += red[i];
  __syncthreads();
  return t;
}

template <typename T>
__global__ void __launch_bounds__(ROW_THREADS)
row_norm_kernel(const nfn_row_norm_args p) {
  extern __shared__ float row_smem[];   // [ld] base, then [ld] y
  __shared__ float red[ROW_THREADS / 32];
  float* base = row_smem;
  float* yrow = row_smem + p.ld;
  const int r = blockIdx.x;
  const int vecs = p.ld / 4;
  const float inv_w = 1.f / (float)p.width;
  const __nv_bfloat16* emb = nullptr;
  const float* x = nullptr;
  if (p.tokens) {
    const int t = min(max(p.tokens[r], 0), p.vocab - 1);
    emb = static_cast<const __nv_bfloat16*>(p.embed) + (size_t)t * p.ld;
  } else {
    x = p.x + (size_t)(p.src_rows ? p.src_rows[r] : r) * p.ld;
  }
  float ry = 0.f;
  if (p.y) {
    float ss = 0.f;
    const T* y = static_cast<const T*>(p.y) + (size_t)r * p.ld;
    for (int v = threadIdx.x; v < vecs; v += ROW_THREADS) {
      const float4 f = load4(y + 4 * v);
      if (x) reinterpret_cast<float4*>(base)[v] = load4(x + 4 * v);      // both rows are on their way together
      reinterpret_cast<float4*>(yrow)[v] = f;
      ss += f.x * f.x + f.y * f.y + f.z * f.z + f.w * f.w;
    }
    ry = 1.f / sqrtf(block_sum(ss, red) * inv_w + p.eps);
  }
  float ss = 0.f;
  for (int v = threadIdx.x; v < vecs; v += ROW_THREADS) {
    float4 b;
    if (emb) {
      b = load4(emb + 4 * v);
      b.x *= p.embed_scale; b.y *= p.embed_scale; b.z *= p.embed_scale; b.w *= p.embed_scale;
    } else {
      b = p.y ? reinterpret_cast<const float4*>(base)[v] : load4(x + 4 * v);
    }
    if (p.y) {
      const float4 f = reinterpret_cast<const float4*>(yrow)[v];
      const float4 w = load4(static_cast<const __nv_bfloat16*>(p.y_weight) + 4 * v);
      b.x += f.x * ry * w.x; b.y += f.y * ry * w.y; b.z += f.z * ry * w.z; b.w += f.w * ry * w.w;
    }
    if (p.x_out) reinterpret_cast<float4*>(p.x_out + (size_t)r * p.ld)[v] = b;
    reinterpret_cast<float4*>(base)[v] = b;
    ss += b.x * b.x + b.y * b.y + b.z * b.z + b.w * b.w;
  }
  if (!p.h) return;
  const float rx = 1.f / sqrtf(block_sum(ss, red) * inv_w + p.eps);
  T* h = static_cast<T*>(p.h) + (size_t)r * p.ld;
  for (int v = threadIdx.x; v < vecs; v += ROW_THREADS) {
    const float4 b = reinterpret_cast<const float4*>(base)[v];
    const float4 w = load4(static_cast<const __nv_bfloat16*>(p.weight) + 4 * v);
    store4(h + 4 * v, make_float4(b.x * rx * w.x, b.y * rx * w.y, b.z * rx * w.z, b.w * rx * w.w));
  }
}

// ----------------------------------------------------------------------------- after the input projection --
constexpr int MIX_THREADS = 128, MIX_ROWS = 16;

// Projected value row `back` positions before row index ti of the entry: this step's rows, the stored history, or zero before
// the sequence's start.
template <typename T>
__device__ __forceinline__ bool mix_source(const nfn_mix_args& p, const nfn_row_tile& t, int idx, int col, float (&v)[8]) {
  if (idx >= 0) {
    load8(static_cast<const T*>(p.in) + (size_t)(t.e_row0 + idx) * p.ld_in + col, v);
    return true;
  }
  if (t.e_pos0 + idx < 0) return false;
  const int C = p.nq + p.nk + p.nv, hist = p.taps - 1;
  load8(static_cast<const T*>(p.state) + (size_t)t.parity * p.state_half + ((size_t)t.slot * hist + hist + idx) * C + col, v);
  return true;
}

// Convolved values of up to N consecutive rows of a tile, starting at row index ti of the entry. TAPS > 0: the window slides through
// registers, so every projected row is read once; TAPS = 0: any number of taps, rows are read again (they stay in L1).
template <typename T, int TAPS, int N>
struct MixWindow {
  float hist[TAPS > 1 ? TAPS - 1 : 1][8], w[TAPS > 0 ? TAPS : 1][8];
  __device__ __forceinline__ void start(const nfn_mix_args& p, const nfn_row_tile& t, int ti, int col) {
    if constexpr (TAPS > 0) {
      const int C = p.nq + p.nk + p.nv;
#pragma unroll
      for (int j = 0; j < TAPS; ++j) load8(static_cast<const __nv_bfloat16*>(p.conv) + (size_t)j * C + col, w[j]);
#pragma unroll
      for (int j = 0; j < TAPS - 1; ++j)
        if (!mix_source<T>(p, t, ti - (TAPS - 1) + j, col, hist[j]))
          for (float& f : hist[j]) f = 0.f;
    }
  }
  // rows [ti, ti + n), n <= N; rows past n are left undefined
  __device__ __forceinline__ void next(const nfn_mix_args& p, const nfn_row_tile& t, int ti, int n, int col, float (&out)[N][8]) {
    if (TAPS == 0 && p.conv) {
      const int C = p.nq + p.nk + p.nv;
#pragma unroll
      for (int i = 0; i < N; ++i) {
#pragma unroll
        for (int e = 0; e < 8; ++e) out[i][e] = 0.f;
        if (i < n)
          for (int j = 0; j < p.taps; ++j) {
            float u[8], wj[8];
            if (!mix_source<T>(p, t, ti + i - (p.taps - 1) + j, col, u)) continue;
            load8(static_cast<const __nv_bfloat16*>(p.conv) + (size_t)j * C + col, wj);
#pragma unroll
            for (int e = 0; e < 8; ++e) out[i][e] += wj[e] * u[e];
          }
      }
      return;
    }
    const T* in = static_cast<const T*>(p.in) + (size_t)(t.e_row0 + ti) * p.ld_in + col;
#pragma unroll
    for (int i = 0; i < N; ++i)
      if (i < n) load8(in + (size_t)i * p.ld_in, out[i]);
    if constexpr (TAPS > 0) {
#pragma unroll
      for (int i = 0; i < N; ++i)
        if (i < n) {
#pragma unroll
          for (int e = 0; e < 8; ++e) {
            const float u = out[i][e];
            float acc = w[TAPS - 1][e] * u;
#pragma unroll
            for (int j = 0; j < TAPS - 1; ++j) acc += w[j][e] * hist[j][e];
#pragma unroll
            for (int j = 0; j + 1 < TAPS - 1; ++j) hist[j][e] = hist[j + 1][e];
            if constexpr (TAPS > 1) hist[TAPS - 2][e] = u;
            out[i][e] = acc;
          }
        }
    }
  }
};

template <typename T, int TAPS>
__global__ void __launch_bounds__(MIX_THREADS, 4)
mix_rows_kernel(const nfn_mix_args p) {
  constexpr int N = 4;                                     // rows in flight per thread
  const nfn_row_tile t = p.tiles[blockIdx.y];
  if (t.slot < 0) return;
  const int C = p.nq + p.nk + p.nv;
  const int vec = blockIdx.x * MIX_THREADS + threadIdx.x;
  const int ti0 = t.row0 - t.e_row0;                       // first row's index inside the entry
  if (vec * 8 >= C) {
    // feed-forward columns of single-row tiles: ff_out = act(gate) * up (larger calls: ff_rows_kernel)
    const int c = vec * 8 - C;
    if (p.tile_rows != 1 || c >= p.ff) return;
    const T* in = static_cast<const T*>(p.in) + (size_t)t.row0 * p.ld_in;
    T* out = static_cast<T*>(p.ff_out) + (size_t)t.row0 * p.ld_ff + c;
    float g[8], u[8];
    load8(in + p.off_gate + c, g);
    load8(in + p.off_up + c, u);
#pragma unroll
    for (int e = 0; e < 8; ++e) g[e] = ff_act(g[e], p.act) * u[e];
    store8(out, g);
    return;
  }
  const int col = vec * 8, taps = p.taps;
  // the history the entry leaves behind: its newest taps - 1 projected rows (older ones move up when it brought fewer). The
  // register window holds exactly these rows after the tile's last row; otherwise they are gathered.
  const bool last = taps > 1 && t.row0 + t.n == t.e_row0 + t.e_n;
  T* st = static_cast<T*>(p.state) + (size_t)(1 - t.parity) * p.state_half + (size_t)t.slot * (taps - 1) * C + col;
  if (TAPS == 0 && last) {
    for (int i = 0; i < taps - 1; ++i) {
      float v[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
      mix_source<T>(p, t, t.e_n - (taps - 1) + i, col, v);
      store8(st + (size_t)i * C, v);
    }
  }
  MixWindow<T, TAPS, N> win;
  win.start(p, t, ti0, col);
  auto leave = [&]() {
    if constexpr (TAPS > 1) {
      if (last) {
#pragma unroll
        for (int i = 0; i < TAPS - 1; ++i) store8(st + (size_t)i * C, win.hist[i]);
      }
    }
  };
  float v[N][8];
  if (col < p.nq) {
    T* out = static_cast<T*>(p.q_out) + (size_t)t.row0 * p.ld_q + col;
    for (int i0 = 0; i0 < t.n; i0 += N) {
      win.next(p, t, ti0 + i0, t.n - i0, col, v);
#pragma unroll
      for (int i = 0; i < N; ++i)
        if (i0 + i < t.n) {
          if (p.conv_act == NFN_ACT_SILU) {
#pragma unroll
            for (int e = 0; e < 8; ++e) v[i][e] *= sigmoid_for<T>(v[i][e]);
          }
          if (p.temp_every > 0) {
            const int pos = t.e_pos0 + ti0 + i0 + i;
            const float f = 1.f + p.temp_coef * logf((float)((pos + 1) / p.temp_every + 1));
#pragma unroll
            for (int e = 0; e < 8; ++e) v[i][e] *= f;
          }
          store8(out + (size_t)(i0 + i) * p.ld_q, v[i]);
        }
    }
    leave();
    return;
  }
  // keys and values: the tile lies inside one page
  const int pos0 = t.e_pos0 + ti0;
  const size_t page = (size_t)p.table[(size_t)t.slot * p.table_ld + pos0 / NFN_PAGE];
  const int in_page = pos0 % NFN_PAGE;
  if (col < p.nq + p.nk) {
    const int c = col - p.nq, head = c / p.dim_p, d = c % p.dim_p;
    T* out = static_cast<T*>(p.k_pool) + ((page * p.kv_heads + head) * NFN_PAGE + in_page) * p.dim_p + d;
    for (int i0 = 0; i0 < t.n; i0 += N) {
      win.next(p, t, ti0 + i0, t.n - i0, col, v);
#pragma unroll
      for (int i = 0; i < N; ++i)
        if (i0 + i < t.n) store8(out + (size_t)(i0 + i) * p.dim_p, v[i]);
    }
    leave();
    return;
  }
  const int c = col - p.nq - p.nk, head = c / p.vdim_p, d = c % p.vdim_p;
  T* out = static_cast<T*>(p.v_pool) + ((page * p.kv_heads + head) * p.vdim_p + d) * NFN_PAGE + in_page;   // [vdim_p][64]
  if (t.n == MIX_ROWS) {
    // whole tile: eight consecutive tokens of every channel at a time, in 16-byte stores
#pragma unroll 1
    for (int i0 = 0; i0 < MIX_ROWS; i0 += 8) {
      T buf[8][8];
#pragma unroll
      for (int q = 0; q < 2; ++q) {
        win.next(p, t, ti0 + i0 + q * N, N, col, v);
#pragma unroll
        for (int i = 0; i < N; ++i)
#pragma unroll
          for (int e = 0; e < 8; ++e) buf[e][q * N + i] = from_float<T>(v[i][e]);
      }
#pragma unroll
      for (int e = 0; e < 8; ++e)
#pragma unroll
        for (int q = 0; q < (int)(sizeof(T) / 2); ++q)
          reinterpret_cast<uint4*>(out + (size_t)e * NFN_PAGE + i0)[q] = pack16(&buf[e][q * (16 / sizeof(T))]);
    }
    leave();
    return;
  }
  for (int i0 = 0; i0 < t.n; i0 += N) {
    win.next(p, t, ti0 + i0, t.n - i0, col, v);
#pragma unroll
    for (int i = 0; i < N; ++i)
      if (i0 + i < t.n)
#pragma unroll
        for (int e = 0; e < 8; ++e) out[(size_t)e * NFN_PAGE + i0 + i] = from_float<T>(v[i][e]);
  }
  leave();
}

// out = act(gate) * up over all rows of a call: two rows per thread, few registers. off_up < 0: out = act(gate)
template <typename T>
__global__ void __launch_bounds__(256)
ff_rows_kernel(const T* __restrict__ src, int ld_in, int off_gate, int off_up, int ff, int act, nfn_gate_clamp clamp, T* __restrict__ dst, int ld_out, int rows) {
  const int c = (blockIdx.x * 256 + threadIdx.x) * 8, r0 = blockIdx.y * 2;
  if (c >= ff) return;
  const T* in = src + (size_t)r0 * ld_in + c;
  T* out = dst + (size_t)r0 * ld_out + c;
  const bool two = r0 + 1 < rows, up = off_up >= 0;
  float g[2][8], u[2][8];
#pragma unroll
  for (int i = 0; i < 2; ++i)
    if (i == 0 || two) {
      load8(in + (size_t)i * ld_in + off_gate, g[i]);
      if (up) load8(in + (size_t)i * ld_in + off_up, u[i]);
    }
#pragma unroll
  for (int i = 0; i < 2; ++i)
    if (i == 0 || two) {
#pragma unroll
      for (int e = 0; e < 8; ++e) g[i][e] = up ? ff_gated<T>(g[i][e], u[i][e], act, clamp) : ff_act(g[i][e], act);
      store8(out + (size_t)i * ld_out, g[i]);
    }
}

template <typename T>
static void launch_ff_rows(const void* in, int ld_in, int off_gate, int off_up, int ff, int act, const nfn_gate_clamp& clamp, void* out, int ld_out, int rows, cudaStream_t st) {
  ff_rows_kernel<T><<<dim3(ceil_div(ff, 256 * 8), ceil_div(rows, 2)), 256, 0, st>>>(static_cast<const T*>(in), ld_in, off_gate, off_up, ff, act, clamp, static_cast<T*>(out),
                                                                                    ld_out, rows);
}

template <typename T>
static void launch_mix_rows(const nfn_mix_args& a, const dim3& grid, cudaStream_t st) {
  switch (a.taps) {
    case 2: mix_rows_kernel<T, 2><<<grid, MIX_THREADS, 0, st>>>(a); break;
    case 3: mix_rows_kernel<T, 3><<<grid, MIX_THREADS, 0, st>>>(a); break;
    case 4: mix_rows_kernel<T, 4><<<grid, MIX_THREADS, 0, st>>>(a); break;
    default: mix_rows_kernel<T, 0><<<grid, MIX_THREADS, 0, st>>>(a); break;
  }
}

// --------------------------------------------------------------------------------- plain paged attention --
// One warp per (row, query head): 32 keys at a time, one per lane, running maximum and sum, the value sum over channels held
// lane-wise. Any size; 32-bit throughout. The yardstick of the tensor-core kernels and the only path in 32-bit mode.
constexpr int PLAIN_WARPS = 4, PLAIN_MAX_VEC = 16;   // 32 * 16 value channels of a head per CTA

template <typename T>
__global__ void __launch_bounds__(PLAIN_WARPS * 32)
paged_attention_plain_kernel(const nfn_paged_attention_args p) {
  extern __shared__ float plain_smem[];                 // [PLAIN_WARPS][dim_p] queries, [PLAIN_WARPS][32] weights
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int row = p.row0 + blockIdx.x;
  const int h = blockIdx.y * PLAIN_WARPS + warp;
  if (h >= p.heads) return;
  const int slot = p.row_slot[row];
  if (slot < 0) return;
  const int pos = p.row_pos[row];
  const int hk = h / (p.heads / p.kv_heads);
  float* q = plain_smem + warp * p.dim_p;
  float* wgt = plain_smem + PLAIN_WARPS * p.dim_p + warp * 32;
  for (int d = lane; d < p.dim_p; d += 32) q[d] = to_float(static_cast<const T*>(p.q)[(size_t)row * p.ld_q + h * p.dim_p + d]);
  __syncwarp();
  const float slope = p.slopes ? p.slopes[h] : 0.f;
  const int lo = first_visible(p, pos);
  const int keep = min(p.keep_first, pos + 1);
  const int* table = p.table + (size_t)slot * p.table_ld;
  const int v0 = blockIdx.z * 32 * PLAIN_MAX_VEC, v_n = min(p.vdim_p - v0, 32 * PLAIN_MAX_VEC);      // this CTA's value channels
  const int nvec = (v_n + 31) / 32;
  float acc[PLAIN_MAX_VEC];
#pragma unroll
  for (int i = 0; i < PLAIN_MAX_VEC; ++i) acc[i] = 0.f;
  float m = has_sink(p) ? sink_score(p, h) : -INFINITY, l = has_sink(p) ? 1.f : 0.f;      // the sink is an element seen before all others
  for (int base = keep > 0 ? 0 : lo / 32 * 32; base <= pos; base += 32) {   // a chunk never crosses a page
    if (base >= keep && base + 32 <= lo) base = lo / 32 * 32;      // from the kept tokens to the window
    const size_t tile = (size_t)table[base / NFN_PAGE] * p.kv_heads + hk;
    const int in_page = base % NFN_PAGE, j = base + lane;
    float s = -INFINITY;
    if ((j >= lo || j < keep) && j <= pos) {
      const T* k = static_cast<const T*>(p.k_pool) + (tile * NFN_PAGE + in_page + lane) * p.dim_p;
      float d0 = 0.f, d1 = 0.f, d2 = 0.f, d3 = 0.f;
      for (int d = 0; d < p.dim_p; d += 4) {
        const float4 kv = load4(k + d);
        d0 += kv.x * q[d]; d1 += kv.y * q[d + 1]; d2 += kv.z * q[d + 2]; d3 += kv.w * q[d + 3];
      }
      s = ((d0 + d1) + (d2 + d3)) * p.scale;
      if (p.softcap > 0.f) s = p.softcap * tanhf(s / p.softcap);
      s -= slope * (float)(pos - j);
    }
    float mx = s;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
    const float m_new = fmaxf(m, mx);                    // the chunk holds a visible key, so this is finite
    const float alpha = m == -INFINITY ? 0.f : expf(m - m_new);
    const float e = s == -INFINITY ? 0.f : expf(s - m_new);
    float sum = e;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
    l = l * alpha + sum;
    m = m_new;
    wgt[lane] = e;
    __syncwarp();
    if (!p.v_pool) {                                     // values are the keys' first channels
      const int live = min(32, pos - base + 1);
      const T* v = static_cast<const T*>(p.k_pool) + (tile * NFN_PAGE + in_page) * p.dim_p + v0;
#pragma unroll
      for (int i = 0; i < PLAIN_MAX_VEC; ++i) {
        if (i >= nvec) break;
        const int c = lane + 32 * i;
        if (c < v_n) {
          float t = 0.f;
          for (int k = 0; k < live; ++k) t += to_float(v[(size_t)k * p.dim_p + c]) * wgt[k];
          acc[i] = acc[i] * alpha + t;
        }
      }
      __syncwarp();
      continue;
    }
    const T* v = static_cast<const T*>(p.v_pool) + (tile * p.vdim_p + v0) * NFN_PAGE + in_page;
#pragma unroll
    for (int i = 0; i < PLAIN_MAX_VEC; ++i) {
      if (i >= nvec) break;
      const int c = lane + 32 * i;
      if (c < v_n) {
        const T* vc = v + (size_t)c * NFN_PAGE;
        float t = 0.f;
        for (int k = 0; k < 32; k += 4) {
          const float4 f = load4(vc + k);
          t += f.x * wgt[k] + f.y * wgt[k + 1] + f.z * wgt[k + 2] + f.w * wgt[k + 3];
        }
        acc[i] = acc[i] * alpha + t;
      }
    }
    __syncwarp();
  }
  const float inv = l > 0.f ? 1.f / l : 0.f;
#pragma unroll
  for (int i = 0; i < PLAIN_MAX_VEC; ++i) {
    if (i >= nvec) break;
    const int c = lane + 32 * i;
    if (c < v_n) {
      float o = acc[i] * inv;
      if (p.gate) o *= sigmoid_exact(to_float(static_cast<const T*>(p.gate)[(size_t)row * p.ld_gate + h * p.vdim_p + v0 + c]));
      static_cast<T*>(p.out)[(size_t)row * p.ld_o + h * p.vdim_p + v0 + c] = from_float<T>(o);
    }
  }
}

int paged_attention_plain(const nfn_paged_attention_args& a, cudaStream_t st) {
  const size_t smem = (size_t)PLAIN_WARPS * (a.dim_p + 32) * sizeof(float);
  if (smem > 48 * 1024) return fail(-1, "paged attention: query head too wide");
  const dim3 grid(a.rows, ceil_div(a.heads, PLAIN_WARPS), ceil_div(a.vdim_p, 32 * PLAIN_MAX_VEC));
  if (a.f32) paged_attention_plain_kernel<float><<<grid, PLAIN_WARPS * 32, smem, st>>>(a);
  else paged_attention_plain_kernel<__nv_bfloat16><<<grid, PLAIN_WARPS * 32, smem, st>>>(a);
  return launch_check("paged_attention_plain");
}

// ------------------------------------------------------------------------------------- token input's gate --
template <typename T>
__global__ void side_mul_kernel(const float* gate, const int* tokens, const __nv_bfloat16* embed, long long ld_embed, int col0, int vocab,
                                T* out, int ld, int rows, int width) {
  const int vecs = width / 8;
  const int i = blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= rows * vecs) return;
  const int r = i / vecs, c = (i % vecs) * 8;
  float g[8], e[8];
  load8(gate + (size_t)r * ld + c, g);
  load8(embed + (size_t)min(max(tokens[r], 0), vocab - 1) * ld_embed + col0 + c, e);
#pragma unroll
  for (int k = 0; k < 8; ++k) g[k] = gelu_tanh_exact(g[k]) * e[k];
  store8(out + (size_t)r * ld + c, g);
}

// ---------------------------------------------------------------------------------- 32-bit matrix product --
// 64 x 64 tile, 16-deep slices, 4 x 4 outputs per thread; fp32 FMA only. Weights are read as the bf16 values they are stored as.
constexpr int SG_BM = 64, SG_BN = 64, SG_BK = 16;

__global__ void __launch_bounds__(256)
gemm_f32_kernel(const float* __restrict__ a, int lda, const __nv_bfloat16* __restrict__ b, int ldb, float* c, int ldc, int m, int n, int k,
                int accumulate, const __nv_bfloat16* __restrict__ bias) {
  __shared__ float sa[SG_BK][SG_BM + 4], sb[SG_BK][SG_BN + 4];
  const int m0 = blockIdx.y * SG_BM, n0 = blockIdx.x * SG_BN;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  const int lr = threadIdx.x >> 2, lk = (threadIdx.x & 3) * 4;     // this thread loads row lr, k values lk .. lk + 3 of both tiles
  float acc[4][4] = {};
  for (int k0 = 0; k0 < k; k0 += SG_BK) {
    float4 va = make_float4(0.f, 0.f, 0.f, 0.f), vb = va;
    if (k0 + lk < k) {
      if (m0 + lr < m) va = load4(a + (size_t)(m0 + lr) * lda + k0 + lk);
      if (n0 + lr < n) vb = load4(b + (size_t)(n0 + lr) * ldb + k0 + lk);
    }
    sa[lk][lr] = va.x; sa[lk + 1][lr] = va.y; sa[lk + 2][lr] = va.z; sa[lk + 3][lr] = va.w;
    sb[lk][lr] = vb.x; sb[lk + 1][lr] = vb.y; sb[lk + 2][lr] = vb.z; sb[lk + 3][lr] = vb.w;
    __syncthreads();
#pragma unroll
    for (int kk = 0; kk < SG_BK; ++kk) {
      const float4 x = *reinterpret_cast<const float4*>(&sa[kk][ty * 4]), y = *reinterpret_cast<const float4*>(&sb[kk][tx * 4]);
      const float xs[4] = {x.x, x.y, x.z, x.w}, ys[4] = {y.x, y.y, y.z, y.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] += xs[i] * ys[j];
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int r = m0 + ty * 4 + i;
    if (r >= m) continue;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int col = n0 + tx * 4 + j;
      if (col < n) {
        float* cp = c + (size_t)r * ldc + col;
        const float v = acc[i][j] + (bias ? __bfloat162float(bias[col]) : 0.f);
        *cp = accumulate ? *cp + v : v;
      }
    }
  }
}

__global__ void logit_cap_kernel(float* logits, int ld, int rows, int vecs, float scale, float cap) {
  const int i = blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= rows * vecs) return;
  float* p = logits + (size_t)(i / vecs) * ld + (i % vecs) * 4;
  const float4 f = load4(p);
  float v[4] = {f.x, f.y, f.z, f.w};
#pragma unroll
  for (float& x : v) x = cap > 0.f ? cap * tanhf(x * scale / cap) : x * scale;
  store4(p, make_float4(v[0], v[1], v[2], v[3]));
}

}  // namespace nfn

using namespace nfn;

extern "C" int nfn_logit_cap(float* logits, int ld, int rows, int cols, float scale, float cap, nfn_stream_t stream) {
  if (rows <= 0) return 0;
  if ((ld | cols) & 3) return fail(-1, "logit_cap: widths must be multiples of 4");
  const int vecs = cols / 4;
  if ((long long)rows * vecs > 0x7fffff00LL) return fail(-1, "logit_cap: too many values for one launch");
  logit_cap_kernel<<<ceil_div(rows * vecs, 256), 256, 0, static_cast<cudaStream_t>(stream)>>>(logits, ld, rows, vecs, scale, cap);
  return launch_check("logit_cap");
}

extern "C" int nfn_row_norm(const nfn_row_norm_args* args, nfn_stream_t stream) {
  if (!args) return fail(-1, "row_norm: null args");
  const nfn_row_norm_args& a = *args;
  if (a.rows <= 0) return 0;
  if ((a.ld & 15) || a.width <= 0 || a.width > a.ld) return fail(-1, "row_norm: the row pitch must be a multiple of 16 that holds the width");
  if (!a.tokens && !a.x) return fail(-1, "row_norm: neither tokens nor rows");
  const size_t smem = (size_t)a.ld * sizeof(float) * (a.y ? 2 : 1);
  if (smem > 200 * 1024) return fail(-1, "row_norm: rows too wide");
  auto kern = a.f32 ? row_norm_kernel<float> : row_norm_kernel<__nv_bfloat16>;
  static bool raised[64][2] = {};
  int dev = 0;
  cudaGetDevice(&dev);
  if (smem > 48 * 1024 && !raised[dev & 63][a.f32 ? 1 : 0]) {
    if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024) != cudaSuccess) return launch_check("row_norm attr", 0);
    raised[dev & 63][a.f32 ? 1 : 0] = true;
  }
  kern<<<a.rows, ROW_THREADS, smem, static_cast<cudaStream_t>(stream)>>>(a);
  return launch_check("row_norm");
}

extern "C" int nfn_mix_rows(const nfn_mix_args* args, nfn_stream_t stream) {
  if (!args) return fail(-1, "mix_rows: null args");
  const nfn_mix_args& a = *args;
  if (a.n_tiles <= 0) return 0;
  if ((a.nq | a.nk | a.nv | a.ff | a.ld_in | a.ld_q | a.ld_ff | a.off_gate | a.off_up | a.dim_p | a.vdim_p) & 7)
    return fail(-1, "mix_rows: widths and offsets must be multiples of 8");
  if (a.conv_act != NFN_ACT_NONE && (a.conv_act != NFN_ACT_SILU || a.nk || a.nv)) return fail(-1, "mix_rows: the activation (SiLU) goes with rows that stay out of the cache");
  if ((a.taps > 0) != (a.conv != nullptr) || (a.taps > 1 && !a.state)) return fail(-1, "mix_rows: a convolution needs its weights and history");
  if (a.n_tiles > 65535) return fail(-1, "mix_rows: too many row tiles in one launch");
  if (a.tile_rows < 1 || a.tile_rows > MIX_ROWS) return fail(-1, "mix_rows: tiles hold 1 to 16 rows");
  const bool split = a.ff > 0 && a.tile_rows > 1;
  if (split && (a.rows < 1 || ceil_div(a.rows, 2) > 65535)) return fail(-1, "mix_rows: too many rows in one launch");
  const int vecs = (a.nq + a.nk + a.nv + (a.tile_rows == 1 ? a.ff : 0)) / 8;
  const dim3 grid(ceil_div(vecs, MIX_THREADS), a.n_tiles);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (a.f32) launch_mix_rows<float>(a, grid, st);
  else launch_mix_rows<__nv_bfloat16>(a, grid, st);
  if (split) {
    if (a.f32) launch_ff_rows<float>(a.in, a.ld_in, a.off_gate, a.off_up, a.ff, a.act, nfn_gate_clamp{}, a.ff_out, a.ld_ff, a.rows, st);
    else launch_ff_rows<__nv_bfloat16>(a.in, a.ld_in, a.off_gate, a.off_up, a.ff, a.act, nfn_gate_clamp{}, a.ff_out, a.ld_ff, a.rows, st);
  }
  return launch_check("mix_rows", split ? 2 : 1);
}

extern "C" int nfn_ff_rows(int f32, const void* in, int ld_in, int off_gate, int off_up, int ff, int act, const nfn_gate_clamp* clamp, void* out, int ld_out, int rows,
                           nfn_stream_t stream) {
  if (rows <= 0 || ff <= 0) return 0;
  if ((ld_in | off_gate | ff | ld_out) & 7 || (off_up >= 0 && (off_up & 7))) return fail(-1, "ff_rows: widths and offsets must be multiples of 8");
  if (ceil_div(rows, 2) > 65535) return fail(-1, "ff_rows: too many rows in one launch");
  if (act == NFN_ACT_CLAMPED && (!clamp || off_up < 0)) return fail(-1, "ff_rows: the clamped gate needs its limits and an up value");
  const nfn_gate_clamp limits = clamp ? *clamp : nfn_gate_clamp{};
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (f32) launch_ff_rows<float>(in, ld_in, off_gate, off_up, ff, act, limits, out, ld_out, rows, st);
  else launch_ff_rows<__nv_bfloat16>(in, ld_in, off_gate, off_up, ff, act, limits, out, ld_out, rows, st);
  return launch_check("ff_rows");
}

extern "C" int nfn_side_mul(int f32, const float* gate, const int* tokens, const void* side_embed, long long ld_embed, int col0, int vocab,
                            void* out, int ld, int rows, int width, nfn_stream_t stream) {
  if (rows <= 0) return 0;
  if ((ld | width | col0) & 7 || (ld_embed & 7)) return fail(-1, "side_mul: widths must be multiples of 8");
  const int total = rows * (width / 8);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const __nv_bfloat16* e = static_cast<const __nv_bfloat16*>(side_embed);
  if (f32) side_mul_kernel<float><<<ceil_div(total, 128), 128, 0, st>>>(gate, tokens, e, ld_embed, col0, vocab, static_cast<float*>(out), ld, rows, width);
  else side_mul_kernel<__nv_bfloat16><<<ceil_div(total, 128), 128, 0, st>>>(gate, tokens, e, ld_embed, col0, vocab, static_cast<__nv_bfloat16*>(out), ld, rows, width);
  return launch_check("side_mul");
}

extern "C" int nfn_gemm_f32(const float* a, int lda, const void* b, int ldb, float* c, int ldc, int m, int n, int k, int accumulate,
                            const void* bias, nfn_stream_t stream) {
  if (m <= 0 || n <= 0 || k <= 0) return fail(-1, "gemm_f32: empty problem");
  if ((lda | ldb | k) & 3) return fail(-1, "gemm_f32: K and the leading dimensions must be multiples of 4");
  const dim3 grid(ceil_div(n, SG_BN), ceil_div(m, SG_BM));
  gemm_f32_kernel<<<grid, 256, 0, static_cast<cudaStream_t>(stream)>>>(a, lda, static_cast<const __nv_bfloat16*>(b), ldb, c, ldc, m, n, k, accumulate,
                                                                        static_cast<const __nv_bfloat16*>(bias));
  return launch_check("gemm_f32");
}
