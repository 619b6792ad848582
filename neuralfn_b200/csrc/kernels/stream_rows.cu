// Residual streams: the pass between two sublayers. A row's residual is a handful of fp32 rows ("streams"); a finished sublayer's
// output enters all of them through a small mixing matrix, the next sublayer reads a weighted sum of them through its norm. One CTA
// per row does both: every stream is read and written once, the weighted sum waits in shared memory until its norm is known.
// A single plain residual is the case of one stream with unit weights. The update may have a norm of its own (designs that norm a sublayer's output
// instead of its input), its rows may carry weights (routed experts) and a row every token has (a shared expert). Where every row is the next token of
// its own sequence the pass also adds the short convolution of designs whose sublayers read their input that way; other batches take a
// launch of its own for it, since a row then needs its neighbours' norms.
#include "common.h"
#include "paged.cuh"

namespace nfn {

template <int ST_THREADS>
__device__ __forceinline__ float st_block_sum(float v, float* red) {
#pragma unroll
  for (int s = 16; s > 0; s >>= 1) v += __shfl_xor_sync(0xffffffffu, v, s);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float t = 0.f;
#pragma unroll
  for (int i = 0; i < ST_THREADS / 32; ++i) t += red[i];
  return t;
}

template <typename T>
struct alignas(4 * sizeof(T)) StPiece { T v[4]; };
constexpr int ST_HIST = 3;      // history rows fetched ahead

// a norm's weights of channels 4 v .. 4 v + 3, as they lie in memory; scalar: one number for all of them
__device__ __forceinline__ StPiece<__nv_bfloat16> st_weight(const void* w, int v, int scalar) {
  const __nv_bfloat16* p = static_cast<const __nv_bfloat16*>(w);
  if (!scalar) return *reinterpret_cast<const StPiece<__nv_bfloat16>*>(p + 4 * v);
  return StPiece<__nv_bfloat16>{{*p, *p, *p, *p}};
}

// S: streams held in registers (an upper bound; the mixing weights past p.streams are zero). CONV: with the short convolution. Few rows take many threads each, so that a
// row's loads are all on their way at once
template <typename T, int S, int ST_THREADS, bool CONV>
__global__ void __launch_bounds__(ST_THREADS)
stream_pass_kernel(const nfn_stream_args p) {
  extern __shared__ float st_row[];                        // [ld] u
  __shared__ float red[ST_THREADS / 32], red_y[ST_THREADS / 32], w_mix[S][S], w_out[S], w_in[S];
  const int r = blockIdx.x, n = p.streams, vecs = p.ld / 4;
  const int src = p.src_rows ? p.src_rows[r] : r;
  const __nv_bfloat16* emb = nullptr;
  if (p.tokens) emb = static_cast<const __nv_bfloat16*>(p.embed) + (size_t)min(max(p.tokens[r], 0), p.vocab - 1) * p.ld;
  const float* x = p.x + (size_t)src * n * p.ld;
  float* x_out = p.x_out ? p.x_out + (size_t)r * n * p.ld : nullptr;
  const T* y = static_cast<const T*>(p.y);
  nfn_row_tile tile{};
  if constexpr (CONV) tile = p.tiles[r];                   // the first of all: the history's place depends on it
  float4 b[S], f;
  auto fetch_x = [&](int v) {
    if (emb) {
      b[0] = load4(emb + 4 * v);
    } else {
#pragma unroll
      for (int s = 0; s < S; ++s) b[s] = s < n ? load4(x + (size_t)s * p.ld + 4 * v) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
  };
  auto fetch_y = [&](int v) {
    f = make_float4(0.f, 0.f, 0.f, 0.f);
    if (p.y) {
#pragma unroll 4
      for (int j = 0; j < p.y_rows; ++j) {
        const int at = src * p.y_rows + j, yr = p.y_index ? p.y_index[at] : at;
        const float4 g = load4(y + (size_t)yr * p.ld + 4 * v);
        const float a = p.y_item ? p.y_item[at] : 1.f;
        f.x += a * g.x; f.y += a * g.y; f.z += a * g.z; f.w += a * g.w;
      }
      if (p.y_plus) {
        const float4 g = load4(static_cast<const T*>(p.y_plus) + (size_t)src * p.ld + 4 * v);
        f.x += g.x; f.y += g.y; f.z += g.z; f.w += g.w;
      }
    }
  };
  if (threadIdx.x < S * S) {
    const int s = threadIdx.x / S, t = threadIdx.x % S;
    w_mix[s][t] = (s < n && t < n) ? (p.mix ? __bfloat162float(static_cast<const __nv_bfloat16*>(p.mix)[s * n + t]) : (s == t ? 1.f : 0.f)) : 0.f;
  }
  if (threadIdx.x < S) {
    const int s = threadIdx.x;
    w_out[s] = s < n ? (p.out ? __bfloat162float(static_cast<const __nv_bfloat16*>(p.out)[s]) : 1.f) : 0.f;
    w_in[s] = s < n ? (p.in ? __bfloat162float(static_cast<const __nv_bfloat16*>(p.in)[s]) : 1.f) : 0.f;
  }
  if (threadIdx.x < vecs) {
    fetch_x(threadIdx.x);
    fetch_y(threadIdx.x);
  }
  StPiece<__nv_bfloat16> wt{}, wy{};                       // the norms' weights of the first piece come along
  if (p.y_weight && threadIdx.x < vecs) wy = st_weight(p.y_weight, threadIdx.x, p.scalar_norms);
  if (p.h && p.weight && threadIdx.x < vecs) wt = st_weight(p.weight, threadIdx.x, p.scalar_norms);
  const T* old = nullptr;                                  // the sequence's stored rows; none before its start
  StPiece<T> past[ST_HIST];                                // as they lie in memory
  StPiece<__nv_bfloat16> taps[ST_HIST + 1];
  const int hist = p.conv_taps - 1;
  const __nv_bfloat16* conv = static_cast<const __nv_bfloat16*>(p.conv);
  auto stored = [&](int i, int v) { return old && tile.e_pos0 - hist + i >= 0 ? *reinterpret_cast<const StPiece<T>*>(old + (size_t)i * p.ld + 4 * v) : StPiece<T>{}; };
  auto tap = [&](int i, int v) { return *reinterpret_cast<const StPiece<__nv_bfloat16>*>(conv + (size_t)i * p.ld + 4 * v); };
  if constexpr (CONV) {
    if (tile.slot >= 0 && hist > 0) old = static_cast<const T*>(p.history) + (size_t)tile.parity * p.history_half + (size_t)tile.slot * hist * p.ld;
    if (threadIdx.x < vecs) {
#pragma unroll
      for (int i = 0; i < ST_HIST; ++i)
        if (i < hist) past[i] = stored(i, threadIdx.x);
    }
  }
  __syncthreads();
  float ry = 0.f;
  if (p.y_weight) {                                        // the update's own norm: its pieces past the first one wait in shared memory
    float sy = threadIdx.x < vecs ? f.x * f.x + f.y * f.y + f.z * f.z + f.w * f.w : 0.f;
    const float4 first = f;
    for (int v = threadIdx.x + ST_THREADS; v < vecs; v += ST_THREADS) {
      fetch_y(v);
      store4(st_row + 4 * v, f);
      sy += f.x * f.x + f.y * f.y + f.z * f.z + f.w * f.w;
    }
    f = first;
    ry = p.y_scale / sqrtf(st_block_sum<ST_THREADS>(sy, red_y) / (float)p.width + p.eps);
  }
  float ss = 0.f;
  for (int v = threadIdx.x; v < vecs; v += ST_THREADS) {
    if (v != threadIdx.x) {
      fetch_x(v);
      if (p.y_weight) f = load4(st_row + 4 * v);
      else fetch_y(v);
    }
    if (p.y_weight) {
      if (v != threadIdx.x) wy = st_weight(p.y_weight, v, p.scalar_norms);
      const float4 w = load4(wy.v);
      f.x *= ry * w.x; f.y *= ry * w.y; f.z *= ry * w.z; f.w *= ry * w.w;
    }
    if (emb) {
      b[0].x *= p.embed_scale; b[0].y *= p.embed_scale; b[0].z *= p.embed_scale; b[0].w *= p.embed_scale;
#pragma unroll
      for (int s = 1; s < S; ++s) b[s] = b[0];
    }
    if (p.y) {
      float4 c[S];
#pragma unroll
      for (int t = 0; t < S; ++t) {
        const float o = w_out[t];
        c[t] = make_float4(o * f.x, o * f.y, o * f.z, o * f.w);
#pragma unroll
        for (int s = 0; s < S; ++s) {
          const float m = w_mix[s][t];
          c[t].x += m * b[s].x; c[t].y += m * b[s].y; c[t].z += m * b[s].z; c[t].w += m * b[s].w;
        }
      }
#pragma unroll
      for (int t = 0; t < S; ++t) b[t] = c[t];
    }
    if (x_out) {
#pragma unroll
      for (int s = 0; s < S; ++s)
        if (s < n) store4(x_out + (size_t)s * p.ld + 4 * v, b[s]);
    }
    if (p.h) {
      float4 u = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
      for (int s = 0; s < S; ++s) {
        const float m = w_in[s];
        u.x += m * b[s].x; u.y += m * b[s].y; u.z += m * b[s].z; u.w += m * b[s].w;
      }
      if (!p.weight) {                                     // no norm: the row leaves as it is
        store4(static_cast<T*>(p.h) + (size_t)r * p.ld + 4 * v, u);
        continue;
      }
      store4(st_row + 4 * v, u);
      ss += u.x * u.x + u.y * u.y + u.z * u.z + u.w * u.w;
    }
  }
  if (!p.h || !p.weight) return;
  if constexpr (CONV) {                                    // on their way during the sum
    if (threadIdx.x < vecs) {
#pragma unroll
      for (int i = 0; i <= ST_HIST; ++i)
        if (i <= hist) taps[i] = tap(i, threadIdx.x);
    }
  }
  const float rms = 1.f / sqrtf(st_block_sum<ST_THREADS>(ss, red) / (float)p.width + p.eps);
  T* h = static_cast<T*>(p.h) + (size_t)r * p.ld;
  for (int v = threadIdx.x; v < vecs; v += ST_THREADS) {
    if (v != threadIdx.x) wt = st_weight(p.weight, v, p.scalar_norms);
    const float4 u = load4(st_row + 4 * v), w = load4(wt.v);
    const float4 n = make_float4(u.x * rms * (w.x + p.weight_offset), u.y * rms * (w.y + p.weight_offset), u.z * rms * (w.z + p.weight_offset), u.w * rms * (w.w + p.weight_offset));
    if constexpr (CONV) {
      float4 c = n;
      T* left = tile.slot >= 0 && hist > 0 ? static_cast<T*>(p.history) + (size_t)(1 - tile.parity) * p.history_half + (size_t)tile.slot * hist * p.ld + 4 * v : nullptr;
      auto add = [&](int i, const float4& x, const float4& t) {
        c.x += t.x * x.x; c.y += t.y * x.y; c.z += t.z * x.z; c.w += t.w * x.w;
        if (left && i > 0) store4(left + (size_t)(i - 1) * p.ld, x);
      };
      const bool ahead = v == threadIdx.x && hist <= ST_HIST;
      if (ahead) {
#pragma unroll
        for (int i = 0; i < ST_HIST; ++i)
          if (i < hist) add(i, load4(past[i].v), load4(taps[i].v));
#pragma unroll
        for (int i = 0; i <= ST_HIST; ++i)
          if (i == hist) add(i, n, load4(taps[i].v));
      } else {
        for (int i = 0; i < hist; ++i) {
          const StPiece<T> x = stored(i, v);
          add(i, load4(x.v), load4(conv + (size_t)i * p.ld + 4 * v));
        }
        add(hist, n, load4(conv + (size_t)hist * p.ld + 4 * v));
      }
      store4(h + 4 * v, c);
    } else {
      store4(h + 4 * v, n);
    }
  }
}

// The convolution over the rows of any entries. A warp takes 256 channels of four rows of a tile, a lane eight channels: the rows and the ones before
// them are all on their way at once, and what the warps of a tile have in common comes out of L1.
constexpr int IC_WARPS = 4, IC_ROWS = 4, IC_COLS = 256;

template <typename T>
struct alignas(16) Piece8 { T v[8]; };

// TAPS = 0: any number of taps, one at a time
template <typename T, int TAPS>
__global__ void __launch_bounds__(IC_WARPS * 32)
input_conv_kernel(const nfn_input_conv_args p) {
  const nfn_row_tile t = p.tiles[blockIdx.y];
  const int i0 = threadIdx.x / 32 * IC_ROWS, col = blockIdx.x * IC_COLS + threadIdx.x % 32 * 8;
  if (t.slot < 0 || col >= p.ld || i0 >= t.n) return;
  const int taps = TAPS ? TAPS : p.taps, hist = taps - 1, at = t.row0 - t.e_row0 + i0, n = min(IC_ROWS, t.n - i0);      // of the entry
  const T* rows = static_cast<const T*>(p.h) + (size_t)t.e_row0 * p.ld + col;
  const T* old = static_cast<const T*>(p.history) + (size_t)t.parity * p.history_half + (size_t)t.slot * hist * p.ld + col;
  const __nv_bfloat16* conv = static_cast<const __nv_bfloat16*>(p.conv) + col;
  T* out = static_cast<T*>(p.out) + (size_t)(t.row0 + i0) * p.ld + col;
  // row `idx` of the entry: this step's, a stored one, or zero before the sequence's start
  auto source = [&](int idx) {
    if (idx >= 0) return *reinterpret_cast<const Piece8<T>*>(rows + (size_t)idx * p.ld);
    return t.e_pos0 + idx >= 0 ? *reinterpret_cast<const Piece8<T>*>(old + (size_t)(hist + idx) * p.ld) : Piece8<T>{};
  };
  auto tap = [&](int j) { return *reinterpret_cast<const Piece8<__nv_bfloat16>*>(conv + (size_t)j * p.ld); };
  if constexpr (TAPS == 0) {
    for (int i = 0; i < n; ++i) {
      float acc[8];
      const Piece8<T> x = source(at + i);
#pragma unroll
      for (int e = 0; e < 8; ++e) acc[e] = to_float(x.v[e]);
      for (int j = 0; j < taps; ++j) {
        const Piece8<T> y = source(at + i - hist + j);
        const Piece8<__nv_bfloat16> w = tap(j);
#pragma unroll
        for (int e = 0; e < 8; ++e) acc[e] += to_float(w.v[e]) * to_float(y.v[e]);
      }
      store8(out + (size_t)i * p.ld, acc);
    }
  } else {
    Piece8<T> x[IC_ROWS + TAPS - 1];
    Piece8<__nv_bfloat16> w[TAPS];
    if (n == IC_ROWS && at >= TAPS - 1) {                  // inside the entry: nothing to decide between the loads
      const T* first = rows + (size_t)(at - (TAPS - 1)) * p.ld;
#pragma unroll
      for (int i = 0; i < IC_ROWS + TAPS - 1; ++i) x[i] = *reinterpret_cast<const Piece8<T>*>(first + (size_t)i * p.ld);
    } else {
#pragma unroll
      for (int i = 0; i < IC_ROWS + TAPS - 1; ++i)
        if (i < n + TAPS - 1) x[i] = source(at - (TAPS - 1) + i);
    }
#pragma unroll
    for (int j = 0; j < TAPS; ++j) w[j] = tap(j);
#pragma unroll
    for (int i = 0; i < IC_ROWS; ++i) {
      if (i >= n) break;
      float acc[8];
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        float a = to_float(x[i + TAPS - 1].v[e]);
#pragma unroll
        for (int j = 0; j < TAPS; ++j) a += to_float(w[j].v[e]) * to_float(x[i + j].v[e]);
        acc[e] = a;
      }
      store8(out + (size_t)i * p.ld, acc);
    }
  }
  // the history the entry leaves behind: its newest taps - 1 rows (older ones move up when it brought fewer)
  if (i0 == 0 && hist > 0 && t.row0 + t.n == t.e_row0 + t.e_n) {
    T* left = static_cast<T*>(p.history) + (size_t)(1 - t.parity) * p.history_half + (size_t)t.slot * hist * p.ld + col;
    for (int i = 0; i < hist; ++i) *reinterpret_cast<Piece8<T>*>(left + (size_t)i * p.ld) = source(t.e_n - hist + i);
  }
}

template <typename T>
static int pick_input_conv(const nfn_input_conv_args& a, cudaStream_t st) {
  const dim3 grid(ceil_div(a.ld, IC_COLS), a.n_tiles);                     // neighbouring CTAs read neighbouring columns of the same rows
  switch (a.taps) {
    case 1: input_conv_kernel<T, 1><<<grid, IC_WARPS * 32, 0, st>>>(a); break;
    case 2: input_conv_kernel<T, 2><<<grid, IC_WARPS * 32, 0, st>>>(a); break;
    case 3: input_conv_kernel<T, 3><<<grid, IC_WARPS * 32, 0, st>>>(a); break;
    case 4: input_conv_kernel<T, 4><<<grid, IC_WARPS * 32, 0, st>>>(a); break;
    default: input_conv_kernel<T, 0><<<grid, IC_WARPS * 32, 0, st>>>(a); break;
  }
  return launch_check("input_conv");
}

template <typename T, int S, int THREADS, bool CONV = false>
static int launch_stream(const nfn_stream_args& a, cudaStream_t st) {
  const size_t smem = a.h || a.y_weight ? (size_t)a.ld * sizeof(float) : 0;
  auto kern = stream_pass_kernel<T, S, THREADS, CONV>;
  static bool raised[64] = {};
  int dev = 0;
  cudaGetDevice(&dev);
  if (smem > 40 * 1024 && !raised[dev & 63]) {
    if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024) != cudaSuccess) return launch_check("stream_pass attr", 0);
    raised[dev & 63] = true;
  }
  kern<<<a.rows, THREADS, smem, st>>>(a);
  return launch_check("stream_pass");
}

template <typename T>
static int pick_stream(const nfn_stream_args& a, cudaStream_t st) {
  const bool few = a.rows <= 2 * sm_count() && a.ld >= 2048;
  if (a.conv) return few ? launch_stream<T, 1, 1024, true>(a, st) : launch_stream<T, 1, 256, true>(a, st);
  switch (a.streams) {
    case 1: return few ? launch_stream<T, 1, 1024>(a, st) : launch_stream<T, 1, 256>(a, st);
    case 2: return few ? launch_stream<T, 2, 1024>(a, st) : launch_stream<T, 2, 256>(a, st);
    case 3: return few ? launch_stream<T, 3, 1024>(a, st) : launch_stream<T, 3, 256>(a, st);
    case 4: return few ? launch_stream<T, 4, 1024>(a, st) : launch_stream<T, 4, 256>(a, st);
    default: return a.streams <= 8 ? launch_stream<T, 8, 256>(a, st) : launch_stream<T, NFN_MAX_STREAMS, 256>(a, st);
  }
}

}  // namespace nfn

using namespace nfn;

extern "C" int nfn_stream_pass(const nfn_stream_args* args, nfn_stream_t stream) {
  if (!args) return fail(-1, "stream_pass: null args");
  const nfn_stream_args& a = *args;
  if (a.rows <= 0) return 0;
  if ((a.ld & 15) || a.width <= 0 || a.width > a.ld) return fail(-1, "stream_pass: the row pitch must be a multiple of 16 that holds the width");
  if (a.streams < 1 || a.streams > NFN_MAX_STREAMS) return fail(-1, "stream_pass: 1 to 16 streams");
  if (!a.tokens && !a.x) return fail(-1, "stream_pass: neither tokens nor rows");
  if (a.y && a.y_rows < 1) return fail(-1, "stream_pass: an update needs at least one row");
  if ((size_t)a.ld * 4 > 200 * 1024) return fail(-1, "stream_pass: rows too wide");
  if (a.conv && (a.streams != 1 || !a.h || !a.weight || !a.tiles || a.conv_taps < 1 || (a.conv_taps > 1 && !a.history)))
    return fail(-1, "stream_pass: the convolution goes with one stream, a norm, a tile per row and a history");
  return a.f32 ? pick_stream<float>(a, static_cast<cudaStream_t>(stream)) : pick_stream<__nv_bfloat16>(a, static_cast<cudaStream_t>(stream));
}

extern "C" int nfn_input_conv(const nfn_input_conv_args* args, nfn_stream_t stream) {
  if (!args) return fail(-1, "input_conv: null args");
  const nfn_input_conv_args& a = *args;
  if (a.n_tiles <= 0) return 0;
  if (a.n_tiles > 65535) return fail(-1, "input_conv: too many row tiles in one launch");
  if ((a.ld & 15) || a.taps < 1 || !a.h || !a.conv || !a.out || a.h == a.out || !a.tiles || (a.taps > 1 && !a.history)) return fail(-1, "input_conv: rows padded to multiples of 16, two buffers, a history");
  return a.f32 ? pick_input_conv<float>(a, static_cast<cudaStream_t>(stream)) : pick_input_conv<__nv_bfloat16>(a, static_cast<cudaStream_t>(stream));
}
