// Residual streams: the pass between two sublayers. A row's residual is a handful of fp32 rows ("streams"); a finished sublayer's
// output enters all of them through a small mixing matrix, the next sublayer reads a weighted sum of them through its norm. One CTA
// per row does both: every stream is read and written once, the weighted sum waits in shared memory until its norm is known.
// A single plain residual is the case of one stream with unit weights. The update may have a norm of its own (designs that norm a sublayer's output
// instead of its input), its rows may carry weights (routed experts) and a row every token has (a shared expert).
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

// S: streams held in registers (an upper bound; the mixing weights past p.streams are zero). Few rows take many threads each, so that a
// row's loads are all on their way at once
template <typename T, int S, int ST_THREADS>
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
  float4 wt = make_float4(0.f, 0.f, 0.f, 0.f);             // the norm's weights of the first piece come along
  if (p.h && p.weight && threadIdx.x < vecs) wt = load4(static_cast<const __nv_bfloat16*>(p.weight) + 4 * threadIdx.x);
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
      const float4 w = load4(static_cast<const __nv_bfloat16*>(p.y_weight) + 4 * v);
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
  const float rms = 1.f / sqrtf(st_block_sum<ST_THREADS>(ss, red) / (float)p.width + p.eps);
  T* h = static_cast<T*>(p.h) + (size_t)r * p.ld;
  for (int v = threadIdx.x; v < vecs; v += ST_THREADS) {
    const float4 u = load4(st_row + 4 * v), w = v == threadIdx.x ? wt : load4(static_cast<const __nv_bfloat16*>(p.weight) + 4 * v);
    store4(h + 4 * v, make_float4(u.x * rms * (w.x + p.weight_offset), u.y * rms * (w.y + p.weight_offset), u.z * rms * (w.z + p.weight_offset),
                                  u.w * rms * (w.w + p.weight_offset)));
  }
}

template <typename T, int S, int THREADS>
static int launch_stream(const nfn_stream_args& a, cudaStream_t st) {
  const size_t smem = a.h || a.y_weight ? (size_t)a.ld * sizeof(float) : 0;
  auto kern = stream_pass_kernel<T, S, THREADS>;
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
  return a.f32 ? pick_stream<float>(a, static_cast<cudaStream_t>(stream)) : pick_stream<__nv_bfloat16>(a, static_cast<cudaStream_t>(stream));
}
