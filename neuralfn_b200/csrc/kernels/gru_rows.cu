// A gated recurrence whose gates read only the current token: per channel s <- (1 - z) s + z c, out = s * silu(g), with z = sigmoid(a) and a candidate c
// formed from b. Everything but the loads and stores is fp32.
//
// Short entries (single tokens, portions of a few rows) go token after token. Long ones are an affine scan: a CTA takes 32 channels, 16 lanes with two
// channels each, and 256 rows at a time in 32 segments of eight; every segment's rows become one step of the same form, the state in front
// of a segment follows from those of the segments before it, and the rows are run again from there, out of registers.
//
// A step is taken as s <- s + z (c - s). Where z is small a state lasts for thousands of tokens, and a factor 1 - z that is rounded on its own would leave
// each time a little less or more than the share z took.
#include <type_traits>

#include "common.h"
#include "paged.cuh"

namespace nfn {

// what a token does to a channel: s <- s + z (c - s)
struct GruStep { float z, c; };
template <typename T>
__device__ __forceinline__ GruStep gru_step(float a, float b) {
  return GruStep{sigmoid_for<T>(a), b >= 0.f ? b + 0.5f : sigmoid_for<T>(b)};
}
__device__ __forceinline__ float gru_take(float s, float z, float c) { return s + z * (c - s); }
template <typename T>
__device__ __forceinline__ float gru_out(float s, float g) { return s * g * sigmoid_for<T>(g); }

template <typename T>
using GruPair = typename std::conditional<sizeof(T) == 4, float2, uint32_t>::type;      // two neighbouring channels as they lie in memory
__device__ __forceinline__ float2 gru_unpack(float2 v) { return v; }
__device__ __forceinline__ float2 gru_unpack(uint32_t v) { return unpack_bf16x2(v); }
__device__ __forceinline__ void gru_store(float* p, float x, float y) { *reinterpret_cast<float2*>(p) = make_float2(x, y); }
__device__ __forceinline__ void gru_store(__nv_bfloat16* p, float x, float y) { *reinterpret_cast<uint32_t*>(p) = pack_bf16x2(x, y); }

constexpr int GR_THREADS = 128;
template <typename T>
__global__ void __launch_bounds__(GR_THREADS)
gru_short_kernel(const nfn_gru_args p) {
  const nfn_seq_rows seq = p.seqs[blockIdx.y];
  const int c = 2 * (blockIdx.x * GR_THREADS + threadIdx.x);
  if (seq.slot < 0 || c >= p.width) return;
  float2* st = reinterpret_cast<float2*>(p.state + (size_t)seq.slot * p.width + c);
  float2 s = make_float2(0.f, 0.f);
  if (seq.pos0 > 0) s = *st;
  for (int t = 0; t < seq.n; ++t) {
    const T* x = static_cast<const T*>(p.in) + (size_t)(seq.row0 + t) * p.ld_in + c;
    const float2 a = gru_unpack(*reinterpret_cast<const GruPair<T>*>(x)), b = gru_unpack(*reinterpret_cast<const GruPair<T>*>(x + p.width)),
                 g = gru_unpack(*reinterpret_cast<const GruPair<T>*>(x + 2 * p.width));
    const GruStep u = gru_step<T>(a.x, b.x), v = gru_step<T>(a.y, b.y);
    s = make_float2(gru_take(s.x, u.z, u.c), gru_take(s.y, v.z, v.c));
    gru_store(static_cast<T*>(p.out) + (size_t)(seq.row0 + t) * p.ld_out + c, gru_out<T>(s.x, g.x), gru_out<T>(s.y, g.y));
  }
  *st = s;
}

constexpr int GS_LANES = 16, GS_SEGS = 32, GS_ROWS = 8, GS_THREADS = GS_LANES * GS_SEGS, GS_SPAN = GS_SEGS * GS_ROWS;
template <typename T>
__global__ void __launch_bounds__(GS_THREADS, 1)
gru_scan_kernel(const nfn_gru_args p) {
  constexpr bool AHEAD = sizeof(T) == 2;                    // the next rows are on their way while these are used
  __shared__ float4 segs[2][GS_SEGS][GS_LANES];             // of both channels: share of the state before it that goes, what comes in its place
  const nfn_seq_rows seq = p.seqs[p.n_short + blockIdx.y];
  if (seq.slot < 0) return;
  const int lane = threadIdx.x % GS_LANES, seg = threadIdx.x / GS_LANES, c = blockIdx.x * 2 * GS_LANES + 2 * lane;
  const bool on = c < p.width;
  float2* st = reinterpret_cast<float2*>(p.state + (size_t)seq.slot * p.width + c);
  float2 s = make_float2(0.f, 0.f);
  if (on && seq.pos0 > 0) s = *st;
  const T* in = static_cast<const T*>(p.in) + (size_t)seq.row0 * p.ld_in + c;
  T* out = static_cast<T*>(p.out) + (size_t)seq.row0 * p.ld_out + c;
  GruPair<T> a[GS_ROWS], b[GS_ROWS], g[GS_ROWS], na[AHEAD ? GS_ROWS : 1], nb[AHEAD ? GS_ROWS : 1], ng[AHEAD ? GS_ROWS : 1];
  auto fetch = [&](int r0, GruPair<T>* fa, GruPair<T>* fb, GruPair<T>* fg) {
#pragma unroll
    for (int i = 0; i < GS_ROWS; ++i) {
      const int r = r0 + seg * GS_ROWS + i;
      if (on && r < seq.n) {
        const T* x = in + (size_t)r * p.ld_in;
        fa[i] = *reinterpret_cast<const GruPair<T>*>(x);
        fb[i] = *reinterpret_cast<const GruPair<T>*>(x + p.width);
        fg[i] = *reinterpret_cast<const GruPair<T>*>(x + 2 * p.width);
      }
    }
  };
  fetch(0, a, b, g);
  int buf = 0;
  for (int r0 = 0; r0 < seq.n; r0 += GS_SPAN, buf ^= 1) {
    if constexpr (AHEAD) fetch(r0 + GS_SPAN, na, nb, ng);
    const int live = on ? min(GS_ROWS, seq.n - r0 - seg * GS_ROWS) : 0;
    float2 z[GS_ROWS], cand[GS_ROWS];
    float4 f = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int i = 0; i < GS_ROWS; ++i)
      if (i < live) {
        const float2 x = gru_unpack(a[i]), y = gru_unpack(b[i]);
        const GruStep u = gru_step<T>(x.x, y.x), v = gru_step<T>(x.y, y.y);
        z[i] = make_float2(u.z, v.z);
        cand[i] = make_float2(u.c, v.c);
        f = make_float4(gru_take(f.x, u.z, 1.f), gru_take(f.y, u.z, u.c), gru_take(f.z, v.z, 1.f), gru_take(f.w, v.z, v.c));
      }
    segs[buf][seg][lane] = f;
    __syncthreads();                                        // the other buffer was read before the last one of these
    float2 mine = s;
#pragma unroll
    for (int q = 0; q < GS_SEGS; ++q) {
      if (q == seg) mine = s;
      const float4 e = segs[buf][q][lane];
      s = make_float2(s.x + (e.y - e.x * s.x), s.y + (e.w - e.z * s.y));
    }
#pragma unroll
    for (int i = 0; i < GS_ROWS; ++i)
      if (i < live) {
        mine = make_float2(gru_take(mine.x, z[i].x, cand[i].x), gru_take(mine.y, z[i].y, cand[i].y));
        const float2 h = gru_unpack(g[i]);
        gru_store(out + (size_t)(r0 + seg * GS_ROWS + i) * p.ld_out, gru_out<T>(mine.x, h.x), gru_out<T>(mine.y, h.y));
      }
    if constexpr (AHEAD) {
#pragma unroll
      for (int i = 0; i < GS_ROWS; ++i) { a[i] = na[i]; b[i] = nb[i]; g[i] = ng[i]; }
    } else {
      fetch(r0 + GS_SPAN, a, b, g);
    }
  }
  if (on && seg == 0) *st = s;
}

template <typename T>
static int launch_gru(const nfn_gru_args& a, cudaStream_t st) {
  const int longs = a.n_seqs - a.n_short;
  if (a.n_short > 0) gru_short_kernel<T><<<dim3(ceil_div(a.width, 2 * GR_THREADS), a.n_short), GR_THREADS, 0, st>>>(a);
  if (longs > 0) gru_scan_kernel<T><<<dim3(ceil_div(a.width, 2 * GS_LANES), longs), GS_THREADS, 0, st>>>(a);
  return launch_check("gru_rows", (a.n_short > 0) + (longs > 0));
}

}  // namespace nfn

using namespace nfn;

extern "C" int nfn_gru_rows(const nfn_gru_args* args, nfn_stream_t stream) {
  if (!args) return fail(-1, "gated recurrence: null args");
  const nfn_gru_args& a = *args;
  if (a.n_seqs <= 0) return 0;
  if ((a.width & 15) || a.width <= 0 || ((a.ld_in | a.ld_out) & 7)) return fail(-1, "gated recurrence: widths and pitches must be multiples of 16 and 8");
  if (!a.in || !a.state || !a.out || !a.seqs || a.n_short < 0 || a.n_short > a.n_seqs || a.n_seqs > 65535) return fail(-1, "gated recurrence: null operand or too many sequences");
  return a.f32 ? launch_gru<float>(a, static_cast<cudaStream_t>(stream)) : launch_gru<__nv_bfloat16>(a, static_cast<cudaStream_t>(stream));
}
