// A gated recurrence that decides from the current token alone: per channel s <- (1 - z) s + z c, out = s * silu(g), with z = sigmoid(a) and a candidate c
// formed from b. Everything but the loads and stores is fp32.
//
// Short entries (single tokens, portions of a few rows) go token after token. Long ones are an affine scan: a CTA takes 32 channels, 16 lanes with two
// channels each, and 256 rows at a time in 32 segments of eight (two to a warp); every segment's rows become one step of the same form, the state in front
// of a segment follows from those of the segments before it, and the rows are run again from there, out of registers.
//
// A step is taken as s <- s + z (c - s). Where z is small a state lasts for thousands of tokens, and a factor 1 - z that is rounded on its own would leave
// each time a little less or more than the share z took.
#include <type_traits>

#include "attention_v2.cuh"
#include "common.h"
#include "paged.cuh"

namespace nfn {

// what a token does to a channel: s <- s + z (c - s)
struct GruStep { float z, c; };
template <typename T>
__device__ __forceinline__ GruStep gru_step(float a, float b) {
  return GruStep{sigmoid_for<T>(a), fmaxf(b + 0.5f, sigmoid_for<T>(b))};      // the line is the larger one where b >= 0, the sigmoid where b < 0
}
__device__ __forceinline__ float gru_take(float s, float z, float c) { return s + z * (c - s); }
__device__ __forceinline__ float2 gru_take2(float2 s, float2 z, float2 c) {
  float2 d, r;
  add2f(d.x, d.y, c.x, c.y, -s.x, -s.y);
  fma2(r.x, r.y, z.x, z.y, d.x, d.y, s.x, s.y);
  return r;
}
// the state behind several steps of which share `go` of it went and `come` came
__device__ __forceinline__ float2 gru_after(float2 s, float2 go, float2 come) {
  float2 d, r;
  fma2(d.x, d.y, -go.x, -go.y, s.x, s.y, come.x, come.y);
  add2f(r.x, r.y, s.x, s.y, d.x, d.y);
  return r;
}
template <typename T>
__device__ __forceinline__ float gru_out(float s, float g) { return s * g * sigmoid_for<T>(g); }

template <typename T>
using GruPair = typename std::conditional<sizeof(T) == 4, float2, uint32_t>::type;      // two neighbouring channels as they lie in memory
__device__ __forceinline__ float2 gru_unpack(float2 v) { return v; }
__device__ __forceinline__ float2 gru_unpack(uint32_t v) { return unpack_bf16x2(v); }
// a share's input of minus infinity
template <typename T>
__device__ __forceinline__ GruPair<T> gru_never();
template <>
__device__ __forceinline__ float2 gru_never<float>() { return make_float2(-INFINITY, -INFINITY); }
template <>
__device__ __forceinline__ uint32_t gru_never<__nv_bfloat16>() { return 0xff80ff80u; }
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

constexpr int GS_LANES = 16, GS_WARPS = 16, GS_ROWS = 8, GS_THREADS = GS_WARPS * 32, GS_SPAN = 2 * GS_WARPS * GS_ROWS;
template <typename T>
__global__ void __launch_bounds__(GS_THREADS, 1)
gru_scan_kernel(const nfn_gru_args p) {
  constexpr bool AHEAD = sizeof(T) == 2;                    // the next rows are on their way while these are used
  __shared__ float4 warps[2][GS_WARPS][GS_LANES];           // of a warp's two segments and both channels: share of the state that goes, what comes in its place
  const nfn_seq_rows seq = p.seqs[p.n_short + blockIdx.y];
  if (seq.slot < 0) return;
  const int warp = threadIdx.x / 32, lane = threadIdx.x % GS_LANES, seg = threadIdx.x / GS_LANES, c = blockIdx.x * 2 * GS_LANES + 2 * lane;
  const bool on = c < p.width, second = seg & 1;
  float2* st = reinterpret_cast<float2*>(p.state + (size_t)seq.slot * p.width + c);
  float2 s = make_float2(0.f, 0.f);
  if (on && seq.pos0 > 0) s = *st;
  const T* in = static_cast<const T*>(p.in) + (size_t)seq.row0 * p.ld_in + c;
  T* out = static_cast<T*>(p.out) + (size_t)seq.row0 * p.ld_out + c;
  GruPair<T> a[GS_ROWS], b[GS_ROWS], g[GS_ROWS], na[AHEAD ? GS_ROWS : 1], nb[AHEAD ? GS_ROWS : 1], ng[AHEAD ? GS_ROWS : 1];
  auto fetch = [&](int r0, GruPair<T>* fa, GruPair<T>* fb, GruPair<T>* fg) {
    const int first = r0 + seg * GS_ROWS;
    const T* x = in + (size_t)first * p.ld_in;
#pragma unroll
    for (int i = 0; i < GS_ROWS; ++i, x += p.ld_in) {
      fa[i] = gru_never<T>();                               // rows that do not exist leave the state alone
      fb[i] = fg[i] = GruPair<T>{};
      if (on && first + i < seq.n) {
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
    float2 z[GS_ROWS], cand[GS_ROWS], go = make_float2(0.f, 0.f), come = go;
#pragma unroll
    for (int i = 0; i < GS_ROWS; ++i) {
      const float2 x = gru_unpack(a[i]), y = gru_unpack(b[i]);
      const GruStep u = gru_step<T>(x.x, y.x), v = gru_step<T>(x.y, y.y);
      z[i] = make_float2(u.z, v.z);
      cand[i] = make_float2(u.c, v.c);
      go = gru_take2(go, z[i], make_float2(1.f, 1.f));
      come = gru_take2(come, z[i], cand[i]);
    }
    // both segments of the warp as one step, the first one's kept for the second
    const float2 go1 = make_float2(__shfl_xor_sync(0xffffffffu, go.x, GS_LANES), __shfl_xor_sync(0xffffffffu, go.y, GS_LANES));
    const float2 come1 = make_float2(__shfl_xor_sync(0xffffffffu, come.x, GS_LANES), __shfl_xor_sync(0xffffffffu, come.y, GS_LANES));
    if (!second) {
      const float2 f = gru_after(go, go1, go1), e = gru_after(come, go1, come1);
      warps[buf][warp][lane] = make_float4(f.x, f.y, e.x, e.y);
    }
    __syncthreads();                                        // the other buffer was read before the last one of these
    float2 mine = s;
#pragma unroll
    for (int q = 0; q < GS_WARPS; ++q) {
      if (q == warp) mine = s;
      const float4 e = warps[buf][q][lane];
      s = gru_after(s, make_float2(e.x, e.y), make_float2(e.z, e.w));
    }
    if (second) mine = gru_after(mine, go1, come1);
    const int first = r0 + seg * GS_ROWS;
    T* dst = out + (size_t)first * p.ld_out;
#pragma unroll
    for (int i = 0; i < GS_ROWS; ++i, dst += p.ld_out) {
      mine = gru_take2(mine, z[i], cand[i]);
      const float2 h = gru_unpack(g[i]);
      if (on && first + i < seq.n) gru_store(dst, gru_out<T>(mine.x, h.x), gru_out<T>(mine.y, h.y));
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
