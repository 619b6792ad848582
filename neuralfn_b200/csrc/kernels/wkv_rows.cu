// Time mixing with a token shift and a recurrence that gives the current token a bonus: the shifted inputs, the rule token after token (single
// tokens, short portions, any length in 32-bit mode; prompt portions in bf16 take wkv_chunk.cu) and the fused decode step.
//
// Per head and value column c the rule needs the state column S[:, c] only, so a warp owns eight columns - four lanes across, two columns
// each, eight lanes down the key channels - and keeps them in registers from the first token of its entry to the last. Decays, state,
// bonus and read-outs are fp32.
#include <algorithm>

#include "common.h"
#include "paged.cuh"
#include "wkv.cuh"

namespace nfn {

// ------------------------------------------------------------------------------------------------- token shift --
constexpr int SH_THREADS = 256, SH_MAX = 8;

template <typename TS, typename T>
__global__ void __launch_bounds__(SH_THREADS)
shift_rows_kernel(const nfn_shift_args p) {
  const nfn_row_tile t = p.tiles[blockIdx.x];
  if (t.slot < 0) return;
  const int c = (blockIdx.y * SH_THREADS + threadIdx.x) * 4;
  if (c >= p.ld) return;
  float4 mu[SH_MAX];
#pragma unroll
  for (int s = 0; s < SH_MAX; ++s)
    if (s < p.n) mu[s] = load4(static_cast<const __nv_bfloat16*>(p.mu) + (size_t)s * p.ld + c);
  const TS* src = static_cast<const TS*>(p.src) + (size_t)t.row0 * p.ld + c;
  T* out = static_cast<T*>(p.out) + (size_t)t.row0 * p.ld + c;
  float4 back = make_float4(0.f, 0.f, 0.f, 0.f);
  if (t.row0 > t.e_row0) back = load4(src - p.ld);
  else if (t.e_pos0 > 0) back = load4(p.prev + (size_t)t.parity * p.prev_half + (size_t)t.slot * p.ld + c);
  for (int i = 0; i < t.n; ++i) {
    const float4 h = load4(src + (size_t)i * p.ld);
    const float4 d = make_float4(back.x - h.x, back.y - h.y, back.z - h.z, back.w - h.w);
#pragma unroll
    for (int s = 0; s < SH_MAX; ++s)
      if (s < p.n)
        store4(out + s * p.out_stride + (size_t)i * p.ld, make_float4(h.x + d.x * mu[s].x, h.y + d.y * mu[s].y, h.z + d.z * mu[s].z, h.w + d.w * mu[s].w));
    back = h;
  }
  if (t.row0 + t.n == t.e_row0 + t.e_n) store4(p.prev + (size_t)(1 - t.parity) * p.prev_half + (size_t)t.slot * p.ld + c, back);
}

// --------------------------------------------------------------------------------------------- token after token --
constexpr int WR_WARPS = 4, WR_COLS = 8;

// NR: key channels per lane (dim_p <= 8 NR)
template <typename T, int NR>
__global__ void __launch_bounds__(WR_WARPS * 32)
wkv_rows_kernel(const nfn_wkv_args p) {
  extern __shared__ float wr_smem[];                        // [WR_WARPS][3][dim_p]: r, k, w of the token at hand
  const nfn_seq_rows seq = p.seqs[blockIdx.z];
  if (seq.slot < 0) return;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, rg = lane >> 2, cl = lane & 3;
  const int h = blockIdx.y, DP = p.dim_p, HD = p.heads * DP;
  const int col0 = (blockIdx.x * WR_WARPS + warp) * WR_COLS;
  if (col0 >= DP) return;
  const int col = col0 + 2 * cl;
  float* sr = wr_smem + warp * 3 * DP;
  float *sk = sr + DP, *sw = sk + DP;
  float* st = p.state + ((size_t)seq.slot * p.heads + h) * DP * DP + col;
  float s[NR][2];
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int d = rg + 8 * i;
    float2 v = make_float2(0.f, 0.f);
    if (seq.pos0 > 0 && d < DP) v = *reinterpret_cast<const float2*>(st + (size_t)d * DP);
    s[i][0] = v.x;
    s[i][1] = v.y;
  }
  const __nv_bfloat16* w0 = static_cast<const __nv_bfloat16*>(p.w0) + (size_t)h * DP;
  const __nv_bfloat16* u = static_cast<const __nv_bfloat16*>(p.u) + (size_t)h * DP;
  for (int t = 0; t < seq.n; ++t) {
    const size_t row = (size_t)(seq.row0 + t);
    const T* x = static_cast<const T*>(p.rkv) + row * p.ld_rkv + (size_t)h * DP;
    const float* z = p.z + row * p.ld_z + (size_t)h * DP;
    float bonus = 0.f;
    for (int d = lane * 4; d < DP; d += 128) {
      const float4 r = load4(x + d), k = load4(x + HD + d), f = load4(z + d), b = load4(w0 + d), uu = load4(u + d);
      bonus += r.x * (uu.x * k.x) + r.y * (uu.y * k.y) + r.z * (uu.z * k.z) + r.w * (uu.w * k.w);
      store4(sr + d, r);
      store4(sk + d, k);
      store4(sw + d, make_float4(wkv_decay(f.x + b.x), wkv_decay(f.y + b.y), wkv_decay(f.z + b.z), wkv_decay(f.w + b.w)));
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) bonus += __shfl_xor_sync(0xffffffffu, bonus, o);
    const float v0 = to_float(x[2 * HD + col]), v1 = to_float(x[2 * HD + col + 1]);
    __syncwarp();
    float o0 = 0.f, o1 = 0.f;
#pragma unroll
    for (int i = 0; i < NR; ++i) {
      const int d = rg + 8 * i;
      if (d < DP) {
        const float r = sr[d], k = sk[d], w = sw[d];
        o0 += s[i][0] * r;
        o1 += s[i][1] * r;
        s[i][0] = s[i][0] * w + k * v0;
        s[i][1] = s[i][1] * w + k * v1;
      }
    }
#pragma unroll
    for (int o = 4; o < 32; o <<= 1) {
      o0 += __shfl_xor_sync(0xffffffffu, o0, o);
      o1 += __shfl_xor_sync(0xffffffffu, o1, o);
    }
    if (rg == 0) *reinterpret_cast<float2*>(p.o + row * p.ld_o + (size_t)h * DP + col) = make_float2(o0 + bonus * v0, o1 + bonus * v1);
    __syncwarp();
  }
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int d = rg + 8 * i;
    if (d < DP) *reinterpret_cast<float2*>(st + (size_t)d * DP) = make_float2(s[i][0], s[i][1]);
  }
}

// ----------------------------------------------------------------------------------------------- one token, fused --
// A CTA takes a head of a row, its warps eight value columns each; the state's loads are on their way while the decays are formed.
constexpr int WS_THREADS = 512;

template <typename T, int NR>
__global__ void __launch_bounds__(WS_THREADS)
wkv_step_kernel(const nfn_wkv_step_args p) {
  extern __shared__ float ws_low[];                        // [rank_p] tanh of the inner decay projection
  __shared__ float sr[8 * NR], sk[8 * NR], sw[8 * NR], sb[8 * NR], red[WS_THREADS / 32];
  const nfn_row_tile tile = p.tiles[blockIdx.y];
  if (tile.slot < 0) return;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, rg = lane >> 2, cl = lane & 3;
  const int h = blockIdx.x, DP = p.dim_p, HD = p.heads * DP, row = tile.row0;
  const int col = warp * WR_COLS + 2 * cl;
  float* st = p.state + ((size_t)tile.slot * p.heads + h) * DP * DP + col;
  float s[NR][2];
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int d = rg + 8 * i;
    float2 v = make_float2(0.f, 0.f);
    if (tile.e_pos0 > 0 && d < DP) v = *reinterpret_cast<const float2*>(st + (size_t)d * DP);
    s[i][0] = v.x;
    s[i][1] = v.y;
  }
  const T* x = static_cast<const T*>(p.rkvg) + (size_t)row * p.ld_rkvg + (size_t)h * DP;
  // whatever else the token brings is asked for before anything waits
  const T v0_raw = x[2 * HD + col], v1_raw = x[2 * HD + col + 1], g0_raw = x[3 * HD + col], g1_raw = x[3 * HD + col + 1];
  const __nv_bfloat16* weight = static_cast<const __nv_bfloat16*>(p.weight) + (size_t)h * DP;
  const __nv_bfloat16 n0 = weight[col], n1 = weight[col + 1];
  for (int i = tid; i < p.rank_p; i += blockDim.x) ws_low[i] = tanhf(p.low[(size_t)row * p.ld_low + i]);
  __syncthreads();
  // decays: four threads per channel share the contraction
  for (int q = tid; q < 4 * DP; q += blockDim.x) {
    const int d = q >> 2, part = q & 3;
    const __nv_bfloat16* w2 = static_cast<const __nv_bfloat16*>(p.w2) + (size_t)(h * DP + d) * p.ld_w2;
    float z = 0.f;
    for (int i = part * 4; i < p.rank_p; i += 16) {
      const float4 w = load4(w2 + i);
      z += w.x * ws_low[i] + w.y * ws_low[i + 1] + w.z * ws_low[i + 2] + w.w * ws_low[i + 3];
    }
    z += __shfl_xor_sync(0xffffffffu, z, 1);
    z += __shfl_xor_sync(0xffffffffu, z, 2);
    if (part == 0) {
      const float r = to_float(x[d]), k = to_float(x[HD + d]);
      sr[d] = r;
      sk[d] = k;
      sb[d] = r * (k * __bfloat162float(static_cast<const __nv_bfloat16*>(p.u)[(size_t)h * DP + d]));
      sw[d] = wkv_decay(z + __bfloat162float(static_cast<const __nv_bfloat16*>(p.w0)[(size_t)h * DP + d]));
    }
  }
  __syncthreads();
  float bonus = 0.f;
  for (int d = lane; d < DP; d += 32) bonus += sb[d];
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) bonus += __shfl_xor_sync(0xffffffffu, bonus, o);
  const float v0 = to_float(v0_raw), v1 = to_float(v1_raw);
  float o0 = 0.f, o1 = 0.f;
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int d = rg + 8 * i;
    if (d < DP) {
      const float r = sr[d], k = sk[d], w = sw[d];
      o0 += s[i][0] * r;
      o1 += s[i][1] * r;
      *reinterpret_cast<float2*>(st + (size_t)d * DP) = make_float2(s[i][0] * w + k * v0, s[i][1] * w + k * v1);
    }
  }
#pragma unroll
  for (int o = 4; o < 32; o <<= 1) {
    o0 += __shfl_xor_sync(0xffffffffu, o0, o);
    o1 += __shfl_xor_sync(0xffffffffu, o1, o);
  }
  o0 += bonus * v0;
  o1 += bonus * v1;
  float ss = o0 * o0 + o1 * o1;                                   // over the warp's eight columns
  ss += __shfl_xor_sync(0xffffffffu, ss, 1);
  ss += __shfl_xor_sync(0xffffffffu, ss, 2);
  if (lane == 0) red[warp] = ss;
  __syncthreads();
  ss = 0.f;
  for (int w = 0; w < DP / WR_COLS; ++w) ss += red[w];
  if (rg == 0) {
    const float r = 1.f / sqrtf(ss / (float)p.dim + p.eps);
    const float g0 = to_float(g0_raw), g1 = to_float(g1_raw);
    T* out = static_cast<T*>(p.out) + (size_t)row * p.ld_out + (size_t)h * DP + col;
    out[0] = from_float<T>(o0 * r * __bfloat162float(n0) * g0 * sigmoid_for<T>(g0));
    out[1] = from_float<T>(o1 * r * __bfloat162float(n1) * g1 * sigmoid_for<T>(g1));
  }
}

__global__ void __launch_bounds__(256)
tanh_split_kernel(const float* __restrict__ in, int ld_in, __nv_bfloat16* __restrict__ out, int ld_out, int rows, int rank_p) {
  const int i = blockIdx.x * 256 + threadIdx.x;
  if (i >= rows * rank_p) return;
  const int r = i / rank_p, c = i % rank_p;
  const float t = tanhf(in[(size_t)r * ld_in + c]);
  const __nv_bfloat16 hi = __float2bfloat16(t);
  out[(size_t)r * ld_out + c] = hi;
  out[(size_t)r * ld_out + rank_p + c] = __float2bfloat16(t - __bfloat162float(hi));
}
__global__ void __launch_bounds__(256)
tanh_rows_kernel(const float* __restrict__ in, int ld_in, float* __restrict__ out, int ld_out, int rows, int rank_p) {
  const int i = blockIdx.x * 256 + threadIdx.x;
  if (i < rows * rank_p) out[(size_t)(i / rank_p) * ld_out + i % rank_p] = tanhf(in[(size_t)(i / rank_p) * ld_in + i % rank_p]);
}

template <typename T, int NR>
static int launch_wkv_rows(const nfn_wkv_args& a, cudaStream_t st) {
  const size_t smem = (size_t)WR_WARPS * 3 * a.dim_p * sizeof(float);
  wkv_rows_kernel<T, NR><<<dim3(ceil_div(a.dim_p, WR_WARPS * WR_COLS), a.heads, a.n_seqs), WR_WARPS * 32, smem, st>>>(a);
  return launch_check("wkv_rows");
}
template <typename T>
static int pick_wkv_rows(const nfn_wkv_args& a, cudaStream_t st) {
  if (a.dim_p <= 64) return launch_wkv_rows<T, 8>(a, st);
  if (a.dim_p <= 128) return launch_wkv_rows<T, 16>(a, st);
  if (a.dim_p <= 256) return launch_wkv_rows<T, 32>(a, st);
  return launch_wkv_rows<T, 64>(a, st);
}

template <typename T>
static int launch_wkv_step(const nfn_wkv_step_args& a, cudaStream_t st) {
  const dim3 grid(a.heads, a.rows);
  const int threads = a.dim_p / WR_COLS * 32;
  const size_t smem = (size_t)a.rank_p * sizeof(float);
  if (a.dim_p <= 64) wkv_step_kernel<T, 8><<<grid, threads, smem, st>>>(a);
  else wkv_step_kernel<T, 16><<<grid, threads, smem, st>>>(a);
  return launch_check("wkv_step");
}

const char* wkv_args_problem(const nfn_wkv_args& a) {
  if (a.heads <= 0 || (a.dim_p & 15) || a.dim <= 0 || a.dim > a.dim_p) return "wkv: head sizes must be padded to multiples of 16";
  if (a.dim_p > 512) return "wkv: more than 512 channels per head";
  if (a.heads > 65535 || a.n_seqs > 65535) return "wkv: too many heads or sequences for one launch";
  if (!a.rkv || !a.z || !a.w0 || !a.u || !a.state || !a.o || !a.seqs) return "wkv: null operand";
  if ((a.ld_o & 3) || (a.ld_z & 3) || (a.ld_rkv & 7)) return "wkv: misaligned rows";
  return nullptr;
}

}  // namespace nfn

using namespace nfn;

extern "C" int nfn_shift_rows(const nfn_shift_args* args, nfn_stream_t stream) {
  if (!args) return fail(-1, "shift_rows: null args");
  const nfn_shift_args& a = *args;
  if (a.n_tiles <= 0) return 0;
  if ((a.ld & 15) || a.n < 1 || a.n > SH_MAX || (a.out_stride & 7)) return fail(-1, "shift_rows: one to eight outputs of rows padded to multiples of 16");
  const dim3 grid(a.n_tiles, ceil_div(a.ld, SH_THREADS * 4));
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (a.f32) shift_rows_kernel<float, float><<<grid, SH_THREADS, 0, st>>>(a);
  else if (a.src_act) shift_rows_kernel<__nv_bfloat16, __nv_bfloat16><<<grid, SH_THREADS, 0, st>>>(a);
  else shift_rows_kernel<float, __nv_bfloat16><<<grid, SH_THREADS, 0, st>>>(a);
  return launch_check("shift_rows");
}

extern "C" int nfn_wkv_rows(const nfn_wkv_args* args, nfn_stream_t stream) {
  if (!args) return fail(-1, "wkv: null args");
  if (args->n_seqs <= 0) return 0;
  if (const char* why = wkv_args_problem(*args)) return fail(-1, why);
  return args->f32 ? pick_wkv_rows<float>(*args, static_cast<cudaStream_t>(stream)) : pick_wkv_rows<__nv_bfloat16>(*args, static_cast<cudaStream_t>(stream));
}

extern "C" int nfn_tanh_split(int f32, const float* in, int ld_in, void* out, int ld_out, int rows, int rank_p, nfn_stream_t stream) {
  if (rows <= 0 || rank_p <= 0) return 0;
  if ((long long)rows * rank_p > 0x7fffff00LL) return fail(-1, "tanh_split: too many values for one launch");
  const int blocks = ceil_div(rows * rank_p, 256);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (f32) tanh_rows_kernel<<<blocks, 256, 0, st>>>(in, ld_in, static_cast<float*>(out), ld_out, rows, rank_p);
  else tanh_split_kernel<<<blocks, 256, 0, st>>>(in, ld_in, static_cast<__nv_bfloat16*>(out), ld_out, rows, rank_p);
  return launch_check("tanh_split");
}

extern "C" int nfn_wkv_step_fits(int rows, int dim_p) { return dim_p <= WS_THREADS / 32 * WR_COLS && rows <= 65535; }

extern "C" int nfn_wkv_step(const nfn_wkv_step_args* args, nfn_stream_t stream) {
  if (!args) return fail(-1, "wkv step: null args");
  const nfn_wkv_step_args& a = *args;
  if (a.rows <= 0) return 0;
  if (a.heads <= 0 || (a.dim_p & 15) || a.dim > a.dim_p || !nfn_wkv_step_fits(a.rows, a.dim_p)) return fail(-1, "wkv step: heads of at most 128 channels, padded to multiples of 16, and at most 65535 rows");
  if ((a.rank_p & 15) || a.rank_p <= 0 || a.rank_p > 8192 || (a.ld_w2 & 3) || (a.ld_rkvg & 7)) return fail(-1, "wkv step: misaligned rows");
  return a.f32 ? launch_wkv_step<float>(a, static_cast<cudaStream_t>(stream)) : launch_wkv_step<__nv_bfloat16>(a, static_cast<cudaStream_t>(stream));
}
