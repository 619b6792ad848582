// Linear attention with a constant decay per head, S <- decay S + k v^T, o = S^T q: token after token (short portions, any length in 32-bit mode; prompt
// portions in bf16 take linear_chunk.cu), the norm and gate behind it, and the fused decode step. State and read-outs are fp32.
#include <algorithm>

#include "common.h"
#include "paged.cuh"

namespace nfn {

// --------------------------------------------------------------------------------------------- token after token --
// A warp owns eight value columns - four lanes across, two columns each, eight lanes down the key channels - from the first token of its entry to
// the last.
constexpr int LR_WARPS = 4, LR_COLS = 8;

// NR: key channels per lane (dim_p <= 8 NR)
template <typename T, int NR>
__global__ void __launch_bounds__(LR_WARPS * 32)
linear_rows_kernel(const nfn_linear_args p) {
  extern __shared__ float lr_smem[];                        // [LR_WARPS][2][dim_p]: q, k of the token at hand
  const nfn_seq_rows seq = p.seqs[blockIdx.z];
  if (seq.slot < 0) return;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, rg = lane >> 2, cl = lane & 3;
  const int h = blockIdx.y, DP = p.dim_p, VP = p.vdim_p, HD = p.heads * DP;
  const int col0 = (blockIdx.x * LR_WARPS + warp) * LR_COLS;
  if (col0 >= VP) return;
  const int col = col0 + 2 * cl;
  float *sq = lr_smem + warp * 2 * DP, *sk = sq + DP;
  float* st = p.state + ((size_t)seq.slot * p.heads + h) * DP * VP + col;
  const float w = p.powers[(size_t)h * (NFN_LINEAR_CHUNK + 1) + 1];
  float s[NR][2];
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int d = rg + 8 * i;
    float2 v = make_float2(0.f, 0.f);
    if (seq.pos0 > 0 && d < DP) v = *reinterpret_cast<const float2*>(st + (size_t)d * VP);
    s[i][0] = v.x;
    s[i][1] = v.y;
  }
  for (int t = 0; t < seq.n; ++t) {
    const size_t row = (size_t)(seq.row0 + t);
    const T* x = static_cast<const T*>(p.qkv) + row * p.ld_qkv + (size_t)h * DP;
    for (int d = lane * 4; d < DP; d += 128) {
      store4(sq + d, load4(x + d));
      store4(sk + d, load4(x + HD + d));
    }
    const T* v = static_cast<const T*>(p.qkv) + row * p.ld_qkv + 2 * HD + (size_t)h * VP + col;
    const float v0 = to_float(v[0]), v1 = to_float(v[1]);
    __syncwarp();
    float o0 = 0.f, o1 = 0.f;
#pragma unroll
    for (int i = 0; i < NR; ++i) {
      const int d = rg + 8 * i;
      if (d < DP) {
        const float q = sq[d], k = sk[d];
        s[i][0] = s[i][0] * w + k * v0;
        s[i][1] = s[i][1] * w + k * v1;
        o0 += s[i][0] * q;
        o1 += s[i][1] * q;
      }
    }
#pragma unroll
    for (int o = 4; o < 32; o <<= 1) {
      o0 += __shfl_xor_sync(0xffffffffu, o0, o);
      o1 += __shfl_xor_sync(0xffffffffu, o1, o);
    }
    if (rg == 0) *reinterpret_cast<float2*>(p.o + row * p.ld_o + (size_t)h * VP + col) = make_float2(o0, o1);
    __syncwarp();
  }
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int d = rg + 8 * i;
    if (d < DP) *reinterpret_cast<float2*>(st + (size_t)d * VP) = make_float2(s[i][0], s[i][1]);
  }
}

// ------------------------------------------------------------------------------------------- norm and gate of a row --
template <int THREADS>
__device__ __forceinline__ float row_sum(float v, float* red) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float t = 0.f;
#pragma unroll
  for (int i = 0; i < THREADS / 32; ++i) t += red[i];
  return t;
}

// out = o / rms(o) * weight * sigmoid(gate), `live` of the `cols` values counted by the mean (padding is zero)
template <typename T, int THREADS>
__device__ __forceinline__ void finish_row(const float* o, const T* gate, const __nv_bfloat16* weight, float eps, T* out, int cols, int live, float* red) {
  constexpr int KEEP = 4;                                   // pieces per thread that stay in registers
  float4 held[KEEP];
  float ss = 0.f;
  auto fetch = [&](int c) { return __ldcg(reinterpret_cast<const float4*>(o + c)); };
#pragma unroll
  for (int i = 0; i < KEEP; ++i) {
    const int c = 4 * (threadIdx.x + i * THREADS);
    held[i] = c < cols ? fetch(c) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
#pragma unroll
  for (int i = 0; i < KEEP; ++i) ss += held[i].x * held[i].x + held[i].y * held[i].y + held[i].z * held[i].z + held[i].w * held[i].w;
  for (int c = 4 * (threadIdx.x + KEEP * THREADS); c < cols; c += 4 * THREADS) {
    const float4 f = fetch(c);
    ss += f.x * f.x + f.y * f.y + f.z * f.z + f.w * f.w;
  }
  const float r = 1.f / sqrtf(row_sum<THREADS>(ss, red) / (float)live + eps);
  auto leave = [&](const float4& f, int c) {
    const float4 w = load4(weight + c), g = load4(gate + c);
    store4(out + c, make_float4(f.x * r * w.x * sigmoid_for<T>(g.x), f.y * r * w.y * sigmoid_for<T>(g.y), f.z * r * w.z * sigmoid_for<T>(g.z), f.w * r * w.w * sigmoid_for<T>(g.w)));
  };
#pragma unroll
  for (int i = 0; i < KEEP; ++i) {
    const int c = 4 * (threadIdx.x + i * THREADS);
    if (c < cols) leave(held[i], c);
  }
  for (int c = 4 * (threadIdx.x + KEEP * THREADS); c < cols; c += 4 * THREADS) leave(fetch(c), c);
}

constexpr int RO_THREADS = 256;
template <typename T>
__global__ void __launch_bounds__(RO_THREADS)
row_out_kernel(const float* __restrict__ o, int ld_o, const T* __restrict__ gate, int ld_gate, const __nv_bfloat16* __restrict__ weight, float eps, T* __restrict__ out,
               int ld_out, int cols, int live) {
  __shared__ float red[RO_THREADS / 32];
  const size_t r = blockIdx.x;
  finish_row<T, RO_THREADS>(o + r * ld_o, gate + r * ld_gate, weight, eps, out + r * ld_out, cols, live, red);
}

// ----------------------------------------------------------------------------------------------- one token, fused --
// A CTA takes a head of a row: VP / 4 threads across four value columns each, the others down the key channels, so that a row of the state is read in
// whole lines. The CTA that finishes last of its row applies the norm over all heads, weight and gate.
constexpr int LS_THREADS = 512, LS_MAX = 512, LS_AHEAD = 8;

template <typename T>
__global__ void __launch_bounds__(LS_THREADS)
linear_step_kernel(const nfn_linear_step_args p) {
  __shared__ float sq[LS_MAX], sk[LS_MAX], red[LS_THREADS / 32];
  __shared__ __align__(16) float part[4 * LS_THREADS];      // [groups][VP]
  __shared__ int sh_last;
  const nfn_row_tile tile = p.tiles[blockIdx.y];
  if (tile.slot < 0) return;
  const int tid = threadIdx.x, h = blockIdx.x, DP = p.dim_p, VP = p.vdim_p, HD = p.heads * DP, HV = p.heads * VP, row = tile.row0;
  const int quads = VP / 4, groups = min(LS_THREADS / quads, DP), cg = tid / quads, c = tid % quads * 4;
  const bool on = cg < groups;
  float* st = p.state + ((size_t)tile.slot * p.heads + h) * DP * VP + c;
  const bool held = tile.e_pos0 > 0;
  float4 s[LS_AHEAD];
  auto fetch = [&](int d0) {
#pragma unroll
    for (int i = 0; i < LS_AHEAD; ++i) {
      const int d = d0 + i * groups;
      s[i] = on && held && d < DP ? load4(st + (size_t)d * VP) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
  };
  fetch(cg);                                                // on its way while the token's vectors are formed
  const T* x = static_cast<const T*>(p.qkvg) + (size_t)row * p.ld_qkvg;
  float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
  if (on) v = load4(x + 2 * HD + h * VP + c);
  for (int d = tid; d < DP; d += LS_THREADS) {
    const float q = to_float(x[h * DP + d]), k = to_float(x[HD + h * DP + d]);
    sq[d] = q * sigmoid_for<T>(q);
    sk[d] = k * sigmoid_for<T>(k);
  }
  const float w = p.powers[(size_t)h * (NFN_LINEAR_CHUNK + 1) + 1];
  v.x *= sigmoid_for<T>(v.x); v.y *= sigmoid_for<T>(v.y); v.z *= sigmoid_for<T>(v.z); v.w *= sigmoid_for<T>(v.w);
  __syncthreads();
  if (on) {
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int d0 = cg; d0 < DP; d0 += LS_AHEAD * groups) {
      if (d0 != cg) fetch(d0);
#pragma unroll
      for (int i = 0; i < LS_AHEAD; ++i) {
        const int d = d0 + i * groups;
        if (d >= DP) break;
        const float q = sq[d], k = sk[d];
        const float4 f = make_float4(s[i].x * w + k * v.x, s[i].y * w + k * v.y, s[i].z * w + k * v.z, s[i].w * w + k * v.w);
        store4(st + (size_t)d * VP, f);
        o.x += f.x * q; o.y += f.y * q; o.z += f.z * q; o.w += f.w * q;
      }
    }
    store4(part + cg * VP + c, o);
  }
  __syncthreads();
  float* o_row = p.o + (size_t)row * p.ld_o;
  for (int i = tid; i < VP; i += LS_THREADS) {
    float t = 0.f;
    for (int g = 0; g < groups; ++g) t += part[g * VP + i];
    o_row[h * VP + i] = t;
  }
  __threadfence();
  __syncthreads();
  if (tid == 0) sh_last = atomicAdd(&p.counters[row], 1) == p.heads - 1;
  __syncthreads();
  if (!sh_last) return;
  __threadfence();
  finish_row<T, LS_THREADS>(o_row, x + 2 * HD + HV, static_cast<const __nv_bfloat16*>(p.weight), p.eps, static_cast<T*>(p.out) + (size_t)row * p.ld_out, HV, p.heads * p.vdim, red);
  if (tid == 0) p.counters[row] = 0;
}

template <typename T, int NR>
static int launch_linear_rows(const nfn_linear_args& a, cudaStream_t st) {
  const size_t smem = (size_t)LR_WARPS * 2 * a.dim_p * sizeof(float);
  linear_rows_kernel<T, NR><<<dim3(ceil_div(a.vdim_p, LR_WARPS * LR_COLS), a.heads, a.n_seqs), LR_WARPS * 32, smem, st>>>(a);
  return launch_check("linear_rows");
}
template <typename T>
static int pick_linear_rows(const nfn_linear_args& a, cudaStream_t st) {
  if (a.dim_p <= 64) return launch_linear_rows<T, 8>(a, st);
  if (a.dim_p <= 128) return launch_linear_rows<T, 16>(a, st);
  if (a.dim_p <= 256) return launch_linear_rows<T, 32>(a, st);
  return launch_linear_rows<T, 64>(a, st);
}

const char* linear_args_problem(const nfn_linear_args& a) {
  if (a.heads <= 0 || ((a.dim_p | a.vdim_p) & 15) || a.dim_p <= 0 || a.vdim_p <= 0) return "linear attention: head sizes must be padded to multiples of 16";
  if (a.dim_p > 512) return "linear attention: more than 512 key channels per head";
  if (a.heads > 65535 || a.n_seqs > 65535) return "linear attention: too many heads or sequences for one launch";
  if (!a.qkv || !a.powers || !a.state || !a.o || !a.seqs) return "linear attention: null operand";
  if ((a.ld_o & 3) || (a.ld_qkv & 7)) return "linear attention: misaligned rows";
  return nullptr;
}

}  // namespace nfn

using namespace nfn;

extern "C" int nfn_linear_rows(const nfn_linear_args* args, nfn_stream_t stream) {
  if (!args) return fail(-1, "linear attention: null args");
  if (args->n_seqs <= 0) return 0;
  if (const char* why = linear_args_problem(*args)) return fail(-1, why);
  return args->f32 ? pick_linear_rows<float>(*args, static_cast<cudaStream_t>(stream)) : pick_linear_rows<__nv_bfloat16>(*args, static_cast<cudaStream_t>(stream));
}

extern "C" int nfn_row_out(int f32, const float* o, int ld_o, const void* gate, int ld_gate, const void* weight, float eps, void* out, int ld_out, int rows, int cols, int live,
                           nfn_stream_t stream) {
  if (rows <= 0) return 0;
  if ((cols & 15) || live <= 0 || live > cols || (ld_o & 3) || ((ld_gate | ld_out) & 7)) return fail(-1, "row_out: rows padded to multiples of 16");
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const __nv_bfloat16* w = static_cast<const __nv_bfloat16*>(weight);
  if (f32) row_out_kernel<float><<<rows, RO_THREADS, 0, st>>>(o, ld_o, static_cast<const float*>(gate), ld_gate, w, eps, static_cast<float*>(out), ld_out, cols, live);
  else row_out_kernel<__nv_bfloat16><<<rows, RO_THREADS, 0, st>>>(o, ld_o, static_cast<const __nv_bfloat16*>(gate), ld_gate, w, eps, static_cast<__nv_bfloat16*>(out), ld_out, cols, live);
  return launch_check("row_out");
}

extern "C" int nfn_linear_step_fits(int rows, int dim_p, int vdim_p) { return dim_p <= LS_MAX && vdim_p <= LS_MAX && rows <= 65535; }

extern "C" int nfn_linear_step(const nfn_linear_step_args* args, nfn_stream_t stream) {
  if (!args) return fail(-1, "linear step: null args");
  const nfn_linear_step_args& a = *args;
  if (a.rows <= 0) return 0;
  if (a.heads <= 0 || ((a.dim_p | a.vdim_p) & 15) || a.dim_p <= 0 || a.vdim <= 0 || a.vdim > a.vdim_p || !nfn_linear_step_fits(a.rows, a.dim_p, a.vdim_p))
    return fail(-1, "linear step: heads of at most 512 channels, padded to multiples of 16, and at most 65535 rows");
  if (!a.qkvg || !a.powers || !a.state || !a.o || !a.counters || !a.weight || !a.out || !a.tiles) return fail(-1, "linear step: null operand");
  if ((a.ld_o & 3) || ((a.ld_qkvg | a.ld_out) & 7)) return fail(-1, "linear step: misaligned rows");
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (a.f32) linear_step_kernel<float><<<dim3(a.heads, a.rows), LS_THREADS, 0, st>>>(a);
  else linear_step_kernel<__nv_bfloat16><<<dim3(a.heads, a.rows), LS_THREADS, 0, st>>>(a);
  return launch_check("linear_step");
}
