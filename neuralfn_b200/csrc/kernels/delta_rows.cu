// Gated delta rule with a decay per key channel, token after token: single tokens, short portions, and any length in 32-bit mode.
// (Prompt portions in bf16 take the chunked form of delta_chunk.cu.)
//
// The columns of a head's state never meet: S^T k, the correction and the read-out of value column c use S[:, c] only. So a warp owns
// eight columns of one head for all tokens of its entry - four lanes across, two columns each, eight lanes down the key channels -
// keeps them in registers from the first token to the last, and needs nothing but shuffles. Everything past the convolved q, k, v is
// fp32: unit vectors, decays (softplus, exponentials), step sizes, the state.
#include "common.h"
#include "delta.cuh"

namespace nfn {

constexpr int DR_WARPS = 4, DR_COLS = 8;

// NR: key channels per lane (dim_p <= 8 NR)
template <typename T, int NR>
__global__ void __launch_bounds__(DR_WARPS * 32)
delta_rows_kernel(const nfn_delta_args p) {
  extern __shared__ float dr_smem[];                        // [DR_WARPS][3][dim_p]: q, k, g of the token at hand
  const nfn_seq_rows seq = p.seqs[blockIdx.z];
  if (seq.slot < 0) return;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, rg = lane >> 2, cl = lane & 3;
  const int h = blockIdx.y, hk = h / (p.heads / p.kv_heads), DP = p.dim_p, VP = p.vdim_p;
  const int col0 = (blockIdx.x * DR_WARPS + warp) * DR_COLS;
  if (col0 >= VP) return;
  const int col = col0 + 2 * cl;
  float* sq = dr_smem + warp * 3 * DP;
  float *sk = sq + DP, *sg = sk + DP;
  float* st = p.state + ((size_t)seq.slot * p.heads + h) * DP * VP + col;
  float s[NR][2];
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int d = rg + 8 * i;
    float2 v = make_float2(0.f, 0.f);
    if (seq.pos0 > 0 && d < DP) v = *reinterpret_cast<const float2*>(st + (size_t)d * VP);
    s[i][0] = v.x;
    s[i][1] = v.y;
  }
  const float rate = -expf(__bfloat162float(static_cast<const __nv_bfloat16*>(p.a_log)[h]));
  const __nv_bfloat16* bias = static_cast<const __nv_bfloat16*>(p.dt_bias) + (size_t)h * DP;
  const float q_scale = 1.f / sqrtf((float)p.dim);
  const int off_k = p.kv_heads * DP, off_v = 2 * off_k;
  for (int t = 0; t < seq.n; ++t) {
    const size_t row = (size_t)(seq.row0 + t);
    const T* x = static_cast<const T*>(p.qkv) + row * p.ld_qkv;
    const float* dec = p.decay + row * p.ld_decay + (size_t)h * DP;
    float nq = 0.f, nk = 0.f;
    for (int d = lane * 4; d < DP; d += 128) {
      const float4 q = load4(x + hk * DP + d), k = load4(x + off_k + hk * DP + d), z = load4(dec + d), b = load4(bias + d);
      nq += q.x * q.x + q.y * q.y + q.z * q.z + q.w * q.w;
      nk += k.x * k.x + k.y * k.y + k.z * k.z + k.w * k.w;
      store4(sq + d, q);
      store4(sk + d, k);
      store4(sg + d, make_float4(delta_decay(z.x + b.x, rate), delta_decay(z.y + b.y, rate), delta_decay(z.z + b.z, rate), delta_decay(z.w + b.w, rate)));
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      nq += __shfl_xor_sync(0xffffffffu, nq, o);
      nk += __shfl_xor_sync(0xffffffffu, nk, o);
    }
    const float fq = q_scale / sqrtf(nq + p.unit_eps), fk = 1.f / sqrtf(nk + p.unit_eps);
    const float beta = sigmoid_exact(to_float(static_cast<const T*>(p.beta)[row * p.ld_beta + h]));
    const float v0 = to_float(x[off_v + h * VP + col]), v1 = to_float(x[off_v + h * VP + col + 1]);
    __syncwarp();
    float a0 = 0.f, a1 = 0.f;
#pragma unroll
    for (int i = 0; i < NR; ++i) {
      const int d = rg + 8 * i;
      if (d < DP) {
        const float g = sg[d], k = sk[d] * fk;
        s[i][0] *= g;
        s[i][1] *= g;
        a0 += s[i][0] * k;
        a1 += s[i][1] * k;
      }
    }
#pragma unroll
    for (int o = 4; o < 32; o <<= 1) {
      a0 += __shfl_xor_sync(0xffffffffu, a0, o);
      a1 += __shfl_xor_sync(0xffffffffu, a1, o);
    }
    const float u0 = beta * (v0 - a0), u1 = beta * (v1 - a1);
    float o0 = 0.f, o1 = 0.f;
#pragma unroll
    for (int i = 0; i < NR; ++i) {
      const int d = rg + 8 * i;
      if (d < DP) {
        const float k = sk[d] * fk, q = sq[d] * fq;
        s[i][0] += k * u0;
        s[i][1] += k * u1;
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

// One token per sequence with everything around the rule fused (decoding). A CTA takes a head of a row, its warps eight value columns each; the
// state's loads are on their way while the convolutions and decays are formed.
constexpr int STEP_THREADS = 512;

template <typename T, int NR>
__global__ void __launch_bounds__(STEP_THREADS)
delta_step_kernel(const nfn_delta_step_args p) {
  __shared__ float sq[8 * NR], sk[8 * NR], sg[8 * NR], sv[STEP_THREADS / 4], red[STEP_THREADS / 32];
  const nfn_row_tile tile = p.tiles[blockIdx.y];
  if (tile.slot < 0) return;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, rg = lane >> 2, cl = lane & 3;
  const int h = blockIdx.x, rep = p.heads / p.kv_heads, hk = h / rep, DP = p.dim_p, VP = p.vdim_p, row = tile.row0;
  const int col = warp * DR_COLS + 2 * cl;
  float* st = p.state + ((size_t)tile.slot * p.heads + h) * DP * VP + col;
  float s[NR][2];
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int d = rg + 8 * i;
    float2 v = make_float2(0.f, 0.f);
    if (tile.e_pos0 > 0 && d < DP) v = *reinterpret_cast<const float2*>(st + (size_t)d * VP);
    s[i][0] = v.x;
    s[i][1] = v.y;
  }
  const T* in = static_cast<const T*>(p.in) + (size_t)row * p.ld_in;
  const T* gate = static_cast<const T*>(p.gate) + (size_t)row * p.ld_gate + (size_t)h * VP + col;
  // whatever else the token brings is asked for before anything waits
  const T z0 = gate[0], z1 = gate[1], beta_raw = in[p.off_beta + h];
  const __nv_bfloat16 w0 = static_cast<const __nv_bfloat16*>(p.weight)[col], w1 = static_cast<const __nv_bfloat16*>(p.weight)[col + 1];
  const __nv_bfloat16 rate_raw = static_cast<const __nv_bfloat16*>(p.a_log)[h];
  const int dd = blockDim.x - 1 - tid;                            // decays from the last thread on: the first ones have the convolutions
  const float dec_raw = dd < DP ? p.decay[(size_t)row * p.ld_decay + (size_t)h * DP + dd] : 0.f;
  const __nv_bfloat16 dt_raw = dd < DP ? static_cast<const __nv_bfloat16*>(p.dt_bias)[(size_t)h * DP + dd] : __float2bfloat16(0.f);
  // ---- four channels of q, k or v per thread: convolution, SiLU, history ----
  const int quads = (2 * DP + VP) / 4, C = 2 * p.kv_heads * DP + p.heads * VP, taps = p.taps;
  for (int u = tid; u < quads; u += blockDim.x) {
    const int c = 4 * u, part = c < DP ? 0 : c < 2 * DP ? 1 : 2;
    const int ch = part == 0 ? hk * DP + c : part == 1 ? (p.kv_heads + hk) * DP + c - DP : 2 * p.kv_heads * DP + h * VP + c - 2 * DP;
    const bool keeper = part == 2 || h % rep == 0;            // one head of a group leaves its q and k history
    const T* old = static_cast<const T*>(p.history) + (size_t)tile.parity * p.history_half + (size_t)tile.slot * (taps - 1) * C + ch;
    T* next = static_cast<T*>(p.history) + (size_t)(1 - tile.parity) * p.history_half + (size_t)tile.slot * (taps - 1) * C + ch;
    const __nv_bfloat16* w = static_cast<const __nv_bfloat16*>(p.conv) + ch;
    const float4 now = load4(in + ch), w_now = load4(w + (size_t)(taps - 1) * C);
    float4 y = make_float4(w_now.x * now.x, w_now.y * now.y, w_now.z * now.z, w_now.w * now.w);
    for (int t0 = 0; t0 < taps - 1; t0 += 3) {                  // three history rows at a time, loads before stores
      float4 f[3], wt[3];
#pragma unroll
      for (int e = 0; e < 3; ++e) {
        const int t = t0 + e;
        const bool live = t < taps - 1 && tile.e_pos0 - (taps - 1) + t >= 0;
        f[e] = live ? load4(old + (size_t)t * C) : make_float4(0.f, 0.f, 0.f, 0.f);
        wt[e] = live ? load4(w + (size_t)t * C) : make_float4(0.f, 0.f, 0.f, 0.f);
      }
#pragma unroll
      for (int e = 0; e < 3; ++e) {
        const int t = t0 + e;
        y.x += wt[e].x * f[e].x; y.y += wt[e].y * f[e].y; y.z += wt[e].z * f[e].z; y.w += wt[e].w * f[e].w;
        if (keeper && t > 0 && t < taps - 1) store4(next + (size_t)(t - 1) * C, f[e]);
      }
    }
    if (keeper && taps > 1) store4(next + (size_t)(taps - 2) * C, now);
    float* dst = part == 0 ? sq + c : part == 1 ? sk + c - DP : sv + c - 2 * DP;
    dst[0] = y.x * sigmoid_for<T>(y.x); dst[1] = y.y * sigmoid_for<T>(y.y); dst[2] = y.z * sigmoid_for<T>(y.z); dst[3] = y.w * sigmoid_for<T>(y.w);
  }
  const float rate = -expf(__bfloat162float(rate_raw));
  if (dd < DP) sg[dd] = delta_decay(dec_raw + __bfloat162float(dt_raw), rate);
  for (int d = dd + blockDim.x; d < DP; d += blockDim.x)
    sg[d] = delta_decay(p.decay[(size_t)row * p.ld_decay + (size_t)h * DP + d] + __bfloat162float(static_cast<const __nv_bfloat16*>(p.dt_bias)[(size_t)h * DP + d]), rate);
  __syncthreads();
  float nq = 0.f, nk = 0.f;
  for (int d = lane; d < DP; d += 32) {
    nq += sq[d] * sq[d];
    nk += sk[d] * sk[d];
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    nq += __shfl_xor_sync(0xffffffffu, nq, o);
    nk += __shfl_xor_sync(0xffffffffu, nk, o);
  }
  const float fq = 1.f / (sqrtf((float)p.dim) * sqrtf(nq + p.unit_eps)), fk = 1.f / sqrtf(nk + p.unit_eps);
  float a0 = 0.f, a1 = 0.f;
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int d = rg + 8 * i;
    if (d < DP) {
      const float g = sg[d], k = sk[d] * fk;
      s[i][0] *= g;
      s[i][1] *= g;
      a0 += s[i][0] * k;
      a1 += s[i][1] * k;
    }
  }
#pragma unroll
  for (int o = 4; o < 32; o <<= 1) {
    a0 += __shfl_xor_sync(0xffffffffu, a0, o);
    a1 += __shfl_xor_sync(0xffffffffu, a1, o);
  }
  const float beta = sigmoid_exact(to_float(beta_raw));
  const float u0 = beta * (sv[col] - a0), u1 = beta * (sv[col + 1] - a1);
  float o0 = 0.f, o1 = 0.f;
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int d = rg + 8 * i;
    if (d < DP) {
      const float k = sk[d] * fk, q = sq[d] * fq;
      s[i][0] += k * u0;
      s[i][1] += k * u1;
      *reinterpret_cast<float2*>(st + (size_t)d * VP) = make_float2(s[i][0], s[i][1]);
      o0 += s[i][0] * q;
      o1 += s[i][1] * q;
    }
  }
#pragma unroll
  for (int o = 4; o < 32; o <<= 1) {
    o0 += __shfl_xor_sync(0xffffffffu, o0, o);
    o1 += __shfl_xor_sync(0xffffffffu, o1, o);
  }
  float ss = o0 * o0 + o1 * o1;                                   // over the warp's eight columns
  ss += __shfl_xor_sync(0xffffffffu, ss, 1);
  ss += __shfl_xor_sync(0xffffffffu, ss, 2);
  if (lane == 0) red[warp] = ss;
  __syncthreads();
  ss = 0.f;
  for (int w = 0; w < VP / DR_COLS; ++w) ss += red[w];
  if (rg == 0) {
    const float r = 1.f / sqrtf(ss / (float)p.vdim + p.norm_eps);
    T* out = static_cast<T*>(p.out) + (size_t)row * p.ld_out + (size_t)h * VP + col;
    out[0] = from_float<T>(o0 * r * __bfloat162float(w0) * sigmoid_for<T>(to_float(z0)));
    out[1] = from_float<T>(o1 * r * __bfloat162float(w1) * sigmoid_for<T>(to_float(z1)));
  }
}

template <typename T>
static int launch_delta_step(const nfn_delta_step_args& a, cudaStream_t st) {
  const dim3 grid(a.heads, a.rows);
  const int threads = a.vdim_p / DR_COLS * 32;
  if (a.dim_p <= 64) delta_step_kernel<T, 8><<<grid, threads, 0, st>>>(a);
  else if (a.dim_p <= 128) delta_step_kernel<T, 16><<<grid, threads, 0, st>>>(a);
  else delta_step_kernel<T, 32><<<grid, threads, 0, st>>>(a);
  return launch_check("delta_step");
}

// One warp per (row, head): o / rms(o) * weight * sigmoid(gate), with SILU also times gate. Weights weight_pitch apart for every head (0: shared).
template <typename T, bool SILU>
__global__ void __launch_bounds__(256)
delta_out_kernel(const float* __restrict__ o, int ld_o, const T* __restrict__ gate, int ld_gate, const __nv_bfloat16* __restrict__ weight, int weight_pitch,
                 float eps, T* __restrict__ out, int ld_out, int rows, int heads, int vdim, int vdim_p) {
  const long long item = (long long)blockIdx.x * 8 + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (item >= (long long)rows * heads) return;
  const int row = (int)(item / heads), h = (int)(item % heads);
  const float* src = o + (size_t)row * ld_o + (size_t)h * vdim_p;
  float ss = 0.f;
  for (int c = lane * 4; c < vdim_p; c += 128) {
    const float4 f = load4(src + c);
    ss += f.x * f.x + f.y * f.y + f.z * f.z + f.w * f.w;
  }
#pragma unroll
  for (int s = 16; s > 0; s >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, s);
  const float r = 1.f / sqrtf(ss / (float)vdim + eps);
  const T* g = gate + (size_t)row * ld_gate + (size_t)h * vdim_p;
  T* dst = out + (size_t)row * ld_out + (size_t)h * vdim_p;
  for (int c = lane * 4; c < vdim_p; c += 128) {
    const float4 f = load4(src + c), z = load4(g + c);
    float4 w = load4(weight + (size_t)h * weight_pitch + c);
    if (SILU) { w.x *= z.x; w.y *= z.y; w.z *= z.z; w.w *= z.w; }
    store4(dst + c, make_float4(f.x * r * w.x * sigmoid_for<T>(z.x), f.y * r * w.y * sigmoid_for<T>(z.y), f.z * r * w.z * sigmoid_for<T>(z.z),
                                f.w * r * w.w * sigmoid_for<T>(z.w)));
  }
}

template <typename T, int NR>
static int launch_delta_rows(const nfn_delta_args& a, cudaStream_t st) {
  const size_t smem = (size_t)DR_WARPS * 3 * a.dim_p * sizeof(float);
  const dim3 grid(ceil_div(a.vdim_p, DR_WARPS * DR_COLS), a.heads, a.n_seqs);
  delta_rows_kernel<T, NR><<<grid, DR_WARPS * 32, smem, st>>>(a);
  return launch_check("delta_rows");
}

template <typename T>
static int pick_delta_rows(const nfn_delta_args& a, cudaStream_t st) {
  if (a.dim_p <= 64) return launch_delta_rows<T, 8>(a, st);
  if (a.dim_p <= 128) return launch_delta_rows<T, 16>(a, st);
  if (a.dim_p <= 256) return launch_delta_rows<T, 32>(a, st);
  return launch_delta_rows<T, 64>(a, st);
}

const char* delta_args_problem(const nfn_delta_args& a) {
  if (a.heads <= 0 || a.kv_heads <= 0 || a.heads % a.kv_heads) return "delta rule: heads must divide into query / key heads";
  if (((a.dim_p | a.vdim_p) & 15) || a.dim <= 0 || a.dim > a.dim_p) return "delta rule: head sizes must be padded to multiples of 16";
  if (a.dim_p > 512) return "delta rule: more than 512 key channels per head";
  if (a.heads > 65535 || a.n_seqs > 65535) return "delta rule: too many heads or sequences for one launch";
  if (!a.qkv || !a.beta || !a.decay || !a.a_log || !a.dt_bias || !a.state || !a.o || !a.seqs) return "delta rule: null operand";
  if ((a.ld_o & 3) || (a.ld_decay & 3) || (a.ld_qkv & 7)) return "delta rule: misaligned rows";
  return nullptr;
}

}  // namespace nfn

using namespace nfn;

extern "C" int nfn_delta_rows(const nfn_delta_args* args, nfn_stream_t stream) {
  if (!args) return fail(-1, "delta rule: null args");
  if (args->n_seqs <= 0) return 0;
  if (const char* why = delta_args_problem(*args)) return fail(-1, why);
  return args->f32 ? pick_delta_rows<float>(*args, static_cast<cudaStream_t>(stream)) : pick_delta_rows<__nv_bfloat16>(*args, static_cast<cudaStream_t>(stream));
}

extern "C" int nfn_delta_step_fits(int rows, int heads, int dim_p, int vdim_p) {
  return dim_p <= 256 && vdim_p <= STEP_THREADS / 32 * DR_COLS && (long long)rows * heads <= 2LL * sm_count();
}

extern "C" int nfn_delta_step(const nfn_delta_step_args* args, nfn_stream_t stream) {
  if (!args) return fail(-1, "delta step: null args");
  const nfn_delta_step_args& a = *args;
  if (a.rows <= 0) return 0;
  if (a.heads <= 0 || a.kv_heads <= 0 || a.heads % a.kv_heads || ((a.dim_p | a.vdim_p) & 15) || a.dim > a.dim_p || a.vdim > a.vdim_p)
    return fail(-1, "delta step: bad head sizes");
  if (!nfn_delta_step_fits(1, 1, a.dim_p, a.vdim_p)) return fail(-1, "delta step: at most 256 key and 128 value channels per head");
  if (a.taps < 1 || !a.conv || (a.taps > 1 && !a.history)) return fail(-1, "delta step: a convolution needs its weights and history");
  if (((a.ld_in | a.ld_decay | a.ld_out | a.ld_gate) & 7) || a.rows > 65535) return fail(-1, "delta step: misaligned rows, or too many");
  return a.f32 ? launch_delta_step<float>(a, static_cast<cudaStream_t>(stream)) : launch_delta_step<__nv_bfloat16>(a, static_cast<cudaStream_t>(stream));
}

template <typename T, bool SILU>
static void launch_head_out(const float* o, int ld_o, const void* gate, int ld_gate, const void* weight, int weight_pitch, float eps, void* out, int ld_out, int rows,
                            int heads, int vdim, int vdim_p, cudaStream_t st) {
  const unsigned blocks = (unsigned)(((long long)rows * heads + 7) / 8);
  delta_out_kernel<T, SILU><<<blocks, 256, 0, st>>>(o, ld_o, static_cast<const T*>(gate), ld_gate, static_cast<const __nv_bfloat16*>(weight), weight_pitch, eps,
                                                    static_cast<T*>(out), ld_out, rows, heads, vdim, vdim_p);
}

extern "C" int nfn_head_out(int f32, const float* o, int ld_o, const void* gate, int ld_gate, int gate_act, const void* weight, int weight_pitch, float eps, void* out,
                            int ld_out, int rows, int heads, int vdim, int vdim_p, nfn_stream_t stream) {
  if (rows <= 0) return 0;
  if ((vdim_p & 15) || vdim <= 0 || vdim > vdim_p || ((ld_o | ld_gate | ld_out | weight_pitch) & 7)) return fail(-1, "head_out: misaligned rows or head sizes");
  if (((long long)rows * heads + 7) / 8 > 0x7fffffffLL) return fail(-1, "head_out: too many rows for one launch");
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const bool silu = gate_act == NFN_ACT_SILU;
  auto run = f32 ? (silu ? launch_head_out<float, true> : launch_head_out<float, false>) : (silu ? launch_head_out<__nv_bfloat16, true> : launch_head_out<__nv_bfloat16, false>);
  run(o, ld_o, gate, ld_gate, weight, weight_pitch, eps, out, ld_out, rows, heads, vdim, vdim_p, st);
  return launch_check("head_out");
}

extern "C" int nfn_delta_out(int f32, const float* o, int ld_o, const void* gate, int ld_gate, const void* weight, float eps, void* out, int ld_out, int rows,
                             int heads, int vdim, int vdim_p, nfn_stream_t stream) {
  return nfn_head_out(f32, o, ld_o, gate, ld_gate, NFN_ACT_NONE, weight, 0, eps, out, ld_out, rows, heads, vdim, vdim_p, stream);
}
