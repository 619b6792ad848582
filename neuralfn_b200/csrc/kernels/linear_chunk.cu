// Linear attention with a constant decay w per head over prompt portions, 64 tokens at a time on the tensor cores (bf16 activations, fp32 state).
//
// With S the state before a chunk of n tokens, token r of it reads O_r = w^(r + 1) S^T q_r + sum_(j <= r) w^(r - j) (q_r . k_j) v_j and the next state is
// S' = w^n S + sum_j w^(n - 1 - j) k_j v_j^T. Every product's operands are the bf16 values as projected, or fp32 values (state, decayed scores, decayed
// values) as the sum of two bf16 numbers.
//
// A CTA takes one head and 64 of its value columns and walks the chunks; each of its four warps keeps the state of 16 columns, transposed, in mma.sync
// accumulators from the first chunk to the last: as they stand they are the second operand of the read-out S^T q. The scores of a chunk are
// formed once per CTA, 16 rows per warp, and cross shared memory. Queries, keys and values of the next chunk arrive (cp.async) while
// this one is in use. Where heads and columns leave SMs idle, a long sequence runs in segments side by side, after a pass that forms the
// state each of them adds.
#include <algorithm>

#include "chunk_scan.cuh"
#include "common.h"
#include "paged.cuh"

namespace nfn {

constexpr int LC_T = NFN_LINEAR_CHUNK, LC_WARPS = 4, LC_THREADS = LC_WARPS * 32, LC_COLS = 16 * LC_WARPS;
constexpr int LC_VP = LC_COLS * 2 + 16, LC_PP = LC_T * 2 + 16;          // bytes of a row of values, of scores
constexpr int LC_MAX_SEGS = 9, LC_MIN_SEG = 4;                          // segments of a sequence, and fewest chunks of one
__host__ __device__ constexpr int lc_pitch(int dk) { return dk * 2 + 16; }
__host__ __device__ constexpr int lc_stage(int dk) { return 2 * LC_T * lc_pitch(dk) + LC_T * LC_VP; }
__host__ __device__ constexpr int lc_smem(int dk) { return 2 * lc_stage(dk) + 2 * LC_T * LC_PP; }

struct LinearChunkParams {
  nfn_linear_args a;
  int segs;
  float* seg_init;            // [seq][head][dim_p][vdim_p]: the state before the sequence's rows
  float* seg_state;           // [seq][seg][head][dim_p][vdim_p]: what a segment adds (the first one: the state after it)
};

__device__ __forceinline__ void lc_mma(float (&d)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
  asm("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
      : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
      : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void lc_load(uint32_t (&r)[4], uint32_t at) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(at) : "memory");
}
__device__ __forceinline__ void lc_load_t(uint32_t (&r)[4], uint32_t at) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(at) : "memory");
}
// 16 bytes to shared memory; zeros where the row does not exist
__device__ __forceinline__ void lc_copy(uint32_t dst, const void* src, bool live) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(live ? 16 : 0) : "memory");
}

// STATE: only what a segment adds to the state
template <int DK, bool STATE>
__global__ void __launch_bounds__(LC_THREADS, 2)
linear_chunk_kernel(const LinearChunkParams p) {
  constexpr int PITCH = lc_pitch(DK), STAGE = lc_stage(DK), NT = DK / 8;
  extern __shared__ __align__(128) unsigned char lc_bytes[];
  __shared__ float sw[LC_T + 1];
  const nfn_linear_args& a = p.a;
  const int runs = STATE ? p.segs - 1 : p.segs, sq = blockIdx.z / runs, seg = blockIdx.z % runs;
  const nfn_seq_rows seq = a.seqs[sq];
  const int total = (seq.n + LC_T - 1) / LC_T, per = (total + p.segs - 1) / p.segs, c0 = seg * per, c1 = min(total, c0 + per);
  if (seq.slot < 0 || c0 >= c1 || (STATE && c1 == total && seg > 0)) return;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, j = lane & 3;
  const int h = blockIdx.y, DP = a.dim_p, VP = a.vdim_p, HD = a.heads * DP, v0 = blockIdx.x * LC_COLS;
  const bool on = v0 + 16 * warp < VP;
  const uint32_t smem = smem_u32(lc_bytes), sP = smem + 2 * STAGE;
  const __nv_bfloat16* rows = static_cast<const __nv_bfloat16*>(a.qkv) + (size_t)seq.row0 * a.ld_qkv;

  auto load = [&](int c) {
    const uint32_t stage = smem + ((c - c0) & 1) * STAGE;
    const __nv_bfloat16* x = rows + (size_t)c * LC_T * a.ld_qkv;
    const int n = seq.n - c * LC_T;
    constexpr int PIECES = DK / 8, STEP = LC_THREADS / PIECES, VPIECES = LC_COLS / 8, VSTEP = LC_THREADS / VPIECES;      // 16 bytes each; rows at a time
    {
      const int q = tid % PIECES, r0 = tid / PIECES;
      const __nv_bfloat16* src = x + (size_t)r0 * a.ld_qkv + h * DP + q * 8;
      uint32_t dst = stage + r0 * PITCH + q * 16;
      if (q * 8 < DP) {
#pragma unroll
        for (int r = 0; r < LC_T; r += STEP, src += (size_t)STEP * a.ld_qkv, dst += STEP * PITCH) {
          const bool live = r0 + r < n;
          if (!STATE) lc_copy(dst, live ? src : x, live);
          lc_copy(dst + LC_T * PITCH, live ? src + HD : x, live);
        }
      }
    }
    {
      const int q = tid % VPIECES, r0 = tid / VPIECES;
      const __nv_bfloat16* src = x + (size_t)r0 * a.ld_qkv + 2 * HD + h * VP + v0 + q * 8;
      uint32_t dst = stage + 2 * LC_T * PITCH + r0 * LC_VP + q * 16;
      if (v0 + q * 8 < VP) {
#pragma unroll
        for (int r = 0; r < LC_T; r += VSTEP, src += (size_t)VSTEP * a.ld_qkv, dst += VSTEP * LC_VP) {
          const bool live = r0 + r < n;
          lc_copy(dst, live ? src : x, live);
        }
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  if (DP < DK) {                                            // channels that do not exist
    const int gap = (DK - DP) / 8;
    for (int i = tid; i < 4 * LC_T * gap; i += LC_THREADS) {
      const int r = i / gap;                                // rows of queries and keys in both stages
      *reinterpret_cast<uint4*>(lc_bytes + (r / (2 * LC_T)) * STAGE + (r % (2 * LC_T)) * PITCH + (DP / 8 + i % gap) * 16) = make_uint4(0u, 0u, 0u, 0u);
    }
  }
  load(c0);
  if (c0 + 1 < c1) load(c0 + 1);
  for (int i = tid; i <= LC_T; i += LC_THREADS) sw[i] = a.powers[(size_t)h * (LC_T + 1) + i];

  // S^T: rows are value columns (g, g + 8), columns key channels 8 t + 2 j, + 1
  const size_t block = (size_t)DP * VP, at0 = v0 + 16 * warp + g;
  float* st = a.state + ((size_t)seq.slot * a.heads + h) * block + at0;
  float* init = p.seg_init + ((size_t)sq * a.heads + h) * block + at0;
  const size_t cell = (size_t)sq * p.segs * a.heads + h;    // of the first segment
  float s[NT][4];
  auto each = [&](auto&& fn) {                              // every element that exists, with its offset from column at0
#pragma unroll
    for (int t = 0; t < NT; ++t)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int d = 8 * t + 2 * j + (e & 1);
        if (on && d < DP) fn(s[t][e], (size_t)d * VP + (e >> 1) * 8);
      }
  };
#pragma unroll
  for (int t = 0; t < NT; ++t)
#pragma unroll
    for (int e = 0; e < 4; ++e) s[t][e] = 0.f;
  const bool fresh = seq.pos0 == 0;
  if (STATE) {
    if (seg == 0) {
      if (!fresh) each([&](float& x, size_t o) { x = st[o]; });
      each([&](float& x, size_t o) { init[o] = x; });
    }
  } else if (p.segs == 1) {
    if (!fresh) each([&](float& x, size_t o) { x = st[o]; });
  } else if (seg == 0) {
    each([&](float& x, size_t o) { x = init[o]; });
  } else {
    const float* add = p.seg_state + cell * block + at0;
    each([&](float& x, size_t o) { x = add[o]; });
    float left = 1.f, f = a.powers[(size_t)h * (LC_T + 1) + LC_T];      // w^(64 per), by squaring
    for (int e = per; e > 0; e >>= 1, f *= f)
      if (e & 1) left *= f;
    for (int q = 1; q < seg; ++q) {
      add += a.heads * block;
      each([&](float& x, size_t o) { x = x * left + add[o]; });
    }
  }

  for (int c = c0; c < c1; ++c) {
    const uint32_t sQ = smem + ((c - c0) & 1) * STAGE, sK = sQ + LC_T * PITCH, sV = sK + LC_T * PITCH;
    const int n = min(LC_T, seq.n - c * LC_T);
    if (c + 1 < c1) asm volatile("cp.async.wait_group 1;" ::: "memory");
    else asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    if constexpr (!STATE) {
      // ---- scores of rows 16 warp .. + 15, decayed, below and on the diagonal ----
      float acc[8][4];
#pragma unroll
      for (int t = 0; t < 8; ++t)
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[t][e] = 0.f;
#pragma unroll
      for (int kk = 0; kk < DK / 16; ++kk) {
        uint32_t q[4];
        lc_load(q, sQ + (16 * warp + (lane & 15)) * PITCH + kk * 32 + (lane >> 4) * 16);
#pragma unroll
        for (int np = 0; np < 4; ++np)
          if (np <= warp) {
            uint32_t k[4];
            lc_load(k, sK + (16 * np + (lane & 7) + (lane >> 4) * 8) * PITCH + kk * 32 + ((lane >> 3) & 1) * 16);
            lc_mma(acc[2 * np], q[0], q[1], q[2], q[3], k[0], k[1]);
            lc_mma(acc[2 * np + 1], q[0], q[1], q[2], q[3], k[2], k[3]);
          }
      }
#pragma unroll
      for (int t = 0; t < 8; ++t)
        if (t <= 2 * warp + 1) {
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            const int r = 16 * warp + g + 8 * e, k = 8 * t + 2 * j;
            const float x = k <= r ? acc[t][2 * e] * sw[max(r - k, 0)] : 0.f, y = k + 1 <= r ? acc[t][2 * e + 1] * sw[max(r - k - 1, 0)] : 0.f;
            uint32_t hi, lo;
            split_bf16(x, y, hi, lo);
            unsigned char* dst = lc_bytes + 2 * STAGE + r * LC_PP + k * 2;
            *reinterpret_cast<uint32_t*>(dst) = hi;
            *reinterpret_cast<uint32_t*>(dst + LC_T * LC_PP) = lo;
          }
        }
      __syncthreads();
    }
    if (on) {
      uint32_t v[4][4];                                     // values of 16 tokens at a time, transposed: rows are columns g, g + 8
#pragma unroll
      for (int kk = 0; kk < 4; ++kk) lc_load_t(v[kk], sV + (16 * kk + (lane & 7) + (lane >> 4) * 8) * LC_VP + (16 * warp + ((lane >> 3) & 1) * 8) * 2);
      if constexpr (!STATE) {
        float o[4][2][4];
#pragma unroll
        for (int m = 0; m < 4; ++m)
#pragma unroll
          for (int t = 0; t < 2; ++t)
#pragma unroll
            for (int e = 0; e < 4; ++e) o[m][t][e] = 0.f;
#pragma unroll
        for (int kk = 0; kk < DK / 16; ++kk) {
          uint32_t hi[4], lo[4];
          split_bf16(s[2 * kk][0], s[2 * kk][1], hi[0], lo[0]);
          split_bf16(s[2 * kk + 1][0], s[2 * kk + 1][1], hi[1], lo[1]);
          split_bf16(s[2 * kk][2], s[2 * kk][3], hi[2], lo[2]);
          split_bf16(s[2 * kk + 1][2], s[2 * kk + 1][3], hi[3], lo[3]);
#pragma unroll
          for (int m0 = 0; m0 < 4; m0 += 2) {               // four products in a row that do not wait for one another
            uint32_t q[2][4];
#pragma unroll
            for (int m = 0; m < 2; ++m) lc_load(q[m], sQ + (16 * (m0 + m) + (lane & 15)) * PITCH + kk * 32 + (lane >> 4) * 16);
#pragma unroll
            for (int m = 0; m < 2; ++m)
#pragma unroll
              for (int t = 0; t < 2; ++t) lc_mma(o[m0 + m][t], q[m][0], q[m][1], q[m][2], q[m][3], hi[2 * t], hi[2 * t + 1]);
#pragma unroll
            for (int m = 0; m < 2; ++m)
#pragma unroll
              for (int t = 0; t < 2; ++t) lc_mma(o[m0 + m][t], q[m][0], q[m][1], q[m][2], q[m][3], lo[2 * t], lo[2 * t + 1]);
          }
        }
#pragma unroll
        for (int m = 0; m < 4; ++m) {
          const float f0 = sw[16 * m + g + 1], f1 = sw[16 * m + g + 9];
#pragma unroll
          for (int t = 0; t < 2; ++t) {
            o[m][t][0] *= f0; o[m][t][1] *= f0; o[m][t][2] *= f1; o[m][t][3] *= f1;
          }
#pragma unroll
          for (int kk = 0; kk <= m; ++kk) {
            uint32_t hi[4], lo[4];
            const uint32_t at = sP + (16 * m + (lane & 15)) * LC_PP + kk * 32 + (lane >> 4) * 16;
            lc_load(hi, at);
            lc_load(lo, at + LC_T * LC_PP);
            lc_mma(o[m][0], hi[0], hi[1], hi[2], hi[3], v[kk][0], v[kk][2]);
            lc_mma(o[m][1], hi[0], hi[1], hi[2], hi[3], v[kk][1], v[kk][3]);
            lc_mma(o[m][0], lo[0], lo[1], lo[2], lo[3], v[kk][0], v[kk][2]);
            lc_mma(o[m][1], lo[0], lo[1], lo[2], lo[3], v[kk][1], v[kk][3]);
          }
          float* dst = a.o + (size_t)(seq.row0 + c * LC_T + 16 * m + g) * a.ld_o + (size_t)h * VP + v0 + 16 * warp + 2 * j;
#pragma unroll
          for (int t = 0; t < 2; ++t) {
            if (16 * m + g < n) *reinterpret_cast<float2*>(dst + 8 * t) = make_float2(o[m][t][0], o[m][t][1]);
            if (16 * m + g + 8 < n) *reinterpret_cast<float2*>(dst + (size_t)8 * a.ld_o + 8 * t) = make_float2(o[m][t][2], o[m][t][3]);
          }
        }
      }
      // ---- the next state ----
      const float keep = sw[n];
#pragma unroll
      for (int t = 0; t < NT; ++t)
#pragma unroll
        for (int e = 0; e < 4; ++e) s[t][e] *= keep;
#pragma unroll
      for (int kk = 0; kk < 4; ++kk) {
        uint32_t hi[4], lo[4];
#pragma unroll
        for (int q = 0; q < 2; ++q) {                       // tokens r, r + 1
          const int r = 16 * kk + 8 * q + 2 * j;
          const float f0 = r < n ? sw[max(n - 1 - r, 0)] : 0.f, f1 = r + 1 < n ? sw[max(n - 2 - r, 0)] : 0.f;
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            const float2 x = unpack_bf16x2(v[kk][2 * q + e]);
            split_bf16(x.x * f0, x.y * f1, hi[2 * q + e], lo[2 * q + e]);
          }
        }
#pragma unroll
        for (int t0 = 0; t0 < NT; t0 += 4) {
          uint32_t k[2][4];
#pragma unroll
          for (int t = 0; t < 2; ++t) lc_load_t(k[t], sK + (16 * kk + (lane & 15)) * PITCH + (t0 + 2 * t) * 16 + (lane >> 4) * 16);
#pragma unroll
          for (int t = 0; t < 4; ++t) lc_mma(s[t0 + t], hi[0], hi[1], hi[2], hi[3], k[t / 2][2 * (t & 1)], k[t / 2][2 * (t & 1) + 1]);
#pragma unroll
          for (int t = 0; t < 4; ++t) lc_mma(s[t0 + t], lo[0], lo[1], lo[2], lo[3], k[t / 2][2 * (t & 1)], k[t / 2][2 * (t & 1) + 1]);
        }
      }
    }
    __syncthreads();                                        // every warp is done with the stage and the scores
    if (c + 2 < c1) load(c + 2);
  }
  if (STATE) {
    float* dst = p.seg_state + (cell + (size_t)seg * a.heads) * block + at0;
    each([&](float& x, size_t o) { dst[o] = x; });
  } else if (c1 == total) {
    each([&](float& x, size_t o) { st[o] = x; });
  }
}

template <int DK, bool STATE>
static int launch_linear_chunk(const LinearChunkParams& p, cudaStream_t st) {
  auto kern = linear_chunk_kernel<DK, STATE>;
  static bool raised[64] = {};
  int dev = 0;
  cudaGetDevice(&dev);
  if (lc_smem(DK) > 48 * 1024 && !raised[dev & 63]) {
    if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, lc_smem(DK)) != cudaSuccess) return launch_check("linear_chunk attr", 0);
    raised[dev & 63] = true;
  }
  kern<<<dim3(ceil_div(p.a.vdim_p, LC_COLS), p.a.heads, p.a.n_seqs * (STATE ? p.segs - 1 : p.segs)), LC_THREADS, lc_smem(DK), st>>>(p);
  return launch_check("linear_chunk");
}

const char* linear_args_problem(const nfn_linear_args& a);   // linear_rows.cu; null: fine

// bytes the segments of one sequence's head take
static long long linear_segment_bytes(int dim_p, int vdim_p) { return (LC_MAX_SEGS + 1LL) * dim_p * vdim_p * 4; }

}  // namespace nfn

using namespace nfn;

extern "C" long long nfn_linear_chunk_workspace_bytes(int heads, int dim_p, int vdim_p, int max_seqs) {
  if (dim_p > 128) return 0;
  return std::min<long long>((long long)heads * max_seqs, 160) * linear_segment_bytes(dim_p, vdim_p);      // segments are for few heads and sequences
}

extern "C" int nfn_linear_chunks(const nfn_linear_args* args, int max_rows, void* workspace, long long workspace_bytes, nfn_stream_t stream) {
  if (!args) return fail(-1, "linear attention: null args");
  if (args->n_seqs <= 0 || max_rows <= 0) return 0;
  if (const char* why = linear_args_problem(*args)) return fail(-1, why);
  const nfn_linear_args& a = *args;
  if (a.f32 || a.dim_p > 128) return fail(-1, "linear attention: chunks are for bf16 activations and at most 128 key channels per head");
  LinearChunkParams p{};
  p.a = a;
  const long long cells = (long long)a.heads * a.n_seqs, ctas = cells * ceil_div(a.vdim_p, LC_COLS);
  // as many as leave the fewest chunks per slot, two CTAs to an SM; more of them only where it pays
  const int chunks = ceil_div(max_rows, LC_T), slots = 2 * sm_count();
  double best = 1e30;
  p.segs = 1;
  for (int n = 1; n <= LC_MAX_SEGS && (n == 1 || n * LC_MIN_SEG <= chunks); ++n) {
    const double cost = (double)((ctas * n + slots - 1) / slots) * ceil_div(chunks, n) * (n > 1 ? 1.4 : 1.0) + n;      // the states in front take two fifths of a pass
    if (cost < best) {
      best = cost;
      p.segs = n;
    }
  }
  if (!workspace || cells * linear_segment_bytes(a.dim_p, a.vdim_p) > workspace_bytes) p.segs = 1;
  p.segs = std::max(p.segs, 1);
  if ((long long)a.n_seqs * p.segs > 65535) return fail(-1, "linear attention: too many sequences for one launch");
  p.seg_init = static_cast<float*>(workspace);
  p.seg_state = p.seg_init + cells * a.dim_p * a.vdim_p;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (p.segs > 1)
    if (const int rc = a.dim_p <= 64 ? launch_linear_chunk<64, true>(p, st) : launch_linear_chunk<128, true>(p, st)) return rc;
  return a.dim_p <= 64 ? launch_linear_chunk<64, false>(p, st) : launch_linear_chunk<128, false>(p, st);
}
