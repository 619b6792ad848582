// Gated delta rule over prompt portions, sixteen tokens at a time (bf16 activations; state and everything that enters it fp32).
//
// Inside a chunk let G_r be the running sum of the log decays (per key channel), S the state before the chunk and, with unit vectors k, q,
//   A_rj = sum_c k_rc k_jc e^(G_rc - G_jc)  (j < r),   P_rj = sum_c q_rc k_jc e^(G_rc - G_jc)  (j <= r),   T = (I + diag(beta) A)^-1 diag(beta).
// The corrections of the chunk are U = T V - W S with W = T (e^G k), its read-outs O = P T V + Q S with Q = e^G q - P W, and the state after it
// S' = e^G_last S + K^T U with K_j = k_j e^(G_last - G_j). Every exponent is a sum of decays between two tokens, never positive, so
// nothing overflows however fast a channel forgets.
//
//   delta_prepare_kernel  one CTA per (chunk, head), all chunks at once: W, Q, K and T V, P T V. A thread owns two channels; their
//                         products for all pairs of tokens are formed in registers and summed over channels through shared memory.
//   delta_scan_kernel     one warp per (head, 16 value columns, 64 key channels), one chunk after another: the state, transposed, sits in
//                         the accumulator registers of mma.m16n8k16 and is the A operand of the next chunk's W S and Q S as it stands; W, Q
//                         and K arrive in fragment order by bulk copies through a ring of shared memory stages.
//
// The products with the state are formed from fp32 values split into two bf16 parts each (high x high + high x low + low x high), which
// keeps sixteen bits of every factor. The scan also runs recurrences without corrections (U = V, no W: wkv_chunk.cu).
// Their states are linear in what comes before, so where heads are few a round is cut into segments: segment_state_kernel runs every segment but the
// last from zero, without read-outs, and the scan of each segment starts from the sum of what the earlier ones leave. Rounds of as many chunks as the workspace holds alternate between the two kernels, small enough
// to stay in L2.
#include <algorithm>

#include "attention_v2.cuh"
#include "common.h"
#include "chunk_scan.cuh"
#include "delta.cuh"

namespace nfn {

// log2(1 + e^z): the series of log(1 + t) for small t = e^z keeps slow decays exact
__device__ __forceinline__ float softplus_log2(float z) {
  const float y = z * 1.4426950408889634f, t = fast_exp2(y);
  const float s = t * (1.f - t * (0.5f - t * (0.33333333f - t * (0.25f - t * (0.2f - t * (0.16666667f - t * 0.14285714f))))));
  const float l = t < 0.125f ? s * 1.4426950408889634f : __log2f(1.f + t);
  return y > 28.f ? y : l;
}

// NT threads, two neighbouring key channels each (dk = 2 NT), and value columns in pairs
template <int NT>
__global__ void __launch_bounds__(NT, 448 / NT)
delta_prepare_kernel(const DeltaChunkParams p) {
  constexpr int PITCH = NT == 128 ? 136 : NT + 4;                 // partial sums [64 values][NT]; rows are read in 16-byte pieces
  extern __shared__ __align__(128) unsigned char dc_smem[];       // partial sums, then the operand block
  __shared__ __align__(16) float sA[DC_T][DC_T + 4], sP[DC_T][DC_T + 4], sT[DC_T][DC_T + 4];
  __shared__ float s_norm[2][DC_T], s_beta[DC_T];
  const nfn_delta_args& a = p.a;
  const nfn_seq_rows seq = a.seqs[blockIdx.z];
  const int r0 = (p.chunk0 + blockIdx.x) * DC_T, n = min(DC_T, seq.n - r0);
  if (seq.slot < 0 || n <= 0) return;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int h = blockIdx.y, hk = h / (a.heads / a.kv_heads), DP = a.dim_p, VP = a.vdim_p;
  const int off_k = a.kv_heads * DP, off_v = 2 * off_k;
  const size_t row0 = (size_t)(seq.row0 + r0);
  const __nv_bfloat16* x = static_cast<const __nv_bfloat16*>(a.qkv) + row0 * a.ld_qkv;
  const int c0 = 2 * tid;
  const bool on = c0 < DP;

  // ---- this thread's channels; unit vectors, step sizes ----
  float q[DC_T][2], k[DC_T][2], G[DC_T][2];
  {
    uint32_t qw[DC_T], kw[DC_T];
#pragma unroll
    for (int r = 0; r < DC_T; ++r) {
      const bool live = on && r < n;
      qw[r] = live ? *reinterpret_cast<const uint32_t*>(x + (size_t)r * a.ld_qkv + hk * DP + c0) : 0u;
      kw[r] = live ? *reinterpret_cast<const uint32_t*>(x + (size_t)r * a.ld_qkv + off_k + hk * DP + c0) : 0u;
      const float2 z = live ? *reinterpret_cast<const float2*>(a.decay + (row0 + r) * a.ld_decay + (size_t)h * DP + c0) : make_float2(0.f, 0.f);
      G[r][0] = z.x;
      G[r][1] = z.y;
    }
    // squared lengths: 32 sums over the channels, NT / 32 neighbouring threads each
    float* part = reinterpret_cast<float*>(dc_smem);
#pragma unroll
    for (int r = 0; r < DC_T; ++r) {
      const float2 fq = unpack_bf16x2(qw[r]), fk = unpack_bf16x2(kw[r]);
      q[r][0] = fq.x; q[r][1] = fq.y; k[r][0] = fk.x; k[r][1] = fk.y;
      part[r * PITCH + tid] = fq.x * fq.x + fq.y * fq.y;
      part[(DC_T + r) * PITCH + tid] = fk.x * fk.x + fk.y * fk.y;
    }
    __syncthreads();
    constexpr int SHARE = NT / 32;
    const int v = tid / SHARE;
    const float* src = part + v * PITCH + tid % SHARE * 32;
    float4 f = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const float4 g = *reinterpret_cast<const float4*>(src + 4 * i);
      f.x += g.x; f.y += g.y; f.z += g.z; f.w += g.w;
    }
    float t = (f.x + f.y) + (f.z + f.w);
#pragma unroll
    for (int o = 1; o < SHARE; o <<= 1) t += __shfl_xor_sync(0xffffffffu, t, o);
    const float inv = 1.f / sqrtf(t + a.unit_eps);
    s_norm[v / DC_T][v % DC_T] = v < DC_T ? inv / sqrtf((float)a.dim) : inv;
    if (tid < DC_T) s_beta[tid] = tid < n ? sigmoid_exact(__bfloat162float(static_cast<const __nv_bfloat16*>(a.beta)[(row0 + tid) * a.ld_beta + h])) : 0.f;
    __syncthreads();
  }
  {
    const float rate = -expf(__bfloat162float(static_cast<const __nv_bfloat16*>(a.a_log)[h]));
    const float2 bias = on ? unpack_bf16x2(*reinterpret_cast<const uint32_t*>(static_cast<const __nv_bfloat16*>(a.dt_bias) + (size_t)h * DP + c0)) : make_float2(0.f, 0.f);
    float s0 = 0.f, s1 = 0.f;                                     // sums of log2 decays
#pragma unroll
    for (int r = 0; r < DC_T; ++r) {
      const float fq = s_norm[0][r], fk = s_norm[1][r];
      q[r][0] *= fq; q[r][1] *= fq; k[r][0] *= fk; k[r][1] *= fk;
      if (r < n) {
        s0 += rate * softplus_log2(G[r][0] + bias.x);
        s1 += rate * softplus_log2(G[r][1] + bias.y);
      }
      G[r][0] = s0;
      G[r][1] = s1;
    }
  }
  // ---- A and P: rows 2t, 15 - 2t, 2t + 1, 14 - 2t together have 64 values ----
  float* part = reinterpret_cast<float*>(dc_smem);
#pragma unroll
  for (int t = 0; t < 4; ++t) {
    const int rows[4] = {2 * t, 15 - 2 * t, 2 * t + 1, 14 - 2 * t};
    int at = 0;
#pragma unroll
    for (int w = 0; w < 4; ++w) {
      const int r = rows[w];
#pragma unroll
      for (int j = 0; j < DC_T; ++j) {
        if (j > r) continue;
        float k0 = k[j][0], k1 = k[j][1];
        if (j < r) {
          float d0 = G[r][0], d1 = G[r][1];
          add2f(d0, d1, d0, d1, -G[j][0], -G[j][1]);
          mul2(k0, k1, k0, k1, fast_exp2(d0), fast_exp2(d1));
        }
        part[at++ * PITCH + tid] = q[r][0] * k0 + q[r][1] * k1;
        if (j < r) part[at++ * PITCH + tid] = k[r][0] * k0 + k[r][1] * k1;
      }
    }
    __syncthreads();
    // every thread sums 64 numbers: two values (NT = 32), one (64) or half of one (128)
#pragma unroll
    for (int v0 = 0; v0 < (NT == 32 ? 64 : 32); v0 += 32) {
      const int v = NT == 32 ? tid + v0 : NT == 64 ? tid : tid >> 1;
      const float* src = part + v * PITCH + (NT == 128 ? 4 * (tid & 1) : 0);
      float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
      for (int i = 0; i < (NT == 32 ? 8 : 16); ++i) {
        const float4 f = *reinterpret_cast<const float4*>(src + i * (NT == 128 ? 8 : 4));
        add2(s.x, s.y, f.x, f.y);
        add2(s.z, s.w, f.z, f.w);
      }
      float sum = (s.x + s.y) + (s.z + s.w);
      if (NT == 128) sum += __shfl_xor_sync(0xffffffffu, sum, 1);
      // where it belongs: the rows of the pass hold 2 r + 1 values each, P_rj and A_rj in turn
      int rest = v, r = rows[0];
      if (rest >= 2 * r + 1) { rest -= 2 * r + 1; r = rows[1];
        if (rest >= 2 * r + 1) { rest -= 2 * r + 1; r = rows[2];
          if (rest >= 2 * r + 1) { rest -= 2 * r + 1; r = rows[3]; } } }
      ((rest & 1) ? sA : sP)[r][rest >> 1] = sum;
      if (NT != 32) break;
    }
    __syncthreads();
  }
  // powers of the decays are formed again below instead of being kept in registers
#pragma unroll
  for (int r = 0; r < DC_T; ++r) asm volatile("" : "+f"(G[r][0]), "+f"(G[r][1]));
  // ---- T = (I + diag(beta) A)^-1 diag(beta): one column per lane, forward substitution ----
  if (tid < DC_T) {
    float y[DC_T];
#pragma unroll
    for (int r = 0; r < DC_T; ++r) {
      float s0 = 0.f, s1 = 0.f;
#pragma unroll
      for (int i = 0; i < r; ++i) ((i & 1) ? s1 : s0) += sA[r][i] * y[i];
      y[r] = (r == tid ? 1.f : 0.f) - s_beta[r] * (s0 + s1);
    }
    const float b = s_beta[tid];
#pragma unroll
    for (int r = 0; r < DC_T; ++r) sT[r][tid] = y[r] * b;
  }
  __syncthreads();
  // rows of T and P times two columns at once
  auto lower = [](const float (&m)[DC_T + 4], const float (&v)[DC_T][2], int last, float& o0, float& o1) {
#pragma unroll
    for (int j4 = 0; j4 <= last; j4 += 4) {
      const float4 f = *reinterpret_cast<const float4*>(&m[j4]);
      const float t[4] = {f.x, f.y, f.z, f.w};
#pragma unroll
      for (int e = 0; e < 4; ++e)
        if (j4 + e <= last) fma2(o0, o1, t[e], t[e], v[j4 + e][0], v[j4 + e][1], o0, o1);
    }
  };
  const size_t block = ((size_t)blockIdx.z * p.n_chunks + blockIdx.x) * a.heads + h;
  // ---- W, Q, K of this thread's key channels, in the order of the scan's fragments: {first eight of the contraction: high, low; second: high, low} ----
  unsigned char* stage = dc_smem;
  *reinterpret_cast<float2*>(stage + dc_gamma_at(p.dk, true) + c0 * 4) = make_float2(fast_exp2(G[DC_T - 1][0]), fast_exp2(G[DC_T - 1][1]));
#pragma unroll
  for (int r = 0; r < DC_T; r += 2)
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      uint2 w;
      split_bf16(k[r][i] * fast_exp2(G[DC_T - 1][i] - G[r][i]), k[r + 1][i] * fast_exp2(G[DC_T - 1][i] - G[r + 1][i]), w.x, w.y);
      *reinterpret_cast<uint2*>(stage + dc_piece(4 * (p.dk / 16) + (c0 + i) / 8, (c0 + i) % 8 * 4 + (r % 8) / 2, true) + (r / 8) * 8) = w;
    }
  float w[DC_T][2];
#pragma unroll
  for (int r = 0; r < DC_T; ++r) {
    const float e0 = fast_exp2(G[r][0]), e1 = fast_exp2(G[r][1]);
    q[r][0] *= e0; q[r][1] *= e1; k[r][0] *= e0; k[r][1] *= e1;
  }
#pragma unroll
  for (int r = 0; r < DC_T; ++r) {
    w[r][0] = w[r][1] = 0.f;
    lower(sT[r], k, r, w[r][0], w[r][1]);
    float p0 = 0.f, p1 = 0.f;
    lower(sP[r], w, r, p0, p1);
    uint2 f;
    const uint32_t half = ((c0 % 16) / 8) * 8;
    const int piece_lane = r % 8 * 4 + (c0 % 8) / 2;
    split_bf16(w[r][0], w[r][1], f.x, f.y);
    *reinterpret_cast<uint2*>(stage + dc_piece(4 * (c0 / 16) + r / 8, piece_lane, false) + half) = f;
    split_bf16(q[r][0] - p0, q[r][1] - p1, f.x, f.y);
    *reinterpret_cast<uint2*>(stage + dc_piece(4 * (c0 / 16) + 2 + r / 8, piece_lane, false) + half) = f;
  }
  asm volatile("" ::: "memory");                                 // T and P are read again, not kept in registers
  // ---- T V and P T V of this thread's value columns ----
  float* uo = p.uo + block * dc_uo_floats(VP);
  for (int c = c0; c < VP; c += 2 * NT) {
    float v[DC_T][2], u[DC_T][2];
#pragma unroll
    for (int r = 0; r < DC_T; ++r) {
      const float2 f = r < n ? unpack_bf16x2(*reinterpret_cast<const uint32_t*>(x + (size_t)r * a.ld_qkv + off_v + h * VP + c)) : make_float2(0.f, 0.f);
      v[r][0] = f.x;
      v[r][1] = f.y;
    }
#pragma unroll
    for (int r = 0; r < DC_T; ++r) {
      u[r][0] = u[r][1] = 0.f;
      lower(sT[r], v, r, u[r][0], u[r][1]);
    }
    float* dst = uo + (c / 16) * 512 + (c & 7) * 16 + ((c & 15) >> 3) * 2;      // [2][2 row tiles][lane = column % 8, row pair][column half, row]
#pragma unroll
    for (int r = 0; r < DC_T; r += 2) {
      float o[2][2] = {};
#pragma unroll
      for (int e = 0; e < 2; ++e) lower(sP[r + e], u, r + e, o[e][0], o[e][1]);
      const int at = (r / 8) * 128 + ((r % 8) / 2) * 4;
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        *reinterpret_cast<float2*>(dst + i * 16 + at) = make_float2(u[r][i], u[r + 1][i]);
        *reinterpret_cast<float2*>(dst + i * 16 + 256 + at) = make_float2(o[0][i], o[1][i]);
      }
    }
  }
  // the finished operand block leaves in one bulk copy
  fence_proxy_async();
  __syncthreads();
  if (tid == 0) {
    dc_bulk_store(p.blocks + block * dc_block_bytes(p.dk, true), smem_u32(stage), dc_block_bytes(p.dk, true));
    asm volatile("cp.async.bulk.commit_group;" ::: "memory");
    asm volatile("cp.async.bulk.wait_group 0;" ::: "memory");
  }
}

__device__ __forceinline__ void dc_mma(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// the first product of a sum
__device__ __forceinline__ void dc_mma0(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%10,%10,%10,%10};"
      : "=f"(d[0]), "=f"(d[1]), "=f"(d[2]), "=f"(d[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1), "f"(0.f));
}
__device__ __forceinline__ void dc_bulk_load(uint32_t dst, const void* src, uint32_t bytes, uint32_t bar) {
  asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"(dst), "l"(src), "r"(bytes), "r"(bar) : "memory");
}

// KS: warps that share a head's key channels, 64 each; the CTA's four warps take 4 / KS tiles of 16 value columns
constexpr int DS_WARPS = 4, DS_CH = 64, DS_K = DS_CH / 16, DS_N = DS_CH / 8;      // a warp's steps of 16 and tiles of 8 channels
// shared memory of a stage: the head's operand block, then T V and P T V of the CTA's column tiles
__host__ __device__ constexpr int ds_stage_bytes(int ks, bool corrections) { return dc_block_bytes(DS_CH * ks, corrections) + DS_WARPS / ks * 2048; }
__host__ __device__ constexpr int ds_stages(int ks) { return ks == 4 ? 3 : 4; }
template <int KS, bool CORRECTIONS>
__global__ void __launch_bounds__(DS_WARPS * 32)
delta_scan_kernel(const DeltaChunkParams p) {
  constexpr int DK = DS_CH * KS, TILES = DS_WARPS / KS, WT = CORRECTIONS ? 4 : 2, BLOCK = dc_block_bytes(DK, CORRECTIONS), STAGE = ds_stage_bytes(KS, CORRECTIONS), STAGES = ds_stages(KS);
  extern __shared__ __align__(128) unsigned char dc_smem[];       // [STAGES][STAGE], then partial sums [2][warps][4 row tiles][32][4]
  __shared__ __align__(8) uint64_t bar_full[STAGES];
  __shared__ int cta_abort_s;
  volatile int* cta_abort = &cta_abort_s;
  const nfn_delta_args& a = p.a;
  const int segs = CORRECTIONS ? 1 : p.segs, sq = blockIdx.z / segs, seg = blockIdx.z % segs, i0 = seg * (CORRECTIONS ? 0 : p.seg_chunks);
  const nfn_seq_rows seq = a.seqs[sq];
  const int total = (seq.n + DC_T - 1) / DC_T, here = min(p.n_chunks, total - p.chunk0), n_chunks = segs > 1 ? min(p.seg_chunks, here - i0) : here;
  if (seq.slot < 0 || n_chunks <= 0) return;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, j = lane & 3;
  const int ks = warp % KS, h = blockIdx.y, DP = a.dim_p, VP = a.vdim_p;
  const int vt = blockIdx.x * TILES + warp / KS;
  const bool on = vt * 16 < VP;                                   // warps past the last column tile keep the others company
  float* xch = reinterpret_cast<float*>(dc_smem + STAGES * STAGE);
  const unsigned char* blocks = p.blocks + (((size_t)sq * p.n_chunks + i0) * a.heads + h) * BLOCK;
  const size_t block_step = (size_t)a.heads * BLOCK;
  const float* uo = p.uo + (((size_t)sq * p.n_chunks + i0) * a.heads + h) * dc_uo_floats(VP) + blockIdx.x * TILES * 512;
  const size_t uo_step = (size_t)a.heads * dc_uo_floats(VP);
  const uint32_t uo_bytes = min(TILES, VP / 16 - (int)blockIdx.x * TILES) * 2048;

  auto load = [&](int i) {
    const uint32_t bar = smem_u32(&bar_full[i % STAGES]), dst = smem_u32(dc_smem + (i % STAGES) * STAGE);
    mbar_expect_tx(bar, BLOCK + uo_bytes);
    dc_bulk_load(dst, blocks + i * block_step, BLOCK, bar);
    dc_bulk_load(dst + BLOCK, uo + i * uo_step, uo_bytes, bar);
  };
  if (tid == 0) {
    cta_abort_s = 0;
    for (int s = 0; s < STAGES; ++s) mbar_init(smem_u32(&bar_full[s]), 1);
    fence_mbar_init();
    for (int i = 0; i < min(STAGES, n_chunks); ++i) load(i);
  }
  // S^T: rows are value columns (g, g + 8), columns key channels 64 ks + 8 t + 2 j, + 1
  float* st = a.state + ((size_t)seq.slot * a.heads + h) * DP * VP + vt * 16 + g;
  const bool fresh = seq.pos0 == 0 && p.chunk0 == 0;
  float s[DS_N][4];
  auto take = [&](const float* from, bool live) {                // a state as it lies in memory
#pragma unroll
    for (int t = 0; t < DS_N; ++t)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int d = DS_CH * ks + 8 * t + 2 * j + (e & 1);
        s[t][e] = (live && on && d < DP) ? from[(size_t)d * VP + (e >> 1) * 8] : 0.f;
      }
  };
  if (segs == 1) {
    take(st, !fresh);
  } else if (seg == 0) {
    take(p.seg_init + ((size_t)sq * a.heads + h) * DP * VP + vt * 16 + g, true);
  } else {
    const size_t cell = (size_t)sq * segs * a.heads + h;         // of the first segment
    take(p.seg_state + cell * DP * VP + vt * 16 + g, true);
    for (int q = 1; q < seg; ++q) {
      const float* add = p.seg_state + (cell + (size_t)q * a.heads) * DP * VP + vt * 16 + g;
      const float* left = p.seg_gamma + (cell + (size_t)q * a.heads) * DK + DS_CH * ks + 2 * j;
#pragma unroll
      for (int t = 0; t < DS_N; ++t) {
        const float2 f = *reinterpret_cast<const float2*>(left + 8 * t);
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int d = DS_CH * ks + 8 * t + 2 * j + (e & 1);
          if (on && d < DP) s[t][e] = s[t][e] * ((e & 1) ? f.y : f.x) + add[(size_t)d * VP + (e >> 1) * 8];
        }
      }
    }
  }
  __syncthreads();
  // Products that every warp of a column tile adds up: W S of this chunk, which the next state waits for, and Q S of the chunk before, which
  // nothing waits for and which is formed while the partial sums of W S cross shared memory.
  int at = 0, phase = 0;
  uint32_t hi[DS_K][4], lo[DS_K][4];                           // S, split
  auto product = [&](const unsigned char* stage, int nt0, float (&acc)[2][4]) {      // two row tiles of [W, Q] times S, transposed
    float low[2][4];
#pragma unroll
    for (int kk = 0; kk < DS_K; ++kk) {
      uint4 b[2];
#pragma unroll
      for (int nt = 0; nt < 2; ++nt) b[nt] = *reinterpret_cast<const uint4*>(stage + dc_piece<CORRECTIONS>((DS_K * ks + kk) * WT + nt0 + nt, lane, false));
#pragma unroll
      for (int nt = 0; nt < 2; ++nt) {
        if (kk == 0) dc_mma0(acc[nt], hi[kk], b[nt].x, b[nt].z);
        else dc_mma(acc[nt], hi[kk], b[nt].x, b[nt].z);
      }
#pragma unroll
      for (int nt = 0; nt < 2; ++nt) {
        if (kk == 0) dc_mma0(low[nt], hi[kk], b[nt].y, b[nt].w);
        else dc_mma(low[nt], hi[kk], b[nt].y, b[nt].w);
      }
#pragma unroll
      for (int nt = 0; nt < 2; ++nt) dc_mma((kk & 1) == 0 ? acc[nt] : low[nt], lo[kk], b[nt].x, b[nt].z);
    }
#pragma unroll
    for (int nt = 0; nt < 2; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[nt][e] += low[nt][e];
  };
  auto put = [&](int i, int nt0, const float (&acc)[2][4]) {
    float* mine = xch + ((i & 1) * DS_WARPS + warp) * 512 + lane * 4;
#pragma unroll
    for (int nt = 0; nt < 2; ++nt) *reinterpret_cast<float4*>(mine + (nt0 + nt) * 128) = make_float4(acc[nt][0], acc[nt][1], acc[nt][2], acc[nt][3]);
  };
  auto sum = [&](int i, int nt) {
    const float* all = xch + ((i & 1) * DS_WARPS + warp / KS * KS) * 512 + lane * 4;
    float4 t = *reinterpret_cast<const float4*>(all + nt * 128);
#pragma unroll
    for (int w = 1; w < KS; ++w) {
      const float4 b = *reinterpret_cast<const float4*>(all + w * 512 + nt * 128);
      t.x += b.x; t.y += b.y; t.z += b.z; t.w += b.w;
    }
    return t;
  };
  // read-outs of chunk i, whose partial sums were exchanged with those of step `x`, shared out among the warps of a column tile: each takes some of
  // (row tile, column half)
  constexpr int PARTS = 4 / KS;
  auto read_out = [&](int i, int x) {
    if (!on) return;
#pragma unroll
    for (int n = 0; n < PARTS; ++n) {
      const int tile = (ks * PARTS + n) >> 1, c = 2 * ((ks * PARTS + n) & 1);
      float2 t = *reinterpret_cast<const float2*>(dc_smem + (i % STAGES) * STAGE + BLOCK + ((warp / KS) * 512 + 256 + tile * 128 + lane * 4 + c) * 4);
      const float* all = xch + ((x & 1) * DS_WARPS + warp / KS * KS) * 512 + (2 + tile) * 128 + lane * 4 + c;
#pragma unroll
      for (int w = 0; w < KS; ++w) {
        const float2 f = *reinterpret_cast<const float2*>(all + w * 512);
        t.x += f.x; t.y += f.y;
      }
      const int r0 = (p.chunk0 + i0 + i) * DC_T + 8 * tile + 2 * j;
      float* dst = a.o + (size_t)(seq.row0 + r0) * a.ld_o + (size_t)h * VP + vt * 16 + g + 4 * c;
      if (r0 < seq.n) dst[0] = t.x;
      if (r0 + 1 < seq.n) dst[a.ld_o] = t.y;
    }
  };
  float qs[2][4];
  for (int i = 0; i < n_chunks; ++i) {
    mbar_wait_bounded(smem_u32(&bar_full[at]), phase, cta_abort, p.status, NFN_ERR_WAIT_FULL);
    const unsigned char* stage = dc_smem + at * STAGE;
#pragma unroll
    for (int kk = 0; kk < DS_K; ++kk) {
      split_bf16(s[2 * kk][0], s[2 * kk][1], hi[kk][0], lo[kk][0]);
      split_bf16(s[2 * kk][2], s[2 * kk][3], hi[kk][1], lo[kk][1]);
      split_bf16(s[2 * kk + 1][0], s[2 * kk + 1][1], hi[kk][2], lo[kk][2]);
      split_bf16(s[2 * kk + 1][2], s[2 * kk + 1][3], hi[kk][3], lo[kk][3]);
    }
    if (i > 0) put(i, 2, qs);
    if constexpr (CORRECTIONS) {
      float ws[2][4];
      product(stage, 0, ws);
      put(i, 0, ws);
    }
    // every warp is done with chunk i - 2 here: its stage takes the next load
    __syncthreads();
    const int gave_up = *cta_abort;                      // set before the barrier by a thread whose wait ran out: all leave together
    if (tid == 0 && i > 1 && i - 2 + STAGES < n_chunks) load(i - 2 + STAGES);
    float4 w0 = make_float4(0.f, 0.f, 0.f, 0.f), w1 = w0;
    if constexpr (CORRECTIONS) {
      w0 = sum(i, 0);
      w1 = sum(i, 1);
    }
    product(stage, WT - 2, qs);
    // U^T, as the A operand of S'^T = e^G_last S^T + U^T K
    const float* tv = reinterpret_cast<const float*>(stage + BLOCK) + (warp / KS) * 512 + lane * 4;
    const float4 v0 = *reinterpret_cast<const float4*>(tv), v1 = *reinterpret_cast<const float4*>(tv + 128);
    uint32_t uh[4], ul[4];
    split_bf16(v0.x - w0.x, v0.y - w0.y, uh[0], ul[0]);
    split_bf16(v0.z - w0.z, v0.w - w0.w, uh[1], ul[1]);
    split_bf16(v1.x - w1.x, v1.y - w1.y, uh[2], ul[2]);
    split_bf16(v1.z - w1.z, v1.w - w1.w, uh[3], ul[3]);
    const float* gamma = reinterpret_cast<const float*>(stage + dc_gamma_at(DK, CORRECTIONS)) + DS_CH * ks + 2 * j;
    uint4 kb[DS_N];
#pragma unroll
    for (int t = 0; t < DS_N; ++t) {
      const float2 f = *reinterpret_cast<const float2*>(gamma + 8 * t);
      kb[t] = *reinterpret_cast<const uint4*>(stage + dc_piece<CORRECTIONS>(WT * (DK / 16) + DS_N * ks + t, lane, true));
      s[t][0] *= f.x; s[t][1] *= f.y; s[t][2] *= f.x; s[t][3] *= f.y;
    }
#pragma unroll
    for (int t = 0; t < DS_N; ++t) dc_mma(s[t], uh, kb[t].x, kb[t].z);
#pragma unroll
    for (int t = 0; t < DS_N; ++t) dc_mma(s[t], uh, kb[t].y, kb[t].w);
    if constexpr (CORRECTIONS) {                         // values on their own are bf16: nothing was left out
#pragma unroll
      for (int t = 0; t < DS_N; ++t) dc_mma(s[t], ul, kb[t].x, kb[t].z);
    }
    if (gave_up) break;
    if (i > 0) read_out(i - 1, i);
    if (++at == STAGES) { at = 0; phase ^= 1; }
  }
  if (!*cta_abort) put(n_chunks, 2, qs);
  __syncthreads();
  if (!*cta_abort) read_out(n_chunks - 1, n_chunks);
  if (*cta_abort) {
    for (int i = 0; i < 64; ++i) __nanosleep(1000);     // copies in flight land
    return;
  }
  if (!on || i0 + n_chunks < here) return;                        // the last segment leaves the state
#pragma unroll
  for (int t = 0; t < DS_N; ++t)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int d = DS_CH * ks + 8 * t + 2 * j + (e & 1);
      if (d < DP) st[(size_t)d * VP + (e >> 1) * 8] = s[t][e];
    }
}

// What each segment but the last adds to the state and leaves of the one before it. Roles and fragments as in the scan.
constexpr int SG_STAGES = 4;
__host__ __device__ constexpr int sg_stage_bytes(int ks) { return DS_CH * ks * 68 + DS_WARPS / ks * 1024; }      // K, e^G_last; V of the CTA's column tiles
template <int KS>
__global__ void __launch_bounds__(DS_WARPS * 32)
segment_state_kernel(const DeltaChunkParams p) {
  constexpr int DK = DS_CH * KS, TILES = DS_WARPS / KS, BLOCK = dc_block_bytes(DK, false), PART = DK * 68, STAGE = sg_stage_bytes(KS);
  extern __shared__ __align__(128) unsigned char dc_smem[];       // [SG_STAGES][STAGE]
  __shared__ __align__(8) uint64_t bar_full[SG_STAGES];
  __shared__ int cta_abort_s;
  volatile int* cta_abort = &cta_abort_s;
  const nfn_delta_args& a = p.a;
  const int sq = blockIdx.z / (p.segs - 1), seg = blockIdx.z % (p.segs - 1), i0 = seg * p.seg_chunks;
  const nfn_seq_rows seq = a.seqs[sq];
  const int total = (seq.n + DC_T - 1) / DC_T, here = min(p.n_chunks, total - p.chunk0);
  if (seq.slot < 0 || i0 >= here) return;
  const int n_chunks = i0 + p.seg_chunks < here ? p.seg_chunks : 0;      // 0: the last one, only the state before the round is noted
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, j = lane & 3;
  const int ks = warp % KS, h = blockIdx.y, DP = a.dim_p, VP = a.vdim_p;
  const int vt = blockIdx.x * TILES + warp / KS, tiles = min(TILES, VP / 16 - (int)blockIdx.x * TILES);
  const bool on = vt * 16 < VP;
  const unsigned char* blocks = p.blocks + (((size_t)sq * p.n_chunks + i0) * a.heads + h) * BLOCK + DK * 64;
  const float* uo = p.uo + (((size_t)sq * p.n_chunks + i0) * a.heads + h) * dc_uo_floats(VP) + blockIdx.x * TILES * 512;
  const size_t block_step = (size_t)a.heads * BLOCK, uo_step = (size_t)a.heads * dc_uo_floats(VP);
  auto load = [&](int i) {
    const uint32_t bar = smem_u32(&bar_full[i % SG_STAGES]), dst = smem_u32(dc_smem + (i % SG_STAGES) * STAGE);
    mbar_expect_tx(bar, PART + tiles * 1024);
    dc_bulk_load(dst, blocks + i * block_step, PART, bar);
    for (int t = 0; t < tiles; ++t) dc_bulk_load(dst + PART + t * 1024, uo + i * uo_step + t * 512, 1024, bar);
  };
  if (tid == 0) {
    cta_abort_s = 0;
    for (int s = 0; s < SG_STAGES; ++s) mbar_init(smem_u32(&bar_full[s]), 1);
    fence_mbar_init();
    for (int i = 0; i < min(SG_STAGES, n_chunks); ++i) load(i);
  }
  const size_t cell = ((size_t)sq * p.segs + seg) * a.heads + h;
  float s[DS_N][4], left[DS_N][2];
#pragma unroll
  for (int t = 0; t < DS_N; ++t) {
    left[t][0] = left[t][1] = 1.f;
#pragma unroll
    for (int e = 0; e < 4; ++e) s[t][e] = 0.f;
  }
  if (seg == 0 && on) {
    const float* st = a.state + ((size_t)seq.slot * a.heads + h) * DP * VP + vt * 16 + g;
    float* init = p.seg_init + ((size_t)sq * a.heads + h) * DP * VP + vt * 16 + g;
    const bool fresh = seq.pos0 == 0 && p.chunk0 == 0;
#pragma unroll
    for (int t = 0; t < DS_N; ++t)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int d = DS_CH * ks + 8 * t + 2 * j + (e & 1);
        if (d < DP) {
          s[t][e] = fresh ? 0.f : st[(size_t)d * VP + (e >> 1) * 8];
          init[(size_t)d * VP + (e >> 1) * 8] = s[t][e];
        }
      }
  }
  __syncthreads();
  for (int i = 0; i < n_chunks; ++i) {
    mbar_wait_bounded(smem_u32(&bar_full[i % SG_STAGES]), (i / SG_STAGES) & 1, cta_abort, p.status, NFN_ERR_WAIT_FULL);
    const unsigned char* stage = dc_smem + (i % SG_STAGES) * STAGE;
    const float* tv = reinterpret_cast<const float*>(stage + PART) + (on ? warp / KS : 0) * 256 + lane * 4;
    const float4 v0 = *reinterpret_cast<const float4*>(tv), v1 = *reinterpret_cast<const float4*>(tv + 128);
    const uint32_t uh[4] = {pack_bf16x2(v0.x, v0.y), pack_bf16x2(v0.z, v0.w), pack_bf16x2(v1.x, v1.y), pack_bf16x2(v1.z, v1.w)};
    const float* gamma = reinterpret_cast<const float*>(stage + DK * 64) + DS_CH * ks + 2 * j;
    uint4 kb[DS_N];
#pragma unroll
    for (int t = 0; t < DS_N; ++t) {
      const float2 f = *reinterpret_cast<const float2*>(gamma + 8 * t);
      kb[t] = *reinterpret_cast<const uint4*>(stage + dc_piece<false>(DS_N * ks + t, lane, true));
      s[t][0] *= f.x; s[t][1] *= f.y; s[t][2] *= f.x; s[t][3] *= f.y;
      left[t][0] *= f.x; left[t][1] *= f.y;
    }
#pragma unroll
    for (int t = 0; t < DS_N; ++t) dc_mma(s[t], uh, kb[t].x, kb[t].z);
#pragma unroll
    for (int t = 0; t < DS_N; ++t) dc_mma(s[t], uh, kb[t].y, kb[t].w);
    __syncthreads();                                    // every warp is done with the stage
    if (*cta_abort) break;                              // set before the barrier: all leave together
    if (tid == 0 && i + SG_STAGES < n_chunks) load(i + SG_STAGES);
  }
  if (*cta_abort) {
    for (int i = 0; i < 64; ++i) __nanosleep(1000);     // copies in flight land
    return;
  }
  if (n_chunks == 0 || !on) return;
  float* add = p.seg_state + cell * DP * VP + vt * 16 + g;
#pragma unroll
  for (int t = 0; t < DS_N; ++t)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int d = DS_CH * ks + 8 * t + 2 * j + (e & 1);
      if (d < DP) add[(size_t)d * VP + (e >> 1) * 8] = s[t][e];
    }
  if (vt == 0 && g == 0) {
    float* gm = p.seg_gamma + cell * DK + DS_CH * ks + 2 * j;
#pragma unroll
    for (int t = 0; t < DS_N; ++t) *reinterpret_cast<float2*>(gm + 8 * t) = make_float2(left[t][0], left[t][1]);
  }
}

template <int KS>
static int launch_segments(const DeltaChunkParams& p, cudaStream_t st) {
  constexpr int SMEM = SG_STAGES * sg_stage_bytes(KS);
  auto kern = segment_state_kernel<KS>;
  static bool raised[64] = {};
  int dev = 0;
  cudaGetDevice(&dev);
  if (SMEM > 40 * 1024 && !raised[dev & 63]) {
    if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, SMEM) != cudaSuccess) return launch_check("segment_state attr", 0);
    raised[dev & 63] = true;
  }
  kern<<<dim3(ceil_div(p.a.vdim_p, 16 * (DS_WARPS / KS)), p.a.heads, p.a.n_seqs * (p.segs - 1)), DS_WARPS * 32, SMEM, st>>>(p);
  return launch_check("segment_state");
}

template <int KS, bool CORRECTIONS>
static int launch_scan(const DeltaChunkParams& p, cudaStream_t st) {
  constexpr int SMEM = ds_stages(KS) * ds_stage_bytes(KS, CORRECTIONS) + 2 * DS_WARPS * 512 * 4;
  auto kern = delta_scan_kernel<KS, CORRECTIONS>;
  static bool raised[64] = {};
  int dev = 0;
  cudaGetDevice(&dev);
  if (SMEM > 48 * 1024 && !raised[dev & 63]) {
    if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, SMEM) != cudaSuccess) return launch_check("delta_scan attr", 0);
    raised[dev & 63] = true;
  }
  kern<<<dim3(ceil_div(p.a.vdim_p, 16 * (DS_WARPS / KS)), p.a.heads, p.a.n_seqs * (CORRECTIONS ? 1 : p.segs)), DS_WARPS * 32, SMEM, st>>>(p);
  return launch_check("delta_scan");
}

int chunk_scan(const DeltaChunkParams& p, bool corrections, cudaStream_t st) {
  if (corrections) return p.dk == 64 ? launch_scan<1, true>(p, st) : p.dk == 128 ? launch_scan<2, true>(p, st) : launch_scan<4, true>(p, st);
  if (p.segs > 1)
    if (const int rc = p.dk == 64 ? launch_segments<1>(p, st) : p.dk == 128 ? launch_segments<2>(p, st) : launch_segments<4>(p, st)) return rc;
  return p.dk == 64 ? launch_scan<1, false>(p, st) : p.dk == 128 ? launch_scan<2, false>(p, st) : launch_scan<4, false>(p, st);
}

template <int NT>
static int launch_prepare(const DeltaChunkParams& p, cudaStream_t st) {
  constexpr int SMEM = std::max(64 * (NT == 128 ? 136 : NT + 4) * 4, dc_block_bytes(2 * NT, true));
  auto kern = delta_prepare_kernel<NT>;
  static bool raised[64] = {};
  int dev = 0;
  cudaGetDevice(&dev);
  if (!raised[dev & 63]) {
    if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, SMEM) != cudaSuccess ||
        cudaFuncSetAttribute(kern, cudaFuncAttributePreferredSharedMemoryCarveout, 100) != cudaSuccess)
      return launch_check("delta_prepare attr", 0);
    raised[dev & 63] = true;
  }
  kern<<<dim3(p.n_chunks, p.a.heads, p.a.n_seqs), NT, SMEM, st>>>(p);
  return launch_check("delta_prepare");
}

}  // namespace nfn

using namespace nfn;

extern "C" long long nfn_delta_chunk_workspace_bytes(int heads, int dim_p, int vdim_p, int max_seqs) {
  if (dim_p > 256) return 0;
  const int dk = dim_p <= 64 ? 64 : dim_p <= 128 ? 128 : 256;
  // at least one chunk of every head and sequence
  return std::max<long long>(DC_WORKSPACE, (long long)max_seqs * heads * (dc_block_bytes(dk, true) + dc_uo_floats(vdim_p) * 4LL));
}

extern "C" int nfn_delta_chunks(const nfn_delta_args* args, int max_rows, void* workspace, long long workspace_bytes, nfn_stream_t stream) {
  if (!args) return fail(-1, "delta rule: null args");
  if (args->n_seqs <= 0 || max_rows <= 0) return 0;
  if (const char* why = delta_args_problem(*args)) return fail(-1, why);
  if (args->f32 || args->dim_p > 256) return fail(-1, "delta rule: chunks are for bf16 activations and at most 256 key channels");
  DeltaChunkParams p{};
  p.a = *args;
  p.segs = 1;
  p.dk = args->dim_p <= 64 ? 64 : args->dim_p <= 128 ? 128 : 256;
  p.status = status_ptr();
  const long long per_chunk = (long long)args->n_seqs * args->heads * (dc_block_bytes(p.dk, true) + dc_uo_floats(args->vdim_p) * 4LL);
  const int total = ceil_div(max_rows, DC_T), round = (int)std::min<long long>(total, workspace_bytes / per_chunk);
  if (!workspace || round < 1) return fail(-1, "delta rule: the workspace holds no chunk");
  p.blocks = static_cast<unsigned char*>(workspace);
  p.uo = reinterpret_cast<float*>(p.blocks + (size_t)round * args->n_seqs * args->heads * dc_block_bytes(p.dk, true));
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  for (p.chunk0 = 0; p.chunk0 < total; p.chunk0 += round) {
    p.n_chunks = std::min(round, total - p.chunk0);
    int rc = p.dk == 64 ? launch_prepare<32>(p, st) : p.dk == 128 ? launch_prepare<64>(p, st) : launch_prepare<128>(p, st);
    if (rc == 0) rc = chunk_scan(p, true, st);
    if (rc) return rc;
  }
  return 0;
}
