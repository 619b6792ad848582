// The bonus recurrence over prompt portions, sixteen tokens at a time (bf16 activations; state and everything that enters it fp32).
//
// Inside a chunk let G_r be the running sum of the log decays (per key channel) up to and with token r and S the state before the chunk. Token r reads
// the state left by token r - 1, so with
//   P_rj = sum_c r_rc k_jc e^(G_(r-1)c - G_jc)  (j < r),   P_rr = sum_c r_rc u_c k_rc
// the read-outs are O = P V + Q S with Q_r = e^G_(r-1) r_r, and the next state is S' = e^G_last S + K^T V with K_j = k_j e^(G_last - G_j). Exponents are sums
// of decays between two tokens, never positive. wkv_prepare_kernel forms Q, K, V and P V of all chunks at once (one CTA per chunk and head, two
// channels per thread); the scan of delta_chunk.cu runs from state to state with U = V.
#include <algorithm>

#include "chunk_scan.cuh"
#include "common.h"
#include "wkv.cuh"

namespace nfn {

// A token's log2 decay is cut off here: what is left after it, 2^-64, is below the rounding of every other term, and sums of sixteen stay small
// enough that their differences keep their digits.
constexpr float WC_FLOOR = -64.f;

struct WkvChunkParams {
  DeltaChunkParams c;
  nfn_wkv_args a;
};

// NT threads, two neighbouring channels each (dk = 2 NT)
template <int NT>
__global__ void __launch_bounds__(NT, 512 / NT)
wkv_prepare_kernel(const WkvChunkParams p) {
  constexpr int PITCH = NT == 128 ? 136 : NT + 4;                 // partial sums [60 values][NT]; rows are read in 16-byte pieces
  extern __shared__ __align__(128) unsigned char dc_smem[];       // partial sums, then the operand block
  __shared__ __align__(16) float sP[DC_T][DC_T + 4];
  const nfn_wkv_args& a = p.a;
  const nfn_seq_rows seq = a.seqs[blockIdx.z];
  const int r0 = (p.c.chunk0 + blockIdx.x) * DC_T, n = min(DC_T, seq.n - r0);
  if (seq.slot < 0 || n <= 0) return;
  const int tid = threadIdx.x, h = blockIdx.y, DP = a.dim_p, HD = a.heads * DP, dk = p.c.dk;
  const size_t row0 = (size_t)(seq.row0 + r0);
  const __nv_bfloat16* x = static_cast<const __nv_bfloat16*>(a.rkv) + row0 * a.ld_rkv + (size_t)h * DP;
  const int c0 = 2 * tid;
  const bool on = c0 < DP;
  float* part = reinterpret_cast<float*>(dc_smem);

  float q[DC_T][2], k[DC_T][2], G[DC_T][2];                       // G[r]: sum up to and with token r
  {
    uint32_t qw[DC_T], kw[DC_T];
#pragma unroll
    for (int r = 0; r < DC_T; ++r) {
      const bool live = on && r < n;
      qw[r] = live ? *reinterpret_cast<const uint32_t*>(x + (size_t)r * a.ld_rkv + c0) : 0u;
      kw[r] = live ? *reinterpret_cast<const uint32_t*>(x + (size_t)r * a.ld_rkv + HD + c0) : 0u;
      const float2 z = live ? *reinterpret_cast<const float2*>(a.z + (row0 + r) * a.ld_z + (size_t)h * DP + c0) : make_float2(0.f, 0.f);
      G[r][0] = z.x;
      G[r][1] = z.y;
    }
    const float2 w0 = on ? unpack_bf16x2(*reinterpret_cast<const uint32_t*>(static_cast<const __nv_bfloat16*>(a.w0) + (size_t)h * DP + c0)) : make_float2(0.f, 0.f);
    const float2 u = on ? unpack_bf16x2(*reinterpret_cast<const uint32_t*>(static_cast<const __nv_bfloat16*>(a.u) + (size_t)h * DP + c0)) : make_float2(0.f, 0.f);
    float s0 = 0.f, s1 = 0.f;
#pragma unroll
    for (int r = 0; r < DC_T; ++r) {
      const float2 fq = unpack_bf16x2(qw[r]), fk = unpack_bf16x2(kw[r]);
      q[r][0] = fq.x; q[r][1] = fq.y; k[r][0] = fk.x; k[r][1] = fk.y;
      if (r < n) {
        s0 += fmaxf(expf(G[r][0] + w0.x) * -1.4426950408889634f, WC_FLOOR);
        s1 += fmaxf(expf(G[r][1] + w0.y) * -1.4426950408889634f, WC_FLOOR);
      }
      G[r][0] = s0;
      G[r][1] = s1;
      part[r * PITCH + tid] = fq.x * (u.x * fk.x) + fq.y * (u.y * fk.y);
    }
  }
  // ---- the bonus: 16 sums over the channels, NT / 16 neighbouring threads each ----
  __syncthreads();
  {
    constexpr int SHARE = NT / 16;
    const int v = tid / SHARE;
    const float* src = part + v * PITCH + tid % SHARE * 16;
    float4 f = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const float4 g = *reinterpret_cast<const float4*>(src + 4 * i);
      f.x += g.x; f.y += g.y; f.z += g.z; f.w += g.w;
    }
    float t = (f.x + f.y) + (f.z + f.w);
#pragma unroll
    for (int o = 1; o < SHARE; o <<= 1) t += __shfl_xor_sync(0xffffffffu, t, o);
    sP[v][v] = t;
  }
  __syncthreads();
  // ---- P below its diagonal: rows r and 15 - r together have 15 values; four such pairs per pass ----
#pragma unroll
  for (int t = 0; t < 2; ++t) {
    int at = 0;
#pragma unroll
    for (int w = 0; w < 8; ++w) {
      const int r = w % 2 ? 15 - (4 * t + w / 2) : 4 * t + w / 2;
#pragma unroll
      for (int j = 0; j < DC_T - 1; ++j) {
        if (j >= r) continue;
        float k0 = k[j][0], k1 = k[j][1];
        if (j + 1 < r) {                                          // between neighbours nothing decays
          float d0 = G[r - 1][0], d1 = G[r - 1][1];
          add2f(d0, d1, d0, d1, -G[j][0], -G[j][1]);
          mul2(k0, k1, k0, k1, fast_exp2(d0), fast_exp2(d1));
        }
        part[at++ * PITCH + tid] = q[r][0] * k0 + q[r][1] * k1;
      }
    }
    __syncthreads();
#pragma unroll
    for (int v0 = 0; v0 < (NT == 32 ? 64 : 32); v0 += 32) {
      const int v = NT == 32 ? tid + v0 : NT == 64 ? tid : tid >> 1;
      if (v < 60) {                                               // NT = 128: both threads of a value agree
        const float* src = part + v * PITCH + (NT == 128 ? 4 * (tid & 1) : 0);
        float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int i = 0; i < (NT == 32 ? 8 : 16); ++i) {
          const float4 f = *reinterpret_cast<const float4*>(src + i * (NT == 128 ? 8 : 4));
          add2(s.x, s.y, f.x, f.y);
          add2(s.z, s.w, f.z, f.w);
        }
        float sum = (s.x + s.y) + (s.z + s.w);
        if (NT == 128) sum += __shfl_xor_sync(__activemask(), sum, 1);
        const int pair = v / 15, rest = v % 15, lo = 4 * t + pair;
        sP[rest < lo ? lo : 15 - lo][rest < lo ? rest : rest - lo] = sum;
      }
      if (NT != 32) break;
    }
    __syncthreads();
  }
  const size_t block = ((size_t)blockIdx.z * p.c.n_chunks + blockIdx.x) * a.heads + h;
  // ---- Q, K of this thread's channels, in the order of the scan's fragments: {first eight of the contraction: high, low; second: high, low} ----
  unsigned char* stage = dc_smem;
  *reinterpret_cast<float2*>(stage + dc_gamma_at(dk, false) + c0 * 4) = make_float2(fast_exp2(G[DC_T - 1][0]), fast_exp2(G[DC_T - 1][1]));
#pragma unroll
  for (int r = 0; r < DC_T; r += 2)
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      uint2 w;
      split_bf16(k[r][i] * fast_exp2(G[DC_T - 1][i] - G[r][i]), k[r + 1][i] * fast_exp2(G[DC_T - 1][i] - G[r + 1][i]), w.x, w.y);
      *reinterpret_cast<uint2*>(stage + dc_piece<false>(2 * (dk / 16) + (c0 + i) / 8, (c0 + i) % 8 * 4 + (r % 8) / 2, true) + (r / 8) * 8) = w;
    }
#pragma unroll
  for (int r = 0; r < DC_T; ++r) {
    uint2 f;
    split_bf16(r ? q[r][0] * fast_exp2(G[r ? r - 1 : 0][0]) : q[0][0], r ? q[r][1] * fast_exp2(G[r ? r - 1 : 0][1]) : q[0][1], f.x, f.y);
    *reinterpret_cast<uint2*>(stage + dc_piece<false>(2 * (c0 / 16) + r / 8, r % 8 * 4 + (c0 % 8) / 2, false) + (c0 % 16) / 8 * 8) = f;
  }
  // ---- V and P V of this thread's value columns ----
  float* uo = p.c.uo + block * dc_uo_floats(DP);
  for (int c = c0; c < DP; c += 2 * NT) {
    float v[DC_T][2];
#pragma unroll
    for (int r = 0; r < DC_T; ++r) {
      const float2 f = r < n ? unpack_bf16x2(*reinterpret_cast<const uint32_t*>(x + (size_t)r * a.ld_rkv + 2 * HD + c)) : make_float2(0.f, 0.f);
      v[r][0] = f.x;
      v[r][1] = f.y;
    }
    float* dst = uo + (c / 16) * 512 + (c & 7) * 16 + ((c & 15) >> 3) * 2;      // [2][2 row tiles][lane = column % 8, row pair][column half, row]
#pragma unroll
    for (int r = 0; r < DC_T; r += 2) {
      float o[2][2] = {};
#pragma unroll
      for (int e = 0; e < 2; ++e)
#pragma unroll
        for (int j4 = 0; j4 <= r + e; j4 += 4) {
          const float4 f = *reinterpret_cast<const float4*>(&sP[r + e][j4]);
          const float m[4] = {f.x, f.y, f.z, f.w};
#pragma unroll
          for (int i = 0; i < 4; ++i)
            if (j4 + i <= r + e) fma2(o[e][0], o[e][1], m[i], m[i], v[j4 + i][0], v[j4 + i][1], o[e][0], o[e][1]);
        }
      const int at = (r / 8) * 128 + ((r % 8) / 2) * 4;
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        *reinterpret_cast<float2*>(dst + i * 16 + at) = make_float2(v[r][i], v[r + 1][i]);
        *reinterpret_cast<float2*>(dst + i * 16 + 256 + at) = make_float2(o[0][i], o[1][i]);
      }
    }
  }
  // the finished operand block leaves in one bulk copy
  fence_proxy_async();
  __syncthreads();
  if (tid == 0) {
    dc_bulk_store(p.c.blocks + block * dc_block_bytes(dk, false), smem_u32(stage), dc_block_bytes(dk, false));
    asm volatile("cp.async.bulk.commit_group;" ::: "memory");
    asm volatile("cp.async.bulk.wait_group 0;" ::: "memory");
  }
}

template <int NT>
static int launch_wkv_prepare(const WkvChunkParams& p, cudaStream_t st) {
  constexpr int SMEM = std::max(60 * (NT == 128 ? 136 : NT + 4) * 4, dc_block_bytes(2 * NT, false));
  static_assert(SMEM <= 48 * 1024, "static limit of dynamic shared memory");
  wkv_prepare_kernel<NT><<<dim3(p.c.n_chunks, p.a.heads, p.a.n_seqs), NT, SMEM, st>>>(p);
  return launch_check("wkv_prepare");
}

}  // namespace nfn

using namespace nfn;

static int wkv_dk(int dim_p) { return dim_p <= 64 ? 64 : dim_p <= 128 ? 128 : 256; }

constexpr int WC_MAX_SEGS = 8, WC_MIN_SEG = 8;           // segments of a round, and fewest chunks of one
// bytes the segments of a sequence take beside the operands
static long long segment_bytes(int heads, int dim_p) { return (long long)heads * ((WC_MAX_SEGS + 1LL) * dim_p * dim_p + (long long)WC_MAX_SEGS * wkv_dk(dim_p)) * 4; }

extern "C" long long nfn_wkv_chunk_workspace_bytes(int heads, int dim_p, int max_seqs) {
  if (dim_p > 256) return 0;
  // at least one chunk of every head and sequence; segments are for few sequences
  return std::max<long long>(DC_WORKSPACE, (long long)max_seqs * heads * (dc_block_bytes(wkv_dk(dim_p), false) + dc_uo_floats(dim_p) * 4LL)) + segment_bytes(heads, dim_p);
}

extern "C" int nfn_wkv_chunks(const nfn_wkv_args* args, int max_rows, void* workspace, long long workspace_bytes, nfn_stream_t stream) {
  if (!args) return fail(-1, "wkv: null args");
  if (args->n_seqs <= 0 || max_rows <= 0) return 0;
  if (const char* why = wkv_args_problem(*args)) return fail(-1, why);
  if (args->f32 || args->dim_p > 256) return fail(-1, "wkv: chunks are for bf16 activations and at most 256 channels per head");
  WkvChunkParams p{};
  p.a = *args;
  nfn_delta_args& d = p.c.a;                     // what the scan reads
  d.heads = d.kv_heads = args->heads;
  d.dim = args->dim;
  d.dim_p = d.vdim_p = args->dim_p;
  d.state = args->state;
  d.o = args->o;
  d.ld_o = args->ld_o;
  d.seqs = args->seqs;
  d.n_seqs = args->n_seqs;
  p.c.dk = wkv_dk(args->dim_p);
  p.c.status = status_ptr();
  const int block = dc_block_bytes(p.c.dk, false);
  // where heads and columns leave SMs idle, a round runs in segments side by side
  const int ctas = ceil_div(args->dim_p, 16 * (256 / p.c.dk)) * args->heads * args->n_seqs;
  const long long seg_bytes = args->n_seqs * segment_bytes(args->heads, args->dim_p);
  int segs = std::min(WC_MAX_SEGS, 2 * sm_count() / ctas);
  // two would cost in extra passes what they gain
  if (segs > 2 && workspace_bytes > 2 * seg_bytes) workspace_bytes = (workspace_bytes - seg_bytes) / 256 * 256;
  else segs = 1;
  const long long per_chunk = (long long)args->n_seqs * args->heads * (block + dc_uo_floats(args->dim_p) * 4LL);
  const int total = ceil_div(max_rows, DC_T), round = (int)std::min<long long>(total, workspace_bytes / per_chunk);
  if (!workspace || round < 1) return fail(-1, "wkv: the workspace holds no chunk");
  p.c.blocks = static_cast<unsigned char*>(workspace);
  p.c.uo = reinterpret_cast<float*>(p.c.blocks + (size_t)round * args->n_seqs * args->heads * block);
  p.c.seg_init = reinterpret_cast<float*>(static_cast<unsigned char*>(workspace) + workspace_bytes);
  p.c.seg_state = p.c.seg_init + (size_t)args->n_seqs * args->heads * args->dim_p * args->dim_p;
  p.c.seg_gamma = p.c.seg_state + (size_t)args->n_seqs * WC_MAX_SEGS * args->heads * args->dim_p * args->dim_p;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  for (p.c.chunk0 = 0; p.c.chunk0 < total; p.c.chunk0 += round) {
    p.c.n_chunks = std::min(round, total - p.c.chunk0);
    p.c.segs = std::max(1, std::min(segs, p.c.n_chunks / WC_MIN_SEG));
    p.c.seg_chunks = ceil_div(p.c.n_chunks, p.c.segs);
    int rc = p.c.dk == 64 ? launch_wkv_prepare<32>(p, st) : p.c.dk == 128 ? launch_wkv_prepare<64>(p, st) : launch_wkv_prepare<128>(p, st);
    if (rc == 0) rc = chunk_scan(p.c, false, st);
    if (rc) return rc;
  }
  return 0;
}
