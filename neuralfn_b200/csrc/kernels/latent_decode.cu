// Attention of single query rows over latent caches: one cached row per token, [latent | rotated key part], is key and value of every head. The
// queries come with the key projection folded in (q . W_uk c = W_uk^T q . c), the outputs are weighted sums of latents whose value
// projection follows, so a token's row is read once for all heads and twice from shared memory: as the key operand and, transposed by
// ldmatrix, as the value operand.
//
// One CTA takes one row, a block of 16 or 32 heads and a share of the visible pages. Per page: sixteen warps form the scores (8 keys x half of the
// channels each, on mma.m16n8k16), a softmax pass merges the halves, then each warp owns a slice of the latent channels of the output.
// Pages arrive one ahead, a bulk copy per row (rows in shared memory are 16 bytes longer than in the page: no bank conflicts). Scores, softmax
// and sums are fp32; a second launch merges the shares, in order.
#include <algorithm>

#include "common.h"
#include "paged.cuh"

namespace nfn {

constexpr int LD_WARPS = 16, LD_THREADS = LD_WARPS * 32, LD_S = NFN_PAGE + 4, LD_P = NFN_PAGE + 8;

struct LatentDecodeParams {
  nfn_paged_attention_args a;
  int splits, pitch;           // pitch: elements between rows in shared memory (an odd number of 16-byte pieces: no bank conflicts)
  float* partial;              // [rows][heads][splits][vdim_p] values
  float2* stats;               // [rows][heads][splits] maximum and sum
  int* status;
};

__device__ __forceinline__ void ld_x4(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ld_x4_t(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ld_mma(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ld_bulk(uint32_t dst, const void* src, uint32_t bytes, uint32_t bar) {
  asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"(dst), "l"(src), "r"(bytes), "r"(bar) : "memory");
}

// MT: 16-head tiles of a CTA; VN: 8-channel tiles of the output per warp (an upper bound)
template <int MT, int VN>
__global__ void __launch_bounds__(LD_THREADS)
latent_decode_kernel(const LatentDecodeParams p) {
  constexpr int NH = MT * 16;
  extern __shared__ __align__(16) unsigned char ld_smem[];
  __shared__ float s_alpha[NH], s_m[NH], s_l[NH];
  __shared__ __align__(8) uint64_t bar_full[2];
  __shared__ int abort_s;
  const nfn_paged_attention_args& a = p.a;
  const int row = a.row0 + blockIdx.z, slot = a.row_slot[row];
  if (slot < 0) return;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, j = lane & 3;
  const int DP = a.dim_p, VP = a.vdim_p, pitch = p.pitch;
  const int h0 = blockIdx.y * NH, n_heads = min(NH, a.heads - h0);
  __nv_bfloat16* sQ = reinterpret_cast<__nv_bfloat16*>(ld_smem);               // [NH][pitch]
  __nv_bfloat16* sK = sQ + (size_t)NH * pitch;                                 // [2][64][pitch]
  float* sS = reinterpret_cast<float*>(sK + (size_t)2 * NFN_PAGE * pitch);     // [2][NH][LD_S]: the two halves' scores
  __nv_bfloat16* sP = reinterpret_cast<__nv_bfloat16*>(sS + 2 * NH * LD_S);    // [NH][LD_P]
  const int pos = a.row_pos[row], lo = first_visible(a, pos);
  const int page0 = lo / NFN_PAGE, n_pages = pos / NFN_PAGE + 1 - page0;
  const int p_lo = (int)((long long)n_pages * blockIdx.x / p.splits), p_hi = (int)((long long)n_pages * (blockIdx.x + 1) / p.splits);
  const int* table = a.table + (size_t)slot * a.table_ld;
  const __nv_bfloat16* pool = static_cast<const __nv_bfloat16*>(a.k_pool);
  const int vecs = DP / 8;
  auto load = [&](int i) {                                       // warp 0: two rows per lane
    const uint32_t bar = smem_u32(&bar_full[i & 1]), dst = smem_u32(sK + (size_t)(i & 1) * NFN_PAGE * pitch);
    const __nv_bfloat16* src = pool + (size_t)table[page0 + i] * NFN_PAGE * DP;
    if (lane == 0) mbar_expect_tx(bar, (uint32_t)(NFN_PAGE * DP * 2));
    __syncwarp();
#pragma unroll
    for (int r = lane; r < NFN_PAGE; r += 32) ld_bulk(dst + (uint32_t)(r * pitch) * 2, src + (size_t)r * DP, (uint32_t)DP * 2, bar);
  };
  if (tid == 0) {
    abort_s = 0;
    mbar_init(smem_u32(&bar_full[0]), 1);
    mbar_init(smem_u32(&bar_full[1]), 1);
    fence_mbar_init();
  }
  __syncthreads();
  if (warp == 0 && p_lo < p_hi) load(p_lo);
  {
    const __nv_bfloat16* q = static_cast<const __nv_bfloat16*>(a.q) + (size_t)row * a.ld_q + (size_t)h0 * DP;
    const uint4 zero4 = make_uint4(0u, 0u, 0u, 0u);
    for (int x = tid; x < NH * vecs; x += LD_THREADS) {
      const int r = x / vecs, c = x - r * vecs;
      *reinterpret_cast<uint4*>(sQ + (size_t)r * pitch + c * 8) = r < n_heads ? *reinterpret_cast<const uint4*>(q + (size_t)x * 8) : zero4;
    }
    if (tid < NH) {
      s_m[tid] = -INFINITY;
      s_l[tid] = 0.f;
    }
  }
  const float mul = a.scale * 1.4426950408889634f;
  float acc[MT][VN][4];
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int v = 0; v < VN; ++v)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[m][v][e] = 0.f;
  const int kg = warp & 7, half = warp >> 3, steps = DP / 16, ks0 = steps * half / 2, ks1 = steps * (half + 1) / 2;
  const uint32_t aq = smem_u32(sQ) + (uint32_t)((lane & 15) * pitch + (lane >> 4) * 8) * 2;
  const uint32_t ap = smem_u32(sP) + (uint32_t)((lane & 15) * LD_P + (lane >> 4) * 8) * 2;
  const uint32_t bk = (uint32_t)((kg * 8 + (lane & 7)) * pitch + (lane >> 3) * 8) * 2;
  const uint32_t bv = (uint32_t)((((lane >> 3) & 1) * 8 + (lane & 7)) * pitch + warp * VN * 8 + (lane >> 4) * 8) * 2;

  __syncthreads();                                                  // queries are in place
  for (int i = p_lo; i < p_hi; ++i) {
    if (warp == 0 && i + 1 < p_hi) load(i + 1);
    mbar_wait_bounded(smem_u32(&bar_full[i & 1]), ((i - p_lo) >> 1) & 1, &abort_s, p.status, NFN_ERR_WAIT_FULL);
    const uint32_t stage = smem_u32(sK + (size_t)(i & 1) * NFN_PAGE * pitch);
    // ---- scores: 8 keys, half of the channels, two steps of 16 per load of keys ----
    float s[MT][4];
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int e = 0; e < 4; ++e) s[m][e] = 0.f;
#pragma unroll 3
    for (int k = ks0; k < ks1; k += 2) {
      uint32_t b[4], q[MT][4];
      ld_x4(b, stage + bk + k * 32);
#pragma unroll
      for (int m = 0; m < MT; ++m) ld_x4(q[m], aq + (uint32_t)(m * 16 * pitch) * 2 + k * 32);
#pragma unroll
      for (int m = 0; m < MT; ++m) ld_mma(s[m], q[m], b[0], b[1]);
      if (k + 1 < ks1) {
#pragma unroll
        for (int m = 0; m < MT; ++m) ld_x4(q[m], aq + (uint32_t)(m * 16 * pitch) * 2 + k * 32 + 32);
#pragma unroll
        for (int m = 0; m < MT; ++m) ld_mma(s[m], q[m], b[2], b[3]);
      }
    }
#pragma unroll
    for (int m = 0; m < MT; ++m) {
      float* dst = sS + (size_t)(half * NH + m * 16 + g) * LD_S + kg * 8 + 2 * j;
      *reinterpret_cast<float2*>(dst) = make_float2(s[m][0], s[m][1]);
      *reinterpret_cast<float2*>(dst + 8 * LD_S) = make_float2(s[m][2], s[m][3]);
    }
    __syncthreads();
    if (*static_cast<volatile int*>(&abort_s)) break;               // a wait ran out: set before the barrier, so all leave together
    // ---- softmax: LD_THREADS / NH threads per head, a few keys each ----
    {
      constexpr int SHARE = LD_THREADS / NH, KEYS = NFN_PAGE / SHARE;
      const int h = tid / SHARE, k0 = tid % SHARE * KEYS, key0 = (page0 + i) * NFN_PAGE + k0;
      const float *s0 = sS + (size_t)h * LD_S + k0, *s1 = s0 + (size_t)NH * LD_S;
      float x[KEYS], mx = -INFINITY;
#pragma unroll
      for (int e = 0; e < KEYS; ++e) {
        x[e] = key0 + e >= lo && key0 + e <= pos ? (s0[e] + s1[e]) * mul : -INFINITY;
        mx = fmaxf(mx, x[e]);
      }
#pragma unroll
      for (int o = 1; o < SHARE; o <<= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
      const float m_old = s_m[h], m_new = fmaxf(m_old, mx);         // every page holds a visible key: finite
      float sum = 0.f;
#pragma unroll
      for (int e = 0; e < KEYS; ++e) {
        x[e] = exp2f(x[e] - m_new);
        sum += x[e];
      }
#pragma unroll
      for (int o = 1; o < SHARE; o <<= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
#pragma unroll
      for (int e = 0; e < KEYS; e += 2) *reinterpret_cast<uint32_t*>(sP + (size_t)h * LD_P + k0 + e) = pack_bf16x2(x[e], x[e + 1]);
      __syncwarp();                                                 // a head's threads share a warp: its maximum is read by all before it changes
      if (tid % SHARE == 0) {
        const float alpha = exp2f(m_old - m_new);                   // 0 on the first page
        s_alpha[h] = alpha;
        s_l[h] = s_l[h] * alpha + sum;
        s_m[h] = m_new;
      }
    }
    __syncthreads();
    // ---- output: this warp's latent channels ----
#pragma unroll
    for (int m = 0; m < MT; ++m) {
      const float a0 = s_alpha[m * 16 + g], a1 = s_alpha[m * 16 + g + 8];
#pragma unroll
      for (int v = 0; v < VN; ++v) {
        acc[m][v][0] *= a0; acc[m][v][1] *= a0; acc[m][v][2] *= a1; acc[m][v][3] *= a1;
      }
    }
#pragma unroll
    for (int kk = 0; kk < NFN_PAGE / 16; ++kk) {
      uint32_t pf[MT][4];
#pragma unroll
      for (int m = 0; m < MT; ++m) ld_x4(pf[m], ap + (uint32_t)(m * 16 * LD_P) * 2 + kk * 32);
#pragma unroll
      for (int v = 0; v < VN; v += 2) {
        if ((warp * VN + v) * 8 >= VP) break;                       // channels come in whole sixteens
        uint32_t b[4];
        ld_x4_t(b, stage + bv + (uint32_t)(kk * 16 * pitch) * 2 + v * 16);
#pragma unroll
        for (int m = 0; m < MT; ++m) {
          ld_mma(acc[m][v], pf[m], b[0], b[1]);
          ld_mma(acc[m][v + 1], pf[m], b[2], b[3]);
        }
      }
    }
    __syncthreads();                                                // the stage takes the page after the next
  }
  __syncthreads();
  if (abort_s) {
    for (int i = 0; i < 64; ++i) __nanosleep(1000);                 // copies in flight land
    return;
  }

  __nv_bfloat16* out = static_cast<__nv_bfloat16*>(a.out) + (size_t)row * a.ld_o + (size_t)h0 * VP;
  const size_t cell = (size_t)blockIdx.z * a.heads + h0;
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int e2 = 0; e2 < 2; ++e2) {
      const int h = m * 16 + g + 8 * e2;
      const float inv = s_l[h] > 0.f ? 1.f / s_l[h] : 0.f;
      if (h >= n_heads) continue;
      float* part = p.partial + ((cell + h) * p.splits + blockIdx.x) * VP;
#pragma unroll
      for (int v = 0; v < VN; ++v) {
        const int c = (warp * VN + v) * 8 + 2 * j;
        if (c >= VP) break;
        if (p.splits == 1) *reinterpret_cast<uint32_t*>(out + (size_t)h * VP + c) = pack_bf16x2(acc[m][v][2 * e2] * inv, acc[m][v][2 * e2 + 1] * inv);
        else *reinterpret_cast<float2*>(part + c) = make_float2(acc[m][v][2 * e2], acc[m][v][2 * e2 + 1]);
      }
      if (p.splits > 1 && warp == 0 && j == 0) p.stats[(cell + h) * p.splits + blockIdx.x] = make_float2(s_m[h], s_l[h]);
    }
}

// A CTA takes one head of a row, a thread four channels.
__global__ void __launch_bounds__(128)
latent_merge_kernel(const LatentDecodeParams p) {
  const nfn_paged_attention_args& a = p.a;
  const int row = a.row0 + blockIdx.y, h = blockIdx.x, c = threadIdx.x * 4;
  if (a.row_slot[row] < 0 || c >= a.vdim_p) return;
  const size_t cell = (size_t)blockIdx.y * a.heads + h;
  const float2* stats = p.stats + cell * p.splits;
  const float* part = p.partial + cell * p.splits * a.vdim_p + c;
  float m = -INFINITY, l = 0.f;
  float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
  for (int s0 = 0; s0 < p.splits; s0 += 8) {
    float2 t[8];
    float4 v[8];
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const int s = min(s0 + i, p.splits - 1);
      t[i] = stats[s];
      v[i] = load4(part + (size_t)s * a.vdim_p);
      if (s0 + i >= p.splits) t[i] = make_float2(-INFINITY, 0.f);
    }
    float m_new = m;
#pragma unroll
    for (int i = 0; i < 8; ++i) m_new = fmaxf(m_new, t[i].x);
    if (m_new == -INFINITY) continue;                       // shares without pages
    const float keep = exp2f(m - m_new);
    l *= keep;
    o.x *= keep; o.y *= keep; o.z *= keep; o.w *= keep;
    m = m_new;
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const float f = exp2f(t[i].x - m_new);
      l += f * t[i].y;
      o.x += f * v[i].x; o.y += f * v[i].y; o.z += f * v[i].z; o.w += f * v[i].w;
    }
  }
  const float inv = 1.f / l;
  store4(static_cast<__nv_bfloat16*>(a.out) + (size_t)row * a.ld_o + (size_t)h * a.vdim_p + c, make_float4(o.x * inv, o.y * inv, o.z * inv, o.w * inv));
}

template <int MT, int VN>
static int launch_latent_decode(LatentDecodeParams p, size_t smem, cudaStream_t st) {
  auto kern = latent_decode_kernel<MT, VN>;
  static size_t raised[64] = {};
  int dev = 0;
  cudaGetDevice(&dev);
  if (smem > 40 * 1024 && raised[dev & 63] < smem) {
    if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess) return launch_check("latent_decode attr", 0);
    raised[dev & 63] = smem;
  }
  const nfn_paged_attention_args a = p.a;
  const int blocks = ceil_div(a.heads, MT * 16);
  for (int r = 0; r < a.rows; r += 65535) {
    p.a.row0 = a.row0 + r;
    const int n = std::min(a.rows - r, 65535);
    kern<<<dim3(p.splits, blocks, n), LD_THREADS, smem, st>>>(p);
    if (p.splits > 1) latent_merge_kernel<<<dim3(a.heads, n), 128, 0, st>>>(p);
  }
  return launch_check("latent_decode", p.splits > 1 ? 2 : 1);
}

// 1: sizes outside the kernel's limits
int latent_decode(const nfn_paged_attention_args& a, cudaStream_t st) {
  if (a.vdim_p > 512 || (a.dim_p & 15) || (a.vdim_p & 15) || (a.ld_q & 7) || a.slopes || a.softcap > 0.f || a.sink || a.keep_first > 0 || a.gate) return 1;
  LatentDecodeParams p;
  p.a = a;
  p.pitch = a.dim_p + 8;
  p.status = status_ptr();
  const int mt = a.heads > 16 ? 2 : 1, nh = 16 * mt;
  const size_t smem = (size_t)(nh + 2 * NFN_PAGE) * p.pitch * 2 + (size_t)2 * nh * LD_S * 4 + (size_t)nh * LD_P * 2;
  if (smem > 220 * 1024) return 1;
  // one wave of what is resident at a time, at least one page each
  const long long ctas = (long long)a.rows * ceil_div(a.heads, nh), cells = (long long)a.rows * a.heads;
  const int resident = (int)std::max<size_t>(1, (size_t)(220 * 1024) / smem);
  long long splits = std::min<long long>(ceil_div(a.max_keys, NFN_PAGE) + 1, std::max<long long>(1, (long long)sm_count() * std::min(resident, 4) / ctas));
  splits = std::min<long long>(std::min<long long>(splits, 64), (a.workspace_bytes - PAGED_COUNTER_BYTES) / (cells * (a.vdim_p * 4 + 8)));
  p.splits = (int)std::max<long long>(splits, 1);
  p.partial = reinterpret_cast<float*>(static_cast<char*>(a.workspace) + PAGED_COUNTER_BYTES);
  p.stats = reinterpret_cast<float2*>(p.partial + cells * p.splits * a.vdim_p);
  if (mt == 1) return a.vdim_p <= 256 ? launch_latent_decode<1, 2>(p, smem, st) : launch_latent_decode<1, 4>(p, smem, st);
  return a.vdim_p <= 256 ? launch_latent_decode<2, 2>(p, smem, st) : launch_latent_decode<2, 4>(p, smem, st);
}

}  // namespace nfn
