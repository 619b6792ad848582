// Attention of single query rows over latent caches (tcgen05): one cached row per token, [latent | rotated key part], is key and value of every
// head. The queries come with the key projection folded in (q . W_uk c = W_uk^T q . c), the outputs are weighted sums of latents whose value
// projection follows.
//
// One CTA takes one row, a block of up to 32 heads and a share of the visible pages. A page arrives once, as 64-channel panels [64 tokens][64 channels],
// and is used twice as it stands: as the K-major operand of the scores S = q C^T (heads are accumulator rows, the queries wait in TMEM as its
// other operand) and as the MN-major operand of the outputs, which are transposed, O^T = C^T P^T (latent channels, 128 at a time, are accumulator
// rows, heads the narrow side), so that few heads waste no accumulators. Roles: warp 0 turns scores into weights, a head per thread; warps 0 - 3
// rescale outputs, only when a maximum grew by more than 2^8, and write them, a channel per thread; one MMA warp, one TMA warp. Up to three
// pages are in shared memory or on their way.
//
// Scores, softmax and sums are fp32; a second launch merges the shares, in order. Sizes outside the limits take the plain kernel of paged_rows.cu.
#include <algorithm>

#include "attention_v2.cuh"
#include "common.h"
#include "paged.cuh"

namespace nfn {

constexpr uint32_t LD_PANEL = NFN_PAGE * 128;      // bytes of 64 channels of a page
constexpr int LD_MAX_STAGES = 3;

struct LatentDecodeParams {
  nfn_paged_attention_args a;
  int splits, stages;           // shares of a row's pages; pages in shared memory
  int panels, m_tiles;          // 64-channel panels of a cached row; 128-channel tiles of the latent
  uint32_t smem, tmem_cols;
  float* partial;               // [rows][heads][splits][vdim_p] values
  float2* stats;                // [rows][heads][splits] maximum and sum
  int* status;
};

// NH: heads of a CTA
template <int NH>
__global__ void __launch_bounds__(AV2_THREADS, 1)
latent_decode_kernel(const __grid_constant__ CUtensorMap tm_q, const __grid_constant__ CUtensorMap tm_c, const LatentDecodeParams p) {
  constexpr uint32_t Q_PANEL = NH * 128;
  extern __shared__ uint8_t smem_raw[];
  __shared__ float s_alpha[2][NH], s_sum[NH];
  __shared__ int s_flag[2];
  __shared__ __align__(8) uint64_t bars[4 + 2 * LD_MAX_STAGES + 2];
  __shared__ uint32_t tmem_slot;
  __shared__ int abort_s;
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~static_cast<uintptr_t>(1023));
  const nfn_paged_attention_args& a = p.a;
  const int row = a.row0 + blockIdx.z, slot = a.row_slot[row];
  if (slot < 0) return;
  const uint32_t stage_bytes = p.panels * LD_PANEL;
  uint8_t* sK = smem;                                    // [stages][panels][64][128 B]
  uint8_t* sP = sK + p.stages * stage_bytes;             // [NH][64 keys]
  uint8_t* sQ = sK + (p.stages - 1) * stage_bytes;       // the queries pass through the last stage
  uint64_t* bar_q = bars;          // TMA: queries landed
  uint64_t* bar_qt = bars + 1;     // warp 0: queries are in TMEM, their stage is free
  uint64_t* bar_s = bars + 2;      // MMA: scores complete
  uint64_t* bar_sfree = bars + 3;  // warp 0: scores are in registers
  uint64_t* bar_p = bars + 4;      // 4 arrivals: weights in shared memory (and O rescaled if needed)
  uint64_t* bar_o = bars + 5;      // MMA: O += ... retired
  uint64_t* bar_k = bars + 6;                      // [stages] TMA: page landed
  uint64_t* bar_free = bars + 6 + LD_MAX_STAGES;   // [stages] MMA: the page's last product retired
  volatile int* cta_abort = &abort_s;

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int h0 = blockIdx.y * NH, n_heads = min(NH, a.heads - h0), VP = a.vdim_p;
  const int pos = a.row_pos[row], lo = first_visible(a, pos);
  const int page0 = lo / NFN_PAGE, n_pages = pos / NFN_PAGE + 1 - page0;
  const int p_lo = page0 + (int)((long long)n_pages * blockIdx.x / p.splits), n = page0 + (int)((long long)n_pages * (blockIdx.x + 1) / p.splits) - p_lo;
  const int* table = a.table + (size_t)slot * a.table_ld;
  const size_t cell = (size_t)blockIdx.z * a.heads + h0;
  if (n <= 0) {                                          // more shares than pages
    for (int x = threadIdx.x; x < n_heads * VP; x += AV2_THREADS) p.partial[((cell + x / VP) * p.splits + blockIdx.x) * VP + x % VP] = 0.f;
    if ((int)threadIdx.x < n_heads) p.stats[(cell + threadIdx.x) * p.splits + blockIdx.x] = make_float2(-INFINITY, 0.f);
    return;
  }
  {
    uint32_t dyn;
    asm volatile("mov.u32 %0, %%dynamic_smem_size;" : "=r"(dyn));
    if (static_cast<uint32_t>(smem - smem_raw) + p.smem > dyn) {
      if (threadIdx.x == 0 && p.status) atomicCAS(p.status, 0, NFN_ERR_WAIT_MISC);
      return;
    }
  }
  if (threadIdx.x == 0) {
    abort_s = 0;
    mbar_init(smem_u32(bar_q), 1);
    mbar_init(smem_u32(bar_qt), 1);
    mbar_init(smem_u32(bar_s), 1);
    mbar_init(smem_u32(bar_sfree), 1);
    mbar_init(smem_u32(bar_p), AV2_MATH_WARPS);
    mbar_init(smem_u32(bar_o), 1);
    for (int i = 0; i < LD_MAX_STAGES; ++i) {
      mbar_init(smem_u32(&bar_k[i]), 1);
      mbar_init(smem_u32(&bar_free[i]), 1);
    }
    fence_mbar_init();
  }
  if (warp == AV2_MMA_WARP) {
    tmem_alloc(smem_u32(&tmem_slot), p.tmem_cols);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = tmem_slot, q_col = NFN_PAGE, o_col = q_col + a.dim_p / 2;      // scores, queries, outputs

  if (warp == AV2_TMA_WARP) {
    // ------------------------------------------------------------ TMA producer --
    if (lane == 0) {
      auto load = [&](int j) {
        const int st = j % p.stages;
        const uint32_t fb = smem_u32(&bar_k[st]), dst = smem_u32(sK + st * stage_bytes);
        const int r = table[p_lo + j] * NFN_PAGE;
        mbar_expect_tx(fb, stage_bytes);
        for (int d = 0; d < p.panels; ++d) tma_load_2d(dst + d * LD_PANEL, &tm_c, fb, d * 64, r);
      };
      mbar_expect_tx(smem_u32(bar_q), p.panels * Q_PANEL);
      for (int d = 0; d < p.panels; ++d) tma_load_2d(smem_u32(sQ) + d * Q_PANEL, &tm_q, smem_u32(bar_q), d * 64, row * a.heads + h0);
      const int ahead = min(n, p.stages - 1);
      for (int j = 0; j < ahead; ++j) load(j);
      for (int j = ahead; j < n; ++j) {
        const bool ok = j == p.stages - 1 ? mbar_wait_bounded(smem_u32(bar_qt), 0, cta_abort, p.status, 0x700 + 1)
                                          : mbar_wait_bounded(smem_u32(&bar_free[j % p.stages]), (j / p.stages - 1) & 1, cta_abort, p.status, 0x700 + 1);
        if (!ok) break;
        load(j);
      }
    }
  } else if (warp == AV2_MMA_WARP) {
    // -------------------------------------------------------------- MMA issuer --
    if (lane == 0) {
      const uint32_t idesc_s = make_idesc_bf16(128, NFN_PAGE, 0, 0), idesc_o = make_idesc_bf16(128, NH, 1, 0);
      const int k_steps = a.dim_p / 16;
      auto issue_s = [&](int j) {
        const uint32_t sk = smem_u32(sK + (j % p.stages) * stage_bytes);
        tc_fence_after();
#pragma unroll 4
        for (int kk = 0; kk < k_steps; ++kk)             // 16 channels of the queries are 8 TMEM columns
          umma_bf16_ts(tmem_base, tmem_base + q_col + kk * 8, make_smem_desc_sw128(sk + (kk / 4) * LD_PANEL + (kk % 4) * 32, 16, 1024), idesc_s, kk != 0);
        umma_commit(smem_u32(bar_s));
      };
      auto page_here = [&](int j) { return mbar_wait_bounded(smem_u32(&bar_k[j % p.stages]), (j / p.stages) & 1, cta_abort, p.status, 0x700 + 2); };
      bool ok = mbar_wait_bounded(smem_u32(bar_qt), 0, cta_abort, p.status, 0x700 + 3) && page_here(0);
      if (ok) issue_s(0);
      for (int j = 0; j < n && ok; ++j) {
        // the next scores first if their page is here, else this page's outputs
        bool ahead = j + 1 >= n;
        ok = mbar_wait_bounded(smem_u32(bar_sfree), j & 1, cta_abort, p.status, 0x700 + 4);
        if (!ok) break;
        if (!ahead && mbar_try_wait(smem_u32(&bar_k[(j + 1) % p.stages]), ((j + 1) / p.stages) & 1)) {
          issue_s(j + 1);
          ahead = true;
        }
        ok = mbar_wait_bounded(smem_u32(bar_p), j & 1, cta_abort, p.status, 0x700 + 5);
        if (!ok) break;
        tc_fence_after();
        const uint32_t sv = smem_u32(sK + (j % p.stages) * stage_bytes), sp = smem_u32(sP);
        for (int t = 0; t < p.m_tiles; ++t)
#pragma unroll
          for (int kk = 0; kk < NFN_PAGE / 16; ++kk)
            umma_bf16_ss(tmem_base + o_col + t * NH, make_smem_desc_sw128(sv + 2 * t * LD_PANEL + kk * (16 * 128), LD_PANEL, 1024),
                         make_smem_desc_sw128(sp + kk * 32, 16, 1024), idesc_o, (j | kk) != 0);
        umma_commit(smem_u32(bar_o));
        umma_commit(smem_u32(&bar_free[j % p.stages]));
        if (!ahead) {
          ok = page_here(j + 1);
          if (ok) issue_s(j + 1);
        }
      }
    }
  } else {
    // ------------------------------------------------------------- math threads --
    const uint32_t t_row = tmem_base + (static_cast<uint32_t>(warp * 32) << 16);
    const float mul = a.scale * 1.4426950408889634f;
    const int head = lane % NH;                          // of warp 0's threads
    float m_run = -INFINITY, l_run = 0.f;
    bool ok = true;
    if (warp == 0) {                                     // queries to TMEM: a head's row is a lane's
      ok = mbar_wait_bounded(smem_u32(bar_q), 0, cta_abort, p.status, 0x700 + 6);
      ok = __all_sync(0xffffffffu, ok);
#pragma unroll 1
      for (int c = 0; c < a.dim_p / 32; ++c) {
        uint32_t u[16];
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int ch = c * 4 + e;                      // 16-byte piece of the row
          *reinterpret_cast<uint4*>(&u[4 * e]) = *reinterpret_cast<const uint4*>(sQ + (ch / 8) * Q_PANEL + head * 128 + (((ch % 8) ^ (head & 7)) << 4));
        }
        tmem_st_32x16(t_row + q_col + c * 16, u);
      }
      if (a.dim_p % 32) {                                // the last sixteen channels; what is stored behind them is overwritten by the first output
        const int c = a.dim_p / 32;
        uint32_t u[16] = {};
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int ch = c * 4 + e;
          *reinterpret_cast<uint4*>(&u[4 * e]) = *reinterpret_cast<const uint4*>(sQ + (ch / 8) * Q_PANEL + head * 128 + (((ch % 8) ^ (head & 7)) << 4));
        }
        tmem_st_32x16(t_row + q_col + c * 16, u);
      }
      tmem_st_wait();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(smem_u32(bar_qt));
    }
    for (int j = 0; j < n; ++j) {
      uint32_t s[NFN_PAGE];
      float m_new = m_run;
      if (warp == 0) {
        ok = mbar_wait_bounded(smem_u32(bar_s), j & 1, cta_abort, p.status, 0x700 + 7);
        ok = __all_sync(0xffffffffu, ok);
        tc_fence_after();
        tmem_ld_row<NFN_PAGE>(t_row, s);
        tmem_ld_wait();
        tc_fence_before();
        __syncwarp();
        if (lane == 0) mbar_arrive(smem_u32(bar_sfree));
        const int kbase = (p_lo + j) * NFN_PAGE;
#pragma unroll
        for (int i = 0; i < NFN_PAGE; i += 2) {
          float x0, x1;
          mul2(x0, x1, __uint_as_float(s[i]), __uint_as_float(s[i + 1]), mul, mul);
          s[i] = __float_as_uint(x0);
          s[i + 1] = __float_as_uint(x1);
        }
        if (kbase < lo || kbase + NFN_PAGE - 1 > pos) {
#pragma unroll
          for (int i = 0; i < NFN_PAGE; ++i)
            if (kbase + i < lo || kbase + i > pos) s[i] = 0xff800000u;      // -inf
        }
        float mx[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
        for (int i = 0; i < NFN_PAGE; i += 8)
#pragma unroll
          for (int e = 0; e < 4; ++e) mx[e] = fmax3(mx[e], __uint_as_float(s[i + 2 * e]), __uint_as_float(s[i + 2 * e + 1]));
        m_new = fmaxf(m_run, fmaxf(fmaxf(mx[0], mx[1]), fmaxf(mx[2], mx[3])));      // every page holds a visible key: finite
        const bool grow = __any_sync(0xffffffffu, m_new - m_run > 8.f);
        if (grow) s_alpha[j & 1][head] = exp2f(m_run - m_new);
        if (lane == 0) s_flag[j & 1] = grow;
      }
      asm volatile("bar.sync 1, 128;" ::: "memory");
      if (*cta_abort) ok = false;                        // set before the barrier by whoever ran out of patience
      ok = __all_sync(0xffffffffu, ok);
      if (!ok) break;
      const bool rescale = s_flag[j & 1];
      if (warp == 0) {
        if (rescale) {
          l_run *= exp2f(m_run - m_new);
          m_run = m_new;
        }
#pragma unroll
        for (int i = 0; i < NFN_PAGE; i += 2) {
          float x0, x1;
          add2f(x0, x1, __uint_as_float(s[i]), __uint_as_float(s[i + 1]), -m_run, -m_run);
          s[i] = __float_as_uint(x0);
          s[i + 1] = __float_as_uint(x1);
        }
#pragma unroll
        for (int i = 0; i < NFN_PAGE; ++i) s[i] = __float_as_uint(fast_exp2(__uint_as_float(s[i])));
        float l0 = 0.f, l1 = 0.f, l2 = 0.f, l3 = 0.f;
#pragma unroll
        for (int i = 0; i < NFN_PAGE; i += 4) {
          add2(l0, l1, __uint_as_float(s[i]), __uint_as_float(s[i + 1]));
          add2(l2, l3, __uint_as_float(s[i + 2]), __uint_as_float(s[i + 3]));
        }
        l_run += (l0 + l1) + (l2 + l3);
      }
      if (j > 0 && (warp == 0 || rescale)) {
        // the last product must have retired before its weights are overwritten and O is rescaled
        ok = mbar_wait_bounded(smem_u32(bar_o), (j - 1) & 1, cta_abort, p.status, 0x700 + 8);
        ok = __all_sync(0xffffffffu, ok);
        if (!ok) continue;                               // all four warps leave together, at the next barrier
        tc_fence_after();
        if (rescale) {
#pragma unroll 1
          for (int c = 0; c < p.m_tiles * (NH / 16); ++c) {
            uint32_t o[16];
            tmem_ld_32x16(t_row + o_col + c * 16, o);
            tmem_ld_wait();
#pragma unroll
            for (int i = 0; i < 16; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * s_alpha[j & 1][(c * 16 + i) % NH]);
            tmem_st_32x16(t_row + o_col + c * 16, o);
          }
          tmem_st_wait();
        }
      }
      if (warp == 0) {
        if (lane < NH) {
#pragma unroll
          for (int c = 0; c < NFN_PAGE / 8; ++c) {
            const uint32_t* e = &s[c * 8];
            st_swizzled_row_chunk(sP, NH, lane, c,
                                  make_uint4(pack_bf16x2(__uint_as_float(e[0]), __uint_as_float(e[1])), pack_bf16x2(__uint_as_float(e[2]), __uint_as_float(e[3])),
                                             pack_bf16x2(__uint_as_float(e[4]), __uint_as_float(e[5])), pack_bf16x2(__uint_as_float(e[6]), __uint_as_float(e[7]))));
          }
        }
        fence_proxy_async();
      }
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(smem_u32(bar_p));
    }
    // ---- O^T: a thread holds one channel of all heads ----
    if (warp == 0) s_sum[head] = l_run + (has_sink(a) && head < n_heads ? exp2f(sink_score(a, h0 + head) * 1.4426950408889634f - m_run) : 0.f);
    asm volatile("bar.sync 1, 128;" ::: "memory");
    if (*cta_abort) ok = false;
    if (ok) ok = mbar_wait_bounded(smem_u32(bar_o), (n - 1) & 1, cta_abort, p.status, 0x700 + 9);
    ok = __all_sync(0xffffffffu, ok);
    if (ok) {
      tc_fence_after();
      if (p.splits > 1 && warp == 0 && lane < n_heads) p.stats[(cell + lane) * p.splits + blockIdx.x] = make_float2(m_run, l_run);
      __nv_bfloat16* out = static_cast<__nv_bfloat16*>(a.out) + (size_t)row * a.ld_o + (size_t)h0 * VP;
#pragma unroll 1
      for (int t = 0; t < p.m_tiles; ++t) {
        uint32_t o[NH];
#pragma unroll
        for (int c = 0; c < NH / 16; ++c) tmem_ld_32x16(t_row + o_col + t * NH + c * 16, *reinterpret_cast<uint32_t(*)[16]>(&o[c * 16]));
        tmem_ld_wait();
        const int ch = t * 128 + warp * 32 + lane;
        if (ch < VP) {
#pragma unroll
          for (int h = 0; h < NH; ++h) {
            if (h >= n_heads) break;
            if (p.splits == 1) out[(size_t)h * VP + ch] = __float2bfloat16(__uint_as_float(o[h]) / s_sum[h]);
            else p.partial[((cell + h) * p.splits + blockIdx.x) * VP + ch] = __uint_as_float(o[h]);
          }
        }
      }
    }
  }

  tc_fence_before();
  __syncthreads();
  if (*cta_abort) {
    for (int i = 0; i < 64; ++i) __nanosleep(1000);       // copies in flight land
  }
  if (warp == AV2_MMA_WARP) {
    tc_fence_after();
    tmem_dealloc(tmem_base, p.tmem_cols);
  }
}

// A CTA takes one head of a row, a thread four channels.
__global__ void __launch_bounds__(128)
latent_merge_kernel(const LatentDecodeParams p) {
  constexpr int AT_ONCE = 8;
  const nfn_paged_attention_args& a = p.a;
  const int row = a.row0 + blockIdx.y, h = blockIdx.x, c = threadIdx.x * 4;
  if (a.row_slot[row] < 0 || c >= a.vdim_p) return;
  const size_t cell = (size_t)blockIdx.y * a.heads + h;
  const float2* stats = p.stats + cell * p.splits;
  const float* part = p.partial + cell * p.splits * a.vdim_p + c;
  float m = has_sink(a) ? sink_score(a, h) * 1.4426950408889634f : -INFINITY, l = has_sink(a) ? 1.f : 0.f;
  float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
  for (int s0 = 0; s0 < p.splits; s0 += AT_ONCE) {
    float2 t[AT_ONCE];
    float4 v[AT_ONCE];
#pragma unroll
    for (int i = 0; i < AT_ONCE; ++i) {
      const int s = min(s0 + i, p.splits - 1);
      t[i] = stats[s];
      v[i] = load4(part + (size_t)s * a.vdim_p);
      if (s0 + i >= p.splits) t[i] = make_float2(-INFINITY, 0.f);
    }
    float m_new = m;
#pragma unroll
    for (int i = 0; i < AT_ONCE; ++i) m_new = fmaxf(m_new, t[i].x);
    if (m_new == -INFINITY) continue;                     // shares without pages
    const float keep = exp2f(m - m_new);
    l *= keep;
    o.x *= keep; o.y *= keep; o.z *= keep; o.w *= keep;
    m = m_new;
#pragma unroll
    for (int i = 0; i < AT_ONCE; ++i) {
      const float f = exp2f(t[i].x - m_new);
      l += f * t[i].y;
      o.x += f * v[i].x; o.y += f * v[i].y; o.z += f * v[i].z; o.w += f * v[i].w;
    }
  }
  const float inv = 1.f / l;
  store4(static_cast<__nv_bfloat16*>(a.out) + (size_t)row * a.ld_o + (size_t)h * a.vdim_p + c, make_float4(o.x * inv, o.y * inv, o.z * inv, o.w * inv));
}

template <int NH>
static int launch_latent_decode(LatentDecodeParams p, const CUtensorMap& tq, const CUtensorMap& tc, cudaStream_t st) {
  auto kern = latent_decode_kernel<NH>;
  static uint32_t raised[64] = {};
  int dev = 0;
  cudaGetDevice(&dev);
  if (raised[dev & 63] < p.smem + 1024) {
    if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)p.smem + 1024) != cudaSuccess) return launch_check("latent_decode attr", 0);
    raised[dev & 63] = p.smem + 1024;
  }
  const nfn_paged_attention_args& a = p.a;
  kern<<<dim3(p.splits, ceil_div(a.heads, NH), a.rows), AV2_THREADS, p.smem + 1024, st>>>(tq, tc, p);
  if (p.splits > 1) latent_merge_kernel<<<dim3(a.heads, a.rows), 128, 0, st>>>(p);
  return launch_check("latent_decode", p.splits > 1 ? 2 : 1);
}

// What lies behind the stages: the weights, and at least a panel where a product over whole 128-channel tiles reads past the last panel.
static uint32_t latent_tail(int panels, int m_tiles, int nh) { return std::max<uint32_t>(nh * 128, 2 * m_tiles > panels ? LD_PANEL : 0); }

// 1: sizes outside the kernel's limits
int latent_decode(const nfn_paged_attention_args& a, cudaStream_t st) {
  constexpr uint32_t LIMIT = 227 * 1024 - 2048;            // static shared memory and the alignment of the dynamic part aside
  if (a.vdim_p > 512 || ((a.dim_p | a.vdim_p) & 15) || a.ld_q != a.heads * a.dim_p || a.rows > 65535 || a.slopes || a.softcap > 0.f || a.keep_first > 0 || a.gate) return 1;
  LatentDecodeParams p{};
  p.a = a;
  p.panels = ceil_div(a.dim_p, 64);
  p.m_tiles = ceil_div(a.vdim_p, 128);
  const int nh = a.heads > 16 && NFN_PAGE + a.dim_p / 2 + p.m_tiles * 32 <= 512 ? 32 : 16;
  const int cols = NFN_PAGE + a.dim_p / 2 + std::max(p.m_tiles * nh, 8);      // the queries' last store may reach eight columns further
  const uint32_t stage = p.panels * LD_PANEL, tail = latent_tail(p.panels, p.m_tiles, nh);
  p.stages = 3 * stage + tail <= LIMIT ? 3 : 2;
  p.smem = p.stages * stage + tail;
  if (cols > 512 || p.smem > LIMIT || p.panels * nh * 128 > (int)stage) return 1;
  p.tmem_cols = cols <= 128 ? 128 : cols <= 256 ? 256 : 512;
  p.status = status_ptr();
  // one wave of what is resident at a time, at least a page each
  const long long ctas = (long long)a.rows * ceil_div(a.heads, nh), cells = (long long)a.rows * a.heads;
  const int resident = std::min<int>(228 * 1024 / (p.smem + 3072), 512 / p.tmem_cols);
  long long splits = std::min<long long>(ceil_div(a.max_keys, NFN_PAGE) + 1, std::max<long long>(1, (long long)sm_count() * std::max(resident, 1) / ctas));
  splits = std::min<long long>(std::min<long long>(splits, 64), (a.workspace_bytes - PAGED_COUNTER_BYTES) / (cells * (a.vdim_p * 4 + 8)));
  p.splits = (int)std::max<long long>(splits, 1);
  p.partial = reinterpret_cast<float*>(static_cast<char*>(a.workspace) + PAGED_COUNTER_BYTES);
  p.stats = reinterpret_cast<float2*>(p.partial + cells * p.splits * a.vdim_p);
  CUtensorMap tq, tc;
  if (!make_tmap_2d(&tq, a.q, 2, a.dim_p, (uint64_t)(a.row0 + a.rows) * a.heads, a.dim_p, 64, nh, 128)) return -3;
  if (!make_tmap_2d(&tc, a.k_pool, 2, a.dim_p, (uint64_t)a.pages * NFN_PAGE, a.dim_p, 64, NFN_PAGE, 128)) return -3;
  return nh == 32 ? launch_latent_decode<32>(p, tq, tc, st) : launch_latent_decode<16>(p, tq, tc, st);
}

}  // namespace nfn
