// Attention of prompt portions over paged caches (tcgen05): tiles of consecutive rows of one sequence, any length of history.
//
// A tile's 128 accumulator rows are (query row, query head of the group) pairs - 128 / group rows of all heads that share a key /
// value head - so the group reads every page once and a sliding window costs window + 128 / group keys per tile instead of
// window + 128. A block of keys is a page: keys arrive as 64-channel panels [64 tokens][64 channels], values, which the cache
// stores channel-major, as [channels][64 tokens]; both are K-major operands, and the page table only enters the TMA coordinates.
// Roles as in attention_fwd2.cu: four softmax warps (one thread per accumulator row), one MMA warp, one TMA warp, two stages of
// keys and values; S of the next page is issued as soon as this one is in registers, the output is rescaled in TMEM only when a
// row maximum grew by more than 2^8. Pages are visited from the newest to the oldest: under a distance bias the maximum then
// settles in the first page instead of growing with every one.
//
// Latent attention (EXPANDED): every head's unrotated keys and its values were formed from the cached latents as rows of one matrix, 64 rows per
// page; the rotated key part, shared by the heads, still comes from the pages as further panels of the same score product. Values then
// are [64 tokens][64 channels] panels, an MN-major operand. Queries and keys take a panel more, so P stays in TMEM (a TMEM-sourced product) and
// values have one stage where two would cost the second CTA of an SM its place.
//
// Head sizes are run-time values (multiples of 16 up to 256; channels past a head's end are zero-filled by TMA). The distance
// bias and the window are applied to the fp32 scores in registers; the output gate is applied on the way out.
#include "attention_v2.cuh"
#include "paged.cuh"

namespace nfn {

constexpr int PP_BM = 128, PP_BN = NFN_PAGE;
constexpr uint32_t PP_P_COL = PP_BN;          // EXPANDED: P behind the scores, PP_BN / 2 columns

struct PagedPrefillParams {
  nfn_paged_attention_args a;
  int hg, nq;                 // query heads per key / value head, query rows per tile
  int panels;                 // 64-channel panels of a query / key head (EXPANDED: of its unrotated part)
  nfn_latent_expanded x;      // EXPANDED
  int panels_r, panels_v;     // panels of the rotated part, of a value head
  uint32_t q_bytes, k_bytes, v_bytes, q_tx;
  int v_stages;
  uint32_t o_col, tmem_cols;
  uint32_t smem;
  int* status;
};

// GATED: with an output gate. tm_k, tm_v: the pages (EXPANDED: the pages for the rotated key part, the matrix of unrotated keys and values)
template <bool EXPANDED, bool GATED>
__global__ void __launch_bounds__(AV2_THREADS, 2)
paged_prefill_kernel(const __grid_constant__ CUtensorMap tm_q, const __grid_constant__ CUtensorMap tm_k,
                     const __grid_constant__ CUtensorMap tm_v, const PagedPrefillParams p) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~static_cast<uintptr_t>(1023));
  {
    uint32_t dyn;
    asm volatile("mov.u32 %0, %%dynamic_smem_size;" : "=r"(dyn));
    if (static_cast<uint32_t>(smem - smem_raw) + p.smem > dyn) {
      if (threadIdx.x == 0 && p.status) atomicCAS(p.status, 0, NFN_ERR_WAIT_MISC);
      return;
    }
  }
  const nfn_paged_attention_args& a = p.a;
  const int vs = p.v_stages;
  uint8_t* sQ = smem;
  uint8_t* sK = sQ + p.q_bytes;
  uint8_t* sV = sK + 2 * p.k_bytes;
  uint8_t* sP = sV + vs * p.v_bytes;
  uint64_t* bars = reinterpret_cast<uint64_t*>(sP + (EXPANDED ? 0 : PP_BM * PP_BN * 2));
  uint64_t* bar_q = bars;          // TMA: Q landed
  uint64_t* bar_k = bars + 1;      // [2] TMA: key stage landed
  uint64_t* bar_v = bars + 3;      // [2] TMA: value stage landed
  uint64_t* bar_s = bars + 5;      // MMA: S_j complete
  uint64_t* bar_sfree = bars + 6;  // 4 arrivals: S_j is in registers
  uint64_t* bar_p = bars + 7;      // 4 arrivals: P_j in shared memory (and O rescaled if needed)
  uint64_t* bar_o = bars + 8;      // MMA: O += P_j V_j retired
  uint64_t* bar_kfree = bars + 9;  // [2] MMA: the product that read key stage s retired
  uint64_t* bar_vfree = bars + 11; // [2]
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 13);
  volatile int* cta_abort = reinterpret_cast<volatile int*>(tmem_slot + 1);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int4 tile = reinterpret_cast<const int4*>(a.tiles)[gridDim.x - 1 - blockIdx.x];   // later tiles see more keys: first
  const int row0 = tile.x, n_rows = tile.y, slot = tile.z, pos0 = tile.w;
  const int hk = blockIdx.y;
  const int* table = a.table + (size_t)slot * a.table_ld;
  const int k_lo = first_visible(a, pos0);
  // visited from the newest page back to the window's edge, then the pages of the kept first tokens that lie before it
  const int jb_hi = (pos0 + n_rows - 1) / PP_BN, n_win = jb_hi + 1 - k_lo / PP_BN;
  const int n_keep = min(k_lo / PP_BN, (a.keep_first + PP_BN - 1) / PP_BN), nblk = n_win + n_keep;
  auto page_at = [&](int j) { return j < n_win ? jb_hi - j : n_keep - 1 - (j - n_win); };

  if (threadIdx.x == 0) {
    *cta_abort = 0;
    mbar_init(smem_u32(bar_q), 1);
    for (int s2 = 0; s2 < 2; ++s2) {
      mbar_init(smem_u32(&bar_k[s2]), 1);
      mbar_init(smem_u32(&bar_v[s2]), 1);
      mbar_init(smem_u32(&bar_kfree[s2]), 1);
      mbar_init(smem_u32(&bar_vfree[s2]), 1);
    }
    mbar_init(smem_u32(bar_s), 1);
    mbar_init(smem_u32(bar_sfree), AV2_MATH_WARPS);
    mbar_init(smem_u32(bar_p), AV2_MATH_WARPS);
    mbar_init(smem_u32(bar_o), 1);
    fence_mbar_init();
  }
  if (warp == AV2_MMA_WARP) {
    tmem_alloc(smem_u32(tmem_slot), p.tmem_cols);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;

  if (warp == AV2_TMA_WARP) {
    // ------------------------------------------------------------ TMA producer --
    if (lane == 0) {
      const int x_base = EXPANDED ? p.x.x_base[slot] : 0;
      auto load_k = [&](int j, int stage) {
        const uint32_t fb = smem_u32(&bar_k[stage]);
        const uint32_t sk = smem_u32(sK + stage * p.k_bytes);
        mbar_expect_tx(fb, p.k_bytes);
        if (EXPANDED) {
          const int r = x_base + page_at(j) * PP_BN;
          for (int d = 0; d < p.panels; ++d) tma_load_2d(sk + d * (PP_BN * 128), &tm_v, fb, hk * p.x.dim_u + d * 64, r);
          for (int d = 0; d < p.panels_r; ++d)
            tma_load_2d(sk + (p.panels + d) * (PP_BN * 128), &tm_k, fb, p.x.rank_p + d * 64, table[page_at(j)] * PP_BN);
        } else {
          const int r = (table[page_at(j)] * a.kv_heads + hk) * PP_BN;
          for (int d = 0; d < p.panels; ++d) tma_load_2d(sk + d * (PP_BN * 128), &tm_k, fb, d * 64, r);
        }
      };
      auto load_v = [&](int j, int stage) {
        const uint32_t fb = smem_u32(&bar_v[stage]);
        const uint32_t sv = smem_u32(sV + stage * p.v_bytes);
        mbar_expect_tx(fb, p.v_bytes);
        if (EXPANDED) {
          for (int d = 0; d < p.panels_v; ++d)
            tma_load_2d(sv + d * (PP_BN * 128), &tm_v, fb, a.heads * p.x.dim_u + hk * a.vdim_p + d * 64, x_base + page_at(j) * PP_BN);
        } else {
          tma_load_2d(sv, &tm_v, fb, 0, (table[page_at(j)] * a.kv_heads + hk) * a.vdim_p);
        }
      };
      mbar_expect_tx(smem_u32(bar_q), p.q_tx);
      for (int d = 0; d < p.panels; ++d) tma_load_3d(smem_u32(sQ) + d * (PP_BM * 128), &tm_q, smem_u32(bar_q), d * 64, hk * p.hg, row0);
      if (EXPANDED)
        for (int d = 0; d < p.panels_r; ++d)
          tma_load_3d(smem_u32(sQ) + (p.panels + d) * (PP_BM * 128), &tm_q, smem_u32(bar_q), p.x.dim_u + d * 64, hk, row0);
      load_k(0, 0);
      load_v(0, 0);
      if (nblk > 1) load_k(1, 1);
      if (nblk > 1 && vs > 1) load_v(1, 1);
      for (int j = 0; j + vs < nblk; ++j) {
        if (j + 2 < nblk) {
          if (!mbar_wait_bounded(smem_u32(&bar_kfree[j & 1]), (j >> 1) & 1, cta_abort, p.status, 0x600 + 1)) break;
          load_k(j + 2, j & 1);
        }
        const int st = vs > 1 ? j & 1 : 0;
        if (!mbar_wait_bounded(smem_u32(&bar_vfree[st]), (vs > 1 ? j >> 1 : j) & 1, cta_abort, p.status, 0x600 + 2)) break;
        load_v(j + vs, st);
      }
    }
  } else if (warp == AV2_MMA_WARP) {
    // -------------------------------------------------------------- MMA issuer --
    if (lane == 0) {
      const uint32_t idesc_s = make_idesc_bf16(PP_BM, PP_BN, 0, 0);
      const uint32_t idesc_o = EXPANDED ? make_idesc_bf16(PP_BM, p.panels_v * 64, 0, 1) : make_idesc_bf16(PP_BM, a.vdim_p, 0, 0);   // whole panels
      const int k_steps = (EXPANDED ? p.x.dim_u : a.dim_p) / 16;
      auto issue_s = [&](int stage) {
        const uint32_t sq = smem_u32(sQ);
        const uint32_t sk = smem_u32(sK + stage * p.k_bytes);
#pragma unroll 4
        for (int kk = 0; kk < k_steps; ++kk) {
          const uint32_t a_off = (kk / 4) * (PP_BM * 128) + (kk % 4) * 32;
          const uint32_t b_off = (kk / 4) * (PP_BN * 128) + (kk % 4) * 32;
          umma_bf16_ss(tmem_base, make_smem_desc_sw128(sq + a_off, 16, 1024), make_smem_desc_sw128(sk + b_off, 16, 1024), idesc_s, kk != 0);
        }
        if (EXPANDED) {
          const uint32_t sqr = sq + p.panels * (PP_BM * 128), skr = sk + p.panels * (PP_BN * 128);
          for (int kk = 0; kk < p.x.rot_p / 16; ++kk) {
            const uint32_t a_off = (kk / 4) * (PP_BM * 128) + (kk % 4) * 32;
            const uint32_t b_off = (kk / 4) * (PP_BN * 128) + (kk % 4) * 32;
            umma_bf16_ss(tmem_base, make_smem_desc_sw128(sqr + a_off, 16, 1024), make_smem_desc_sw128(skr + b_off, 16, 1024), idesc_s, 1);
          }
        }
        umma_commit(smem_u32(bar_s));
        umma_commit(smem_u32(&bar_kfree[stage]));
      };
      bool ok = mbar_wait_bounded(smem_u32(bar_q), 0, cta_abort, p.status, 0x600 + 3);
      ok = ok && mbar_wait_bounded(smem_u32(&bar_k[0]), 0, cta_abort, p.status, 0x600 + 4);
      if (ok) { tc_fence_after(); issue_s(0); }
      for (int j = 0; j < nblk && ok; ++j) {
        if (j + 1 < nblk) {
          const int ns = (j + 1) & 1;
          ok = mbar_wait_bounded(smem_u32(bar_sfree), j & 1, cta_abort, p.status, 0x600 + 5);
          ok = ok && mbar_wait_bounded(smem_u32(&bar_k[ns]), ((j + 1) >> 1) & 1, cta_abort, p.status, 0x600 + 6);
          if (!ok) break;
          tc_fence_after();
          issue_s(ns);
        }
        ok = mbar_wait_bounded(smem_u32(bar_p), j & 1, cta_abort, p.status, 0x600 + 7);
        const int st = vs > 1 ? j & 1 : 0;
        ok = ok && mbar_wait_bounded(smem_u32(&bar_v[st]), (vs > 1 ? j >> 1 : j) & 1, cta_abort, p.status, 0x600 + 8);
        if (!ok) break;
        tc_fence_after();
        const uint32_t sp = smem_u32(sP);
        const uint32_t sv = smem_u32(sV + st * p.v_bytes);
#pragma unroll
        for (int kk = 0; kk < PP_BN / 16; ++kk) {
          if (EXPANDED)  // 16 keys of P = 8 TMEM columns of bf16 pairs
            umma_bf16_ts(tmem_base + p.o_col, tmem_base + PP_P_COL + kk * 8, make_smem_desc_sw128(sv + kk * (16 * 128), PP_BN * 128, 1024), idesc_o, (j | kk) != 0);
          else
            umma_bf16_ss(tmem_base + p.o_col, make_smem_desc_sw128(sp + kk * 32, 16, 1024), make_smem_desc_sw128(sv + kk * 32, 16, 1024), idesc_o, (j | kk) != 0);
        }
        umma_commit(smem_u32(bar_o));
        umma_commit(smem_u32(&bar_vfree[st]));
      }
    }
  } else {
    // --------------------------------------------------------- softmax threads --
    const int r = warp * 32 + lane;  // accumulator row == TMEM lane: (query row r / hg, head r % hg)
    const int qi = r / p.hg, h = hk * p.hg + r % p.hg;
    const bool row_ok = qi < n_rows && r < p.nq * p.hg;
    const int pos = pos0 + qi;
    const uint32_t t_row = tmem_base + (static_cast<uint32_t>(warp * 32) << 16);
    const float LOG2E = 1.4426950408889634f;
    const float c_mul = a.scale * LOG2E;
    const float cap = a.softcap * LOG2E, cap_in = a.softcap > 0.f ? 2.f * c_mul / a.softcap : 0.f;
    // tanh(x) / x in powers of the raw score's square, x = score * to_x
    const float to_x = a.softcap > 0.f ? a.scale / a.softcap : 0.f, x2 = to_x * to_x, small = to_x != 0.f ? 0.6f / fabsf(to_x) : 0.f;
    const float th1 = -0.33332309f * x2, th2 = 0.13310173f * x2 * x2, th3 = -0.05210146f * x2 * x2 * x2, th4 = 0.015475395f * x2 * x2 * x2 * x2;
    const float slope = (a.slopes && row_ok) ? a.slopes[h] * LOG2E : 0.f;
    // visible keys of this row: [v_lo, v_hi)
    const int v_hi = row_ok ? pos + 1 : 0;
    const int v_lo = row_ok ? first_visible(a, pos) : 0;
    const int lo_last = first_visible(a, pos0 + n_rows - 1);
    const int v_keep = min(a.keep_first, v_hi);
    float m_run = has_sink(a) ? sink_score(a, h) * LOG2E : -INFINITY, l_run = has_sink(a) ? 1.f : 0.f;  // units of log2; the sink counts as seen before all keys
    bool ok = true;
    for (int j = 0; j < nblk; ++j) {
      ok = mbar_wait_bounded(smem_u32(bar_s), j & 1, cta_abort, p.status, 0x600 + 9);
      ok = __all_sync(0xffffffffu, ok);
      if (!ok) break;
      tc_fence_after();
      uint32_t s[PP_BN];
      tmem_ld_row<PP_BN>(t_row, s);
      tmem_ld_wait();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(smem_u32(bar_sfree));

      const int kbase = page_at(j) * PP_BN;
      float mul = c_mul;
      if (a.softcap > 0.f) {
        float big = 0.f;
#pragma unroll
        for (int i = 0; i < PP_BN; i += 2) big = fmax3(big, fabsf(__uint_as_float(s[i])), fabsf(__uint_as_float(s[i + 1])));
        if (!__any_sync(0xffffffffu, big > small)) {
          // every score of the warp's tile is small against the cap: tanh(x) = x P(x^2), a fit of relative error below 1e-7 for |x| <= 0.6
#pragma unroll
          for (int i = 0; i < PP_BN; i += 2) {
            const float s0 = __uint_as_float(s[i]), s1 = __uint_as_float(s[i + 1]);
            float u0, u1, t0, t1;
            mul2(u0, u1, s0, s1, s0, s1);
            fma2_bcast(t0, t1, u0, u1, th4, th3);
            fma2(t0, t1, u0, u1, t0, t1, th2, th2);
            fma2(t0, t1, u0, u1, t0, t1, th1, th1);
            fma2(t0, t1, u0, u1, t0, t1, 0.99999994f, 0.99999994f);
            mul2(t0, t1, t0, t1, s0, s1);
            s[i] = __float_as_uint(t0);
            s[i + 1] = __float_as_uint(t1);
          }
        } else {
          // cap tanh(x) = cap (1 - 2 / (1 + e^(2x))), two scores per reciprocal
#pragma unroll
          for (int i = 0; i < PP_BN; i += 2) {
            const float e0 = 1.f + fast_exp2(fminf(__uint_as_float(s[i]) * cap_in, 60.f)), e1 = 1.f + fast_exp2(fminf(__uint_as_float(s[i + 1]) * cap_in, 60.f));
            const float r2 = cap * -2.f * fast_rcp(e0 * e1);
            s[i] = __float_as_uint(fmaf(r2, e1, cap));
            s[i + 1] = __float_as_uint(fmaf(r2, e0, cap));
          }
          mul = 1.f;
        }
      }
      const float b0 = slope * (float)(kbase - pos);
#pragma unroll
      for (int i = 0; i < PP_BN; i += 2) {
        float t0, t1, y0, y1;
        fma2_bcast(t0, t1, (float)i, (float)(i + 1), slope, b0);
        fma2(y0, y1, __uint_as_float(s[i]), __uint_as_float(s[i + 1]), mul, mul, t0, t1);
        s[i] = __float_as_uint(y0);
        s[i + 1] = __float_as_uint(y1);
      }
      if (kbase + PP_BN - 1 > pos0 || kbase < lo_last) {
        const int lo_rel = v_lo - kbase, keep_rel = v_keep - kbase;
        const unsigned span = (unsigned)max(0, v_hi - v_lo);
#pragma unroll
        for (int i = 0; i < PP_BN; ++i)
          if ((unsigned)(i - lo_rel) >= span && i >= keep_rel) s[i] = 0xff800000u;  // -inf
      }
      float mx0 = -INFINITY, mx1 = -INFINITY, mx2 = -INFINITY, mx3 = -INFINITY;
#pragma unroll
      for (int i = 0; i < PP_BN; i += 8) {
        mx0 = fmax3(mx0, __uint_as_float(s[i]), __uint_as_float(s[i + 1]));
        mx1 = fmax3(mx1, __uint_as_float(s[i + 2]), __uint_as_float(s[i + 3]));
        mx2 = fmax3(mx2, __uint_as_float(s[i + 4]), __uint_as_float(s[i + 5]));
        mx3 = fmax3(mx3, __uint_as_float(s[i + 6]), __uint_as_float(s[i + 7]));
      }
      const float m_new = fmaxf(fmaxf(fmaxf(mx0, mx1), fmaxf(mx2, mx3)), m_run);
      const bool grow = m_new - m_run > 8.f;  // also true for -inf -> finite, false for -inf -> -inf
      const bool rescale = __any_sync(0xffffffffu, grow);
      float alpha = 1.f;
      if (rescale) {
        alpha = (m_run == -INFINITY) ? 0.f : fast_exp2(m_run - m_new);
        l_run *= alpha;
        m_run = m_new;
      }
      const float moff = (m_run == -INFINITY) ? 0.f : m_run;
#pragma unroll
      for (int i = 0; i < PP_BN; i += 2) {
        float x0, x1;
        add2f(x0, x1, __uint_as_float(s[i]), __uint_as_float(s[i + 1]), -moff, -moff);
        s[i] = __float_as_uint(x0);
        s[i + 1] = __float_as_uint(x1);
      }
#pragma unroll
      for (int i = 0; i < PP_BN; ++i) s[i] = __float_as_uint(fast_exp2(__uint_as_float(s[i])));
      float l0 = 0.f, l1 = 0.f, l2 = 0.f, l3 = 0.f;
#pragma unroll
      for (int i = 0; i < PP_BN; i += 4) {
        add2(l0, l1, __uint_as_float(s[i]), __uint_as_float(s[i + 1]));
        add2(l2, l3, __uint_as_float(s[i + 2]), __uint_as_float(s[i + 3]));
      }
      l_run += (l0 + l1) + (l2 + l3);
      if (j > 0) {
        // O += P_{j-1} V_{j-1} must have retired before P is overwritten and O rescaled
        ok = mbar_wait_bounded(smem_u32(bar_o), (j - 1) & 1, cta_abort, p.status, 0x600 + 10);
        ok = __all_sync(0xffffffffu, ok);
        if (!ok) break;
        tc_fence_after();
        if (rescale) {
#pragma unroll 1
          for (int c = 0; c < a.vdim_p / 16; ++c) {
            uint32_t o[16];
            tmem_ld_32x16(t_row + p.o_col + c * 16, o);
            tmem_ld_wait();
#pragma unroll
            for (int i = 0; i < 16; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * alpha);
            tmem_st_32x16(t_row + p.o_col + c * 16, o);
          }
          tmem_st_wait();
        }
      }
      if (EXPANDED) {
        // packed in place, then straight into TMEM
#pragma unroll
        for (int i = 0; i < PP_BN / 2; ++i) s[i] = pack_bf16x2(__uint_as_float(s[2 * i]), __uint_as_float(s[2 * i + 1]));
        tmem_st_32x32(t_row + PP_P_COL, *reinterpret_cast<uint32_t(*)[32]>(&s[0]));
        tmem_st_wait();
      } else {
#pragma unroll
        for (int c = 0; c < PP_BN / 8; ++c) {
          const uint32_t* e = &s[c * 8];
          st_swizzled_row_chunk(sP, PP_BM, r, c,
                                make_uint4(pack_bf16x2(__uint_as_float(e[0]), __uint_as_float(e[1])), pack_bf16x2(__uint_as_float(e[2]), __uint_as_float(e[3])),
                                           pack_bf16x2(__uint_as_float(e[4]), __uint_as_float(e[5])), pack_bf16x2(__uint_as_float(e[6]), __uint_as_float(e[7]))));
        }
        fence_proxy_async();
      }
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(smem_u32(bar_p));
    }
    // ---- O / l, output gate -> global: 64 channels at a time, their gates on the way before O is waited for ----
    __nv_bfloat16* orow = static_cast<__nv_bfloat16*>(a.out) + (size_t)(row0 + qi) * a.ld_o + (size_t)h * a.vdim_p;
    const __nv_bfloat16* grow_ = (GATED && row_ok) ? static_cast<const __nv_bfloat16*>(a.gate) + (size_t)(row0 + qi) * a.ld_gate + (size_t)h * a.vdim_p : nullptr;
    uint4 gv[8];
    auto fetch_gate = [&](int c0) {
#pragma unroll
      for (int g = 0; g < 8; ++g)
        if (GATED && grow_ && c0 + g * 8 < a.vdim_p) gv[g] = __ldg(reinterpret_cast<const uint4*>(grow_ + c0 + g * 8));
    };
    fetch_gate(0);
    if (ok) {
      ok = mbar_wait_bounded(smem_u32(bar_o), (nblk - 1) & 1, cta_abort, p.status, 0x600 + 11);
      ok = __all_sync(0xffffffffu, ok);
    }
    if (ok) {
      tc_fence_after();
      const float inv = l_run > 0.f ? 1.f / l_run : 0.f;
#pragma unroll 1
      for (int c0 = 0; c0 < a.vdim_p; c0 += 64) {
        if (c0 > 0) fetch_gate(c0);
        uint32_t o[64];
#pragma unroll
        for (int c = 0; c < 4; ++c)                                     // warp-collective: every lane issues them
          if (c0 + c * 16 < a.vdim_p) tmem_ld_32x16(t_row + p.o_col + c0 + c * 16, *reinterpret_cast<uint32_t(*)[16]>(&o[c * 16]));
        tmem_ld_wait();
        if (row_ok) {
#pragma unroll
          for (int g = 0; g < 8; ++g) {
            if (c0 + g * 8 >= a.vdim_p) break;
            float v[8];
#pragma unroll
            for (int i = 0; i < 8; ++i) v[i] = __uint_as_float(o[g * 8 + i]) * inv;
            if (GATED) {
              const float2 g0 = unpack_bf16x2(gv[g].x), g1 = unpack_bf16x2(gv[g].y), g2 = unpack_bf16x2(gv[g].z), g3 = unpack_bf16x2(gv[g].w);
              const float gf[8] = {g0.x, g0.y, g1.x, g1.y, g2.x, g2.y, g3.x, g3.y};
#pragma unroll
              for (int i = 0; i < 8; ++i) v[i] *= sigmoid_for<__nv_bfloat16>(gf[i]);
            }
            store8(orow + c0 + g * 8, v);
          }
        }
      }
    }
  }

  tc_fence_before();
  __syncthreads();
  if (*cta_abort) {
    for (int i = 0; i < 64; ++i) __nanosleep(1000);
  }
  if (warp == AV2_MMA_WARP) {
    tc_fence_after();
    tmem_dealloc(tmem_base, p.tmem_cols);
  }
}

}  // namespace nfn

using namespace nfn;

// shared memory of a tile with this many panels and bytes of values per page; the limit is what one CTA may have
static uint32_t paged_tile_smem(uint32_t panels, uint32_t v_bytes) {
  return panels * PP_BM * 128 + 2 * (panels * PP_BN * 128 + v_bytes) + PP_BM * PP_BN * 2 + 128;
}
static uint32_t latent_tile_smem(int panels, int panels_v, int v_stages) {
  return panels * PP_BM * 128 + 2 * panels * PP_BN * 128 + v_stages * panels_v * PP_BN * 128 + 128;
}
constexpr uint32_t PP_SMEM_MAX = 226 * 1024, PP_SMEM_HALF = 113 * 1024;     // of one CTA; so that two share an SM

extern "C" int nfn_paged_tile_rows(int f32, int heads, int kv_heads, int dim_p, int vdim_p) {
  const int hg = heads / kv_heads;
  if (f32 || dim_p > 256 || vdim_p > 256 || hg > PP_BM || paged_tile_smem((dim_p + 63) / 64, vdim_p * 128) > PP_SMEM_MAX) return 0;
  return PP_BM / hg;
}

template <bool EXPANDED, bool GATED>
static int launch_paged_prefill(PagedPrefillParams& p, const CUtensorMap& tq, const CUtensorMap& tk, const CUtensorMap& tv, cudaStream_t st) {
  const nfn_paged_attention_args& a = p.a;
  p.o_col = EXPANDED ? PP_BN + PP_BN / 2 : PP_BN;
  const int cols = (int)p.o_col + (EXPANDED ? p.panels_v * 64 : a.vdim_p);
  p.tmem_cols = cols <= 128 ? 128 : cols <= 256 ? 256 : 512;
  p.status = status_ptr();
  auto kern = paged_prefill_kernel<EXPANDED, GATED>;
  static uint32_t raised[64] = {};
  int dev = 0;
  cudaGetDevice(&dev);
  if (raised[dev & 63] < p.smem) {
    if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)p.smem) != cudaSuccess) return launch_check("paged_prefill attr", 0);
    raised[dev & 63] = p.smem;
  }
  kern<<<dim3(a.n_tiles, a.kv_heads), AV2_THREADS, p.smem, st>>>(tq, tk, tv, p);
  return launch_check("paged_prefill");
}

extern "C" int nfn_paged_attention_tiles(const nfn_paged_attention_args* args, nfn_stream_t stream) {
  if (!args) return fail(-1, "paged attention: null args");
  const nfn_paged_attention_args& a = *args;
  if (a.n_tiles <= 0) return 0;
  PagedPrefillParams p{};
  p.a = a;
  p.nq = nfn_paged_tile_rows(a.f32, a.heads, a.kv_heads, a.dim_p, a.vdim_p);
  if (p.nq <= 0) return fail(-1, "paged attention: these head sizes run one row at a time");
  if ((a.dim_p | a.vdim_p | a.ld_q | a.ld_o) & 15 || (a.gate && (a.ld_gate & 7))) return fail(-1, "paged attention: head sizes and row pitches must be multiples of 16");
  p.hg = a.heads / a.kv_heads;
  p.panels = (a.dim_p + 63) / 64;
  p.q_bytes = p.panels * PP_BM * 128;
  p.k_bytes = p.panels * PP_BN * 128;
  // the value stage keeps the next key stage on a 1024-byte boundary
  p.v_bytes = a.vdim_p * 128;
  p.q_tx = p.panels * p.nq * p.hg * 128;
  p.v_stages = 2;
  p.smem = paged_tile_smem(p.panels, p.v_bytes);
  CUtensorMap tq, tk, tv;
  if (!make_tmap_3d(&tq, a.q, 2, a.dim_p, a.heads, a.total_rows, a.dim_p, a.ld_q, 64, p.hg, p.nq, 128)) return -3;
  const uint64_t cells = (uint64_t)a.pages * a.kv_heads;
  if (!make_tmap_2d(&tk, a.k_pool, 2, a.dim_p, cells * NFN_PAGE, a.dim_p, 64, PP_BN, 128)) return -3;
  if (!make_tmap_2d(&tv, a.v_pool, 2, NFN_PAGE, cells * a.vdim_p, NFN_PAGE, NFN_PAGE, a.vdim_p, 128)) return -3;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  return a.gate ? launch_paged_prefill<false, true>(p, tq, tk, tv, st) : launch_paged_prefill<false, false>(p, tq, tk, tv, st);
}

// stages of values for these panels: two, or one where that lets a second CTA in or is all there is room for; 0: no room
static int latent_v_stages(int panels, int panels_v) {
  if (latent_tile_smem(panels, panels_v, 2) <= PP_SMEM_HALF) return 2;
  if (latent_tile_smem(panels, panels_v, 1) <= PP_SMEM_HALF) return 1;
  return latent_tile_smem(panels, panels_v, 2) <= PP_SMEM_MAX ? 2 : latent_tile_smem(panels, panels_v, 1) <= PP_SMEM_MAX ? 1 : 0;
}

extern "C" int nfn_latent_tile_rows(int f32, int dim_u, int rot_p, int vdim_p) {
  return f32 || vdim_p > 256 || latent_v_stages((dim_u + 63) / 64 + (rot_p + 63) / 64, (vdim_p + 63) / 64) == 0 ? 0 : PP_BM;
}

extern "C" int nfn_latent_attention_tiles(const nfn_paged_attention_args* args, const nfn_latent_expanded* x, nfn_stream_t stream) {
  if (!args || !x) return fail(-1, "latent attention: null args");
  const nfn_paged_attention_args& a = *args;
  if (a.n_tiles <= 0) return 0;
  if (nfn_latent_tile_rows(a.f32, x->dim_u, x->rot_p, a.vdim_p) <= 0) return fail(-1, "latent attention: these head sizes run one row at a time");
  if (a.kv_heads != a.heads || a.dim_p != x->dim_u + x->rot_p || a.keep_first > 0) return fail(-1, "latent attention: every head has expanded keys and values of its own");
  if ((x->dim_u | x->rot_p | x->rank_p | a.vdim_p | a.ld_q | a.ld_o) & 15 || (a.gate && (a.ld_gate & 7))) return fail(-1, "latent attention: head sizes and row pitches must be multiples of 16");
  PagedPrefillParams p{};
  p.a = a;
  p.x = *x;
  p.nq = PP_BM;
  p.hg = 1;
  p.panels = (x->dim_u + 63) / 64;
  p.panels_r = (x->rot_p + 63) / 64;
  p.panels_v = (a.vdim_p + 63) / 64;
  const int panels = p.panels + p.panels_r;
  p.q_bytes = p.q_tx = panels * PP_BM * 128;
  p.k_bytes = panels * PP_BN * 128;
  p.v_bytes = p.panels_v * PP_BN * 128;
  p.v_stages = latent_v_stages(panels, p.panels_v);
  p.smem = latent_tile_smem(panels, p.panels_v, p.v_stages);
  const int lp = x->rank_p + x->rot_p, cols = a.heads * (x->dim_u + a.vdim_p);
  CUtensorMap tq, tk, tx;
  if (!make_tmap_3d(&tq, a.q, 2, a.dim_p, a.heads, a.total_rows, a.dim_p, a.ld_q, 64, 1, PP_BM, 128)) return -3;
  if (!make_tmap_2d(&tk, a.k_pool, 2, lp, (uint64_t)a.pages * NFN_PAGE, lp, 64, PP_BN, 128)) return -3;
  if (!make_tmap_2d(&tx, x->x, 2, cols, x->x_rows, cols, 64, PP_BN, 128)) return -3;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  return a.gate ? launch_paged_prefill<true, true>(p, tq, tk, tx, st) : launch_paged_prefill<true, false>(p, tq, tk, tx, st);
}
