// Attention of single query rows (decoded tokens, very short portions) over paged caches, on the tensor cores.
//
// One CTA takes one row, one key / value head and a share of the visible keys; its four warps walk that share in steps of 32 keys.
// Nothing is staged in shared memory: a contraction does not care about the order of its index, so every fragment of
// mma.m16n8k16 comes from ONE 16-byte load per lane. For S^T = K q^T lane (g, j) reads 8 consecutive channels of a key row and
// of the query heads; for O^T = V^T P^T, with values stored channel-major, it reads 8 consecutive keys of a channel row. The key
// that sits in row g of a score tile is chosen such that the transposed probability tile (movmatrix) is the second product's
// operand as it stands. The query heads of a group are the 8-column operand, so grouped heads share every load.
//
// Scores, distance bias, softmax and the running sums are fp32. A row's shares (and warps) are merged in a fixed order: the CTA
// that finishes last adds them up, applies the output gate and stores. Sizes outside the kernel's limits and 32-bit mode take the
// plain kernel of paged_rows.cu.
#include <algorithm>

#include "common.h"
#include "paged.cuh"

namespace nfn {

int paged_attention_plain(const nfn_paged_attention_args& a, cudaStream_t st);  // paged_rows.cu
int latent_decode(const nfn_paged_attention_args& a, cudaStream_t st);           // latent_decode.cu; 1: sizes outside its limits

constexpr int PD_WARPS = 4, PD_THREADS = PD_WARPS * 32, PD_KEYS = 32;
constexpr int PD_COUNTERS = PAGED_COUNTER_BYTES / 4;
constexpr long long PD_PARTIAL_BYTES = 16LL << 20;

__device__ __forceinline__ void pd_mma(float (&d)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
               : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}
// 8 x 8 matrix of 16-bit values, two per lane: rows become columns
__device__ __forceinline__ uint32_t pd_transpose(uint32_t v) {
  uint32_t r;
  asm volatile("movmatrix.sync.aligned.m8n8.trans.b16 %0, %1;" : "=r"(r) : "r"(v));
  return r;
}
__device__ __forceinline__ uint32_t pd_word(const uint4& v, int i) { return i == 0 ? v.x : i == 1 ? v.y : i == 2 ? v.z : v.w; }

struct PagedDecodeParams {
  nfn_paged_attention_args a;
  int splits, head_blocks;     // shares of a row's keys; blocks of NT * 8 query heads per key / value head
  int* counters;               // [rows][kv_heads * head_blocks]
  float* partial;              // [rows][kv_heads * head_blocks][splits][NT * 8][vdim_p + 2]: values, maximum, sum
};

// DC: 32-channel chunks of a query / key head; VT: 16-channel tiles of a value head; NT: 8-head tiles (upper bounds, the actual
// sizes are checked inside)
template <int DC, int VT, int NT>
__global__ void __launch_bounds__(PD_THREADS, 2)
paged_decode_kernel(const PagedDecodeParams p) {
  constexpr int NH = NT * 8;
  extern __shared__ float pd_smem[];   // [PD_WARPS][NH][vdim_p] values, then [PD_WARPS][NH] maxima, [PD_WARPS][NH] sums
  __shared__ int sh_last;
  const nfn_paged_attention_args& a = p.a;
  const int row = a.row0 + blockIdx.z;
  const int slot = a.row_slot[row];
  if (slot < 0) return;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, g = lane >> 2, j = lane & 3;
  const int hk = blockIdx.y / p.head_blocks, hb = blockIdx.y % p.head_blocks;
  const int hg = a.heads / a.kv_heads, h_lo = hb * NH, n_heads = min(NH, hg - h_lo), h0 = hk * hg + h_lo;
  const int pos = a.row_pos[row];
  const int lo = first_visible(a, pos);
  // chunks in the order kept tokens, window: number i of them is chunk i of the sequence, or c_first + i - n_keep
  const int keep = min(a.keep_first, pos + 1);
  const int c_first = lo / PD_KEYS, n_keep = min(c_first, (keep + PD_KEYS - 1) / PD_KEYS), n_chunks = n_keep + pos / PD_KEYS + 1 - c_first;
  const int c_lo = (int)((long long)n_chunks * blockIdx.x / p.splits), c_hi = (int)((long long)n_chunks * (blockIdx.x + 1) / p.splits);
  auto chunk_base = [&](int i) { return (i < n_keep ? i : c_first + i - n_keep) * PD_KEYS; };
  const int DP = a.dim_p, VP = a.vdim_p;
  const int* table = a.table + (size_t)slot * a.table_ld;
  const __nv_bfloat16* kp = static_cast<const __nv_bfloat16*>(a.k_pool);
  const __nv_bfloat16* vp = static_cast<const __nv_bfloat16*>(a.v_pool);
  const uint4 zero4 = make_uint4(0u, 0u, 0u, 0u);

  uint4 qf[DC][NT];
#pragma unroll
  for (int c = 0; c < DC; ++c)
#pragma unroll
    for (int nt = 0; nt < NT; ++nt) {
      const int h = nt * 8 + g, d = c * 32 + 8 * j;
      qf[c][nt] = (h < n_heads && d < DP)
                      ? *reinterpret_cast<const uint4*>(static_cast<const __nv_bfloat16*>(a.q) + (size_t)row * a.ld_q + (size_t)(h0 + h) * DP + d) : zero4;
    }
  // this lane's two heads per tile: columns 2 j, 2 j + 1
  const float LOG2E = 1.4426950408889634f;
  const float mul = a.scale * LOG2E;
  // cap tanh(s / cap) = cap (1 - 2 / (1 + e^(2 s / cap)))
  const float cap = a.softcap * LOG2E, cap_in = a.softcap > 0.f ? 2.f * mul / a.softcap : 0.f;
  float slope[NT][2], m[NT][2], l[NT][2];
  float acc[VT][NT][4];
#pragma unroll
  for (int nt = 0; nt < NT; ++nt)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int h = nt * 8 + 2 * j + e;
      slope[nt][e] = (a.slopes && h < n_heads) ? a.slopes[h0 + h] * LOG2E : 0.f;
      m[nt][e] = -INFINITY;
      l[nt][e] = 0.f;
    }
#pragma unroll
  for (int v = 0; v < VT; ++v)
#pragma unroll
    for (int nt = 0; nt < NT; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[v][nt][e] = 0.f;

  // row g of score tile t is key 8 (g / 2) + g % 2 + 4 t of the 32, row g + 8 the key two further
  const int key0 = 8 * (g >> 1) + (g & 1);
  uint4 kf[2][2][DC];                                       // key fragments of the chunk at hand: [tile][row g, row g + 8]
  auto load_keys = [&](int c) {
    const int base = chunk_base(c), in_page = base % NFN_PAGE;
    const size_t tile = (size_t)table[base / NFN_PAGE] * a.kv_heads + hk;
    const __nv_bfloat16* krow = kp + (tile * NFN_PAGE + in_page + key0) * DP + 8 * j;
#pragma unroll
    for (int t = 0; t < 2; ++t)
#pragma unroll
      for (int half = 0; half < 2; ++half)
#pragma unroll
        for (int d = 0; d < DC; ++d)
          kf[t][half][d] = d * 32 + 8 * j < DP ? __ldg(reinterpret_cast<const uint4*>(krow + (size_t)(4 * t + 2 * half) * DP + d * 32)) : zero4;
  };
  if (c_lo + warp < c_hi) load_keys(c_lo + warp);
  for (int c = c_lo + warp; c < c_hi; c += PD_WARPS) {
    const int base = chunk_base(c), in_page = base % NFN_PAGE;
    const size_t tile = (size_t)table[base / NFN_PAGE] * a.kv_heads + hk;
    // this chunk's values are on their way while the scores are formed, the next chunk's keys while these are used
    constexpr int VF = (NT == 1 && VT <= 8) ? VT : 2;                    // value tiles held ahead
    const __nv_bfloat16* vrow = vp + (tile * VP + g) * NFN_PAGE + in_page + 8 * j;
    uint4 vf[VF][2];
#pragma unroll
    for (int v = 0; v < VF; ++v)
#pragma unroll
      for (int half = 0; half < 2; ++half)
        vf[v][half] = v * 16 < VP ? __ldg(reinterpret_cast<const uint4*>(vrow + (size_t)(v * 16 + 8 * half) * NFN_PAGE)) : zero4;
    float s[2][NT][4];
#pragma unroll
    for (int t = 0; t < 2; ++t)
#pragma unroll
      for (int nt = 0; nt < NT; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) s[t][nt][e] = 0.f;
#pragma unroll
    for (int t = 0; t < 2; ++t)
#pragma unroll
      for (int d = 0; d < DC; ++d) {
        if (d * 32 >= DP) break;
        const uint4 k0 = kf[t][0][d], k1 = kf[t][1][d];
#pragma unroll
        for (int nt = 0; nt < NT; ++nt) {
          pd_mma(s[t][nt], k0.x, k1.x, k0.y, k1.y, qf[d][nt].x, qf[d][nt].y);
          pd_mma(s[t][nt], k0.z, k1.z, k0.w, k1.w, qf[d][nt].z, qf[d][nt].w);
        }
      }
    if (c + PD_WARPS < c_hi) load_keys(c + PD_WARPS);
    // scaled and biased scores in units of log2, invisible keys out
    const int rel = pos - base - key0;      // distance of this lane's first key
#pragma unroll
    for (int t = 0; t < 2; ++t)
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int dist = rel - 4 * t - 2 * half;
        const bool seen = dist >= 0 && (pos - dist >= lo || pos - dist < keep);
#pragma unroll
        for (int nt = 0; nt < NT; ++nt)
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            float& x = s[t][nt][2 * half + e];
            const float y = cap > 0.f ? cap * (1.f - __fdividef(2.f, 1.f + exp2f(x * cap_in))) : x * mul;
            x = seen ? y - slope[nt][e] * (float)dist : -INFINITY;
          }
      }
    uint32_t b[2][NT][2];
#pragma unroll
    for (int nt = 0; nt < NT; ++nt) {
      float alpha[2];
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        float mx = fmaxf(fmaxf(s[0][nt][e], s[0][nt][2 + e]), fmaxf(s[1][nt][e], s[1][nt][2 + e]));
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 4));
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 8));
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 16));
        const float m_new = fmaxf(m[nt][e], mx);           // every chunk holds a visible key: finite
        alpha[e] = exp2f(m[nt][e] - m_new);                 // 0 on the first chunk
        m[nt][e] = m_new;
        float sum = 0.f;
#pragma unroll
        for (int t = 0; t < 2; ++t)
#pragma unroll
          for (int half = 0; half < 2; ++half) {
            float& x = s[t][nt][2 * half + e];
            x = exp2f(x - m_new);
            sum += x;
          }
        l[nt][e] = l[nt][e] * alpha[e] + sum;
      }
#pragma unroll
      for (int v = 0; v < VT; ++v) {
        acc[v][nt][0] *= alpha[0]; acc[v][nt][1] *= alpha[1]; acc[v][nt][2] *= alpha[0]; acc[v][nt][3] *= alpha[1];
      }
#pragma unroll
      for (int t = 0; t < 2; ++t)
#pragma unroll
        for (int half = 0; half < 2; ++half) b[t][nt][half] = pd_transpose(pack_bf16x2(s[t][nt][2 * half], s[t][nt][2 * half + 1]));
    }
#pragma unroll
    for (int v = 0; v < VT; ++v) {
      if (v * 16 >= VP) break;
      const uint4 v0 = v < VF ? vf[v < VF ? v : 0][0] : __ldg(reinterpret_cast<const uint4*>(vrow + (size_t)(v * 16) * NFN_PAGE));
      const uint4 v1 = v < VF ? vf[v < VF ? v : 0][1] : __ldg(reinterpret_cast<const uint4*>(vrow + (size_t)(v * 16 + 8) * NFN_PAGE));
#pragma unroll
      for (int t = 0; t < 2; ++t)
#pragma unroll
        for (int nt = 0; nt < NT; ++nt)
          pd_mma(acc[v][nt], pd_word(v0, 2 * t), pd_word(v1, 2 * t), pd_word(v0, 2 * t + 1), pd_word(v1, 2 * t + 1), b[t][nt][0], b[t][nt][1]);
    }
  }

  // merge the warps
  float* so = pd_smem;
  float* sm = so + PD_WARPS * NH * VP;
  float* sl = sm + PD_WARPS * NH;
#pragma unroll
  for (int nt = 0; nt < NT; ++nt)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      float t = l[nt][e];
      t += __shfl_xor_sync(0xffffffffu, t, 4);
      t += __shfl_xor_sync(0xffffffffu, t, 8);
      t += __shfl_xor_sync(0xffffffffu, t, 16);
      const int h = nt * 8 + 2 * j + e;
      if (g == 0) {
        sm[warp * NH + h] = m[nt][e];
        sl[warp * NH + h] = t;
      }
#pragma unroll
      for (int v = 0; v < VT; ++v) {
        if (v * 16 >= VP) break;
        float* o = so + (size_t)(warp * NH + h) * VP + v * 16 + g;
        o[0] = acc[v][nt][e];
        o[8] = acc[v][nt][2 + e];
      }
    }
  __syncthreads();
  const __nv_bfloat16* gate = static_cast<const __nv_bfloat16*>(a.gate);
  __nv_bfloat16* out = static_cast<__nv_bfloat16*>(a.out);
  auto finish = [&](int h, int ch, float o) {
    const int col = (h0 + h) * VP + ch;
    if (gate) o *= 1.f / (1.f + __expf(-__bfloat162float(gate[(size_t)row * a.ld_gate + col])));
    out[(size_t)row * a.ld_o + col] = __float2bfloat16(o);
  };
  const size_t cell = (size_t)blockIdx.z * gridDim.y + blockIdx.y;
  float* part = p.partial + (cell * p.splits + blockIdx.x) * NH * (VP + 2);
  for (int i = threadIdx.x; i < n_heads * VP; i += PD_THREADS) {
    const int h = i / VP, ch = i % VP;
    const float sink = has_sink(a) ? sink_score(a, h0 + h) * LOG2E : -INFINITY;
    float mx = p.splits == 1 ? sink : -INFINITY;
#pragma unroll
    for (int w = 0; w < PD_WARPS; ++w) mx = fmaxf(mx, sm[w * NH + h]);
    float o = 0.f, sum = 0.f;
    if (mx != -INFINITY) {
#pragma unroll
      for (int w = 0; w < PD_WARPS; ++w) {
        const float f = exp2f(sm[w * NH + h] - mx);
        o += f * so[(size_t)(w * NH + h) * VP + ch];
        sum += f * sl[w * NH + h];
      }
    }
    if (p.splits == 1) {
      if (has_sink(a)) sum += exp2f(sink - mx);
      finish(h, ch, o / sum);
    } else {
      part[(size_t)h * (VP + 2) + ch] = o;
      if (ch == 0) {
        part[(size_t)h * (VP + 2) + VP] = mx;
        part[(size_t)h * (VP + 2) + VP + 1] = sum;
      }
    }
  }
  if (p.splits == 1) return;
  // the share that finishes last adds them up, in order
  __threadfence();
  __syncthreads();
  if (threadIdx.x == 0) sh_last = atomicAdd(&p.counters[cell], 1) == p.splits - 1;
  __syncthreads();
  if (!sh_last) return;
  __threadfence();
  const float* all = p.partial + cell * p.splits * NH * (VP + 2);
  for (int i = threadIdx.x; i < n_heads * VP; i += PD_THREADS) {
    const int h = i / VP, ch = i % VP;
    const float sink = has_sink(a) ? sink_score(a, h0 + h) * LOG2E : -INFINITY;
    float mx = sink;
    for (int s2 = 0; s2 < p.splits; ++s2) mx = fmaxf(mx, __ldcg(&all[((size_t)s2 * NH + h) * (VP + 2) + VP]));
    float o = 0.f, sum = 0.f;
    for (int s2 = 0; s2 < p.splits; ++s2) {
      const float* q = &all[((size_t)s2 * NH + h) * (VP + 2)];
      const float f = exp2f(__ldcg(q + VP) - mx);
      o += f * __ldcg(q + ch);
      sum += f * __ldcg(q + VP + 1);
    }
    if (has_sink(a)) sum += exp2f(sink - mx);
    finish(h, ch, o / sum);
  }
  if (threadIdx.x == 0) p.counters[cell] = 0;
}

template <int DC, int VT, int NT>
static int launch_paged_decode(const nfn_paged_attention_args& a, cudaStream_t st) {
  PagedDecodeParams p;
  p.a = a;
  const int hg = a.heads / a.kv_heads;
  p.head_blocks = ceil_div(hg, NT * 8);
  const int cells_y = a.kv_heads * p.head_blocks;
  const long long cells = (long long)a.rows * cells_y;
  p.counters = static_cast<int*>(a.workspace);
  p.partial = reinterpret_cast<float*>(static_cast<char*>(a.workspace) + PAGED_COUNTER_BYTES);
  // about two CTAs per SM (what is resident at a time), at least one chunk of keys per warp
  long long splits = std::min<long long>(ceil_div(a.max_keys, PD_KEYS * PD_WARPS), std::max<long long>(1, 2LL * sm_count() / cells));
  const long long per_split = cells * NT * 8 * (a.vdim_p + 2) * 4;
  splits = std::min<long long>(splits, (a.workspace_bytes - PAGED_COUNTER_BYTES) / per_split);
  if (cells > PD_COUNTERS || splits < 1) splits = 1;
  p.splits = (int)std::min<long long>(splits, 64);
  const size_t smem = (size_t)PD_WARPS * NT * 8 * (a.vdim_p + 2) * sizeof(float);
  auto kern = paged_decode_kernel<DC, VT, NT>;
  static bool raised[64] = {};
  int dev = 0;
  cudaGetDevice(&dev);
  if (smem > 48 * 1024 && !raised[dev & 63]) {
    if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 100 * 1024) != cudaSuccess) return launch_check("paged_decode attr", 0);
    raised[dev & 63] = true;
  }
  for (int r = 0; r < a.rows; r += 65535) {          // grid.z limit
    PagedDecodeParams part = p;
    part.a.row0 = a.row0 + r;
    const dim3 grid(p.splits, cells_y, std::min(a.rows - r, 65535));
    kern<<<grid, PD_THREADS, smem, st>>>(part);
  }
  return launch_check("paged_decode");
}

}  // namespace nfn

using namespace nfn;

extern "C" long long nfn_paged_attention_workspace_bytes(int rows, int heads, int vdim_p) {
  (void)rows; (void)heads; (void)vdim_p;
  return PAGED_COUNTER_BYTES + PD_PARTIAL_BYTES;
}

extern "C" int nfn_paged_attention_rows(const nfn_paged_attention_args* args, nfn_stream_t stream) {
  if (!args) return fail(-1, "paged attention: null args");
  const nfn_paged_attention_args& a = *args;
  if (a.rows <= 0) return 0;
  if (a.kv_heads <= 0 || a.heads % a.kv_heads) return fail(-1, "paged attention: query heads must divide into key / value heads");
  if ((a.dim_p | a.vdim_p | a.ld_q) & 15) return fail(-1, "paged attention: head sizes and the query pitch must be multiples of 16");
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (!a.v_pool) {
    if (a.kv_heads != 1 || a.vdim_p > a.dim_p) return fail(-1, "paged attention: values out of the keys need one key head at least as wide");
    const int rc = a.f32 || !a.workspace ? 1 : latent_decode(a, st);
    return rc == 1 ? paged_attention_plain(a, st) : rc;
  }
  if (a.f32 || a.dim_p > 256 || a.vdim_p > 256 || !a.workspace) return paged_attention_plain(a, st);
  if (a.dim_p > 128 || a.vdim_p > 128) return launch_paged_decode<8, 16, 1>(a, st);
  return a.heads / a.kv_heads > 8 ? launch_paged_decode<4, 8, 2>(a, st) : launch_paged_decode<4, 8, 1>(a, st);
}
