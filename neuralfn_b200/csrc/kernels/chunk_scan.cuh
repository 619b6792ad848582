// Recurrences with a decay per key channel over prompt portions, sixteen tokens at a time: what the kernels that form a chunk's operands (delta_chunk.cu,
// wkv_chunk.cu) share with the scan that runs from state to state (delta_chunk.cu).
#pragma once
#include "attention_v2.cuh"
#include "delta.cuh"

namespace nfn {

constexpr int DC_T = 16;                               // tokens of a chunk
constexpr long long DC_WORKSPACE = 96LL << 20;

// A (chunk, head) block of the scan's operands: [W, Q: dk / 16 steps x 4 tiles of 8 rows][K: dk / 8 tiles] x 32 lanes x 16 bytes, then e^G_last of every
// channel. Without corrections there is no W: two tiles per step.
__host__ __device__ constexpr int dc_gamma_at(int dk, bool corrections) { return (corrections ? 192 : 128) * dk; }
__host__ __device__ constexpr int dc_block_bytes(int dk, bool corrections) { return dc_gamma_at(dk, corrections) + dk * 4; }
__host__ __device__ constexpr int dc_uo_floats(int vdim_p) { return vdim_p * 32; }      // T V and P T V: [column tile][2][2 row tiles][32 lanes][4]

struct DeltaChunkParams {
  nfn_delta_args a;
  int dk;                     // padded key channels: 64, 128 or 256
  int chunk0, n_chunks;       // chunks [chunk0, chunk0 + n_chunks) of every sequence in this round
  unsigned char* blocks;      // [seq][chunk][head][dc_block_bytes]
  float* uo;                  // [seq][chunk][head][dc_uo_floats]
  int* status;
  // segs > 1 (without corrections only): a round's chunks in segments of seg_chunks that run side by side
  int segs, seg_chunks;
  float* seg_init;            // [seq][head][dim_p][vdim_p]: the state before the round
  float* seg_state;           // [seq][seg][head][dim_p][vdim_p]: what a segment adds (the first one: with seg_init decayed)
  float* seg_gamma;           // [seq][seg][head][dk]: what it leaves of the state before it
};

// two fp32 values as bf16 pairs: the rounded values and what they leave out
__device__ __forceinline__ void split_bf16(float a, float b, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16x2(a, b);
  const float2 f = unpack_bf16x2(hi);
  lo = pack_bf16x2(a - f.x, b - f.y);
}

__device__ __forceinline__ void dc_bulk_store(void* dst, uint32_t src, uint32_t bytes) {
  asm volatile("cp.async.bulk.global.shared::cta.bulk_group [%0], [%1], %2;" ::"l"(dst), "r"(src), "r"(bytes) : "memory");
}

// Where the 16-byte piece of lane `lane` lies inside operand tile `tile` of a block: the order keeps the writers of both kinds of tile, and
// the scan's reads, on different banks.
template <bool CORRECTIONS = true>
__device__ __forceinline__ uint32_t dc_piece(int tile, int lane, bool of_k) {
  const int turn = of_k ? ((lane >> 3) & 3) | ((tile & 1) << 2) : ((tile >> (CORRECTIONS ? 2 : 1)) & 1) << 2;
  return (uint32_t)(tile * 32 + (lane ^ turn)) * 16;
}

// The scan over the chunks of a round (delta_chunk.cu); corrections: with W, else U = V.
int chunk_scan(const DeltaChunkParams& p, bool corrections, cudaStream_t st);

}  // namespace nfn
