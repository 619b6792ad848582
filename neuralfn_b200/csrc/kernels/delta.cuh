// Shared by the kernels of the gated delta rule (delta_rows.cu, delta_chunk.cu).
#pragma once
#include "paged.cuh"

namespace nfn {

__device__ __forceinline__ float softplus_exact(float z) { return z > 20.f ? z : log1pf(expf(z)); }
// logarithm of a channel's decay: rate = -exp(A_log)
__device__ __forceinline__ float delta_log_decay(float z, float rate) { return rate * softplus_exact(z); }
__device__ __forceinline__ float delta_decay(float z, float rate) { return expf(delta_log_decay(z, rate)); }

const char* delta_args_problem(const nfn_delta_args& a);   // delta_rows.cu; null: fine

}  // namespace nfn
