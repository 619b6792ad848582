// Shared by the kernels of the bonus recurrence (wkv_rows.cu, wkv_chunk.cu).
#pragma once
#include "paged.cuh"

namespace nfn {

// a channel's decay from its projected value: exp(-exp(z))
__device__ __forceinline__ float wkv_decay(float z) { return expf(-expf(z)); }

const char* wkv_args_problem(const nfn_wkv_args& a);   // wkv_rows.cu; null: fine

}  // namespace nfn
