// Attention of single query rows over cache pages.
#include "common.h"
#include "paged.cuh"

namespace nfn {
int paged_attention_plain(const nfn_paged_attention_args& a, cudaStream_t st);  // paged_rows.cu
}

extern "C" long long nfn_paged_attention_workspace_bytes(int rows, int heads, int vdim_p) { return nfn::PAGED_COUNTER_BYTES; }
extern "C" int nfn_paged_attention_rows(const nfn_paged_attention_args* args, nfn_stream_t stream) {
  return nfn::paged_attention_plain(*args, static_cast<cudaStream_t>(stream));
}
