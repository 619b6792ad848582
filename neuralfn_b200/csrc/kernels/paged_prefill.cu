// Attention of prompt portions over cache pages.
#include "common.h"
#include "paged.cuh"
extern "C" int nfn_paged_tile_rows(int f32, int heads, int kv_heads, int dim_p, int vdim_p) { return 0; }
extern "C" int nfn_paged_attention_tiles(const nfn_paged_attention_args* args, nfn_stream_t stream) { return nfn::fail(-1, "tiles"); }
