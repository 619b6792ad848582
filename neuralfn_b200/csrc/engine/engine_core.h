// What every resident engine shares: the device, the stream, the weights by name, slot lengths, launch counts and the virtual
// interface behind the C ABI of nfn_engine.h. Two engines implement it: the fixed block families (resident_engine.cpp: GPT-2,
// Llama, Glimmer; one ring or plain cache per slot) and the layer-list engine (layered_engine.cpp: layers described one by one,
// paged caches, steps that mix prompt portions with single tokens). Operations an engine does not have report an error.
#pragma once
#include <cuda_runtime.h>

#include <algorithm>
#include <map>
#include <string>
#include <utility>
#include <vector>

#include "../kernels/nfn_kernels.h"
#include "nfn_engine.h"

extern "C" long long nfn_launch_count(void);

namespace nfn_eng {

int efail(const std::string& m);   // records the message for nfn_engine_last_error, returns -1

struct DevTensor {
  void* ptr = nullptr;
  long long numel = 0;
  int qtype = 0;  // 0: bf16 values; NFN_QTYPE_Q4_K / Q5_K / Q6_K: packed super-blocks of 256 values, rows back to back
};

}  // namespace nfn_eng

#define CU(call)                                                                                                \
  do {                                                                                                          \
    cudaError_t e__ = (call);                                                                                   \
    if (e__ != cudaSuccess) return nfn_eng::efail(std::string(#call) + ": " + cudaGetErrorString(e__));         \
  } while (0)
#define K(call)                                                                                 \
  do {                                                                                          \
    int rc__ = (call);                                                                          \
    if (rc__ != 0) return nfn_eng::efail(std::string(#call) + " failed: " + nfn_last_error()); \
  } while (0)

struct nfn_engine {
  int device = 0;
  cudaStream_t stream = nullptr;
  std::map<std::string, nfn_eng::DevTensor> w;
  std::vector<std::pair<std::string, long long>> expected;   // tensor name, element count
  bool finalized = false;
  long long bytes = 0;
  std::vector<int> len;                                      // tokens held per slot
  unsigned long long steps = 0;
  long long launches = 0;

  virtual ~nfn_engine();
  int alloc(void** p, long long nbytes) {
    CU(cudaMalloc(p, (size_t)nbytes));
    bytes += nbytes;
    return 0;
  }
  const void* W(const std::string& n) const { return w.at(n).ptr; }
  bool has(const std::string& n) const { return w.count(n) != 0; }
  int slots() const { return (int)len.size(); }
  int missing_tensor() const;   // 0, or -1 with the name of the first expected tensor that was not set

  int set_tensor(const char* name, const void* host_bf16, long long numel);
  virtual int set_tensor_kquant(const char*, int, const void*, long long, long long) { return unavailable("set_tensor_kquant"); }
  virtual int load_dense_v5(const char*) { return unavailable("load_dense_v5"); }
  virtual int set_turboquant(const void*) { return unavailable("set_turboquant"); }
  virtual int finalize() = 0;
  virtual int release(int slot) = 0;
  virtual int prefill(int slot, const int32_t* tokens, int n, const nfn_sampling* s, int32_t* next_token) = 0;
  virtual int prefill_rows(int, const void*, int, int, const nfn_sampling*, int32_t*) { return unavailable("prefill_rows"); }
  virtual int decode(const int32_t* tokens_in, const uint8_t* active, const nfn_sampling* s, const nfn_sampling* per_slot,
                     int32_t* next_tokens) = 0;
  virtual int step(const nfn_step_entry*, int, const int32_t*, const int32_t*, int, const nfn_sampling*, int32_t*, float*) {
    return unavailable("step");
  }
  virtual int last_logits(int slot, float* out_vocab) = 0;
  virtual int enable_verify(int) { return unavailable("enable_verify"); }
  virtual int verify(const int32_t*, const int32_t*, int, int32_t*) { return unavailable("verify"); }
  virtual int verify_logits(int, int, float*) { return unavailable("verify_logits"); }
  virtual int commit(const int32_t*) { return unavailable("commit"); }
  virtual int truncate(int slot, int n) = 0;
  virtual int fork(int src_slot, int dst_slot, int n) = 0;
  virtual int enable_taps(const int32_t*, int) { return unavailable("enable_taps"); }
  virtual int read_taps(int, int, int, void*, int) { return unavailable("read_taps"); }
  virtual long long free_tokens() const { return -1; }   // cache room in tokens (paged engines)
  int unavailable(const char* what) const { return nfn_eng::efail(std::string("engine: ") + what + " is not available for this kind of model"); }
};
