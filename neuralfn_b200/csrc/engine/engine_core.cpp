// C ABI of the resident engines: argument checks that do not depend on the kind of model, then the virtual call.
#include "engine_core.h"

#include <cstring>

namespace nfn_eng {

static thread_local std::string t_err;
int efail(const std::string& m) {
  t_err = m;
  return -1;
}

}  // namespace nfn_eng

using nfn_eng::efail;

nfn_engine::~nfn_engine() {
  for (auto& kv : w) cudaFree(kv.second.ptr);
  if (stream) cudaStreamDestroy(stream);
}

int nfn_engine::missing_tensor() const {
  for (const auto& kv : expected)
    if (!has(kv.first)) return efail("engine_finalize: missing tensor " + kv.first);
  return 0;
}

int nfn_engine::set_tensor(const char* name, const void* host_bf16, long long numel) {
  CU(cudaSetDevice(device));
  long long want = -1;
  for (const auto& kv : expected)
    if (kv.first == name) want = kv.second;
  if (want < 0) return efail(std::string("engine_set_tensor: this configuration has no tensor named ") + name);
  if (want != numel) return efail(std::string("engine_set_tensor: ") + name + " has " + std::to_string(numel) + " elements, expected " + std::to_string(want));
  nfn_eng::DevTensor& t = w[name];
  if (t.qtype) return efail(std::string("engine_set_tensor: ") + name + " holds K-quant blocks");
  if (!t.ptr) {
    if (alloc(&t.ptr, numel * 2)) return -1;
    t.numel = numel;
  }
  CU(cudaMemcpyAsync(t.ptr, host_bf16, (size_t)numel * 2, cudaMemcpyHostToDevice, stream));
  CU(cudaStreamSynchronize(stream));
  return 0;
}

extern "C" {

int nfn_engine_abi_version(void) { return 1; }
const char* nfn_engine_last_error(void) { return nfn_eng::t_err.c_str(); }

void nfn_engine_destroy(nfn_engine* e) {
  if (!e) return;
  cudaSetDevice(e->device);
  if (e->stream) cudaStreamSynchronize(e->stream);
  delete e;
}

int nfn_engine_set_tensor(nfn_engine* e, const char* name, const void* host_bf16, long long numel) {
  if (!e || !name || !host_bf16 || numel <= 0) return efail("engine_set_tensor: bad arguments");
  return e->set_tensor(name, host_bf16, numel);
}

int nfn_engine_set_tensor_kquant(nfn_engine* e, const char* name, int qtype, const void* host_blocks, long long nbytes, long long numel) {
  if (!e || !name || !host_blocks || numel <= 0) return efail("engine_set_tensor_kquant: bad arguments");
  return e->set_tensor_kquant(name, qtype, host_blocks, nbytes, numel);
}

int nfn_engine_expected_tensors(const nfn_engine* e, char* buf, int cap) {
  if (!e) return efail("engine_expected_tensors: null engine");
  std::string s;
  for (const auto& kv : e->expected) s += kv.first + " " + std::to_string(kv.second) + "\n";
  if (buf && cap > 0) {
    const size_t n = std::min<size_t>(s.size(), (size_t)cap - 1);
    std::memcpy(buf, s.data(), n);
    buf[n] = 0;
  }
  return (int)s.size();
}

int nfn_engine_load_dense_v5(nfn_engine* e, const char* path) {
  if (!e || !path) return efail("engine_load_dense_v5: bad arguments");
  return e->load_dense_v5(path);
}

int nfn_engine_set_turboquant(nfn_engine* e, const void* tq_tables) {
  if (!e || !tq_tables) return efail("engine_set_turboquant: null argument");
  return e->set_turboquant(tq_tables);
}

int nfn_engine_finalize(nfn_engine* e) {
  if (!e) return efail("engine_finalize: null engine");
  return e->finalized ? 0 : e->finalize();
}

long long nfn_engine_device_bytes(const nfn_engine* e) { return e ? e->bytes : -1; }
int nfn_engine_slot_length(const nfn_engine* e, int slot) { return (e && slot >= 0 && slot < e->slots()) ? e->len[slot] : -1; }
long long nfn_engine_launches(const nfn_engine* e) { return e ? e->launches : -1; }
void* nfn_engine_stream(const nfn_engine* e) { return e ? e->stream : nullptr; }
long long nfn_engine_free_tokens(const nfn_engine* e) { return e ? e->free_tokens() : -1; }

int nfn_engine_release(nfn_engine* e, int slot) {
  if (!e || slot < 0 || slot >= e->slots()) return efail("engine_release: bad slot");
  return e->release(slot);
}

int nfn_engine_prefill(nfn_engine* e, int slot, const int32_t* tokens, int n, const nfn_sampling* s, int32_t* next_token) {
  if (!e || !tokens || !s || !next_token) return efail("engine_prefill: null argument");
  if (!e->finalized) return efail("engine_prefill: call nfn_engine_finalize first");
  if (slot < 0 || slot >= e->slots()) return efail("engine_prefill: bad slot");
  return e->prefill(slot, tokens, n, s, next_token);
}

int nfn_engine_prefill_rows(nfn_engine* e, int slot, const void* rows_bf16, int n, int rows_on_device, const nfn_sampling* s, int32_t* next_token) {
  if (!e || !rows_bf16 || !s || !next_token) return efail("engine_prefill_rows: null argument");
  if (!e->finalized) return efail("engine_prefill_rows: call nfn_engine_finalize first");
  if (slot < 0 || slot >= e->slots()) return efail("engine_prefill_rows: bad slot");
  return e->prefill_rows(slot, rows_bf16, n, rows_on_device, s, next_token);
}

int nfn_engine_decode(nfn_engine* e, const int32_t* tokens_in, const uint8_t* active, const nfn_sampling* s, const nfn_sampling* per_slot,
                      int32_t* next_tokens) {
  if (!e || !tokens_in || !active || !s || !next_tokens) return efail("engine_decode: null argument");
  if (!e->finalized) return efail("engine_decode: call nfn_engine_finalize first");
  return e->decode(tokens_in, active, s, per_slot, next_tokens);
}

int nfn_engine_step(nfn_engine* e, const nfn_step_entry* entries, int n_entries, const int32_t* tokens, const int32_t* want_rows, int n_want,
                    const nfn_sampling* want_sampling, int32_t* want_tokens, float* want_logits) {
  if (!e || (n_entries > 0 && (!entries || !tokens)) || n_entries < 0 || n_want < 0 || (n_want > 0 && !want_rows))
    return efail("engine_step: bad arguments");
  if (!e->finalized) return efail("engine_step: call nfn_engine_finalize first");
  return e->step(entries, n_entries, tokens, want_rows, n_want, want_sampling, want_tokens, want_logits);
}

int nfn_engine_last_logits(nfn_engine* e, int slot, float* out_vocab) {
  if (!e || !out_vocab || slot < 0 || slot >= e->slots() || !e->finalized) return efail("engine_last_logits: bad arguments");
  return e->last_logits(slot, out_vocab);
}

int nfn_engine_enable_verify(nfn_engine* e, int max_rows) {
  if (!e || !e->finalized) return efail("engine_enable_verify: finalize the engine first");
  return e->enable_verify(max_rows);
}

int nfn_engine_verify(nfn_engine* e, const int32_t* tokens, const int32_t* n_rows, int rows, int32_t* argmax_out) {
  if (!e || !tokens || !n_rows || !argmax_out) return efail("engine_verify: null argument");
  return e->verify(tokens, n_rows, rows, argmax_out);
}

int nfn_engine_verify_logits(nfn_engine* e, int slot, int row, float* out_vocab) {
  if (!e || !out_vocab || slot < 0 || slot >= e->slots()) return efail("engine_verify_logits: no such verification row");
  return e->verify_logits(slot, row, out_vocab);
}

int nfn_engine_commit(nfn_engine* e, const int32_t* accepted) {
  if (!e || !accepted) return efail("engine_commit: null argument");
  return e->commit(accepted);
}

int nfn_engine_truncate(nfn_engine* e, int slot, int n) {
  if (!e || slot < 0 || slot >= e->slots()) return efail("engine_truncate: bad slot");
  if (n < 0 || n > e->len[slot]) return efail("engine_truncate: length outside [0, current length]");
  return e->truncate(slot, n);
}

int nfn_engine_fork(nfn_engine* e, int src_slot, int dst_slot, int n) {
  if (!e || !e->finalized) return efail("engine_fork: engine not ready");
  if (src_slot < 0 || src_slot >= e->slots() || dst_slot < 0 || dst_slot >= e->slots() || src_slot == dst_slot) return efail("engine_fork: bad slots");
  if (n < 0 || n > e->len[src_slot]) return efail("engine_fork: prefix longer than the source");
  return e->fork(src_slot, dst_slot, n);
}

int nfn_engine_enable_taps(nfn_engine* e, const int32_t* layers, int n) {
  if (!e || !e->finalized || !layers) return efail("engine_enable_taps: finalize the engine first");
  return e->enable_taps(layers, n);
}

int nfn_engine_read_taps(nfn_engine* e, int slot, int pos0, int n, void* dst, int dst_on_device) {
  if (!e || !dst) return efail("engine_read_taps: null argument");
  if (slot < 0 || slot >= e->slots() || pos0 < 0 || n < 0 || pos0 + n > e->len[slot]) return efail("engine_read_taps: positions outside the slot's cached tokens");
  return n == 0 ? 0 : e->read_taps(slot, pos0, n, dst, dst_on_device);
}

}  // extern "C"
