// C ABI of the resident inference engine: weights, KV caches and activation buffers stay on
// the device for the life of the engine; the host sends token ids and receives token ids.
//
// One engine serves up to max_batch concurrent sequences ("slots"). `prefill` runs a whole
// prompt of one slot through the tcgen05 GEMM / flash-attention path and fills that slot's
// KV cache; `decode` advances every active slot by one token in a single batched step
// (split-KV decode attention with fused QK-norm + RoPE + cache append, on-device sampling)
// which is captured into a CUDA graph on first use and replayed afterwards.
//
// `step` (layer-list engines) is the general form: any mix of prompt portions and single tokens of
// different slots in one batch.
//
// Families: 0 = GPT-2 style (LayerNorm, learned positions, GELU MLP, biases, MHA, tied head),
//           1 = Llama style (RMSNorm, RoPE, grouped-query attention, SwiGLU, optional per-head
//               QK norm with weights, optional sliding-window layers with ring caches).
// Behavioural counterpart in the reference: csrc/native_gpt2/resident_dense.{h,cpp},
// resident_llama.{h,cpp} and the `_native_inference` module (resident_binding.cpp).
#pragma once
#include <stdint.h>

#ifdef __cplusplus
extern "C" {
#endif

typedef struct nfn_engine nfn_engine;

typedef struct {
  int family;
  int n_layer, d_model, n_head, n_kv_head, head_dim, d_ff;
  int vocab, padded_vocab, max_seq, max_batch;
  int qk_norm;          // 0 none, 1 weightless, 2 with bf16 weights [head_dim]
  int rope_hf;          // rotary convention: 1 = hf, 0 = legacy (family 1)
  float rope_theta;
  float norm_eps, qk_norm_eps;
  float logit_softcap;  // 0 = off
  int tie_embeddings;
  int window;           // sliding window of local layers (0 = every layer global)
  int global_every;     // with window > 0: layers l with (l + 1) % global_every == 0 are global
  float embed_scale;    // multiplies the token embedding (1 = off)
  int use_cuda_graph;
  // Glimmer-style blocks (family 1 only); all zero = plain Llama
  int gated_attention;  // wqkv carries n_head * head_dim extra gate rows; attention output *= sigmoid(gate)
  int sandwich_norms;   // h += RMS(branch; post_*_norm) instead of h += branch (needs post_attn_norm / post_ffn_norm tensors)
  int centered_norms;   // block norms apply (1 + w); the final norm never does
  int embed_norm;       // weightless RMS norm of the token embedding
  int rope_local_only;  // rotary embedding on sliding-window layers only (global layers have no position signal)
  float q_scale;        // multiplies the normalised, rotated query (0 = 1)
  float output_multiplier;  // multiplies the logits before the soft cap (0 = 1)
  float post_norm_eps;  // epsilon of the sandwich norms (0 = norm_eps)
  int mlp_activation;   // family 0: NFN_ACT_* id of the MLP activation (0 = GELU, tanh form); mixture-of-activations checkpoints name theirs
  int kv_cache_mode;    // 0: bf16 K / V rows; 1: TurboQuant records (nfn_engine_set_turboquant before finalize; decode only, no verification blocks)
} nfn_engine_config;

typedef struct {
  float temperature;    // <= 0: greedy
  int top_k;            // 0: off
  float top_p;          // 0 or 1: off
  uint64_t seed;
} nfn_sampling;

// ---- layer-list engine ------------------------------------------------------------------------------
// A decoder given as a list of layers, each with its own sizes and constants. Layer: h = RMS(x) * norm1; x += mixer(h) + ff(h)
// (both branches read h; one product adds both to the 32-bit residual stream); then, with side_dim > 0, a per-layer token
// input: x += RMS(proj(gelu_tanh(gate x) * side_embed[token, layer])) * side_norm. The output norm and the head follow.
// With `chained` set in the configuration mixer and feed-forward are two sublayers, each with a norm of its own, and the residual may be
// several streams: u = sum_s in[s] x_s, y = sublayer(RMS(u) * norm), x_t <- sum_s mix[s][t] x_s + out[t] y.
// With `post_norm` the sublayers of such a layer read the residual itself and their outputs are normed: x <- x + residual_mult * RMS(sublayer(x)) * norm.
// With `sandwich` they have a norm before and one after them: x <- x + residual_mult * RMS(sublayer(RMS(x) * norm)) * norm_b; `input_taps` then adds to what a
// sublayer reads a short causal convolution of it over the sequence, h + conv(h).
enum { NFN_MIXER_ATTENTION = 0, NFN_MIXER_DELTA = 1, NFN_MIXER_LATENT = 2, NFN_MIXER_WKV = 3, NFN_MIXER_LINEAR = 4, NFN_MIXER_GRU = 5 };
typedef struct {
  int heads, kv_heads;   // query head h reads key / value head h / (heads / kv_heads)
  int dim, vdim;         // per-head query / key size and value size
  int conv_taps;         // causal depthwise convolution on the projected q, k, v (0: none; 1: a factor per channel)
  int window;            // key j is visible to query i when 0 <= i - j < window (0: every earlier key)
  int kv_from;           // >= 0: keys and values are those of that earlier layer (this one has none); -1: its own
  float scale;           // score = q . k * scale - slope_h * (i - j)
  float alibi;           // slope_h = 2^(-alibi (h + 1) / heads); 0: no distance bias
  float q_temp_coef;     // q *= 1 + coef * ln(floor((pos + 1) / every) + 1); every = 0: off
  int q_temp_every;
  int out_gate;          // heads *= sigmoid(W_g h)
  int ff;                // width of the gated feed-forward down(act(gate h) * (up h)); 0: none
  int ff_act;            // NFN_ACT_RELU, NFN_ACT_SILU, NFN_ACT_GELU_TANH, NFN_ACT_RELU2, NFN_ACT_CLAMPED (gated ones, with ff_limit and ff_slope)
  int mixer;             // NFN_MIXER_*. Delta: gated delta rule with a decay per key channel (nfn_delta_rows); conv_taps >= 1 with SiLU after it
  int qkv_bias;          // biases on the projected q, k, v (gru: on the share and the candidate)
  int keep_first;        // with a window: the sequence's first keys stay visible
  float softcap;         // score <- softcap * tanh(score / softcap); 0: off
  int sink;              // 1: one more score of 0, without a value, in the softmax; 2: one of a learned size per head
  int rank_decay, rank_gate;   // delta: inner sizes of the decay and output-gate projections
  int experts, top, expert_ff; // chained: routed experts instead of a dense feed-forward (sigmoid scores, weight on the expert's input)
  int weights_of;        // >= 0: this layer runs with the tensors of that earlier one (a loop over layers); -1: its own
  int chunk;             // > 0: keys of the query's own chunk of that many positions only (counted from the sequence's start), instead of a window
  int qk_norm;           // per-head RMS norm on queries and keys before the rotation, a weight shared by the heads
  int rot_dims;          // rotary positions on the first rot_dims dimensions of queries and keys, pairs (2i, 2i + 1); latent: on the rot_dim part
  double rot_base;       // frequency of pair i: rot_base^(-2i / rot_dims)
  int key_values;        // the values are the keys as projected, before norm and rotation; no value projection
  int kv_rank, rot_dim;  // latent: size of the cached latent and of the rotated key part all heads share; dim: the unrotated part. With kv_from the earlier
                         // layer's latents are read through this layer's own key and value projections
  int expert_plain;      // experts down(act(up h)), weighted at their output, instead of gated ones weighted at their input
  int shared_ff;         // width of an expert of the same (plain) form that every token has; 0: none
  int route_correction;  // choice scores s + correction
  int route_groups, route_keep;   // consecutive experts form groups, the choice is limited to the best of them (nfn_route_rule; 0: no groups)
  int route_normalise;   // weights divided by their sum
  float route_scale;     // times this; 0 counts as 1
  int route_softmax;     // weights are the softmax over the chosen experts' logits
  int expert_weigh_out;  // gated experts weighted at their output instead of their input
  float ff_limit, ff_slope;   // NFN_ACT_CLAMPED: g = min(gate, limit), u = clamp(up, +-limit), g * sigmoid(slope * g) * (u + 1); feed-forward and experts
  int ff_bias;           // biases on the dense feed-forward's three products
  const double* decay;   // linear: factor of each head's state per token [heads], copied
} nfn_layer_desc;
// Latent (NFN_MIXER_LATENT): q per head [dim | rot_dim], c = RMS(W_dkv h) cached with the rotated key part; score = (q . W_uk c + q_rot . k_rot) * scale, value W_uv c.
// Latent layers may have an output gate and a sink. Linear (NFN_MIXER_LINEAR): SiLU on q, k, v, the rule of nfn_linear_rows, RMS norm over all heads together,
// sigmoid gate. Gru (NFN_MIXER_GRU): the rule of nfn_gru_rows over vdim channels (heads = kv_heads = dim = 1).
// Wkv (NFN_MIXER_WKV): heads x dim, vdim = dim; token shift, bonus recurrence (nfn_wkv_rows), rank_decay the inner size of the decay projection.

typedef struct {
  int n_layer, width, vocab;
  int side_dim;          // per-layer token input size (0: none)
  float embed_scale, norm_eps;
  int dtype;             // 0: bf16 products and activations (norms, softmax, residual in 32-bit); 1: everything in 32-bit
  int max_seq;           // most tokens of one sequence
  int max_batch;         // slots
  int kv_tokens;         // cache pool: tokens all live sequences hold together, each rounded up to a page (0: max_batch * max_seq)
  int max_step_rows;     // most rows one internal pass runs; longer steps are cut
  int use_cuda_graph;
  int chained;           // two sublayers per layer
  int streams;           // residual streams (chained only); 0: one plain residual
  int untied_head;       // head of its own instead of the embedding table
  float norm_offset;     // norms multiply by weight + norm_offset
  float logit_scale;     // logits *= logit_scale
  float logit_softcap;   // logits <- cap * tanh(logits / cap); 0: off
  int post_norm;         // chained, one residual: norms on the sublayers' outputs
  float residual_mult;   // post_norm, sandwich: factor of the normed output
  int sandwich;          // chained, one residual: norms before and after every sublayer
  int scalar_norms;      // sandwich: every norm of the residual has one factor for all channels
  int input_taps;        // sandwich: taps of the convolution on the sublayers' inputs; 0: none
} nfn_layered_config;

enum { NFN_KV_PAGE = 64 };   // tokens per cache page

typedef struct {
  int32_t slot;          // sequence
  int32_t count;         // its next tokens in this step
} nfn_step_entry;

int nfn_engine_abi_version(void);
const char* nfn_engine_last_error(void);
nfn_engine* nfn_engine_create(const nfn_engine_config* cfg, int device);
void nfn_engine_destroy(nfn_engine* e);
// Copies one bf16 tensor to the device under `name` (replacing any earlier one).
int nfn_engine_set_tensor(nfn_engine* e, const char* name, const void* host_bf16, long long numel);
// Names the engine expects for its configuration, '\n'-separated "name numel" lines.
// A projection weight kept resident in its K-quant blocks (qtype 12 / 13 / 14 = Q4_K / Q5_K / Q6_K, the GGUF row layout).
// Products with up to eight rows read the blocks directly (quantised GEMV); larger ones decode the tensor into one shared
// bf16 scratch buffer first. Before nfn_engine_finalize; embeddings, norms and biases stay bf16.
int nfn_engine_set_tensor_kquant(nfn_engine* e, const char* name, int qtype, const void* host_blocks, long long nbytes, long long numel);
int nfn_engine_expected_tensors(const nfn_engine* e, char* buf, int cap);
// Loads a dense GPT checkpoint (model_%08d.bin, version 5) into a family-0 engine.
int nfn_engine_load_dense_v5(nfn_engine* e, const char* path);
// kv_cache_mode 1: the codec tables (device pointers that stay valid for the engine's life, see nfn_tq_tables in
// nfn_kernels.h; D must equal head_dim). K and V of every layer are then kept as compressed records - keys after QK norm
// and rotary embedding - and decode attention runs on the records. Call before nfn_engine_finalize.
int nfn_engine_set_turboquant(nfn_engine* e, const void* tq_tables);
// Verifies that every expected tensor is present with the right size.
int nfn_engine_finalize(nfn_engine* e);
long long nfn_engine_device_bytes(const nfn_engine* e);

// Runs the prompt of `slot` (resets the slot first). Writes the sampled next token.
int nfn_engine_prefill(nfn_engine* e, int slot, const int32_t* tokens, int n, const nfn_sampling* s, int32_t* next_token);
// The same for a prompt given as its layer-0 input rows (bf16 [n][d_model], host or device memory): token embeddings after
// the embedding norm, with rows replaced by projected media features where the prompt holds media placeholders.
// Llama-family layouts only (the GPT-2 layout adds learned position embeddings inside the engine).
int nfn_engine_prefill_rows(nfn_engine* e, int slot, const void* rows_bf16, int n, int rows_on_device, const nfn_sampling* s,
                            int32_t* next_token);
// One step for all slots: tokens_in[slot] is consumed for every slot with active[slot] != 0,
// next_tokens[slot] receives its successor. per_slot (optional, max_batch entries) overrides `s`.
int nfn_engine_decode(nfn_engine* e, const int32_t* tokens_in, const uint8_t* active, const nfn_sampling* s,
                      const nfn_sampling* per_slot, int32_t* next_tokens);
// Layer-list engines: `layers` has cfg->n_layer entries.
nfn_engine* nfn_engine_create_layered(const nfn_layered_config* cfg, const nfn_layer_desc* layers, int device);
// Runs the next tokens of any number of slots as one batch: `tokens` holds the entries' tokens one after another, want_rows
// (ascending places in `tokens`) the ones whose logits are asked for. want_sampling (n_want) and want_tokens (n_want) are given
// together or not at all: the token drawn after each wanted place. want_logits (optional): fp32 [n_want, vocab].
int nfn_engine_step(nfn_engine* e, const nfn_step_entry* entries, int n_entries, const int32_t* tokens, const int32_t* want_rows, int n_want,
                    const nfn_sampling* want_sampling, int32_t* want_tokens, float* want_logits);
// Tokens the page pool still has room for (whole free pages); -1 for engines without pages.
long long nfn_engine_free_tokens(const nfn_engine* e);
// The CUDA stream the engine launches on (for events around its calls).
void* nfn_engine_stream(const nfn_engine* e);
int nfn_engine_release(nfn_engine* e, int slot);
int nfn_engine_slot_length(const nfn_engine* e, int slot);
// Copies the bf16 logits of the last step for `slot` to the host as fp32 (vocab entries).
int nfn_engine_last_logits(nfn_engine* e, int slot, float* out_vocab);

// ---- block verification (speculative decoding, appends at a position > 0) ---------------------
// Allocates the staging buffers once (max_rows <= 128 rows per slot and call;
// max_batch * max_rows must not exceed max(max_seq, max_batch)).
int nfn_engine_enable_verify(nfn_engine* e, int max_rows);
// Runs `rows` tokens per slot (tokens[slot * rows + r]; n_rows[slot] of them live, 0 = slot not
// in this call) through the model at positions length[slot] ..., WITHOUT touching the KV caches:
// attention reads the cache prefix plus the block, the block's K/V go to per-layer staging
// buffers. argmax_out[slot * rows + r] = most likely successor after row r.
int nfn_engine_verify(nfn_engine* e, const int32_t* tokens, const int32_t* n_rows, int rows, int32_t* argmax_out);
// fp32 logits of row `row` of `slot` in the last verification.
int nfn_engine_verify_logits(nfn_engine* e, int slot, int row, float* out_vocab);
// Appends the first accepted[slot] rows of the last verification to the caches (one launch for
// all layers) and advances the slot lengths; rows that were not accepted leave no trace.
int nfn_engine_commit(nfn_engine* e, const int32_t* accepted);
// Shortens a slot to its first n tokens. Fails when a sliding-window cache of the slot has
// already wrapped (its older rows are gone).
int nfn_engine_truncate(nfn_engine* e, int slot, int n);
// Copies the first n cached tokens of src_slot into dst_slot (device-to-device; the two slots
// are independent afterwards).
int nfn_engine_fork(nfn_engine* e, int src_slot, int dst_slot, int n);

// ---- hidden-state taps (context of a block-diffusion draft model) ------------------------------
// Keeps the residual stream after each listed layer (0-based) for every cached position of every slot:
// [max_batch][max_seq][d_model] bf16 per tap. Prefill, decode steps and verification blocks all write
// their rows; rows of a block that is not committed are overwritten before they can be read. Must be
// called after finalize and before the first decode step.
int nfn_engine_enable_taps(nfn_engine* e, const int32_t* layers, int n);
// Copies positions [pos0, pos0 + n) of `slot` to dst as bf16 [n][taps * d_model] (taps side by side in
// the order they were enabled). dst is device memory when dst_on_device != 0, else host memory.
int nfn_engine_read_taps(nfn_engine* e, int slot, int pos0, int n, void* dst, int dst_on_device);
// Kernel launches issued so far by this engine (graph replays count their captured launches).
long long nfn_engine_launches(const nfn_engine* e);

#ifdef __cplusplus
}
#endif
