// C ABI of the sm_100a kernel library (libnfn_b200_kernels.so).
//
// Every entry point takes raw device pointers plus the CUDA stream to launch on
// and returns 0 on success or a negative argument/launch error. Kernels never
// allocate; scratch is passed in by the caller. Waits inside kernels are bounded
// and report through a per-device status word (nfn_status_read_reset).
//
// Plays the role of the reference's dlopen kernel boundary
// (neuralfn/csrc/native_train/tile_ops.h), redesigned around tcgen05/TMA kernels.
#pragma once
#include <stdint.h>

#ifdef __cplusplus
extern "C" {
#endif

typedef void* nfn_stream_t;

// ---- library / status -------------------------------------------------------
int nfn_abi_version(void);
// Returns the first non-zero error code recorded by any kernel on the current
// device since the last call (0 = none) and clears it. Synchronises the device.
int nfn_status_read_reset(void);
// Same, but does not synchronise (reads whatever has landed) and does not clear.
int nfn_status_peek(void);
// Host-side test hook: sets the status word of the current device.
int nfn_status_set(int code);
const char* nfn_last_error(void);

// ---- GEMM family (tcgen05 + TMEM + TMA) -------------------------------------
// C[M,N] = epilogue( sum_k opA[m,k] * opB[n,k] )
//   a_mn = 0: A is stored [M,K] (K contiguous, leading dim lda)
//   a_mn = 1: A is stored [K,M] (M contiguous, leading dim lda)
//   b_mn = 0: B is stored [N,K] (K contiguous, leading dim ldb)
//   b_mn = 1: B is stored [K,N] (N contiguous, leading dim ldb)
// A, B are bf16. C is bf16 unless NFN_EPI_OUT_F32.
// Epilogue order: acc*alpha -> +bias[n] -> (save pre-activation to aux_out)
//   -> activation -> * act'(aux_in) (DACT) -> + aux_in (RESID) -> + C (ACCUM).
enum {
  NFN_EPI_BIAS = 1 << 0,      // add bf16 bias[N]
  NFN_EPI_SAVE_PRE = 1 << 1,  // write pre-activation to aux_out (bf16, ld = ld_aux_out)
  NFN_EPI_RESID = 1 << 2,     // add bf16 residual aux_in[M,N]
  NFN_EPI_DACT = 1 << 3,      // multiply by act'(aux_in[M,N]) (aux_in = saved pre-activation)
  NFN_EPI_ACCUM = 1 << 4,     // C += result
  NFN_EPI_OUT_F32 = 1 << 5,   // C is fp32
  NFN_EPI_COPY_BF16 = 1 << 6, // with OUT_F32: also write bf16 of the final C to aux_out (ld = ld_aux_out)
  NFN_EPI_ACT_SHIFT = 8,      // activation id in bits 8..11
};
enum { NFN_ACT_NONE = 0, NFN_ACT_GELU_TANH = 1, NFN_ACT_GELU_ERF = 2, NFN_ACT_SILU = 3,
       NFN_ACT_RELU2 = 4, NFN_ACT_TANH_CAP = 5 /* cap*tanh(x/cap), cap = act_param */, NFN_ACT_RELU = 6,
       NFN_ACT_CLAMPED = 7 /* feed-forward gates only, see nfn_gate_clamp */ };

typedef struct {
  const void* a; const void* b; void* c;
  int m, n, k;
  int lda, ldb, ldc;
  int a_mn, b_mn;
  int flags;
  float alpha;
  float act_param;
  const void* bias;
  const void* aux_in; int ld_aux_in;
  void* aux_out; int ld_aux_out;
  // split-K (plain products only): 0 = choose automatically, 1 = never, n > 1 = force n.
  // Needs an fp32 workspace of split * M * N elements; without one no split happens.
  void* workspace; long long workspace_bytes; int split_k;
} nfn_gemm_args;

int nfn_gemm_bf16(const nfn_gemm_args* args, nfn_stream_t stream);
// Grouped contraction for expert weight gradients: C[g] = A[K rows of group g, M]^T . B[same rows, N] for every group in one
// launch. Both operands MN-major; group_rows = groups + 1 device ints (multiples of 64; padding rows zero); C slices
// group_stride elements apart. Only alpha, fp32 output and accumulate of the epilogue flags apply.
int nfn_gemm_grouped_k(const nfn_gemm_args* args, const int* group_rows, int groups, long long group_stride, nfn_stream_t stream);
// Routes eligible products (K-major A and B, bf16 output, no split-K, at least one 256 x 256
// tile per SM pair) to the CTA-pair kernel (tcgen05 cta_group::2, 256 x 256 tile per 2-CTA
// cluster). Returns the previous setting. On by default; NFN_GEMM_PAIR=0 turns it off.
int nfn_gemm_set_gemv_mode(int on);  // 1 (default): M <= 2 products use the weight-streaming GEMV kernel; returns the old setting
int nfn_gemm_set_pair_mode(int on);

// ---- GEMMs fused with their collective (gemm_tp.cu) ----------------------------------------
// K-major bf16 operands: A [M, K], B [N, K] (out x in), C = A . B^T. Buffers named "peer"
// are the same allocation on every rank (symmetric memory), indexed by rank.
//   NFN_TP_AG_A: `a` is the local gathered buffer [M, K] (lda == K); this rank's rows
//                [rank * rows_per_rank, +rows_per_rank) are already in it, the other rows are
//                pulled from peer_bufs[r] inside the kernel. C [M, N] = bias/activation epilogue.
//   NFN_TP_AG_B: the same with the gathered operand on the B side (`b` [N, K], ldb == K).
//   NFN_TP_RS:   C is not written; partial tiles go to peer_bufs[owner] (bf16 slots
//                [world, rows_per_rank, N]); the kernel then reduces this rank's slots into
//                `out` [rows_per_rank, N] (+ bias + resid).
// ctrl_*: per-rank control block of ctrl_ints int32 (zero-initialised once): [0, 8) flags
// written by peers, [16] ticket, [32, 32 + blocks) block flags. epoch must grow by one per
// call on every rank alike; the value used is epoch + *epoch_dev (epoch_dev may be NULL).
//   NFN_TP_GROUPED: single-rank grouped GEMM (mixture-of-experts): A rows sorted by group and
//                padded to 128-row tiles, B = [groups, N, K]; tile t uses B[tile_group[t]];
//                only the first *num_m_tiles_dev tiles are computed (device-side count).
enum { NFN_TP_AG_A = 0, NFN_TP_AG_B = 1, NFN_TP_RS = 2, NFN_TP_GROUPED = 3 };
typedef struct {
  int mode;
  const void* a; const void* b; void* c;
  int m, n, k;
  int lda, ldb, ldc;
  int flags; float act_param; const void* bias;   // NFN_EPI_BIAS and activation bits
  int rank, world, rows_per_rank;
  int epoch; const int* epoch_dev;
  const void* peer_bufs[8];
  int* ctrl_local; int* ctrl_peer[8]; int ctrl_ints;
  void* out; int ld_out; const void* resid; int ld_resid;   // NFN_TP_RS only
  int n_copy;                                               // gather CTAs (0 = default 16)
  const int* tile_group; const int* num_m_tiles_dev; int groups;   // NFN_TP_GROUPED only
} nfn_gemm_tp_args;
int nfn_gemm_tp(const nfn_gemm_tp_args* args, nfn_stream_t stream);

// ---- one-shot all-reduce + residual + RMS norm (allreduce_fused.cu) ---------------------------
// peer_bufs[r]: rank r's copy of the symmetric bf16 [rows, ld] partial-result buffer;
// multicast_buf: multicast address of that buffer (NVSwitch reduction) or NULL for peer loads.
// resid (optional) is updated in place with sum + bias + resid; out receives the RMS-normed
// row (norm_weight != NULL) or the reduced row itself. ctrl blocks: >= 32 int32, zeroed once.
int nfn_allreduce_resid_norm(const void* const* peer_bufs, const void* multicast_buf, int* ctrl_local, int* const* ctrl_peer,
                             int rank, int world, int epoch, const int* epoch_dev, int rows, int n, int ld,
                             const void* bias, void* resid, int ld_resid, const void* norm_weight, float eps,
                             int centered, void* out, int ld_out, nfn_stream_t stream);
// Stream-ordered wait until every peer finished reading this rank's buffer in call `epoch`.
int nfn_allreduce_wait_readers(const int* ctrl_local, int world, int epoch, const int* epoch_dev, nfn_stream_t stream);

// ---- flash attention for training and prefill (attention_fwd2.cu, attention_bwd2.cu) ----------------
// q: bf16 rows [B*T] x (Hq*D) with row stride ld_q; k, v: rows x (Hkv*D); o: rows x (Hq*D);
// lse: fp32 [B, Hq, T] (optional in the forward pass). head_dim D is 64 or 128.
//   causal = 1: keys <= query.  window = W > 0: causal keys in (q - W, q], or |q - k| < W when
//   not causal.  seq_ids (optional int32 [B*T]): a key is visible only when its id equals the
//   query's (packed sequences).  softcap = c > 0: scores become c * tanh(s * scale / c).
//   gate (optional bf16 [rows, Hq*D], forward only): o *= sigmoid(gate).
// The backward pass needs delta scratch (fp32 [B, Hq, T]); it runs two kernels, one that owns a
// key block (dK, dV) and one that owns a query tile (dQ), so no gradient is accumulated with atomics.
typedef struct {
  const void* q; const void* k; const void* v; void* o; float* lse;
  int B, T, Hq, Hkv, D;
  int ld_q, ld_k, ld_v, ld_o;
  int causal, window;
  float scale, softcap;
  const int* seq_ids;
  const void* gate; int ld_gate;
  // backward only
  const void* d_o; int ld_do;
  float* delta;
  void* dq; void* dk; void* dv; int ld_dq, ld_dk, ld_dv;
} nfn_attention_args;
int nfn_attention_forward_ex(const nfn_attention_args* args, nfn_stream_t stream);
int nfn_attention_backward_ex(const nfn_attention_args* args, nfn_stream_t stream);
int nfn_attention_forward(const void* q, const void* k, const void* v, void* o, float* lse, int B, int T, int Hq,
                          int Hkv, int D, int ld_q, int ld_k, int ld_v, int ld_o, int causal, int window, float scale,
                          nfn_stream_t stream);
int nfn_attention_backward(const void* dout, const void* q, const void* k, const void* v, const void* o, const float* lse,
                           float* delta, float* dq_accum, void* dq, void* dk, void* dv, int B, int T, int Hq, int Hkv,
                           int D, int ld_do, int ld_q, int ld_k, int ld_v, int ld_o, int ld_dq, int ld_dk, int ld_dv,
                           int causal, int window, float scale, nfn_stream_t stream);
// 2 (default): pipelined kernels; 1: the first-generation kernels (plain masks only). Returns the old value.
int nfn_attention_set_impl(int impl);

// ---- rotary embedding (rope.cu) -----------------------------------------------------------------
// In place on the q and k heads of packed rows (q | k | v). sign = +1: "hf" convention,
// -1: "legacy"; the backward pass is the same call with the opposite sign. Tables are fp32
// [max_pos, rot_dim/2]; positions (optional int32 per row) default to row % T.
int nfn_rope_inplace(void* qkv, int ld, long long tokens, int T, int n_q_heads, int n_kv_heads, int head_dim,
                     int rot_dim, const float* cos_table, const float* sin_table, const int* positions,
                     int max_pos, float sign, float q_scale, nfn_stream_t stream);
// Per-head RMS norm (optional bf16 weights [head_dim]) + rotation + query scale in one pass.
int nfn_qk_norm_rope_forward(void* qkv, int ld, long long tokens, int T, int n_q_heads, int n_kv_heads, int head_dim,
                             const void* q_weight, const void* k_weight, const float* cos_table,
                             const float* sin_table, const int* positions, int max_pos, float sign, float eps,
                             float q_scale, float* rstd_out, nfn_stream_t stream);

// ---- token selection (sampling.cu) --------------------------------------------------------------
// logits: bf16 (is_fp32 = 0) or fp32 rows of V entries, row stride ld. Ties go to the lowest
// index. index_offset is added to every result (vocabulary shard offset under tensor
// parallelism). argmax workspace: rows * 8 bytes at least, rows * 512 for full parallelism.
int nfn_argmax_rows(const void* logits, int is_fp32, long long ld, int rows, int V, int* out_idx, float* out_val,
                    void* workspace, long long workspace_bytes, int index_offset, nfn_stream_t stream);
// Merges per-rank winners laid out [world, rows] (values and already-offset indices).
int nfn_argmax_merge(const float* vals, const int* idx, int world, int rows, int* out_idx, float* out_val,
                     nfn_stream_t stream);
// temperature <= 0 or top_k == 1: greedy. top_k = 0 and top_p in {0, 1}: no truncation.
// row_params (optional, fp32 [rows, 3] = temperature, top_k, top_p) overrides the scalars per
// row. Randomness: Philox4x32-10 keyed by seed, counter (element/4, row, offset + *offset_dev).
int nfn_sample_rows(const void* logits, int is_fp32, long long ld, int rows, int V, int* out_idx, float* out_logprob,
                    float temperature, int top_k, float top_p, const float* row_params, unsigned long long seed,
                    unsigned long long offset, const unsigned long long* offset_dev, int index_offset,
                    nfn_stream_t stream);

// ---- decode attention (decode_attention.cu) -----------------------------------------------------
// One new token per sequence. qkv: bf16 [B, ld] packed (q | k | v) rows of the new token;
// caches: bf16 [B, n_kv_heads, cap, head_dim] with cache_batch_stride elements between
// sequences; lengths[b] counts the new token; out: bf16 [B, n_q_heads * head_dim]. The call
// appends the (normed, rotated) k and v of the new token at slot (len - 1) % cap. The
// workspace must be zero-filled once before its first use and is left ready for the next call.
long long nfn_decode_attention_workspace_bytes(int B, int n_q_heads, int n_kv_heads, int head_dim, int max_splits);
// 1 (default): mma.sync kernel, 16 cache positions per warp step; 0: SIMT kernel. Returns the previous setting.
int nfn_decode_attention_set_impl(int impl);
int nfn_decode_attention(const void* qkv, int ld, void* k_cache, void* v_cache, long long cache_batch_stride,
                         const int* lengths, void* out, int B, int n_q_heads, int n_kv_heads, int head_dim, int cap,
                         const void* q_norm_weight, const void* k_norm_weight, int qk_norm, float eps,
                         const float* cos_table, const float* sin_table, int max_pos, float rope_sign, float scale,
                         void* workspace, long long workspace_bytes, int splits, nfn_stream_t stream);

// ---- block attention over a KV cache (block_attention.cu) ------------------------------------------
// `rows` (<= 128) new rows per sequence attend to the sequence's cached keys plus the block's own
// keys; the caches are only read. qkv: [B*rows, ld] packed q | k | v (norm / rotary already
// applied); caches [B][n_kv_heads][cap][head_dim]; lengths[b] = tokens already cached (the block
// starts at that position); n_rows (optional) = live rows per sequence, 0 skips the sequence.
// window = 0: every cached key is visible; otherwise keys inside (q - window, q] (window <= cap).
// causal = 0 lets every block row see the whole block (draft blocks). stage_k / stage_v
// (optional, [B*rows, n_kv_heads*head_dim]) receive the block's own K / V rows for a later
// nfn_kv_commit_layers. splits = 0 picks the KV split count.
long long nfn_block_attention_workspace_bytes(int B, int rows, int n_q_heads, int n_kv_heads, int head_dim, int max_splits);
int nfn_block_attention(const void* qkv, int ld, const void* k_cache, const void* v_cache, const int* lengths, const int* n_rows,
                        void* out, int ld_o, void* stage_k, void* stage_v, int B, int rows, int n_q_heads, int n_kv_heads,
                        int head_dim, int cap, int window, int causal, float scale, void* workspace, long long workspace_bytes,
                        int splits, nfn_stream_t stream);
// Appends the first accepted[b] staged rows of every layer to that layer's cache at positions
// lengths[b] ... (ring rows position % caps[layer]). All pointer arrays live in device memory.
int nfn_kv_commit_layers(const void* const* stage_k, const void* const* stage_v, void* const* k_caches, void* const* v_caches,
                         const int* caps, const int* lengths, const int* accepted, int n_layers, int B, int rows, int n_kv_heads,
                         int head_dim, nfn_stream_t stream);

// Products with a few rows over large K-major weights (decode batches, verification blocks): 1 (default) = 3 - 16 rows take the
// mma.sync weight-streaming kernel of gemm_skinny.cu, 2 = up to 64 rows do, 0 = none (tcgen05 split-K path). Returns the previous setting.
int nfn_gemm_skinny_set_impl(int mode);

// Hidden-state taps: row r of x (bf16 [rows, ldx], C columns used) belongs to sequence r / block_rows and is copied to
// position lengths[sequence] + r % block_rows + pos_offset of dst [sequences][max_pos][C] (slot_stride elements between
// sequences). live_rows (optional): rows at or past live_rows[sequence] are skipped. Positions outside [0, max_pos) are skipped.
int nfn_rows_to_slots(const void* x, int ldx, int rows, int C, void* dst, long long slot_stride, int max_pos, const int* lengths,
                      int block_rows, int pos_offset, const int* live_rows, nfn_stream_t stream);

// ---- GEMM over K-quant weights, dequantisation fused into the operand pipeline (gemm_kquant.cu) ----
// C[M, N] = A[M, K] . dequant(W)^T with args->b pointing at N rows of K / 256 super-blocks
// (qtype: NFN_QTYPE_Q4_K / Q5_K / Q6_K, declared below). K-major A, bf16 output, the bias /
// activation / residual epilogues of nfn_gemm_bf16; ldb, a_mn, b_mn and split_k are ignored or refused.
int nfn_gemm_kquant(int qtype, const nfn_gemm_args* args, nfn_stream_t stream);
// The same with NF4 base weights (qtype NFN_QTYPE_NF4: args->b = N rows of K / 2 code bytes, low
// nibble = even element; absmax fp32 [N, K / 64]) and / or a fused LoRA branch: lora_t = bf16
// [M, >= 64] holding scale * (x A^T) in its first r columns and zeros up to column 64, lora_b =
// bf16 [N, >= 64] holding the adapter's B matrix likewise. Pass NULL adapters for none.
int nfn_gemm_quant_lora(int qtype, const nfn_gemm_args* args, const float* absmax, const void* lora_t, int ld_t,
                        const void* lora_b, int ld_b, nfn_stream_t stream);

// ---- TurboQuant KV cache (turboquant.cu) ------------------------------------------------------------
// Device tables of one codec: rotation / projection [D, D] fp32 (rotated = R x), centroids [5][16]
// fp32 (row = bit width), fields [D][2] int32 (bit offset inside the index area, width).
// Record: [norm f32 | residual norm f32 + D/8 sign bytes (qjl keys) | packed indices | pad to 16].
typedef struct {
  const float* rotation; const float* projection; const float* centroids;
  const int* key_fields; const int* value_fields;
  int D, qjl, key_rec_bytes, value_rec_bytes;
} nfn_tq_tables;
// Encodes head vectors x[row, h * D ...] (bf16, row stride ld) into records[seq[row]][h][slot[row]].
int nfn_turboquant_encode(const nfn_tq_tables* tables, const void* x, long long ld, const int* seq, const int* slot, int rows,
                          int n_heads, int cap, int is_key, void* records, nfn_stream_t stream);
// One query row per sequence against records [B][n_kv_heads][cap]; the first min(lengths[b], cap)
// rows of every head are live. q: bf16 [B, ld_q]; out: bf16 [B, ld_o].
int nfn_turboquant_attention(const nfn_tq_tables* tables, const void* q, int ld_q, const void* k_records, const void* v_records,
                             const int* lengths, void* out, int ld_o, int B, int n_q_heads, int n_kv_heads, int cap, float scale,
                             nfn_stream_t stream);

// ---- quantised weights (quant.cu) ---------------------------------------------------------------
enum { NFN_QTYPE_Q4_K = 12, NFN_QTYPE_Q5_K = 13, NFN_QTYPE_Q6_K = 14, NFN_QTYPE_NF4 = 100 };  // GGUF type ids; NF4 is this library's own
int nfn_quant_block_bytes(int qtype);
int nfn_dequant_kquant(int qtype, const void* blocks, long long n_blocks, void* out_bf16, nfn_stream_t stream);
int nfn_dequant_nf4(const void* codes, const float* absmax, long long n_weights, int group, void* out_bf16,
                    nfn_stream_t stream);
// y[b, n] = W1[n, :] . x[b, :]  (silu(W1 x) * (W2 x) when w2 != NULL) + bias[n] + resid[b, n];
// W rows are K/256 consecutive super-blocks; B <= 8.
int nfn_kquant_gemv(int qtype, const void* w1, const void* w2, const void* x, int ldx, void* y, int ldy,
                    const void* bias, const void* resid, int ld_resid, int B, int N, int K, nfn_stream_t stream);

int nfn_allreduce_sandwich_norm(const void* const* peer_bufs, const void* multicast_buf, int* ctrl_local, int* const* ctrl_peer,
                                int rank, int world, int epoch, const int* epoch_dev, int rows, int n, int ld, const void* bias,
                                const void* post_weight, float post_eps, void* resid, int ld_resid, const void* norm_weight,
                                float eps, int centered, void* out, int ld_out, nfn_stream_t stream);

// ---- gated attention, training (gate.cu) ----
int nfn_sigmoid_gate_forward(const void* att, int ld_att, const void* gate, int ld_gate, void* out, int ld_out, long long rows, int width,
                             nfn_stream_t stream);
int nfn_sigmoid_gate_backward(const void* dout, int ld_dout, const void* att, int ld_att, const void* gate, int ld_gate, void* datt,
                              int ld_datt, void* dgate, int ld_dgate, long long rows, int width, nfn_stream_t stream);

// ---- counter-based dropout for the LoRA adapter branch (dropout.cu) ----
// out (+)= keep ? x / (1 - p) : 0 with keep = f(seed, stream_id, *step_dev, row, column): calling it again with the same ids
// reproduces the mask (backward pass, recomputation). bf16 [rows, width], width a multiple of 8.
int nfn_dropout_apply(const void* x, int ld_x, void* out, int ld_out, long long rows, int width, float p, unsigned long long seed,
                      int stream_id, const long long* step_dev, int accumulate, nfn_stream_t stream);

// ---- differential attention glue (diff_attention.cu) ----
int nfn_diff_partials(void);
int nfn_diff_q_expand(const void* q, int ldq, void* q2, long long tokens, int H, int D, nfn_stream_t stream);
int nfn_diff_q_collapse(const void* dq2, void* dq, int lddq, long long tokens, int H, int D, nfn_stream_t stream);
int nfn_diff_combine(const void* a, const void* lambda, float out_scale, float eps, void* out, float* rstd,
                     long long tokens, int H, int D, nfn_stream_t stream);
int nfn_diff_combine_backward(const void* dout, const void* a, const void* lambda, float out_scale, const float* rstd,
                              void* da, float* partial, void* dlambda, long long tokens, int H, int D, nfn_stream_t stream);

// ---- steps of mixed batches over paged caches (paged_rows.cu, paged_decode.cu, paged_prefill.cu) ----------------------------
// A step's rows are the next tokens of several sequences, one sequence ("entry") after another. Activations are bf16 (f32 = 0)
// or fp32 (f32 = 1), weights bf16, the residual stream fp32. Row widths are multiples of 16.
// Cache pages hold NFN_KV_PAGE = 64 tokens: keys [page][kv_heads][64][dim_p], values transposed [page][kv_heads][vdim_p][64];
// table[slot * table_ld + position / 64] names the page.
typedef struct {
  int row0, n;         // rows of this tile (at most 16, not crossing a multiple of 16 positions)
  int e_row0, e_n;     // first row and row count of the entry it belongs to
  int e_pos0;          // position of the entry's first row
  int slot;            // < 0: padding, skipped
  int parity;          // which half of the convolution state holds the entry's history (the other one is written)
  int pad;
} nfn_row_tile;
// Row pass: base = embed[token] * embed_scale (tokens != NULL) or x[src_rows ? src_rows[r] : r]; with y: base += y / rms(y) *
// y_weight; x_out (optional) = base; h (optional) = base / rms(base) * weight. rms(z) = sqrt(sum z^2 / width + eps).
typedef struct {
  int f32, rows, width, ld;               // ld: row pitch of x, y, h and of the embedding table
  const float* x; float* x_out; const int* src_rows;
  const int* tokens; const void* embed; float embed_scale; int vocab;
  const void* y; const void* y_weight;
  void* h; const void* weight;
  float eps;
} nfn_row_norm_args;
int nfn_row_norm(const nfn_row_norm_args* args, nfn_stream_t stream);
// After the input projection [q | k | v | g | gate | up] of a layer: causal depthwise convolution on q, k, v over the entry's
// rows and the stored history (conv: bf16 [taps][nq + nk + nv], NULL and taps = 0: none), query temperature, keys and values into
// their pages, ff_out = act(gate) * up. nk = nv = 0: the layer reads another layer's cache.
typedef struct {
  int f32;
  const void* in; int ld_in;
  int nq, nk, nv, off_gate, off_up, ff, act;
  const void* conv; int taps;
  int conv_act;                           // NFN_ACT_NONE or NFN_ACT_SILU on the convolved values
  void* state; long long state_half;      // [2][slots][taps - 1][nq + nk + nv]; elements between the halves
  void* q_out; int ld_q;
  void* k_pool; void* v_pool; int kv_heads, dim_p, vdim_p;
  const int* table; int table_ld;
  float temp_coef; int temp_every;
  void* ff_out; int ld_ff;
  const nfn_row_tile* tiles; int n_tiles;
  int tile_rows;                          // most rows of a tile of this call
  int rows;                               // rows of the call
} nfn_mix_args;
int nfn_mix_rows(const nfn_mix_args* args, nfn_stream_t stream);
// NFN_ACT_CLAMPED, the gate of a feed-forward with bounded inputs: g = min(gate, limit), u = max(-limit, min(up, limit)), g * sigmoid(slope * g) * (u + shift).
typedef struct { float limit, slope, shift; } nfn_gate_clamp;
// out[r] = act(gate) * up of rows [.. off_gate: gate .. off_up: up ..]; off_up < 0: out[r] = act(gate). clamp: with NFN_ACT_CLAMPED (which needs both).
int nfn_ff_rows(int f32, const void* in, int ld_in, int off_gate, int off_up, int ff, int act, const nfn_gate_clamp* clamp, void* out, int ld_out, int rows,
                nfn_stream_t stream);
// Attention of a step's rows over the pages. score = q . k * scale, capped to softcap * tanh(score / softcap) (0: off), minus
// slopes[h] * (i - j); keys 0 <= i - j < window (0: all) and the first keep_first ones of the sequence, with chunk > 0 only those of the query's own
// chunk of that many positions; softmax, with sink != 0 over one more score of 0 that has no value, with sinks over one of
// sinks[h] (not scaled, not capped); out = P V * sigmoid(gate) (gate optional).
// q: [rows, heads * dim_p]; out: row pitch ld_o, head pitch vdim_p. v_pool = NULL: a key's value is its first vdim_p channels (latent caches).
typedef struct {
  int f32;
  const void* q; int ld_q;
  const void* k_pool; const void* v_pool; int kv_heads, dim_p, vdim_p; long long pages;
  const int* table; int table_ld;
  int heads, window;
  float scale; const float* slopes;       // fp32 [heads], NULL: no distance bias
  const void* gate; int ld_gate;
  void* out; int ld_o;
  const int* row_slot; const int* row_pos; // per row (slot < 0: skipped)
  int rows;                               // nfn_paged_attention_rows: rows [row0, row0 + rows)
  int row0;
  int max_keys;                           // most keys a row of this call sees (sizes the split)
  void* workspace; long long workspace_bytes;   // split partials; the first 64 KB are counters, zeroed once
  const int* tiles; int n_tiles;          // nfn_paged_attention_tiles: {row0, rows, slot, pos0} each
  int total_rows;                         // rows of the q buffer
  int keep_first; float softcap; int sink;
  int chunk;
  const void* sinks;                      // bf16 [heads]
} nfn_paged_attention_args;
// One query row at a time (single tokens, very short portions): bf16 goes to the tensor cores in 32-key steps, fp32 and sizes
// outside its limits to the plain kernel.
int nfn_paged_attention_rows(const nfn_paged_attention_args* args, nfn_stream_t stream);
long long nfn_paged_attention_workspace_bytes(int rows, int heads, int vdim_p);
// Tiles of consecutive rows of one sequence (prompt portions), tcgen05. nfn_paged_tile_rows: rows per tile for these sizes, 0 when
// the sizes need nfn_paged_attention_rows.
int nfn_paged_tile_rows(int f32, int heads, int kv_heads, int dim_p, int vdim_p);
int nfn_paged_attention_tiles(const nfn_paged_attention_args* args, nfn_stream_t stream);

// ---- heads of a step's rows (head_rows.cu) ---------------------------------------------------------------------------------------
// After the input projection of an attention layer: per head of dim values (pitch dim_p), RMS norm with a weight shared by the heads (NULL: none),
// then rotation of the first rot_dims dimensions, pairs (2i, 2i + 1) by position * freq_i; freq: rot_dims / 2 pairs (high, low part of the
// frequency). Queries [rows][heads] -> q_out, keys and values into their pages; off_v = off_k: the values are the keys as projected.
typedef struct {
  int f32;
  const void* in; int ld_in, off_k, off_v;
  int heads, kv_heads, dim, dim_p, vdim_p;         // kv_heads = 0: queries only
  const void* q_norm; const void* k_norm; float eps;
  const float* freq; int rot_dims;
  void* q_out; int ld_q;
  void* k_pool; void* v_pool;
  const int* table; int table_ld;
  const nfn_row_tile* tiles; int n_tiles, tile_rows;
} nfn_head_rows_args;
int nfn_head_rows(const nfn_head_rows_args* args, nfn_stream_t stream);
// The same for latent attention. in: queries [heads][dim_p + rot_p] and, with k_pool, [rank_p latent | rot_p shared key part] at off_kv. The latent is
// normed, the key part rotated, both go into the page [64][rank_p + rot_p]. Rotated query parts go to q_out ([heads][dim_p + rot_p], with
// the unrotated ones) from row q_row0 on and to q_lat ([heads][rank_p + rot_p], at column rank_p) before it.
typedef struct {
  int f32;
  const void* in; int ld_in, off_kv;
  int heads, dim_p, rot_dim, rot_p, rank, rank_p;
  const void* c_norm; float eps;
  const float* freq;
  void* q_out; int ld_q, q_row0;
  void* q_lat;
  void* k_pool;
  const int* table; int table_ld;
  const nfn_row_tile* tiles; int n_tiles, tile_rows;
} nfn_latent_rows_args;
int nfn_latent_rows(const nfn_latent_rows_args* args, nfn_stream_t stream);
// out[r][g][n] = act(sum_k in[r][g][k] w[g][n][k]): one small product per group and row (the per-head projections around a latent cache, several inputs
// with a matrix each). in, out: activation type, group pitches in elements; w bf16. Sizes are multiples of 16. tail_n > 0: one more product of the same
// depth, from the input tail_in elements into each row, with an fp32 result and no activation. gate: out *= sigmoid(gate[r][g][n]).
typedef struct {
  int f32, rows, groups, n, k;
  const void* in; long long ld_in, in_group;
  const void* w;
  void* out; long long ld_out, out_group;
  int act, tail_n;
  long long tail_in;
  const void* tail_w;
  float* tail_out; int ld_tail;
  const void* gate; long long ld_gate, gate_group;
} nfn_group_products_args;
int nfn_group_products(const nfn_group_products_args* args, nfn_stream_t stream);

// ---- latent attention over prompt portions (paged_prefill.cu, head_rows.cu) --------------------------------------------------------
// A portion's visible latents, page by page, as rows of one matrix: page first_page + i of the slot to rows [row0 + 64 i, ...), i < n_pages.
typedef struct { int slot, first_page, n_pages, row0; } nfn_latent_span;
int nfn_latent_gather(int f32, const void* pool, int ld_pool, int cols, const int* table, int table_ld, const nfn_latent_span* spans, int n_spans,
                      int max_pages, void* out, nfn_stream_t stream);
// nfn_paged_attention_tiles with keys and values formed from the latents: x [x_rows][heads * dim_u unrotated keys | heads * vdim_p values], the rotated
// key part (rot_p channels at column rank_p) still in the pages. args: dim_p = dim_u + rot_p, kv_heads = heads; tiles hold 128 rows;
// x_base[slot]: row of x that belongs to position 0 of the sequence (may be negative).
typedef struct { const void* x; int x_rows, dim_u, rot_p, rank_p; const int* x_base; } nfn_latent_expanded;
int nfn_latent_tile_rows(int f32, int dim_u, int rot_p, int vdim_p);
int nfn_latent_attention_tiles(const nfn_paged_attention_args* args, const nfn_latent_expanded* x, nfn_stream_t stream);
// out = gelu_tanh(gate) * side_embed[token][col0 + c]: gate fp32 [rows, ld], out bf16 / fp32 with the same pitch.
int nfn_side_mul(int f32, const float* gate, const int* tokens, const void* side_embed, long long ld_embed, int col0, int vocab, void* out,
                 int ld, int rows, int width, nfn_stream_t stream);
// C[M, N] (fp32) (+)= A[M, K] (fp32) . B[N, K]^T (bf16) + bias[N] (bf16, optional), true 32-bit arithmetic. K, leading dimensions
// multiples of 4.
int nfn_gemm_f32(const float* a, int lda, const void* b, int ldb, float* c, int ldc, int m, int n, int k, int accumulate, const void* bias,
                 nfn_stream_t stream);
// logits <- cap * tanh(scale * logits / cap) (cap = 0: scale only) on fp32 rows.
int nfn_logit_cap(float* logits, int ld, int rows, int cols, float scale, float cap, nfn_stream_t stream);

// ---- residual streams (stream_rows.cu) -------------------------------------------------------------------------------------
// A row's residual is `streams` fp32 rows of pitch ld, x [rows][streams][ld]. One pass finishes a sublayer and starts the next:
// all streams at once, x_t <- sum_s mix[s][t] x_s + out[t] y (mix, out: bf16; NULL: identity, ones; y = NULL: no update), then
// u = sum_s in[s] x_s (in: bf16; NULL: ones) and h = u / rms(u) * (weight + weight_offset), rms(z) = sqrt(sum z^2 / width + eps).
// The base is embed[token] * embed_scale in every stream (tokens != NULL) or row src_rows[r] (NULL: r) of x; y is the row of the
// same number, or with y_rows > 1 the sum of rows y_index[r * y_rows + j] (y_index NULL: r * y_rows + j), each times y_item[r * y_rows + j]
// (NULL: 1), plus row r of y_plus (NULL: none). With y_weight the update is normed first: y <- y_scale * y / rms(y) * y_weight.
// weight = NULL: h = u. scalar_norms: weight and y_weight are one number each, for all channels.
// With conv (bf16 [conv_taps][ld]) every row is an entry of its own (tiles: one per row) and h gets a causal convolution of itself over the sequence added,
// h + sum_j conv[j] h_(t - conv_taps + 1 + j), zero before its start; one stream. history: see nfn_input_conv.
enum { NFN_MAX_STREAMS = 16 };
typedef struct {
  int f32, rows, width, ld, streams;
  const float* x; float* x_out; const int* src_rows;
  const int* tokens; const void* embed; float embed_scale; int vocab;
  const void* y; int y_rows; const int* y_index;
  const void* mix; const void* out;
  const void* in; void* h; const void* weight;
  float eps, weight_offset;
  const float* y_item; const void* y_plus;
  const void* y_weight; float y_scale;
  int scalar_norms;
  const void* conv; int conv_taps; void* history; long long history_half;
  const nfn_row_tile* tiles;
} nfn_stream_args;
int nfn_stream_pass(const nfn_stream_args* args, nfn_stream_t stream);
// The same convolution over the rows of any entries: out[r] = h[r] + sum_j conv[j] h_(t - taps + 1 + j). h and out are different buffers of pitch ld in the
// activation type; history [2][slots][taps - 1][ld], its newest rows last: the half named by the tile's parity is read, the other written.
typedef struct {
  int f32, ld, taps;
  const void* h; const void* conv;        // bf16 [taps][ld]
  void* history; long long history_half;
  void* out;
  const nfn_row_tile* tiles; int n_tiles;
} nfn_input_conv_args;
int nfn_input_conv(const nfn_input_conv_args* args, nfn_stream_t stream);

// ---- gated delta rule with a decay per key channel (delta_rows.cu, delta_chunk.cu) -------------------------------------------
// Per head (query / key head h / (heads / kv_heads)), with the fp32 state S [dim][vdim] of the sequence:
//   q, k made unit vectors, z / sqrt(sum z^2 + unit_eps), q also times dim^-1/2;  g = exp(-exp(a_log_h) softplus(decay + dt_bias)) per channel;
//   S <- g * S;  u = sigmoid(beta) (v - S^T k);  S <- S + k u^T;  o = S^T q.
// qkv: rows [q: kv_heads * dim_p | k | v: heads * vdim_p] after convolution and activation; state [slots][heads][dim_p][vdim_p]; a
// sequence at position 0 starts from zero whatever the slot holds. o: fp32 rows of heads * vdim_p. Padded channels are zero in q, k, v.
typedef struct { int row0, n, slot, pos0; } nfn_seq_rows;   // slot < 0: skipped
typedef struct {
  int f32;
  const void* qkv; int ld_qkv;
  const void* beta; int ld_beta;          // projected, before the sigmoid
  const float* decay; int ld_decay;       // [rows][heads * dim_p]
  const void* a_log; const void* dt_bias; // bf16 [heads], [heads * dim_p]
  int heads, kv_heads, dim, dim_p, vdim_p;
  float unit_eps;
  float* state;
  float* o; int ld_o;
  const nfn_seq_rows* seqs; int n_seqs;
} nfn_delta_args;
int nfn_delta_rows(const nfn_delta_args* args, nfn_stream_t stream);     // token after token, any length
// Sixteen tokens at a time on the tensor cores (bf16, dim_p <= 256), for sequences of up to max_rows rows.
long long nfn_delta_chunk_workspace_bytes(int heads, int dim_p, int vdim_p, int max_seqs);   // 0: these sizes go token after token
int nfn_delta_chunks(const nfn_delta_args* args, int max_rows, void* workspace, long long workspace_bytes, nfn_stream_t stream);
// One token of every sequence, from the input product to the rows the output product reads: convolution with its history (tiles: one per row),
// SiLU, the rule, the output norm and gate. in: [q | k | v] at column 0, beta at off_beta; conv [taps][channels], taps >= 1; history as in
// nfn_mix_args. nfn_delta_step_fits: the sizes it takes, and few enough heads and rows for its large CTAs (more rows run faster as
// nfn_mix_rows, nfn_delta_rows, nfn_delta_out).
typedef struct {
  int f32, rows;
  const void* in; int ld_in, off_beta;
  const void* conv; int taps; void* history; long long history_half;
  const float* decay; int ld_decay; const void* a_log; const void* dt_bias;
  int heads, kv_heads, dim, vdim, dim_p, vdim_p;
  float unit_eps, norm_eps;
  float* state;
  const void* gate; int ld_gate; const void* weight;
  void* out; int ld_out;
  const nfn_row_tile* tiles;
} nfn_delta_step_args;
int nfn_delta_step_fits(int rows, int heads, int dim_p, int vdim_p);
int nfn_delta_step(const nfn_delta_step_args* args, nfn_stream_t stream);
// out = o / rms(o) * weight * sigmoid(gate) per head of vdim values (pitch vdim_p); weight bf16 [vdim_p], out and gate in the activation type.
// nfn_head_out: the same with weights per head (weight_pitch = vdim_p; 0: shared) and gate_act NFN_ACT_SILU (silu(gate)) or NFN_ACT_NONE (sigmoid).
int nfn_head_out(int f32, const float* o, int ld_o, const void* gate, int ld_gate, int gate_act, const void* weight, int weight_pitch, float eps, void* out,
                 int ld_out, int rows, int heads, int vdim, int vdim_p, nfn_stream_t stream);
int nfn_delta_out(int f32, const float* o, int ld_o, const void* gate, int ld_gate, const void* weight, float eps, void* out, int ld_out, int rows,
                  int heads, int vdim, int vdim_p, nfn_stream_t stream);

// ---- token shift and the bonus recurrence (wkv_rows.cu, wkv_chunk.cu) --------------------------------------------------------------------
// out[s][r] = h + (h' - h) * mu[s], s < n: h the row, h' the previous token's (the row before it in its entry, the stored one of the slot, zero at
// position 0). src fp32 or, with src_act, in the activation type; prev fp32 [2][slots][ld], the half named by the tile's parity is read, the other written.
typedef struct {
  int f32, src_act, width, ld, n;
  const void* src;
  const void* mu;                         // bf16 [n][ld]
  float* prev; long long prev_half;
  void* out; long long out_stride;        // elements between the outputs; row pitch ld
  const nfn_row_tile* tiles; int n_tiles;
} nfn_shift_args;
int nfn_shift_rows(const nfn_shift_args* args, nfn_stream_t stream);
// Per head, with the fp32 state S [dim][dim] of the sequence: o = S^T r + (r . (u k)) v;  S <- w S + k v^T,  w = exp(-exp(z + w0)) per key channel.
// rkv: rows [r | k | v] of heads * dim_p each; z fp32 [rows][heads * dim_p]; u, w0 bf16 [heads * dim_p]; state [slots][heads][dim_p][dim_p]; a sequence at
// position 0 starts from zero. o: fp32 rows. Padded channels are zero in r, k, v.
typedef struct {
  int f32;
  const void* rkv; int ld_rkv;
  const float* z; int ld_z;
  const void* w0; const void* u;
  int heads, dim, dim_p;
  float* state;
  float* o; int ld_o;
  const nfn_seq_rows* seqs; int n_seqs;
} nfn_wkv_args;
int nfn_wkv_rows(const nfn_wkv_args* args, nfn_stream_t stream);         // token after token, any length
long long nfn_wkv_chunk_workspace_bytes(int heads, int dim_p, int max_seqs);   // 0: these sizes go token after token
int nfn_wkv_chunks(const nfn_wkv_args* args, int max_rows, void* workspace, long long workspace_bytes, nfn_stream_t stream);
// tanh of the inner decay projection, ready for the outer product: fp32 in; out in the activation type, [rows][2 * rank_p] = rounded value | what rounding
// left out in bf16, [rows][rank_p] in 32-bit mode.
int nfn_tanh_split(int f32, const float* in, int ld_in, void* out, int ld_out, int rows, int rank_p, nfn_stream_t stream);
// One token of every sequence: decay (with its outer projection w2 [heads * dim_p][ld_w2], low fp32 [rows][rank_p] before the tanh), rule, output norm, gate.
// rkvg: rows [r | k | v | g]; tiles: one per row. nfn_wkv_step_fits: the sizes it takes.
typedef struct {
  int f32, rows;
  const void* rkvg; int ld_rkvg;
  const float* low; int ld_low, rank_p;
  const void* w2; int ld_w2;
  const void* w0; const void* u;
  int heads, dim, dim_p;
  float* state;
  const void* weight; float eps;
  void* out; int ld_out;
  const nfn_row_tile* tiles;
} nfn_wkv_step_args;
int nfn_wkv_step_fits(int rows, int dim_p);
int nfn_wkv_step(const nfn_wkv_step_args* args, nfn_stream_t stream);

// ---- linear attention with a constant decay per head (linear_rows.cu, linear_chunk.cu) ------------------------------------------------------
// Per head, with the fp32 state S [dim][vdim] of the sequence: S <- decay_h S + k v^T;  o = S^T q.
// qkv: rows [q: heads * dim_p | k | v: heads * vdim_p], activated; state [slots][heads][dim_p][vdim_p]; a sequence at position 0 starts from zero.
// powers: fp32 [heads][NFN_LINEAR_CHUNK + 1], decay_h^i. o: fp32 rows of heads * vdim_p. Padded channels are zero in q, k, v.
enum { NFN_LINEAR_CHUNK = 64 };
typedef struct {
  int f32;
  const void* qkv; int ld_qkv;
  const float* powers;
  int heads, dim_p, vdim_p;
  float* state;
  float* o; int ld_o;
  const nfn_seq_rows* seqs; int n_seqs;
} nfn_linear_args;
int nfn_linear_rows(const nfn_linear_args* args, nfn_stream_t stream);      // token after token, any length
// NFN_LINEAR_CHUNK tokens at a time on the tensor cores (bf16), for sequences of up to max_rows rows. The workspace lets the segments of a long sequence
// run side by side; 0 bytes: these sizes go token after token.
long long nfn_linear_chunk_workspace_bytes(int heads, int dim_p, int vdim_p, int max_seqs);
int nfn_linear_chunks(const nfn_linear_args* args, int max_rows, void* workspace, long long workspace_bytes, nfn_stream_t stream);
// One token of every sequence from the input product on: qkvg rows [q | k | v | g] before their activations; SiLU on q, k, v, the rule, then o / rms(o) *
// weight * sigmoid(g), the norm over all heads of a row together (vdim values each). Tiles: one per row. o: scratch, fp32 rows of heads * vdim_p; counters:
// one int per row, zero before the first call.
typedef struct {
  int f32, rows;
  const void* qkvg; int ld_qkvg;
  const float* powers;
  int heads, vdim, dim_p, vdim_p;
  float* state;
  float* o; int ld_o; int* counters;
  const void* weight; float eps;
  void* out; int ld_out;
  const nfn_row_tile* tiles;
} nfn_linear_step_args;
int nfn_linear_step_fits(int rows, int dim_p, int vdim_p);
int nfn_linear_step(const nfn_linear_step_args* args, nfn_stream_t stream);
// out = o / rms(o) * weight * sigmoid(gate) over whole rows of `cols` values of which `live` count; weight bf16 [cols], out and gate in the activation type.
int nfn_row_out(int f32, const float* o, int ld_o, const void* gate, int ld_gate, const void* weight, float eps, void* out, int ld_out, int rows, int cols, int live,
                nfn_stream_t stream);

// ---- gated recurrence without a matrix in its loop (gru_rows.cu) ------------------------------------------------------------------------------------------
// Per channel, with the fp32 state s of the sequence: z = sigmoid(a), c = b + 1/2 (b >= 0) or sigmoid(b), s <- (1 - z) s + z c, out = s * silu(g).
// in: rows [a | b | g] of `width` channels each (a multiple of 16), biases added; state [slots][width]; a sequence at position 0 starts from zero. Entries
// of at most 16 rows go token after token (n_short of them, first in seqs), longer ones in segments that a scan joins.
typedef struct {
  int f32, width;
  const void* in; int ld_in;
  float* state;
  void* out; int ld_out;
  const nfn_seq_rows* seqs; int n_seqs, n_short;
} nfn_gru_args;
int nfn_gru_rows(const nfn_gru_args* args, nfn_stream_t stream);

// ---- mixture of experts for the rows of a step (moe.cu, moe_rows.cu) ----------------------------------------------------------
// item i = token i / top, choice i % top. Gated experts take the routing weight at their INPUT: mid = act(w G h) * (w U h); with weigh_output, and plain
// ones (w_gate_up [E][ff][width], mid = act(U h)), they leave it to whoever sums the items.
// nfn_route_rule: how experts are chosen and weighted. s = sigmoid(logits). The choice goes by s + correction (bf16, NULL: by s). groups > 0: group g is
// experts [g E / groups, (g + 1) E / groups); the keep_groups whose two best members add up to most stay open, the rest are out of the choice.
// Weights: s, with normalise / (sum of the chosen ones + 1e-20), times scale. Ties: the lower index. softmax: the choice goes by the logits and the weights
// are the softmax over the chosen ones alone, times scale (no correction, no groups).
typedef struct { const void* correction; int groups, keep_groups, normalise; float scale; int softmax; } nfn_route_rule;
// logits[r][e] = h[r] . w[e] for a handful of rows (bf16, fp32 sums): a CTA per expert and eight rows. width: a multiple of 16.
int nfn_router_rows(const void* h, int ld_h, const void* w, int rows, int experts, int width, float* logits, int ld_logits, nfn_stream_t stream);
int nfn_moe_choose(const float* logits, int ld, int T, int E, int k, const nfn_route_rule* rule, int* idx, float* weight, int* counts, nfn_stream_t stream);
int nfn_moe_route(const float* logits, int ld, int T, int E, int k, int score_fn, int norm_topk, float route_scale, int* topk_idx, float* topk_w,
                  int* counts, nfn_stream_t stream);
int nfn_moe_plan(const int* counts, int E, int max_tiles, int* offsets, int* cursor, int* tile_expert, int* plan, nfn_stream_t stream);
// nfn_moe_permute that also leaves each sorted row's routing weight in row_w.
int nfn_moe_permute_weighted(const void* x, int ldx, int T, int k, int d, const int* topk_idx, const float* topk_w, const int* offsets, int* cursor,
                             int capacity_rows, void* xs, int* row_of, float* row_w, nfn_stream_t stream);
// mid[r] = act(w G) * (w U) over the first plan[1] rows of gate_up [rows][2 * ff] (bf16), w = row_w[r] (NULL: 1); clamp as in nfn_ff_rows.
int nfn_moe_act_rows(const void* gate_up, const float* row_w, const int* plan, int capacity_rows, int ff, int act, const nfn_gate_clamp* clamp, void* mid,
                     nfn_stream_t stream);
// Few rows: routing and a list of items per expert in one launch (order: items by expert; offsets: experts + 1; active: experts with items,
// active[experts] their number), then the products of the chosen experts only, item by item. w_gate_up [E][2 ff][width], w_down [E][width][ff].
typedef struct {
  int f32, rows, width, ff, experts, top, act;
  const float* logits; int ld_logits;
  const void* h; int ld_h;
  const void* w_gate_up; const void* w_down;
  int* idx; float* weight; int* order; int* offsets; int* active;
  void* mid;                              // [rows * top][ff]
  void* y; int ld_y;                      // [rows * top][ld_y]
  int plain;
  nfn_route_rule rule;                    // scale 0 counts as 1
  // shared_ff > 0: the second product of an expert that every row has, y_shared [rows][ld_y] = w_shared_down shared_mid [rows][shared_ff], beside the others
  int shared_ff; const void* shared_mid; const void* w_shared_down; void* y_shared;
  int weigh_output;
  nfn_gate_clamp clamp;                   // of NFN_ACT_CLAMPED
} nfn_moe_rows_args;
int nfn_moe_rows(const nfn_moe_rows_args* args, nfn_stream_t stream);

#ifdef __cplusplus
}
#endif
