// Layer-list engine (see nfn_engine.h): a decoder described layer by layer, served from paged caches in steps that run any mix of
// prompt portions and single tokens as one batch.
//
// Cache manager. Every layer that owns keys and values has page pools (keys [page][kv_heads][64][dim], values transposed
// [page][kv_heads][vdim][64]); layers that read an earlier layer's cache have none. Owner layers whose readers look equally far
// back form a group with one free list and one page table per slot, so a page number means the same tokens in all of them. When
// all readers of a group have windows, pages behind the widest one go back to the free list as the sequence moves on. The short
// convolutions keep taps - 1 projected rows per slot and layer in two halves: a step reads one half and writes the other, so no
// launch reads what it overwrites.
//
// Layers whose keys are limited to chunks of positions give pages back when a chunk ends. Latent layers cache one row per token, [latent | rotated key
// part], for all heads; single tokens and short portions attend to the latents themselves, long portions to keys and values formed from the
// visible latents for the pass.
//
// Recurrent layers have no pages: a slot keeps one fp32 state per head, read and written in place (and, for the token shift, the previous input in two
// halves like the convolutions' history; convolutions on the sublayers' inputs keep theirs the same way, in every layer). Layers of a loop share tensors and have caches and states of their own.
//
// A step lays its rows out short entries first (single tokens and portions below kTileMin rows: one query row at a time), then
// the long ones (tcgen05 tiles). Per layer it launches: input projection (q | k | v | gates | feed-forward in one product), the
// row mix (convolution, temperature, cache append, feed-forward gate), attention with the output gate, one output product that
// adds mixer and feed-forward to the 32-bit residual stream, and the token input's two products with their norm, which also
// produces the next layer's normalised rows. `chained` models run mixer and feed-forward as two sublayers with a stream pass after each
// (chained_pass; post_pass where outputs are normed). Steps of single tokens run with a padded row count and are replayed as CUDA graphs.
#include <cmath>
#include <cstring>
#include <memory>

#include "engine_core.h"

using nfn_eng::efail;

namespace {

constexpr int kPage = NFN_KV_PAGE, kTileMin = 16, kMixRows = 16;
constexpr int kFewRows = 32;                        // up to here several products of a layer run as one weight-streaming launch
constexpr float kUnitEps = 1e-6f;                   // of the delta rule's unit vectors

int up(int v, int m) { return (v + m - 1) / m * m; }

struct Layer {
  nfn_layer_desc d{};
  int dp = 0, vp = 0, ff = 0;                       // padded head sizes and feed-forward width
  int nq = 0, nk = 0, nv = 0, off_g = 0, off_gate = 0, off_up = 0, n_in = 0, n_cat = 0;
  int owner = 0, group = 0;
  int n_conv = 0;                                   // channels that pass the convolution
  int off_b = 0, off_a1 = 0, off_g1 = 0, ra = 0, rg = 0;   // delta: step size, decay and gate projections inside the input product
  int ep = 0, ef = 0;                               // padded number of experts (router rows) and expert width
  void *k_pool = nullptr, *v_pool = nullptr, *state = nullptr;
  long long state_half = 0;
  float* memory = nullptr;                          // delta: [slots][heads][dp][vp]
  float* slopes = nullptr;
  const void *norm1 = nullptr, *w_in = nullptr, *conv = nullptr, *w_out = nullptr, *side_gate = nullptr, *side_proj = nullptr, *side_norm = nullptr;
  const void *norm2 = nullptr, *bias_in = nullptr, *w_a2 = nullptr, *w_g2 = nullptr, *a_log = nullptr, *dt_bias = nullptr, *out_norm = nullptr;
  const void *router = nullptr, *w_gate_up = nullptr, *w_down = nullptr;
  int rp = 0, lr = 0, off_kv = 0;                   // latent: padded rotated part and latent size, latent columns of the input product
  int shp = 0;                                      // padded width of the shared expert
  float* freq = nullptr;                            // rotation: rot_dims / 2 frequencies in two parts
  const void *q_norm = nullptr, *k_norm = nullptr, *c_norm = nullptr, *w_ukv = nullptr, *w_uk_t = nullptr, *w_uv = nullptr;
  const void *mu = nullptr, *w1 = nullptr, *w2 = nullptr, *w0 = nullptr, *u = nullptr;
  const void *w_shared_up = nullptr, *w_shared_down = nullptr, *correction = nullptr;
  float* prev = nullptr;                            // token shift: [2][slots][wp]
  struct { const void *norm_b = nullptr, *conv = nullptr; void* history = nullptr; } sub[2];   // sandwich: mixer, feed-forward; [2][slots][taps - 1][wp]
  const void *sinks = nullptr, *bias_gate_up = nullptr, *bias_down = nullptr;
  float* powers = nullptr;                          // linear: [heads][NFN_LINEAR_CHUNK + 1]
  std::vector<double> decay;
  bool paged() const { return d.mixer == NFN_MIXER_ATTENTION || d.mixer == NFN_MIXER_LATENT; }
  bool latent() const { return d.mixer == NFN_MIXER_LATENT; }
  int key_row() const { return latent() ? lr + rp : d.kv_heads * dp; }       // values of one token's key and value rows in the pages
  int value_row() const { return latent() ? 0 : d.kv_heads * vp; }
  long long memory_floats() const { return d.mixer == NFN_MIXER_GRU ? vp : d.mixer == NFN_MIXER_DELTA || d.mixer == NFN_MIXER_WKV || d.mixer == NFN_MIXER_LINEAR ? (long long)d.heads * dp * vp : 0; }
  nfn_gate_clamp clamp() const { return nfn_gate_clamp{d.ff_limit, d.ff_slope, 1.f}; }
  bool has_ff() const { return d.experts > 0 || d.ff > 0; }
  int look() const { return d.chunk > 0 ? d.chunk : d.window; }              // most positions a query sees, 0: all
  struct { const void *in = nullptr, *out = nullptr, *mix = nullptr; } hc[2];   // streams: mixer, feed-forward
  int tile_rows = 0;                                // query rows per tcgen05 tile, 0: one row at a time
};

struct Group {
  bool all = false;                                 // a reader sees everything: everything stays
  int window = 0;                                   // widest reader with a window
  std::vector<int> chunks;                          // chunk sizes of the readers that have them
  int keep = 0;                                     // first pages that stay whatever the window
  int look() const {                                // most positions a reader sees, 0: all
    int n = window;
    for (int k : chunks) n = std::max(n, k);
    return all ? 0 : n;
  }
  int oldest(int next) const {                      // first position a query at `next` or later can see
    int p = window > 0 ? std::max(0, next - window + 1) : next;
    for (int k : chunks) p = std::min(p, next / k * k);
    return all ? 0 : p;
  }
  bool like(const Group& o) const { return all == o.all && window == o.window && chunks == o.chunks && keep == o.keep; }
  int pages = 0;
  bool held(int slot, int p) const { return p < keep || p >= first[slot]; }   // of pages below next[slot]
  std::vector<int> free_pages;
  int* d_table = nullptr;                           // [slots][max_pages]
  int* h_table = nullptr;                           // pinned mirror
  std::vector<int> first, next;                     // per slot: pages [first, next) of the sequence are held
};

struct layered_engine final : nfn_engine {
  nfn_layered_config c{};
  std::vector<Layer> layers;
  std::vector<Group> groups;
  std::vector<int> tile_kinds;                      // distinct tile heights
  int es = 2;                                       // bytes per activation
  int wp = 0, vp = 0, sp = 0, max_pages = 0, rows_max = 0, logit_rows = 0, n_in_max = 0, nq_max = 0, cat_max = 0;
  float* x = nullptr;
  void *xb = nullptr, *h = nullptr, *hc = nullptr, *in = nullptr, *q = nullptr, *cat = nullptr, *s_act = nullptr, *y = nullptr, *hw = nullptr;
  float *s_gate = nullptr, *logits = nullptr, *saved = nullptr;
  float *decay = nullptr, *d_o = nullptr;           // delta: projected decays, read-outs
  void *d_gate = nullptr, *delta_ws = nullptr;
  long long delta_ws_bytes = 0;
  struct { float *logits = nullptr, *weight = nullptr, *row_w = nullptr; int *idx = nullptr, *order = nullptr, *offsets = nullptr, *active = nullptr, *counts = nullptr,
           *cursor = nullptr, *tile_expert = nullptr, *plan = nullptr, *row_of = nullptr; void *xs = nullptr, *gate_up = nullptr, *mid = nullptr, *y = nullptr; } ex;
  void *q_lat = nullptr, *o_lat = nullptr, *lat_rows = nullptr, *lat_x = nullptr;   // latent: absorbed queries and outputs of short rows; gathered latents, expansion
  int lat_cap = 0;                                  // rows of the last two
  void *shift = nullptr, *low_act = nullptr, *shared_mid = nullptr, *y_shared = nullptr;
  const void* hx = nullptr;                         // what the sublayer at hand reads: h, or hc behind the convolution on its input
  int* row_count = nullptr;                         // linear: one counter per row
  void* linear_ws = nullptr;
  long long linear_ws_bytes = 0;
  float* low = nullptr;
  void* wkv_ws = nullptr;
  long long wkv_ws_bytes = 0;
  nfn_stream_args pend{};                           // chained: the last sublayer's update, applied on the way to the head
  void *att_ws = nullptr, *gemm_ws = nullptr;
  long long att_ws_bytes = 0, gemm_ws_bytes = 0;
  std::vector<uint8_t> parity;                      // per slot: the half that holds its convolution history
  std::vector<int> logit_at;                        // per slot: row of `logits`, -1: none, -2: `saved`
  // per-step block, one copy to the device: offsets in bytes
  struct { long long tok, slot, pos, want, params, offset, mix, att, seq, spans, base, out, total; } io{};
  unsigned char *h_io = nullptr, *d_io = nullptr;
  std::map<int, cudaGraphExec_t> graphs;            // by padded row count
  std::map<int, long long> graph_launches;
  std::map<int, int> graph_calls;

  ~layered_engine() override;
  int build();
  int finalize() override;
  int release(int slot) override;
  int prefill(int slot, const int32_t* tokens, int n, const nfn_sampling* s, int32_t* next_token) override;
  int decode(const int32_t* tokens_in, const uint8_t* active, const nfn_sampling* s, const nfn_sampling* per_slot, int32_t* next_tokens) override;
  int step(const nfn_step_entry* entries, int n_entries, const int32_t* tokens, const int32_t* want_rows, int n_want, const nfn_sampling* want_sampling,
           int32_t* want_tokens, float* want_logits) override;
  int last_logits(int slot, float* out_vocab) override;
  int truncate(int slot, int n) override;
  int fork(int src_slot, int dst_slot, int n) override;
  long long free_tokens() const override;

  int add(void** p, long long n) {
    if (alloc(p, n)) return -1;
    owned.push_back(*p);
    return 0;
  }
  std::vector<void*> owned;
  template <typename P>
  P* dev(long long off) const { return reinterpret_cast<P*>(d_io + off); }
  template <typename P>
  P* host(long long off) const { return reinterpret_cast<P*>(h_io + off); }

  int reserve(int slot, int upto);                  // pages for positions < upto
  void trim(int slot);                              // pages no later query of this slot can see
  int lin(const void* a, int lda, const void* w, int rows, int n, int k, void* out, int ldo, int kind, const void* bias = nullptr, int act = NFN_ACT_NONE);
  // the rows of one pass: short entries first, then the long ones
  struct Batch { int rows = 0, short_rows = 0, n_mix = 0, n_seq = 0, n_short_seq = 0, longest = 0; bool single = false; std::vector<int> att_off, att_n;
                 // latent layers: the long entries whose latents one expansion holds, by layer
                 struct Round { int span0, n_spans, max_pages, rows, tile0, n_tiles; };
                 std::vector<std::vector<Round>> expand; };
  int mix_rows(const Layer& L, const Batch& b, void* ff_out);
  int attention(const Layer& L, const Batch& b);
  int delta(const Layer& L, const Batch& b);
  int rotated_attention(const Layer& L, const Batch& b);
  int latent_attention(const Layer& L, const Batch& b);
  int wkv(const Layer& L, const Batch& b);
  int linear(const Layer& L, const Batch& b);
  int gru(const Layer& L, const Batch& b);
  int mixer(const Layer& L, const Batch& b);
  int dense_ff(const Layer& L, int rows);
  bool rotated(const Layer& L) const { return L.d.mixer == NFN_MIXER_ATTENTION && (L.d.rot_dims > 0 || L.d.qk_norm || L.d.key_values); }
  void attention_args(const Layer& L, nfn_paged_attention_args* a);
  int post_pass(const Batch& b);
  int enter(nfn_stream_args* s, const Layer& L, int which, const Batch& b);
  // wkv: single tokens in one launch after the products, few rows through one launch for the four projections
  bool wkv_step(const Layer& L, const Batch& b) const { return b.single && nfn_wkv_step_fits(b.rows, L.dp); }
  bool grouped(const Layer& L, int rows) const { return c.dtype == 0 && L.d.experts <= 256 && L.d.top <= 32 && (long long)rows * L.d.top > 8LL * L.d.experts; }
  bool linear_step(const Layer& L, const Batch& b) const { return b.single && nfn_linear_step_fits(b.rows, L.dp, L.vp); }
  // single tokens of delta layers: convolution, rule, norm and gate in one launch
  bool one_step(const Layer& L, const Batch& b) const { return b.single && L.d.mixer == NFN_MIXER_DELTA && nfn_delta_step_fits(b.rows, L.d.heads, L.dp, L.vp); }
  int experts(const Layer& L, int rows, nfn_stream_args* sp);
  int pass(const Batch& b);
  int chained_pass(const Batch& b);
  int head(const int* src_rows, int rows);
  int sample(int rows);
  int run(const std::vector<nfn_step_entry>& part, const int32_t* const* part_tokens, std::vector<int>& row_of, bool single);
};

enum { kOutAct = 0, kOutF32 = 1, kOutResidual = 2 };

std::string lname(int l, const char* s) { return "layers." + std::to_string(l) + "." + s; }

}  // namespace

layered_engine::~layered_engine() {
  for (auto& g : graphs) cudaGraphExecDestroy(g.second);
  for (void* p : owned) cudaFree(p);
  for (Group& g : groups)
    if (g.h_table) cudaFreeHost(g.h_table);
  if (h_io) cudaFreeHost(h_io);
}

// sizes, tensor names and groups; no device memory yet
int layered_engine::build() {
  es = c.dtype == 1 ? 4 : 2;
  wp = up(c.width, 16);
  vp = up(c.vocab, 16);
  sp = c.side_dim > 0 ? up(c.side_dim, 16) : 0;
  max_pages = (c.max_seq + kPage - 1) / kPage;
  auto want = [&](const std::string& n, long long numel) { expected.emplace_back(n, numel); };
  want("embed", (long long)vp * wp);
  if (sp) want("side_embed", (long long)c.vocab * c.n_layer * sp);
  if (c.untied_head) want("head", (long long)vp * wp);
  for (int l = 0; l < c.n_layer; ++l) {
    Layer& L = layers[l];
    const nfn_layer_desc& d = L.d;
    const std::string bad = "engine: layer " + std::to_string(l);
    if (d.weights_of >= 0) {
      if (d.weights_of >= l || layers[d.weights_of].d.weights_of >= 0) return efail(bad + " must take its tensors from an earlier layer that has its own");
      nfn_layer_desc a = d, o = layers[d.weights_of].d;
      a.weights_of = o.weights_of = -1;
      a.decay = o.decay = nullptr;
      if (L.decay != layers[d.weights_of].decay) return efail(bad + " and the layer whose tensors it uses differ");
      if (std::memcmp(&a, &o, sizeof a)) return efail(bad + " and the layer whose tensors it uses differ");
    }
    if (c.chained ? ((d.out_gate && d.mixer != NFN_MIXER_LATENT) || (d.ff > 0 && d.experts > 0)) : (d.mixer != NFN_MIXER_ATTENTION || d.experts > 0 || d.qkv_bias || d.rot_dims > 0 || d.qk_norm || d.key_values))
      return efail(bad + (c.chained ? ": sublayers one after another have one feed-forward and no output gate"
                                    : ": recurrent and latent mixers, rotation, experts and biases need sublayers one after another"));
    if (d.mixer == NFN_MIXER_WKV && !c.post_norm) return efail(bad + ": the token shift reads the residual itself (post_norm)");
    if ((rotated(L) || d.mixer == NFN_MIXER_LATENT) && (d.conv_taps > 0 || d.q_temp_every > 0 || d.qkv_bias))
      return efail(bad + ": rotated and latent attention have no convolutions, query temperature or biases");
    if (!d.expert_plain && (d.shared_ff > 0 || d.route_correction || d.route_groups > 0 || d.route_normalise)) return efail(bad + ": gated experts have plain sigmoid routing and no shared expert");
    if ((d.route_softmax || d.ff_act == NFN_ACT_CLAMPED) && d.experts > 0 && (d.expert_plain || !d.expert_weigh_out)) return efail(bad + ": softmax routing and clamped gates go with gated experts weighted at their output");
    if ((d.mixer == NFN_MIXER_LINEAR || d.mixer == NFN_MIXER_GRU) && (d.conv_taps > 0 || (d.qkv_bias && d.mixer == NFN_MIXER_LINEAR))) return efail(bad + ": these recurrences have no convolution or such biases of their own");
    L.ep = d.experts > 0 ? up(d.experts, 16) : 0;
    L.ef = d.experts > 0 ? up(d.expert_ff, 16) : 0;
    L.dp = up(d.dim, 16);
    L.vp = up(d.vdim, 16);
    L.ff = d.ff > 0 ? up(d.ff, 16) : 0;
    L.owner = l;
    if (d.kv_from >= 0) {
      const Layer& o = layers[d.kv_from];
      if (d.kv_from >= l || o.d.kv_from >= 0) return efail("engine: layer " + std::to_string(l) + " must read an earlier layer with keys and values of its own");
      if (o.d.mixer != d.mixer || (d.mixer == NFN_MIXER_LATENT ? (o.d.kv_rank != d.kv_rank || o.d.rot_dim != d.rot_dim || o.d.rot_dims != d.rot_dims || o.d.rot_base != d.rot_base)
                                                               : (o.d.kv_heads != d.kv_heads || o.d.dim != d.dim || o.d.vdim != d.vdim)))
        return efail("engine: layer " + std::to_string(l) + " and the layer whose cache it reads have different caches");
      L.owner = d.kv_from;
    }
    const bool own = L.owner == l;
    if (d.mixer == NFN_MIXER_DELTA) {   // q, k, v leave the convolution as one row; no pages
      L.nq = 2 * d.kv_heads * L.dp + d.heads * L.vp;
      L.ra = up(d.rank_decay, 16);
      L.rg = up(d.rank_gate, 16);
      L.off_b = L.nq;
      L.off_a1 = L.off_b + up(d.heads, 16);
      L.off_g1 = L.off_a1 + L.ra;
      L.off_gate = L.off_up = L.n_in = L.off_g1 + L.rg;
    } else if (d.mixer == NFN_MIXER_LATENT) {
      L.lr = up(d.kv_rank, 16);
      L.rp = up(d.rot_dim, 16);
      L.nq = d.heads * (L.dp + L.rp);
      L.off_kv = L.nq;
      L.off_g = L.nq + (own ? L.lr + L.rp : 0);
      L.n_in = L.off_g + (d.out_gate ? d.heads * L.vp : 0);
    } else if (d.mixer == NFN_MIXER_WKV) {
      L.ra = up(d.rank_decay, 16);
      L.nq = d.heads * L.dp;                       // each of r, k, v, g
      L.n_in = 4 * L.nq;
    } else if (d.mixer == NFN_MIXER_LINEAR) {        // [q | k | v | gate]
      L.nq = 2 * d.heads * L.dp + d.heads * L.vp;
      L.off_g = L.nq;
      L.n_in = L.nq + d.heads * L.vp;
    } else if (d.mixer == NFN_MIXER_GRU) {           // [share | candidate | gate]
      L.nq = 3 * L.vp;
      L.n_in = L.nq;
    } else {
      L.nq = d.heads * L.dp;
      L.nk = own ? d.kv_heads * L.dp : 0;
      L.nv = own && !d.key_values ? d.kv_heads * L.vp : 0;
      L.off_g = L.nq + L.nk + L.nv;
      L.off_gate = L.off_g + (d.out_gate ? d.heads * L.vp : 0);
      L.off_up = L.off_gate + (c.chained ? 0 : L.ff);
      L.n_in = L.off_up + (c.chained ? 0 : L.ff);
    }
    L.shp = d.shared_ff > 0 ? up(d.shared_ff, 16) : 0;
    L.n_conv = L.nq + L.nk + L.nv;
    L.n_cat = d.heads * L.vp + (c.chained ? 0 : L.ff);
    n_in_max = std::max(n_in_max, std::max(L.n_in, c.chained ? 2 * L.ff : 0));
    if (!rotated(L) && (d.mixer == NFN_MIXER_ATTENTION || d.mixer == NFN_MIXER_DELTA)) nq_max = std::max(nq_max, L.nq);      // others keep their queries in place
    cat_max = std::max(cat_max, std::max(L.n_cat, L.ff));
    if (d.weights_of < 0) {
      const long long nw = c.scalar_norms ? 1 : wp;
      want(lname(l, "norm1"), nw);
      for (int q = 0; c.sandwich && q < (L.has_ff() ? 2 : 1); ++q) {
        want(lname(l, q ? "norm2_b" : "norm1_b"), nw);
        if (c.input_taps > 0) want(lname(l, q ? "in_conv2" : "in_conv1"), (long long)c.input_taps * wp);
      }
      if (d.sink == 2) want(lname(l, "sink"), d.heads);
      if (d.mixer == NFN_MIXER_LINEAR) want(lname(l, "out_norm"), (long long)d.heads * L.vp);
      want(lname(l, "w_in"), (long long)L.n_in * wp);
      if (d.qk_norm) {
        want(lname(l, "q_norm"), L.dp);
        if (own) want(lname(l, "k_norm"), L.dp);
      }
      if (d.mixer == NFN_MIXER_LATENT) {
        if (own) want(lname(l, "c_norm"), L.lr);
        want(lname(l, "w_ukv"), (long long)d.heads * (L.dp + L.vp) * L.lr);
        want(lname(l, "w_uk_t"), (long long)d.heads * L.lr * L.dp);
      }
      if (d.mixer == NFN_MIXER_WKV) {
        want(lname(l, "mu"), 5LL * wp);
        want(lname(l, "w1"), (long long)L.ra * wp);
        want(lname(l, "w2"), 2LL * L.nq * L.ra);
        want(lname(l, "w0"), L.nq);
        want(lname(l, "u"), L.nq);
        want(lname(l, "out_norm"), L.nq);
      }
      if (c.chained && d.ff > 0) {
        want(lname(l, "norm2"), nw);
        want(lname(l, "w_gate_up"), 2LL * L.ff * wp);
        want(lname(l, "w_down"), (long long)wp * L.ff);
        if (d.ff_bias) {
          want(lname(l, "bias_gate_up"), 2LL * L.ff);
          want(lname(l, "bias_down"), wp);
        }
      }
      if (d.shared_ff > 0) {
        want(lname(l, "w_shared_up"), (long long)L.shp * wp);
        want(lname(l, "w_shared_down"), (long long)wp * L.shp);
      }
      if (d.route_correction) want(lname(l, "correction"), L.ep);
      if (d.conv_taps > 0) want(lname(l, "conv"), (long long)d.conv_taps * L.n_conv);
      want(lname(l, "w_out"), (long long)wp * L.n_cat);
      if (sp) {
        want(lname(l, "side_gate"), (long long)sp * wp);
        want(lname(l, "side_proj"), (long long)wp * sp);
        want(lname(l, "side_norm"), wp);
      }
      if (d.qkv_bias) want(lname(l, "bias_in"), L.n_in);
      if (d.mixer == NFN_MIXER_DELTA) {
        want(lname(l, "w_a2"), (long long)d.heads * L.dp * L.ra);
        want(lname(l, "w_g2"), (long long)d.heads * L.vp * L.rg);
        want(lname(l, "a_log"), d.heads);
        want(lname(l, "dt_bias"), (long long)d.heads * L.dp);
        want(lname(l, "out_norm"), L.vp);
      }
      if (d.experts > 0) {
        want(lname(l, "norm2"), nw);
        want(lname(l, "router"), (long long)L.ep * wp);
        want(lname(l, "w_gate_up"), (long long)d.experts * (d.expert_plain ? 1 : 2) * L.ef * wp);
        want(lname(l, "w_down"), (long long)d.experts * wp * L.ef);
      }
      for (int q = 0; q < (c.streams > 0 ? (d.experts > 0 || d.ff > 0 ? 2 : 1) : 0); ++q) {
        const std::string hc = q ? "hc2_" : "hc1_";
        want(lname(l, (hc + "in").c_str()), c.streams);
        want(lname(l, (hc + "out").c_str()), c.streams);
        want(lname(l, (hc + "mix").c_str()), (long long)c.streams * c.streams);
      }
    }
    if (!L.paged()) continue;
    L.tile_rows = L.latent() ? nfn_latent_tile_rows(c.dtype, L.dp, L.rp, L.vp) : nfn_paged_tile_rows(c.dtype, d.heads, d.kv_heads, L.dp, L.vp);
    if (L.tile_rows > 0 && std::find(tile_kinds.begin(), tile_kinds.end(), L.tile_rows) == tile_kinds.end()) tile_kinds.push_back(L.tile_rows);
  }
  want("final_norm", c.scalar_norms ? 1 : wp);
  // how far back the readers of each owner look, and one group per distinct answer
  for (int l = 0; l < c.n_layer; ++l) {
    if (layers[l].owner != l || !layers[l].paged()) continue;
    Group n;
    for (const Layer& r : layers)
      if (r.owner == l) {
        n.all |= r.look() <= 0;
        if (r.d.chunk > 0) n.chunks.push_back(r.d.chunk);
        else n.window = std::max(n.window, r.d.window);
        n.keep = std::max(n.keep, (r.d.keep_first + kPage - 1) / kPage);
      }
    std::sort(n.chunks.begin(), n.chunks.end());
    n.chunks.erase(std::unique(n.chunks.begin(), n.chunks.end()), n.chunks.end());
    if (n.all) {
      n.window = n.keep = 0;
      n.chunks.clear();
    }
    int g = 0;
    while (g < (int)groups.size() && !groups[g].like(n)) ++g;
    if (g == (int)groups.size()) groups.push_back(n);
    for (Layer& r : layers)
      if (r.owner == l) r.group = g;
  }
  if (groups.empty()) {   // no layer has pages: the pool still counts tokens
    groups.emplace_back();
    groups.back().all = true;
  }
  len.assign(c.max_batch, 0);
  parity.assign(c.max_batch, 0);
  logit_at.assign(c.max_batch, -1);
  return 0;
}

extern "C" nfn_engine* nfn_engine_create_layered(const nfn_layered_config* cfg, const nfn_layer_desc* layers, int device) {
  if (!cfg || !layers) {
    efail("engine_create: null config");
    return nullptr;
  }
  const nfn_layered_config& c = *cfg;
  if (c.n_layer <= 0 || c.width <= 0 || c.vocab <= 0 || c.side_dim < 0 || (c.dtype != 0 && c.dtype != 1) || c.max_seq <= 0 || c.max_batch <= 0 ||
      c.kv_tokens < 0 || c.max_step_rows <= 0 || !(c.norm_eps >= 0.f) || c.streams < 0 || c.streams > NFN_MAX_STREAMS || (c.streams > 0 && !c.chained) ||
      (c.chained && c.side_dim > 0) || !(c.logit_softcap >= 0.f) || (!c.chained && c.norm_offset != 0.f) ||
      (c.post_norm && (!c.chained || c.streams > 0 || c.norm_offset != 0.f)) || (c.sandwich && (!c.chained || c.streams > 0 || c.norm_offset != 0.f || c.post_norm)) ||
      (!c.sandwich && (c.scalar_norms || c.input_taps)) || c.input_taps < 0) {
    efail("engine_create: invalid geometry");
    return nullptr;
  }
  auto e = std::make_unique<layered_engine>();
  e->c = c;
  if (e->c.kv_tokens == 0) e->c.kv_tokens = (int)std::min<long long>((long long)c.max_batch * up(c.max_seq, kPage), 0x7fffffc0LL);
  e->layers.resize(c.n_layer);
  for (int l = 0; l < c.n_layer; ++l) {
    const nfn_layer_desc& d = layers[l];
    if (d.heads <= 0 || d.kv_heads <= 0 || d.heads % d.kv_heads || d.dim <= 0 || d.vdim <= 0 || d.conv_taps < 0 || d.ff < 0 || d.window < 0 ||
        d.q_temp_every < 0 || d.keep_first < 0 || d.softcap < 0.f || d.experts < 0 || (d.experts > 0 && (d.top < 1 || d.top > d.experts || d.expert_ff < 1)) ||
        d.mixer < NFN_MIXER_ATTENTION || d.mixer > NFN_MIXER_GRU || d.chunk < 0 || (d.chunk > 0 && (d.window > 0 || d.keep_first > 0)) || d.rot_dims < 0 ||
        (d.rot_dims & 1) || (d.rot_dims > 0 && !(d.rot_base > 0.0)) || (d.mixer == NFN_MIXER_ATTENTION && (d.rot_dims > d.dim || (d.key_values && d.vdim != d.dim) || ((d.rot_dims > 0 || d.qk_norm) && d.dim > 512))) ||
        (d.mixer == NFN_MIXER_LATENT && (d.kv_rank <= 0 || d.rot_dim <= 0 || d.rot_dims != d.rot_dim || d.rot_dim > 512 || d.kv_heads != 1 || d.keep_first > 0 || d.qk_norm || d.softcap > 0.f || d.alibi != 0.f)) ||
        d.sink < 0 || d.sink > 2 || (d.sink && d.mixer != NFN_MIXER_ATTENTION && d.mixer != NFN_MIXER_LATENT) || (d.mixer == NFN_MIXER_LINEAR && (!d.decay || d.kv_heads != d.heads || d.dim > 512)) ||
        (d.mixer == NFN_MIXER_GRU && (d.heads != 1 || d.dim != 1)) || (d.ff_act == NFN_ACT_CLAMPED && !(d.ff_limit > 0.f)) ||
        (d.mixer == NFN_MIXER_WKV && (d.rank_decay < 1 || d.dim > 512 || d.vdim != d.dim || d.kv_heads != d.heads)) || d.shared_ff < 0 || (d.shared_ff > 0 && d.experts <= 0) ||
        (d.route_groups > 0 && (d.experts % d.route_groups || d.route_keep < 1 || d.route_keep > d.route_groups || d.route_keep * (d.experts / d.route_groups) < d.top)) || d.route_groups < 0 ||
        (d.mixer == NFN_MIXER_DELTA && (d.conv_taps < 1 || d.rank_decay < 1 || d.rank_gate < 1 || d.dim > 512)) || (d.ff_act != NFN_ACT_RELU && d.ff_act != NFN_ACT_SILU && d.ff_act != NFN_ACT_GELU_TANH && d.ff_act != NFN_ACT_RELU2 && d.ff_act != NFN_ACT_CLAMPED)) {
      efail("engine_create: invalid sizes in layer " + std::to_string(l));
      return nullptr;
    }
    e->layers[l].d = d;
    if (d.mixer == NFN_MIXER_LINEAR) e->layers[l].decay.assign(d.decay, d.decay + d.heads);
    e->layers[l].d.decay = nullptr;
  }
  e->device = device;
  if (cudaSetDevice(device) != cudaSuccess || cudaStreamCreateWithFlags(&e->stream, cudaStreamNonBlocking) != cudaSuccess) {
    efail("engine_create: cannot select the device or create a stream");
    return nullptr;
  }
  if (e->build()) return nullptr;
  return e.release();
}

int layered_engine::finalize() {
  CU(cudaSetDevice(device));
  if (missing_tensor()) return -1;
  rows_max = up(std::max(std::min(c.max_step_rows, std::max(c.max_seq, c.max_batch)), c.max_batch), 16);
  logit_rows = std::max(c.max_batch, 64);
  const long long R = rows_max, S = c.max_batch;
  auto zero = [&](void** p, long long n) -> int {
    if (add(p, n)) return -1;
    CU(cudaMemset(*p, 0, (size_t)n));
    return 0;
  };
  if (zero((void**)&x, R * wp * 4 * std::max(c.streams, 1)) || zero(&h, R * wp * es) || zero(&in, R * n_in_max * es) || (nq_max > 0 && zero(&q, R * nq_max * es)) || zero(&cat, R * cat_max * es) ||
      zero(&hw, (long long)logit_rows * wp * es) || zero((void**)&logits, (long long)logit_rows * vp * 4) || zero((void**)&saved, S * vp * 4))
    return -1;
  if (c.dtype == 0 && zero(&xb, R * wp * 2)) return -1;
  if (sp && (zero((void**)&s_gate, R * sp * 4) || zero(&s_act, R * sp * es))) return -1;
  if ((sp || c.chained) && zero(&y, R * wp * es)) return -1;
  if (c.input_taps > 0 && zero(&hc, R * wp * es)) return -1;
  // scratch of the delta mixers and of the experts: the largest any layer asks for
  long long n_q_lat = 0, n_o_lat = 0, n_lat = 0, n_lat_x = 0, n_low = 0, n_shift = 0, n_shared = 0;
  // rows that attend to latents themselves: short entries, or all of them where the sizes have no tiles
  const long long r_short = std::min<long long>(R, S * (kTileMin - 1));
  long long n_dec = 0, n_do = 0, n_lin = 0, e_log = 0, e_max = 0, e_items = 0, e_sorted = 0, e_gu = 0, e_mid = 0, e_rows = 0;
  for (const Layer& L : layers) {
    const nfn_layer_desc& d = L.d;
    if (d.mixer == NFN_MIXER_DELTA) {
      n_dec = std::max(n_dec, R * d.heads * L.dp);
      n_do = std::max(n_do, R * d.heads * L.vp);
      if (c.dtype == 0) delta_ws_bytes = std::max(delta_ws_bytes, nfn_delta_chunk_workspace_bytes(d.heads, L.dp, L.vp, c.max_batch));
    }
    if (L.latent()) {
      const long long rows = L.tile_rows > 0 ? std::max<long long>(r_short, c.max_batch) : R;
      n_q_lat = std::max(n_q_lat, rows * d.heads * (L.lr + L.rp));
      n_o_lat = std::max(n_o_lat, rows * d.heads * L.lr);
      if (L.tile_rows > 0) {   // at least the longest portion with its window; several portions per round where they fit
        const long long look = L.look() > 0 ? std::min(L.look(), c.max_seq) : c.max_seq;
        lat_cap = std::max(lat_cap, up((int)std::min<long long>(look + R, up(c.max_seq, kPage)) + 2 * kPage, kPage));
        n_lat = std::max<long long>(n_lat, L.lr);
        n_lat_x = std::max<long long>(n_lat_x, (long long)d.heads * (L.dp + L.vp));
      }
    }
    if (d.mixer == NFN_MIXER_WKV) {
      n_dec = std::max(n_dec, R * L.nq);
      n_do = std::max(n_do, R * L.nq);
      n_low = std::max(n_low, R * L.ra);
      n_shift = 5 * R * wp;
      if (c.dtype == 0) wkv_ws_bytes = std::max(wkv_ws_bytes, nfn_wkv_chunk_workspace_bytes(d.heads, L.dp, c.max_batch));
    }
    if (d.mixer == NFN_MIXER_LINEAR) {
      n_lin = std::max(n_lin, R * d.heads * L.vp);
      if (c.dtype == 0) linear_ws_bytes = std::max(linear_ws_bytes, nfn_linear_chunk_workspace_bytes(d.heads, L.dp, L.vp, c.max_batch));
    }
    n_shared = std::max(n_shared, R * L.shp);
    if (d.experts > 0) {
      const bool g = grouped(L, (int)R);
      const long long sorted = g ? (R * d.top + d.experts * 127LL + 127) / 128 * 128 : 0;
      const long long single = std::min(R * d.top, c.dtype == 0 && g ? 8LL * d.experts : R * d.top);   // items of the largest step outside the sorted form
      e_log = std::max(e_log, R * L.ep);
      e_max = std::max<long long>(e_max, d.experts);
      e_items = std::max(e_items, R * d.top);
      e_sorted = std::max(e_sorted, sorted);
      e_gu = std::max(e_gu, sorted * 2 * L.ef);
      e_mid = std::max(e_mid, std::max(sorted, single) * L.ef);
      e_rows = std::max(e_rows, std::max(sorted, single));
    }
  }
  lat_cap = std::max(lat_cap, n_lat > 0 ? rows_max : 0);
  if ((n_q_lat && (zero(&q_lat, n_q_lat * es) || zero(&o_lat, n_o_lat * es))) || (n_lat && (zero(&lat_rows, lat_cap * n_lat * es) || zero(&lat_x, lat_cap * n_lat_x * es)))) return -1;
  if (n_low && (zero((void**)&low, n_low * 4) || zero(&low_act, 2 * n_low * es) || zero(&shift, n_shift * es))) return -1;
  if (n_shared && (zero(&shared_mid, n_shared * es) || zero(&y_shared, R * wp * es))) return -1;
  if (wkv_ws_bytes > 0 && add(&wkv_ws, wkv_ws_bytes)) return -1;
  if (delta_ws_bytes > 0 && add(&delta_ws, delta_ws_bytes)) return -1;
  if (n_dec && (zero((void**)&decay, n_dec * 4) || zero(&d_gate, n_do * es))) return -1;
  if (std::max(n_do, n_lin) > 0 && zero((void**)&d_o, std::max(n_do, n_lin) * 4)) return -1;
  if (n_lin && zero((void**)&row_count, R * 4)) return -1;
  if (linear_ws_bytes > 0 && add(&linear_ws, linear_ws_bytes)) return -1;
  if (e_max && (zero((void**)&ex.logits, e_log * 4) || zero((void**)&ex.weight, e_items * 4) || zero((void**)&ex.idx, e_items * 4) ||
                zero((void**)&ex.order, e_items * 4) || zero((void**)&ex.row_of, e_items * 4) || zero((void**)&ex.offsets, (e_max + 1) * 4) ||
                zero((void**)&ex.active, (e_max + 1) * 4) || zero((void**)&ex.counts, e_max * 4) || zero((void**)&ex.cursor, e_max * 4) ||
                zero((void**)&ex.plan, 16) || zero(&ex.mid, e_mid * es) || zero(&ex.y, e_rows * wp * es)))
    return -1;
  if (e_sorted && (zero((void**)&ex.row_w, e_sorted * 4) || zero((void**)&ex.tile_expert, e_sorted / 128 * 4) || zero(&ex.xs, e_sorted * wp * 2) ||
                   zero(&ex.gate_up, e_gu * 2)))
    return -1;
  for (Group& g : groups) {
    g.pages = (c.kv_tokens + kPage - 1) / kPage;
    if (g.look() > 0) g.pages = (int)std::min<long long>(g.pages, S * ((g.look() + R) / kPage + 2 + g.keep));
    for (int p = g.pages - 1; p >= 0; --p) g.free_pages.push_back(p);
    g.first.assign(S, 0);
    g.next.assign(S, 0);
    if (zero((void**)&g.d_table, S * max_pages * 4)) return -1;
    CU(cudaMallocHost((void**)&g.h_table, (size_t)S * max_pages * 4));
    std::memset(g.h_table, 0, (size_t)S * max_pages * 4);
  }
  long long ws = 0;
  for (int l = 0; l < c.n_layer; ++l) {
    Layer& L = layers[l];
    const nfn_layer_desc& d = L.d;
    if (L.memory_floats() > 0) {
      if (zero((void**)&L.memory, S * L.memory_floats() * 4) || (d.mixer == NFN_MIXER_WKV && zero((void**)&L.prev, 2 * S * wp * 4))) return -1;
    } else if (L.owner == l) {
      const long long tokens = (long long)groups[L.group].pages * kPage;
      if (zero(&L.k_pool, tokens * L.key_row() * es) || (L.value_row() > 0 && zero(&L.v_pool, tokens * L.value_row() * es))) return -1;
    } else {
      L.k_pool = layers[L.owner].k_pool;
      L.v_pool = layers[L.owner].v_pool;
    }
    if (d.conv_taps > 1) {
      L.state_half = S * (d.conv_taps - 1) * L.n_conv;
      if (zero(&L.state, 2 * L.state_half * es)) return -1;
    }
    const int wl = d.weights_of >= 0 ? d.weights_of : l;
    if (d.conv_taps > 0) L.conv = W(lname(wl, "conv"));
    for (int q = 0; c.sandwich && q < (L.has_ff() ? 2 : 1); ++q) {
      L.sub[q].norm_b = W(lname(wl, q ? "norm2_b" : "norm1_b"));
      if (c.input_taps <= 0) continue;
      L.sub[q].conv = W(lname(wl, q ? "in_conv2" : "in_conv1"));
      if (c.input_taps > 1 && zero(&L.sub[q].history, 2 * S * (c.input_taps - 1) * wp * es)) return -1;
    }
    if (d.sink == 2) L.sinks = W(lname(wl, "sink"));
    if (d.mixer == NFN_MIXER_LINEAR) {
      L.out_norm = W(lname(wl, "out_norm"));
      std::vector<float> pw((size_t)d.heads * (NFN_LINEAR_CHUNK + 1));
      for (int i = 0; i < d.heads; ++i)
        for (int n = 0; n <= NFN_LINEAR_CHUNK; ++n) pw[(size_t)i * (NFN_LINEAR_CHUNK + 1) + n] = (float)std::pow(L.decay[i], n);
      if (zero((void**)&L.powers, (long long)pw.size() * 4)) return -1;
      CU(cudaMemcpy(L.powers, pw.data(), pw.size() * 4, cudaMemcpyHostToDevice));
    }
    if (d.alibi != 0.f) {
      std::vector<float> sl(d.heads);
      for (int i = 0; i < d.heads; ++i) sl[i] = (float)std::exp2(-(double)d.alibi * (i + 1) / d.heads);
      if (zero((void**)&L.slopes, 4LL * d.heads)) return -1;
      CU(cudaMemcpy(L.slopes, sl.data(), sl.size() * 4, cudaMemcpyHostToDevice));
    }
    if (d.rot_dims > 0) {
      std::vector<float> f(d.rot_dims);
      for (int i = 0; i < d.rot_dims / 2; ++i) {
        const double v = std::pow(d.rot_base, -2.0 * i / d.rot_dims);
        f[2 * i] = (float)v;
        f[2 * i + 1] = (float)(v - (double)f[2 * i]);
      }
      if (zero((void**)&L.freq, 4LL * d.rot_dims)) return -1;
      CU(cudaMemcpy(L.freq, f.data(), f.size() * 4, cudaMemcpyHostToDevice));
    }
    if (d.qk_norm) {
      L.q_norm = W(lname(wl, "q_norm"));
      if (L.owner == l) L.k_norm = W(lname(wl, "k_norm"));
    }
    if (L.latent()) {
      if (L.owner == l) L.c_norm = W(lname(wl, "c_norm"));
      L.w_ukv = W(lname(wl, "w_ukv"));
      L.w_uk_t = W(lname(wl, "w_uk_t"));
      L.w_uv = static_cast<const char*>(L.w_ukv) + 2LL * d.heads * L.dp * L.lr;
    }
    if (d.mixer == NFN_MIXER_WKV) {
      L.mu = W(lname(wl, "mu"));
      L.w1 = W(lname(wl, "w1"));
      L.w2 = W(lname(wl, "w2"));
      L.w0 = W(lname(wl, "w0"));
      L.u = W(lname(wl, "u"));
      L.out_norm = W(lname(wl, "out_norm"));
    }
    if (c.chained && d.ff > 0) {
      L.norm2 = W(lname(wl, "norm2"));
      L.w_gate_up = W(lname(wl, "w_gate_up"));
      L.w_down = W(lname(wl, "w_down"));
      if (d.ff_bias) {
        L.bias_gate_up = W(lname(wl, "bias_gate_up"));
        L.bias_down = W(lname(wl, "bias_down"));
      }
    }
    if (d.shared_ff > 0) {
      L.w_shared_up = W(lname(wl, "w_shared_up"));
      L.w_shared_down = W(lname(wl, "w_shared_down"));
    }
    if (d.route_correction) L.correction = W(lname(wl, "correction"));
    L.norm1 = W(lname(wl, "norm1"));
    L.w_in = W(lname(wl, "w_in"));
    L.w_out = W(lname(wl, "w_out"));
    if (d.qkv_bias) L.bias_in = W(lname(wl, "bias_in"));
    if (d.mixer == NFN_MIXER_DELTA) {
      L.w_a2 = W(lname(wl, "w_a2"));
      L.w_g2 = W(lname(wl, "w_g2"));
      L.a_log = W(lname(wl, "a_log"));
      L.dt_bias = W(lname(wl, "dt_bias"));
      L.out_norm = W(lname(wl, "out_norm"));
    }
    if (d.experts > 0) {
      L.norm2 = W(lname(wl, "norm2"));
      L.router = W(lname(wl, "router"));
      L.w_gate_up = W(lname(wl, "w_gate_up"));
      L.w_down = W(lname(wl, "w_down"));
    }
    for (int q = 0; q < (c.streams > 0 ? (d.experts > 0 || d.ff > 0 ? 2 : 1) : 0); ++q) {
      const std::string hc = q ? "hc2_" : "hc1_";
      L.hc[q].in = W(lname(wl, (hc + "in").c_str()));
      L.hc[q].out = W(lname(wl, (hc + "out").c_str()));
      L.hc[q].mix = W(lname(wl, (hc + "mix").c_str()));
    }
    if (sp) {
      L.side_gate = W(lname(wl, "side_gate"));
      L.side_proj = W(lname(wl, "side_proj"));
      L.side_norm = W(lname(wl, "side_norm"));
    }
    ws = std::max(ws, nfn_paged_attention_workspace_bytes(rows_max, d.heads, L.vp));
  }
  att_ws_bytes = ws;
  gemm_ws_bytes = 64LL << 20;
  if (zero(&att_ws, att_ws_bytes) || add(&gemm_ws, gemm_ws_bytes)) return -1;
  auto up256 = [](long long v) { return (v + 255) / 256 * 256; };
  const long long kinds = (long long)tile_kinds.size();
  io.tok = 0;
  io.slot = io.tok + up256(R * 4);
  io.pos = io.slot + up256(R * 4);
  io.want = io.pos + up256(R * 4);
  io.params = io.want + up256(R * 4);
  io.offset = io.params + up256((long long)logit_rows * 12);
  io.mix = io.offset + 256;
  io.att = io.mix + up256(R * (long long)sizeof(nfn_row_tile));
  io.seq = io.att + up256(kinds * R * 16);
  io.spans = io.seq + up256(S * (long long)sizeof(nfn_seq_rows));
  io.base = io.spans + up256(c.n_layer * S * (long long)sizeof(nfn_latent_span));
  io.out = io.base + up256(c.n_layer * S * 4);
  io.total = io.out + up256((long long)logit_rows * 4);
  CU(cudaMallocHost((void**)&h_io, (size_t)io.total));
  std::memset(h_io, 0, (size_t)io.total);
  if (zero((void**)&d_io, io.total)) return -1;
  CU(cudaDeviceSynchronize());
  finalized = true;
  return 0;
}

// ---- cache manager ------------------------------------------------------------------------------------

long long layered_engine::free_tokens() const {
  long long n = -1;
  for (const Group& g : groups) {
    const long long t = (long long)g.free_pages.size() * kPage;
    n = n < 0 ? t : std::min(n, t);
  }
  return n;
}

// Pages for every position below `upto` of the slot; the new table entries go to the device. All groups or none.
int layered_engine::reserve(int slot, int upto) {
  const int need = (upto + kPage - 1) / kPage;
  for (const Group& g : groups)
    if (need - g.next[slot] > (int)g.free_pages.size())
      return efail("engine_step: the cache pool is full (slot " + std::to_string(slot) + " needs " + std::to_string(need - g.next[slot]) + " more pages)");
  for (Group& g : groups) {
    const int from = g.next[slot];
    if (need <= from) continue;
    int* row = g.h_table + (size_t)slot * max_pages;
    for (int p = from; p < need; ++p) {
      row[p] = g.free_pages.back();
      g.free_pages.pop_back();
    }
    g.next[slot] = need;
    CU(cudaMemcpyAsync(g.d_table + (size_t)slot * max_pages + from, row + from, (size_t)(need - from) * 4, cudaMemcpyHostToDevice, stream));
  }
  return 0;
}

// The next query of the slot sits at len[slot].
void layered_engine::trim(int slot) {
  for (Group& g : groups) {
    if (g.look() <= 0) continue;
    const int live = g.oldest(len[slot]) / kPage;
    for (; g.first[slot] < std::min(live, g.next[slot]); ++g.first[slot])
      if (g.first[slot] >= g.keep) g.free_pages.push_back(g.h_table[(size_t)slot * max_pages + g.first[slot]]);
  }
}

int layered_engine::release(int slot) {
  for (Group& g : groups) {
    for (int p = 0; p < g.next[slot]; ++p)
      if (g.held(slot, p)) g.free_pages.push_back(g.h_table[(size_t)slot * max_pages + p]);
    g.first[slot] = g.next[slot] = 0;
  }
  len[slot] = 0;
  logit_at[slot] = -1;
  return 0;
}

int layered_engine::truncate(int slot, int n) {
  if (n == len[slot]) return 0;
  if (n == 0) return release(slot);
  return efail("engine_truncate: recurrent state and short convolutions keep the newest rows only; a shorter prefix has to be run again");
}

int layered_engine::fork(int src, int dst, int n) {
  if (n != len[src]) return efail("engine_fork: recurrent state and short convolutions keep the newest rows only; a shorter prefix has to be run again");
  CU(cudaSetDevice(device));
  release(dst);
  if (n == 0) return 0;
  for (Group& g : groups)   // pages the source gave back hold nothing the copy needs
    if (g.next[src] - g.first[src] + std::min(g.first[src], g.keep) > (int)g.free_pages.size()) return efail("engine_fork: the cache pool is full");
  for (size_t gi = 0; gi < groups.size(); ++gi) {
    Group& g = groups[gi];
    int *from = g.h_table + (size_t)src * max_pages, *to = g.h_table + (size_t)dst * max_pages;
    g.first[dst] = g.first[src];
    g.next[dst] = g.next[src];
    for (int p = 0; p < g.next[src]; ++p) {
      if (!g.held(src, p)) continue;
      to[p] = g.free_pages.back();
      g.free_pages.pop_back();
      for (int l = 0; l < c.n_layer; ++l) {
        const Layer& L = layers[l];
        if (L.owner != l || L.group != (int)gi || !L.paged()) continue;
        const size_t kb = (size_t)kPage * L.key_row() * es, vb = (size_t)kPage * L.value_row() * es;
        CU(cudaMemcpyAsync(static_cast<char*>(L.k_pool) + to[p] * kb, static_cast<char*>(L.k_pool) + from[p] * kb, kb, cudaMemcpyDeviceToDevice, stream));
        if (vb) CU(cudaMemcpyAsync(static_cast<char*>(L.v_pool) + to[p] * vb, static_cast<char*>(L.v_pool) + from[p] * vb, vb, cudaMemcpyDeviceToDevice, stream));
      }
    }
    CU(cudaMemcpyAsync(g.d_table + (size_t)dst * max_pages, to, (size_t)max_pages * 4, cudaMemcpyHostToDevice, stream));
  }
  parity[dst] = parity[src];
  for (const Layer& L : layers) {
    if (L.memory) {
      const size_t n = (size_t)L.memory_floats();
      CU(cudaMemcpyAsync(L.memory + dst * n, L.memory + src * n, n * 4, cudaMemcpyDeviceToDevice, stream));
    }
    if (L.prev) {
      float* half = L.prev + (size_t)parity[src] * c.max_batch * wp;
      CU(cudaMemcpyAsync(half + (size_t)dst * wp, half + (size_t)src * wp, (size_t)wp * 4, cudaMemcpyDeviceToDevice, stream));
    }
    for (const auto& u : L.sub) {
      if (!u.history) continue;
      const size_t row = (size_t)(c.input_taps - 1) * wp * es;
      char* half = static_cast<char*>(u.history) + (size_t)parity[src] * c.max_batch * row;
      CU(cudaMemcpyAsync(half + dst * row, half + src * row, row, cudaMemcpyDeviceToDevice, stream));
    }
    if (!L.state) continue;
    const size_t row = (size_t)(L.d.conv_taps - 1) * L.n_conv * es;
    char* half = static_cast<char*>(L.state) + (size_t)parity[src] * L.state_half * es;
    CU(cudaMemcpyAsync(half + dst * row, half + src * row, row, cudaMemcpyDeviceToDevice, stream));
  }
  CU(cudaStreamSynchronize(stream));
  len[dst] = n;
  return 0;
}

// ---- one pass over the rows of a step -----------------------------------------------------------------

// out = a . w^T: kOutAct in the activation type, kOutF32 in fp32, kOutResidual added to the residual stream x
int layered_engine::lin(const void* a, int lda, const void* wt, int rows, int n, int k, void* out, int ldo, int kind, const void* bias, int act) {
  if (c.dtype == 1) {
    K(nfn_gemm_f32(static_cast<const float*>(a), lda, wt, k, static_cast<float*>(out), ldo, rows, n, k, kind == kOutResidual, bias, stream));
    if (act != NFN_ACT_NONE) K(nfn_ff_rows(1, out, ldo, 0, -1, n, act, nullptr, out, ldo, rows, stream));
    return 0;
  }
  nfn_gemm_args g{};
  g.a = a; g.b = wt; g.c = out;
  g.m = rows; g.n = n; g.k = k;
  g.lda = lda; g.ldb = k; g.ldc = ldo;
  g.alpha = 1.f;
  g.flags = (kind == kOutAct ? 0 : NFN_EPI_OUT_F32) | (act << NFN_EPI_ACT_SHIFT);
  if (kind == kOutResidual) {
    g.flags |= NFN_EPI_ACCUM | NFN_EPI_COPY_BF16;
    g.aux_out = xb;
    g.ld_aux_out = wp;
  }
  if (bias) {
    g.flags |= NFN_EPI_BIAS;
    g.bias = bias;
  }
  g.workspace = gemm_ws;
  g.workspace_bytes = gemm_ws_bytes;
  K(nfn_gemm_bf16(&g, stream));
  return 0;
}

// The step between a layer's input product and its mixer. Delta layers: the convolved and activated [q | k | v] rows stay in `q`.
int layered_engine::mix_rows(const Layer& L, const Batch& b, void* ff_out) {
  const nfn_layer_desc& d = L.d;
  nfn_mix_args m{};
  m.f32 = c.dtype == 1; m.in = in; m.ld_in = L.n_in;
  m.nq = L.nq; m.nk = L.nk; m.nv = L.nv; m.off_gate = L.off_gate; m.off_up = L.off_up; m.ff = c.chained ? 0 : L.ff; m.act = d.ff_act;
  m.conv = L.conv; m.taps = d.conv_taps; m.state = L.state; m.state_half = L.state_half;
  m.conv_act = d.mixer == NFN_MIXER_DELTA ? NFN_ACT_SILU : NFN_ACT_NONE;
  m.q_out = q; m.ld_q = L.nq;
  m.k_pool = L.k_pool; m.v_pool = L.v_pool; m.kv_heads = d.kv_heads; m.dim_p = L.dp; m.vdim_p = L.vp;
  m.table = groups[L.group].d_table; m.table_ld = max_pages;
  m.temp_coef = d.q_temp_coef; m.temp_every = d.q_temp_every;
  m.ff_out = ff_out; m.ld_ff = L.n_cat;
  m.tiles = dev<nfn_row_tile>(io.mix); m.n_tiles = b.n_mix; m.tile_rows = b.n_mix == b.rows ? 1 : kMixRows; m.rows = b.rows;
  K(nfn_mix_rows(&m, stream));
  return 0;
}

// What the attention calls of a layer have in common.
void layered_engine::attention_args(const Layer& L, nfn_paged_attention_args* out) {
  const nfn_layer_desc& d = L.d;
  nfn_paged_attention_args& a = *out;
  a.f32 = c.dtype == 1; a.total_rows = rows_max;
  a.k_pool = L.k_pool; a.v_pool = L.v_pool; a.pages = groups[L.group].pages;
  a.table = groups[L.group].d_table; a.table_ld = max_pages;
  a.heads = d.heads; a.window = d.window; a.chunk = d.chunk; a.scale = d.scale; a.slopes = L.slopes;
  a.keep_first = d.window > 0 ? d.keep_first : 0; a.softcap = d.softcap; a.sink = d.sink == 1; a.sinks = L.sinks;
  a.row_slot = dev<int>(io.slot); a.row_pos = dev<int>(io.pos);
  a.max_keys = L.look() > 0 ? std::min(L.look() + d.keep_first, c.max_seq) : c.max_seq;
  a.workspace = att_ws; a.workspace_bytes = att_ws_bytes;
}

// q rows over the layer's pages -> the first columns of `cat`
int layered_engine::attention(const Layer& L, const Batch& b) {
  const nfn_layer_desc& d = L.d;
  nfn_paged_attention_args a{};
  attention_args(L, &a);
  const bool in_place = rotated(L);
  a.q = in_place ? in : q; a.ld_q = in_place ? L.n_in : L.nq;
  a.kv_heads = d.kv_heads; a.dim_p = L.dp; a.vdim_p = L.vp;
  a.gate = d.out_gate ? static_cast<char*>(in) + (size_t)L.off_g * es : nullptr; a.ld_gate = L.n_in;
  a.out = cat; a.ld_o = L.n_cat;
  const int single = L.tile_rows > 0 ? b.short_rows : b.rows;
  if (single > 0) {
    a.rows = single;
    K(nfn_paged_attention_rows(&a, stream));
  }
  if (L.tile_rows > 0 && b.rows > b.short_rows) {
    const int k = (int)(std::find(tile_kinds.begin(), tile_kinds.end(), L.tile_rows) - tile_kinds.begin());
    a.tiles = dev<int>(io.att) + b.att_off[k] * 4;
    a.n_tiles = b.att_n[k];
    K(nfn_paged_attention_tiles(&a, stream));
  }
  return 0;
}

// Gated delta rule over the convolved rows -> the first columns of `cat`
int layered_engine::delta(const Layer& L, const Batch& b) {
  const nfn_layer_desc& d = L.d;
  const int n_dec = d.heads * L.dp, n_o = d.heads * L.vp;
  const char* low = static_cast<const char*>(in);
  if (lin(low + (size_t)L.off_a1 * es, L.n_in, L.w_a2, b.rows, n_dec, L.ra, decay, n_dec, kOutF32)) return -1;
  if (lin(low + (size_t)L.off_g1 * es, L.n_in, L.w_g2, b.rows, n_o, L.rg, d_gate, n_o, kOutAct)) return -1;
  if (one_step(L, b)) {
    nfn_delta_step_args t{};
    t.f32 = c.dtype == 1; t.rows = b.rows; t.in = in; t.ld_in = L.n_in; t.off_beta = L.off_b;
    t.conv = L.conv; t.taps = d.conv_taps; t.history = L.state; t.history_half = L.state_half;
    t.decay = decay; t.ld_decay = n_dec; t.a_log = L.a_log; t.dt_bias = L.dt_bias;
    t.heads = d.heads; t.kv_heads = d.kv_heads; t.dim = d.dim; t.vdim = d.vdim; t.dim_p = L.dp; t.vdim_p = L.vp;
    t.unit_eps = kUnitEps; t.norm_eps = c.norm_eps; t.state = L.memory;
    t.gate = d_gate; t.ld_gate = n_o; t.weight = L.out_norm; t.out = cat; t.ld_out = L.n_cat; t.tiles = dev<nfn_row_tile>(io.mix);
    K(nfn_delta_step(&t, stream));
    return 0;
  }
  nfn_delta_args a{};
  a.f32 = c.dtype == 1; a.qkv = q; a.ld_qkv = L.nq;
  a.beta = low + (size_t)L.off_b * es; a.ld_beta = L.n_in;
  a.decay = decay; a.ld_decay = n_dec; a.a_log = L.a_log; a.dt_bias = L.dt_bias;
  a.heads = d.heads; a.kv_heads = d.kv_heads; a.dim = d.dim; a.dim_p = L.dp; a.vdim_p = L.vp; a.unit_eps = kUnitEps;
  a.state = L.memory; a.o = d_o; a.ld_o = n_o;
  const bool chunks = c.dtype == 0 && L.dp <= 256;
  a.seqs = dev<nfn_seq_rows>(io.seq); a.n_seqs = chunks ? b.n_short_seq : b.n_seq;
  if (a.n_seqs > 0) K(nfn_delta_rows(&a, stream));
  if (chunks && b.n_seq > b.n_short_seq) {
    a.seqs += b.n_short_seq;
    a.n_seqs = b.n_seq - b.n_short_seq;
    K(nfn_delta_chunks(&a, b.longest, delta_ws, delta_ws_bytes, stream));
  }
  K(nfn_delta_out(a.f32, d_o, n_o, d_gate, n_o, L.out_norm, c.norm_eps, cat, L.n_cat, b.rows, d.heads, d.vdim, L.vp, stream));
  return 0;
}

// Attention whose queries and keys are normed and rotated, in place inside the input product -> the first columns of `cat`
int layered_engine::rotated_attention(const Layer& L, const Batch& b) {
  const nfn_layer_desc& d = L.d;
  nfn_head_rows_args r{};
  r.f32 = c.dtype == 1; r.in = in; r.ld_in = L.n_in; r.off_k = L.nq; r.off_v = d.key_values ? L.nq : L.nq + L.nk;
  r.heads = d.heads; r.kv_heads = L.nk > 0 ? d.kv_heads : 0; r.dim = d.dim; r.dim_p = L.dp; r.vdim_p = L.vp;
  r.q_norm = L.q_norm; r.k_norm = L.k_norm; r.eps = c.norm_eps; r.freq = L.freq; r.rot_dims = d.rot_dims;
  r.q_out = in; r.ld_q = L.n_in;
  r.k_pool = L.k_pool; r.v_pool = L.v_pool; r.table = groups[L.group].d_table; r.table_ld = max_pages;
  r.tiles = dev<nfn_row_tile>(io.mix); r.n_tiles = b.n_mix; r.tile_rows = b.n_mix == b.rows ? 1 : kMixRows;
  K(nfn_head_rows(&r, stream));
  return attention(L, b);
}

// Latent attention -> the first columns of `cat`. Short entries: queries and outputs pass through the key and value projections, attention runs on
// the cached latents. Long ones: keys and values of the visible latents are formed first, as many entries at a time as the buffers hold.
int layered_engine::latent_attention(const Layer& L, const Batch& b) {
  const nfn_layer_desc& d = L.d;
  const int f32 = c.dtype == 1, H = d.heads, lp = L.lr + L.rp, qp = L.dp + L.rp, single = L.tile_rows > 0 ? b.short_rows : b.rows;
  nfn_latent_rows_args r{};
  r.f32 = f32; r.in = in; r.ld_in = L.n_in; r.off_kv = L.off_kv;
  r.heads = H; r.dim_p = L.dp; r.rot_dim = d.rot_dim; r.rot_p = L.rp; r.rank = d.kv_rank; r.rank_p = L.lr;
  r.c_norm = L.c_norm; r.eps = c.norm_eps; r.freq = L.freq;
  r.q_out = in; r.ld_q = L.n_in; r.q_row0 = single; r.q_lat = q_lat;
  r.k_pool = L.c_norm ? L.k_pool : nullptr;              // readers of another layer's cache leave it alone
  r.table = groups[L.group].d_table; r.table_ld = max_pages;
  r.tiles = dev<nfn_row_tile>(io.mix); r.n_tiles = b.n_mix; r.tile_rows = b.n_mix == b.rows ? 1 : kMixRows;
  K(nfn_latent_rows(&r, stream));
  nfn_paged_attention_args a{};
  attention_args(L, &a);
  if (single > 0) {
    nfn_group_products_args g{};
    g.f32 = f32; g.rows = single; g.groups = H;
    g.n = L.lr; g.k = L.dp; g.in = in; g.ld_in = L.n_in; g.in_group = qp; g.w = L.w_uk_t; g.out = q_lat; g.ld_out = (long long)H * lp; g.out_group = lp;
    K(nfn_group_products(&g, stream));
    a.q = q_lat; a.ld_q = H * lp; a.kv_heads = 1; a.dim_p = lp; a.vdim_p = L.lr; a.v_pool = nullptr;
    a.out = o_lat; a.ld_o = H * L.lr; a.rows = single;
    K(nfn_paged_attention_rows(&a, stream));
    if (d.out_gate) { g.gate = static_cast<const char*>(in) + (size_t)L.off_g * es; g.ld_gate = L.n_in; g.gate_group = L.vp; }
    g.n = L.vp; g.k = L.lr; g.in = o_lat; g.ld_in = (long long)H * L.lr; g.in_group = L.lr; g.w = L.w_uv; g.out = cat; g.ld_out = L.n_cat; g.out_group = L.vp;
    K(nfn_group_products(&g, stream));
  }
  const int l = (int)(&L - layers.data()), cols = H * (L.dp + L.vp);
  a.q = in; a.ld_q = L.n_in; a.kv_heads = H; a.dim_p = qp; a.vdim_p = L.vp; a.out = cat; a.ld_o = L.n_cat;
  a.gate = d.out_gate ? static_cast<const char*>(in) + (size_t)L.off_g * es : nullptr; a.ld_gate = L.n_in;
  const int k = (int)(std::find(tile_kinds.begin(), tile_kinds.end(), L.tile_rows) - tile_kinds.begin());
  for (const Batch::Round& o : b.expand[l]) {
    K(nfn_latent_gather(f32, L.k_pool, lp, L.lr, groups[L.group].d_table, max_pages, dev<nfn_latent_span>(io.spans) + (size_t)l * c.max_batch + o.span0, o.n_spans, o.max_pages,
                        lat_rows, stream));
    if (lin(lat_rows, L.lr, L.w_ukv, o.rows, cols, L.lr, lat_x, cols, kOutAct)) return -1;
    nfn_latent_expanded x{};
    x.x = lat_x; x.x_rows = o.rows; x.dim_u = L.dp; x.rot_p = L.rp; x.rank_p = L.lr; x.x_base = dev<int>(io.base) + (size_t)l * c.max_batch;
    a.tiles = dev<int>(io.att) + (size_t)(b.att_off[k] + o.tile0) * 4;
    a.n_tiles = o.n_tiles;
    K(nfn_latent_attention_tiles(&a, &x, stream));
  }
  return 0;
}

// Time mixing with the bonus recurrence -> the first columns of `cat`
int layered_engine::wkv(const Layer& L, const Batch& b) {
  const nfn_layer_desc& d = L.d;
  const int f32 = c.dtype == 1, rows = b.rows, nq = L.nq;
  const long long stride = (long long)rows_max * wp;
  nfn_shift_args s{};
  s.f32 = f32; s.width = c.width; s.ld = wp; s.n = 5; s.src = x; s.mu = L.mu;
  s.prev = L.prev; s.prev_half = (long long)c.max_batch * wp; s.out = shift; s.out_stride = stride;
  s.tiles = dev<nfn_row_tile>(io.mix); s.n_tiles = b.n_mix;
  K(nfn_shift_rows(&s, stream));
  auto mixed = [&](int i) { return static_cast<const char*>(shift) + (size_t)i * stride * es; };
  if (!f32 && rows <= kFewRows) {                        // r, k, v, gate and the inner decay projection in one launch
    nfn_group_products_args g{};
    g.rows = rows; g.groups = 4; g.n = nq; g.k = wp; g.in = shift; g.ld_in = wp; g.in_group = stride; g.w = L.w_in;
    g.out = in; g.ld_out = L.n_in; g.out_group = nq;
    g.tail_n = L.ra; g.tail_in = 4 * stride; g.tail_w = L.w1; g.tail_out = low; g.ld_tail = L.ra;
    K(nfn_group_products(&g, stream));
  } else {
    for (int i = 0; i < 4; ++i)
      if (lin(mixed(i), wp, static_cast<const char*>(L.w_in) + 2LL * i * nq * wp, rows, nq, wp, static_cast<char*>(in) + (size_t)i * nq * es, L.n_in, kOutAct)) return -1;
    if (lin(mixed(4), wp, L.w1, rows, L.ra, wp, low, L.ra, kOutF32)) return -1;
  }
  if (wkv_step(L, b)) {
    nfn_wkv_step_args t{};
    t.f32 = f32; t.rows = rows; t.rkvg = in; t.ld_rkvg = L.n_in; t.low = low; t.ld_low = t.rank_p = L.ra; t.w2 = L.w2; t.ld_w2 = 2 * L.ra;
    t.w0 = L.w0; t.u = L.u; t.heads = d.heads; t.dim = d.dim; t.dim_p = L.dp; t.state = L.memory; t.weight = L.out_norm; t.eps = c.norm_eps;
    t.out = cat; t.ld_out = L.n_cat; t.tiles = dev<nfn_row_tile>(io.mix);
    K(nfn_wkv_step(&t, stream));
    return 0;
  }
  const int ld = f32 ? L.ra : 2 * L.ra;                  // w2 rows stand twice: for the rounded tanh and for what rounding left out
  K(nfn_tanh_split(f32, low, L.ra, low_act, ld, rows, L.ra, stream));
  if (f32) K(nfn_gemm_f32(static_cast<const float*>(low_act), ld, L.w2, 2 * L.ra, decay, nq, rows, nq, L.ra, 0, nullptr, stream));
  else if (lin(low_act, ld, L.w2, rows, nq, ld, decay, nq, kOutF32)) return -1;
  nfn_wkv_args a{};
  a.f32 = f32; a.rkv = in; a.ld_rkv = L.n_in; a.z = decay; a.ld_z = nq; a.w0 = L.w0; a.u = L.u;
  a.heads = d.heads; a.dim = d.dim; a.dim_p = L.dp; a.state = L.memory; a.o = d_o; a.ld_o = nq;
  const bool chunks = !f32 && L.dp <= 256;
  a.seqs = dev<nfn_seq_rows>(io.seq); a.n_seqs = chunks ? b.n_short_seq : b.n_seq;
  if (a.n_seqs > 0) K(nfn_wkv_rows(&a, stream));
  if (chunks && b.n_seq > b.n_short_seq) {
    a.seqs += b.n_short_seq;
    a.n_seqs = b.n_seq - b.n_short_seq;
    K(nfn_wkv_chunks(&a, b.longest, wkv_ws, wkv_ws_bytes, stream));
  }
  K(nfn_head_out(f32, d_o, nq, static_cast<char*>(in) + 3LL * nq * es, L.n_in, NFN_ACT_SILU, L.out_norm, L.dp, c.norm_eps, cat, L.n_cat, rows, d.heads, d.dim, L.dp, stream));
  return 0;
}

// Linear attention with a decay per head -> the first columns of `cat`
int layered_engine::linear(const Layer& L, const Batch& b) {
  const nfn_layer_desc& d = L.d;
  const int f32 = c.dtype == 1, rows = b.rows, n_o = d.heads * L.vp;
  if (linear_step(L, b)) {                               // the products in one, activations in the step
    if (lin(hx, wp, L.w_in, rows, L.n_in, wp, in, L.n_in, kOutAct)) return -1;
    nfn_linear_step_args t{};
    t.f32 = f32; t.rows = rows; t.qkvg = in; t.ld_qkvg = L.n_in; t.powers = L.powers; t.heads = d.heads; t.vdim = d.vdim; t.dim_p = L.dp; t.vdim_p = L.vp;
    t.state = L.memory; t.o = d_o; t.ld_o = n_o; t.counters = row_count; t.weight = L.out_norm; t.eps = c.norm_eps; t.out = cat; t.ld_out = L.n_cat;
    t.tiles = dev<nfn_row_tile>(io.mix);
    K(nfn_linear_step(&t, stream));
    return 0;
  }
  char* gate = static_cast<char*>(in) + (size_t)L.off_g * es;
  if (lin(hx, wp, L.w_in, rows, L.nq, wp, in, L.n_in, kOutAct, nullptr, NFN_ACT_SILU) ||
      lin(hx, wp, static_cast<const char*>(L.w_in) + 2LL * L.off_g * wp, rows, n_o, wp, gate, L.n_in, kOutAct))
    return -1;
  nfn_linear_args a{};
  a.f32 = f32; a.qkv = in; a.ld_qkv = L.n_in; a.powers = L.powers; a.heads = d.heads; a.dim_p = L.dp; a.vdim_p = L.vp; a.state = L.memory; a.o = d_o; a.ld_o = n_o;
  const bool chunks = !f32 && nfn_linear_chunk_workspace_bytes(d.heads, L.dp, L.vp, 1) > 0;
  a.seqs = dev<nfn_seq_rows>(io.seq); a.n_seqs = chunks ? b.n_short_seq : b.n_seq;
  if (a.n_seqs > 0) K(nfn_linear_rows(&a, stream));
  if (chunks && b.n_seq > b.n_short_seq) {
    a.seqs += b.n_short_seq;
    a.n_seqs = b.n_seq - b.n_short_seq;
    K(nfn_linear_chunks(&a, b.longest, linear_ws, linear_ws_bytes, stream));
  }
  K(nfn_row_out(f32, d_o, n_o, gate, L.n_in, L.out_norm, c.norm_eps, cat, L.n_cat, rows, n_o, d.heads * d.vdim, stream));
  return 0;
}

// The gated recurrence over the projected rows -> `cat`
int layered_engine::gru(const Layer& L, const Batch& b) {
  nfn_gru_args a{};
  a.f32 = c.dtype == 1; a.width = L.vp; a.in = in; a.ld_in = L.n_in; a.state = L.memory; a.out = cat; a.ld_out = L.n_cat;
  a.seqs = dev<nfn_seq_rows>(io.seq); a.n_seqs = b.n_seq; a.n_short = b.n_short_seq;
  K(nfn_gru_rows(&a, stream));
  return 0;
}

// A chained layer's mixer on the rows hx -> y
int layered_engine::mixer(const Layer& L, const Batch& b) {
  const int kind = L.d.mixer;
  if (kind != NFN_MIXER_WKV && kind != NFN_MIXER_LINEAR && lin(hx, wp, L.w_in, b.rows, L.n_in, wp, in, L.n_in, kOutAct, L.bias_in)) return -1;
  int rc;
  if (kind == NFN_MIXER_WKV) rc = wkv(L, b);
  else if (kind == NFN_MIXER_LATENT) rc = latent_attention(L, b);
  else if (kind == NFN_MIXER_LINEAR) rc = linear(L, b);
  else if (kind == NFN_MIXER_GRU) rc = gru(L, b);
  else if (rotated(L)) rc = rotated_attention(L, b);
  else {
    if (!one_step(L, b) && mix_rows(L, b, nullptr)) return -1;
    rc = kind == NFN_MIXER_DELTA ? delta(L, b) : attention(L, b);
  }
  return rc ? -1 : lin(cat, L.n_cat, L.w_out, b.rows, wp, L.n_cat, y, wp, kOutAct);
}

// A chained layer's gated feed-forward on the rows hx -> y
int layered_engine::dense_ff(const Layer& L, int rows) {
  if (lin(hx, wp, L.w_gate_up, rows, 2 * L.ff, wp, in, 2 * L.ff, kOutAct, L.bias_gate_up)) return -1;
  const nfn_gate_clamp clamp = L.clamp();
  K(nfn_ff_rows(c.dtype == 1, in, 2 * L.ff, 0, L.ff, L.ff, L.d.ff_act, &clamp, cat, L.ff, rows, stream));
  return lin(cat, L.ff, L.w_down, rows, wp, L.ff, y, wp, kOutAct, L.bias_down);
}

// Routed experts on the rows hx; says in `sp` where the next stream pass finds each row's outputs.
int layered_engine::experts(const Layer& L, int rows, nfn_stream_args* sp) {
  const nfn_layer_desc& d = L.d;
  const bool few = !grouped(L, rows), shared = d.shared_ff > 0;
  if (shared && c.dtype == 0 && rows <= kFewRows) {        // router and the shared expert's first product in one launch
    nfn_group_products_args g{};
    g.rows = rows; g.groups = 1; g.n = L.shp; g.k = wp; g.in = hx; g.ld_in = wp; g.w = L.w_shared_up; g.out = shared_mid; g.ld_out = L.shp; g.act = d.ff_act;
    g.tail_n = L.ep; g.tail_w = L.router; g.tail_out = ex.logits; g.ld_tail = L.ep;
    K(nfn_group_products(&g, stream));
  } else if (!shared && c.dtype == 0 && rows <= kFewRows) {
    K(nfn_router_rows(hx, wp, L.router, rows, d.experts, wp, ex.logits, L.ep, stream));
  } else if (lin(hx, wp, L.router, rows, L.ep, wp, ex.logits, L.ep, kOutF32) || (shared && lin(hx, wp, L.w_shared_up, rows, L.shp, wp, shared_mid, L.shp, kOutAct, nullptr, d.ff_act))) {
    return -1;
  }
  if (shared && !few && lin(shared_mid, L.shp, L.w_shared_down, rows, wp, L.shp, y_shared, wp, kOutAct)) return -1;
  sp->y = ex.y;
  sp->y_rows = d.top;
  const bool weigh_out = d.expert_plain || d.expert_weigh_out;
  const nfn_gate_clamp clamp = L.clamp();
  sp->y_item = weigh_out ? ex.weight : nullptr;
  sp->y_plus = shared ? y_shared : nullptr;
  nfn_route_rule rule{};
  rule.correction = L.correction; rule.groups = d.route_groups; rule.keep_groups = d.route_keep; rule.normalise = d.route_normalise; rule.scale = d.route_scale; rule.softmax = d.route_softmax;
  if (few) {
    nfn_moe_rows_args a{};
    a.f32 = c.dtype == 1; a.rows = rows; a.width = wp; a.ff = L.ef; a.experts = d.experts; a.top = d.top; a.act = d.ff_act;
    a.logits = ex.logits; a.ld_logits = L.ep; a.h = hx; a.ld_h = wp; a.w_gate_up = L.w_gate_up; a.w_down = L.w_down;
    a.idx = ex.idx; a.weight = ex.weight; a.order = ex.order; a.offsets = ex.offsets; a.active = ex.active;
    a.mid = ex.mid; a.y = ex.y; a.ld_y = wp; a.plain = d.expert_plain; a.rule = rule; a.weigh_output = weigh_out; a.clamp = clamp;
    if (shared) { a.shared_ff = L.shp; a.shared_mid = shared_mid; a.w_shared_down = L.w_shared_down; a.y_shared = y_shared; }
    K(nfn_moe_rows(&a, stream));
    sp->y_index = nullptr;
    return 0;
  }
  const int cap = (int)(((long long)rows * d.top + d.experts * 127LL + 127) / 128 * 128);
  CU(cudaMemsetAsync(ex.counts, 0, (size_t)d.experts * 4, stream));
  if (weigh_out) K(nfn_moe_choose(ex.logits, L.ep, rows, d.experts, d.top, &rule, ex.idx, ex.weight, ex.counts, stream));
  else K(nfn_moe_route(ex.logits, L.ep, rows, d.experts, d.top, 1, 0, 1.f, ex.idx, ex.weight, ex.counts, stream));
  K(nfn_moe_plan(ex.counts, d.experts, cap / 128, ex.offsets, ex.cursor, ex.tile_expert, ex.plan, stream));
  K(nfn_moe_permute_weighted(hx, wp, rows, d.top, wp, ex.idx, ex.weight, ex.offsets, ex.cursor, cap, ex.xs, ex.row_of, ex.row_w, stream));
  nfn_gemm_tp_args g{};
  g.mode = NFN_TP_GROUPED;
  g.tile_group = ex.tile_expert; g.num_m_tiles_dev = ex.plan; g.groups = d.experts; g.m = cap;
  g.a = ex.xs; g.b = L.w_gate_up;
  g.k = g.lda = g.ldb = wp;
  if (d.expert_plain) {
    g.c = ex.mid; g.n = g.ldc = L.ef; g.flags = d.ff_act << NFN_EPI_ACT_SHIFT;
    K(nfn_gemm_tp(&g, stream));
    g.flags = 0;
  } else {
    g.c = ex.gate_up; g.n = g.ldc = 2 * L.ef;
    K(nfn_gemm_tp(&g, stream));
    K(nfn_moe_act_rows(ex.gate_up, weigh_out ? nullptr : ex.row_w, ex.plan, cap, L.ef, d.ff_act, &clamp, ex.mid, stream));
  }
  g.a = ex.mid; g.b = L.w_down; g.c = ex.y;
  g.n = wp; g.k = g.lda = g.ldb = L.ef; g.ldc = wp;
  K(nfn_gemm_tp(&g, stream));
  sp->y_index = ex.row_of;
  return 0;
}

// Layers whose mixer and feed-forward read one norm
int layered_engine::pass(const Batch& b) {
  hx = h;
  if (c.post_norm || c.sandwich) return post_pass(b);
  if (c.chained) return chained_pass(b);
  const int f32 = c.dtype == 1, rows = b.rows;
  nfn_row_norm_args rn{};
  rn.f32 = f32; rn.rows = rows; rn.width = c.width; rn.ld = wp; rn.eps = c.norm_eps;
  rn.tokens = dev<int>(io.tok); rn.embed = W("embed"); rn.embed_scale = c.embed_scale; rn.vocab = c.vocab;
  rn.x_out = x; rn.h = h; rn.weight = layers[0].norm1;
  K(nfn_row_norm(&rn, stream));
  rn.tokens = nullptr; rn.embed = nullptr; rn.x = x;
  for (int l = 0; l < c.n_layer; ++l) {
    const Layer& L = layers[l];
    if (lin(h, wp, L.w_in, rows, L.n_in, wp, in, L.n_in, kOutAct)) return -1;
    if (mix_rows(L, b, static_cast<char*>(cat) + (size_t)L.d.heads * L.vp * es) || attention(L, b)) return -1;
    if (lin(cat, L.n_cat, L.w_out, rows, wp, L.n_cat, x, wp, kOutResidual)) return -1;
    const bool last = l + 1 == c.n_layer;
    if (sp) {
      if (lin(f32 ? (const void*)x : xb, wp, L.side_gate, rows, sp, wp, s_gate, sp, kOutF32)) return -1;
      K(nfn_side_mul(f32, s_gate, dev<int>(io.tok), W("side_embed"), (long long)c.n_layer * sp, l * sp, c.vocab, s_act, sp, rows, sp, stream));
      if (lin(s_act, sp, L.side_proj, rows, wp, sp, y, wp, kOutAct)) return -1;
    }
    if (sp || !last) {
      rn.y = sp ? y : nullptr; rn.y_weight = L.side_norm;
      rn.x_out = sp ? x : nullptr;
      rn.h = last ? nullptr : h; rn.weight = last ? nullptr : layers[l + 1].norm1;
      K(nfn_row_norm(&rn, stream));
    }
  }
  return 0;
}

// Layers of two sublayers. A stream pass after each one applies its output to the residual and norms the next one's input; the last
// update is left to the head, which needs it for the wanted rows only.
int layered_engine::chained_pass(const Batch& b) {
  nfn_stream_args s{};
  s.f32 = c.dtype == 1; s.rows = b.rows; s.width = c.width; s.ld = wp; s.streams = std::max(c.streams, 1);
  s.eps = c.norm_eps; s.weight_offset = c.norm_offset;
  s.tokens = dev<int>(io.tok); s.embed = W("embed"); s.embed_scale = c.embed_scale; s.vocab = c.vocab;
  s.x = x; s.x_out = x; s.h = h;
  s.in = layers[0].hc[0].in; s.weight = layers[0].norm1;
  K(nfn_stream_pass(&s, stream));
  s.tokens = nullptr; s.embed = nullptr;
  for (int l = 0; l < c.n_layer; ++l) {
    const Layer& L = layers[l];
    if (mixer(L, b)) return -1;
    s.y = y; s.y_rows = 1; s.y_index = nullptr; s.y_item = nullptr; s.y_plus = nullptr; s.mix = L.hc[0].mix; s.out = L.hc[0].out;
    if (L.d.experts > 0 || L.d.ff > 0) {
      s.in = L.hc[1].in; s.weight = L.norm2;
      K(nfn_stream_pass(&s, stream));
      if (L.d.experts > 0 ? experts(L, b.rows, &s) : dense_ff(L, b.rows)) return -1;
      s.mix = L.hc[1].mix; s.out = L.hc[1].out;
    }
    if (l + 1 < c.n_layer) {
      s.in = layers[l + 1].hc[0].in; s.weight = layers[l + 1].norm1;
      K(nfn_stream_pass(&s, stream));
    }
  }
  pend = s;
  return 0;
}

// The stream pass in front of a sublayer (0: mixer, 1: feed-forward): its norm if it has one, and the convolution on its input - in the same launch when
// every row is a sequence of its own.
int layered_engine::enter(nfn_stream_args* s, const Layer& L, int which, const Batch& b) {
  const auto& u = L.sub[which];
  const long long half = (long long)c.max_batch * (c.input_taps - 1) * wp;
  s->weight = !c.sandwich ? nullptr : which ? L.norm2 : L.norm1;
  const bool fused = u.conv && b.single;
  s->conv = fused ? u.conv : nullptr;
  s->conv_taps = c.input_taps; s->history = u.history; s->history_half = half; s->tiles = dev<nfn_row_tile>(io.mix);
  K(nfn_stream_pass(s, stream));
  s->conv = nullptr;
  hx = h;
  if (!u.conv || fused) return 0;
  nfn_input_conv_args a{};
  a.f32 = c.dtype == 1; a.ld = wp; a.taps = c.input_taps; a.h = h; a.conv = u.conv; a.history = u.history; a.history_half = half; a.out = hc;
  a.tiles = dev<nfn_row_tile>(io.mix); a.n_tiles = b.n_mix;
  K(nfn_input_conv(&a, stream));
  hx = hc;
  return 0;
}

// Layers whose sublayers' outputs are normed before they are added. Sublayers read the residual itself, in the activation type, or (sandwich) its norm. The
// last update is left to the head.
int layered_engine::post_pass(const Batch& b) {
  nfn_stream_args s{};
  s.f32 = c.dtype == 1; s.rows = b.rows; s.width = c.width; s.ld = wp; s.streams = 1;
  s.eps = c.norm_eps; s.y_scale = c.residual_mult;
  s.tokens = dev<int>(io.tok); s.embed = W("embed"); s.embed_scale = c.embed_scale; s.vocab = c.vocab;
  s.x = x; s.x_out = x; s.h = h; s.scalar_norms = c.scalar_norms;
  if (enter(&s, layers[0], 0, b)) return -1;
  s.tokens = nullptr; s.embed = nullptr;
  for (int l = 0; l < c.n_layer; ++l) {
    const Layer& L = layers[l];
    if (mixer(L, b)) return -1;
    s.y = y; s.y_rows = 1; s.y_index = nullptr; s.y_item = nullptr; s.y_plus = nullptr; s.y_weight = c.sandwich ? L.sub[0].norm_b : L.norm1;
    if (L.has_ff()) {
      if (enter(&s, L, 1, b)) return -1;
      if (L.d.experts > 0 ? experts(L, b.rows, &s) : dense_ff(L, b.rows)) return -1;
      s.y_weight = c.sandwich ? L.sub[1].norm_b : L.norm2;
    }
    if (l + 1 < c.n_layer && enter(&s, layers[l + 1], 0, b)) return -1;
  }
  pend = s;
  return 0;
}

// output norm and head of `rows` rows of x (src_rows: device indices, NULL: the first ones) -> logits
int layered_engine::head(const int* src_rows, int rows) {
  if (c.chained) {
    nfn_stream_args s = pend;
    s.rows = rows; s.src_rows = src_rows; s.x_out = nullptr;
    s.in = nullptr; s.h = hw; s.weight = W("final_norm");
    K(nfn_stream_pass(&s, stream));
  } else {
    nfn_row_norm_args rn{};
    rn.f32 = c.dtype == 1; rn.rows = rows; rn.width = c.width; rn.ld = wp; rn.eps = c.norm_eps;
    rn.x = x; rn.src_rows = src_rows; rn.h = hw; rn.weight = W("final_norm");
    K(nfn_row_norm(&rn, stream));
  }
  if (lin(hw, wp, W(c.untied_head ? "head" : "embed"), rows, vp, wp, logits, vp, kOutF32)) return -1;
  if (c.logit_softcap > 0.f || c.logit_scale != 1.f) K(nfn_logit_cap(logits, vp, rows, vp, c.logit_scale, c.logit_softcap, stream));
  return 0;
}

int layered_engine::sample(int rows) {
  K(nfn_sample_rows(logits, 1, vp, rows, c.vocab, dev<int>(io.out), nullptr, 1.f, 0, 1.f, dev<float>(io.params), 0x5eedULL, 0ULL,
                    dev<unsigned long long>(io.offset), 0, stream));
  return 0;
}

// Runs one batch of at most rows_max rows. row_of[i]: row of the i-th token (in the order of the entries). single: every entry
// brings one token, and the pass, the head over all rows and the sampling run as one (replayed) launch sequence.
int layered_engine::run(const std::vector<nfn_step_entry>& part, const int32_t* const* part_tokens, std::vector<int>& row_of, bool single) {
  int total = 0, short_rows = 0;
  Batch b;
  std::vector<int> first(part.size());
  for (size_t i = 0; i < part.size(); ++i) {
    if (reserve(part[i].slot, len[part[i].slot] + part[i].count)) return -1;
    if (part[i].count < kTileMin) {
      first[i] = short_rows;
      short_rows += part[i].count;
    }
    total += part[i].count;
  }
  int at = short_rows;
  for (size_t i = 0; i < part.size(); ++i)
    if (part[i].count >= kTileMin) {
      first[i] = at;
      at += part[i].count;
    }
  int *tok = host<int>(io.tok), *slot = host<int>(io.slot), *pos = host<int>(io.pos);
  nfn_row_tile* mix = host<nfn_row_tile>(io.mix);
  int n_mix = 0, hist_max = 0;
  for (const Layer& L : layers) hist_max = std::max(std::max(hist_max, c.input_taps - 1), L.prev ? 1 : L.d.conv_taps - 1);
  row_of.clear();
  for (size_t i = 0; i < part.size(); ++i) {
    const int s = part[i].slot, p0 = len[s], n = part[i].count;
    for (int r = 0; r < n; ++r) {
      tok[first[i] + r] = part_tokens[i][r];
      slot[first[i] + r] = s;
      pos[first[i] + r] = p0 + r;
      row_of.push_back(first[i] + r);
    }
    for (int r = 0; r < n;) {
      const int k = std::min(n - r, kMixRows - (p0 + r) % kMixRows);
      mix[n_mix++] = nfn_row_tile{first[i] + r, k, first[i], n, p0, s, parity[s], 0};
      r += k;
    }
  }
  int rows = total;
  if (single) {
    rows = 1;
    while (rows < total) rows *= 2;
    rows = std::min(rows, c.max_batch);
    for (int r = total; r < rows; ++r) {
      tok[r] = 0; slot[r] = -1; pos[r] = 0;
      mix[n_mix++] = nfn_row_tile{r, 1, r, 1, 0, -1, 0, 0};
    }
    short_rows = rows;
  }
  nfn_seq_rows* seq = host<nfn_seq_rows>(io.seq);
  for (int longs = 0; longs < 2; ++longs) {
    for (size_t i = 0; i < part.size(); ++i)
      if ((part[i].count >= kTileMin) == (longs == 1)) b.longest = std::max(b.longest, part[i].count), seq[b.n_seq++] = nfn_seq_rows{first[i], part[i].count, part[i].slot, len[part[i].slot]};
    if (!longs) {
      for (int r = total; r < rows; ++r) seq[b.n_seq++] = nfn_seq_rows{r, 1, -1, 0};
      b.n_short_seq = b.n_seq;
    }
  }
  std::vector<int>&att_off = b.att_off, &att_n = b.att_n;
  att_off.assign(tile_kinds.size(), 0);
  att_n.assign(tile_kinds.size(), 0);
  int* att = host<int>(io.att);
  int n_att = 0;
  for (size_t k = 0; k < tile_kinds.size(); ++k) {
    att_off[k] = n_att;
    for (size_t i = 0; i < part.size(); ++i) {
      if (part[i].count < kTileMin) continue;
      for (int r = 0; r < part[i].count; r += tile_kinds[k]) {
        int* t = att + (size_t)n_att++ * 4;
        t[0] = first[i] + r; t[1] = std::min(tile_kinds[k], part[i].count - r); t[2] = part[i].slot; t[3] = len[part[i].slot] + r;
      }
    }
    att_n[k] = n_att - att_off[k];
  }
  // what the latent layers expand: the visible pages of every long entry, in rounds that fit
  b.expand.resize(c.n_layer);
  for (int l = 0; l < c.n_layer; ++l) {
    const Layer& L = layers[l];
    if (!L.latent() || L.tile_rows <= 0) continue;
    nfn_latent_span* spans = host<nfn_latent_span>(io.spans) + (size_t)l * c.max_batch;
    int* base = host<int>(io.base) + (size_t)l * c.max_batch;
    int n_spans = 0, tile = 0;
    for (size_t i = 0; i < part.size(); ++i) {
      if (part[i].count < kTileMin) continue;
      const int s = part[i].slot, p0 = len[s], oldest = L.d.chunk > 0 ? p0 / L.d.chunk * L.d.chunk : L.d.window > 0 ? std::max(0, p0 - L.d.window + 1) : 0;
      const int page0 = oldest / kPage, pages = (p0 + part[i].count - 1) / kPage + 1 - page0, tiles = (part[i].count + L.tile_rows - 1) / L.tile_rows;
      if (b.expand[l].empty() || b.expand[l].back().rows + pages * kPage > lat_cap) b.expand[l].push_back(Batch::Round{n_spans, 0, 0, 0, tile, 0});
      Batch::Round& o = b.expand[l].back();
      spans[n_spans++] = nfn_latent_span{s, page0, pages, o.rows};
      base[s] = o.rows - page0 * kPage;
      o.n_spans += 1;
      o.max_pages = std::max(o.max_pages, pages);
      o.rows += pages * kPage;
      o.n_tiles += tiles;
      tile += tiles;
      if (o.rows > lat_cap) return efail("engine_step: a portion's latents do not fit their buffer");
    }
  }
  // row metadata, then the tile lists
  CU(cudaMemcpyAsync(d_io + io.tok, h_io + io.tok, (size_t)(io.pos - io.tok) + (size_t)rows * 4, cudaMemcpyHostToDevice, stream));
  CU(cudaMemcpyAsync(d_io + io.mix, h_io + io.mix, (size_t)n_mix * sizeof(nfn_row_tile), cudaMemcpyHostToDevice, stream));
  if (n_att > 0) CU(cudaMemcpyAsync(d_io + io.att, h_io + io.att, (size_t)n_att * 16, cudaMemcpyHostToDevice, stream));

  CU(cudaMemcpyAsync(d_io + io.seq, h_io + io.seq, (size_t)b.n_seq * sizeof(nfn_seq_rows), cudaMemcpyHostToDevice, stream));
  if (lat_cap > 0 && rows > short_rows) CU(cudaMemcpyAsync(d_io + io.spans, h_io + io.spans, (size_t)(io.out - io.spans), cudaMemcpyHostToDevice, stream));

  b.rows = rows;
  b.short_rows = short_rows;
  b.n_mix = n_mix;
  b.single = single;
  const long long before = nfn_launch_count();
  auto body = [&]() -> int {
    if (pass(b)) return -1;
    return single ? (head(nullptr, rows) || sample(rows) ? -1 : 0) : 0;
  };
  if (!single || !c.use_cuda_graph) {
    if (body()) return -1;
    launches += nfn_launch_count() - before;
  } else if (graphs.count(rows)) {
    CU(cudaGraphLaunch(graphs[rows], stream));
    launches += graph_launches[rows];
  } else if (graph_calls[rows]++ == 0) {
    if (body()) return -1;                          // first call with this row count: attributes and tensor maps get set up
    launches += nfn_launch_count() - before;
  } else {
    cudaGraph_t g = nullptr;
    CU(cudaStreamBeginCapture(stream, cudaStreamCaptureModeThreadLocal));
    const int rc = body();
    const cudaError_t ce = cudaStreamEndCapture(stream, &g);
    if (rc != 0 || ce != cudaSuccess || !g) {
      if (g) cudaGraphDestroy(g);
      return rc != 0 ? -1 : efail("engine_step: stream capture failed");
    }
    cudaGraphExec_t ge = nullptr;
    CU(cudaGraphInstantiate(&ge, g, 0));
    cudaGraphDestroy(g);
    graphs[rows] = ge;
    graph_launches[rows] = nfn_launch_count() - before;
    CU(cudaGraphLaunch(ge, stream));
    launches += graph_launches[rows];
  }
  for (const nfn_step_entry& p : part) {
    len[p.slot] += p.count;
    parity[p.slot] ^= hist_max > 0;
    trim(p.slot);
  }
  return 0;
}

int layered_engine::step(const nfn_step_entry* entries, int n_entries, const int32_t* tokens, const int32_t* want_rows, int n_want,
                         const nfn_sampling* want_sampling, int32_t* want_tokens, float* want_logits) {
  CU(cudaSetDevice(device));
  if ((want_sampling == nullptr) != (want_tokens == nullptr)) return efail("engine_step: sampling parameters and a place for the tokens go together");
  std::vector<uint8_t> seen(c.max_batch, 0);
  long long total = 0;
  bool single = n_entries > 0;
  for (int i = 0; i < n_entries; ++i) {
    const nfn_step_entry& e = entries[i];
    if (e.slot < 0 || e.slot >= c.max_batch || seen[e.slot]) return efail("engine_step: bad or repeated slot");
    if (e.count <= 0 || e.count > c.max_seq || len[e.slot] + e.count > c.max_seq) return efail("engine_step: slot " + std::to_string(e.slot) + " would pass max_seq");
    seen[e.slot] = 1;
    total += e.count;
    single &= e.count == 1;
  }
  for (long long i = 0; i < total; ++i)
    if (tokens[i] < 0 || tokens[i] >= c.vocab) return efail("engine_step: token id outside the vocabulary");
  for (int i = 0; i < n_want; ++i)
    if (want_rows[i] < 0 || want_rows[i] >= total || (i > 0 && want_rows[i] <= want_rows[i - 1])) return efail("engine_step: wanted places must ascend inside the step");
  {
    // enough pages for the whole step before anything runs (portions longer than a pass get pages back on the way: see run)
    if (total <= rows_max)
      for (const Group& g : groups) {
        long long need = 0;
        for (int i = 0; i < n_entries; ++i) need += std::max(0, (len[entries[i].slot] + entries[i].count + kPage - 1) / kPage - g.next[entries[i].slot]);
        if (need > (long long)g.free_pages.size()) return efail("engine_step: the cache pool is full");
      }
  }
  for (int b = 0; b < c.max_batch; ++b)
    if (seen[b]) logit_at[b] = -1;

  auto stash = [&]() -> int {   // logits of slots that are not part of what comes next
    for (int b = 0; b < c.max_batch; ++b)
      if (logit_at[b] >= 0) {
        CU(cudaMemcpyAsync(saved + (size_t)b * vp, logits + (size_t)logit_at[b] * vp, (size_t)vp * 4, cudaMemcpyDeviceToDevice, stream));
        logit_at[b] = -2;
      }
    return 0;
  };
  auto draw_params = [&](int row, const nfn_sampling* s) {
    float* rp = host<float>(io.params) + 3 * row;
    rp[0] = s ? s->temperature : 0.f;
    rp[1] = s ? (float)s->top_k : 0.f;
    rp[2] = s ? s->top_p : 1.f;
  };
  auto send_params = [&](int rows, const nfn_sampling* s) -> int {
    *host<unsigned long long>(io.offset) = ((s ? s->seed : 0ull) << 20) ^ (++steps);
    CU(cudaMemcpyAsync(d_io + io.params, h_io + io.params, (size_t)rows * 12, cudaMemcpyHostToDevice, stream));
    CU(cudaMemcpyAsync(d_io + io.offset, h_io + io.offset, 8, cudaMemcpyHostToDevice, stream));
    return 0;
  };
  auto fetch = [&](int want0, int n, const std::vector<int>& at) -> int {   // results of wants [want0, want0 + n), rows `at` of logits / out
    if (want_logits)
      for (int i = 0; i < n; ++i)
        CU(cudaMemcpyAsync(want_logits + (size_t)(want0 + i) * c.vocab, logits + (size_t)at[i] * vp, (size_t)c.vocab * 4, cudaMemcpyDeviceToHost, stream));
    if (want_tokens) CU(cudaMemcpyAsync(h_io + io.out, d_io + io.out, (size_t)logit_rows * 4, cudaMemcpyDeviceToHost, stream));
    CU(cudaStreamSynchronize(stream));
    if (want_tokens)
      for (int i = 0; i < n; ++i) want_tokens[want0 + i] = host<int>(io.out)[at[i]];
    return 0;
  };

  int ei = 0, used = 0, w = 0;       // entry, its tokens already run, next want
  long long base = 0;                // tokens run by earlier passes
  const int32_t* cursor = tokens;
  while (ei < n_entries) {
    std::vector<nfn_step_entry> part;
    std::vector<const int32_t*> ptok;
    int rows = 0;
    while (ei < n_entries && rows < rows_max) {
      const int n = std::min(entries[ei].count - used, rows_max - rows);
      part.push_back(nfn_step_entry{entries[ei].slot, n});
      ptok.push_back(cursor);
      cursor += n;
      rows += n;
      used += n;
      if (used == entries[ei].count) { ++ei; used = 0; }
    }
    std::vector<int> row_of, slot_of;
    for (const nfn_step_entry& p : part) slot_of.insert(slot_of.end(), p.count, p.slot);
    if (single) {
      if (stash()) return -1;
      std::vector<int> want_of(rows, -1);
      for (int i = 0; i < n_want; ++i) want_of[want_rows[i]] = i;
      for (int r = 0; r < logit_rows; ++r) draw_params(r, (r < rows && want_sampling && want_of[r] >= 0) ? &want_sampling[want_of[r]] : nullptr);
      if (send_params(logit_rows, (want_sampling && n_want > 0) ? want_sampling : nullptr)) return -1;
      if (run(part, ptok.data(), row_of, true)) return -1;
      for (int r = 0; r < rows; ++r) logit_at[slot_of[r]] = row_of[r];
      std::vector<int> at;
      for (int i = 0; i < n_want; ++i) at.push_back(row_of[want_rows[i]]);
      if (fetch(0, n_want, at)) return -1;
      break;
    }
    if (run(part, ptok.data(), row_of, false)) return -1;
    while (w < n_want && want_rows[w] < base + rows) {
      if (stash()) return -1;
      int n = 0;
      std::vector<int> at;
      for (; w + n < n_want && n < logit_rows && want_rows[w + n] < base + rows; ++n) {
        host<int>(io.want)[n] = row_of[want_rows[w + n] - base];
        logit_at[slot_of[want_rows[w + n] - base]] = n;
        at.push_back(n);
        draw_params(n, want_sampling ? &want_sampling[w + n] : nullptr);
      }
      CU(cudaMemcpyAsync(d_io + io.want, h_io + io.want, (size_t)n * 4, cudaMemcpyHostToDevice, stream));
      const long long before = nfn_launch_count();
      if (head(dev<int>(io.want), n)) return -1;
      if (want_sampling && (send_params(n, &want_sampling[w]) || sample(n))) return -1;
      launches += nfn_launch_count() - before;
      if (fetch(w, n, at)) return -1;
      w += n;
    }
    base += rows;
    CU(cudaStreamSynchronize(stream));   // the pinned blocks are written again by the next pass
  }
  if (nfn_status_peek() != 0) return efail("engine_step: a kernel reported error code " + std::to_string(nfn_status_read_reset()));
  return 0;
}

// ---- the one-sequence and all-slots forms ---------------------------------------------------------------

int layered_engine::prefill(int slot, const int32_t* tokens, int n, const nfn_sampling* s, int32_t* next_token) {
  if (n <= 0 || n >= c.max_seq) return efail("engine_prefill: the prompt must hold between 1 and max_seq - 1 tokens");
  release(slot);
  const nfn_step_entry e{slot, n};
  const int32_t want = n - 1;
  return step(&e, 1, tokens, &want, 1, s, next_token, nullptr);
}

int layered_engine::decode(const int32_t* tokens_in, const uint8_t* active, const nfn_sampling* s, const nfn_sampling* per_slot, int32_t* next_tokens) {
  std::vector<nfn_step_entry> entries;
  std::vector<int32_t> tok, want, out;
  std::vector<nfn_sampling> sam;
  for (int b = 0; b < c.max_batch; ++b) {
    if (!active[b]) continue;
    if (len[b] <= 0) return efail("engine_decode: slot " + std::to_string(b) + " is active but was never prefilled");
    if (len[b] + 1 > c.max_seq) return efail("engine_decode: slot " + std::to_string(b) + " reached max_seq");
    want.push_back((int32_t)entries.size());
    entries.push_back(nfn_step_entry{b, 1});
    tok.push_back(tokens_in[b]);
    sam.push_back(per_slot ? per_slot[b] : *s);
    sam.back().seed = s->seed;
  }
  if (entries.empty()) return 0;
  out.resize(entries.size());
  if (step(entries.data(), (int)entries.size(), tok.data(), want.data(), (int)want.size(), sam.data(), out.data(), nullptr)) return -1;
  for (size_t i = 0; i < entries.size(); ++i) next_tokens[entries[i].slot] = out[i];
  return 0;
}

int layered_engine::last_logits(int slot, float* out_vocab) {
  if (logit_at[slot] == -1) return efail("engine_last_logits: the slot's newest tokens were run without asking for logits");
  CU(cudaSetDevice(device));
  const float* src = logit_at[slot] == -2 ? saved + (size_t)slot * vp : logits + (size_t)logit_at[slot] * vp;
  CU(cudaMemcpy(out_vocab, src, (size_t)c.vocab * 4, cudaMemcpyDeviceToHost));
  return 0;
}
