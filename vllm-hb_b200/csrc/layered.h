// Models described layer by layer: every layer has a mixer (attention, a gated linear
// recurrence, or both side by side) and possibly a feed-forward (one gated layer, or a mixture of
// them), over one or several residual streams held in fp32.  The mechanisms and their constants are
// data (LayeredSpec); a design's reader (latarax.cc, biberax.cc, badolix.cc, muzopel.cc) turns its config.json and tensor
// names into it.
#pragma once

#include <cstdint>
#include <map>
#include <memory>
#include <string>
#include <vector>

#include "common.h"
#include "gemm.h"

namespace hb {

struct Json;

// Softmax attention over a paged K/V cache: per-head sizes of keys and values may differ;
// position i sees j <= i with i - j < window (0 = all) or j < keep_first, or (chunk > 0) the j <= i
// of its own chunk of positions.
struct AttentionSpec {
  int heads = 0, kv_heads = 0, dim = 0, vdim = 0;
  float scale = 1.f;
  int window = 0, keep_first = 0, chunk = 0;
  float softcap = 0.f;              // scores s become softcap * tanh(s / softcap) (0: they stay)
  // rotation of the first 2 * rotation.size() channels of queries and keys, channel 2i with 2i + 1 or
  // (halves) channel i with i + rotation.size(); the angle of pair i is position * rotation[i], and sines
  // and cosines are multiplied by rotation_gain
  std::vector<double> rotation;
  bool rotation_halves = false;
  float rotation_gain = 1.f;
  int kv_from = -1;                 // the layer whose keys and values are used (-1: the layer's own)
  // Latent attention (rank > 0): keys and values of all heads are products of one normed latent of
  // `rank` channels; a query head is [dim | rot_dim], its second part and one key part of rot_dim
  // channels that all heads share are rotated.  The cache holds [latent | rotated key part], and the
  // attention runs over the latent itself (as keys and as values, with the heads' matrices applied to
  // queries and outputs).
  int rank = 0, rot_dim = 0;
  int q_rank = 0;                   // > 0: the queries are a product of a normed latent of their own
  bool gate_per_head = false;       // the output gate is one number per head (else one per channel)
  int cached_heads() const { return rank ? 1 : kv_heads; }
  int key_width() const { return rank ? rank + rot_dim : dim; }
  int value_width() const { return rank ? rank : vdim; }
  int64_t value_pool_width() const { return rank || values_are_keys ? 0 : vdim; }
  bool values_are_keys = false;     // the values are the keys as projected (before their norm)
  bool unit_sink = false;           // the softmax denominator has one more member of score 0
  // learned bias by distance: row bucket(i - j) of a [buckets, heads] table; the lower half of the
  // buckets is exact, the upper half logarithmic up to distance bias_far
  double bias_far = 0;
};

// A gated feed-forward W_down act(W_gate h, W_up h); act: gemm.h.
struct FeedForwardSpec {
  int64_t ff = 0;                   // 0: none
  GatedAct act;
  std::string gate, up, down;
  std::string gate_bias, up_bias, down_bias;  // empty: none
};

// `top` of the experts run for every token, weighted by the softmax over their router logits, or
// (sigmoid) by their sigmoid scores over the scores' sum, chosen among the best `keep` of `groups`
// equal groups of neighbours.
struct ExpertsSpec {
  int experts = 0, top = 0;         // 0: no mixture
  bool sigmoid = false;
  int groups = 1, keep = 1;
  // softmax_all: weighted by the softmax over all outputs of the router, chosen by that plus `correction`;
  // the last `identity` outputs are no experts, they hand the input on
  bool softmax_all = false;
  int identity = 0;
  int64_t ff = 0;
  GatedAct act;                     // single: W_down act(W_up h)
  std::string router, router_bias, correction;
  std::string prefix;               // expert e: prefix + "<e>." + gate | up | down
  int outputs() const { return experts + identity; }
  // experts a random row chooses
  double picks() const { return (double)top * experts / outputs(); }
};

// S_t = diag(a_t) S_(t-1) + k_t v_t^T, o_t = S_t^T q_t per head, fp32 state of [dim, vdim].
struct RecurrenceSpec {
  int heads = 0, dim = 0, vdim = 0;
  int qk_heads = 0;                 // heads of q and k, each serving heads / qk_heads neighbours (0: one each)
  // Selective state space: v, k and q pass through a causal convolution of conv_taps taps and SiLU; a
  // step softplus(dt + bias) per token and head gives the decay exp(-exp(a_log) step) and scales the
  // key, and the output gets skip * v
  bool per_token_decay = false;
  int conv_taps = 0;
  float q_scale = 1.f;
  bool silu_qkv = false;            // q, k and v pass through SiLU
  // decay: a constant per head, or sigmoid(W2 (W1 h) + bias)^(1/tau) per key channel
  bool low_rank_decay = false;
  std::vector<double> decay;        // [heads]
  double tau = 1.0;
  int rank = 0;
  // the outputs are RMS-normed per head (weight [vdim]) or all heads together (weight
  // [heads * vdim]) and multiplied by a gate
  bool norm_per_head = false;
  bool gate_silu = false;           // gate activation: SiLU, else sigmoid
  int gated_norm_groups = 0;        // > 0: the gate comes first, then the norm in that many equal parts
  int64_t conv_channels() const { return (int64_t)heads * vdim + 2 * (int64_t)qk_heads * dim; }
};

// Rows of the layer's input projection that come from one checkpoint tensor.
struct ProjPart {
  std::string tensor;
  int64_t rows = 0;
  int64_t offset = 0;  // first column of the projection's output (a multiple of 8)
  int64_t first = 0, of = 0;  // of > 0: the rows from `first` on of a tensor of `of` rows
};

struct MixerSpec {
  bool has_attn = false, has_rec = false;
  AttentionSpec attn;
  RecurrenceSpec rec;
  // tensors: projections that read h, concatenated into one matrix
  ProjPart aq, ak, av, ag;                   // attention (ag: gate of the heads' outputs)
  ProjPart rq, rk, rv, rg, ra1;              // recurrence (ra1: low-rank decay)
  ProjPart rx, rdt;                          // selective state space: [v | k | q] before the convolution, steps
  std::string rec_conv, rec_conv_bias, rec_dt_bias, rec_a_log, rec_skip;
  std::string attn_latent_norm, attn_uk, attn_uv;  // latent attention (ak: [latent | shared key part])
  std::string attn_q_latent_norm, attn_uq;         // with q_rank (aq: the queries' latent)
  std::string attn_o, rec_o, rec_norm, rec_a2, rec_a2_bias;
  // attention, empty where the design has none: biases of the projections, norms over the whole
  // query and key projections, distance bias table, learned sinks [heads]
  std::string attn_q_bias, attn_k_bias, attn_o_bias, attn_q_norm, attn_k_norm, attn_rel, attn_sink;
  std::string attn_out_norm, rec_out_norm;   // both branches: each normed, then averaged
};

struct LayerSpec {
  std::string prefix;                        // tensor name prefix, "l0."
  MixerSpec mixer;
  std::string norm1, norm2;
  std::string conv1, conv2;                  // convolutions of the sublayers' inputs (input_taps)
  std::string depth;                         // weights of the sum over all results so far (empty: none)
  std::string hc1_in, hc1_out, hc1_mix, hc2_in, hc2_out, hc2_mix;  // empty: one plain residual stream
  FeedForwardSpec ffn;                       // the layer's feed-forward, or what every token takes beside `moe`
  ExpertsSpec moe;
  bool has_ffn() const { return ffn.ff > 0 || moe.experts > 0; }
};

struct LayeredSpec {
  std::string design;
  int64_t width = 0, vocab = 0, max_positions = 0;
  int streams = 1;
  float eps = 1e-6f;
  float norm_offset = 0.f;                   // of norm1, norm2, final norm: 0 stored as they apply, 1 around zero
  float embed_scale = 1.f, residual_mult = 1.f, logit_scale = 1.f;  // residual_mult: of designs with one plain stream
  std::string embed, pos, final_norm, head;  // pos empty: no learned positions; head empty: the embedding table
  // post_norm: the norms are on the sublayers' outputs (and on the embedding), in norm_groups equal parts;
  // the sublayers read the residual itself, to which a causal convolution of input_taps taps per channel is
  // added (0: none).  One stream, residual.cu.
  bool post_norm = false;
  int norm_groups = 1;
  int input_taps = 0;
  std::string embed_norm;
  float logit_cap = 0.f;                     // > 0: logits z become cap * tanh(z / cap)
  std::vector<LayerSpec> layers;
};

// Design readers: config.json (and, for sizes it does not give, tensor shapes) -> spec.
bool is_latarax(const Json& config);
int read_latarax(const Json& config, LayeredSpec* out);
bool is_biberax(const Json& config);
int read_biberax(const Json& config, LayeredSpec* out);
bool is_badolix(const Json& config);
int read_badolix(const Json& config, LayeredSpec* out);
bool is_muzopel(const Json& config);
int read_muzopel(const Json& config, LayeredSpec* out);

// ---------------------------------------------------------------------------- weights
struct LayeredLinear {
  void* w = nullptr;        // [N, K] engine dtype; N, K are padded to multiples of 8 with zeros
  int64_t N = 0, K = 0;
};

struct SublayerMix {        // how a sublayer's output goes back into the streams (fp32, device)
  float* in = nullptr;      // [streams]
  float* out = nullptr;     // [streams]
  float* mix = nullptr;     // [streams from, streams to]
  float* norm = nullptr;    // [width]
  // convolution of the sublayer's input: [taps, width]; inputs of earlier steps [slots, taps - 1, width]
  float *conv = nullptr, *conv_state = nullptr;
};

struct LayeredExperts {     // experts' matrices one after another; the expert every token passes through
  LayeredLinear gate_up, down;   // one expert's [2 * ffp, K] (without a gate [ffp, K]) and [N, ffp]
  LayeredLinear shared_gate_up, shared_down;
  int64_t ffp = 0, shared_ffp = 0;
  int64_t ld() const { return ffp > shared_ffp ? ffp : shared_ffp; }  // row stride of the activations
  void* router = nullptr;        // [outputs, width] engine dtype
  float *router_bias = nullptr, *correction = nullptr;  // [outputs]
};

struct LayeredLayer {
  LayeredLinear proj;                        // all projections of h
  LayeredLinear attn_o, rec_o, gate_up, down;
  int64_t ffp = 0;                           // padded feed-forward width
  float *decay = nullptr;                    // [heads] (constant decay)
  float *a2 = nullptr, *a2_bias = nullptr;   // [heads * dim, rank], [heads * dim]
  float *rec_norm = nullptr, *attn_out_norm = nullptr, *rec_out_norm = nullptr;
  double* rotation = nullptr;                // [pairs] frequencies
  float *q_bias = nullptr, *k_bias = nullptr, *o_bias = nullptr, *q_norm = nullptr, *k_norm = nullptr, *sink = nullptr;
  float *rel = nullptr, *dist_bias = nullptr;  // [buckets, heads]; the same by distance, [heads, dist_len]
  int dist_len = 0, buckets = 0;
  // latent attention: per head W_uk^T [rank, dim] and W_uv [vdim, rank]; whether the tensor-core kernel
  // takes these products
  void *uk_t = nullptr, *ukv = nullptr, *uv = nullptr;  // ukv [heads * dim | heads * vdim, rank]: W_uk, then W_uv
  bool expand = false;                       // prompts attend to keys and values of the heads grown out of the latents
  float* latent_norm = nullptr;
  LayeredLinear uq;                          // queries out of their latent
  float* q_latent_norm = nullptr;
  bool latent_tc = false;
  // selective state space
  float *conv_w = nullptr, *conv_b = nullptr, *dt_bias = nullptr, *a_log = nullptr, *skip = nullptr;
  void* conv_state = nullptr;                // [slots, taps - 1, channels] engine dtype
  float *gate_b = nullptr, *up_b = nullptr, *down_b = nullptr;  // biases of a dense feed-forward
  LayeredExperts moe;
  int kv_pool = -1;                          // index into hb_engine::kc / vc
  int tile_kind = -1, expand_kind = -1;      // indices into LayeredModel::tile_kinds (-1: row by row)
  float* state = nullptr;                    // [slots, heads, dim, vdim]
  SublayerMix sub1, sub2;
  float* depth = nullptr;                    // [layers before this one + 2]
};

// Plans of all matrix products for one bucket of batch rows.
struct LayeredPlans {
  std::vector<TcGemmPlan> proj, uq, latent_q, latent_v, attn_o, rec_o, gate_up, down, moe_gate_up, moe_down;
};

struct LayeredGraph {
  cudaGraphExec_t exec = nullptr;
  int64_t launches = 0;
};

// Tiles of query positions: how many positions one has, and which segments are cut into them.
struct TileKind {
  int positions;
  enum Which { kAll, kNotExpanded, kExpanded } which;
  bool operator==(const TileKind& o) const { return positions == o.positions && which == o.which; }
};
constexpr int kTileKinds = 6;  // different kinds in one model

// Where a step's inputs lie in the (pinned and device) input block, and what it contains.
struct LayeredStep {
  int rows = 0, segs = 0, want = 0;
  int n_short = 0;        // segments the token-by-token recurrence kernel takes
  int n_chunks = 0;       // chunks of the longer segments (chunked recurrence kernels)
  int n_long = 0;         // longer segments
  int n_tiles[kTileKinds] = {0};  // query tiles of the tiled attention kernel, by tile size
  int n_expand = 0;       // blocks of the contexts whose keys and values are grown out of latents
  int n_not_expanded = 0; // rows of the other segments
  int n_runs = 0;         // runs of tokens of the residual kernel, run_rows each at most
  int run_rows = 0;
  int n_token_rows = 0;   // rows that are single decoded tokens (first in the list of rows)
  bool decode = false;    // every segment is one token
  size_t off_ids = 0, off_pos = 0, off_slots = 0, off_row_seg = 0, off_want = 0, off_seg = 0, off_short = 0,
         off_long = 0, off_chunk = 0, off_tile[kTileKinds] = {0}, off_row_list = 0, off_tables = 0, off_run = 0,
         off_expand_base = 0, off_expand_list = 0;
  LayeredPlans* plans = nullptr;
  TcGemmPlan* head_plan = nullptr;
  std::vector<TcGemmPlan>* expand_plans = nullptr;  // by layer
};

struct LayeredModel {
  LayeredSpec spec;
  std::vector<LayeredLayer> layers;
  void *embed = nullptr, *pos = nullptr;     // [vocab, width], [max_positions, width] engine dtype, dense rows
  LayeredLinear head;                        // [vocab (padded), width (padded)]
  float *final_norm = nullptr, *embed_norm = nullptr;
  float* ones = nullptr;                     // [streams] of 1
  int64_t Hp = 0;                            // width padded to a multiple of 8
  int64_t params = 0;                        // elements of all tensors
  int64_t row_cap = 0;                       // rows of the step buffers
  // buffers
  int64_t max_proj = 0;                      // widest projection row
  float* x = nullptr;                        // [rows, streams, width]
  void* h = nullptr;                         // [rows, Hp]
  // post_norm: the feed-forward's input [rows, Hp], a second x, results of the embedding and all layers
  // [layers + 1, row_cap, width]
  void* h2 = nullptr;
  float *x2 = nullptr, *results = nullptr;
  float* part_scale = nullptr;               // [rows, norm_groups]
  void *q_latent = nullptr, *q = nullptr;    // queries out of a latent: [rows, q_rank], [rows, heads * (dim + rot_dim)]
  void* proj = nullptr;                      // [rows, max_proj]
  void *attn = nullptr, *rec = nullptr;      // branch outputs before their output projection
  float* o = nullptr;                        // [rows, heads * vdim] recurrence outputs
  void* conv = nullptr;                      // [rows, channels] after the convolution
  void *latent_q = nullptr, *latent_o = nullptr;  // [rows, heads * (rank + rot_dim)], [rows, heads * rank]
  float *y1 = nullptr, *y2 = nullptr;        // [rows, Hp] sublayer outputs
  void *gu = nullptr, *act = nullptr;        // feed-forward
  void* hf = nullptr;                        // [logits rows, Hp] final normed rows
  float* cum = nullptr;                      // [rows, heads * dim] running log2 decay inside a chunk
  float* chunk_state = nullptr;              // [chunks, heads, dim, vdim]
  float* attn_part = nullptr;                // split partials of the per-token attention
  // mixture of experts: what the router decided, the rows of every expert side by side
  void *moe_x = nullptr, *moe_act = nullptr, *moe_y = nullptr;  // [places, Hp], [places, ffp], [places, Hp]
  void* moe_gu = nullptr;                    // fp32 engines: gate | up before the activation
  int32_t *moe_ids = nullptr, *moe_rank = nullptr, *moe_place = nullptr;  // [rows, picks]
  float* moe_weight = nullptr;               // [rows, picks]
  int64_t moe_places = 0;
  int32_t *moe_count = nullptr, *moe_first = nullptr, *moe_tiles = nullptr;
  int max_segs = 0, max_chunks = 0;
  std::vector<TileKind> tile_kinds;          // as the layers need them
  // contexts of prompts whose latents are expanded: the latents side by side, keys and values of all heads
  int64_t expand_blocks = 0;                 // capacity
  void *expand_latent = nullptr, *expand_kv = nullptr;
  std::map<int, std::vector<TcGemmPlan>> expand_plans;  // by rows bucket
  std::map<int, LayeredPlans> plans;         // by rows bucket
  std::map<int, TcGemmPlan> head_plans;      // by wanted-rows bucket
  std::map<int, LayeredGraph> graphs;        // by number of decoded sequences
  ~LayeredModel();
};

}  // namespace hb
