// Models described layer by layer: every layer has a mixer (attention, a gated linear
// recurrence, or both side by side) and possibly a feed-forward (one gated layer, or a mixture of
// them), over one or several residual streams held in fp32.  The mechanisms and their constants are
// data (LayeredSpec); a design's reader (latarax.cc, biberax.cc) turns its config.json and tensor
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
  // interleaved rotation of the first 2 * rotation.size() channels of queries and keys; the
  // angle of pair i is position * rotation[i]
  std::vector<double> rotation;
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
};

// `top` of the experts run for every token, weighted by the softmax over their router logits.
struct ExpertsSpec {
  int experts = 0, top = 0;         // 0: no mixture
  int64_t ff = 0;
  GatedAct act;
  std::string router, router_bias;
  std::string prefix;               // expert e: prefix + "<e>." + gate | up | down
};

// S_t = diag(a_t) S_(t-1) + k_t v_t^T, o_t = S_t^T q_t per head, fp32 state of [dim, vdim].
struct RecurrenceSpec {
  int heads = 0, dim = 0, vdim = 0;
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
};

// Rows of the layer's input projection that come from one checkpoint tensor.
struct ProjPart {
  std::string tensor;
  int64_t rows = 0;
  int64_t offset = 0;  // first column of the projection's output (a multiple of 8)
};

struct MixerSpec {
  bool has_attn = false, has_rec = false;
  AttentionSpec attn;
  RecurrenceSpec rec;
  // tensors: projections that read h, concatenated into one matrix
  ProjPart aq, ak, av, ag;                   // attention (ag: gate of the heads' outputs)
  ProjPart rq, rk, rv, rg, ra1;              // recurrence (ra1: low-rank decay)
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
  std::string embed, pos, final_norm, head;  // pos empty: no learned positions
  std::vector<LayerSpec> layers;
};

// Design readers: config.json (and, for sizes it does not give, tensor shapes) -> spec.
bool is_latarax(const Json& config);
int read_latarax(const Json& config, LayeredSpec* out);
bool is_biberax(const Json& config);
int read_biberax(const Json& config, LayeredSpec* out);

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
};

struct LayeredExperts {     // experts' matrices one after another; the expert every token passes through
  LayeredLinear gate_up, down;   // one expert's [2 * ffp, K] and [N, ffp]
  LayeredLinear shared_gate_up, shared_down;
  int64_t ffp = 0, shared_ffp = 0;
  int64_t ld() const { return ffp > shared_ffp ? ffp : shared_ffp; }  // row stride of the activations
  void* router = nullptr;        // [experts, width] engine dtype
  float* router_bias = nullptr;  // [experts]
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
  LayeredExperts moe;
  int kv_pool = -1;                          // index into hb_engine::kc / vc
  float* state = nullptr;                    // [slots, heads, dim, vdim]
  SublayerMix sub1, sub2;
};

// Plans of all matrix products for one bucket of batch rows.
struct LayeredPlans {
  std::vector<TcGemmPlan> proj, attn_o, rec_o, gate_up, down, moe_gate_up, moe_down;
};

struct LayeredGraph {
  cudaGraphExec_t exec = nullptr;
  int64_t launches = 0;
};

// Where a step's inputs lie in the (pinned and device) input block, and what it contains.
struct LayeredStep {
  int rows = 0, segs = 0, want = 0;
  int n_short = 0;        // segments the token-by-token recurrence kernel takes
  int n_chunks = 0;       // chunks of the longer segments (chunked recurrence kernels)
  int n_long = 0;         // longer segments
  int n_tiles = 0;        // query tiles of the tiled attention kernel
  int n_token_rows = 0;   // rows that are single decoded tokens (first in the list of rows)
  bool decode = false;    // every segment is one token
  size_t off_ids = 0, off_pos = 0, off_slots = 0, off_row_seg = 0, off_want = 0, off_seg = 0, off_short = 0,
         off_long = 0, off_chunk = 0, off_tile = 0, off_row_list = 0, off_tables = 0;
  LayeredPlans* plans = nullptr;
  TcGemmPlan* head_plan = nullptr;
};

struct LayeredModel {
  LayeredSpec spec;
  std::vector<LayeredLayer> layers;
  void *embed = nullptr, *pos = nullptr;     // [vocab, width], [max_positions, width] engine dtype, dense rows
  LayeredLinear head;                        // [vocab (padded), width (padded)]
  float* final_norm = nullptr;
  float* ones = nullptr;                     // [streams] of 1
  int64_t Hp = 0;                            // width padded to a multiple of 8
  int64_t params = 0;                        // elements of all tensors
  int64_t row_cap = 0;                       // rows of the step buffers
  // buffers
  int64_t max_proj = 0;                      // widest projection row
  float* x = nullptr;                        // [rows, streams, width]
  void* h = nullptr;                         // [rows, Hp]
  void* proj = nullptr;                      // [rows, max_proj]
  void *attn = nullptr, *rec = nullptr;      // branch outputs before their output projection
  float* o = nullptr;                        // [rows, heads * vdim] recurrence outputs
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
  int tile_positions = 0;                    // positions of an attention tile that suit every layer (0: no tiles)
  std::map<int, LayeredPlans> plans;         // by rows bucket
  std::map<int, TcGemmPlan> head_plans;      // by wanted-rows bucket
  std::map<int, LayeredGraph> graphs;        // by number of decoded sequences
  ~LayeredModel();
};

}  // namespace hb
