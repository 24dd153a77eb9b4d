// Launchers of the kernels the layered family is made of.  Every constant of a mechanism is a
// parameter; rows of a step belong to segments (StepSeg) and carry their position and KV slot.
#pragma once

#include "common.h"

namespace hb {

// One segment of a step on the device: rows [row0, row0 + n), positions pos0 .., state slot.
struct SegInfo {
  int32_t row0, n, pos0, slot;
};
// A chunk of a longer segment (chunked recurrence) or a tile of query positions (tiled
// attention): `n` consecutive rows from `row0`, part of segment `seg`; `index` counts the chunks of
// the segment from 0.
struct RowRange {
  int32_t seg, row0, n, index;
};

// ------------------------------------------------------------------ residual streams (streams.cu)
constexpr int kMaxStreams = 16;
// A norm's weight applies as norm_offset + norm (offset 1: stored around zero).
// x[r, s, :] = embed[ids[r]] * embed_scale + pos_table[pos[r]] for every stream s (fp32; pos_table null: no learned
// positions), then h[r] = rms(sum_s in[s] x[r, s]) * (offset + norm).
int streams_embed(cudaStream_t st, float* x, void* h, const void* embed, const void* pos_table, const uint32_t* ids,
                  const int32_t* pos, const float* in, const float* norm, float norm_offset, int64_t rows, int streams,
                  int64_t width, int64_t ld_h, int64_t vocab, int64_t max_positions, float eps, hb_dtype dtype,
                  float embed_scale = 1.f);
// One sublayer boundary: y (fp32 rows of stride ld_y) goes back into the streams,
//   x[r, t] = sum_s mix[s, t] x[r, s] + out[t] y[r],
// and the next sublayer's input is read: h[r] = rms(sum_t next_in[t] x[r, t]) * (offset + next_norm)
// (next_norm null: no further sublayer).  With y2, y is the mean of two branch outputs, each
// RMS-normed over the width with its plain weight: (rms(y) w1 + rms(y2) w2) / 2.  Else y may be null
// (nothing), `bias` [width] is added to it, and so are the outputs of the experts of a mixture:
//   sum_k expert_weight[r, k] * expert_y[expert_place[r, k]]   (rows of `dtype`, stride ld_y).
struct StreamMix {
  const float *mix, *out, *next_in, *next_norm;
  const float *w1 = nullptr, *w2 = nullptr;
  float norm_offset = 1.f;
  const float* bias = nullptr;
  const void* expert_y = nullptr;
  const int32_t* expert_place = nullptr;
  const float* expert_weight = nullptr;
  int top = 0;
};
int streams_mix(cudaStream_t st, float* x, void* h, const float* y, const float* y2, int64_t ld_y, const StreamMix& m,
                int64_t rows, int streams, int64_t width, int64_t ld_h, float eps, hb_dtype dtype);
// h[i] = rms(sum_s x[want[i], s]) * (offset + norm) * scale
int streams_final(cudaStream_t st, void* h, const float* x, const int32_t* want, const float* norm, float norm_offset,
                  int64_t n_want, int streams, int64_t width, int64_t ld_h, float eps, hb_dtype dtype, float scale = 1.f);
// out[r, g * size + i] = rms over the group of o[r, g, :] * weight * act(gate[r, g * size + i]), act = SiLU
// or sigmoid; with gate_first the product o * act(gate) is what is normed.  weight [size] is shared by
// the groups, or own_weights: [groups * size].
struct GroupNorm {
  int groups = 1, size = 0;
  bool gate_silu = true, gate_first = false, own_weights = false;
  float eps = 0.f;
};
int gated_group_norm(cudaStream_t st, void* out, int64_t ld_out, const float* o, int64_t ld_o, const void* gate,
                     int64_t ld_gate, const float* weight, int64_t rows, const GroupNorm& n, hb_dtype dtype);

// ------------------------------------- residual with normed sublayer outputs (residual.cu)
// Rows of `tiles` (runs of consecutive tokens of a segment that together are all rows of the step):
//   v = the output of a row: its embedding row, or y plus the weighted outputs of its experts (place -1:
//       the row of `input` itself);
//   x' = x + rms(v in `groups` equal parts of the width) * norm       (x null: zero) -> result
//   x' = sum_l depth[l] earlier[l] + depth[n_earlier] x'                (depth null: as it is) -> x_out
//   h = x' + sum_j conv[j] x'[t - (taps - 1) + j]                        (conv null: x')
// with zeros before the sequence's start.  x_out, result and h may be null; none of them is a buffer that
// is read here.  state [slots, taps - 1, width]: what earlier steps left of the convolution's inputs, the
// one of position p at entry p mod (taps - 1); past: the same of the convolution that read x, which is
// brought up to date here.
constexpr int kResidualMaxTaps = 32;
constexpr int kResidualRun = 16;       // most rows of a run where the step goes in two kernels
struct ResidualStep {
  const float* y = nullptr;            // rows of stride ld_y
  int64_t ld_y = 0;
  const void* expert_y = nullptr;      // rows of the step's dtype, stride ld_y
  const int32_t* expert_place = nullptr;
  const float* expert_weight = nullptr;
  int top = 0;
  const void* input = nullptr;
  int64_t ld_input = 0;
  const void* embed = nullptr;         // [vocab, width]
  const uint32_t* ids = nullptr;
  int64_t vocab = 0;
  const float* norm = nullptr;
  int groups = 1;
  float eps = 0.f;
  const float* x = nullptr;            // [rows, width]
  float *result = nullptr, *x_out = nullptr;
  const float* earlier = nullptr;      // n_earlier times [rows, width], `step` elements apart
  int64_t step = 0;
  int n_earlier = 0;
  const float* depth = nullptr;
  const float* conv = nullptr;         // [taps, width]
  int taps = 1;
  const float* state = nullptr;
  float* past = nullptr;
  void* h = nullptr;
  int64_t ld_h = 0;
  // With scale [rows, groups] and, for experts, mixed [rows, ld_y] (scratch) and up to four taps the step goes in two kernels, the faster form for
  // many rows: rows of the step, none of the runs longer than kResidualRun.
  float *scale = nullptr, *mixed = nullptr;
  int64_t rows = 0;
};
inline bool residual_in_two(const ResidualStep& a) { return a.scale && a.rows > 0 && a.taps <= 4 && (a.mixed || !a.top); }
int residual_step(cudaStream_t st, const ResidualStep& a, const RowRange* tiles, int n_tiles, const SegInfo* segs, int64_t width,
                  hb_dtype dtype);
// out[r] = rms of in[list ? list[r] : r] in `groups` parts of `size` channels * weight [groups * size]; in
// rows of `dtype`, or (in_f32) fp32.
int parts_norm(cudaStream_t st, void* out, int64_t ld_out, const void* in, int64_t ld_in, bool in_f32, const int32_t* list,
               const float* weight, int64_t rows, int groups, int64_t size, float eps, hb_dtype dtype);

// --------------------------------------------------------------- attention (attention_span.cu)
// Paged attention whose queries see the last `window` positions (0 = all) and the first
// `keep_first`, or (chunk > 0) the positions of their own chunk; keys and values of different
// widths.  Pools per layer: K [num_blocks, kv_heads, 16, dim], V [num_blocks, kv_heads, 16, vdim].
//   score(i, j) = cap(scale * q_i . k_j [* key_scale[slot of j]]) [+ dist_bias[h, min(i - j, dist_len - 1)]]
// with cap(s) = softcap * tanh(s / softcap), or s where softcap is 0.  Without a V pool (vc null) the
// values are the first vdim channels of the keys (a latent that both are made of); with key_scale
// [num_blocks * 16] the K pool then holds the values, and a key is its value times a scale of its own
// (a norm over the whole projection; the norm's weight is part of q).  sink [heads]: one more member of the softmax with this score and no value.  gate (row r,
// head h at gate + r * ld_gate + h * vdim): the output is multiplied by its sigmoid.  With gate_per_head
// a head has one number, at gate + r * ld_gate + h.
struct SpanAttention {
  const void* q = nullptr;     // row r, head h at q + r * ld_q + h * dim
  int64_t ld_q = 0;
  void* out = nullptr;         // row r, head h at out + r * ld_out + h * vdim
  int64_t ld_out = 0;
  void *kc = nullptr, *vc = nullptr;
  const int32_t* tables = nullptr;   // [segs, max_blocks]
  int64_t max_blocks = 0, num_blocks = 0;
  const int32_t* row_seg = nullptr;  // segment of a row
  const int32_t* pos = nullptr;      // position of a row
  int heads = 0, kv_heads = 0, dim = 0, vdim = 0, window = 0, keep_first = 0, chunk = 0;
  float scale = 1.f, softcap = 0.f;
  int slice = 0;               // query heads of a kv head that one CTA takes (set by the launchers)
  const float* key_scale = nullptr;
  const float* dist_bias = nullptr;  // [heads, dist_len]
  int dist_len = 0;
  const float* sink = nullptr;
  const void* gate = nullptr;
  int64_t ld_gate = 0;
  int gate_per_head = 0;
  // element of `gate` that meets channel c of a head
  __host__ __device__ __forceinline__ int64_t gate_at(int64_t row, int64_t head, int c) const {
    return row * ld_gate + (gate_per_head ? head : head * vdim + c);
  }
  // Where keys and values lie, in elements: token j of a block at block * step.block + head * step.head +
  // j * step.token (all zero: the pools above).  With `linear` tables holds one number per segment and
  // its blocks follow one another from there.  The last `tail` channels of every key are one vector per
  // token for all heads, rows of kt of stride ld_kt numbered like the tokens.  (span_attention_tiles only.)
  struct Steps {
    int64_t block = 0, head = 0, token = 0;
  } k_step, v_step;
  int linear = 0, tail = 0;
  const void* kt = nullptr;
  int64_t ld_kt = 0;
  int* err = nullptr;          // set to HB_ERR_TIMEOUT when a bounded wait inside a kernel ran out (may be null)
  // first position a query at `pos` sees besides the first keep_first
  __host__ __device__ __forceinline__ int first_seen(int pos) const {
    if (chunk > 0) return pos - pos % chunk;
    return window > 0 && pos >= window ? pos - window + 1 : 0;
  }
  // The query heads of a kv head are cut into equal slices (the last may be smaller) of at most `most`.
  void cut(int most) {
    const int R = heads / kv_heads, n = (R + most - 1) / most;
    slice = (R + n - 1) / n;
  }
  __host__ __device__ __forceinline__ int slices() const { return (heads / kv_heads + slice - 1) / slice; }
};
// The query heads one CTA takes: `n` of them from `first`, on kv head `kvh`; unit = blockIdx.y.
struct HeadSlice {
  int kvh, first, n;
  __device__ __forceinline__ HeadSlice(const SpanAttention& a, int unit) {
    const int R = a.heads / a.kv_heads, S = a.slices();
    kvh = unit / S;
    const int h0 = unit % S * a.slice;
    first = kvh * R + h0;
    n = min(a.slice, R - h0);
  }
};
// K/V of the step's rows to their slots (slot = block * 16 + offset; negative: skipped).
int span_kv_write(cudaStream_t st, const SpanAttention& a, const void* k, const void* v, int64_t ld_kv, const int64_t* slots,
                  int64_t rows, hb_dtype dtype);
// One CTA per (row of `row_list`, kv head): any dtype and any sizes.
int span_attention_rows(cudaStream_t st, const SpanAttention& a, const int32_t* row_list, int n_rows, hb_dtype dtype);

// Tensor-core forms (attention_span_mma.cu): prompt portions as tiles of up to
// span_attention_tile_positions() consecutive positions (0: these sizes are not taken) and decoded
// tokens as single rows, their keys split over n_splits CTAs when the rows alone leave SMs idle
// (`part`: n_rows * heads * n_splits * (vdim + 2) floats).
int span_attention_tile_positions(const SpanAttention& a, hb_dtype dtype);
// CTAs of the per-token kernel that are resident at once, and how many one row has (splits apart).
int span_attention_token_units(const SpanAttention& a);
int span_attention_tokens_slots(const SpanAttention& a);
bool span_attention_tokens_supported(const SpanAttention& a, hb_dtype dtype);
int span_attention_tiles(cudaStream_t st, const SpanAttention& a, const RowRange* tiles, int n_tiles);
int span_attention_tokens(cudaStream_t st, const SpanAttention& a, const int32_t* rows, int n_rows, int n_splits, float* part);
// Whether sizes and alignments suit the tensor-core kernels; the sum of a row's split partials.
bool span_attention_mma_ok(const SpanAttention& a, hb_dtype dtype);
int span_attention_merge(cudaStream_t st, const SpanAttention& a, const int32_t* rows, int n_rows, int n_splits, const float* part);
// Per-token kernel for wide values inside the keys (attention_latent.cu); span_attention_tokens takes it
// where it is supported.
bool latent_tokens_supported(const SpanAttention& a, hb_dtype dtype);
int latent_tokens_units(const SpanAttention& a);
int latent_tokens(cudaStream_t st, const SpanAttention& a, const int32_t* rows, int n_rows, int n_splits, float* part);

// ----------------------------------------------- queries and keys of a step (attention_prep.cu)
// One pass over projection rows: biases added, RMS norms over all query and all key rows, or a
// rotation of the first 2 * pairs channels of every head (channel 2i with 2i + 1, or with `halves`
// channel i with i + pairs); queries stay in their place (in `dtype`), keys and values go to their
// slots of the pools (kc null: queries only).  With key_scale the K pool takes the
// keys before their norm (they are the values as well), key_scale[slot] the norm's factor, and the
// queries are multiplied by the key norm's weight.
struct AttentionPrep {
  void* p = nullptr;
  int64_t ld = 0;
  int off_q = 0, off_k = 0, off_v = 0;
  int heads = 0, kv_heads = 0, dim = 0, vdim = 0;
  const int32_t* pos = nullptr;
  const int64_t* slots = nullptr;      // block * 16 + offset; negative: skipped
  void *kc = nullptr, *vc = nullptr;
  int64_t num_blocks = 0;
  const float *q_bias = nullptr, *k_bias = nullptr;
  const float *q_norm = nullptr, *k_norm = nullptr;
  float eps = 0.f;
  const double* rotation = nullptr;    // [pairs] frequencies
  int pairs = 0, halves = 0;
  float rotation_gain = 1.f;           // factor on sines and cosines
  float* key_scale = nullptr;
};
// Attention over a latent (no V pool; SpanAttention): row r of p holds the heads' queries of
// [dim | rot_dim] channels (head h at off_q + h * (dim + rot_dim)) and, from off_c on, the latent of
// `rank` channels and a key part of rot_dim channels that all heads share.  The latent is RMS-normed
// (weight norm), the key part rotated, and both go to the token's slot of kc [num_blocks, 16, rank +
// rot_dim]; the rotated parts of the queries go back to their place and to q, head h at q + r * ld_q + h *
// (rank + rot_dim) + rank.  With qs the queries lie there instead, head h of row r at qs + r * ld_qs + h * (dim +
// rot_dim).  (The other `rank` channels there come from a product of heads: W_uk^T on the first dim
// channels, so that a query meets the latent itself.)
struct LatentPrep {
  void* p = nullptr;
  int64_t ld = 0;
  int off_q = 0, off_c = 0;
  void* qs = nullptr;
  int64_t ld_qs = 0;
  int heads = 0, dim = 0, rot_dim = 0, rank = 0;
  void* q = nullptr;
  int64_t ld_q = 0;
  const int32_t* pos = nullptr;
  const int64_t* slots = nullptr;
  void* kc = nullptr;
  int64_t num_blocks = 0;
  const float* norm = nullptr;
  float eps = 0.f;
  const double* rotation = nullptr;    // [pairs]
  int pairs = 0, halves = 1;           // channel i with i + pairs, or (0) 2i with 2i + 1
  float rotation_gain = 1.f;
};
int latent_prepare(cudaStream_t st, const LatentPrep& a, int64_t rows, hb_dtype dtype);
// Rows of whole contexts side by side: block i of dst (16 rows of `width` elements) is block list[i] of pool.
int latent_gather(cudaStream_t st, void* dst, const void* pool, const int32_t* list, int n_blocks, int width, int64_t num_blocks,
                  hb_dtype dtype);
// dst [n, cols, rows] = src [n, rows, cols] transposed, elements of es bytes (2 or 4).
int transpose_matrices(cudaStream_t st, void* dst, const void* src, int64_t n, int64_t rows, int64_t cols, size_t es);
int attention_prepare(cudaStream_t st, const AttentionPrep& a, int64_t rows, hb_dtype dtype);
// out[h, d] = rel[bucket[d], h] (rel [buckets, heads]), d < dist_len
int expand_distance_bias(cudaStream_t st, float* out, const float* rel, const int32_t* bucket, int heads, int dist_len);

// ------------------------------------------------------- mixture of experts (moe_experts.cu)
constexpr int kMoeMaxExperts = 1024;
struct MoeRouting {
  int experts = 0, top = 0;
  int shared = 0;                      // 1: every row also goes to the further group (TcGroups), with weight 1
  // sigmoid: scores sigmoid(logit), the chosen ones divided by their sum as weights (else softmax over
  // the chosen logits); only experts of the `keep` best of `groups` equal groups of neighbours can be
  // chosen, a group counting the sum of its two largest scores
  int sigmoid = 0, groups = 1, keep = 1;
  // softmax_all: scores and weights are the softmax over all outputs, the choice is by score + correction
  // [experts + identity] (may be null)
  int softmax_all = 0;
  const float* correction = nullptr;
  int identity = 0;                    // router outputs behind the experts that hand the row on: place -1
  int m_pad = 0, max_tiles = 0;        // TcGroups
  int32_t *ids = nullptr, *rank = nullptr, *place = nullptr;  // [rows, picks()]
  float* weight = nullptr;             // [rows, picks()]
  int32_t* count = nullptr;            // [experts + 1], zero between calls
  int32_t* first = nullptr;            // [experts + shared] first place of an expert
  int32_t* tile_group = nullptr;       // [max_tiles]
  __host__ __device__ __forceinline__ int picks() const { return top + shared; }
  __host__ __device__ __forceinline__ int outputs() const { return experts + identity; }
};
// Router logits h . router^T (+ bias) in fp32; the `top` largest per row (the lower expert among
// equals), their weights, every chosen (row, expert) a rank among the expert's rows, and
// the batch tiles of the experts: expert e has tiles of m_pad places from first[e] on.
int moe_route_top(cudaStream_t st, const MoeRouting& m, const void* h, int64_t ld_h, const void* router, const float* bias,
                  int64_t rows, int64_t width, hb_dtype dtype);
// place[r, k] = first[expert] + rank (-1: no expert, the row itself), and row r of h goes to these places of x (rows of ld elements).
int moe_gather(cudaStream_t st, const MoeRouting& m, void* x, const void* h, int64_t ld, int64_t rows, hb_dtype dtype);

// ------------------------------------------------------------ linear recurrence (recurrence.cu)
struct Recurrence {
  const void* p = nullptr;     // projection rows: q, k, v (and the low-rank decay input) at offsets
  int64_t ld = 0;
  int off_q = 0, off_k = 0, off_v = 0, off_a1 = 0;
  int heads = 0, dim = 0, vdim = 0;
  float q_scale = 1.f;
  int silu_qkv = 0;
  const float* decay = nullptr;      // [heads] constant decay, or null:
  const float* a2 = nullptr;         // [heads * dim, rank] low-rank decay
  const float* a2_bias = nullptr;    // [heads * dim]
  int rank = 0;
  float inv_tau = 1.f;
  // Or a decay per token and head (selective state space): a step t = softplus(dt + dt_bias), decay
  // exp(-exp(a_log) t), keys scaled by t, and skip * v added to the output.  dt: row r at dt + r * ld_dt
  // ([heads] of the rows' dtype); dt_bias, a_log, skip [heads].
  const void* dt = nullptr;
  int64_t ld_dt = 0;
  const float *dt_bias = nullptr, *a_log = nullptr, *skip = nullptr;
  int qk_heads = 0;            // heads of q and k, each serving heads / qk_heads neighbours (0: one each)
  float* state = nullptr;            // [slots, heads, dim, vdim]
  float* o = nullptr;                // [rows, heads * vdim]
  int64_t ld_o = 0;
  const SegInfo* segs = nullptr;
  __host__ __device__ __forceinline__ int qk(int h) const { return qk_heads ? h / (heads / qk_heads) : h; }
};
// Token by token, state in and out of HBM once per segment where it fits the registers:
// decoded tokens and short portions.  `list` holds segment numbers.
int recurrence_tokens(cudaStream_t st, const Recurrence& a, const int32_t* list, int n_list, hb_dtype dtype);

// Prompt portions in chunks of kRecChunk tokens on tensor cores (recurrence_chunk.cu, bf16
// projections): every chunk's own contribution to the state, a scan over the chunks of a segment,
// every chunk's outputs.  Chunks of a segment are neighbours in `chunks`.
constexpr int kRecChunk = 64;
struct RecurrenceChunks {
  const RowRange* chunks = nullptr;   // device
  int n_chunks = 0;
  const RowRange* segs = nullptr;     // longer segments: seg, first chunk (row0), number of chunks (n)
  int n_segs = 0;
  // running log2 decay inside a chunk: [rows, heads * dim]; of a decay per token [rows, heads] and,
  // behind them in the row, the steps
  float* cum = nullptr;
  float* state = nullptr;             // [n_chunks, heads, dim, vdim]
};
// Floats of a row of RecurrenceChunks::cum.
inline int64_t recurrence_cum_width(const Recurrence& a) {
  return a.dt ? 2 * (int64_t)a.heads : a.decay ? 0 : (int64_t)a.heads * a.dim;
}
bool recurrence_chunks_supported(const Recurrence& a, hb_dtype dtype);
int recurrence_chunks(cudaStream_t st, const Recurrence& a, const RecurrenceChunks& c, int64_t* launches);

// ---------------------------------------------------- causal convolution per channel (conv.cu)
// out = SiLU(bias + sum_j w[j] x[t - (taps - 1) + j]) over the tokens of a sequence, zeros before its
// start.  The last taps - 1 inputs of every sequence stay in its state slot.
constexpr int kConvMaxTaps = kRecChunk + 1;
struct ShortConv {
  const void* p = nullptr;     // row r, channel c at p + r * ld + off + c
  int64_t ld = 0;
  int off = 0, channels = 0, taps = 0;
  const float *w = nullptr, *bias = nullptr;  // [taps, channels], [channels]
  void* out = nullptr;         // row r, channel c at out + r * ld_out + c
  int64_t ld_out = 0;
  void* state = nullptr;       // [slots, taps - 1, channels]
  const SegInfo* segs = nullptr;
};
// Every segment of the step is either in `list` (as a whole: up to kRecChunk tokens) or cut into
// `chunks` of kRecChunk tokens.
int short_conv(cudaStream_t st, const ShortConv& a, const int32_t* list, int n_list, const RowRange* chunks, int n_chunks,
               hb_dtype dtype);

}  // namespace hb
