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
// x[r, s, :] = embed[ids[r]] + pos_table[pos[r]] for every stream s (fp32; pos_table null: no learned
// positions), then h[r] = rms(sum_s in[s] x[r, s]) * (offset + norm).
int streams_embed(cudaStream_t st, float* x, void* h, const void* embed, const void* pos_table, const uint32_t* ids,
                  const int32_t* pos, const float* in, const float* norm, float norm_offset, int64_t rows, int streams,
                  int64_t width, int64_t ld_h, int64_t vocab, int64_t max_positions, float eps, hb_dtype dtype);
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
// h[i] = rms(sum_s x[want[i], s]) * (offset + norm)
int streams_final(cudaStream_t st, void* h, const float* x, const int32_t* want, const float* norm, float norm_offset,
                  int64_t n_want, int streams, int64_t width, int64_t ld_h, float eps, hb_dtype dtype);
// out[r, g * size + i] = rms over the group of o[r, g, :] * weight * act(gate[r, g * size + i]);
// weight [size] is shared by the groups; act = SiLU or sigmoid.
int gated_group_norm(cudaStream_t st, void* out, int64_t ld_out, const float* o, int64_t ld_o, const void* gate,
                     int64_t ld_gate, const float* weight, int64_t rows, int groups, int size, bool gate_silu, float eps,
                     hb_dtype dtype);

// --------------------------------------------------------------- attention (attention_span.cu)
// Paged attention whose queries see the last `window` positions (0 = all) and the first
// `keep_first`, or (chunk > 0) the positions of their own chunk; keys and values of different
// widths.  Pools per layer: K [num_blocks, kv_heads, 16, dim], V [num_blocks, kv_heads, 16, vdim].
//   score(i, j) = scale * q_i . k_j [* key_scale[slot of j]] [+ dist_bias[h, min(i - j, dist_len - 1)]]
// With key_scale [num_blocks * 16] the K pool holds the values too (vc null, vdim == dim): a key is
// its value times a scale of its own (a norm over the whole projection; the norm's weight is part
// of q).  sink [heads]: one more member of the softmax with this score and no value.  gate (row r,
// head h at gate + r * ld_gate + h * vdim): the output is multiplied by its sigmoid.
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
  float scale = 1.f;
  const float* key_scale = nullptr;
  const float* dist_bias = nullptr;  // [heads, dist_len]
  int dist_len = 0;
  const float* sink = nullptr;
  const void* gate = nullptr;
  int64_t ld_gate = 0;
  // first position a query at `pos` sees besides the first keep_first
  __host__ __device__ __forceinline__ int first_seen(int pos) const {
    if (chunk > 0) return pos - pos % chunk;
    return window > 0 && pos >= window ? pos - window + 1 : 0;
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
// CTAs of the per-token kernel that are resident at once.
int span_attention_tokens_slots(const SpanAttention& a);
bool span_attention_tokens_supported(const SpanAttention& a, hb_dtype dtype);
int span_attention_tiles(cudaStream_t st, const SpanAttention& a, const RowRange* tiles, int n_tiles);
int span_attention_tokens(cudaStream_t st, const SpanAttention& a, const int32_t* rows, int n_rows, int n_splits, float* part);

// ----------------------------------------------- queries and keys of a step (attention_prep.cu)
// One pass over projection rows: biases added, RMS norms over all query and all key rows, or an
// interleaved rotation of the first 2 * pairs channels of every head; queries stay in their place
// (in `dtype`), keys and values go to their slots of the pools.  With key_scale the K pool takes the
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
  int pairs = 0;
  float* key_scale = nullptr;
};
int attention_prepare(cudaStream_t st, const AttentionPrep& a, int64_t rows, hb_dtype dtype);
// out[h, d] = rel[bucket[d], h] (rel [buckets, heads]), d < dist_len
int expand_distance_bias(cudaStream_t st, float* out, const float* rel, const int32_t* bucket, int heads, int dist_len);

// ------------------------------------------------------- mixture of experts (moe_experts.cu)
constexpr int kMoeMaxExperts = 1024;
struct MoeRouting {
  int experts = 0, top = 0;
  int shared = 0;                      // 1: every row also goes to the further group (TcGroups), with weight 1
  int m_pad = 0, max_tiles = 0;        // TcGroups
  int32_t *ids = nullptr, *rank = nullptr, *place = nullptr;  // [rows, picks()]
  float* weight = nullptr;             // [rows, picks()]
  int32_t* count = nullptr;            // [experts + 1], zero between calls
  int32_t* first = nullptr;            // [experts + shared] first place of an expert
  int32_t* tile_group = nullptr;       // [max_tiles]
  __host__ __device__ __forceinline__ int picks() const { return top + shared; }
};
// Router logits h . router^T + bias in fp32; the `top` largest per row (the lower expert among
// equals), their softmax as weights, every chosen (row, expert) a rank among the expert's rows, and
// the batch tiles of the experts: expert e has tiles of m_pad places from first[e] on.
int moe_route_top(cudaStream_t st, const MoeRouting& m, const void* h, int64_t ld_h, const void* router, const float* bias,
                  int64_t rows, int64_t width, hb_dtype dtype);
// place[r, k] = first[expert] + rank, and row r of h goes to these places of x (rows of ld elements).
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
  float* state = nullptr;            // [slots, heads, dim, vdim]
  float* o = nullptr;                // [rows, heads * vdim]
  int64_t ld_o = 0;
  const SegInfo* segs = nullptr;
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
  float* cum = nullptr;               // [rows, heads * dim] running log2 decay inside a chunk
  float* state = nullptr;             // [n_chunks, heads, dim, vdim]
};
bool recurrence_chunks_supported(const Recurrence& a, hb_dtype dtype);
int recurrence_chunks(cudaStream_t st, const Recurrence& a, const RecurrenceChunks& c, int64_t* launches);

}  // namespace hb
