// Public entry points of the layered models' mechanisms.
#include "gemm.h"
#include "layered_ops.h"

namespace hb {

static SpanAttention span_of(const hb_span_attention_args* p) {
  SpanAttention a;
  a.q = p->q; a.ld_q = p->ld_q; a.out = p->out; a.ld_out = p->ld_out;
  a.kc = p->k_cache; a.vc = p->v_cache;
  a.tables = p->block_tables; a.max_blocks = p->max_blocks; a.num_blocks = p->num_blocks;
  a.row_seg = p->row_segment; a.pos = p->positions;
  a.heads = p->heads; a.kv_heads = p->kv_heads; a.dim = p->dim; a.vdim = p->vdim;
  a.window = p->window; a.keep_first = p->keep_first; a.chunk = p->chunk; a.scale = p->scale;
  a.key_scale = p->key_scale; a.dist_bias = p->dist_bias; a.dist_len = p->dist_len; a.sink = p->sink;
  a.gate = p->gate; a.ld_gate = p->ld_gate;
  a.softcap = p->softcap;
  a.gate_per_head = p->gate_per_head;
  if (a.key_scale) a.vc = nullptr;
  return a;
}

static int check_span(const hb_span_attention_args* p) {
  HB_CHECK_ARG(p && p->k_cache, "span attention: null argument");
  HB_CHECK_ARG(p->heads > 0 && p->kv_heads > 0 && p->heads % p->kv_heads == 0 && p->dim > 0 && p->vdim > 0,
               "span attention: bad sizes");
  HB_CHECK_ARG(p->window >= 0 && p->keep_first >= 0 && p->chunk >= 0 && p->num_blocks > 0, "span attention: bad window or pool");
  HB_CHECK_ARG(p->v_cache || p->vdim <= p->dim, "span attention: values inside the keys are no wider than they are");
  HB_CHECK_ARG(p->softcap >= 0.f, "span attention: a negative cap");
  HB_CHECK_ARG(!p->key_scale || p->dim == p->vdim, "span attention: keys that are the values have their width");
  HB_CHECK_ARG(!p->dist_bias || p->dist_len > 0, "span attention: an empty bias table");
  return HB_OK;
}

static Recurrence recurrence_of(const hb_linear_recurrence_args* p) {
  Recurrence a;
  a.p = p->p; a.ld = p->ld;
  a.off_q = p->off_q; a.off_k = p->off_k; a.off_v = p->off_v; a.off_a1 = p->off_a1;
  a.heads = p->heads; a.dim = p->dim; a.vdim = p->vdim;
  a.q_scale = p->q_scale; a.silu_qkv = p->silu_qkv;
  a.decay = p->decay; a.a2 = p->a2; a.a2_bias = p->a2_bias;
  a.rank = p->decay ? 0 : p->rank;
  a.inv_tau = p->decay ? 1.f : (float)(1.0 / p->tau);
  a.state = p->state; a.o = p->o; a.ld_o = p->ld_o;
  a.segs = (const SegInfo*)p->segments;
  a.dt = p->dt; a.ld_dt = p->ld_dt; a.dt_bias = p->dt_bias; a.a_log = p->a_log; a.skip = p->skip; a.qk_heads = p->qk_heads;
  if (a.dt) { a.decay = nullptr; a.rank = 0; a.inv_tau = 1.f; }
  return a;
}

}  // namespace hb

extern "C" {

int hb_span_attention_tile_positions(const hb_span_attention_args* a, hb_dtype dtype) {
  int rc = hb::check_span(a);
  return rc ? rc : hb::span_attention_tile_positions(hb::span_of(a), dtype);
}

int hb_span_attention(void* stream, const hb_span_attention_args* p, const int32_t* tiles, int n_tiles, const int32_t* rows,
                      int n_rows, int n_splits, float* workspace, hb_dtype dtype) {
  int rc = hb::check_span(p);
  if (rc) return rc;
  HB_CHECK_ARG(p->q && p->out && p->block_tables && p->row_segment && p->positions && p->max_blocks > 0,
               "hb_span_attention: null argument");
  HB_CHECK_ARG((tiles || n_tiles == 0) && (rows || n_rows == 0) && n_tiles >= 0 && n_rows >= 0, "hb_span_attention: bad lists");
  HB_CHECK_ARG(n_splits >= 1 && n_splits <= 64 && (n_splits == 1 || workspace), "hb_span_attention: bad splits");
  const hb::SpanAttention a = hb::span_of(p);
  auto st = (cudaStream_t)stream;
  if (n_tiles) {
    HB_CHECK_ARG(hb::span_attention_tile_positions(a, dtype) > 0, "hb_span_attention: these sizes do not go as tiles");
    if ((rc = hb::span_attention_tiles(st, a, (const hb::RowRange*)tiles, n_tiles))) return rc;
  }
  if (hb::span_attention_tokens_supported(a, dtype)) return hb::span_attention_tokens(st, a, rows, n_rows, n_splits, workspace);
  return hb::span_attention_rows(st, a, rows, n_rows, dtype);
}

int hb_span_kv_write(void* stream, const hb_span_attention_args* p, const void* k, const void* v, int64_t ld,
                     const int64_t* slots, int64_t rows, hb_dtype dtype) {
  int rc = hb::check_span(p);
  if (rc) return rc;
  HB_CHECK_ARG(k && v && slots && rows >= 0 && p->v_cache, "hb_span_kv_write: null argument");
  return rows ? hb::span_kv_write((cudaStream_t)stream, hb::span_of(p), k, v, ld, slots, rows, dtype) : HB_OK;
}

int hb_linear_recurrence_chunked(const hb_linear_recurrence_args* a, hb_dtype dtype) {
  HB_CHECK_ARG(a, "hb_linear_recurrence_chunked: null argument");
  return hb::recurrence_chunks_supported(hb::recurrence_of(a), dtype) ? 1 : 0;
}

int hb_linear_recurrence(void* stream, const hb_linear_recurrence_args* p, const int32_t* list, int n_list,
                         const int32_t* chunks, int n_chunks, const int32_t* long_segments, int n_long, float* cum,
                         float* chunk_state, hb_dtype dtype) {
  HB_CHECK_ARG(p && p->p && p->state && p->o && p->segments, "hb_linear_recurrence: null argument");
  HB_CHECK_ARG(p->heads > 0 && p->dim > 0 && p->vdim > 0, "hb_linear_recurrence: bad sizes");
  HB_CHECK_ARG(p->qk_heads >= 0 && (!p->qk_heads || p->heads % p->qk_heads == 0), "hb_linear_recurrence: bad heads of q and k");
  HB_CHECK_ARG(p->dt ? p->dt_bias && p->a_log : p->decay || (p->a2 && p->a2_bias && p->rank > 0 && p->tau > 0.f), "hb_linear_recurrence: no decay");
  const hb::Recurrence a = hb::recurrence_of(p);
  auto st = (cudaStream_t)stream;
  int rc = hb::recurrence_tokens(st, a, list, n_list, dtype);
  if (rc || n_chunks == 0) return rc;
  HB_CHECK_ARG(chunks && long_segments && n_long > 0 && chunk_state && (p->decay || cum), "hb_linear_recurrence: bad chunk lists");
  HB_CHECK_ARG(hb::recurrence_chunks_supported(a, dtype), "hb_linear_recurrence: these sizes do not go in chunks");
  hb::RecurrenceChunks c;
  c.chunks = (const hb::RowRange*)chunks; c.n_chunks = n_chunks;
  c.segs = (const hb::RowRange*)long_segments; c.n_segs = n_long;
  c.cum = cum; c.state = chunk_state;
  int64_t launches = 0;
  return hb::recurrence_chunks(st, a, c, &launches);
}

int hb_streams_embed(void* stream, float* x, void* h, const void* embed, const void* pos_table, const uint32_t* ids,
                     const int32_t* positions, const float* in, const float* norm, int64_t rows, int streams, int64_t width,
                     int64_t ld_h, int64_t vocab, int64_t max_positions, float eps, hb_dtype dtype) {
  HB_CHECK_ARG(x && h && embed && pos_table && ids && positions && in && norm, "hb_streams_embed: null argument");
  HB_CHECK_ARG(rows >= 0 && streams > 0 && width > 0 && vocab > 0 && max_positions > 0, "hb_streams_embed: bad shape");
  if (rows == 0) return HB_OK;
  return hb::streams_embed((cudaStream_t)stream, x, h, embed, pos_table, ids, positions, in, norm, 1.f, rows, streams, width, ld_h,
                           vocab, max_positions, eps, dtype);
}

int hb_streams_mix(void* stream, float* x, void* h, const float* y, const float* y2, int64_t ld_y, const float* mix,
                   const float* out, const float* next_in, const float* next_norm, const float* w1, const float* w2,
                   int64_t rows, int streams, int64_t width, int64_t ld_h, float eps, hb_dtype dtype) {
  HB_CHECK_ARG(x && y && mix && out && (!next_norm || (next_in && h)) && (!y2 || (w1 && w2)), "hb_streams_mix: null argument");
  HB_CHECK_ARG(rows >= 0 && width > 0, "hb_streams_mix: bad shape");
  if (rows == 0) return HB_OK;
  hb::StreamMix m;
  m.mix = mix; m.out = out; m.next_in = next_in; m.next_norm = next_norm; m.w1 = w1; m.w2 = w2;
  return hb::streams_mix((cudaStream_t)stream, x, h, y, y2, ld_y, m, rows, streams, width, ld_h, eps, dtype);
}

int hb_streams_mix_ex(void* stream, float* x, void* h, const float* y, const float* y2, int64_t ld_y,
                      const hb_stream_mix_args* a, int64_t rows, int streams, int64_t width, int64_t ld_h, float eps,
                      hb_dtype dtype) {
  HB_CHECK_ARG(x && a && a->mix && a->out && (!a->next_norm || (a->next_in && h)), "hb_streams_mix_ex: null argument");
  HB_CHECK_ARG(!y2 || (y && a->w1 && a->w2 && !a->bias && !a->top), "hb_streams_mix_ex: bad second branch");
  HB_CHECK_ARG(rows >= 0 && width > 0 && a->top >= 0 && (!a->top || (a->expert_y && a->expert_place && a->expert_weight)),
               "hb_streams_mix_ex: bad shape");
  if (rows == 0) return HB_OK;
  hb::StreamMix m;
  m.mix = a->mix; m.out = a->out; m.next_in = a->next_in; m.next_norm = a->next_norm; m.w1 = a->w1; m.w2 = a->w2;
  m.norm_offset = a->norm_offset; m.bias = a->bias;
  m.expert_y = a->expert_y; m.expert_place = a->expert_place; m.expert_weight = a->expert_weight; m.top = a->top;
  return hb::streams_mix((cudaStream_t)stream, x, h, y, y2, ld_y, m, rows, streams, width, ld_h, eps, dtype);
}

int hb_attention_prepare(void* stream, const hb_attention_prep_args* p, int64_t rows, hb_dtype dtype) {
  HB_CHECK_ARG(p && p->p && p->positions && p->slots && (!p->k_cache || p->v_cache || p->key_scale) && rows >= 0,
               "hb_attention_prepare: null argument");
  HB_CHECK_ARG(p->heads > 0 && p->kv_heads > 0 && p->heads % p->kv_heads == 0 && p->dim > 0 && p->vdim > 0 && p->num_blocks > 0 &&
               p->pairs >= 0 && (p->pairs == 0 || p->rotation), "hb_attention_prepare: bad sizes");
  hb::AttentionPrep a;
  a.p = p->p; a.ld = p->ld;
  a.off_q = p->off_q; a.off_k = p->off_k; a.off_v = p->off_v;
  a.heads = p->heads; a.kv_heads = p->kv_heads; a.dim = p->dim; a.vdim = p->vdim;
  a.pos = p->positions; a.slots = p->slots; a.kc = p->k_cache; a.vc = p->v_cache; a.num_blocks = p->num_blocks;
  a.q_bias = p->q_bias; a.k_bias = p->k_bias; a.q_norm = p->q_norm; a.k_norm = p->k_norm; a.eps = p->eps;
  a.rotation = p->rotation; a.pairs = p->pairs; a.key_scale = p->key_scale;
  a.halves = p->halves; a.rotation_gain = p->rotation_gain == 0.f ? 1.f : p->rotation_gain;
  return hb::attention_prepare((cudaStream_t)stream, a, rows, dtype);
}

int hb_latent_prepare(void* stream, const hb_latent_prep_args* p, int64_t rows, hb_dtype dtype) {
  HB_CHECK_ARG(p && p->p && p->q && p->positions && p->slots && p->k_cache && p->norm && rows >= 0, "hb_latent_prepare: null argument");
  HB_CHECK_ARG(p->heads > 0 && p->dim > 0 && p->rot_dim >= 0 && p->rank > 0 && p->num_blocks > 0 && p->pairs >= 0 &&
               (p->pairs == 0 || p->rotation), "hb_latent_prepare: bad sizes");
  hb::LatentPrep a;
  a.p = p->p; a.ld = p->ld; a.off_q = p->off_q; a.off_c = p->off_c;
  a.heads = p->heads; a.dim = p->dim; a.rot_dim = p->rot_dim; a.rank = p->rank;
  a.q = p->q; a.ld_q = p->ld_q; a.pos = p->positions; a.slots = p->slots; a.kc = p->k_cache; a.num_blocks = p->num_blocks;
  a.norm = p->norm; a.eps = p->eps; a.rotation = p->rotation; a.pairs = p->pairs;
  a.rotation_gain = p->rotation_gain == 0.f ? 1.f : p->rotation_gain;
  a.qs = p->q_rows; a.ld_qs = p->ld_q_rows; a.halves = p->neighbours ? 0 : 1;
  return hb::latent_prepare((cudaStream_t)stream, a, rows, dtype);
}

int hb_gemm_heads(void* stream, void* Y, const void* X, const void* W, int64_t M, int64_t N, int64_t K, int heads, int64_t ldx,
                  int64_t x_step, int64_t ldy, int64_t y_step, hb_dtype dtype) {
  HB_CHECK_ARG(Y && X && W && M >= 0 && N > 0 && K > 0 && heads > 0, "hb_gemm_heads: bad argument");
  hb::TcHeads h;
  h.heads = heads; h.ldx = ldx; h.x_step = x_step; h.ldy = ldy; h.y_step = y_step;
  auto st = (cudaStream_t)stream;
  auto al = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 15) == 0; };
  if (M && hb::gemm_tc_supported(M, N, K, dtype) && hb::gemm_tc_heads_supported(N, K, false, h) && al(X) && al(W) && al(Y)) {
    int dev = 0;
    HB_CUDA_CHECK(cudaGetDevice(&dev));
    hb::TcGemmPlan plan;
    int rc = hb::gemm_tc_plan(&plan, X, W, M, N, K, hb::kEpiStore, false, dev, 0, nullptr, &h);
    return rc ? rc : hb::gemm_tc_run(plan, st, Y, ldy, nullptr, nullptr);
  }
  return hb::gemm_simt_heads(st, Y, X, W, M, N, K, dtype, false, h);
}

int hb_short_conv(void* stream, const hb_short_conv_args* p, const int32_t* list, int n_list, const int32_t* chunks, int n_chunks,
                  hb_dtype dtype) {
  HB_CHECK_ARG(p && p->p && p->w && p->bias && p->out && p->segments && (p->state || p->taps == 1), "hb_short_conv: null argument");
  HB_CHECK_ARG(n_list >= 0 && n_chunks >= 0 && (list || !n_list) && (chunks || !n_chunks), "hb_short_conv: bad lists");
  hb::ShortConv a;
  a.p = p->p; a.ld = p->ld; a.off = p->off; a.channels = p->channels; a.taps = p->taps; a.w = p->w; a.bias = p->bias;
  a.out = p->out; a.ld_out = p->ld_out; a.state = p->state; a.segs = (const hb::SegInfo*)p->segments;
  return hb::short_conv((cudaStream_t)stream, a, list, n_list, (const hb::RowRange*)chunks, n_chunks, dtype);
}

static hb::MoeRouting routing_of(const hb_moe_routing* p) {
  hb::MoeRouting m;
  m.experts = p->experts; m.top = p->top; m.shared = p->shared ? 1 : 0; m.m_pad = p->m_pad; m.max_tiles = p->max_tiles;
  m.ids = p->ids; m.rank = p->rank; m.place = p->place; m.weight = p->weight;
  m.count = p->count; m.first = p->first; m.tile_group = p->tile_group;
  m.sigmoid = p->sigmoid;
  if (p->groups) { m.groups = p->groups; m.keep = p->keep; }
  m.identity = p->identity; m.softmax_all = p->softmax_all; m.correction = p->correction;
  return m;
}

int hb_moe_route_top(void* stream, const hb_moe_routing* m, const void* h, int64_t ld_h, const void* router,
                     const float* bias, int64_t rows, int64_t width, hb_dtype dtype) {
  HB_CHECK_ARG(m && h && router && m->ids && m->rank && m->weight && m->count && m->first && m->tile_group,
               "hb_moe_route_top: null argument");
  HB_CHECK_ARG(m->identity >= 0, "hb_moe_route_top: a negative number of identities");
  HB_CHECK_ARG(rows >= 0 && width > 0 && m->m_pad > 0 &&
               m->max_tiles >= (rows * m->top < m->experts ? rows * m->top : m->experts) + rows * m->top / m->m_pad +
                                   (m->shared ? (rows + m->m_pad - 1) / m->m_pad : 0),
               "hb_moe_route_top: bad shape");
  return hb::moe_route_top((cudaStream_t)stream, routing_of(m), h, ld_h, router, bias, rows, width, dtype);
}

int hb_moe_gather(void* stream, const hb_moe_routing* m, void* x, const void* h, int64_t ld, int64_t rows, hb_dtype dtype) {
  HB_CHECK_ARG(m && x && h && m->ids && m->rank && m->place && m->first && ld > 0 && rows >= 0, "hb_moe_gather: null argument");
  return hb::moe_gather((cudaStream_t)stream, routing_of(m), x, h, ld, rows, dtype);
}

static hb::GatedAct act_of(const hb_gated_act_spec* p) {
  hb::GatedAct a;
  a.slope = p->slope; a.cubic = p->cubic; a.limit = p->limit; a.shift = p->shift;
  a.form = p->form; a.single = p->single;
  return a;
}

static int check_act(const hb_gated_act_spec* p) {
  HB_CHECK_ARG(p->form >= HB_ACT_LOGISTIC && p->form <= HB_ACT_TANH && (p->form != HB_ACT_TANH || p->single),
               "activation: unknown form %d", p->form);
  return HB_OK;
}

int hb_gated_act(void* stream, void* out, const void* gate_up, int64_t M, int64_t inter, const hb_gated_act_spec* act,
                 hb_dtype dtype) {
  HB_CHECK_ARG(out && gate_up && act && M >= 0 && inter > 0, "hb_gated_act: bad argument");
  if (int rc = check_act(act)) return rc;
  return hb::gated_act((cudaStream_t)stream, out, gate_up, M, inter, act_of(act), dtype);
}

static hb::TcGroups groups_of(const hb_grouped_gemm* p) {
  hb::TcGroups g;
  g.groups = p->groups; g.m_pad = p->m_pad; g.max_tiles = p->max_tiles; g.likely_tiles = p->likely_tiles;
  g.ldx = p->ldx; g.ldy = p->ldy;
  g.shared_w = p->shared_w; g.shared_n = p->shared_n; g.shared_k = p->shared_k;
  if (p->shared_w) g.shared_act = act_of(&p->shared_act);
  return g;
}

static int check_grouped(const hb_grouped_gemm* p) {
  HB_CHECK_ARG(p && p->tile_group && p->groups > 0 && p->N > 0 && p->K > 0 && p->m_pad > 0 && p->max_tiles > 0 &&
               p->likely_tiles > 0 && p->ldx >= p->K && (!p->shared_w || (p->shared_n > 0 && p->shared_k > 0 && p->ldx >= p->shared_k)),
               "grouped gemm: bad argument");
  HB_CHECK_ARG(!p->shared_w || !p->act.single == !p->shared_act.single, "grouped gemm: one activation with a gate, one without");
  return check_act(&p->act);
}

int hb_gemm_grouped(void* stream, void* Y, const void* X, const void* W, const hb_grouped_gemm* p, hb_dtype dtype) {
  int rc = check_grouped(p);
  if (rc) return rc;
  const int64_t wide = p->shared_n > p->N ? p->shared_n : p->N;
  HB_CHECK_ARG(Y && X && W && p->ldy >= (p->gated && !p->act.single ? wide / 2 : wide), "hb_gemm_grouped: bad output");
  const hb::TcGroups g = groups_of(p);
  const int64_t M = (int64_t)p->max_tiles * p->m_pad;
  auto st = (cudaStream_t)stream;
  if (hb::gemm_tc_supported(M, p->N, p->K, dtype) && p->m_pad % 16 == 0) {
    int dev = 0;
    HB_CUDA_CHECK(cudaGetDevice(&dev));
    hb::TcGemmPlan plan;
    rc = hb::gemm_tc_plan(&plan, X, W, M, p->N, p->K, !p->gated ? hb::kEpiStore : p->act.single ? hb::kEpiAct : hb::kEpiSwiGLU, p->out_f32 != 0, dev, 0, &g);
    if (rc) return rc;
    if (p->gated) plan.act = act_of(&p->act);
    return hb::gemm_tc_run(plan, st, Y, p->ldy, nullptr, nullptr, nullptr, p->tile_group);
  }
  HB_CHECK_ARG(!p->gated, "hb_gemm_grouped: the gated form runs on tensor cores (bf16, K %% 8 == 0)");
  return hb::gemm_simt_grouped(st, Y, X, W, p->N, p->K, dtype, p->out_f32 != 0, g, p->tile_group);
}

int hb_gated_act_grouped(void* stream, void* out, const void* gate_up, int64_t ld_gu, const hb_grouped_gemm* p, hb_dtype dtype) {
  int rc = check_grouped(p);
  if (rc) return rc;
  const int per = p->act.single ? 1 : 2;
  HB_CHECK_ARG(out && gate_up && ld_gu >= p->N && ld_gu >= p->shared_n && p->ldy >= p->N / per && p->ldy >= p->shared_n / per,
               "hb_gated_act_grouped: bad argument");
  return hb::gated_act_grouped((cudaStream_t)stream, out, p->ldy, gate_up, ld_gu, p->N / per, act_of(&p->act), dtype, groups_of(p),
                               p->tile_group);
}

int hb_residual_step(void* stream, const hb_residual_args* p, const int32_t* tiles, int n_tiles, const int32_t* segments,
                     int64_t width, hb_dtype dtype) {
  HB_CHECK_ARG(p && p->norm && (tiles || !n_tiles) && n_tiles >= 0 && segments, "hb_residual_step: null argument");
  HB_CHECK_ARG((p->embed ? p->ids && p->vocab > 0 : p->y || p->top > 0) && p->top >= 0 &&
               (!p->top || (p->expert_y && p->expert_place && p->expert_weight)), "hb_residual_step: no output of a sublayer");
  HB_CHECK_ARG(p->n_earlier >= 0 && (!p->depth || p->earlier || !p->n_earlier), "hb_residual_step: bad sum over earlier results");
  HB_CHECK_ARG(p->taps >= 1 && (!p->conv || p->taps == 1 || p->state) && (!p->past || p->x), "hb_residual_step: bad convolution");
  hb::ResidualStep a;
  a.y = p->y; a.ld_y = p->ld_y;
  a.expert_y = p->expert_y; a.expert_place = p->expert_place; a.expert_weight = p->expert_weight; a.top = p->top;
  a.input = p->input; a.ld_input = p->ld_input;
  a.embed = p->embed; a.ids = p->ids; a.vocab = p->vocab;
  a.norm = p->norm; a.groups = p->groups; a.eps = p->eps;
  a.x = p->x; a.result = p->result; a.x_out = p->x_out;
  a.earlier = p->earlier; a.step = p->step; a.n_earlier = p->n_earlier; a.depth = p->depth;
  a.conv = p->conv; a.taps = p->taps; a.state = p->state; a.past = p->past;
  a.h = p->h; a.ld_h = p->ld_h;
  a.scale = p->scale; a.mixed = p->mixed; a.rows = p->rows;
  return hb::residual_step((cudaStream_t)stream, a, (const hb::RowRange*)tiles, n_tiles, (const hb::SegInfo*)segments, width, dtype);
}

int hb_parts_norm(void* stream, void* out, int64_t ld_out, const void* in, int64_t ld_in, int in_f32, const int32_t* list,
                  const float* weight, int64_t rows, int groups, int64_t size, float eps, hb_dtype dtype) {
  HB_CHECK_ARG(out && in && weight && rows >= 0 && groups > 0 && size > 0 && ld_in >= groups * size && ld_out >= groups * size,
               "hb_parts_norm: bad argument");
  return hb::parts_norm((cudaStream_t)stream, out, ld_out, in, ld_in, in_f32 != 0, list, weight, rows, groups, size, eps, dtype);
}

int hb_streams_final(void* stream, void* h, const float* x, const int32_t* want, const float* norm, int64_t n_want,
                     int streams, int64_t width, int64_t ld_h, float eps, hb_dtype dtype) {
  HB_CHECK_ARG(h && x && want && norm && streams > 0 && width > 0, "hb_streams_final: bad argument");
  return hb::streams_final((cudaStream_t)stream, h, x, want, norm, 1.f, n_want, streams, width, ld_h, eps, dtype);
}

int hb_gated_group_norm(void* stream, void* out, int64_t ld_out, const float* o, int64_t ld_o, const void* gate,
                        int64_t ld_gate, const float* weight, int64_t rows, int groups, int size, int gate_mode, float eps,
                        hb_dtype dtype) {
  HB_CHECK_ARG(out && o && gate && weight && groups > 0 && size > 0 && rows >= 0, "hb_gated_group_norm: bad argument");
  if (rows == 0) return HB_OK;
  hb::GroupNorm n;
  n.groups = groups; n.size = size; n.gate_silu = (gate_mode & 1) != 0; n.gate_first = n.own_weights = (gate_mode & 2) != 0;
  n.eps = eps;
  return hb::gated_group_norm((cudaStream_t)stream, out, ld_out, o, ld_o, gate, ld_gate, weight, rows, n, dtype);
}

}  // extern "C"
