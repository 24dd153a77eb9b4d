// The layered family: weights, pools and the step of models described by a LayeredSpec.
#include <algorithm>
#include <cmath>
#include <cstring>

#include "engine.h"
#include "layered_ops.h"

namespace hb {

LayeredModel::~LayeredModel() {
  for (auto& kv : graphs)
    if (kv.second.exec) cudaGraphExecDestroy(kv.second.exec);
}

static int64_t pad8(int64_t n) { return (n + 7) / 8 * 8; }
static int64_t pad_to(int64_t n, int64_t m) { return (n + m - 1) / m * m; }

// ------------------------------------------------------------------------------- load
// The designs of this family: which config.json a reader takes, and the reader.
struct LayeredDesign {
  bool (*serves)(const Json&);
  int (*read)(const Json&, LayeredSpec*);
};
static const LayeredDesign kDesigns[] = {{is_latarax, read_latarax}, {is_biberax, read_biberax}, {is_badolix, read_badolix},
                                          {is_muzopel, read_muzopel}};

static const LayeredDesign* design_of(const Json& config) {
  for (const LayeredDesign& d : kDesigns)
    if (d.serves(config)) return &d;
  return nullptr;
}

static bool layered_serves(const Json& config) { return design_of(config) != nullptr; }

static int layered_configure(hb_engine* e, const Json& config) {
  if (e->ws > 1) return fail(HB_ERR_INVALID_ARG, "this design runs on one rank");
  if (e->dtype == HB_F16) return fail(HB_ERR_UNSUPPORTED_DTYPE, "this design runs in bf16 or f32, not f16");
  e->lm.reset(new LayeredModel);
  int rc = design_of(config)->read(config, &e->lm->spec);
  if (rc) return rc;
  const LayeredSpec& s = e->lm->spec;
  if (s.streams < 1 || s.streams > kMaxStreams)
    return fail(HB_ERR_INVALID_ARG, "%d residual streams (1 to %d)", s.streams, kMaxStreams);
  e->H = s.width; e->V = s.vocab; e->L = (int64_t)s.layers.size();
  e->eps = s.eps;
  e->max_positions = s.max_positions;
  e->use_tc = e->dtype == HB_BF16;
  const char* g = getenv("HB_GEMM");
  if (g && std::string(g) == "simt") e->use_tc = false;
  return HB_OK;
}

namespace {
struct Loader {
  hb_engine* e;
  LayeredModel* m;
  TensorSource& src;

  // [rows, cols] rows of `name` at row r0 of a matrix, columns zero-padded to its K
  int part(const LayeredLinear& lin, const std::string& name, int64_t r0, int64_t rows, int64_t cols) {
    uint8_t* dst = (uint8_t*)lin.w + (size_t)r0 * lin.K * e->es;
    int rc = src.fetch_all(name, rows, cols, dst, e->dtype, lin.K);
    e->named[name] = {dst, rows, cols, lin.K};
    m->params += rows * cols;
    return rc;
  }
  int alloc(LayeredLinear* lin, int64_t n, int64_t k) {
    lin->N = n;
    lin->K = pad8(k);
    return dev_alloc(e, &lin->w, (size_t)n * lin->K * e->es, true);
  }
  int part(const LayeredLinear& lin, const ProjPart& p) {
    if (!p.of) return part(lin, p.tensor, p.offset, p.rows, m->spec.width);
    uint8_t* dst = (uint8_t*)lin.w + (size_t)p.offset * lin.K * e->es;
    m->params += p.rows * m->spec.width;
    return src.fetch(p.tensor, p.of, m->spec.width, p.first, p.rows, 0, m->spec.width, dst, e->dtype, lin.K);
  }
  int linear(LayeredLinear* lin, const std::string& name, int64_t n, int64_t k) {
    int rc = alloc(lin, pad8(n), k);
    return rc ? rc : part(*lin, name, 0, n, k);
  }
  int vector(float** dst, const std::string& name, int64_t n, float neutral) {  // none where the design names none
    return name.empty() ? HB_OK : small(dst, name, 1, n, neutral);
  }
  // fp32 vector or small matrix; generated weights take `neutral` (mix: the identity)
  int small(float** dst, const std::string& name, int64_t rows, int64_t cols, float neutral, bool identity = false) {
    int rc = dev_alloc(e, (void**)dst, (size_t)rows * cols * 4);
    if (rc) return rc;
    e->named[name] = {*dst, rows, cols, 0, HB_F32};
    m->params += rows * cols;
    if (!src.generated()) return src.fetch_all(name, rows, cols, *dst, HB_F32);
    return identity ? constant(*dst, rows, cols) : fill_const(e->stream, *dst, HB_F32, rows * cols, neutral);
  }
  int constant(float* dst, int64_t rows, int64_t cols) {
    std::vector<float> v((size_t)(rows * cols), 0.f);
    for (int64_t i = 0; i < std::min(rows, cols); ++i) v[(size_t)(i * cols + i)] = 1.f;
    return upload(dst, v);
  }
  int upload(float* dst, const std::vector<float>& v) {
    HB_CUDA_CHECK(cudaMemcpyAsync(dst, v.data(), v.size() * 4, cudaMemcpyHostToDevice, e->stream));
    HB_CUDA_CHECK(cudaStreamSynchronize(e->stream));
    return HB_OK;
  }
  // a convolution's weights [channels, taps] as [taps, channels]
  int taps(float** dst, const std::string& name, int64_t channels, int taps) {
    int rc;
    if ((rc = dev_alloc(e, (void**)dst, (size_t)channels * taps * 4))) return rc;
    m->params += channels * taps;
    float* rows = nullptr;
    HB_CUDA_CHECK(cudaMalloc((void**)&rows, (size_t)channels * taps * 4));
    rc = src.fetch_all(name, channels, taps, rows, HB_F32);
    if (!rc) rc = transpose_matrices(e->stream, *dst, rows, 1, channels, taps, 4);
    const cudaError_t ce = cudaStreamSynchronize(e->stream);
    cudaFree(rows);
    if (rc) return rc;
    HB_CUDA_CHECK(ce);
    return HB_OK;
  }
  int sublayer(SublayerMix* q, const std::string& norm, const std::string& conv) {  // post_norm
    const int rc = small(&q->norm, norm, 1, m->spec.width, 1.f);
    return rc || conv.empty() ? rc : taps(&q->conv, conv, m->spec.width, m->spec.input_taps);
  }
  int sublayer(SublayerMix* q, const std::string& in, const std::string& out, const std::string& mix,
               const std::string& norm) {
    const int S = m->spec.streams;
    int rc;
    if (in.empty()) {  // one plain stream: x += mult * y
      for (float** p : {&q->in, &q->out, &q->mix}) {
        if ((rc = dev_alloc(e, (void**)p, 4))) return rc;
        if ((rc = upload(*p, std::vector<float>(1, p == &q->out ? m->spec.residual_mult : 1.f)))) return rc;
      }
    } else {
      if ((rc = small(&q->in, in, 1, S, 1.f / S))) return rc;
      if ((rc = small(&q->out, out, 1, S, 1.f))) return rc;
      if ((rc = small(&q->mix, mix, S, S, 0.f, true))) return rc;
    }
    return small(&q->norm, norm, 1, m->spec.width, 1.f - m->spec.norm_offset);
  }
  int attention(LayeredLayer* l, const MixerSpec& mx) {
    const AttentionSpec& a = mx.attn;
    const int64_t q = (int64_t)a.heads * a.dim, k = (int64_t)a.kv_heads * a.dim;
    int rc;
    if ((rc = linear(&l->attn_o, mx.attn_o, m->spec.width, (int64_t)a.heads * a.vdim))) return rc;
    if ((rc = vector(&l->q_bias, mx.attn_q_bias, q, 0.f))) return rc;
    if ((rc = vector(&l->k_bias, mx.attn_k_bias, k, 0.f))) return rc;
    if ((rc = vector(&l->o_bias, mx.attn_o_bias, m->spec.width, 0.f))) return rc;
    if ((rc = vector(&l->q_norm, mx.attn_q_norm, q, 1.f))) return rc;
    if ((rc = vector(&l->k_norm, mx.attn_k_norm, k, 1.f))) return rc;
    if ((rc = vector(&l->sink, mx.attn_sink, a.heads, 0.f))) return rc;
    if (a.unit_sink) {
      if ((rc = dev_alloc(e, (void**)&l->sink, (size_t)a.heads * 4, true))) return rc;
    }
    if (!mx.attn_rel.empty()) {
      const std::vector<int64_t> shape = src.shape(mx.attn_rel);
      if (!src.generated() && (shape.size() != 2 || shape[0] < 1 || shape[0] > (1 << 20)))
        return fail(HB_ERR_IO, "Weight not found: %s", mx.attn_rel.c_str());
      l->buckets = src.generated() ? 32 : (int)shape[0];  // the number of buckets is the tensor's own
      if ((rc = small(&l->rel, mx.attn_rel, l->buckets, a.heads, 0.f))) return rc;
    }
    if (a.rank && (rc = latent(l, mx))) return rc;
    if (!a.rotation.empty()) {
      if ((rc = dev_alloc(e, (void**)&l->rotation, a.rotation.size() * 8))) return rc;
      HB_CUDA_CHECK(cudaMemcpyAsync(l->rotation, a.rotation.data(), a.rotation.size() * 8, cudaMemcpyHostToDevice, e->stream));
      HB_CUDA_CHECK(cudaStreamSynchronize(e->stream));
    }
    return HB_OK;
  }
  int latent(LayeredLayer* l, const MixerSpec& mx) {
    const AttentionSpec& a = mx.attn;
    const int64_t H = a.heads, C = a.rank;
    const size_t uk = (size_t)H * a.dim * C * e->es;
    int rc;
    if ((rc = vector(&l->latent_norm, mx.attn_latent_norm, C, 1.f))) return rc;
    if ((rc = dev_alloc(e, &l->uk_t, uk)) || (rc = dev_alloc(e, &l->ukv, uk + (size_t)H * a.vdim * C * e->es))) return rc;
    l->uv = (uint8_t*)l->ukv + uk;
    if (a.q_rank) {
      if ((rc = vector(&l->q_latent_norm, mx.attn_q_latent_norm, a.q_rank, 1.f))) return rc;
      if ((rc = linear(&l->uq, mx.attn_uq, H * (a.dim + a.rot_dim), a.q_rank))) return rc;
    }
    if ((rc = src.fetch_all(mx.attn_uv, H * a.vdim, C, l->uv, e->dtype))) return rc;
    e->named[mx.attn_uv] = {l->uv, H * a.vdim, C};
    m->params += H * (a.dim + a.vdim) * C;
    if ((rc = src.fetch_all(mx.attn_uk, H * a.dim, C, l->ukv, e->dtype))) return rc;
    e->named[mx.attn_uk] = {l->ukv, H * a.dim, C};
    return transpose_matrices(e->stream, l->uk_t, l->ukv, H, a.dim, C, e->es);
  }
  // convolution weights [channels, taps] as [taps, channels], steps, decays
  int state_space(LayeredLayer* l, const MixerSpec& mx) {
    const RecurrenceSpec& r = mx.rec;
    const int64_t n = r.conv_channels();
    int rc;
    if ((rc = taps(&l->conv_w, mx.rec_conv, n, r.conv_taps))) return rc;
    if ((rc = vector(&l->conv_b, mx.rec_conv_bias, n, 0.f))) return rc;
    if ((rc = vector(&l->dt_bias, mx.rec_dt_bias, r.heads, 0.f))) return rc;
    if ((rc = vector(&l->a_log, mx.rec_a_log, r.heads, 0.f))) return rc;
    return vector(&l->skip, mx.rec_skip, r.heads, 1.f);
  }
  // biases of a dense feed-forward, as long as the padded rows they meet
  int biases(LayeredLayer* l, const FeedForwardSpec& f) {
    int rc = vector(&l->down_b, f.down_bias, m->spec.width, 0.f);
    for (auto b : {std::make_pair(&l->gate_b, &f.gate_bias), std::make_pair(&l->up_b, &f.up_bias)}) {
      if (rc || b.second->empty()) continue;
      if ((rc = dev_alloc(e, (void**)b.first, (size_t)l->ffp * 4, true))) return rc;
      e->named[*b.second] = {*b.first, 1, f.ff, 0, HB_F32};
      m->params += f.ff;
      if (!src.generated()) rc = src.fetch_all(*b.second, 1, f.ff, *b.first, HB_F32);
    }
    return rc;
  }
  int gated(LayeredLinear* gate_up, LayeredLinear* down, int64_t* ffp, const FeedForwardSpec& f) {
    const int64_t W = m->spec.width;
    int rc;
    *ffp = pad8(f.ff);
    if ((rc = alloc(gate_up, 2 * *ffp, W))) return rc;
    if ((rc = part(*gate_up, f.gate, 0, f.ff, W))) return rc;
    if ((rc = part(*gate_up, f.up, *ffp, f.ff, W))) return rc;
    return linear(down, f.down, W, f.ff);
  }
  int experts(LayeredExperts* x, const ExpertsSpec& s, const FeedForwardSpec& shared) {
    const int64_t W = m->spec.width, E = s.experts, halves = s.act.single ? 1 : 2;
    int rc;
    x->ffp = pad8(s.ff);
    if (s.act.single && shared.ff) return fail(HB_ERR_INVALID_ARG, "experts without gates beside a shared one");
    LayeredLinear all_up, all_down;
    if ((rc = alloc(&all_up, E * halves * x->ffp, W)) || (rc = alloc(&all_down, E * pad8(W), s.ff))) return rc;
    for (int64_t i = 0; i < E; ++i) {
      const std::string t = s.prefix + std::to_string(i) + ".";
      if (halves == 2 && (rc = part(all_up, t + "gate", i * 2 * x->ffp, s.ff, W))) return rc;
      if ((rc = part(all_up, t + "up", (i * halves + halves - 1) * x->ffp, s.ff, W))) return rc;
      if ((rc = part(all_down, t + "down", i * pad8(W), W, s.ff))) return rc;
    }
    x->gate_up = all_up;
    x->gate_up.N = halves * x->ffp;
    x->down = all_down;
    x->down.N = pad8(W);
    const int64_t O = s.outputs();
    if ((rc = dev_alloc(e, &x->router, (size_t)O * W * e->es))) return rc;
    if ((rc = src.fetch_all(s.router, O, W, x->router, e->dtype))) return rc;
    e->named[s.router] = {x->router, O, W};
    m->params += O * W;
    if ((rc = vector(&x->correction, s.correction, O, 0.f))) return rc;
    if (shared.ff && (rc = gated(&x->shared_gate_up, &x->shared_down, &x->shared_ffp, shared))) return rc;
    return vector(&x->router_bias, s.router_bias, O, 0.f);
  }
};
}  // namespace

static int layered_load(hb_engine* e, TensorSource& src) {
  LayeredModel* m = e->lm.get();
  LayeredSpec& s = m->spec;
  Loader ld{e, m, src};
  const int64_t W = s.width;
  int rc;
  m->Hp = pad8(W);
  if ((rc = dev_alloc(e, &m->embed, (size_t)s.vocab * W * e->es))) return rc;
  if ((rc = src.fetch_all(s.embed, s.vocab, W, m->embed, e->dtype))) return rc;
  e->named[s.embed] = {m->embed, s.vocab, W};
  m->params += s.vocab * W;
  if (!s.pos.empty()) {
    if ((rc = dev_alloc(e, &m->pos, (size_t)s.max_positions * W * e->es))) return rc;
    if ((rc = src.fetch_all(s.pos, s.max_positions, W, m->pos, e->dtype))) return rc;
    e->named[s.pos] = {m->pos, s.max_positions, W};
    m->params += s.max_positions * W;
  }
  if (!s.head.empty()) {
    if ((rc = ld.alloc(&m->head, s.vocab, W))) return rc;
    if ((rc = ld.part(m->head, s.head, 0, s.vocab, W))) return rc;
  } else if (W % 8 == 0) {  // the embedding table itself
    m->head.w = m->embed;
    m->head.N = s.vocab;
    m->head.K = W;
  } else {
    if ((rc = ld.alloc(&m->head, s.vocab, W))) return rc;
    if ((rc = src.fetch_all(s.embed, s.vocab, W, m->head.w, e->dtype, m->head.K))) return rc;
  }
  if ((rc = ld.small(&m->final_norm, s.final_norm, 1, W, 1.f - s.norm_offset))) return rc;
  if ((rc = ld.vector(&m->embed_norm, s.embed_norm, W, 1.f))) return rc;
  m->layers.resize(s.layers.size());
  for (size_t i = 0; i < s.layers.size(); ++i) {
    LayerSpec& sp = s.layers[i];
    LayeredLayer& l = m->layers[i];
    MixerSpec& mx = sp.mixer;
    if (mx.has_rec && mx.rec.low_rank_decay) {
      const std::vector<int64_t> shape = src.shape(mx.ra1.tensor);
      if (!src.generated() && shape.size() != 2) return fail(HB_ERR_IO, "Weight not found: %s", mx.ra1.tensor.c_str());
      mx.rec.rank = src.generated() ? 16 : (int)shape[0];  // the low rank is the tensor's own
      mx.ra1.rows = mx.rec.rank;
      if (mx.rec.rank < 1) return fail(HB_ERR_IO, "%s is empty", mx.ra1.tensor.c_str());
    }
    int64_t n = 0;
    const ProjPart* parts[] = {&mx.aq, &mx.ak, &mx.av, &mx.ag, &mx.rq, &mx.rk, &mx.rv, &mx.rg, &mx.ra1, &mx.rx, &mx.rdt};
    for (const ProjPart* p : parts)
      if (p->rows) n = std::max(n, p->offset + p->rows);
    if ((rc = ld.alloc(&l.proj, pad8(n), W))) return rc;
    for (const ProjPart* p : parts)
      if (p->rows && (rc = ld.part(l.proj, *p))) return rc;
    if (mx.has_attn && (rc = ld.attention(&l, mx))) return rc;
    if (mx.has_rec) {
      const RecurrenceSpec& r = mx.rec;
      const int64_t hd = (int64_t)r.heads * r.dim, hv = (int64_t)r.heads * r.vdim;
      if ((rc = ld.linear(&l.rec_o, mx.rec_o, W, hv))) return rc;
      if ((rc = ld.small(&l.rec_norm, mx.rec_norm, 1, r.norm_per_head ? r.vdim : hv, 1.f))) return rc;
      if (r.per_token_decay) {
        if ((rc = ld.state_space(&l, mx))) return rc;
      } else if (r.low_rank_decay) {
        if ((rc = dev_alloc(e, (void**)&l.a2, (size_t)hd * r.rank * 4))) return rc;
        if ((rc = src.fetch_all(mx.rec_a2, hd, r.rank, l.a2, HB_F32))) return rc;
        e->named[mx.rec_a2] = {l.a2, hd, r.rank, 0, HB_F32};
        m->params += hd * r.rank;
        if ((rc = ld.small(&l.a2_bias, mx.rec_a2_bias, 1, hd, 1.f))) return rc;
      } else {
        if ((rc = dev_alloc(e, (void**)&l.decay, (size_t)r.heads * 4))) return rc;
        if ((rc = ld.upload(l.decay, std::vector<float>(r.decay.begin(), r.decay.end())))) return rc;
      }
    }
    if (mx.has_attn && mx.has_rec) {
      if ((rc = ld.small(&l.attn_out_norm, mx.attn_out_norm, 1, W, 1.f))) return rc;
      if ((rc = ld.small(&l.rec_out_norm, mx.rec_out_norm, 1, W, 1.f))) return rc;
    }
    if (s.post_norm) rc = ld.sublayer(&l.sub1, sp.norm1, sp.conv1);
    else rc = ld.sublayer(&l.sub1, sp.hc1_in, sp.hc1_out, sp.hc1_mix, sp.norm1);
    if (rc) return rc;
    if (!sp.depth.empty()) {  // generated: the newest result alone
      const int64_t n = (int64_t)i + 2;
      if ((rc = ld.vector(&l.depth, sp.depth, n, 0.f))) return rc;
      std::vector<float> newest((size_t)n, 0.f);
      newest.back() = 1.f;
      if (src.generated() && (rc = ld.upload(l.depth, newest))) return rc;
    }
    if (sp.moe.experts) rc = ld.experts(&l.moe, sp.moe, sp.ffn);
    else if (sp.ffn.ff) rc = ld.gated(&l.gate_up, &l.down, &l.ffp, sp.ffn);
    if (!rc && sp.ffn.ff && !sp.moe.experts) rc = ld.biases(&l, sp.ffn);
    if (rc) return rc;
    if (sp.has_ffn()) {
      if (s.post_norm) rc = ld.sublayer(&l.sub2, sp.norm2, sp.conv2);
      else rc = ld.sublayer(&l.sub2, sp.hc2_in, sp.hc2_out, sp.hc2_mix, sp.norm2);
      if (rc) return rc;
    }
  }
  return HB_OK;
}

// --------------------------------------------------------------------------- runtime
struct InputLayout {
  size_t bytes = 0;
  size_t take(size_t n) {
    const size_t at = bytes;
    bytes = (bytes + n + 15) / 16 * 16;
    return at;
  }
};

static size_t layered_layout(const hb_engine* e, LayeredStep* s) {
  InputLayout l;
  s->off_ids = l.take((size_t)s->rows * 4);
  s->off_pos = l.take((size_t)s->rows * 4);
  s->off_slots = l.take((size_t)s->rows * 8);
  s->off_row_seg = l.take((size_t)s->rows * 4);
  s->off_want = l.take((size_t)s->want * 4);
  s->off_seg = l.take((size_t)s->segs * sizeof(SegInfo));
  s->off_short = l.take((size_t)s->segs * 4);
  s->off_long = l.take((size_t)s->n_long * sizeof(RowRange));
  s->off_chunk = l.take((size_t)s->n_chunks * sizeof(RowRange));
  for (int k = 0; k < kTileKinds; ++k) s->off_tile[k] = l.take((size_t)s->n_tiles[k] * sizeof(RowRange));
  s->off_row_list = l.take((size_t)s->rows * 4);
  s->off_run = l.take((size_t)s->n_runs * sizeof(RowRange));
  s->off_tables = l.take((size_t)s->segs * e->max_blocks_per_seq * 4);
  s->off_expand_base = l.take(s->n_expand ? (size_t)s->segs * 4 : 0);
  s->off_expand_list = l.take((size_t)s->n_expand * 4);
  return l.bytes;
}

// Segments of up to this many tokens go through the recurrence token by token.
constexpr int kShortSegment = 8;
// Latent attention of prompts: keys and values of the heads are grown out of the latents for portions of
// at least this many tokens (fewer do not pay for it), in at most this much memory.
constexpr int kExpandTokens = 32;
constexpr size_t kExpandBytes = (size_t)512 << 20;
// Decoded tokens: with fewer (row, kv head) units than this the keys may be split over several CTAs.
constexpr int kSplitUnits = 592;
// Most tokens of a run of the residual kernels: long runs repeat less, short ones fill the SMs.
static int residual_run(int rows) { return rows <= 256 ? 4 : kResidualRun; }
constexpr int kResidualTwo = 256;  // more rows than this: the residual in two kernels

static SpanAttention span_args(const hb_engine* e, size_t i, const LayeredStep& s) {
  const LayeredModel* m = e->lm.get();
  const MixerSpec& mx = m->spec.layers[i].mixer;
  const AttentionSpec& as = mx.attn;
  const LayeredLayer& l = m->layers[i];
  SpanAttention a;
  a.q = (const uint8_t*)m->proj + mx.aq.offset * e->es; a.ld_q = l.proj.N;
  a.out = m->attn; a.ld_out = l.attn_o.K;
  a.kc = e->kc[l.kv_pool]; a.vc = e->vc[l.kv_pool];
  a.tables = (const int32_t*)(e->d_inputs + s.off_tables);
  a.max_blocks = e->max_blocks_per_seq; a.num_blocks = e->num_blocks;
  a.row_seg = (const int32_t*)(e->d_inputs + s.off_row_seg);
  a.pos = (const int32_t*)(e->d_inputs + s.off_pos);
  a.heads = as.heads; a.kv_heads = as.cached_heads(); a.dim = as.key_width(); a.vdim = as.value_width();
  a.window = as.window; a.keep_first = as.keep_first; a.chunk = as.chunk; a.scale = as.scale; a.softcap = as.softcap;
  if (as.rank) {
    a.q = m->latent_q; a.ld_q = (int64_t)as.heads * a.dim;
    a.out = m->latent_o; a.ld_out = (int64_t)as.heads * a.vdim;
    a.vc = nullptr;
  }
  if (as.values_are_keys) {  // the second pool holds the keys' scales
    a.key_scale = (const float*)a.vc;
    a.vc = nullptr;
  }
  a.dist_bias = l.dist_bias; a.dist_len = l.dist_len;
  a.err = e->d_err;
  a.sink = l.sink;
  a.gate_per_head = as.gate_per_head ? 1 : 0;
  if (mx.ag.rows) {
    a.gate = (const uint8_t*)m->proj + mx.ag.offset * e->es;
    a.ld_gate = l.proj.N;
  }
  return a;
}

static LatentPrep latent_args(const hb_engine* e, size_t i, const LayeredStep& s) {
  const LayeredModel* m = e->lm.get();
  const MixerSpec& mx = m->spec.layers[i].mixer;
  const LayeredLayer& l = m->layers[i];
  const AttentionSpec& as = mx.attn;
  LatentPrep p;
  p.p = m->proj; p.ld = l.proj.N; p.off_q = (int)mx.aq.offset; p.off_c = (int)mx.ak.offset;
  p.heads = as.heads; p.dim = as.dim; p.rot_dim = as.rot_dim; p.rank = as.rank;
  p.q = m->latent_q; p.ld_q = (int64_t)as.heads * as.key_width();
  p.pos = (const int32_t*)(e->d_inputs + s.off_pos);
  p.slots = (const int64_t*)(e->d_inputs + s.off_slots);
  p.kc = e->kc[l.kv_pool]; p.num_blocks = e->num_blocks;
  p.norm = l.latent_norm; p.eps = m->spec.eps;
  p.rotation = l.rotation; p.pairs = (int)as.rotation.size(); p.rotation_gain = as.rotation_gain;
  p.halves = as.rotation_halves ? 1 : 0;
  if (as.q_rank) { p.qs = m->q; p.ld_qs = l.uq.N; }
  return p;
}

// The heads' queries as projected: part of the input projection, or out of a latent of their own.
static const void* query_rows(const hb_engine* e, size_t i) {
  const LayeredModel* m = e->lm.get();
  const MixerSpec& mx = m->spec.layers[i].mixer;
  return mx.attn.q_rank ? m->q : (const uint8_t*)m->proj + mx.aq.offset * e->es;
}
static int64_t query_stride(const LayeredLayer& l, const AttentionSpec& a) { return a.q_rank ? l.uq.N : l.proj.N; }

// Attention of expanded segments: every head its own keys [dim | shared part] and values.
static SpanAttention expanded_args(const hb_engine* e, size_t i, const LayeredStep& s) {
  const LayeredModel* m = e->lm.get();
  const MixerSpec& mx = m->spec.layers[i].mixer;
  const AttentionSpec& as = mx.attn;
  const LayeredLayer& l = m->layers[i];
  SpanAttention a = span_args(e, i, s);
  a.q = query_rows(e, i); a.ld_q = query_stride(l, as);
  a.out = m->attn; a.ld_out = l.attn_o.K;
  a.kv_heads = as.heads; a.dim = as.dim + as.rot_dim; a.vdim = as.vdim;
  const int64_t row = (int64_t)as.heads * (as.dim + as.vdim);
  a.kc = m->expand_kv; a.vc = (uint8_t*)m->expand_kv + (size_t)as.heads * as.dim * e->es;
  a.k_step = {HB_BLOCK_SIZE * row, as.dim, row};
  a.v_step = {HB_BLOCK_SIZE * row, as.vdim, row};
  a.linear = 1; a.tables = (const int32_t*)(e->d_inputs + s.off_expand_base); a.num_blocks = m->expand_blocks;
  a.tail = as.rot_dim; a.kt = (const uint8_t*)m->expand_latent + (size_t)as.rank * e->es; a.ld_kt = as.key_width();
  return a;
}
static TcHeads expand_rows(const AttentionSpec& a) {
  TcHeads h;
  h.heads = 1;
  h.ldx = h.x_step = a.key_width();
  h.ldy = h.y_step = (int64_t)a.heads * (a.dim + a.vdim);
  return h;
}

// The products of latent attention, head by head: W_uk^T on the queries' first parts, W_uv on what the
// heads gathered from the latents.
static TcHeads latent_q_heads(const LayeredLayer& l, const AttentionSpec& a) {
  TcHeads h;
  h.heads = a.heads;
  h.ldx = query_stride(l, a); h.x_step = a.dim + a.rot_dim;
  h.ldy = (int64_t)a.heads * a.key_width(); h.y_step = a.key_width();
  return h;
}
static TcHeads latent_v_heads(const LayeredLayer& l, const AttentionSpec& a) {
  TcHeads h;
  h.heads = a.heads;
  h.ldx = (int64_t)a.heads * a.rank; h.x_step = a.rank;
  h.ldy = l.attn_o.K; h.y_step = a.vdim;
  return h;
}

// Queries in place, keys and values to their slots; false: the design only needs the K/V write.
static bool prep_args(const hb_engine* e, size_t i, const LayeredStep& s, AttentionPrep* p) {
  const LayeredModel* m = e->lm.get();
  const MixerSpec& mx = m->spec.layers[i].mixer;
  const LayeredLayer& l = m->layers[i];
  const AttentionSpec& as = mx.attn;
  if (!l.rotation && !l.q_norm && !l.q_bias) return false;
  p->p = m->proj; p->ld = l.proj.N;
  p->off_q = (int)mx.aq.offset; p->off_k = (int)mx.ak.offset; p->off_v = (int)mx.av.offset;
  p->heads = as.heads; p->kv_heads = as.kv_heads; p->dim = as.dim; p->vdim = as.vdim;
  p->pos = (const int32_t*)(e->d_inputs + s.off_pos);
  p->slots = (const int64_t*)(e->d_inputs + s.off_slots);
  p->kc = e->kc[l.kv_pool]; p->vc = e->vc[l.kv_pool]; p->num_blocks = e->num_blocks;
  p->q_bias = l.q_bias; p->k_bias = l.k_bias; p->q_norm = l.q_norm; p->k_norm = l.k_norm;
  p->eps = m->spec.eps;
  p->rotation = l.rotation; p->pairs = (int)as.rotation.size();
  p->halves = as.rotation_halves ? 1 : 0; p->rotation_gain = as.rotation_gain;
  if (as.kv_from >= 0) p->kc = p->vc = nullptr;  // that layer has written them
  if (as.values_are_keys) p->key_scale = (float*)p->vc;
  return true;
}

// Row of the bias table for distance n: exact below half of the buckets, logarithmic above.
static int distance_bucket(int64_t n, int buckets, double far) {
  const int half = buckets / 2;
  if (n < half) return (int)n;
  if (half == 0 || far <= half) return buckets - 1;
  const double x = std::log((double)n / half) / std::log(far / half) * (buckets - half);
  return x >= buckets - half ? buckets - 1 : std::min(buckets - 1, half + (int)std::floor(x));
}

// The bias by distance, up to where it no longer changes (or no sequence reaches).
static int build_distance_bias(hb_engine* e, LayeredLayer* l, const AttentionSpec& a, int64_t max_seq) {
  std::vector<int32_t> bucket;
  for (int64_t n = 0; n < max_seq; ++n) {
    bucket.push_back(distance_bucket(n, l->buckets, a.bias_far));
    if (bucket.back() == l->buckets - 1) break;
  }
  l->dist_len = (int)bucket.size();
  int32_t* d = nullptr;
  int rc;
  if ((rc = dev_alloc(e, (void**)&l->dist_bias, (size_t)a.heads * l->dist_len * 4))) return rc;
  HB_CUDA_CHECK(cudaMalloc((void**)&d, bucket.size() * 4));
  rc = cudaMemcpyAsync(d, bucket.data(), bucket.size() * 4, cudaMemcpyHostToDevice, e->stream) == cudaSuccess
           ? expand_distance_bias(e->stream, l->dist_bias, l->rel, d, a.heads, l->dist_len)
           : fail(HB_ERR_CUDA, "upload of the distance buckets failed");
  const cudaError_t ce = cudaStreamSynchronize(e->stream);
  cudaFree(d);
  if (rc) return rc;
  HB_CUDA_CHECK(ce);
  return HB_OK;
}

// Batch tiles of a mixture for `rows` rows of a step: tiles of about the rows an expert gets.
static TcGroups moe_groups(const ExpertsSpec& x, bool shared, int rows, bool tc) {
  TcGroups g;
  const int64_t n = (int64_t)rows * x.top;
  g.groups = x.experts;
  g.m_pad = tc ? (int)std::min<int64_t>(128, pad_to(std::max<int64_t>(1, ((int64_t)(rows * x.picks() * 1.5) + x.experts - 1) / x.experts), 16)) : 16;
  g.max_tiles = (int)(std::min<int64_t>(x.experts, n) + n / g.m_pad);
  // experts that some row of a random batch chooses, and their tiles
  const double picks = rows * x.picks(), active = x.experts * (1.0 - std::pow(1.0 - 1.0 / x.experts, picks));
  const double tiles = active * std::max(1.0, std::ceil(picks / std::max(1.0, active) / g.m_pad));
  g.likely_tiles = (int)std::max<int64_t>(1, std::min<int64_t>((int64_t)tiles, g.max_tiles));
  if (shared) {
    const int more = (rows + g.m_pad - 1) / g.m_pad;
    g.max_tiles += more;
    g.likely_tiles += more;
  }
  return g;
}
// The two products of a mixture: gate | up into rows of activations, and from there back to the width.
static TcGroups up_groups(TcGroups g, const LayeredExperts& w, const GatedAct& shared_act) {
  g.ldx = w.gate_up.K; g.ldy = w.ld();
  if (w.shared_ffp) {
    g.shared_w = w.shared_gate_up.w; g.shared_n = w.shared_gate_up.N; g.shared_k = w.shared_gate_up.K;
    g.shared_act = shared_act;
  }
  return g;
}
static TcGroups down_groups(TcGroups g, const LayeredExperts& w) {
  g.ldx = w.ld(); g.ldy = w.down.N;
  if (w.shared_ffp) { g.shared_w = w.shared_down.w; g.shared_n = w.shared_down.N; g.shared_k = w.shared_down.K; }
  return g;
}

static MoeRouting moe_args(const LayeredModel* m, const ExpertsSpec& x, const LayeredExperts& w, const TcGroups& g) {
  const bool shared = w.shared_ffp > 0;
  MoeRouting r;
  r.correction = w.correction;
  r.experts = x.experts; r.top = x.top; r.shared = shared ? 1 : 0;
  r.softmax_all = x.softmax_all ? 1 : 0; r.identity = x.identity;
  r.sigmoid = x.sigmoid ? 1 : 0; r.groups = x.groups; r.keep = x.keep;
  r.m_pad = g.m_pad; r.max_tiles = g.max_tiles;
  r.ids = m->moe_ids; r.rank = m->moe_rank; r.place = m->moe_place; r.weight = m->moe_weight;
  r.count = m->moe_count; r.first = m->moe_first; r.tile_group = m->moe_tiles;
  return r;
}

// Prompt portions as tiles, decoded tokens as rows; sizes the tensor-core kernels do not take go
// row by row.
static int issue_attention(hb_engine* e, const SpanAttention& a, int kind, const LayeredStep& s) {
  LayeredModel* m = e->lm.get();
  cudaStream_t st = e->stream;
  const int32_t* rows = (const int32_t*)(e->d_inputs + s.off_row_list);
  int rc;
  if (kind < 0) {
    ++e->last_launches;
    return span_attention_rows(st, a, rows, s.rows, e->dtype);
  }
  if (s.n_tiles[kind]) {
    ++e->last_launches;
    if ((rc = span_attention_tiles(st, a, (const RowRange*)(e->d_inputs + s.off_tile[kind]), s.n_tiles[kind]))) return rc;
  }
  if (!s.n_token_rows) return HB_OK;
  ++e->last_launches;
  if (!span_attention_tokens_supported(a, e->dtype)) return span_attention_rows(st, a, rows, s.n_token_rows, e->dtype);
  // the longest span a row can have decides the split: it is the same in every replay of a graph
  const int64_t span = a.chunk > 0 ? a.chunk : a.window;
  const int64_t longest = span > 0 ? span + a.keep_first : a.max_blocks * HB_BLOCK_SIZE;
  const int64_t blocks = std::min<int64_t>(longest / HB_BLOCK_SIZE + 2, a.max_blocks), units = (int64_t)s.n_token_rows * span_attention_token_units(a);
  // as many as are resident at once, every one with some blocks for each of its warps
  const bool latent = latent_tokens_supported(a, e->dtype);
  int64_t splits = std::min<int64_t>(std::min(kSplitUnits, span_attention_tokens_slots(a)) / units, (blocks + 7) / 8);
  splits = std::max<int64_t>(1, std::min<int64_t>(splits, latent ? 64 : 16));
  if (splits > 8 && blocks < 1024 && !latent) splits = 8;  // what a cluster sums up
  if (splits > (latent ? 1 : 8)) ++e->last_launches;  // a kernel sums up
  return span_attention_tokens(st, a, rows, s.n_token_rows, (int)splits, m->attn_part);
}

static int issue_recurrence(hb_engine* e, const Recurrence& r, const LayeredStep& s) {
  LayeredModel* m = e->lm.get();
  const int32_t* list = (const int32_t*)(e->d_inputs + s.off_short);
  const bool chunked = e->use_tc && recurrence_chunks_supported(r, e->dtype);
  const int n_list = chunked ? s.n_short : s.segs;  // short segments first, longer ones after them
  if (n_list) ++e->last_launches;
  int rc = recurrence_tokens(e->stream, r, list, n_list, e->dtype);
  if (rc || !chunked) return rc;
  RecurrenceChunks c;
  c.chunks = (const RowRange*)(e->d_inputs + s.off_chunk); c.n_chunks = s.n_chunks;
  c.segs = (const RowRange*)(e->d_inputs + s.off_long); c.n_segs = s.n_long;
  c.cum = m->cum; c.state = m->chunk_state;
  return recurrence_chunks(e->stream, r, c, &e->last_launches);
}

// Index of the kind of tiles a layer takes; where there are as many as there are lists, the one with the
// most positions that are not too many (-1: none).
static int tile_kind(LayeredModel* m, int positions, TileKind::Which which) {
  if (positions < 1) return -1;
  std::vector<TileKind>& kinds = m->tile_kinds;
  const TileKind want{positions, which};
  auto at = std::find(kinds.begin(), kinds.end(), want);
  if (at != kinds.end()) return (int)(at - kinds.begin());
  if ((int)kinds.size() < kTileKinds) {
    kinds.push_back(want);
    return (int)kinds.size() - 1;
  }
  int best = -1;
  for (size_t k = 0; k < kinds.size(); ++k)
    if (kinds[k].which == which && kinds[k].positions <= positions && (best < 0 || kinds[k].positions > kinds[best].positions)) best = (int)k;
  return best;
}

static int layered_alloc_runtime(hb_engine* e, const hb_model_config* cfg) {
  LayeredModel* m = e->lm.get();
  const LayeredSpec& s = m->spec;
  const size_t es = e->es;
  int rc;
  e->max_batch = cfg->max_batch > 0 ? cfg->max_batch : 256;
  int64_t max_seq = cfg->max_seq_len > 0 ? (int64_t)cfg->max_seq_len : 2048;
  if (s.max_positions > 0) max_seq = std::min(max_seq, s.max_positions);
  e->max_blocks_per_seq = (max_seq + HB_BLOCK_SIZE - 1) / HB_BLOCK_SIZE;
  m->max_segs = std::min(e->max_batch, cfg->max_seqs > 0 ? cfg->max_seqs : e->max_batch);
  e->num_blocks = cfg->num_kv_blocks > 0 ? cfg->num_kv_blocks : e->max_blocks_per_seq * m->max_segs;
  for (int64_t b = 0; b < e->num_blocks; ++b) e->free_blocks.push_back(b);
  const int64_t R = pad_to(e->max_batch, 128);
  m->row_cap = R;
  if (s.post_norm) {
    for (size_t i = 0; i < s.layers.size(); ++i) {
      const int64_t n = (int64_t)m->max_segs * (s.input_taps - 1) * s.width;
      if (n <= 0) break;
      e->num_state_slots = m->max_segs;
      if ((rc = dev_alloc(e, (void**)&m->layers[i].sub1.conv_state, (size_t)n * 4, true))) return rc;
      if (s.layers[i].has_ffn() && (rc = dev_alloc(e, (void**)&m->layers[i].sub2.conv_state, (size_t)n * 4, true))) return rc;
    }
    if ((rc = dev_alloc(e, &m->h2, (size_t)R * m->Hp * es, true))) return rc;
    if ((rc = dev_alloc(e, (void**)&m->x2, (size_t)R * s.width * 4, true))) return rc;
    if ((rc = dev_alloc(e, (void**)&m->part_scale, (size_t)R * s.norm_groups * 4, true))) return rc;
    if ((rc = dev_alloc(e, (void**)&m->results, (size_t)(s.layers.size() + 1) * R * s.width * 4, true))) return rc;
  }
  m->max_chunks = e->max_batch / kRecChunk + std::min(m->max_segs, e->max_batch / (kShortSegment + 1)) + 1;
  int64_t max_attn = 0, max_rec = 0, max_o = 0, max_ffp = 0, max_cum = 0, max_state = 0, max_part = 0;
  int64_t max_experts = 0, max_top = 0, max_eff = 0, max_tiles = 0, max_conv = 0, max_latent_q = 0, max_latent_o = 0, max_expand_row = 0,
          max_expand_latent = 0, max_q_latent = 0, max_q = 0;
  for (size_t i = 0; i < s.layers.size(); ++i) {
    LayeredLayer& l = m->layers[i];
    const MixerSpec& mx = s.layers[i].mixer;
    m->max_proj = std::max(m->max_proj, l.proj.N);
    max_ffp = std::max(max_ffp, l.ffp);
    if (mx.has_attn) {
      const AttentionSpec& a = mx.attn;
      if (a.kv_from >= 0) {
        l.kv_pool = m->layers[a.kv_from].kv_pool;
      } else {
        l.kv_pool = (int)e->kc.size();
        const size_t kb = (size_t)a.cached_heads() * HB_BLOCK_SIZE * a.key_width() * es;
        // values that are the keys: the second pool holds one scale per token; a latent: nothing
        const size_t vb = a.values_are_keys ? (size_t)HB_BLOCK_SIZE * 4 : (size_t)(a.kv_heads * HB_BLOCK_SIZE * a.value_pool_width()) * es;
        void *k = nullptr, *v = nullptr;
        // unwritten slots may be fetched (and masked): keep them finite
        if ((rc = dev_alloc(e, &k, kb * e->num_blocks, true))) return rc;
        if (vb && (rc = dev_alloc(e, &v, vb * e->num_blocks, true))) return rc;
        e->kc.push_back(k);
        e->vc.push_back(v);
        e->k_block_bytes.push_back(kb);
        e->v_block_bytes.push_back(vb);
      }
      max_attn = std::max(max_attn, l.attn_o.K);
      max_part = std::max(max_part, (int64_t)kSplitUnits * 2 * (a.heads / a.cached_heads()) * (a.value_width() + 2));
      if (a.rank) {
        max_latent_q = std::max(max_latent_q, (int64_t)a.heads * a.key_width());
        max_latent_o = std::max(max_latent_o, (int64_t)a.heads * a.rank);
        max_q_latent = std::max(max_q_latent, l.uq.K);
        max_q = std::max(max_q, l.uq.N);
        l.latent_tc = e->use_tc && gemm_tc_heads_supported(a.rank, a.dim, false, latent_q_heads(l, a)) &&
                      gemm_tc_heads_supported(a.vdim, a.rank, false, latent_v_heads(l, a));
        // over the latent a row and key cost more than with a head's own keys and values
        l.expand = l.latent_tc && gemm_tc_heads_supported(a.heads * (a.dim + a.vdim), a.rank, false, expand_rows(a)) &&
                   3 * a.rank > a.dim + 2 * a.vdim;
        if (l.expand) {
          max_expand_row = std::max(max_expand_row, (int64_t)a.heads * (a.dim + a.vdim));
          max_expand_latent = std::max(max_expand_latent, (int64_t)a.key_width());
        }
      }
      if (l.rel && (rc = build_distance_bias(e, &l, a, e->max_blocks_per_seq * HB_BLOCK_SIZE))) return rc;
    }
    if (const ExpertsSpec& x = s.layers[i].moe; x.experts) {
      if (x.outputs() > kMoeMaxExperts) return fail(HB_ERR_INVALID_ARG, "%d experts (at most %d)", x.outputs(), kMoeMaxExperts);
      max_experts = std::max<int64_t>(max_experts, x.experts);
      max_top = std::max<int64_t>(max_top, x.top + 1);
      max_eff = std::max(max_eff, l.moe.ld());
      for (int64_t M = 1; M <= R; M = M < 16 ? M * 2 : M + 16) {
        const TcGroups g = moe_groups(x, l.moe.shared_ffp > 0, (int)M, e->use_tc);
        max_tiles = std::max<int64_t>(max_tiles, g.max_tiles);
        m->moe_places = std::max<int64_t>(m->moe_places, (int64_t)g.max_tiles * g.m_pad);
      }
    }
    if (mx.has_rec) {
      const RecurrenceSpec& r = mx.rec;
      e->num_state_slots = m->max_segs;
      if ((rc = dev_alloc(e, (void**)&l.state, (size_t)m->max_segs * r.heads * r.dim * r.vdim * 4, true))) return rc;
      max_rec = std::max(max_rec, l.rec_o.K);
      max_o = std::max(max_o, (int64_t)r.heads * r.vdim);
      if (r.low_rank_decay) max_cum = std::max(max_cum, (int64_t)r.heads * r.dim);
      if (r.per_token_decay) {
        max_cum = std::max(max_cum, 2 * (int64_t)r.heads);
        max_conv = std::max(max_conv, pad8(r.conv_channels()));
        if (r.conv_taps > 1 &&
            (rc = dev_alloc(e, &l.conv_state, (size_t)m->max_segs * (r.conv_taps - 1) * r.conv_channels() * es, true))) return rc;
      }
      max_state = std::max(max_state, (int64_t)r.heads * r.dim * r.vdim);
    }
  }
  for (int i = 0; i < e->num_state_slots; ++i) e->free_slots.push_back(i);
  e->max_logits_rows = (int)std::min<int64_t>(e->max_batch, std::max<int64_t>(64, (1ll << 28) / s.vocab));
  const int64_t LR = pad_to(e->max_logits_rows, 16);
  if ((rc = dev_alloc(e, (void**)&m->x, (size_t)R * s.streams * s.width * 4, true))) return rc;
  if ((rc = dev_alloc(e, &m->h, (size_t)R * m->Hp * es, true))) return rc;
  if ((rc = dev_alloc(e, &m->proj, (size_t)R * m->max_proj * es, true))) return rc;
  if ((rc = dev_alloc(e, &m->attn, (size_t)R * max_attn * es, true))) return rc;
  if ((rc = dev_alloc(e, &m->rec, (size_t)R * max_rec * es, true))) return rc;
  if ((rc = dev_alloc(e, (void**)&m->o, (size_t)R * max_o * 4, true))) return rc;
  if (max_expand_row) {
    m->expand_blocks = std::min<int64_t>((int64_t)(kExpandBytes / ((size_t)max_expand_row * es * HB_BLOCK_SIZE)),
                                         std::min(e->num_blocks, e->max_blocks_per_seq * m->max_segs));
    m->expand_blocks = std::max<int64_t>(8, pad_to(m->expand_blocks, 8));  // whole batch tiles
    const size_t rows = (size_t)m->expand_blocks * HB_BLOCK_SIZE;
    if ((rc = dev_alloc(e, &m->expand_kv, rows * max_expand_row * es, true))) return rc;
    if ((rc = dev_alloc(e, &m->expand_latent, rows * max_expand_latent * es, true))) return rc;
  }
  if (max_conv && (rc = dev_alloc(e, &m->conv, (size_t)R * max_conv * es, true))) return rc;
  if (max_latent_q && (rc = dev_alloc(e, &m->latent_q, (size_t)R * max_latent_q * es, true))) return rc;
  if (max_q && (rc = dev_alloc(e, &m->q_latent, (size_t)R * max_q_latent * es, true))) return rc;
  if (max_q && (rc = dev_alloc(e, &m->q, (size_t)R * max_q * es, true))) return rc;
  if (max_latent_o && (rc = dev_alloc(e, &m->latent_o, (size_t)R * max_latent_o * es, true))) return rc;
  if (e->use_tc) {
    if ((rc = dev_alloc(e, (void**)&m->cum, (size_t)R * max_cum * 4))) return rc;
    if ((rc = dev_alloc(e, (void**)&m->chunk_state, (size_t)m->max_chunks * max_state * 4))) return rc;
    if ((rc = dev_alloc(e, (void**)&m->attn_part, (size_t)max_part * 4))) return rc;
  }
  for (size_t i = 0; i < s.layers.size(); ++i)
    if (s.layers[i].mixer.has_attn) {
      LayeredLayer& l = m->layers[i];
      const int tp = span_attention_tile_positions(span_args(e, i, LayeredStep()), e->dtype);
      if (l.expand) l.expand_kind = tile_kind(m, span_attention_tile_positions(expanded_args(e, i, LayeredStep()), e->dtype), TileKind::kExpanded);
      l.expand = l.expand_kind >= 0;
      l.tile_kind = tile_kind(m, tp, l.expand ? TileKind::kNotExpanded : TileKind::kAll);
    }
  if ((rc = dev_alloc(e, (void**)&m->y1, (size_t)R * m->Hp * 4, true))) return rc;
  if ((rc = dev_alloc(e, (void**)&m->y2, (size_t)R * m->Hp * 4, true))) return rc;
  if (!e->use_tc && (rc = dev_alloc(e, &m->gu, (size_t)R * 2 * max_ffp * es, true))) return rc;
  if ((rc = dev_alloc(e, &m->act, (size_t)R * max_ffp * es, true))) return rc;
  if (max_experts) {
    const size_t picks = (size_t)R * max_top * 4;
    if ((rc = dev_alloc(e, &m->moe_x, (size_t)m->moe_places * m->Hp * es, true))) return rc;
    if ((rc = dev_alloc(e, &m->moe_act, (size_t)m->moe_places * max_eff * es, true))) return rc;
    if ((rc = dev_alloc(e, &m->moe_y, (size_t)m->moe_places * m->Hp * es, true))) return rc;
    if (!e->use_tc && (rc = dev_alloc(e, &m->moe_gu, (size_t)m->moe_places * 2 * max_eff * es, true))) return rc;
    if ((rc = dev_alloc(e, (void**)&m->moe_ids, picks, true))) return rc;
    if ((rc = dev_alloc(e, (void**)&m->moe_rank, picks, true))) return rc;
    if ((rc = dev_alloc(e, (void**)&m->moe_place, picks, true))) return rc;
    if ((rc = dev_alloc(e, (void**)&m->moe_weight, picks, true))) return rc;
    if ((rc = dev_alloc(e, (void**)&m->moe_count, (size_t)(max_experts + 1) * 4, true))) return rc;
    if ((rc = dev_alloc(e, (void**)&m->moe_first, (size_t)(max_experts + 1) * 4, true))) return rc;
    if ((rc = dev_alloc(e, (void**)&m->moe_tiles, (size_t)max_tiles * 4, true))) return rc;
  }
  if ((rc = dev_alloc(e, &m->hf, (size_t)LR * m->Hp * es, true))) return rc;
  if ((rc = dev_alloc(e, (void**)&e->d_logits, (size_t)LR * s.vocab * 4))) return rc;
  if ((rc = dev_alloc(e, (void**)&e->d_next, (size_t)LR * 4, true))) return rc;
  HB_CUDA_CHECK(cudaMallocHost((void**)&e->h_next, (size_t)LR * 4));
  if ((rc = dev_alloc(e, (void**)&e->d_err, 16, true))) return rc;
  if ((rc = dev_alloc(e, (void**)&e->d_pairs, (size_t)kPairCap * 2 * sizeof(int64_t)))) return rc;
  // the largest step: every list at its longest
  LayeredStep cap;
  cap.rows = e->max_batch;
  cap.want = e->max_batch;
  cap.segs = cap.n_long = m->max_segs;
  cap.n_chunks = m->max_chunks;
  for (size_t k = 0; k < m->tile_kinds.size(); ++k) cap.n_tiles[k] = e->max_batch / m->tile_kinds[k].positions + m->max_segs;
  cap.n_expand = (int)m->expand_blocks;
  if (s.post_norm) cap.n_runs = e->max_batch / residual_run(1) + m->max_segs;
  e->inputs_bytes = layered_layout(e, &cap);
  if ((rc = dev_alloc(e, (void**)&e->d_inputs, e->inputs_bytes, true))) return rc;
  HB_CUDA_CHECK(cudaMallocHost((void**)&e->h_inputs, e->inputs_bytes));
  return HB_OK;
}

// ------------------------------------------------------------------------------- step
// Matrix products are planned for a bucket of rows, so that steps of similar size share plans;
// the rows above the step's own are scratch.
static int row_bucket(int rows) {
  if (rows <= 16) {  // few rows choose few experts: how many decides how their products are cut
    int b = 1;
    while (b < rows) b *= 2;
    return b;
  }
  return (int)(rows <= 256 ? pad_to(rows, 16) : pad_to(rows, 128));
}

static int layered_plans(hb_engine* e, int rows, LayeredPlans** out) {
  LayeredModel* m = e->lm.get();
  const int M = row_bucket(rows);
  auto it = m->plans.find(M);
  if (it != m->plans.end()) { *out = &it->second; return HB_OK; }
  LayeredPlans p;
  const size_t L = m->layers.size();
  for (auto* v : {&p.proj, &p.uq, &p.latent_q, &p.latent_v, &p.attn_o, &p.rec_o, &p.gate_up, &p.down, &p.moe_gate_up, &p.moe_down}) v->resize(L);
  size_t ws = 0;
  int rc;
  auto plan = [&](TcGemmPlan* pl, const void* X, const LayeredLinear& w, int epi, bool f32) -> int {
    if (!w.w) return HB_OK;
    const int r = gemm_tc_plan(pl, X, w.w, M, w.N, w.K, epi, f32, e->device);
    if (!r) ws = std::max(ws, pl->workspace_bytes());
    return r;
  };
  for (size_t i = 0; i < L; ++i) {
    LayeredLayer& l = m->layers[i];
    if ((rc = plan(&p.proj[i], m->h, l.proj, kEpiStore, false))) return rc;
    if ((rc = plan(&p.uq[i], m->q_latent, l.uq, kEpiStore, false))) return rc;
    if (l.latent_tc) {
      const AttentionSpec& a = m->spec.layers[i].mixer.attn;
      const TcHeads q = latent_q_heads(l, a), v = latent_v_heads(l, a);
      if ((rc = gemm_tc_plan(&p.latent_q[i], query_rows(e, i), l.uk_t, M, a.rank, a.dim, kEpiStore, false, e->device, 0, nullptr, &q))) return rc;
      if ((rc = gemm_tc_plan(&p.latent_v[i], m->latent_o, l.uv, M, a.vdim, a.rank, kEpiStore, false, e->device, 0, nullptr, &v))) return rc;
      ws = std::max(ws, std::max(p.latent_q[i].workspace_bytes(), p.latent_v[i].workspace_bytes()));
    }
    if ((rc = plan(&p.attn_o[i], m->attn, l.attn_o, kEpiStore, true))) return rc;
    if ((rc = plan(&p.rec_o[i], m->rec, l.rec_o, kEpiStore, true))) return rc;
    const void* ffn_in = m->spec.post_norm ? m->h2 : m->h;
    if ((rc = plan(&p.gate_up[i], ffn_in, l.gate_up, kEpiSwiGLU, false))) return rc;
    p.gate_up[i].act = m->spec.layers[i].ffn.act;
    p.gate_up[i].gate_bias = l.gate_b; p.gate_up[i].up_bias = l.up_b;
    if ((rc = plan(&p.down[i], m->act, l.down, kEpiStore, true))) return rc;
    const ExpertsSpec& x = m->spec.layers[i].moe;
    if (!x.experts) continue;
    const TcGroups g = moe_groups(x, l.moe.shared_ffp > 0, M, true);
    const TcGroups up = up_groups(g, l.moe, m->spec.layers[i].ffn.act), down = down_groups(g, l.moe);
    if ((int64_t)g.max_tiles * g.m_pad > m->moe_places) return fail(HB_ERR_INVALID_ARG, "experts of %d rows need more places", M);
    if ((rc = gemm_tc_plan(&p.moe_gate_up[i], m->moe_x, l.moe.gate_up.w, m->moe_places, l.moe.gate_up.N, l.moe.gate_up.K,
                           x.act.single ? kEpiAct : kEpiSwiGLU, false, e->device, 0, &up))) return rc;
    p.moe_gate_up[i].act = x.act;
    if ((rc = gemm_tc_plan(&p.moe_down[i], m->moe_act, l.moe.down.w, m->moe_places, l.moe.down.N, l.moe.down.K, kEpiStore, false,
                           e->device, 0, &down))) return rc;
  }
  if ((rc = ensure_gemm_workspace(e, ws))) return rc;
  *out = &m->plans.emplace(M, std::move(p)).first->second;
  return HB_OK;
}

static int layered_expand_plans(hb_engine* e, int blocks, std::vector<TcGemmPlan>** out) {
  LayeredModel* m = e->lm.get();
  const int64_t rows = (int64_t)blocks * HB_BLOCK_SIZE, M = std::min<int64_t>(pad_to(rows, rows <= 1024 ? 128 : 512), m->expand_blocks * HB_BLOCK_SIZE);
  auto it = m->expand_plans.find((int)M);
  if (it != m->expand_plans.end()) { *out = &it->second; return HB_OK; }
  std::vector<TcGemmPlan> p(m->layers.size());
  size_t ws = 0;
  for (size_t i = 0; i < m->layers.size(); ++i) {
    if (!m->layers[i].expand) continue;
    const AttentionSpec& a = m->spec.layers[i].mixer.attn;
    const TcHeads h = expand_rows(a);
    const int rc = gemm_tc_plan(&p[i], m->expand_latent, m->layers[i].ukv, M, h.ldy, a.rank, kEpiStore, false, e->device, 0, nullptr, &h);
    if (rc) return rc;
    ws = std::max(ws, p[i].workspace_bytes());
  }
  const int rc = ensure_gemm_workspace(e, ws);
  if (rc) return rc;
  *out = &m->expand_plans.emplace((int)M, std::move(p)).first->second;
  return HB_OK;
}

// cap * tanh(z / cap), the logits' last step
static GatedAct logit_act(const LayeredSpec& s) {
  GatedAct a;
  a.form = GatedAct::kTanh;
  a.limit = s.logit_cap;
  a.single = 1;
  return a;
}

static int layered_head_plan(hb_engine* e, int want, TcGemmPlan** out) {
  LayeredModel* m = e->lm.get();
  const int M = (int)std::min<int64_t>(row_bucket(want), pad_to(e->max_logits_rows, 16));
  auto it = m->head_plans.find(M);
  if (it != m->head_plans.end()) { *out = &it->second; return HB_OK; }
  TcGemmPlan p;
  int rc = gemm_tc_plan(&p, m->hf, m->head.w, M, m->head.N, m->head.K, m->spec.logit_cap > 0.f ? kEpiAct : kEpiStore, true, e->device);
  if (rc) return rc;
  if (m->spec.logit_cap > 0.f) p.act = logit_act(m->spec);
  if ((rc = ensure_gemm_workspace(e, p.workspace_bytes()))) return rc;
  *out = &m->head_plans.emplace(M, p).first->second;
  return HB_OK;
}

static int layered_prepare(hb_engine* e, const StepBatch& batch, StepExec* x) {
  LayeredModel* m = e->lm.get();
  if ((int)batch.segs.size() > m->max_segs)
    return fail(HB_ERR_INVALID_ARG, "%zu sequences in one step, %d at most", batch.segs.size(), m->max_segs);
  LayeredStep& s = x->layered;
  s.rows = batch.rows;
  s.segs = (int)batch.segs.size();
  s.want = (int)batch.want.size();
  s.decode = s.rows == s.segs;
  for (const StepSeg& t : batch.segs) {
    if (t.n <= kShortSegment) ++s.n_short;
    else { ++s.n_long; s.n_chunks += (t.n + kRecChunk - 1) / kRecChunk; }
    if (t.n == 1) ++s.n_token_rows;
  }
  // expanded segments: as many as the buffers hold
  std::vector<int32_t> expand_base(batch.segs.size(), -1);
  s.n_not_expanded = s.rows;
  for (int g = 0; g < s.segs; ++g) {
    const StepSeg& t = batch.segs[g];
    const int64_t blocks = (t.pos0 + t.n - 1) / HB_BLOCK_SIZE + 1;
    if (t.n >= kExpandTokens && s.n_expand + blocks <= m->expand_blocks) {
      expand_base[g] = s.n_expand;
      s.n_expand += (int)blocks;
      s.n_not_expanded -= t.n;
    }
  }
  auto cut = [&](int g, const TileKind& k) {  // whether a segment is cut into tiles of this kind
    return batch.segs[g].n > 1 && (k.which == TileKind::kAll || (k.which == TileKind::kExpanded) == (expand_base[g] >= 0));
  };
  for (int g = 0; g < s.segs; ++g)
    for (size_t k = 0; k < m->tile_kinds.size(); ++k)
      if (cut(g, m->tile_kinds[k])) s.n_tiles[k] += (batch.segs[g].n + m->tile_kinds[k].positions - 1) / m->tile_kinds[k].positions;
  if (m->spec.post_norm) {
    s.run_rows = residual_run(s.rows);
    for (const StepSeg& t : batch.segs) s.n_runs += (t.n + s.run_rows - 1) / s.run_rows;
  }
  x->rows = batch.rows;
  x->logits_compact = true;
  x->input_bytes = layered_layout(e, &s);
  if (x->input_bytes > e->inputs_bytes) return fail(HB_ERR_INVALID_ARG, "step inputs of %zu bytes", x->input_bytes);
  uint8_t* in = e->h_inputs;
  uint32_t* ids = (uint32_t*)(in + s.off_ids);
  int32_t* pos = (int32_t*)(in + s.off_pos);
  int64_t* slots = (int64_t*)(in + s.off_slots);
  int32_t* row_seg = (int32_t*)(in + s.off_row_seg);
  SegInfo* seg = (SegInfo*)(in + s.off_seg);
  int32_t* shorts = (int32_t*)(in + s.off_short);
  RowRange* longs = (RowRange*)(in + s.off_long);
  RowRange* chunks = (RowRange*)(in + s.off_chunk);
  int32_t* row_list = (int32_t*)(in + s.off_row_list);
  int at_short = 0, at_long = s.n_short, n_long = 0, n_chunks = 0, n_tiles[kTileKinds] = {0}, at_token = 0, at_row = s.n_token_rows;
  int32_t* tables = (int32_t*)(in + s.off_tables);
  RowRange* runs = (RowRange*)(in + s.off_run);
  int n_runs = 0;
  for (int g = 0; g < s.segs; ++g) {
    const StepSeg& t = batch.segs[g];
    seg[g] = {t.row0, t.n, (int32_t)t.pos0, t.state_slot};
    if (t.n <= kShortSegment) {
      shorts[at_short++] = g;
    } else {
      shorts[at_long++] = g;
      RowRange& l = longs[n_long++];
      l = {g, n_chunks, 0, 0};
      for (int i = 0; i < t.n; i += kRecChunk)
        chunks[n_chunks++] = {g, t.row0 + i, std::min(kRecChunk, t.n - i), l.n++};
    }
    if (s.run_rows)
      for (int i = 0; i < t.n; i += s.run_rows) runs[n_runs++] = {g, t.row0 + i, std::min(s.run_rows, t.n - i), i / s.run_rows};
    for (size_t k = 0; k < m->tile_kinds.size(); ++k) {
      if (!cut(g, m->tile_kinds[k])) continue;
      RowRange* tiles = (RowRange*)(in + s.off_tile[k]);
      const int size = m->tile_kinds[k].positions;
      for (int i = 0; i < t.n; i += size) tiles[n_tiles[k]++] = {g, t.row0 + i, std::min(size, t.n - i), i / size};
    }
    for (int i = 0; i < t.n; ++i) {
      const int64_t p = t.pos0 + i;
      ids[t.row0 + i] = t.tokens[i];
      pos[t.row0 + i] = (int32_t)p;
      slots[t.row0 + i] = t.blocks[p / HB_BLOCK_SIZE] * HB_BLOCK_SIZE + p % HB_BLOCK_SIZE;
      row_seg[t.row0 + i] = g;
      row_list[t.n == 1 ? at_token++ : at_row++] = t.row0 + i;
    }
    const int64_t need = (t.pos0 + t.n - 1) / HB_BLOCK_SIZE + 1;
    int32_t* row = tables + (size_t)g * e->max_blocks_per_seq;
    for (int64_t k = 0; k < need; ++k) row[k] = (int32_t)t.blocks[k];
    if (s.n_expand) ((int32_t*)(in + s.off_expand_base))[g] = expand_base[g];
    if (expand_base[g] >= 0) std::copy(row, row + need, (int32_t*)(in + s.off_expand_list) + expand_base[g]);
  }
  std::copy(batch.want.begin(), batch.want.end(), (int32_t*)(in + s.off_want));
  if (e->use_tc) {
    int rc;
    if ((rc = layered_plans(e, s.rows, &s.plans))) return rc;
    if (s.n_expand && (rc = layered_expand_plans(e, s.n_expand, &s.expand_plans))) return rc;
    if (s.want && (rc = layered_head_plan(e, s.want, &s.head_plan))) return rc;
  }
  // a step of decoded tokens whose logits are all wanted replays from a graph
  if (s.decode && s.want == s.rows) {
    LayeredGraph& g = m->graphs[s.rows];
    x->graph = &g.exec;
    x->graph_launches = &g.launches;
  }
  return HB_OK;
}

static int layered_issue(hb_engine* e, const StepExec& x) {
  LayeredModel* m = e->lm.get();
  const LayeredSpec& sp = m->spec;
  const LayeredStep& s = x.layered;
  cudaStream_t st = e->stream;
  const uint8_t* in = e->d_inputs;
  const uint32_t* ids = (const uint32_t*)(in + s.off_ids);
  const int32_t* pos = (const int32_t*)(in + s.off_pos);
  const int64_t* slots = (const int64_t*)(in + s.off_slots);
  const SegInfo* seg = (const SegInfo*)(in + s.off_seg);
  const int S = sp.streams;
  const int64_t W = sp.width, rows = s.rows;
  const size_t es = e->es;
  int rc;
  auto gemm = [&](const std::vector<TcGemmPlan>* plans, size_t i, void* Y, const void* X, const LayeredLinear& w,
                  bool f32) -> int {
    ++e->last_launches;
    if (e->use_tc) return gemm_tc_run((*plans)[i], st, Y, (*plans)[i].N, e->d_gemm_ws, e->d_err);
    return gemm_simt(st, Y, X, w.w, rows, w.N, w.K, e->dtype, f32);
  };
  const LayeredPlans* pl = s.plans;
  auto grouped = [&](const std::vector<TcGemmPlan>* plans, size_t i, void* Y, const void* X, const LayeredLinear& w,
                     const TcGroups& g) -> int {
    ++e->last_launches;
    if (e->use_tc) return gemm_tc_run((*plans)[i], st, Y, (*plans)[i].ldy, e->d_gemm_ws, e->d_err, nullptr, m->moe_tiles);
    return gemm_simt_grouped(st, Y, X, w.w, w.N, w.K, e->dtype, false, g, m->moe_tiles);
  };
  // the experts' outputs of every row, side by side in moe_y
  const void* ffn_in = sp.post_norm ? m->h2 : m->h;
  auto experts = [&](size_t i, const ExpertsSpec& x, const LayeredExperts& w, const GatedAct& shared_act) -> int {
    const bool shared = w.shared_ffp > 0;
    const TcGroups g = moe_groups(x, shared, e->use_tc ? row_bucket((int)rows) : (int)rows, e->use_tc);
    const TcGroups up = up_groups(g, w, shared_act), down = down_groups(g, w);
    const MoeRouting r = moe_args(m, x, w, g);
    prof_mark(e, kCatRouting);
    if ((rc = moe_route_top(st, r, ffn_in, m->Hp, w.router, w.router_bias, rows, W, e->dtype))) return rc;
    if ((rc = moe_gather(st, r, m->moe_x, ffn_in, m->Hp, rows, e->dtype))) return rc;
    e->last_launches += 2;
    prof_mark(e, kCatExpertsUp);
    if (e->use_tc) {
      if ((rc = grouped(&pl->moe_gate_up, i, m->moe_act, m->moe_x, w.gate_up, up))) return rc;
    } else {
      TcGroups raw = up;
      raw.ldy = (x.act.single ? 1 : 2) * w.ld();
      if ((rc = grouped(nullptr, i, m->moe_gu, m->moe_x, w.gate_up, raw))) return rc;
      if ((rc = gated_act_grouped(st, m->moe_act, w.ld(), m->moe_gu, raw.ldy, w.ffp, x.act, e->dtype, up, m->moe_tiles))) return rc;
      ++e->last_launches;
    }
    prof_mark(e, kCatExpertsDown);
    return grouped(pl ? &pl->moe_down : nullptr, i, m->moe_y, m->moe_act, w.down, down);
  };
  auto at = [&](void* p, int64_t elements) { return (void*)((uint8_t*)p + (size_t)elements * es); };

  // post_norm: one boundary, and what lies ahead of it
  const RowRange* runs = (const RowRange*)(in + s.off_run);
  float *x_now = m->results, *x_next = m->x;  // the residual, where the next boundary leaves it
  const SublayerMix* read = nullptr;          // the sublayer whose input was formed last
  auto residual = [&](ResidualStep r, const float* norm, const SublayerMix* next, void* h) -> int {
    r.ld_y = m->Hp;
    r.norm = norm; r.groups = sp.norm_groups; r.eps = sp.eps;
    r.taps = std::max(1, sp.input_taps);
    if (read) r.past = read->conv_state;
    if (next) {
      r.conv = next->conv; r.state = next->conv_state;
      r.h = h; r.ld_h = m->Hp;
    }
    read = next;
    r.rows = rows;
    if (rows > kResidualTwo) {
      r.scale = m->part_scale;
      r.mixed = m->y2;
    }
    e->last_launches += residual_in_two(r) ? 2 : 1;
    prof_mark(e, kCatNorm);
    return residual_step(st, r, runs, s.n_runs, seg, W, e->dtype);
  };
  // the sublayer's output back into the residual; `layer` >= 0: it ends this layer
  auto post = [&](ResidualStep r, const float* norm, int64_t layer, const SublayerMix* next, void* h) -> int {
    r.x = x_now;
    r.x_out = x_next;
    if (layer >= 0 && m->layers[layer].depth) {
      r.earlier = m->results; r.step = m->row_cap * W; r.n_earlier = (int)layer + 1;
      r.depth = m->layers[layer].depth;
      r.result = m->results + (layer + 1) * r.step;
    }
    x_now = x_next;
    x_next = x_next == m->x ? m->x2 : m->x;
    return residual(r, norm, next, h);
  };

  prof_mark(e, kCatOther);
  if (sp.post_norm) {
    ResidualStep r;
    r.embed = m->embed; r.ids = ids; r.vocab = sp.vocab;
    r.x_out = m->results;
    if ((rc = residual(r, m->embed_norm, &m->layers[0].sub1, m->h))) return rc;
  } else if ((rc = streams_embed(st, m->x, m->h, m->embed, m->pos, ids, pos, m->layers[0].sub1.in, m->layers[0].sub1.norm, sp.norm_offset,
                          rows, S, W, m->Hp, sp.vocab, sp.max_positions, sp.eps, e->dtype, sp.embed_scale))) return rc;
  ++e->last_launches;
  for (size_t i = 0; i < m->layers.size(); ++i) {
    LayeredLayer& l = m->layers[i];
    const LayerSpec& lsp = sp.layers[i];
    const MixerSpec& mx = lsp.mixer;
    prof_mark(e, kCatGemm);
    if ((rc = gemm(pl ? &pl->proj : nullptr, i, m->proj, m->h, l.proj, false))) return rc;
    const int64_t ldp = l.proj.N;
    float* y = m->y1;
    if (mx.has_attn) {
      const SpanAttention a = span_args(e, i, s);
      const AttentionSpec& as = mx.attn;
      // one product per head of latent attention
      auto heads = [&](const std::vector<TcGemmPlan>* plans, void* Y, const void* X, const void* w, int64_t N, int64_t K,
                       const TcHeads& h) -> int {
        ++e->last_launches;
        prof_mark(e, kCatLatent);
        if (l.latent_tc) return gemm_tc_run((*plans)[i], st, Y, h.ldy, e->d_gemm_ws, e->d_err);
        return gemm_simt_heads(st, Y, X, w, rows, N, K, e->dtype, false, h);
      };
      if (as.q_rank) {
        prof_mark(e, kCatNorm);
        if ((rc = parts_norm(st, m->q_latent, l.uq.K, at(m->proj, mx.aq.offset), ldp, false, nullptr, l.q_latent_norm, rows, 1, as.q_rank,
                             sp.eps, e->dtype))) return rc;
        ++e->last_launches;
        prof_mark(e, kCatGemm);
        if ((rc = gemm(pl ? &pl->uq : nullptr, i, m->q, m->q_latent, l.uq, false))) return rc;
      }
      const bool expand = l.expand && s.n_expand, latent = as.rank && !(expand && s.n_not_expanded == 0);
      if (latent && (rc = heads(pl ? &pl->latent_q : nullptr, m->latent_q, query_rows(e, i), l.uk_t, as.rank, as.dim,
                                 latent_q_heads(l, as)))) return rc;
      prof_mark(e, kCatRopeKv);
      AttentionPrep prep;
      if (as.rank) rc = latent_prepare(st, latent_args(e, i, s), rows, e->dtype);
      else if (as.kv_from >= 0 && !l.rotation && !l.q_bias) rc = HB_OK;  // queries as projected, keys of another layer
      else if (prep_args(e, i, s, &prep)) rc = attention_prepare(st, prep, rows, e->dtype);
      else rc = span_kv_write(st, a, at(m->proj, mx.ak.offset), at(m->proj, mx.av.offset), ldp, slots, rows, e->dtype);
      if (rc) return rc;
      prof_mark(e, kCatAttention);
      if ((!as.rank || latent) && (rc = issue_attention(e, a, l.tile_kind, s))) return rc;
      if (latent && (rc = heads(pl ? &pl->latent_v : nullptr, m->attn, m->latent_o, l.uv, as.vdim, as.rank, latent_v_heads(l, as))))
        return rc;
      if (expand) {  // (after the product above, which writes all rows)
        prof_mark(e, kCatLatent);
        if ((rc = latent_gather(st, m->expand_latent, e->kc[l.kv_pool], (const int32_t*)(in + s.off_expand_list), s.n_expand,
                                as.key_width(), e->num_blocks, e->dtype))) return rc;
        if ((rc = gemm_tc_run((*s.expand_plans)[i], st, m->expand_kv, expand_rows(as).ldy, e->d_gemm_ws, e->d_err))) return rc;
        prof_mark(e, kCatAttention);
        if ((rc = span_attention_tiles(st, expanded_args(e, i, s), (const RowRange*)(in + s.off_tile[l.expand_kind]),
                                       s.n_tiles[l.expand_kind]))) return rc;
        e->last_launches += 3;
      }
      prof_mark(e, kCatGemmO);
      if ((rc = gemm(pl ? &pl->attn_o : nullptr, i, y, m->attn, l.attn_o, true))) return rc;
      ++e->last_launches;  // the K/V write
      y = m->y2;
    }
    if (mx.has_rec) {
      const RecurrenceSpec& rs = mx.rec;
      Recurrence r;
      r.p = m->proj; r.ld = ldp;
      r.off_q = (int)mx.rq.offset; r.off_k = (int)mx.rk.offset; r.off_v = (int)mx.rv.offset; r.off_a1 = (int)mx.ra1.offset;
      r.heads = rs.heads; r.dim = rs.dim; r.vdim = rs.vdim;
      r.q_scale = rs.q_scale; r.silu_qkv = rs.silu_qkv ? 1 : 0;
      r.decay = l.decay; r.a2 = l.a2; r.a2_bias = l.a2_bias; r.rank = rs.rank; r.inv_tau = (float)(1.0 / rs.tau);
      r.qk_heads = rs.qk_heads;
      if (rs.per_token_decay) {
        ShortConv c;
        c.p = m->proj; c.ld = ldp; c.off = (int)mx.rx.offset; c.channels = (int)rs.conv_channels(); c.taps = rs.conv_taps;
        c.w = l.conv_w; c.bias = l.conv_b; c.out = m->conv; c.ld_out = pad8(rs.conv_channels());
        c.state = l.conv_state; c.segs = seg;
        prof_mark(e, kCatConv);
        if ((rc = short_conv(st, c, (const int32_t*)(in + s.off_short), s.n_short, (const RowRange*)(in + s.off_chunk), s.n_chunks,
                             e->dtype))) return rc;
        e->last_launches += (s.n_short ? 1 : 0) + (s.n_chunks ? 1 : 0);
        r.p = m->conv; r.ld = c.ld_out;
        r.off_v = 0; r.off_k = rs.heads * rs.vdim; r.off_q = r.off_k + rs.qk_heads * rs.dim;
        r.dt = at(m->proj, mx.rdt.offset); r.ld_dt = ldp;
        r.dt_bias = l.dt_bias; r.a_log = l.a_log; r.skip = l.skip;
      }
      r.state = l.state; r.o = m->o; r.ld_o = (int64_t)rs.heads * rs.vdim; r.segs = seg;
      prof_mark(e, kCatRecurrence);
      if ((rc = issue_recurrence(e, r, s))) return rc;
      prof_mark(e, kCatNorm);
      GroupNorm n;
      n.groups = rs.norm_per_head ? rs.heads : std::max(1, rs.gated_norm_groups);
      n.size = rs.heads * rs.vdim / n.groups;
      n.gate_silu = rs.gate_silu; n.gate_first = n.own_weights = rs.gated_norm_groups > 0;
      n.eps = sp.eps;
      if ((rc = gated_group_norm(st, m->rec, l.rec_o.K, m->o, r.ld_o, at(m->proj, mx.rg.offset), ldp, l.rec_norm, rows, n, e->dtype)))
        return rc;
      prof_mark(e, kCatGemmO);
      if ((rc = gemm(pl ? &pl->rec_o : nullptr, i, y, m->rec, l.rec_o, true))) return rc;
      ++e->last_launches;  // the gated norm
    }
    const bool both = mx.has_attn && mx.has_rec;
    const SublayerMix* next = lsp.has_ffn() ? &l.sub2 : (i + 1 < m->layers.size() ? &m->layers[i + 1].sub1 : nullptr);
    auto boundary = [&](const SublayerMix& q, const float* y, bool two, StreamMix sm) -> int {
      sm.mix = q.mix; sm.out = q.out;
      sm.next_in = next ? next->in : nullptr;
      sm.next_norm = next ? next->norm : nullptr;
      sm.w1 = l.attn_out_norm; sm.w2 = l.rec_out_norm;
      sm.norm_offset = sp.norm_offset;
      ++e->last_launches;
      prof_mark(e, kCatNorm);
      return streams_mix(st, m->x, m->h, y, two ? m->y2 : nullptr, m->Hp, sm, rows, S, W, m->Hp, sp.eps, e->dtype);
    };
    const bool more = i + 1 < m->layers.size();
    if (sp.post_norm) {
      ResidualStep r;
      r.y = m->y1;
      if (!lsp.has_ffn()) {
        if ((rc = post(r, l.sub1.norm, (int64_t)i, more ? &m->layers[i + 1].sub1 : nullptr, m->h))) return rc;
        continue;
      }
      if ((rc = post(r, l.sub1.norm, -1, &l.sub2, m->h2))) return rc;
    }
    StreamMix mixed{};
    mixed.bias = l.o_bias;
    if (!sp.post_norm && (rc = boundary(l.sub1, m->y1, both, mixed))) return rc;
    if (!lsp.has_ffn()) continue;
    next = i + 1 < m->layers.size() ? &m->layers[i + 1].sub1 : nullptr;
    StreamMix fed{};
    if (lsp.moe.experts) {
      if ((rc = experts(i, lsp.moe, l.moe, lsp.ffn.act))) return rc;
      fed.expert_y = m->moe_y; fed.expert_place = m->moe_place; fed.expert_weight = m->moe_weight;
      fed.top = lsp.moe.top + (l.moe.shared_ffp ? 1 : 0);
    } else {
      prof_mark(e, kCatGemmGateUp);
      if (e->use_tc) {
        if ((rc = gemm(&pl->gate_up, i, m->act, ffn_in, l.gate_up, false))) return rc;
      } else {
        if ((rc = gemm(nullptr, i, m->gu, ffn_in, l.gate_up, false))) return rc;
        if ((rc = gated_act(st, m->act, m->gu, rows, l.ffp, lsp.ffn.act, e->dtype, l.gate_b, l.up_b))) return rc;
        ++e->last_launches;
      }
      prof_mark(e, kCatGemmDown);
      if ((rc = gemm(pl ? &pl->down : nullptr, i, m->y1, m->act, l.down, true))) return rc;
    }
    if (sp.post_norm) {
      ResidualStep r;
      if (lsp.moe.experts) {
        r.expert_y = fed.expert_y; r.expert_place = fed.expert_place; r.expert_weight = fed.expert_weight; r.top = fed.top;
        r.input = m->h2; r.ld_input = m->Hp;
      } else {
        r.y = m->y1;
      }
      if ((rc = post(r, l.sub2.norm, (int64_t)i, more ? &m->layers[i + 1].sub1 : nullptr, m->h))) return rc;
      continue;
    }
    fed.bias = l.down_b;
    if ((rc = boundary(l.sub2, lsp.moe.experts ? nullptr : m->y1, false, fed))) return rc;
  }
  if (s.want) {
    prof_mark(e, kCatNorm);
    if (sp.post_norm) {
      if ((rc = parts_norm(st, m->hf, m->Hp, x_now, W, true, (const int32_t*)(in + s.off_want), m->final_norm, s.want, sp.norm_groups,
                           W / sp.norm_groups, sp.eps, e->dtype))) return rc;
    } else if ((rc = streams_final(st, m->hf, m->x, (const int32_t*)(in + s.off_want), m->final_norm, sp.norm_offset, s.want, S, W, m->Hp, sp.eps,
                            e->dtype, sp.logit_scale))) return rc;
    prof_mark(e, kCatGemmLmHead);
    if (e->use_tc) rc = gemm_tc_run(*s.head_plan, st, e->d_logits, sp.vocab, e->d_gemm_ws, e->d_err);
    else rc = gemm_simt(st, e->d_logits, m->hf, m->head.w, s.want, m->head.N, m->head.K, e->dtype, true);
    if (rc) return rc;
    if (!e->use_tc && sp.logit_cap > 0.f) {
      if ((rc = gated_act(st, e->d_logits, e->d_logits, s.want, sp.vocab, logit_act(sp), HB_F32))) return rc;
      ++e->last_launches;
    }
    prof_mark(e, kCatOther);
    if ((rc = hb_argmax(st, e->d_next, e->d_logits, s.want, sp.vocab, HB_F32))) return rc;
    e->last_launches += 3;
  }
  prof_mark(e, -1);
  return HB_OK;
}

// Bytes one decode step moves: weights once, K/V and recurrent states of the sequences, streams.
static double layered_step_bytes(const hb_engine* e, const int32_t* ctx_lens, int64_t n_seqs) {
  const LayeredModel* m = e->lm.get();
  const LayeredSpec& s = m->spec;
  const double es = (double)e->es, n = (double)n_seqs;
  double w = (double)m->head.N * m->head.K * es + 2.0 * n * s.width * es;
  for (size_t i = 0; i < s.layers.size(); ++i) {
    const LayeredLayer& l = m->layers[i];
    for (const LayeredLinear* q : {&l.proj, &l.uq, &l.attn_o, &l.rec_o, &l.gate_up, &l.down}) w += (double)q->N * q->K * es;
    const MixerSpec& mx = s.layers[i].mixer;
    if (mx.has_attn) {
      const AttentionSpec& a = mx.attn;
      const double per_key = a.rank ? a.key_width() * es : a.values_are_keys ? a.kv_heads * a.dim * es + 4.0 : a.kv_heads * (a.dim + a.vdim) * es;
      if (a.rank) w += (double)a.heads * (a.dim + a.vdim) * a.rank * es;
      for (int64_t k = 0; k < n_seqs; ++k) {
        const int64_t ctx = ctx_lens ? ctx_lens[k] : 0;
        int64_t seen = ctx;
        if (a.chunk > 0) seen = ctx % a.chunk;
        else if (a.window > 0) seen = std::min<int64_t>(ctx, (int64_t)a.window + std::min<int64_t>(a.keep_first, std::max<int64_t>(0, ctx - a.window)));
        w += ((double)seen + 1.0) * per_key;
      }
    }
    if (mx.has_rec && mx.rec.per_token_decay) w += n * 2.0 * (mx.rec.conv_taps - 1) * mx.rec.conv_channels() * es;
    if (mx.has_rec) w += n * 2.0 * mx.rec.heads * mx.rec.dim * mx.rec.vdim * 4.0;
    w += n * (s.layers[i].has_ffn() ? 2.0 : 1.0) * 2.0 * s.streams * s.width * 4.0;
    if (s.input_taps) w += n * (s.layers[i].has_ffn() ? 2.0 : 1.0) * s.input_taps * s.width * 4.0;
    if (l.depth) w += n * ((double)i + 2.0) * s.width * 4.0;
    if (const ExpertsSpec& x = s.layers[i].moe; x.experts)  // the experts a random batch chooses
      w += x.experts * (1.0 - std::pow(1.0 - 1.0 / x.experts, n * x.picks())) *
               ((double)l.moe.gate_up.N * l.moe.gate_up.K + (double)l.moe.down.N * l.moe.down.K) * es +
           ((double)x.outputs() * s.width + (double)l.moe.shared_gate_up.N * l.moe.shared_gate_up.K +
            (double)l.moe.shared_down.N * l.moe.shared_down.K) * es;
  }
  return w;
}

static double layered_gemm_bytes(const hb_engine* e, int64_t rows) {
  const LayeredModel* m = e->lm.get();
  const double es = (double)e->es, b = (double)rows;
  auto lin = [&](const LayeredLinear& q, double n_out, double out_es) {
    return q.w ? ((double)q.N * q.K + b * q.K) * es + b * n_out * out_es : 0.0;
  };
  auto latent = [&](const AttentionSpec& a) {
    return a.heads * ((double)(a.dim + a.vdim) * a.rank + b * (a.dim + 2.0 * a.rank + a.vdim)) * es;
  };
  double t = lin(m->head, (double)m->head.N, 4.0);
  for (size_t i = 0; i < m->layers.size(); ++i) {
    const LayeredLayer& l = m->layers[i];
    t += lin(l.proj, (double)l.proj.N, es) + lin(l.uq, (double)l.uq.N, es) + lin(l.attn_o, (double)l.attn_o.N, 4.0) + lin(l.rec_o, (double)l.rec_o.N, 4.0) +
         (m->spec.layers[i].mixer.attn.rank ? latent(m->spec.layers[i].mixer.attn) : 0.0) + lin(l.gate_up, (double)l.ffp, es) + lin(l.down, (double)l.down.N, 4.0);
    if (const ExpertsSpec& x = m->spec.layers[i].moe; x.experts) {
      const double picks = b * x.picks(), active = x.experts * (1.0 - std::pow(1.0 - 1.0 / x.experts, picks));
      const LayeredExperts& w = l.moe;
      t += active * ((double)w.gate_up.N * w.gate_up.K + (double)w.down.N * w.down.K) * es +
           picks * ((double)w.gate_up.K + 2.0 * w.ffp + (double)w.down.N) * es +
           lin(w.shared_gate_up, (double)w.shared_ffp, es) + lin(w.shared_down, (double)w.shared_down.N, es);
    }
  }
  return t;
}

const ModelFamily kLayeredFamily = {"layered", layered_serves, layered_configure, layered_load, layered_alloc_runtime,
                                    layered_prepare, layered_issue, layered_step_bytes, layered_gemm_bytes};

}  // namespace hb
