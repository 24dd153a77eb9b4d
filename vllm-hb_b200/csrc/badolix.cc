// Badolix: the reader of its config.json and tensor names.
//
// A pre-norm decoder whose sublayers' outputs carry one factor, with a scaled embedding that is also the
// output projection.  A layer's mixer is "attention" (rotated halves, capped scores, a window that
// keeps its first tokens, possibly another layer's keys and values), "latent_attention" (keys and values
// out of one cached latent) or "mamba2" (selective state space); its feed-forward is dense with biases,
// a mixture of experts chosen by sigmoid scores within groups, or none.
#include <climits>
#include <cmath>

#include "design_reader.h"

namespace hb {

bool is_badolix(const Json& config) { return config.string_or("architecture", "") == "Badolix"; }

static int read_attention(const Json* m, const std::string& t, size_t layer, const LayeredSpec& spec, MixerSpec* out) {
  AttentionSpec& a = out->attn;
  out->has_attn = true;
  a.heads = (int)int_of(m, "heads");
  a.kv_heads = (int)int_of(m, "kv_heads");
  a.dim = (int)int_of(m, "dim");
  a.vdim = (int)int_of(m, "vdim");
  a.scale = (float)m->number_or("scale", 0);
  a.softcap = (float)m->number_or("softcap", 0);
  if (a.heads < 1 || a.kv_heads < 1 || a.heads % a.kv_heads || a.dim < 1 || a.vdim < 1 || !m->get("scale") || a.softcap < 0)
    return fail(HB_ERR_INVALID_ARG, "%s: bad attention sizes", t.c_str());
  if (const Json* mask = object_of(*m, "mask")) {
    const double size = mask->number_or("size", 0), keep = mask->number_or("keep_first", 0);
    if ((mask->get("size") && !(size >= 1)) || keep < 0) return fail(HB_ERR_INVALID_ARG, "%s: bad attention mask", t.c_str());
    a.window = (int)(size > INT_MAX / 2 ? 0 : size);
    a.keep_first = (int)(keep > INT_MAX / 2 ? INT_MAX / 2 : keep);
  }
  int64_t off = 0;
  place(&out->aq, t + "q", (int64_t)a.heads * a.dim, &off);
  if (const Json* from = m->get("kv_from"); from && from->kind == Json::Num) {
    const double j = from->num;
    const MixerSpec* other = j >= 0 && j < (double)layer && j == std::floor(j) ? &spec.layers[(size_t)j].mixer : nullptr;
    if (!other || !other->has_attn || other->attn.rank || other->attn.kv_from >= 0 || other->attn.kv_heads != a.kv_heads ||
        other->attn.dim != a.dim || other->attn.vdim != a.vdim)
      return fail(HB_ERR_INVALID_ARG, "%s: layer %g has no keys and values for it", t.c_str(), j);
    a.kv_from = (int)j;
  } else {
    place(&out->ak, t + "k", (int64_t)a.kv_heads * a.dim, &off);
    place(&out->av, t + "v", (int64_t)a.kv_heads * a.vdim, &off);
  }
  out->attn_o = t + "o";
  const Json* rot = object_of(*m, "rot");
  return rot ? read_rotation(rot, t, a.dim, false, true, &a) : HB_OK;
}

static int read_latent(const Json* m, const std::string& t, MixerSpec* out) {
  AttentionSpec& a = out->attn;
  out->has_attn = true;
  a.heads = a.kv_heads = (int)int_of(m, "heads");
  a.dim = (int)int_of(m, "dim");
  a.rot_dim = (int)int_of(m, "rot_dim");
  a.vdim = (int)int_of(m, "vdim");
  a.rank = (int)int_of(m, "kv_rank");
  a.scale = (float)m->number_or("scale", 0);
  if (a.heads < 1 || a.dim < 1 || a.rot_dim < 0 || a.vdim < 1 || a.rank < 1 || !m->get("scale"))
    return fail(HB_ERR_INVALID_ARG, "%s: bad attention sizes", t.c_str());
  int64_t off = 0;
  place(&out->aq, t + "q", (int64_t)a.heads * (a.dim + a.rot_dim), &off);
  place(&out->ak, t + "dkv", (int64_t)a.rank + a.rot_dim, &off);
  out->attn_latent_norm = t + "dkv.norm";
  out->attn_uk = t + "uk";
  out->attn_uv = t + "uv";
  out->attn_o = t + "o";
  const Json* rot = object_of(*m, "rot");
  return rot ? read_rotation(rot, t, a.rot_dim, true, true, &a) : HB_OK;
}

static int read_mamba2(const Json* m, const std::string& t, MixerSpec* out) {
  RecurrenceSpec& r = out->rec;
  out->has_rec = true;
  r.heads = (int)int_of(m, "heads");
  r.dim = (int)int_of(m, "state");
  r.vdim = (int)int_of(m, "vdim");
  r.qk_heads = (int)int_of(m, "groups");
  r.conv_taps = (int)int_of(m, "conv");
  r.gated_norm_groups = (int)int_of(m, "norm_groups");
  r.per_token_decay = true;
  r.gate_silu = true;
  const int64_t inner = (int64_t)r.heads * r.vdim;
  if (r.heads < 1 || r.dim < 1 || r.vdim < 1 || r.qk_heads < 1 || r.heads % r.qk_heads || r.conv_taps < 1 ||
      r.gated_norm_groups < 1 || inner % r.gated_norm_groups)
    return fail(HB_ERR_INVALID_ARG, "%s: bad recurrence sizes", t.c_str());
  // rows of the one input matrix: gate, [v | k | q] of the convolution, steps
  const int64_t total = inner + r.conv_channels() + r.heads;
  int64_t off = 0, first = 0;
  for (auto p : {std::make_pair(&out->rg, inner), std::make_pair(&out->rx, r.conv_channels()), std::make_pair(&out->rdt, (int64_t)r.heads)}) {
    place(p.first, t + "in", p.second, &off);
    p.first->first = first;
    p.first->of = total;
    first += p.second;
  }
  out->rec_conv = t + "conv";
  out->rec_conv_bias = t + "conv.b";
  out->rec_dt_bias = t + "dt_bias";
  out->rec_a_log = t + "A_log";
  out->rec_skip = t + "D";
  out->rec_norm = t + "norm";
  out->rec_o = t + "o";
  return HB_OK;
}

static int read_mlp(const Json& mlp, const std::string& t, LayerSpec* l) {
  const std::string kind = mlp.string_or("kind", "dense");
  if (kind == "dense") {
    FeedForwardSpec& f = l->ffn;
    f.ff = int_of(&mlp, "ff");
    if (f.ff < 1) return fail(HB_ERR_INVALID_ARG, "%s: ff must be positive", t.c_str());
    f.gate = t + "gate";
    f.up = t + "up";
    f.down = t + "down";
    f.gate_bias = f.gate + ".b";
    f.up_bias = f.up + ".b";
    f.down_bias = f.down + ".b";
    return HB_OK;
  }
  if (kind != "moe") return fail(HB_ERR_INVALID_ARG, "%s: unknown kind '%s'", t.c_str(), kind.c_str());
  const Json *router = object_of(mlp, "router"), *expert = object_of(mlp, "expert");
  if (!router || !expert) return fail(HB_ERR_INVALID_ARG, "%s: a mixture needs router and expert", t.c_str());
  ExpertsSpec& x = l->moe;
  x.experts = (int)int_of(router, "experts");
  x.top = (int)int_of(router, "top");
  x.ff = int_of(expert, "ff");
  x.sigmoid = true;
  if (const Json* g = object_of(*router, "groups")) {
    x.groups = (int)int_of(g, "count");
    x.keep = (int)int_of(g, "keep");
  }
  if (x.experts < 1 || x.top < 1 || x.ff < 1 || x.groups < 1 || x.experts % x.groups || x.keep < 1 || x.keep > x.groups ||
      x.top > x.experts / x.groups * x.keep)
    return fail(HB_ERR_INVALID_ARG, "%s: %d of %d experts, %d of %d groups", t.c_str(), x.top, x.experts, x.keep, x.groups);
  x.router = t + "router";
  x.prefix = t + "e";
  return HB_OK;
}

int read_badolix(const Json& config, LayeredSpec* out) {
  out->design = "Badolix";
  out->width = int_of(&config, "width");
  out->vocab = int_of(&config, "vocab");
  const Json *norm = object_of(config, "norm"), *embedding = object_of(config, "embedding");
  if (!norm || !norm->get("eps")) return fail(HB_ERR_INVALID_ARG, "config.json: norm.eps is missing");
  out->eps = (float)norm->number_or("eps", 0);
  out->embed_scale = (float)(embedding ? embedding->number_or("scale", 1) : 1);
  out->residual_mult = (float)config.number_or("residual_mult", 1);
  out->logit_scale = (float)config.number_or("logit_scale", 1);
  out->embed = "embed";
  out->final_norm = "final.norm";
  const Json* layers = config.get("layers");
  if (!layers || layers->kind != Json::Arr || out->width < 1 || out->vocab < 1)
    return fail(HB_ERR_INVALID_ARG, "config.json: layers, width and vocab are needed");
  for (size_t i = 0; i < layers->arr.size(); ++i) {
    const Json& j = layers->arr[i];
    LayerSpec l;
    l.prefix = "l" + std::to_string(i) + ".";
    const Json* m = object_of(j, "mixer");
    const std::string type = j.string_or("type", ""), t = l.prefix + "mix.";
    if (!m) return fail(HB_ERR_INVALID_ARG, "config.json: layer %zu has no mixer", i);
    int rc;
    if (type == "attention") rc = read_attention(m, t, i, *out, &l.mixer);
    else if (type == "latent_attention") rc = read_latent(m, t, &l.mixer);
    else if (type == "mamba2") rc = read_mamba2(m, t, &l.mixer);
    else return fail(HB_ERR_INVALID_ARG, "config.json: layer %zu has the unknown type '%s'", i, type.c_str());
    if (rc) return rc;
    l.norm1 = l.prefix + "norm1";
    if (const Json* mlp = object_of(j, "mlp")) {
      if ((rc = read_mlp(*mlp, l.prefix + "mlp.", &l))) return rc;
      l.norm2 = l.prefix + "norm2";
    }
    out->layers.push_back(std::move(l));
  }
  if (out->layers.empty()) return fail(HB_ERR_INVALID_ARG, "config.json: no layers");
  return HB_OK;
}

}  // namespace hb
