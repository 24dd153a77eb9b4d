// Latarax: the reader of its config.json and tensor names.
//
// A decoder with learned positions, several residual streams mixed around every sublayer
// (hyper-connections), and per layer either gated linear attention ("gla") or two mixers side by
// side ("parallel": windowed attention that keeps its first tokens, and lightning attention).
#include <climits>
#include <cmath>

#include "design_reader.h"

namespace hb {

bool is_latarax(const Json& config) { return config.string_or("architecture", "") == "Latarax"; }

static int read_window(const Json* mask, AttentionSpec* a) {
  if (!mask || mask->kind == Json::Null) return HB_OK;  // every earlier position is visible
  const double size = mask->number_or("size", 0), keep = mask->number_or("keep_first", 0);
  if (mask->kind != Json::Obj || size < 0 || keep < 0) return fail(HB_ERR_INVALID_ARG, "bad attention mask");
  if (mask->get("size") && size < 1) return fail(HB_ERR_INVALID_ARG, "an attention window of %g positions", size);
  a->window = (int)(size > INT_MAX / 2 ? 0 : size);
  a->keep_first = (int)(keep > INT_MAX / 2 ? INT_MAX / 2 : keep);
  return HB_OK;
}

static int read_gla(const Json* m, const std::string& t, MixerSpec* out) {
  RecurrenceSpec& r = out->rec;
  out->has_rec = true;
  r.heads = (int)int_of(m, "heads");
  r.dim = (int)int_of(m, "dim");
  r.vdim = (int)int_of(m, "vdim");
  r.tau = m->number_or("tau", 0);
  r.low_rank_decay = true;
  r.norm_per_head = true;
  r.gate_silu = true;
  if (r.heads < 1 || r.dim < 1 || r.vdim < 1 || r.tau <= 0)
    return fail(HB_ERR_INVALID_ARG, "%s: heads, dim, vdim and tau must be positive", t.c_str());
  r.q_scale = (float)(1.0 / std::sqrt((double)r.dim));
  int64_t off = 0;
  place(&out->rq, t + "q", (int64_t)r.heads * r.dim, &off);
  place(&out->rk, t + "k", (int64_t)r.heads * r.dim, &off);
  place(&out->rv, t + "v", (int64_t)r.heads * r.vdim, &off);
  place(&out->rg, t + "g", (int64_t)r.heads * r.vdim, &off);
  place(&out->ra1, t + "a1", 0, &off);  // its rows are the tensor's own
  out->rec_a2 = t + "a2";
  out->rec_a2_bias = t + "a2.b";
  out->rec_o = t + "o";
  out->rec_norm = t + "norm";
  return HB_OK;
}

static int read_parallel(const Json* m, const std::string& t, MixerSpec* out) {
  const Json *left = m->get("left"), *right = m->get("right");
  if (!left || !right) return fail(HB_ERR_INVALID_ARG, "%s: a parallel mixer needs left and right", t.c_str());
  AttentionSpec& a = out->attn;
  out->has_attn = true;
  a.heads = (int)int_of(left, "heads");
  a.kv_heads = (int)int_of(left, "kv_heads");
  a.dim = (int)int_of(left, "dim");
  a.vdim = (int)int_of(left, "vdim");
  a.scale = (float)left->number_or("scale", 0);
  if (a.heads < 1 || a.kv_heads < 1 || a.heads % a.kv_heads || a.dim < 1 || a.vdim < 1 || !left->get("scale"))
    return fail(HB_ERR_INVALID_ARG, "%s: bad attention sizes", t.c_str());
  int rc = read_window(left->get("mask"), &a);
  if (rc) return rc;
  RecurrenceSpec& r = out->rec;
  out->has_rec = true;
  r.heads = (int)int_of(right, "heads");
  r.dim = (int)int_of(right, "dim");
  r.vdim = (int)int_of(right, "vdim");
  r.silu_qkv = true;
  if (r.heads < 1 || r.dim < 1 || r.vdim < 1) return fail(HB_ERR_INVALID_ARG, "%s: bad recurrence sizes", t.c_str());
  const Json* decay = right->get("decay");
  if (decay && decay->kind == Json::Num) r.decay.assign((size_t)r.heads, decay->num);
  else if (decay && decay->kind == Json::Arr)
    for (const Json& d : decay->arr) r.decay.push_back(d.num);
  if ((int)r.decay.size() != r.heads)
    return fail(HB_ERR_INVALID_ARG, "%s: %zu decays for %d heads", t.c_str(), r.decay.size(), r.heads);
  for (double d : r.decay)
    if (!(d >= 0.0 && d <= 1.0)) return fail(HB_ERR_INVALID_ARG, "%s: decay %g outside [0, 1]", t.c_str(), d);
  int64_t off = 0;
  const std::string l = t + "left.", rt = t + "right.";
  place(&out->aq, l + "q", (int64_t)a.heads * a.dim, &off);
  place(&out->ak, l + "k", (int64_t)a.kv_heads * a.dim, &off);
  place(&out->av, l + "v", (int64_t)a.kv_heads * a.vdim, &off);
  place(&out->rq, rt + "q", (int64_t)r.heads * r.dim, &off);
  place(&out->rk, rt + "k", (int64_t)r.heads * r.dim, &off);
  place(&out->rv, rt + "v", (int64_t)r.heads * r.vdim, &off);
  place(&out->rg, rt + "g", (int64_t)r.heads * r.vdim, &off);
  out->attn_o = l + "o";
  out->attn_out_norm = l + "out";
  out->rec_o = rt + "o";
  out->rec_norm = rt + "norm";
  out->rec_out_norm = rt + "out";
  return HB_OK;
}

int read_latarax(const Json& config, LayeredSpec* out) {
  out->design = "Latarax";
  out->norm_offset = 1.f;
  out->width = int_of(&config, "width");
  out->vocab = int_of(&config, "vocab");
  out->max_positions = int_of(&config, "max_positions");
  out->streams = config.get("streams") ? (int)int_of(&config, "streams") : 1;
  const bool mixed = config.get("streams") != nullptr;
  const Json* norm = config.get("norm");
  if (!norm || !norm->get("eps")) return fail(HB_ERR_INVALID_ARG, "config.json: norm.eps is missing");
  out->eps = (float)norm->number_or("eps", 0);
  out->embed = "embed";
  out->pos = "pos";
  out->final_norm = "final.norm";
  out->head = "head";
  const Json* layers = config.get("layers");
  if (!layers || layers->kind != Json::Arr || out->width < 1 || out->vocab < 1 || out->max_positions < 1)
    return fail(HB_ERR_INVALID_ARG, "config.json: layers, width, vocab and max_positions are needed");
  for (size_t i = 0; i < layers->arr.size(); ++i) {
    const Json& j = layers->arr[i];
    LayerSpec l;
    l.prefix = "l" + std::to_string(i) + ".";
    const Json* m = j.get("mixer");
    const std::string type = j.string_or("type", "");
    if (!m) return fail(HB_ERR_INVALID_ARG, "config.json: layer %zu has no mixer", i);
    int rc;
    if (type == "gla") rc = read_gla(m, l.prefix + "mix.", &l.mixer);
    else if (type == "parallel") rc = read_parallel(m, l.prefix + "mix.", &l.mixer);
    else return fail(HB_ERR_INVALID_ARG, "config.json: layer %zu has the unknown type '%s'", i, type.c_str());
    if (rc) return rc;
    l.norm1 = l.prefix + "norm1";
    const Json* mlp = j.get("mlp");
    if (mlp && mlp->kind == Json::Obj) {
      const std::string kind = mlp->string_or("kind", "dense");
      l.ffn.ff = int_of(mlp, "ff");
      if (kind != "dense" || l.ffn.ff < 1) return fail(HB_ERR_INVALID_ARG, "config.json: layer %zu has a bad feed-forward", i);
      l.norm2 = l.prefix + "norm2";
      l.ffn.gate = l.prefix + "mlp.gate";
      l.ffn.up = l.prefix + "mlp.up";
      l.ffn.down = l.prefix + "mlp.down";
    }
    if (mixed) {
      l.hc1_in = l.prefix + "hc1.in";
      l.hc1_out = l.prefix + "hc1.out";
      l.hc1_mix = l.prefix + "hc1.mix";
      if (l.ffn.ff) {
        l.hc2_in = l.prefix + "hc2.in";
        l.hc2_out = l.prefix + "hc2.out";
        l.hc2_mix = l.prefix + "hc2.mix";
      }
    }
    out->layers.push_back(std::move(l));
  }
  if (out->layers.empty()) return fail(HB_ERR_INVALID_ARG, "config.json: no layers");
  return HB_OK;
}

}  // namespace hb
