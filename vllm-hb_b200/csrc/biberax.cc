// Biberax: the reader of its config.json and tensor names.
//
// A pre-norm decoder whose layers have one of two attention mixers: "attention" (interleaved
// rotation with stretched long wavelengths, chunks of positions, one added to the softmax
// denominator) or "attention_2" (values are the projected keys, norms over whole projections, a
// learned bias by distance, a learned sink), both with a gate on the heads' outputs; and a dense
// feed-forward, or a mixture of experts with a shared one, or none.
#include <climits>
#include <cmath>

#include "design_reader.h"

namespace hb {

bool is_biberax(const Json& config) { return config.string_or("architecture", "") == "Biberax"; }

// Frequencies base^(-2i / dims); with `scaling` those of wavelengths above original / low are
// divided by factor, those below original / high kept, and the ones between blended linearly in
// original / wavelength.
static int read_rotation(const Json* rot, const std::string& t, AttentionSpec* a) {
  const double pi = 3.14159265358979323846;
  const double base = rot->number_or("base", 0);
  const int64_t dims = int_of(rot, "dims");
  if (base <= 0 || dims % 2 || dims > a->dim) return fail(HB_ERR_INVALID_ARG, "%s: bad rotation", t.c_str());
  const Json* s = object_of(*rot, "scaling");
  const double factor = s ? s->number_or("factor", 0) : 1, low = s ? s->number_or("low", 0) : 1;
  const double high = s ? s->number_or("high", 0) : 1, original = s ? s->number_or("original", 0) : 1;
  if (factor <= 0 || low <= 0 || high < low || original <= 0)
    return fail(HB_ERR_INVALID_ARG, "%s: bad rotation scaling", t.c_str());
  for (int64_t i = 0; i < dims / 2; ++i) {
    double f = std::pow(base, -2.0 * (double)i / (double)dims);
    if (s) {
      const double wave = 2.0 * pi / f;
      if (wave > original / low) {
        f /= factor;
      } else if (wave >= original / high && high > low) {
        const double keep = (original / wave - low) / (high - low);
        f = (1.0 - keep) * f / factor + keep * f;
      }
    }
    a->rotation.push_back(f);
  }
  return HB_OK;
}

static int read_mixer(const Json* m, const std::string& type, const std::string& t, MixerSpec* out) {
  AttentionSpec& a = out->attn;
  out->has_attn = true;
  a.heads = (int)int_of(m, "heads");
  a.kv_heads = (int)int_of(m, "kv_heads");
  a.dim = (int)int_of(m, "dim");
  a.vdim = (int)int_of(m, "vdim");
  a.scale = (float)m->number_or("scale", 0);
  a.values_are_keys = type == "attention_2";
  if (a.values_are_keys && !m->get("vdim")) a.vdim = a.dim;
  if (a.heads < 1 || a.kv_heads < 1 || a.heads % a.kv_heads || a.dim < 1 || a.vdim < 1 || !m->get("scale"))
    return fail(HB_ERR_INVALID_ARG, "%s: bad attention sizes", t.c_str());
  if (a.values_are_keys && a.vdim != a.dim)
    return fail(HB_ERR_INVALID_ARG, "%s: values that are the keys have their width (%d, not %d)", t.c_str(), a.dim, a.vdim);
  int64_t off = 0;
  place(&out->aq, t + "q", (int64_t)a.heads * a.dim, &off);
  place(&out->ak, t + "k", (int64_t)a.kv_heads * a.dim, &off);
  if (!a.values_are_keys) place(&out->av, t + "v", (int64_t)a.kv_heads * a.vdim, &off);
  place(&out->ag, t + "g", (int64_t)a.heads * a.vdim, &off);
  out->attn_o = t + "o";
  if (!a.values_are_keys) {
    a.unit_sink = true;
    if (const Json* mask = object_of(*m, "mask")) {
      const double size = mask->number_or("size", 0);
      if (!(size >= 1)) return fail(HB_ERR_INVALID_ARG, "%s: chunks of %g positions", t.c_str(), size);
      a.chunk = (int)(size > INT_MAX / 2 ? 0 : size);
    }
    if (const Json* rot = object_of(*m, "rot")) return read_rotation(rot, t, &a);
    return HB_OK;
  }
  a.bias_far = m->number_or("bias_max", 0);
  if (!(a.bias_far > 0)) return fail(HB_ERR_INVALID_ARG, "%s: bias_max must be positive", t.c_str());
  out->attn_q_bias = t + "q.b";
  out->attn_k_bias = t + "k.b";
  out->attn_o_bias = t + "o.b";
  out->attn_q_norm = t + "q.norm";
  out->attn_k_norm = t + "k.norm";
  out->attn_rel = t + "rel";
  out->attn_sink = t + "sink";
  return HB_OK;
}

static int read_clamp(const Json* j, const std::string& t, int64_t* ff, GatedAct* act) {
  *ff = int_of(j, "ff");
  if (*ff < 1 || !j->get("limit")) return fail(HB_ERR_INVALID_ARG, "%s: an expert needs ff and limit", t.c_str());
  act->slope = 1.702f;
  act->shift = 1.f;
  act->limit = (float)j->number_or("limit", 0);
  return HB_OK;
}

static void name_ffn(FeedForwardSpec* f, const std::string& t) {
  f->gate = t + "gate";
  f->up = t + "up";
  f->down = t + "down";
}

static int read_mlp(const Json& mlp, const std::string& t, LayerSpec* l) {
  const std::string kind = mlp.string_or("kind", "dense");
  if (kind == "dense") {
    l->ffn.ff = int_of(&mlp, "ff");
    if (l->ffn.ff < 1) return fail(HB_ERR_INVALID_ARG, "%s: ff must be positive", t.c_str());
    l->ffn.act.slope = (float)(2.0 * std::sqrt(2.0 / 3.14159265358979323846));
    l->ffn.act.cubic = 0.044715f;
    name_ffn(&l->ffn, t);
    return HB_OK;
  }
  if (kind != "moe") return fail(HB_ERR_INVALID_ARG, "%s: unknown kind '%s'", t.c_str(), kind.c_str());
  const Json *router = object_of(mlp, "router"), *expert = object_of(mlp, "expert"), *shared = object_of(mlp, "shared");
  if (!router || !expert) return fail(HB_ERR_INVALID_ARG, "%s: a mixture needs router and expert", t.c_str());
  ExpertsSpec& x = l->moe;
  x.experts = (int)int_of(router, "experts");
  x.top = (int)int_of(router, "top");
  if (x.experts < 1 || x.top < 1 || x.top > x.experts)
    return fail(HB_ERR_INVALID_ARG, "%s: %d of %d experts", t.c_str(), x.top, x.experts);
  int rc = read_clamp(expert, t, &x.ff, &x.act);
  if (rc) return rc;
  x.router = t + "router";
  x.router_bias = t + "router.b";
  x.prefix = t + "e";
  if (shared) {
    if ((rc = read_clamp(shared, t + "shared", &l->ffn.ff, &l->ffn.act))) return rc;
    name_ffn(&l->ffn, t + "shared.");
  }
  return HB_OK;
}

int read_biberax(const Json& config, LayeredSpec* out) {
  out->design = "Biberax";
  out->width = int_of(&config, "width");
  out->vocab = int_of(&config, "vocab");
  const Json* norm = object_of(config, "norm");
  if (!norm || !norm->get("eps")) return fail(HB_ERR_INVALID_ARG, "config.json: norm.eps is missing");
  out->eps = (float)norm->number_or("eps", 0);
  out->embed = "embed";
  out->final_norm = "final.norm";
  out->head = "head";
  const Json* layers = config.get("layers");
  if (!layers || layers->kind != Json::Arr || out->width < 1 || out->vocab < 1)
    return fail(HB_ERR_INVALID_ARG, "config.json: layers, width and vocab are needed");
  for (size_t i = 0; i < layers->arr.size(); ++i) {
    const Json& j = layers->arr[i];
    LayerSpec l;
    l.prefix = "l" + std::to_string(i) + ".";
    const Json* m = object_of(j, "mixer");
    const std::string type = j.string_or("type", "");
    if (!m) return fail(HB_ERR_INVALID_ARG, "config.json: layer %zu has no mixer", i);
    if (type != "attention" && type != "attention_2")
      return fail(HB_ERR_INVALID_ARG, "config.json: layer %zu has the unknown type '%s'", i, type.c_str());
    int rc = read_mixer(m, type, l.prefix + "mix.", &l.mixer);
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
