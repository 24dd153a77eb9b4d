// Muzopel: the reader of its config.json and tensor names.
//
// A decoder whose sublayers read the residual itself, with a causal convolution of its channels added,
// and whose outputs are normed in equal parts before they are added; after every layer the residual
// becomes a weighted sum over the embedding and the results of all layers so far.  Mixers: latent attention
// whose queries come from a latent of their own and whose heads are gated ("latent_attention"), or from the
// input ("latent_attention_2").  The feed-forward is a mixture of experts without gates, some of whose
// router outputs hand the input on, or none.  Logits are capped by a hyperbolic tangent.
#include "design_reader.h"

namespace hb {

bool is_muzopel(const Json& config) { return config.string_or("architecture", "") == "Muzopel"; }

static int read_latent(const Json* m, const std::string& t, bool own_latent, MixerSpec* out) {
  AttentionSpec& a = out->attn;
  out->has_attn = true;
  a.heads = a.kv_heads = (int)int_of(m, "heads");
  a.dim = (int)int_of(m, "dim");
  a.rot_dim = (int)int_of(m, "rot_dim");
  a.vdim = (int)int_of(m, "vdim");
  a.rank = (int)int_of(m, "kv_rank");
  a.q_rank = own_latent ? (int)int_of(m, "q_rank") : 0;
  a.scale = (float)m->number_or("scale", 0);
  if (a.heads < 1 || a.dim < 1 || a.rot_dim < 0 || a.vdim < 1 || a.rank < 1 || !m->get("scale") || (own_latent && a.q_rank < 1))
    return fail(HB_ERR_INVALID_ARG, "%s: bad attention sizes", t.c_str());
  int64_t off = 0;
  if (own_latent) {
    place(&out->aq, t + "dq", a.q_rank, &off);
    out->attn_q_latent_norm = t + "dq.norm";
    out->attn_uq = t + "uq";
  } else {
    place(&out->aq, t + "q", (int64_t)a.heads * (a.dim + a.rot_dim), &off);
  }
  place(&out->ak, t + "dkv", (int64_t)a.rank + a.rot_dim, &off);
  if (own_latent) {
    place(&out->ag, t + "g", a.heads, &off);
    a.gate_per_head = true;
  }
  out->attn_latent_norm = t + "dkv.norm";
  out->attn_uk = t + "uk";
  out->attn_uv = t + "uv";
  out->attn_o = t + "o";
  const Json* rot = object_of(*m, "rot");
  return rot ? read_rotation(rot, t, a.rot_dim, true, false, &a) : HB_OK;
}

static int read_experts(const Json& mlp, const std::string& t, ExpertsSpec* x) {
  const std::string kind = mlp.string_or("kind", "moe");
  if (kind != "moe") return fail(HB_ERR_INVALID_ARG, "%s: unknown kind '%s'", t.c_str(), kind.c_str());
  const Json *router = object_of(mlp, "router"), *expert = object_of(mlp, "expert");
  if (!router || !expert) return fail(HB_ERR_INVALID_ARG, "%s: a mixture needs router and expert", t.c_str());
  x->experts = (int)int_of(router, "experts");
  x->identity = (int)int_of(router, "identity");
  x->top = (int)int_of(router, "top");
  x->ff = int_of(expert, "ff");
  if (x->experts < 1 || x->identity < 0 || x->top < 1 || x->top > x->outputs() || x->ff < 1)
    return fail(HB_ERR_INVALID_ARG, "%s: %d of %d experts (%d of them identities)", t.c_str(), x->top, x->outputs(), x->identity);
  x->softmax_all = true;
  x->act.form = GatedAct::kErf;
  x->act.single = 1;
  x->router = t + "router";
  x->correction = t + "correction";
  x->prefix = t + "e";
  return HB_OK;
}

int read_muzopel(const Json& config, LayeredSpec* out) {
  out->design = "Muzopel";
  out->width = int_of(&config, "width");
  out->vocab = int_of(&config, "vocab");
  const Json *norm = object_of(config, "norm"), *canon = object_of(config, "canon");
  if (!norm || !norm->get("eps")) return fail(HB_ERR_INVALID_ARG, "config.json: norm.eps is missing");
  out->eps = (float)norm->number_or("eps", 0);
  out->post_norm = true;
  out->norm_groups = (int)norm->number_or("groups", 1);
  out->input_taps = (int)int_of(canon, "taps");
  out->logit_cap = (float)config.number_or("logit_softcap", 0);
  const Json* layers = config.get("layers");
  if (!layers || layers->kind != Json::Arr || out->width < 1 || out->vocab < 1)
    return fail(HB_ERR_INVALID_ARG, "config.json: layers, width and vocab are needed");
  if (out->norm_groups < 1 || out->width % out->norm_groups || out->input_taps < 1 || out->logit_cap < 0)
    return fail(HB_ERR_INVALID_ARG, "config.json: a width of %lld in %d parts, %d taps", (long long)out->width, out->norm_groups, out->input_taps);
  out->embed = "embed";
  out->embed_norm = "embed.norm";
  out->final_norm = "final.norm";
  out->head = "head";
  for (size_t i = 0; i < layers->arr.size(); ++i) {
    const Json& j = layers->arr[i];
    LayerSpec l;
    l.prefix = "l" + std::to_string(i) + ".";
    const Json* m = object_of(j, "mixer");
    const std::string type = j.string_or("type", "");
    if (!m) return fail(HB_ERR_INVALID_ARG, "config.json: layer %zu has no mixer", i);
    if (type != "latent_attention" && type != "latent_attention_2")
      return fail(HB_ERR_INVALID_ARG, "config.json: layer %zu has the unknown type '%s'", i, type.c_str());
    int rc;
    if ((rc = read_latent(m, l.prefix + "mix.", type == "latent_attention", &l.mixer))) return rc;
    l.norm1 = l.prefix + "norm1";
    l.conv1 = l.prefix + "canon1";
    l.depth = l.prefix + "dwa";
    if (const Json* mlp = object_of(j, "mlp")) {
      if ((rc = read_experts(*mlp, l.prefix + "mlp.", &l.moe))) return rc;
      l.norm2 = l.prefix + "norm2";
      l.conv2 = l.prefix + "canon2";
    }
    out->layers.push_back(std::move(l));
  }
  if (out->layers.empty()) return fail(HB_ERR_INVALID_ARG, "config.json: no layers");
  return HB_OK;
}

}  // namespace hb
