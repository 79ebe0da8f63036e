// Gavodra: config.json -> layer program.
// A decoder whose norms sit on what the sublayers return,
//     x <- x + m norm1(mixer(x)),   x <- x + m norm2(ff(x)),
// with plain rms norms (the weight is stored as it is used), scaled embedding rows that serve (unscaled) as the output matrix, and capped logits.
// Layer type "attention": causal softmax attention without rotation; rms norms per q and k head, a learned bias per head by distance bucket,
// one sigmoid gate per head; in layers that mix values, each value row is blended with the first such layer's row of the same token.
// Feed-forward: none, dense with the clamped gate, or a mixture of such experts behind a sigmoid router (choice by corrected scores, weights
// the plain scores times a constant) plus a shared expert scaled by a per-token sigmoid.
// Every size and constant comes from the config; constants the design fixes live with the mechanisms.
#include "layer_model.hpp"

static void gavodra_mixer(const JsonValue& L, const std::string& pre, int first_mixing, LayerSpec* out) {
  const std::string type = L.at("type").string();
  if (type != "attention") throw std::runtime_error("config: unknown layer type '" + type + "'");
  const JsonValue& m = L.at("mixer");
  const std::string p = pre + "mix.";
  out->mixer = THA_MIX_ATTN;
  AttnSpec& a = out->attn;
  a.heads = m.at("heads").integer();
  a.kv_heads = m.at("kv_heads").integer();
  a.dim = m.at("dim").integer();
  a.vdim = m.at("vdim").integer();
  a.scale = (float)m.at("scale").number();
  a.rel = p + "rel";
  a.rel_far = m.at("bias_max").number();
  a.head_norm = true;
  a.q_norm = p + "q.norm"; a.k_norm = p + "k.norm";
  a.q = p + "q"; a.k = p + "k"; a.v = p + "v"; a.g = p + "g"; a.o = p + "o";
  a.fp32_scores = true;
  if (first_mixing >= 0) { a.v_mix_from = first_mixing; a.v_mix = p + "vmix"; }
}

static void gavodra_ff(const JsonValue& L, const std::string& pre, LayerSpec* out) {
  LayerSpec& ls = *out;
  if (!L.has("mlp")) return;   // absent or null: the layer has no feed-forward
  const JsonValue& f = L.at("mlp");
  const std::string kind = f.at("kind").string();
  const std::string p = pre + "mlp.";
  ls.has_ff = true;
  ls.norm2 = pre + "norm2";
  if (kind == "dense") {
    ls.ff_kind = THA_FF_DENSE;
    ls.dense.ff = f.at("ff").integer();
    ls.dense.act = THA_ACT_GLU_CLAMPED;
    ls.dense.limit = (float)f.at("limit").number();
    ls.dense.gate = p + "gate"; ls.dense.up = p + "up"; ls.dense.down = p + "down";
  } else if (kind == "moe") {
    ls.ff_kind = THA_FF_MOE;
    MoeSpec& e = ls.moe;
    const JsonValue& r = f.at("router");
    e.experts = r.at("experts").integer();
    e.top = r.at("top").integer();
    e.weight_scale = (float)r.at("scale").number();
    e.ff = f.at("expert").at("ff").integer();
    e.limit = (float)f.at("expert").at("limit").number();
    e.act = THA_ACT_GLU_CLAMPED;
    e.route = THA_ROUTE_SIGMOID_GROUPS;
    e.router = p + "router";
    e.correction = p + "correction";
    e.prefix = p;
    if (f.has("shared")) {
      e.shared_ff = f.at("shared").at("ff").integer();
      e.shared_limit = (float)f.at("shared").at("limit").number();
      e.s_gate = p + "shared.gate"; e.s_up = p + "shared.up"; e.s_down = p + "shared.down"; e.s_scale = p + "shared.sg";
    }
  } else {
    throw std::runtime_error("config: unknown feed-forward kind '" + kind + "'");
  }
}

static void gavodra_translate(const JsonValue& c, LayerProgramSpec* out) {
  LayerProgramSpec& s = *out;
  s.width = c.at("width").integer();
  s.vocab = c.at("vocab").integer();
  s.eps = (float)c.at("norm").at("eps").number();
  s.norm_kind = THA_NORM_RMS;
  s.norm_w_offset = 0.0f;
  s.embed = "embed";
  s.embed_scale = (float)c.at("embedding").at("scale").number();
  s.final_norm = "final.norm";
  s.head = s.embed;
  s.logit_scale = (float)c.at("logit_scale").number();
  s.logit_softcap = (float)c.at("logit_softcap").number();
  if (!(s.logit_softcap > 0.f)) throw std::runtime_error("config: 'logit_softcap' must be positive");
  const float res_mult = (float)c.at("residual_mult").number();
  const JsonValue& layers = c.at("layers");
  if (layers.kind != JsonValue::Array) throw std::runtime_error("config: 'layers' must be a list");
  int first_mixing = -1;   // the first layer that says v_mix keeps its values as they are; the later ones blend with them
  for (size_t i = 0; i < layers.arr.size(); i++) {
    const JsonValue& L = layers.arr[i];
    const std::string pre = "l" + std::to_string(i) + ".";
    LayerSpec ls;
    ls.block = THA_BLOCK_POST;
    ls.res_mult = res_mult;
    ls.norm1 = pre + "norm1";
    const JsonValue& m = L.at("mixer");
    const bool mixes = m.has("v_mix") && m.at("v_mix").boolean();
    gavodra_mixer(L, pre, mixes ? first_mixing : -1, &ls);
    if (mixes && first_mixing < 0) first_mixing = (int)i;
    gavodra_ff(L, pre, &ls);
    s.layers.push_back(ls);
  }
}

void register_gavodra() { register_architecture({"Gavodra", ModelFamily::LayerProgram, gavodra_translate}); }
