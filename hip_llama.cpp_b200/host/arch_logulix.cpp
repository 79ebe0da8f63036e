// Logulix: config.json -> layer program.
// A decoder of sequential pre-norm blocks with plain rms norms (the weight is stored as it is used),
//     x <- x + mixer(norm1 x),   x <- x + ff(norm2 x),
// whose embedding rows and logits are multiplied by constants.
// Layer types:
//   "attention"  sliding-window softmax attention without a value projection: q and k carry biases and a short convolution, the values
//                are the convolved keys, not normed or rotated; rms norms over the whole q and k rows, rotary pairs (2i, 2i + 1) with linearly
//                stretched frequencies, capped scores, an output bias;
//   "wkv"        a token-shifted key-value memory: decay per key channel, a bonus for the current token, head norm, silu gate;
//   "retention"  a linear-attention memory whose only decay is a constant per head, rotary pairs (i, i + dims / 2), head norm without a weight, silu gate.
// Feed-forward: none, or dense without a gate and with squared relu.
// "loop" runs a segment of the layer list several times with the same weights, every pass with a cache and state of its own; every
// pass starts by joining x and the embedding output through one map.  Every size and constant comes from the config; constants the
// design fixes live with the mechanisms.
#include "layer_model.hpp"

static void logulix_rotary(const JsonValue& m, bool halves, RotarySpec* rot, bool* on) {
  if (!m.has("rot")) return;
  const JsonValue& r = m.at("rot");
  *on = true;
  rot->dims = r.at("dims").integer();
  rot->base = r.at("base").number();
  rot->halves = halves;
  if (r.has("scaling")) {
    rot->linear = true;
    rot->factor = r.at("scaling").at("factor").number();
  }
}

static void logulix_mixer(const JsonValue& L, const std::string& pre, LayerSpec* out) {
  LayerSpec& ls = *out;
  const std::string type = L.at("type").string();
  const JsonValue& m = L.at("mixer");
  const std::string p = pre + "mix.";
  if (type == "attention") {
    ls.mixer = THA_MIX_ATTN;
    AttnSpec& a = ls.attn;
    a.heads = m.at("heads").integer();
    a.kv_heads = m.at("kv_heads").integer();
    a.dim = m.at("dim").integer();
    a.vdim = m.has("vdim") ? m.at("vdim").integer() : a.dim;
    a.scale = (float)m.at("scale").number();
    a.softcap = m.has("softcap") ? (float)m.at("softcap").number() : 0.f;
    if (m.has("softcap") && !(a.softcap > 0.f)) throw std::runtime_error("config: 'softcap' must be positive");
    logulix_rotary(m, false, &a.rot, &a.rotary);
    if (m.has("mask")) {   // absent: every earlier position is seen
      a.window = m.at("mask").at("size").integer();
      if (a.window < 1) throw std::runtime_error("config: a window must hold at least the token itself");
    }
    if (m.has("conv")) {   // absent: the projections are used as they are
      a.conv_taps = m.at("conv").integer();
      if (a.conv_taps < 1) throw std::runtime_error("config: 'conv' must be at least one tap");
    }
    a.q = p + "q"; a.k = p + "k"; a.o = p + "o";
    a.q_b = p + "q.b"; a.k_b = p + "k.b"; a.o_b = p + "o.b";
    a.q_norm = p + "q.norm"; a.k_norm = p + "k.norm";
    a.v_is_k = true;
    a.fp32_scores = true;
  } else if (type == "wkv") {
    ls.mixer = THA_MIX_WKV;
    WkvSpec& g = ls.wkv;
    g.heads = m.at("heads").integer();
    g.dim = m.at("dim").integer();
    g.mu_r = p + "mu.r"; g.mu_k = p + "mu.k"; g.mu_v = p + "mu.v"; g.mu_g = p + "mu.g"; g.mu_w = p + "mu.w";
    g.r = p + "r"; g.k = p + "k"; g.v = p + "v"; g.g = p + "g";
    g.w1 = p + "w1"; g.w2 = p + "w2"; g.w0 = p + "w0"; g.u = p + "u"; g.norm = p + "norm"; g.o = p + "o";
  } else if (type == "retention") {
    ls.mixer = THA_MIX_RETENTION;
    RetentionSpec& g = ls.retention;
    g.heads = m.at("heads").integer();
    g.dim = m.at("dim").integer();
    g.vdim = m.at("vdim").integer();
    logulix_rotary(m, true, &g.rot, &g.rotary);
    const JsonValue& d = m.at("decay");
    if (d.kind != JsonValue::Array) throw std::runtime_error("config: 'decay' must be a list");
    for (const JsonValue& v : d.arr) g.decay.push_back(v.number());
    g.q = p + "q"; g.k = p + "k"; g.v = p + "v"; g.g = p + "g"; g.o = p + "o";
  } else {
    throw std::runtime_error("config: unknown layer type '" + type + "'");
  }
}

static void logulix_translate(const JsonValue& c, LayerProgramSpec* out) {
  LayerProgramSpec& s = *out;
  s.width = c.at("width").integer();
  s.vocab = c.at("vocab").integer();
  s.eps = (float)c.at("norm").at("eps").number();
  s.norm_kind = THA_NORM_RMS;
  s.norm_w_offset = 0.0f;
  s.embed = "embed";
  s.embed_scale = (float)c.at("embedding").at("scale").number();
  s.final_norm = "final.norm";
  s.head = "head";
  s.logit_scale = (float)c.at("logit_scale").number();
  const JsonValue& layers = c.at("layers");
  if (layers.kind != JsonValue::Array) throw std::runtime_error("config: 'layers' must be a list");
  const int n = (int)layers.arr.size();
  // the order of execution: the looped segment repeated in place
  int start = 0, stop = 0, times = 1;
  if (c.has("loop")) {
    const JsonValue& lp = c.at("loop");
    start = lp.at("start").integer();
    stop = lp.at("stop").integer();
    times = lp.at("times").integer();
    if (start < 0 || stop < start || stop > n || times < 0) throw std::runtime_error("config: 'loop' does not fit the layer list");
  }
  std::vector<int> first_run(n, -1);
  auto run = [&](int i, bool opens_pass) {
    LayerSpec ls;
    const JsonValue& L = layers.arr[i];
    const std::string pre = "l" + std::to_string(i) + ".";
    ls.block = THA_BLOCK_SEQUENTIAL;
    ls.norm1 = pre + "norm1";
    logulix_mixer(L, pre, &ls);
    if (L.has("mlp")) {   // absent or null: the layer has no feed-forward
      const JsonValue& f = L.at("mlp");
      const std::string kind = f.at("kind").string();
      if (kind != "dense") throw std::runtime_error("config: unknown feed-forward kind '" + kind + "'");
      ls.has_ff = true;
      ls.ff_kind = THA_FF_DENSE;
      ls.norm2 = pre + "norm2";
      ls.dense.ff = f.at("ff").integer();
      ls.dense.act = THA_ACT_RELU2;
      ls.dense.up = pre + "mlp.up"; ls.dense.down = pre + "mlp.down";
    }
    if (opens_pass) ls.pre_join = "loop.in";
    if (first_run[i] >= 0) ls.same_weights_as = first_run[i];
    else first_run[i] = (int)s.layers.size();
    s.layers.push_back(ls);
  };
  for (int i = 0; i < start; i++) run(i, false);
  for (int t = 0; t < times; t++)
    for (int i = start; i < stop; i++) run(i, i == start);
  for (int i = stop; i < n; i++) run(i, false);
}

void register_logulix() { register_architecture({"Logulix", ModelFamily::LayerProgram, logulix_translate}); }
