"""Plain float64 statement of the Gavodra design (numpy; one function per mechanism; shares no code with the product).

A model is (cfg, W): cfg the parsed config.json, W a dict name -> float64 array.  The mixer takes the rows of ONE sequence's next
portion and the store that the layer carries for the sequence (its key and value rows), so `Stepper.feed` serves whole prompts,
portions and single tokens alike.

A layer norms what a sublayer returns, not what it reads:  x <- x + m N1(mixer(x)),  x <- x + m N2(ff(x)).
"""
import functools
import math
from fractions import Fraction

import numpy as np


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def rms_unit(x, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


# ---- the distance bias ----------------------------------------------------------------------------------------------------
@functools.lru_cache(maxsize=None)
def bucket(n, rows, far):
    """Which of `rows` table rows the distance n >= 0 reads: its own below rows / 2, then logarithmically wider ones that end at `far`.
    Whole-number comparison: step k of the upper half starts where (n / half)^steps >= (far / half)^k."""
    half = rows // 2
    if n < half:
        return n
    steps, far = rows - half, Fraction(far)
    k = 0
    while k + 1 < steps and n ** steps * half ** (k + 1) >= far ** (k + 1) * half ** steps:
        k += 1
    return half + k


def bias_matrix(table, far, q_pos, n_keys):
    """[heads, queries, keys]; keys after the query get row 0's value (they are masked anyway)"""
    rows = table.shape[0]
    of = np.array([bucket(n, rows, far) for n in range(int(max(q_pos)) + 1)])
    dist = np.maximum(np.asarray(q_pos)[:, None] - np.arange(n_keys)[None, :], 0)
    return table[of[dist]].transpose(2, 0, 1)


# ---- attention ------------------------------------------------------------------------------------------------------------
def mix_values(v, lam, v_first):
    return (1.0 - lam) * v + lam * v_first


def attention_mixer(h, m, W, p, eps, store, pos0, first_values):
    """first_values: the values of the first value-mixing layer for the same tokens (None: this layer mixes nothing in).
    Returns (output, this layer's cached values of the portion)."""
    T = h.shape[0]
    H, G, D, E = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms_unit((h @ W[p + "q"].T).reshape(T, H, D), eps) * W[p + "q.norm"]
    k = rms_unit((h @ W[p + "k"].T).reshape(T, G, D), eps) * W[p + "k.norm"]
    v = h @ W[p + "v"].T
    if first_values is not None:
        v = mix_values(v, float(W[p + "vmix"]), first_values)
    store.setdefault("k", []).extend(k)
    store.setdefault("v", []).extend(v.reshape(T, G, E))
    K, V = np.array(store["k"]), np.array(store["v"])
    pos = pos0 + np.arange(T)
    bias = bias_matrix(W[p + "rel"], m["bias_max"], pos, K.shape[0])
    seen = np.arange(K.shape[0])[None, :] <= pos[:, None]
    out = np.zeros((T, H, E))
    for hh in range(H):
        g = hh // (H // G)
        s = q[:, hh] @ K[:, g].T * m["scale"] + bias[hh]
        s = np.where(seen, s, -np.inf)
        e = np.exp(s - s.max(axis=1, keepdims=True))
        out[:, hh] = (e / e.sum(axis=1, keepdims=True)) @ V[:, g]
    out = out * sigmoid(h @ W[p + "g"].T)[:, :, None]
    return out.reshape(T, H * E) @ W[p + "o"].T, v


# ---- feed-forward ---------------------------------------------------------------------------------------------------------
def clamped_glu(h, W, p, limit):
    g = np.minimum(h @ W[p + "gate"].T, limit)
    u = np.clip(h @ W[p + "up"].T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ W[p + "down"].T


def route(z, correction, top, scale):
    """One row's router logits -> (chosen experts, their weights): chosen by sigmoid + correction, weighted by the sigmoid alone"""
    s = sigmoid(z)
    chosen = np.argsort(-(s + correction), kind="stable")[:top]
    return chosen, s[chosen] * scale


def mixture_ff(h, f, W, p):
    r = f["router"]
    z = h @ W[p + "router"].T
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        for e, w in zip(*route(z[t], W[p + "correction"], r["top"], r["scale"])):
            out[t] += w * clamped_glu(h[t:t + 1], W, p + "e%d." % e, f["expert"]["limit"])[0]
    if f.get("shared"):
        out = out + sigmoid(h @ W[p + "shared.sg"].T) * clamped_glu(h, W, p + "shared.", f["shared"]["limit"])
    return out


# ---- one sequence ---------------------------------------------------------------------------------------------------------
class Stepper:
    """feed(tokens) runs the sequence's next portion and returns (logits [T, vocab], taps [layers, T, width])."""

    def __init__(self, cfg, W):
        self.cfg, self.W = cfg, W
        self.pos = 0
        self.stores = [dict() for _ in cfg["layers"]]

    def feed(self, tokens):
        cfg, W = self.cfg, self.W
        eps, mult = cfg["norm"]["eps"], cfg["residual_mult"]
        x = W["embed"][np.asarray(tokens)] * cfg["embedding"]["scale"]
        taps, first = [], None
        for i, (L, st) in enumerate(zip(cfg["layers"], self.stores)):
            pre, m = "l%d." % i, L["mixer"]
            mixes = bool(m.get("v_mix"))
            y, v = attention_mixer(x, m, W, pre + "mix.", eps, st, self.pos, first if mixes else None)
            if mixes and first is None:
                first = v
            x = x + mult * rms_unit(y, eps) * W[pre + "norm1"]
            f = L.get("mlp")
            if f:
                y = clamped_glu(x, W, pre + "mlp.", f["limit"]) if f["kind"] == "dense" else mixture_ff(x, f, W, pre + "mlp.")
                x = x + mult * rms_unit(y, eps) * W[pre + "norm2"]
            taps.append(x)
        self.pos += len(tokens)
        z = (rms_unit(x, eps) * W["final.norm"]) @ W["embed"].T * cfg["logit_scale"]
        return cfg["logit_softcap"] * np.tanh(z / cfg["logit_softcap"]), np.array(taps)


def forward(cfg, W, tokens):
    return Stepper(cfg, W).feed(tokens)


def forward_tokenwise(cfg, W, tokens):
    s = Stepper(cfg, W)
    outs = [s.feed([t]) for t in tokens]
    return np.concatenate([o[0] for o in outs]), np.concatenate([o[1] for o in outs], axis=1)


def bf16_round(a):
    """float64 -> the nearest bfloat16 (ties to even), as float64"""
    u = np.asarray(a, dtype=np.float32).view(np.uint32).astype(np.uint64)
    u = (u + 0x7FFF + ((u >> 16) & 1)) & 0xFFFF0000
    return u.astype(np.uint32).view(np.float32).astype(np.float64)


# ---- shapes and random weights of a configuration -------------------------------------------------------------------------
def tensor_shapes(cfg, rel_rows=12):
    """`rel_rows`: rows of the distance tables (a property of the tensors, not of the config)"""
    Wd = cfg["width"]
    out = {"embed": (cfg["vocab"], Wd), "final.norm": (Wd,)}

    def glu(p, ff):
        out.update({p + "gate": (ff, Wd), p + "up": (ff, Wd), p + "down": (Wd, ff)})

    for i, L in enumerate(cfg["layers"]):
        pre = "l%d." % i
        m, p = L["mixer"], pre + "mix."
        H, G, D, E = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        out.update({pre + "norm1": (Wd,), p + "q": (H * D, Wd), p + "k": (G * D, Wd), p + "v": (G * E, Wd), p + "q.norm": (D,), p + "k.norm": (D,),
                    p + "rel": (rel_rows, H), p + "g": (H, Wd), p + "o": (Wd, H * E)})
        if m.get("v_mix"):
            out[p + "vmix"] = ()
        f = L.get("mlp")
        if not f:
            continue
        out[pre + "norm2"] = (Wd,)
        p = pre + "mlp."
        if f["kind"] == "dense":
            glu(p, f["ff"])
            continue
        out.update({p + "router": (f["router"]["experts"], Wd), p + "correction": (f["router"]["experts"],)})
        for e in range(f["router"]["experts"]):
            glu(p + "e%d." % e, f["expert"]["ff"])
        if f.get("shared"):
            glu(p + "shared.", f["shared"]["ff"])
            out[p + "shared.sg"] = (1, Wd)
    return out


def random_weights(cfg, seed=0, rel_rows=12):
    """bfloat16-representable float64 values, scaled so that activations stay of order one through the layers"""
    rng = np.random.default_rng(seed)
    W = {}
    for name, shape in tensor_shapes(cfg, rel_rows).items():
        leaf = name.split(".")[-1]
        if "norm" in leaf:
            a = 1.0 + 0.2 * rng.standard_normal(shape)
        elif leaf == "vmix":
            a = rng.uniform(0.2, 0.8)
        elif leaf == "rel":
            a = 0.7 * rng.standard_normal(shape)
        elif leaf == "correction":
            a = 0.3 * rng.standard_normal(shape)
        elif leaf == "embed":
            a = rng.standard_normal(shape)
        else:
            a = rng.standard_normal(shape) / math.sqrt(shape[-1])
        W[name] = bf16_round(a)
    return W


def self_check():
    """The statement agrees with itself: a whole prompt, the same prompt token by token, and in uneven portions."""
    att = {"heads": 4, "kv_heads": 2, "dim": 6, "vdim": 5, "scale": 0.5, "bias_max": 11, "v_mix": True}
    moe = {"kind": "moe", "expert": {"ff": 7, "limit": 0.8}, "router": {"experts": 5, "top": 2, "scale": 1.5}, "shared": {"ff": 6, "limit": 0.6}}
    cfg = {"architecture": "Gavodra", "width": 20, "vocab": 30, "norm": {"eps": 1e-6}, "embedding": {"scale": 1.5}, "logit_scale": 0.7,
           "logit_softcap": 9.0, "residual_mult": 0.6,
           "layers": [{"type": "attention", "mixer": dict(att, v_mix=False), "mlp": {"kind": "dense", "ff": 18, "limit": 1.2}},
                      {"type": "attention", "mixer": att, "mlp": None},
                      {"type": "attention", "mixer": att, "mlp": moe},
                      {"type": "attention", "mixer": dict(att, heads=2), "mlp": moe}]}
    W = random_weights(cfg, 3, rel_rows=8)
    toks = list(np.random.default_rng(1).integers(0, 30, 19))
    a, ta = forward(cfg, W, toks)
    b, tb = forward_tokenwise(cfg, W, toks)
    assert ta.shape == (4, 19, 20)
    assert np.abs(a - b).max() < 1e-9 and np.abs(ta - tb).max() < 1e-9
    s, parts, at = Stepper(cfg, W), [], 0
    for n in (2, 7, 1, 9):
        parts.append(s.feed(toks[at:at + n])[0])
        at += n
    assert np.abs(np.concatenate(parts) - a).max() < 1e-9
    return True


if __name__ == "__main__":
    self_check()
    print("ok")
