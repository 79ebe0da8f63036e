"""Plain float64 statement of the Logulix design (numpy; one function per mechanism; shares no code with the product).

A model is (cfg, W): cfg the parsed config.json, W a dict name -> float64 array.  Every mechanism takes the rows of ONE
sequence's next portion and the store that this run of the layer carries for the sequence (cache rows, recurrent state,
convolution tails, the last normed input), so `Stepper.feed` serves whole prompts, portions and single tokens alike.

Order of runs: the layer list with its looped segment repeated in place; every run has a store of its own.  Ahead of a pass's
first layer x becomes J [x; e], e the embedding output.
"""
import math

import numpy as np


def silu(z):
    return z / (1.0 + np.exp(-z))


def rms_unit(x, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


# ---- causal convolution over time, per channel, continuing from a tail --------------------------------------------------
def causal_conv(u, w, tail):
    """u [T, C], w [C, taps], tail [taps - 1, C] (the inputs before u, oldest first).  Returns (y, new tail)."""
    taps, T = w.shape[1], u.shape[0]
    full = np.concatenate([tail, u], axis=0)
    y = np.zeros_like(u)
    for t in range(T):
        for j in range(taps):
            y[t] += w[:, j] * full[t + j]
    return y, full[T:]


# ---- rotary -------------------------------------------------------------------------------------------------------------
def rotary_angles(rot, pos):
    dims = rot["dims"]
    f = np.array([float(rot["base"]) ** (-2.0 * i / dims) for i in range(dims // 2)])
    if rot.get("scaling"):
        f = f / float(rot["scaling"]["factor"])
    return np.asarray(pos, dtype=np.float64)[:, None] * f[None, :]


def rotate(x, pos, rot, halves):
    """x [T, heads, n]: the first `dims` entries of every head rotated by pairs, (i, i + dims / 2) or (2 i, 2 i + 1)"""
    if not rot:
        return x.copy()
    dims = rot["dims"]
    ang = rotary_angles(rot, pos)
    out = x.copy()
    for i in range(dims // 2):
        a, b = (i, i + dims // 2) if halves else (2 * i, 2 * i + 1)
        c, s = np.cos(ang[:, i])[:, None], np.sin(ang[:, i])[:, None]
        out[..., a] = x[..., a] * c - x[..., b] * s
        out[..., b] = x[..., b] * c + x[..., a] * s
    return out


# ---- mixers -------------------------------------------------------------------------------------------------------------
def attention_mixer(h, m, W, p, eps, store, pos0):
    """Softmax attention under a sliding window; values are the convolved, not yet normed or rotated keys."""
    T = h.shape[0]
    H, G, D = m["heads"], m["kv_heads"], m["dim"]
    pos = pos0 + np.arange(T)

    def projected(name):
        u = h @ W[p + name].T + W[p + name + ".b"]
        tail = store.get("tail_" + name)
        if tail is None:
            tail = np.zeros((m["conv"] - 1, u.shape[1]))
        y, store["tail_" + name] = causal_conv(u, W[p + name + ".conv"], tail)
        return y

    q, k = projected("q"), projected("k")
    v = k.reshape(T, G, D)
    q = rms_unit(q, eps) * W[p + "q.norm"]                   # one mean over all heads' channels
    k = rms_unit(k, eps) * W[p + "k.norm"]
    q = rotate(q.reshape(T, H, D), pos, m.get("rot"), halves=False)
    k = rotate(k.reshape(T, G, D), pos, m.get("rot"), halves=False)
    store.setdefault("k", []).extend(k)
    store.setdefault("v", []).extend(v)
    K, V = np.array(store["k"]), np.array(store["v"])
    dist = pos[:, None] - np.arange(K.shape[0])[None, :]
    vis = (dist >= 0) & (dist < m["mask"]["size"])
    out = np.zeros((T, H, D))
    for hh in range(H):
        g = hh // (H // G)
        s = q[:, hh] @ K[:, g].T * m["scale"]
        s = m["softcap"] * np.tanh(s / m["softcap"])
        s = np.where(vis, s, -np.inf)
        e = np.exp(s - s.max(axis=1, keepdims=True))
        out[:, hh] = (e / e.sum(axis=1, keepdims=True)) @ V[:, g]
    return out.reshape(T, H * D) @ W[p + "o"].T + W[p + "o.b"]


def wkv_mixer(h, m, W, p, eps, store):
    """Token-shifted projections; per head o_t = (S + diag(u) k v^T)^T r, then S <- diag(w) S + k v^T."""
    T, H, D = h.shape[0], m["heads"], m["dim"]
    before = store.get("h")
    if before is None:
        before = np.zeros(h.shape[1])
    prev = np.concatenate([before[None], h[:-1]], axis=0)
    store["h"] = h[-1].copy()
    mixed = {c: h + (prev - h) * W[p + "mu." + c] for c in "rkvgw"}
    r, k, v = ((mixed[c] @ W[p + c].T).reshape(T, H, D) for c in "rkv")
    gate = silu(mixed["g"] @ W[p + "g"].T)
    w = np.exp(-np.exp(np.tanh(mixed["w"] @ W[p + "w1"].T) @ W[p + "w2"].T + W[p + "w0"])).reshape(T, H, D)
    u = W[p + "u"]
    S = store.get("S")
    if S is None:
        S = np.zeros((H, D, D))
    out = np.zeros((T, H, D))
    for t in range(T):
        kv = k[t][:, :, None] * v[t][:, None, :]
        out[t] = np.einsum("hde,hd->he", S + u[:, :, None] * kv, r[t])
        S = w[t][:, :, None] * S + kv
    store["S"] = S
    out = rms_unit(out, eps).reshape(T, H * D) * W[p + "norm"] * gate
    return out @ W[p + "o"].T


def retention_mixer(h, m, W, p, eps, store, pos0):
    """S_t = decay S_(t-1) + k_t v_t^T with one fixed decay per head, o_t = S_t^T q_t."""
    T, H, D, E = h.shape[0], m["heads"], m["dim"], m["vdim"]
    pos = pos0 + np.arange(T)
    q = rotate((h @ W[p + "q"].T).reshape(T, H, D), pos, m.get("rot"), halves=True)
    k = rotate((h @ W[p + "k"].T).reshape(T, H, D), pos, m.get("rot"), halves=True) / math.sqrt(D)
    v = (h @ W[p + "v"].T).reshape(T, H, E)
    decay = np.asarray(m["decay"], dtype=np.float64)
    S = store.get("S")
    if S is None:
        S = np.zeros((H, D, E))
    out = np.zeros((T, H, E))
    for t in range(T):
        S = decay[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = np.einsum("hde,hd->he", S, q[t])
    store["S"] = S
    out = rms_unit(out, eps).reshape(T, H * E) * silu(h @ W[p + "g"].T)
    return out @ W[p + "o"].T


# ---- feed-forward ---------------------------------------------------------------------------------------------------------
def dense_ff(h, W, p):
    return np.maximum(h @ W[p + "up"].T, 0.0) ** 2 @ W[p + "down"].T


# ---- the order of runs: (layer, opens a pass) -------------------------------------------------------------------------------
def layer_runs(cfg):
    n, lp = len(cfg["layers"]), cfg.get("loop")
    if not lp:
        return [(i, False) for i in range(n)]
    runs = [(i, False) for i in range(lp["start"])]
    for _ in range(lp["times"]):
        runs += [(i, i == lp["start"]) for i in range(lp["start"], lp["stop"])]
    return runs + [(i, False) for i in range(lp["stop"], n)]


class Stepper:
    """One sequence: feed(tokens) runs its next portion and returns (logits [T, vocab], taps [runs, T, width])."""

    def __init__(self, cfg, W):
        self.cfg, self.W = cfg, W
        self.pos = 0
        self.runs = layer_runs(cfg)
        self.stores = [dict() for _ in self.runs]

    def feed(self, tokens):
        cfg, W = self.cfg, self.W
        eps = cfg["norm"]["eps"]
        e = W["embed"][np.asarray(tokens)] * cfg["embedding"]["scale"]
        x, taps = e, []
        for (i, opens), st in zip(self.runs, self.stores):
            if opens:
                x = np.concatenate([x, e], axis=1) @ W["loop.in"].T
            L, pre = cfg["layers"][i], "l%d." % i
            m, p = L["mixer"], pre + "mix."
            h = rms_unit(x, eps) * W[pre + "norm1"]
            if L["type"] == "attention":
                y = attention_mixer(h, m, W, p, eps, st, self.pos)
            elif L["type"] == "wkv":
                y = wkv_mixer(h, m, W, p, eps, st)
            elif L["type"] == "retention":
                y = retention_mixer(h, m, W, p, eps, st, self.pos)
            else:
                raise ValueError(L["type"])
            x = x + y
            if L.get("mlp"):
                x = x + dense_ff(rms_unit(x, eps) * W[pre + "norm2"], W, pre + "mlp.")
            taps.append(x)
        self.pos += len(tokens)
        return (rms_unit(x, eps) * W["final.norm"]) @ W["head"].T * cfg["logit_scale"], np.array(taps)


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
def tensor_shapes(cfg, rank=6):
    """`rank`: rows of the wkv mixers' first decay matrix (a property of the tensors, not of the config)"""
    Wd = cfg["width"]
    out = {"embed": (cfg["vocab"], Wd), "final.norm": (Wd,), "head": (cfg["vocab"], Wd)}
    if cfg.get("loop"):
        out["loop.in"] = (Wd, 2 * Wd)
    for i, L in enumerate(cfg["layers"]):
        pre = "l%d." % i
        m, p = L["mixer"], pre + "mix."
        out[pre + "norm1"] = (Wd,)
        if L["type"] == "attention":
            for n, c in (("q", m["heads"] * m["dim"]), ("k", m["kv_heads"] * m["dim"])):
                out.update({p + n: (c, Wd), p + n + ".b": (c,), p + n + ".norm": (c,), p + n + ".conv": (c, m["conv"])})
            out.update({p + "o": (Wd, m["heads"] * m["dim"]), p + "o.b": (Wd,)})
        elif L["type"] == "wkv":
            c = m["heads"] * m["dim"]
            out.update({p + "mu." + n: (Wd,) for n in "rkvgw"})
            out.update({p + n: (c, Wd) for n in "rkvg"})
            out.update({p + "w1": (rank, Wd), p + "w2": (c, rank), p + "w0": (c,), p + "u": (m["heads"], m["dim"]), p + "norm": (c,), p + "o": (Wd, c)})
        else:
            cq, cv = m["heads"] * m["dim"], m["heads"] * m["vdim"]
            out.update({p + "q": (cq, Wd), p + "k": (cq, Wd), p + "v": (cv, Wd), p + "g": (cv, Wd), p + "o": (Wd, cv)})
        if L.get("mlp"):
            out.update({pre + "norm2": (Wd,), pre + "mlp.up": (L["mlp"]["ff"], Wd), pre + "mlp.down": (Wd, L["mlp"]["ff"])})
    return out


def random_weights(cfg, seed=0, rank=6):
    """bfloat16-representable float64 values, scaled so that activations stay of order one through the layers"""
    rng = np.random.default_rng(seed)
    W = {}
    for name, shape in tensor_shapes(cfg, rank).items():
        leaf = name.split(".")[-1]
        if "norm" in leaf:
            a = 1.0 + 0.2 * rng.standard_normal(shape)
        elif leaf == "conv":
            a = 0.5 * rng.standard_normal(shape)
        elif leaf == "b":
            a = 0.3 * rng.standard_normal(shape)
        elif ".mu." in name:
            a = rng.uniform(0.0, 1.0, shape)
        elif leaf == "w0":
            a = rng.uniform(-5.0, 0.5, shape)
        elif leaf == "u":
            a = rng.standard_normal(shape)
        elif leaf == "embed":
            a = rng.standard_normal(shape)
        else:
            a = rng.standard_normal(shape) / math.sqrt(shape[-1])
        W[name] = bf16_round(a)
    return W


def self_check():
    """The statement agrees with itself: a whole prompt, the same prompt token by token, and in uneven portions."""
    att = {"heads": 4, "kv_heads": 2, "dim": 6, "vdim": 6, "conv": 3, "scale": 0.5, "softcap": 4.0, "mask": {"size": 5},
           "rot": {"dims": 4, "base": 50.0, "scaling": {"factor": 3.0}}}
    ret = {"heads": 2, "dim": 5, "vdim": 7, "decay": [0.7, 0.95], "rot": {"dims": 4, "base": 30.0}}
    cfg = {"architecture": "Logulix", "width": 20, "vocab": 30, "norm": {"eps": 1e-6}, "embedding": {"scale": 1.5}, "logit_scale": 0.7,
           "loop": {"start": 1, "stop": 3, "times": 3},
           "layers": [{"type": "retention", "mixer": ret, "mlp": {"kind": "dense", "ff": 18}},
                      {"type": "attention", "mixer": att, "mlp": None},
                      {"type": "wkv", "mixer": {"heads": 3, "dim": 4}, "mlp": {"kind": "dense", "ff": 14}},
                      {"type": "attention", "mixer": dict(att, conv=1, kv_heads=4), "mlp": None}]}
    W = random_weights(cfg, 3)
    toks = list(np.random.default_rng(1).integers(0, 30, 19))
    a, ta = forward(cfg, W, toks)
    b, tb = forward_tokenwise(cfg, W, toks)
    assert ta.shape == (8, 19, 20)
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
