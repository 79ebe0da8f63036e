"""Gavodra through the serving path (ServingEngine -> SequenceEngine -> tha_hyb_step) against the plain float64 statement of the
design in tests/gavodra_oracle.py.

Every test builds its own small configuration with random weights.  float32 runs are compared tightly (they differ from float64 by
rounding only), bfloat16 runs loosely.  Where random weights would hide a fault (one far key among hundreds, a distance one row of the
bias table off, a value mixed with another token's) the weights are made sharp, so that one key or one row of the table carries the
result and reading another moves the output by tens of percent.
"""
import copy
import ctypes as C
import json
import os
import subprocess

import numpy as np
import pytest

import gavodra_oracle as O
from pkgload import load_pkg

pytestmark = pytest.mark.gpu

F32_TOL, BF16_TOL = 1e-4, 6e-2
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def rel_err(got, want):
    got, want = np.asarray(got, np.float64), np.asarray(want, np.float64)
    return float(np.sqrt(((got - want) ** 2).mean()) / (np.sqrt((want ** 2).mean()) + 1e-12))


# ---- configurations ---------------------------------------------------------------------------------------------------
def dense(ff=56, limit=1.3):
    return {"kind": "dense", "ff": ff, "limit": limit}


def moe(experts=6, top=2, ff=24, limit=0.8, scale=1.7, shared=40, shared_limit=1.1):
    f = {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top, "scale": scale}}
    if shared:
        f["shared"] = {"ff": shared, "limit": shared_limit}
    return f


def attention(mlp=None, heads=4, kv_heads=2, dim=16, vdim=12, scale=0.3, bias_max=35, v_mix=True):
    return {"type": "attention", "mlp": mlp, "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale,
                                                       "bias_max": bias_max, "v_mix": v_mix}}


def model(layers, width=64, vocab=130, eps=1e-5, embed=1.4, logit=0.8, cap=12.0, mult=0.6):
    return {"architecture": "Gavodra", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width, "embedding": {"scale": embed},
            "logit_scale": logit, "logit_softcap": cap, "residual_mult": mult}


class Built:
    """A model folder, its oracle view, and engines on demand."""

    def __init__(self, tmp, cfg, seed=0, tweak=None, rel_rows=12):
        self.serving = load_pkg("serving")
        self.cfg = cfg
        self.w = O.random_weights(cfg, seed, rel_rows)
        if tweak:
            tweak(self.w)
            for k in self.w:
                self.w[k] = O.bf16_round(self.w[k])
        self.folder = str(tmp)
        os.makedirs(self.folder, exist_ok=True)
        self.serving.save_model_folder(self.folder, cfg, {k: np.asarray(v, np.float32) for k, v in self.w.items()})
        self._ref = {}

    def engine(self, dtype="float32", max_tokens=1024, max_seqs=4):
        return self.serving.ServingEngine(self.folder, dtype, max_tokens, max_seqs)

    def ref(self, tokens):
        key = tuple(tokens)
        if key not in self._ref:
            self._ref[key] = O.forward(self.cfg, self.w, list(tokens))
        return self._ref[key]


@pytest.fixture(scope="module")
def general(tmp_path_factory):
    # layers with and without value mixing (the first that mixes is not the first layer), every feed-forward, none, head groups of one to
    # three, distances beyond the end of every bias table, one table that ends next to its linear half
    layers = [attention(dense(), v_mix=False, vdim=20), attention(moe(), heads=6, kv_heads=2, dim=8), attention(None, kv_heads=2, v_mix=False, bias_max=61.5),
              attention(moe(experts=9, top=3, shared=None), heads=2, dim=32, bias_max=7), attention(dense(40, 0.7), heads=2, kv_heads=2, scale=0.5),
              attention(moe(top=1, shared=17), bias_max=90)]
    return Built(tmp_path_factory.mktemp("general"), model(layers), seed=1)


def tokens_for(built, n, seed):
    return np.random.default_rng(seed).integers(0, built.cfg["vocab"], n).tolist()


def feed(e, rid, toks, cuts):
    """the tokens in portions of the given sizes (the last size repeats); logits of every position"""
    out, at, i = [], 0, 0
    while at < len(toks):
        c = min(cuts[min(i, len(cuts) - 1)], len(toks) - at)
        out.append(e.step([(rid, toks[at:at + c], list(range(c)))]))
        at += c
        i += 1
    return np.concatenate(out, 0)


# ---- whole prompts, every layer -----------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype,tol", [("float32", F32_TOL), ("bfloat16", BF16_TOL)])
@pytest.mark.parametrize("n", [1, 2, 97])
def test_whole_prompt_every_layer(general, dtype, tol, n):
    toks = tokens_for(general, n, 3)
    z, layers = general.ref(toks)
    logits, taps = general.engine(dtype).step([("a", toks, list(range(n)))], taps=True)
    assert taps.shape == layers.shape
    for i in range(len(layers)):
        assert rel_err(taps[i], layers[i]) < tol, f"residual stream after layer {i}"
    assert rel_err(logits, z) < tol


# ---- each mechanism alone -----------------------------------------------------------------------------------------------
def one_layer(tmp, layer, width=48, seed=2, tweak=None, rel_rows=12, **kw):
    return Built(tmp, model([layer], width=width, vocab=90, **kw), seed, tweak, rel_rows)


def check_all_positions(b, n=70, dtype="float32", tol=F32_TOL, cuts=None):
    toks = tokens_for(b, n, 9)
    z, layers = b.ref(toks)
    if cuts:
        got = feed(b.engine(dtype), "a", toks, cuts)
    else:
        got, taps = b.engine(dtype).step([("a", toks, list(range(n)))], taps=True)
        for g, w in zip(taps, layers):
            assert rel_err(g, w) < tol
    assert rel_err(got, z) < tol


def matters(b, n=70, cfg=None, **changed):
    """how far the statement's logits move when tensors or the config are changed: what a test can tell apart"""
    toks = tokens_for(b, n, 9)
    w = dict(b.w)
    for k, f in changed.items():
        name = k.replace("__", ".")
        w[name] = f(b.w[name].copy())
    return rel_err(O.forward(cfg or b.cfg, w, toks)[0], b.ref(toks)[0])


def changed_config(b, layer, path, value):
    cfg = copy.deepcopy(b.cfg)
    at = cfg["layers"][layer]
    for k in path[:-1]:
        at = at[k]
    at[path[-1]] = value
    return cfg


@pytest.mark.parametrize("heads,kv_heads,dim,vdim", [(4, 2, 16, 12), (3, 3, 20, 16), (6, 2, 48, 40), (5, 1, 7, 9), (70, 1, 16, 8), (1, 1, 1, 1)])
def test_attention_alone(tmp_path, heads, kv_heads, dim, vdim):
    b = one_layer(tmp_path, attention(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim))
    check_all_positions(b)
    check_all_positions(b, cuts=[3, 1, 20, 2])
    check_all_positions(b, dtype="bfloat16", tol=BF16_TOL)
    check_all_positions(b, dtype="bfloat16", tol=BF16_TOL, cuts=[41, 1])
    assert matters(b, l0__mix__rel=np.zeros_like) > 1e-3
    assert matters(b, l0__mix__g=np.zeros_like) > 1e-3
    if dim > 1:
        for t in ("l0__mix__q__norm", "l0__mix__k__norm"):
            assert matters(b, **{t: np.ones_like}) > 1e-4, t


def test_heads_are_normed_one_by_one(tmp_path):
    """heads of very different size: one mean over the row would leave them different"""
    def tweak(w):
        w["l0.mix.q"][:16] *= 8.0
        w["l0.mix.k"][:16] *= 0.1
    b = one_layer(tmp_path, attention(scale=0.8), tweak=tweak)
    check_all_positions(b)
    check_all_positions(b, dtype="bfloat16", tol=BF16_TOL, cuts=[30, 1])


TABLES = [(12, 35), (8, 64), (32, 190), (2, 5), (3, 40), (9, 50), (24, 700), (64, 33), (20, 320), (5, 2.5)]


@pytest.mark.parametrize("rows,far", TABLES)
def test_distance_bias_decides_alone(tmp_path, rows, far):
    """queries and keys say nothing, neighbouring rows of the table differ by several units: a bucket edge that is one distance off shows;
    decoded one by one, in portions, and in one prompt"""
    def tweak(w):
        t = w["l0.mix.rel"]
        t[...] = np.random.default_rng(5).uniform(-3.0, 3.0, t.shape) + 2.0 * np.arange(rows)[:, None] / rows
    b = one_layer(tmp_path, attention(heads=6, kv_heads=2, scale=1e-6, bias_max=far), tweak=tweak, rel_rows=rows)
    if rows > 3:
        assert matters(b, n=130, l0__mix__rel=lambda a: np.roll(a, 1, axis=0)) > 1e-2
    for cuts in (None, [90, 1], [33, 2, 1, 31, 64]):
        check_all_positions(b, n=130, cuts=cuts)
    check_all_positions(b, n=130, dtype="bfloat16", tol=BF16_TOL, cuts=[100, 1])


@pytest.mark.parametrize("rows,far,kv_heads,dim", [(12, 96, 12, 16), (12, 96, 4, 16), (8, 64, 2, 10), (16, 410, 1, 32)])
def test_every_row_of_the_distance_table_by_itself(tmp_path, rows, far, kv_heads, dim):
    """head h is left with the keys of row h only, so its output is the mean over exactly the distances of that row: every position by
    itself, also the first and last distance of every row"""
    def tweak(w):
        w["l0.mix.rel"][...] = -30.0
        np.fill_diagonal(w["l0.mix.rel"], 0.0)
        w["l0.mix.g"][...] = 0.0
    b = one_layer(tmp_path, attention(heads=rows, kv_heads=kv_heads, dim=dim, scale=1e-6, bias_max=far), tweak=tweak, rel_rows=rows)
    n = 3 * 96 + 5 if far < 400 else 450
    toks = tokens_for(b, n, 4)
    base = b.w["embed"][np.asarray(toks)] * b.cfg["embedding"]["scale"]
    want = b.ref(toks)[1][0] - base
    for dtype, tol in (("float32", F32_TOL), ("bfloat16", BF16_TOL)):
        for cuts in ([n], [n - 40, 1], [31, 33, 64]):
            e, at, got, i = b.engine(dtype), 0, [], 0
            while at < n:
                c = min(cuts[min(i, len(cuts) - 1)], n - at)
                got.append(e.step([("a", toks[at:at + c], [])], taps=True)[1][0])
                at += c
                i += 1
            got = np.concatenate(got, 0) - base
            assert max(rel_err(got[p], want[p]) for p in range(n)) < 3 * tol, (dtype, cuts)


def test_the_bias_is_not_scaled_and_each_layer_has_its_own(tmp_path):
    b = Built(tmp_path, model([attention(dense(), scale=0.05), attention(dense(), scale=4.0, bias_max=60)], width=48, vocab=90), 3)
    for i in (0, 1):
        assert matters(b, **{"l%d__mix__rel" % i: lambda a: a * b.cfg["layers"][i]["mixer"]["scale"]}) > 1e-3
    assert matters(b, l1__mix__rel=lambda a: b.w["l0.mix.rel"].copy()) > 1e-3
    check_all_positions(b)
    check_all_positions(b, cuts=[50, 1])


def mixing_model(tmp, pattern, lams=None):
    layers = [attention(dense() if i % 2 else None, v_mix=v, vdim=12, heads=4 if i % 3 else 2) for i, v in enumerate(pattern)]

    def tweak(w):
        for i, v in enumerate(pattern):
            if v and lams:
                w["l%d.mix.vmix" % i] = np.array(lams[i])
    return Built(tmp, model(layers, width=48, vocab=90), 7, tweak)


@pytest.mark.parametrize("pattern", [(1, 1, 1), (0, 1, 1), (0, 0, 1, 0, 1, 1), (1, 0, 0, 1), (0, 0), (1, 0), (0, 1)])
def test_value_mixing(tmp_path, pattern):
    pattern = [bool(v) for v in pattern]
    b = mixing_model(tmp_path, pattern)
    first = pattern.index(True) if any(pattern) else -1
    for i, v in enumerate(pattern):
        if v:
            moved = matters(b, **{"l%d__mix__vmix" % i: np.zeros_like})
            assert moved > 1e-3 if i > first else moved == 0.0      # the first one's share is not used
    check_all_positions(b)
    check_all_positions(b, cuts=[20, 2, 1, 30, 1])
    check_all_positions(b, dtype="bfloat16", tol=BF16_TOL, cuts=[40, 1])


@pytest.mark.parametrize("lams", [(0.5, 0.0, 1.0), (-3.0, 1.0, 1.0), (9.0, -0.5, 1.75)])
def test_value_mixing_shares_outside_the_usual_range(tmp_path, lams):
    """all of the first values, none of them, a negative share; what is blended in is the first mixing layer's values as that layer keeps
    them, not a blend of blends"""
    b = mixing_model(tmp_path, (True, True, True), lams)
    check_all_positions(b)
    check_all_positions(b, cuts=[33, 1, 2])


@pytest.mark.parametrize("ff", [dense(56, 0.3), dense(64, 5.0), dense(33, 1.0), dense(1, 0.5)])
def test_dense_feed_forward(tmp_path, ff):
    def tweak(w):
        for n in ("gate", "up"):
            w["l0.mlp." + n][...] *= 1.5
    b = one_layer(tmp_path, attention(ff), tweak=tweak)
    assert matters(b, cfg=changed_config(b, 0, ("mlp", "limit"), 1e9)) > (-1 if ff["limit"] > 4 else 1e-3)
    check_all_positions(b)
    check_all_positions(b, dtype="bfloat16", tol=BF16_TOL, cuts=[50, 1])


@pytest.mark.parametrize("ff", [moe(), moe(experts=16, top=16), moe(experts=5, top=1, shared=None, scale=0.4), moe(experts=40, top=7, ff=9, shared=3),
                                moe(experts=1, top=1), moe(experts=130, top=4, ff=8, shared=64), moe(limit=0.2, shared_limit=3.0), moe(limit=4.0, shared_limit=0.1)])
def test_mixture(tmp_path, ff):
    def tweak(w):
        w["l0.mlp.router"][...] *= 2.0
        for k in w:
            if k.startswith("l0.mlp.") and k.split(".")[-1] in ("gate", "up"):
                w[k] = w[k] * 1.5
    b = one_layer(tmp_path, attention(ff), tweak=tweak, width=64)
    experts, top = ff["router"]["experts"], ff["router"]["top"]
    if top < experts:
        assert matters(b, l0__mlp__correction=np.zeros_like) > 1e-3    # the corrections change who is chosen
    if ff.get("shared"):
        assert matters(b, l0__mlp__shared__sg=np.zeros_like) > 1e-3
    assert matters(b, cfg=changed_config(b, 0, ("mlp", "expert", "limit"), 1e9)) > (-1 if ff["expert"]["limit"] > 3 else 1e-3)
    check_all_positions(b)
    check_all_positions(b, cuts=[2, 1, 40, 3])


def test_mixture_bfloat16_with_clear_choices(tmp_path):
    """corrections that settle the choice by a margin (a choice within bfloat16's rounding may go either way)"""
    def tweak(w):
        w["l0.mlp.correction"][...] = np.array([3.0, 0.0, -2.0, 2.0, 0.0, 1.0])
    b = one_layer(tmp_path, attention(moe(top=3)), tweak=tweak, width=64)
    check_all_positions(b, dtype="bfloat16", tol=BF16_TOL)
    check_all_positions(b, dtype="bfloat16", tol=BF16_TOL, cuts=[33, 1])


def test_norms_sit_on_the_results(tmp_path):
    """the sublayers read x as it is: making x ten times as large changes them, scaling what they return does not"""
    b = one_layer(tmp_path, attention(dense()), embed=6.0)
    assert matters(b, l0__mix__o=lambda a: 4.0 * a) < 1e-3 and matters(b, l0__mlp__down=lambda a: 4.0 * a) < 1e-3
    for t in ("l0__norm1", "l0__norm2", "final__norm"):
        assert matters(b, **{t: np.ones_like}) > 1e-2, t
    check_all_positions(b)


def test_constants_of_the_model(tmp_path):
    for i, kw in enumerate((dict(embed=0.25, logit=3.0, cap=2.0, mult=1.0), dict(embed=10.0, logit=0.1, cap=50.0, mult=0.1), dict(embed=1.0, logit=1.0, cap=0.7, mult=2.5),
                            dict(eps=0.3), dict(eps=1e-8))):
        b = Built(tmp_path / str(i), model([attention(dense()), attention(moe())], width=24, vocab=50, **kw), 4)
        check_all_positions(b, n=20)


# ---- portions, decoding, batches ------------------------------------------------------------------------------------------
@pytest.mark.parametrize("cuts", [[1], [2], [3, 5, 2, 7, 1, 16, 2], [40, 1], [64, 2, 2, 33]])
def test_portions_equal_the_whole_prompt(general, cuts):
    toks = tokens_for(general, 110, 11)
    assert rel_err(feed(general.engine(), "a", toks, cuts), general.ref(toks)[0]) < F32_TOL


def test_prefill_equals_token_by_token_decoding(general):
    toks = tokens_for(general, 90, 12)
    whole = general.engine().step([("a", toks, list(range(90)))])
    assert rel_err(feed(general.engine(), "a", toks, [1]), whole) < 2e-5
    assert rel_err(whole, O.forward_tokenwise(general.cfg, general.w, toks)[0]) < F32_TOL


def test_portions_bfloat16(general):
    toks = tokens_for(general, 100, 13)
    assert rel_err(feed(general.engine("bfloat16"), "a", toks, [37, 2, 1]), general.ref(toks)[0]) < BF16_TOL


def test_long_decoding(general):
    toks = tokens_for(general, 420, 14)
    z, _ = general.ref(toks)
    got = feed(general.engine(), "a", toks, [20, 1])
    assert rel_err(got, z) < F32_TOL
    assert rel_err(got[-1], z[-1]) < 5 * F32_TOL


@pytest.mark.parametrize("dtype,tol", [("float32", F32_TOL), ("bfloat16", BF16_TOL)])
def test_mixed_batches_equal_each_request_alone(general, dtype, tol):
    """Six unequal requests through an engine with three slots and fewer blocks than their sum: portions of some beside single tokens of
    others, requests ending and their slots and blocks going to the next ones."""
    lens = [70, 5, 131, 33, 18, 90]
    reqs = {f"r{i}": tokens_for(general, n, 20 + i) for i, n in enumerate(lens)}
    e = general.engine(dtype, max_tokens=288, max_seqs=3)
    got, at = {k: [] for k in reqs}, {k: 0 for k in reqs}
    waiting, live, step = list(reqs), [], 0
    sizes = [7, 1, 16, 2, 1, 30, 1, 3]
    while waiting or live:
        while waiting and len(live) < 3 and e.free_blocks() * 16 >= len(reqs[waiting[0]]) + 48:
            live.append(waiting.pop(0))
        entries = []
        for j, k in enumerate(live):
            n = min(sizes[(step + j) % len(sizes)], len(reqs[k]) - at[k])
            entries.append((k, reqs[k][at[k]:at[k] + n], list(range(n))))
        out, o = e.step(entries), 0
        for k, toks, w in entries:
            got[k].append(out[o:o + len(w)])
            o += len(w)
            at[k] += len(toks)
        for k in [k for k in live if at[k] == len(reqs[k])]:
            e.finish(k)
            live.remove(k)
        step += 1
    for k, toks in reqs.items():
        assert rel_err(np.concatenate(got[k], 0), general.ref(toks)[0]) < tol, k


def test_a_request_left_out_of_a_step_goes_on_later(general):
    a, b = tokens_for(general, 40, 51), tokens_for(general, 30, 52)
    e = general.engine(max_seqs=2)
    out = [e.step([("a", a[:10], list(range(10))), ("b", b[:7], list(range(7)))])]
    out.append(e.step([("b", b[7:20], list(range(13)))]))        # a waits
    out.append(e.step([("a", a[10:], list(range(30))), ("b", b[20:], list(range(10)))]))
    assert rel_err(np.concatenate([out[0][:10], out[2][:30]]), general.ref(a)[0]) < F32_TOL
    assert rel_err(np.concatenate([out[0][10:], out[1], out[2][30:]]), general.ref(b)[0]) < F32_TOL


def test_reused_slots_and_blocks_hold_nothing(general):
    a, b = tokens_for(general, 80, 31), tokens_for(general, 45, 32)
    e = general.engine(max_tokens=128, max_seqs=1)
    e.step([("a", a, [])])
    e.finish("a")
    assert rel_err(e.step([("b", b, list(range(45)))]), general.ref(b)[0]) < F32_TOL


def test_pool_exhaustion_is_an_error_not_a_fault(general):
    e = general.engine(max_tokens=64, max_seqs=2)
    with pytest.raises(Exception):
        e.step([("a", tokens_for(general, 100, 1), [])])
    e.finish("a")
    toks = tokens_for(general, 20, 2)
    assert rel_err(e.step([("b", toks, [19])]), general.ref(toks)[0][[19]]) < F32_TOL


# ---- sharp weights: far keys, page borders -----------------------------------------------------------------------------------
HALF = 32


def sharp_attention(tmp, dim=16, vocab=1024, layers=1):
    """Queries read the upper half of the layer's input, keys the lower half through the same matrix, with a large score scale.  The upper
    half of the QUERY probe's embedding is the lower half of the KEY probe's: the query probe puts nearly all its weight on the key
    probe wherever it is, a different token with a different value.  (The norms make every other token's score a few units at most.)"""
    layer = attention(heads=2, kv_heads=1, dim=dim, vdim=24, scale=2.5 if dim < 64 else 1.0, bias_max=200)
    cfg = model([layer] * layers, width=2 * HALF, vocab=vocab, mult=0.9)

    def tweak(w):
        w["embed"][vocab - 2, HALF:] = w["embed"][vocab - 1, :HALF]
        for i in range(layers):
            p = "l%d.mix." % i
            for n in ("q", "k"):
                w[p + n + ".norm"][...] = 1.0
            w[p + "k"][:, HALF:] = 0.0
            q = w[p + "q"].reshape(2, dim, 2 * HALF)
            q[:, :, :HALF] = 0.0
            q[:, :, HALF:] = w[p + "k"][None, :, :HALF]
    return Built(tmp, cfg, 12, tweak)


def with_probes(b, n, key_pos, query_pos, seed):
    """distinct tokens with both probes in place; and the same without the key probe"""
    toks = np.random.default_rng(seed).permutation(b.cfg["vocab"] - 2)[:n + 1].tolist()
    spare = toks.pop()
    toks[key_pos], toks[query_pos] = b.cfg["vocab"] - 1, b.cfg["vocab"] - 2
    other = list(toks)
    other[key_pos] = spare
    return toks, other


def check_probe(b, n, key_pos, query_pos, cut_sets, dtype="float32", shift=0.1):
    """the engine agrees with the statement at the query probe, which depends on the key probe"""
    toks, other = with_probes(b, n, key_pos, query_pos, key_pos * 7 + query_pos)
    z, _ = b.ref(toks)
    moved = rel_err(b.ref(other)[0][query_pos], z[query_pos])
    assert moved > shift, moved
    tol = F32_TOL if dtype == "float32" else BF16_TOL
    for cuts in cut_sets:
        got = feed(b.engine(dtype), "a", toks, [c for c in cuts if c > 0] or [1])
        assert rel_err(got[query_pos], z[query_pos]) < (10 if dtype == "float32" else 1) * tol, cuts
        if dtype == "float32":
            assert rel_err(got, z) < tol, cuts


@pytest.mark.parametrize("key_pos,query_pos", [(0, 1), (0, 149), (15, 16), (16, 17), (63, 64), (64, 65), (63, 127), (64, 128), (127, 128), (1, 63)])
def test_keys_at_the_borders_of_the_block_table(tmp_path, key_pos, query_pos):
    b = sharp_attention(tmp_path, dim=64)
    check_probe(b, 150, key_pos, query_pos, ([150], [query_pos, 1], [key_pos, 2, 1], [key_pos + 1, 1]))


@pytest.mark.parametrize("dtype,decoded", [("float32", False), ("float32", True), ("bfloat16", False), ("bfloat16", True)])
@pytest.mark.parametrize("dim", [16, 64])
def test_one_far_key_among_hundreds(tmp_path, dtype, decoded, dim):
    b = sharp_attention(tmp_path, dim=dim)
    check_probe(b, 700, 3, 690, ([670, 1] if decoded else [300, 400],), dtype)


@pytest.mark.parametrize("key_pos,query_pos", [(0, 300), (63, 64), (64, 200), (170, 171)])
def test_a_far_key_brings_its_own_first_values(tmp_path, key_pos, query_pos):
    """the second layer's read-out at the probe is the blend of the key's two value rows: the blend must be of the same token, wherever the
    portions were cut between writing and reading it"""
    b = sharp_attention(tmp_path, dim=32, layers=2)
    toks, _ = with_probes(b, 310, key_pos, query_pos, key_pos * 7 + query_pos)
    w = dict(b.w)
    w["l1.mix.vmix"] = np.array(0.0)
    z = b.ref(toks)[0]
    assert rel_err(O.forward(b.cfg, w, toks)[0][query_pos], z[query_pos]) > 1e-2
    for cuts in ([310], [query_pos, 1], [key_pos + 1, 2, 1], [100]):
        got = feed(b.engine(), "a", toks, cuts)
        assert rel_err(got[query_pos], z[query_pos]) < 10 * F32_TOL and rel_err(got, z) < F32_TOL, cuts


def test_few_rows_at_a_long_context(tmp_path):
    """steps of one or two rows behind hundreds of positions are cut along the keys and merged; value rows that are no multiple of a warp;
    parts that lie wholly in the far end of the bias beside parts that do not"""
    b = Built(tmp_path, model([attention(dense(), heads=6, kv_heads=2, dim=40, vdim=40, bias_max=300), attention(None, heads=4, kv_heads=2, dim=72, vdim=40)],
                              width=64, vocab=120), 7)
    toks = tokens_for(b, 720, 4)
    z, _ = b.ref(toks)
    for dtype, tol in (("float32", F32_TOL), ("bfloat16", BF16_TOL)):
        got = feed(b.engine(dtype), "a", toks, [600, 38, 2, 1, 1, 2, 3, 1])
        assert max(rel_err(g, w) for g, w in zip(got[600:], z[600:])) < 3 * tol
        assert rel_err(got, z) < tol


@pytest.mark.parametrize("heads,kv_heads,rows,far", [(6, 2, 32, 190), (8, 1, 16, 50), (4, 4, 12, 280), (10, 2, 8, 900)])
@pytest.mark.parametrize("cuts", [[300], [150, 86, 2, 1], [64, 1]])
def test_tensor_core_attention_bfloat16_every_position(tmp_path, cuts, heads, kv_heads, rows, far):
    """heads that take the tensor-core form, peaked scores, strong biases, and a check of EVERY position by itself"""
    def tweak(w):
        w["l0.mix.rel"] *= 4.0
    b = Built(tmp_path, model([attention(heads=heads, kv_heads=kv_heads, dim=48, vdim=40, scale=0.4, bias_max=far)], width=64, vocab=200), 41, tweak, rows)
    n = 300
    toks = tokens_for(b, n, 3)
    base = b.w["embed"][np.asarray(toks)] * b.cfg["embedding"]["scale"]
    mix = b.ref(toks)[1][0] - base
    e, at, got, i = b.engine("bfloat16"), 0, [], 0
    while at < n:
        c = min(cuts[min(i, len(cuts) - 1)], n - at)
        got.append(e.step([("a", toks[at:at + c], [])], taps=True)[1][0])
        at += c
        i += 1
    got = np.concatenate(got, 0) - base
    assert max(rel_err(got[p], mix[p]) for p in range(n)) < 6e-2
    assert rel_err(got, mix) < 2e-2


def test_prompt_sized_mixture_runs_expert_by_expert(tmp_path, monkeypatch):
    """steps of a thousand rows give every expert one tensor-core product of its own; the same rows in small portions use the grouped one"""
    def tweak(w):
        w["l0.mlp.correction"][...] = np.array([2.0, -1.5, 1.0, 0.0])
    b = one_layer(tmp_path, attention(moe(experts=4, top=2, ff=64, shared=48), heads=2, kv_heads=1), tweak=tweak, width=64)
    toks = tokens_for(b, 1100, 6)
    small = feed(b.engine("bfloat16", max_tokens=2048), "a", toks, [300])
    monkeypatch.setenv("THA_HYB_EXPERT_ROWS", "100")
    big = feed(b.engine("bfloat16", max_tokens=2048), "a", toks, [1100])
    z = b.ref(toks)[0]
    assert rel_err(small, z) < BF16_TOL and rel_err(big, z) < BF16_TOL and rel_err(big, small) < 2e-2


# ---- other sizes: values that are often equal, or 1 ------------------------------------------------------------------
@pytest.mark.parametrize("case", ["single", "wide_heads", "everything_small", "odd_sizes", "many_kv_heads", "no_feed_forward", "mixtures_only",
                                  "value_rows_wider_than_keys", "aligned"])
def test_other_sizes(tmp_path, case):
    width, n, rows = 32, 75, 12
    if case == "single":
        layers = [attention(dense(8), heads=1, kv_heads=1, dim=8, vdim=8, v_mix=False), attention(moe(1, 1, 8, shared=8), heads=1, kv_heads=1, dim=24, vdim=24)]
        width, rows = 24, 2
    elif case == "wide_heads":
        layers = [attention(dense(40), heads=2, kv_heads=2, dim=150, vdim=130, scale=0.08), attention(moe(), heads=4, kv_heads=2, dim=288, vdim=130, scale=0.05),
                  attention(dense(), heads=1, kv_heads=1, dim=64, vdim=260)]
        width = 40
    elif case == "everything_small":
        layers = [attention(dense(1), heads=1, kv_heads=1, dim=1, vdim=1, bias_max=3), attention(moe(2, 1, 1, shared=1), heads=1, kv_heads=1, dim=2, vdim=1, bias_max=2)]
        width, rows = 5, 3
    elif case == "odd_sizes":
        layers = [attention(dense(11), heads=6, kv_heads=3, dim=7, vdim=5, bias_max=29.5), attention(moe(7, 3, 13, shared=9), heads=9, kv_heads=3, dim=11, vdim=5)]
        width, rows = 27, 13
    elif case == "many_kv_heads":
        layers = [attention(heads=3, kv_heads=3, v_mix=False), attention(dense(), heads=6, kv_heads=6, dim=8, vdim=4), attention(heads=8, kv_heads=2, dim=8)]
    elif case == "no_feed_forward":
        layers = [attention(), attention(), attention()]
    elif case == "mixtures_only":
        layers = [attention(moe(8, 8, 12)), attention(moe(33, 5, 7, shared=None))]
    elif case == "value_rows_wider_than_keys":
        layers = [attention(dense(), dim=8, vdim=48), attention(moe(), dim=4, vdim=48)]
    else:                                                     # every product on the tensor cores
        layers = [attention(dense(96), heads=4, kv_heads=1, dim=32, vdim=64), attention(moe(8, 3, 64, shared=96), heads=8, kv_heads=2, dim=64, vdim=32),
                  attention(moe(4, 2, 128, shared=64), heads=6, kv_heads=2, dim=16, vdim=32)]
        width, n, rows = 96, 150, 24
    b = Built(tmp_path, model(layers, width=width, vocab=61), 5, rel_rows=rows)
    toks = tokens_for(b, n, 2)
    z, layers_ref = b.ref(toks)
    logits, taps = b.engine().step([("a", toks, list(range(n)))], taps=True)
    for i in range(len(layers_ref)):
        assert rel_err(taps[i], layers_ref[i]) < F32_TOL, f"layer {i}"
    assert rel_err(logits, z) < F32_TOL
    assert rel_err(feed(b.engine(), "a", toks, [9, 2, 1]), z) < F32_TOL
    assert rel_err(feed(b.engine("bfloat16"), "a", toks, [40, 1]), z) < 2.5 * BF16_TOL


# ---- operations by themselves -------------------------------------------------------------------------------------------
class Norm(C.Structure):
    _fields_ = [("kind", C.c_int), ("w", C.c_void_p), ("b", C.c_void_p), ("w_offset", C.c_float), ("alpha", C.c_float)]


@pytest.mark.parametrize("width", [4, 30, 192, 1024, 5120, 13000])
@pytest.mark.parametrize("parts", ["dense", "gated", "mixture", "both"])
def test_end_of_a_post_norm_sublayer(width, parts):
    import torch
    lib = C.CDLL(os.path.join(ROOT, "hip_llama.cpp_b200", "lib", "libtha_b200.so"))
    lib.tha_hyb_post_norm.argtypes = ([C.c_void_p, C.c_int] + [C.c_void_p] * 3 + [C.c_longlong, C.c_int] + [C.c_void_p] * 3 +
                                      [C.c_float, C.POINTER(Norm), C.c_float, C.c_void_p, C.c_void_p, C.c_int, C.c_int])
    g = torch.Generator().manual_seed(width)
    R, top, ldg = 9, 3, 5
    x, dn, w = torch.randn(R, width, generator=g), torch.randn(R, width, generator=g), torch.randn(width, generator=g)
    gate, down = torch.randn(R, ldg, generator=g), torch.randn(R * top, width, generator=g)
    wt, inv = torch.rand(R, top, generator=g), torch.randperm(R * top, generator=g).to(torch.int32)
    y = torch.zeros(R, width, dtype=torch.float64)
    if parts != "mixture":
        y += dn.double() * (torch.sigmoid(gate[:, :1].double()) if parts in ("gated", "both") else 1.0)
    if parts in ("mixture", "both"):
        y += (wt.double()[:, :, None] * down.double()[inv.long()].view(R, top, width)).sum(1)
    want = x.double() + 0.7 * y / torch.sqrt((y * y).mean(1, keepdim=True) + 1e-3) * (0.25 + w.double())
    for dt, tt in ((0, torch.bfloat16), (1, torch.float32)):
        d = {k: v.cuda() for k, v in dict(x=x, dn=dn, w=w, gate=gate, down=down, wt=wt, inv=inv).items()}
        tap, out = torch.empty(R, width, device="cuda"), torch.empty(R, width, device="cuda", dtype=tt)
        n = Norm(0, d["w"].data_ptr(), None, 0.25, 0.0)
        st = lib.tha_hyb_post_norm(None, dt, d["x"].data_ptr(), d["dn"].data_ptr() if parts != "mixture" else None,
                                   d["gate"].data_ptr() if parts in ("gated", "both") else None, ldg, top if parts in ("mixture", "both") else 0, d["wt"].data_ptr(),
                                   d["inv"].data_ptr(), d["down"].data_ptr(), 0.7, C.byref(n), 1e-3, tap.data_ptr(), out.data_ptr(), R, width)
        torch.cuda.synchronize()
        assert st == 0
        assert float((d["x"].cpu().double() - want).abs().max()) < 1e-5 * float(want.abs().max())
        assert torch.equal(tap, d["x"]) and torch.equal(out, d["x"].to(tt))


# ---- generation through the scheduler ---------------------------------------------------------------------------------
def test_greedy_generation_through_the_scheduler(general):
    prompts = [tokens_for(general, n, 40 + n) for n in (5, 23, 70, 12, 3, 41)]
    new = [6, 9, 4, 12, 8, 5]
    e = general.engine(max_tokens=384, max_seqs=3)      # fewer slots than requests
    got = e.generate(prompts, new, temperature=0.0, portion=32)
    assert e.free_blocks() > 0 and e.steps_run() > max(new)
    for p, n, g in zip(prompts, new, got):
        assert len(g) == n
        st = O.Stepper(general.cfg, general.w)
        z = st.feed(p)[0][-1]
        for tok in g:
            best = int(np.argmax(z))
            if tok != best:                                # only a near tie may differ
                assert z[best] - z[tok] < 1e-3 * max(1.0, float(np.abs(z).max()))
            z = st.feed([tok])[0][-1]


def test_sampled_generation_is_reproducible_and_independent_of_the_batch(general):
    prompts = [tokens_for(general, n, 60 + n) for n in (9, 30)]
    a = general.engine(max_seqs=2).generate(prompts, [10, 10], temperature=1.0, topp=0.9, seed=7)
    b = general.engine(max_seqs=1).generate(prompts, [10, 10], temperature=1.0, topp=0.9, seed=7, portion=4)
    assert a == b


def test_the_app_serves_a_model_folder(general, tmp_path):
    app = os.path.join(ROOT, "build", "apps", "llama")
    if not os.path.exists(app):
        pytest.skip("the app is not built")
    prompts = [tokens_for(general, n, 80 + n) for n in (4, 19, 33)]
    (tmp_path / "in.txt").write_text("\n".join(" ".join(map(str, p)) for p in prompts) + "\n")
    r = subprocess.run([app, general.folder, "-m", "test", "-f", str(tmp_path / "in.txt"), "-o", str(tmp_path / "out.txt"), "-n", "7", "-b", "2",
                        "-d", "f32", "-j", "16"], capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    got = [[int(t) for t in line.split()] for line in (tmp_path / "out.txt").read_text().splitlines()]
    assert got == general.engine(max_seqs=2).generate(prompts, [7, 7, 7], temperature=0.0, portion=16)


def test_the_trace_replayer_answers_every_step(general, tmp_path):
    """the replayer on a model folder: steps in, logits files out, requests ended and their slot used again"""
    exe = os.path.join(ROOT, "build", "apps", "trace_run")
    if not os.path.exists(exe):
        pytest.skip("the program is not built")
    a, b = tokens_for(general, 70, 1), tokens_for(general, 20, 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:64], "want": [0, 63]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[64:], "want": [5]}, {"id": "b", "tokens": b[:18], "want": []}], "end": ["a"]},
             {"step": 2, "entries": [{"id": "b", "tokens": b[18:], "want": [0, 1]}], "end": ["b"]}]
    out = tmp_path / "out"
    out.mkdir()
    r = subprocess.run([exe, "--model", general.folder, "--dtype", "float32", "--out", str(out), "--max-tokens", "128", "--max-seqs", "2"],
                       input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2"]
    za, zb = general.ref(a)[0], general.ref(b)[0]
    V = general.cfg["vocab"]
    assert rel_err(np.fromfile(out / "0.f32", np.float32).reshape(-1, V), za[[0, 63]]) < F32_TOL
    assert rel_err(np.fromfile(out / "1.f32", np.float32).reshape(-1, V), za[[69]]) < F32_TOL
    assert rel_err(np.fromfile(out / "2.f32", np.float32).reshape(-1, V), zb[[18, 19]]) < F32_TOL
