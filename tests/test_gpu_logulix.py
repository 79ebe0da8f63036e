"""Logulix through the serving path (ServingEngine -> SequenceEngine -> tha_hyb_step) against the plain float64 statement of the
design in tests/logulix_oracle.py.

Every test builds its own small configuration with random weights.  float32 runs are compared tightly (they differ from float64 by
rounding only), bfloat16 runs loosely.  Where random weights would hide a fault (one far key among hundreds, a key just inside or
just outside the window, a memory that fades over hundreds of tokens) the weights are made sharp, so that one key carries the result
and seeing it or not moves the output by tens of percent.
"""
import copy
import ctypes as C
import json
import os
import subprocess

import numpy as np
import pytest

import logulix_oracle as O
from pkgload import load_pkg

pytestmark = pytest.mark.gpu

F32_TOL, BF16_TOL = 1e-4, 6e-2


def rel_err(got, want):
    got, want = np.asarray(got, np.float64), np.asarray(want, np.float64)
    return float(np.sqrt(((got - want) ** 2).mean()) / (np.sqrt((want ** 2).mean()) + 1e-12))


# ---- configurations ---------------------------------------------------------------------------------------------------
def dense(ff=56):
    return {"kind": "dense", "ff": ff}


def attention(mlp=None, heads=4, kv_heads=2, dim=16, conv=3, window=20, rot=(8, 1000.0, 3.0), scale=0.4, softcap=5.0):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "conv": conv, "mask": {"size": window}, "scale": scale, "softcap": softcap}
    if rot:
        m["rot"] = {"dims": rot[0], "base": rot[1]}
        if rot[2]:
            m["rot"]["scaling"] = {"factor": rot[2]}
    return {"type": "attention", "mixer": m, "mlp": mlp}


def wkv(mlp=None, heads=3, dim=10):
    return {"type": "wkv", "mixer": {"heads": heads, "dim": dim}, "mlp": mlp}


def retention(mlp=None, heads=3, dim=12, vdim=10, rot=(8, 500.0), decay=None):
    m = {"heads": heads, "dim": dim, "vdim": vdim, "decay": list(decay) if decay else [1.0 - 2.0 ** -(2 + 1.7 * i) for i in range(heads)]}
    if rot:
        m["rot"] = {"dims": rot[0], "base": rot[1]}
    return {"type": "retention", "mixer": m, "mlp": mlp}


def model(layers, width=64, vocab=130, loop=None, eps=1e-5, embed=1.7, logit=0.6):
    c = {"architecture": "Logulix", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width, "embedding": {"scale": embed},
         "logit_scale": logit}
    if loop:
        c["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return c


class Built:
    """A model folder, its oracle view, and engines on demand."""

    def __init__(self, tmp, cfg, seed=0, tweak=None, rank=6):
        self.serving = load_pkg("serving")
        self.cfg = cfg
        self.w = O.random_weights(cfg, seed, rank)
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
    # every mixer with and without a feed-forward, sizes that differ between the layers, a segment of three layers that runs three
    # times (its attention, both memories and every tail once per pass), windows shorter than the prompts
    layers = [wkv(dense(), heads=2, dim=20), attention(None, heads=6, kv_heads=3, dim=8, conv=4, window=33, rot=(4, 50.0, 2.0)),
              retention(dense(40), heads=2, dim=16, vdim=24), wkv(None), attention(dense(), window=20), retention(None, rot=(12, 900.0))]
    return Built(tmp_path_factory.mktemp("general"), model(layers, loop=(1, 4, 3)), seed=1)


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


# ---- whole prompts, every layer run -------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype,tol", [("float32", F32_TOL), ("bfloat16", BF16_TOL)])
@pytest.mark.parametrize("n", [1, 2, 97])
def test_whole_prompt_every_layer_run(general, dtype, tol, n):
    toks = tokens_for(general, n, 3)
    z, layers = general.ref(toks)
    assert len(layers) == 12
    logits, taps = general.engine(dtype).step([("a", toks, list(range(n)))], taps=True)
    assert taps.shape == layers.shape
    for i in range(len(layers)):
        assert rel_err(taps[i], layers[i]) < tol, f"residual stream after run {i}"
    assert rel_err(logits, z) < tol


# ---- each mechanism alone -----------------------------------------------------------------------------------------------
def one_layer(tmp, layer, width=48, seed=2, tweak=None, **kw):
    return Built(tmp, model([layer], width=width, vocab=90, **kw), seed, tweak)


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


@pytest.mark.parametrize("rot", [(8, 1000.0, 3.0), (16, 40.0, None), None, (2, 5.0, 0.5)])
def test_attention_alone(tmp_path, rot):
    b = one_layer(tmp_path, attention(rot=rot, window=9))
    check_all_positions(b)
    check_all_positions(b, cuts=[3, 1, 20, 2])
    check_all_positions(b, n=3)                                  # the first tokens: the convolutions read zeros before the start
    check_all_positions(b, dtype="bfloat16", tol=BF16_TOL)
    for t in ("l0__mix__q__b", "l0__mix__k__b", "l0__mix__o__b"):
        assert matters(b, **{t: np.zeros_like}) > 1e-3, t
    for t in ("l0__mix__q__norm", "l0__mix__k__norm"):
        assert matters(b, **{t: np.ones_like}) > 1e-3, t


def test_linear_stretch_of_the_rotation(tmp_path):
    b = one_layer(tmp_path, attention(heads=2, kv_heads=1, rot=(16, 50.0, 8.0), window=300, scale=1.5, softcap=30.0))
    cfg = copy.deepcopy(b.cfg)
    del cfg["layers"][0]["mixer"]["rot"]["scaling"]
    assert matters(b, n=200, cfg=cfg) > 1e-2
    check_all_positions(b, n=200, cuts=[150, 1])


@pytest.mark.parametrize("softcap,scale", [(0.5, 1.0), (3.0, 4.0), (60.0, 4.0)])
def test_score_cap(tmp_path, softcap, scale):
    b = one_layer(tmp_path, attention(scale=scale, softcap=softcap, window=50))
    cfg = copy.deepcopy(b.cfg)
    cfg["layers"][0]["mixer"]["softcap"] = 1e6
    assert matters(b, cfg=cfg) > 1e-3
    check_all_positions(b)
    check_all_positions(b, dtype="bfloat16", tol=BF16_TOL, cuts=[40, 1])


def test_convolution_behind_biased_projections(tmp_path):
    """taps far from the identity and large biases (the tail holds biased rows, the rows before the start are zeros without a bias);
    portions shorter than the taps"""
    def tweak(w):
        for n in ("q", "k"):
            w["l0.mix.%s.conv" % n][...] *= 2.0
            w["l0.mix.%s.b" % n][...] *= 5.0
    for taps in (1, 2, 5, 9):
        b = one_layer(tmp_path / str(taps), attention(conv=taps, window=12), tweak=tweak)
        check_all_positions(b, n=40)
        check_all_positions(b, n=40, cuts=[1, 2, 1, 1, 3, 2, 7, 1])
        check_all_positions(b, n=40, cuts=[2])
        if taps > 1:
            def last_only(a):
                a[:, :-1] = 0.0
                return a
            assert matters(b, n=40, l0__mix__k__conv=last_only) > 1e-2


def test_row_norm_takes_one_mean_over_all_heads(tmp_path):
    """heads of very different size: a norm per head would make them equal"""
    def tweak(w):
        w["l0.mix.q"][:16] *= 8.0
        w["l0.mix.k"][:16] *= 8.0
    b = one_layer(tmp_path, attention(), tweak=tweak)
    check_all_positions(b)
    check_all_positions(b, dtype="bfloat16", tol=BF16_TOL)


def test_key_value_memory_alone(tmp_path):
    b = one_layer(tmp_path, wkv())
    check_all_positions(b)
    check_all_positions(b, cuts=[3, 1, 20, 2])
    check_all_positions(b, n=1)
    check_all_positions(b, n=2, cuts=[1])
    check_all_positions(b, dtype="bfloat16", tol=BF16_TOL, cuts=[33, 2, 1])
    assert matters(b, l0__mix__u=np.zeros_like) > 1e-2           # the current token's bonus
    for c in "rkvgw":                                            # every mix with the previous token
        assert matters(b, **{"l0__mix__mu__" + c: np.zeros_like}) > 1e-3, c


def test_key_value_memory_decay_extremes(tmp_path):
    """decays next to one (nothing is forgotten for hundreds of tokens) and next to zero, and a strong input-dependent part"""
    for i, (w0, gain) in enumerate(((-9.0, 1.0), (3.0, 1.0), (-2.0, 6.0))):
        def tweak(w):
            w["l0.mix.w0"][...] = w0
            w["l0.mix.w2"][...] *= gain
        b = one_layer(tmp_path / str(i), wkv(heads=2, dim=16), tweak=tweak)
        check_all_positions(b, n=300, cuts=[170, 50, 1, 40])


@pytest.mark.parametrize("rot", [(8, 500.0), (12, 20.0), None])
def test_retention_alone(tmp_path, rot):
    b = one_layer(tmp_path, retention(rot=rot))
    check_all_positions(b)
    check_all_positions(b, cuts=[3, 1, 20, 2])
    check_all_positions(b, n=1)
    check_all_positions(b, dtype="bfloat16", tol=BF16_TOL, cuts=[33, 2, 1])


@pytest.mark.parametrize("dim,vdim", [(16, 16), (64, 128), (40, 24), (128, 32), (9, 7)])
def test_retention_long_prompts_and_portions(tmp_path, dim, vdim):
    """portions of every length from one token to several hundred, decays from forgetful to nearly none"""
    b = one_layer(tmp_path, retention(heads=4, dim=dim, vdim=vdim, rot=(dim // 2 * 2, 1e4), decay=(0.3, 0.93, 0.998, 1.0)))
    for cuts in ([400], [63, 1, 64, 2, 65, 31, 33, 128, 1], [2], [127, 129, 140]):
        check_all_positions(b, n=400, cuts=cuts)
    check_all_positions(b, n=400, cuts=[300, 1], dtype="bfloat16", tol=BF16_TOL)


@pytest.mark.parametrize("dim", [24, 64, 128])
def test_long_and_short_portions_in_one_batch(tmp_path, dim):
    """long portions run as segments side by side, short ones and single tokens in the same step do not: every sequence continues from
    its own state, before and after"""
    b = Built(tmp_path, model([wkv(heads=2, dim=dim), retention(heads=2, dim=dim, vdim=dim + 8, rot=None, decay=(0.9, 0.999))], width=48, vocab=90), 8)
    lens = {"a": (5, 390, 1, 200), "b": (1, 64, 1, 1), "c": (40, 260, 3, 1), "d": (2, 1, 300, 2)}
    toks = {k: tokens_for(b, sum(v), 70 + i) for i, (k, v) in enumerate(lens.items())}
    e, got, at = b.engine(max_tokens=2048), {k: [] for k in lens}, dict.fromkeys(lens, 0)
    for i in range(4):
        out, o = e.step([(k, toks[k][at[k]:at[k] + v[i]], list(range(v[i]))) for k, v in lens.items()]), 0
        for k, v in lens.items():
            got[k].append(out[o:o + v[i]])
            o += v[i]
            at[k] += v[i]
    for k in lens:
        assert rel_err(np.concatenate(got[k]), b.ref(toks[k])[0]) < F32_TOL, k


@pytest.mark.parametrize("loop", [(0, 1, 2), (0, 3, 2), (1, 3, 4), (2, 3, 1), (1, 2, 3)])
def test_looped_segment(tmp_path, loop):
    """at the start, at the end, over everything, one layer, one pass; the map that joins x with the embedding output runs once a pass"""
    b = Built(tmp_path, model([attention(conv=3, window=7), wkv(dense()), retention()], width=40, vocab=90, loop=loop), 6)
    check_all_positions(b)
    check_all_positions(b, cuts=[5, 2, 1, 30, 1])

    def no_embedding(a):
        a[:, a.shape[1] // 2:] = 0.0
        return a
    assert matters(b, loop__in=no_embedding) > 1e-2


def test_constants_of_the_embedding_and_the_logits(tmp_path):
    for embed, logit in ((0.25, 3.0), (30.0, 0.1), (1.0, 1.0)):
        b = Built(tmp_path / str(embed), model([retention(dense())], width=24, vocab=50, embed=embed, logit=logit), 4)
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


def test_a_reused_slot_starts_from_zero_state_and_reused_blocks_hold_nothing(general):
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


# ---- sharp weights: far keys, page borders, the edges of the window, fading memories ---------------------------------------
HALF = 32


def sharp_attention(tmp, dim=16, window=40, vocab=1024):
    """Queries read the upper half of the layer's input, keys the lower half through the same matrix, with a large score scale.  The upper
    half of the QUERY probe's embedding is the lower half of the KEY probe's: the query probe puts nearly all its weight on the key
    probe wherever it sees it, a different token with a different value.  The convolutions pass their input through."""
    cfg = model([attention(heads=2, kv_heads=1, dim=dim, window=window, rot=(4, 100.0, 2.0), scale=2.0 if dim < 64 else 1.0, softcap=90.0)],
                width=2 * HALF, vocab=vocab)
    p = "l0.mix."

    def tweak(w):
        w["embed"][vocab - 2, HALF:] = w["embed"][vocab - 1, :HALF]
        w["l0.norm1"][HALF:] = w["l0.norm1"][:HALF]
        for n in ("q", "k"):
            w[p + n + ".conv"][...] = 0.0
            w[p + n + ".conv"][:, -1] = 1.0
            w[p + n + ".b"][...] = 0.0
            w[p + n + ".norm"][...] = 1.0
        w[p + "k"][:, HALF:] = 0.0
        w[p + "k"][:4] *= 0.05                                    # the rotated channels carry little
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


def check_probe(b, n, key_pos, query_pos, seen, cut_sets, dtype="float32"):
    """the engine agrees with the statement at the query probe, which does (seen) or does not depend on the key probe"""
    toks, other = with_probes(b, n, key_pos, query_pos, key_pos * 7 + query_pos)
    z, _ = b.ref(toks)
    moved = rel_err(b.ref(other)[0][query_pos], z[query_pos])
    assert moved > 0.1 if seen else moved < 1e-9, moved
    tol = F32_TOL if dtype == "float32" else BF16_TOL
    for cuts in cut_sets:
        got = feed(b.engine(dtype), "a", toks, [c for c in cuts if c > 0] or [1])
        assert rel_err(got[query_pos], z[query_pos]) < (10 if dtype == "float32" else 1) * tol, cuts
        if dtype == "float32":
            assert rel_err(got, z) < tol, cuts


@pytest.mark.parametrize("query_pos", [41, 64, 95, 130])
@pytest.mark.parametrize("window", [32, 40])
def test_keys_just_inside_and_just_outside_the_window(tmp_path, query_pos, window):
    """the key at distance window - 1 is the last one seen, the key at distance `window` the first one lost -- in whole prompts, in
    portions that start at the key, the query or in between, and with the query decoded alone"""
    b = sharp_attention(tmp_path, window=window)
    for dist, seen in ((window - 1, True), (window, False), (1, True)):
        key_pos = query_pos - dist
        check_probe(b, 140, key_pos, query_pos, seen, ([140], [query_pos, 1], [key_pos, 2, 1], [key_pos + 1, 17, 2], [33, 2]))


def test_window_edges_bfloat16(tmp_path):
    b = sharp_attention(tmp_path, window=40)
    check_probe(b, 140, 94, 133, True, ([140], [133, 1]), "bfloat16")
    check_probe(b, 140, 93, 133, False, ([140], [133, 1]), "bfloat16")


@pytest.mark.parametrize("key_pos,query_pos", [(0, 1), (0, 149), (15, 16), (16, 17), (63, 64), (64, 65), (63, 127), (64, 128), (127, 128), (1, 63)])
def test_keys_at_the_borders_of_the_block_table(tmp_path, key_pos, query_pos):
    b = sharp_attention(tmp_path, dim=64, window=900)
    check_probe(b, 150, key_pos, query_pos, True, ([150], [query_pos, 1], [key_pos, 2, 1], [key_pos + 1, 1]))


@pytest.mark.parametrize("dtype,decoded", [("float32", False), ("float32", True), ("bfloat16", False), ("bfloat16", True)])
def test_one_far_key_among_hundreds(tmp_path, dtype, decoded):
    b = sharp_attention(tmp_path, dim=64, window=900)
    check_probe(b, 700, 3, 690, True, ([670, 1] if decoded else [300, 400],), dtype)


def sharp_memory(tmp, kind, vocab=1024):
    """One memory whose keys read the lower half of the input and whose queries read the upper half; every token but the key probe has a
    small lower half, so that the key probe's write stands out among hundreds of others; slow decays."""
    layer = retention(heads=2, dim=32, vdim=24, rot=None, decay=(0.999, 0.9965)) if kind == "retention" else wkv(heads=2, dim=32)
    p, qn = "l0.mix.", "q" if kind == "retention" else "r"

    def tweak(w):
        w["embed"][:vocab - 1, :HALF] *= 0.03
        w["embed"][vocab - 2, HALF:] = w["embed"][vocab - 1, :HALF]
        w["l0.norm1"][HALF:] = w["l0.norm1"][:HALF]
        w[p + "k"][:, HALF:] = 0.0
        w[p + qn][:, :HALF] = 0.0
        w[p + qn][:, HALF:] = w[p + "k"][:, :HALF]
        if kind == "wkv":
            w[p + "w0"][...] = -7.0
            w[p + "w2"][...] *= 0.3
            for c in "rk":
                w[p + "mu." + c][...] = 0.0
    return Built(tmp, model([layer], width=2 * HALF, vocab=vocab), 15, tweak)


@pytest.mark.parametrize("kind", ["retention", "wkv"])
@pytest.mark.parametrize("key_pos,query_pos", [(0, 500), (3, 690), (63, 64), (64, 128), (31, 257), (255, 600)])
def test_one_far_write_in_a_fading_memory(tmp_path, kind, key_pos, query_pos):
    b = sharp_memory(tmp_path, kind)
    check_probe(b, 700, key_pos, query_pos, True, ([700], [query_pos, 1], [key_pos, 2, 200, 1], [key_pos + 1, 64]))


@pytest.mark.parametrize("kind", ["retention", "wkv"])
def test_one_far_write_bfloat16(tmp_path, kind):
    check_probe(sharp_memory(tmp_path, kind), 700, 3, 690, True, ([700], [690, 1]), "bfloat16")


def test_few_rows_at_a_long_context_with_value_rows_that_are_no_multiple_of_a_warp(tmp_path):
    """steps of one or two rows behind hundreds of positions are cut along the keys and merged"""
    b = Built(tmp_path, model([attention(dense(), heads=6, kv_heads=2, dim=40, window=700), attention(None, heads=4, kv_heads=2, dim=72, window=900)],
                              width=64, vocab=120), 7)
    toks = tokens_for(b, 720, 4)
    z, _ = b.ref(toks)
    for dtype, tol in (("float32", F32_TOL), ("bfloat16", BF16_TOL)):
        got = feed(b.engine(dtype), "a", toks, [600, 38, 2, 1, 1, 2, 3, 1])
        assert max(rel_err(g, w) for g, w in zip(got[600:], z[600:])) < 3 * tol
        assert rel_err(got, z) < tol


@pytest.mark.parametrize("cuts", [[300], [150, 86, 2, 1], [64, 1]])
def test_tensor_core_attention_bfloat16_every_position(tmp_path, cuts):
    """heads that take the tensor-core form, capped peaked scores, and a check of EVERY position by itself"""
    b = Built(tmp_path, model([attention(heads=6, kv_heads=2, dim=48, rot=(24, 1e4, 4.0), scale=0.6, softcap=8.0, window=70)], width=64, vocab=200), 41)
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


# ---- other sizes: values that are often equal, or 1 ------------------------------------------------------------------
@pytest.mark.parametrize("case", ["single", "wide_heads", "everything_small", "odd_sizes", "many_kv_heads", "window_one", "window_beyond",
                                  "no_attention", "attention_only", "wide_memories", "aligned"])
def test_other_sizes(tmp_path, case):
    width, n, rank, loop = 32, 75, 6, None
    if case == "single":
        layers = [attention(dense(8), heads=1, kv_heads=1, dim=8, rot=(2, 9.0, 2.0), conv=1, window=9), wkv(dense(16), heads=1, dim=24),
                  retention(heads=1, dim=8, vdim=40, rot=(2, 10.0), decay=(0.9,))]
        width, rank, loop = 24, 1, (0, 3, 2)
    elif case == "wide_heads":
        layers = [attention(dense(40), heads=2, kv_heads=2, dim=150, rot=(72, 1e3, 3.0), window=30, conv=2),
                  wkv(heads=1, dim=72), retention(dense(), heads=1, dim=72, vdim=140, rot=(72, 1e3))]
        width = 40
    elif case == "everything_small":
        layers = [attention(dense(1), heads=1, kv_heads=1, dim=2, rot=(2, 3.0, 2.0), window=2, conv=2), wkv(dense(1), heads=1, dim=1),
                  retention(heads=1, dim=2, vdim=1, rot=(2, 3.0), decay=(0.5,)), wkv(heads=1, dim=2)]
        width, rank = 8, 1
    elif case == "odd_sizes":
        layers = [attention(dense(11), heads=6, kv_heads=3, dim=7, rot=(2, 30.0, 5.0), window=13, conv=5), wkv(dense(9), heads=3, dim=11),
                  retention(heads=5, dim=9, vdim=7, rot=(6, 40.0))]
        width, rank, loop = 27, 7, (1, 3, 3)
    elif case == "many_kv_heads":
        layers = [attention(heads=3, kv_heads=3), attention(dense(), heads=6, kv_heads=2, dim=8), attention(heads=8, kv_heads=1)]
    elif case == "window_one":
        layers = [attention(dense(), window=1), retention()]
    elif case == "window_beyond":
        layers = [attention(dense(), window=500), wkv()]
    elif case == "no_attention":
        layers = [wkv(), retention(dense())]
        loop = (0, 2, 2)
    elif case == "attention_only":
        layers = [attention(conv=4), attention(dense())]
        loop = (0, 1, 3)
    elif case == "wide_memories":                             # more key channels than a warp's lanes, in every register form
        layers = [wkv(heads=1, dim=130), retention(heads=1, dim=300, vdim=18, rot=(300, 1e3), decay=(0.95,)), wkv(heads=1, dim=260),
                  retention(heads=2, dim=130, vdim=6, rot=None, decay=(0.7, 0.99))]
        rank = 40
    else:                                                     # every product on the tensor cores, groups that are no multiple of a tile
        layers = [wkv(dense(96), heads=3, dim=24), attention(heads=4, kv_heads=1, dim=32), retention(dense(128), heads=2, dim=64, vdim=96, rot=(64, 1e4)),
                  wkv(heads=5, dim=32)]
        width, rank, loop, n = 96, 24, (1, 3, 2), 150
    b = Built(tmp_path, model(layers, width=width, vocab=61, loop=loop), 5, rank=rank)
    toks = tokens_for(b, n, 2)
    z, layers_ref = b.ref(toks)
    logits, taps = b.engine().step([("a", toks, list(range(n)))], taps=True)
    for i in range(len(layers_ref)):
        assert rel_err(taps[i], layers_ref[i]) < F32_TOL, f"run {i}"
    assert rel_err(logits, z) < F32_TOL
    assert rel_err(feed(b.engine(), "a", toks, [9, 2, 1]), z) < F32_TOL
    assert rel_err(feed(b.engine("bfloat16"), "a", toks, [40, 1]), z) < 2 * BF16_TOL


# ---- the grouped product by itself --------------------------------------------------------------------------------------
@pytest.mark.parametrize("M", [1, 7, 64, 200, 700])
@pytest.mark.parametrize("groups,K", [((96, 96, 96, 96, 24), 64), ((256, 256, 128, 40, 8), 320), ((5, 3), 72), ((130,) * 8, 128), ((7, 9), 30)])
def test_grouped_product_equals_one_product_per_group(M, groups, K):
    import torch
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    lib = C.CDLL(os.path.join(root, "hip_llama.cpp_b200", "lib", "libtha_b200.so"))
    g = torch.Generator(device="cpu").manual_seed(M * 1000 + K)
    N = sum(groups)
    gn = (C.c_int * len(groups))(*groups)
    for dt, tt, tol in ((0, torch.bfloat16, 2e-6), (1, torch.float32, 2e-6)):
        A = torch.randn(len(groups), M, K, generator=g).to(tt)
        W = torch.randn(N, K, generator=g).to(tt)
        out = torch.full((M, N + 3), 7.0, device="cuda")
        Ad, Wd = A.cuda(), W.cuda()
        st = lib.tha_hyb_linear_groups(None, dt, C.c_void_p(out.data_ptr()), C.c_longlong(N + 3), C.c_void_p(Ad.data_ptr()), C.c_void_p(Wd.data_ptr()), M, K,
                                       len(groups), gn)
        torch.cuda.synchronize()
        assert st == 0
        want = torch.cat([A[i].double() @ w.double().T for i, w in enumerate(torch.split(W, list(groups)))], 1)
        got = out.cpu().double()
        assert float((got[:, :N] - want).abs().max()) <= tol * float(want.abs().max()) * K ** 0.5
        assert bool((got[:, N:] == 7.0).all())


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
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    app = os.path.join(root, "build", "apps", "llama")
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
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    exe = os.path.join(root, "build", "apps", "trace_run")
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
