"""Fidatar on the layered runtime against the plain restatement in tests/fidatar_oracle.py: every mechanism alone, prefill against
token-by-token decoding, portions of several sizes, interleaved requests, pages and slots used again, keys far away, at page borders
and on both sides of a block's edge, the one in the softmax denominator, the rescaled rotation, norms per head, biases, gates at their
extremes, writes to the memory that last or fade, the denominator of its read-out, groups of experts, norms of the sums, the first
tokens of a sequence, long decoding, sizes that defeat every vector width, values that happen to be equal or 1, and greedy generation
through the engine's own entry points.  Small random models, each written to a temporary folder and loaded like any model folder."""
import copy
import json
import os
import subprocess
import sys

import numpy as np
import pytest

from nano_b200 import engine as E, modeldir as md

import fidatar_oracle as O

pytestmark = pytest.mark.gpu

YARN = {"factor": 6.0, "original": 60, "fast": 8.0, "slow": 0.5}
ATT = {"heads": 6, "kv_heads": 2, "dim": 20, "vdim": 12, "scale": 0.3, "mask": {"size": 41}, "rot": {"dims": 12, "base": 300.0, "scaling": YARN}}
MEM = {"heads": 3, "dim": 20, "vdim": 28, "gate_cap": 9.0}
MOE = {"kind": "moe", "router": {"experts": 12, "top": 3, "groups": {"count": 4, "keep": 2}, "scale": 1.7}, "expert": {"ff": 24}}


def att(**kw):
    m = copy.deepcopy(ATT)
    m.update(kw)
    return {k: v for k, v in m.items() if v is not None}


def mem(**kw):
    return dict(MEM, **kw)


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts=12, top=3, count=4, keep=2, scale=1.7, ff=24):
    return {"kind": "moe", "router": {"experts": experts, "top": top, "groups": {"count": count, "keep": keep}, "scale": scale}, "expert": {"ff": ff}}


def build(tmp_path, cfg, seed=0, f32=True, max_tokens=512, keep=False, chunk=None, name="m", tweak=None):
    w = md.fidatar_random(cfg, seed)
    if tweak:
        tweak(w)
        w = {k: md.bf16_round(v) for k, v in w.items()}          # the file holds bfloat16: the oracle reads the same numbers
    path = md.write_model_dir(str(tmp_path / name), cfg, w)
    os.environ.pop("NB200_KEEP_RESIDUALS", None); os.environ.pop("NB200_CHUNK", None)
    if keep: os.environ["NB200_KEEP_RESIDUALS"] = "1"
    if chunk: os.environ["NB200_CHUNK"] = str(chunk)
    try:
        eng = E.Engine(path, max_tokens, flags=E.FLAG_F32 if f32 else 0)
    finally:
        os.environ.pop("NB200_KEEP_RESIDUALS", None); os.environ.pop("NB200_CHUNK", None)
    return eng, w


def toks(cfg, n, seed=1):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], size=n).astype(np.uint32)


def rows(got, want):
    """rms of the difference over the rms of the reference, per row (mean taken off: logits are shift-invariant)"""
    d = got - want
    d = d - d.mean(-1, keepdims=True)
    return np.sqrt((d ** 2).mean(-1)) / np.sqrt((want ** 2).mean(-1) + 1e-30)


def rel(got, want):
    return float(rows(got, want).max())


F32_TOL, BF16_TOL = 3e-5, 5e-2


def close_bf16(got, want):
    """bfloat16 products: nearly every row stays within the tolerance, the typical row far within it, and no row is far off (tiny random
    models amplify a rounding here and there)"""
    r = rows(got, want)
    return np.median(r) < BF16_TOL / 2 and np.mean(r > BF16_TOL) <= 0.06 and r.max() < 5 * BF16_TOL


def no_close_calls(cfg):
    """every routed feed-forward with all of its experts chosen: random routers make close calls, which bfloat16 may turn the other way"""
    cfg = copy.deepcopy(cfg)
    for L in cfg["layers"]:
        if L["mlp"] and L["mlp"]["kind"] == "moe":
            r = L["mlp"]["router"]
            r["top"], r["scale"] = r["experts"], r["scale"] * r["top"] / r["experts"]
            r["groups"]["keep"] = r["groups"]["count"]
    return cfg


def whole(eng, t, want=None):
    s = eng.seq_open()
    out = eng.step(s, t, range(len(t)) if want is None else want)
    eng.seq_close(s)
    return out


def in_cuts(eng, t, cuts):
    s = eng.seq_open()
    out, at = [], 0
    for c in cuts:
        part = t[at:at + c]
        if len(part):
            out.append(eng.step(s, part, range(len(part))))
        at += c
    eng.seq_close(s)
    assert at >= len(t)
    return np.concatenate(out)


def check_alone(tmp_path, cfg, n=75, tweak=None):
    eng, w = build(tmp_path, cfg, keep=True, tweak=tweak)
    t = toks(cfg, n)
    trace = []
    ref = O.forward(cfg, w, t, trace)
    got = whole(eng, t)
    res = eng.read_residual(0, len(t))
    assert np.abs(res - trace[0]).max() <= 3e-5 * np.abs(trace[0]).max()
    assert rel(got, ref) < F32_TOL
    for cuts in ([1] * n, [2, 3, 4] * (n // 9 + 1), [5, 1, 30, 2, 7, n], [6, 9, 11, 5, 13, n]):
        assert rel(in_cuts(eng, t, cuts), ref) < F32_TOL, cuts[:3]
    eng.close()


MIXERS = [
    ("attention", att()),
    ("attention", att(mask=None, rot=None)),                                                    # every earlier key, no positions
    ("attention", att(rot={"dims": 12, "base": 300.0})),                                        # frequencies as they are
    ("attention", att(heads=1, kv_heads=1, dim=2, vdim=1, mask={"size": 1}, rot={"dims": 2, "base": 5.0})),      # a token sees itself alone
    ("attention", att(heads=4, kv_heads=4, dim=16, vdim=16, mask={"size": 16}, rot={"dims": 16, "base": 1e4, "scaling": YARN})),      # one head per key/value head; sizes all equal
    ("attention", att(heads=11, kv_heads=1, dim=7, vdim=5, mask={"size": 2}, rot={"dims": 2, "base": 9.0})),     # more heads per key/value head than a block takes
    ("attention", att(heads=6, kv_heads=3, dim=64, vdim=128, mask={"size": 32}, rot={"dims": 32, "base": 1e6, "scaling": dict(YARN, original=4096)})),
    ("attention", att(heads=2, kv_heads=1, dim=100, vdim=68, mask={"size": 33}, rot={"dims": 100, "base": 50.0})),
    ("attention", att(heads=2, kv_heads=2, dim=256, vdim=256, scale=0.06, mask={"size": 500}, rot={"dims": 64, "base": 100.0, "scaling": dict(YARN, factor=1.0)})),
    ("mlstm", MEM),
    ("mlstm", mem(heads=1, dim=1, vdim=1)),
    ("mlstm", mem(heads=4, dim=16, vdim=16, gate_cap=1.0)),                                     # sizes all equal
    ("mlstm", mem(heads=2, dim=33, vdim=7)),                                                    # sizes no vector width divides
    ("mlstm", mem(heads=5, dim=64, vdim=64)),
    ("mlstm", mem(heads=2, dim=128, vdim=72)),
    ("mlstm", mem(heads=2, dim=130, vdim=150)),
    ("mlstm", mem(heads=1, dim=256, vdim=33)),
    ("mlstm", mem(heads=1, dim=300, vdim=600)),                                                 # the widest register tile; more value columns than the cluster's threads take at once
    ("mlstm", mem(heads=36, dim=8, vdim=132, gate_cap=30.0)),
]


# ---- each mechanism alone: one layer, no feed-forward, residual after the layer and logits; whole, token by token, portions ----
@pytest.mark.parametrize("kind,mixer", MIXERS)
def test_mixer_alone(tmp_path, kind, mixer):
    check_alone(tmp_path, md.fidatar_config(61, 72, [(kind, mixer, None)]))


@pytest.mark.parametrize("mlp", [dense(56), dense(7), dense(129), dense(1), MOE, moe(1, 1, 1, 1), moe(5, 5, 1, 1, 1.0, 9), moe(6, 2, 6, 3), moe(8, 4, 2, 1, 0.5), moe(16, 2, 4, 4, 3.0, 1), moe(96, 6, 8, 3, 2.5, 12),
                                 moe(66, 1, 33, 2, 1.0, 8)])
def test_feed_forward(tmp_path, mlp):
    """dense widths; experts: one, all of them, one per group, one group kept, every group kept, more than a warp's lanes and groups too"""
    check_alone(tmp_path, md.fidatar_config(50, 40, [("mlstm", mem(heads=2), mlp)]), n=40)


@pytest.mark.parametrize("width,vocab", [(50, 61), (37, 33), (130, 7), (1100, 20)])
def test_ragged_widths(tmp_path, width, vocab):
    """widths and vocabularies that no vector width divides, through every product of a layer"""
    cfg = md.fidatar_config(vocab, width, [("attention", att(), dense(30)), ("mlstm", MEM, None), ("mlstm", mem(dim=10), MOE), ("attention", att(mask={"size": 9}), moe(6, 2, 3, 2))])
    eng, w = build(tmp_path, cfg)
    t = toks(cfg, 45)
    ref = O.forward(cfg, w, t)
    assert rel(whole(eng, t), ref) < F32_TOL
    assert rel(in_cuts(eng, t, [3, 1, 2, 4, 35]), ref) < F32_TOL
    eng.close()
    cfg = no_close_calls(dict(cfg, layers=cfg["layers"][2:]))          # two layers: deeper models of this size amplify roundings
    eng, w = build(tmp_path, cfg, f32=False, name="b")
    ref = O.forward(cfg, w, t)
    assert close_bf16(whole(eng, t), ref) and close_bf16(in_cuts(eng, t, [40, 1, 1, 3]), ref)
    eng.close()


@pytest.mark.parametrize("width", [2051, 4100, 8400])
def test_wide_residual(tmp_path, width):
    """residuals wider than the registers of the norm's block hold, with and without 16-byte rows"""
    check_alone(tmp_path, md.fidatar_config(16, width, [("mlstm", mem(heads=1, dim=8, vdim=8), dense(16))]), n=9)


def mixed_cfg(vocab=67):
    layers = [("attention", att(), dense(40)), ("mlstm", MEM, MOE), ("attention", att(heads=3, kv_heads=3, dim=8, mask={"size": 64}, rot={"dims": 4, "base": 40.0}), None),
              ("mlstm", mem(heads=2, dim=36, gate_cap=14.0), dense(24)), ("attention", att(mask={"size": 30}), moe(8, 2, 4, 3))]
    return md.fidatar_config(vocab, 56, layers, alpha=2.5)          # a calm residual: five layers of this size amplify a rounding some fifty times at 1.5


@pytest.mark.parametrize("order", ["m", "a", "am", "mam", "aamm", "AmMa", "MAXY"])
def test_layer_order(tmp_path, order):
    """the residual after every layer; capitals carry a dense feed-forward, X and Y experts"""
    kinds = {"a": ("attention", ATT), "m": ("mlstm", MEM), "x": ("attention", ATT), "y": ("mlstm", MEM)}
    layers = [(*kinds[c.lower()], (MOE if c in "XY" else dense(33)) if c.isupper() else None) for c in order]
    cfg = md.fidatar_config(40, 48, layers)
    eng, w = build(tmp_path, cfg, keep=True)
    t = toks(cfg, 50)
    trace = []
    ref = O.forward(cfg, w, t, trace)
    assert rel(whole(eng, t), ref) < F32_TOL
    for i, x in enumerate(trace):
        assert np.abs(eng.read_residual(i, len(t)) - x).max() <= 3e-5 * np.abs(x).max(), i
    assert rel(in_cuts(eng, t, [20] + [1] * 30), ref) < F32_TOL
    eng.close()


# ---- prefill against token-by-token decoding, portions down to two tokens, the engine's own chunking ----
@pytest.mark.parametrize("f32", [True, False])
def test_portions_and_decoding(tmp_path, f32):
    cfg = mixed_cfg() if f32 else no_close_calls(mixed_cfg())
    eng, w = build(tmp_path, cfg, f32=f32)
    t = toks(cfg, 150)
    ref = O.forward(cfg, w, t)
    ok = (lambda g, r: rel(g, r) < F32_TOL) if f32 else close_bf16
    full = whole(eng, t)
    assert ok(full, ref)
    for cuts in ([1] * 150, [2] * 75, [3, 2, 64, 5, 1, 1, 33, 2, 39], [100] + [1] * 50, [31, 1, 32, 33, 53], [7] * 22, [5, 6, 7, 8, 9, 10, 11, 12, 82], [149, 1], [4] * 38, [63, 65, 22], [64, 64, 22]):
        got = in_cuts(eng, t, cuts)
        assert ok(got, ref), cuts[:4]
        assert ok(got, full), cuts[:4]
    eng.close()
    for chunk in (16, 5, 3):
        eng, _ = build(tmp_path, cfg, f32=f32, chunk=chunk, name="c%d" % chunk)       # chunks of the engine's own inside one step
        assert ok(whole(eng, t), ref)
        eng.close()


def test_batches_of_unequal_requests_and_reuse(tmp_path):
    """Requests interleaved step by step equal each alone; pages and slots that were freed hold other requests' numbers."""
    cfg = mixed_cfg()
    eng, w = build(tmp_path, cfg, max_tokens=400)
    ts = [toks(cfg, n, seed=10 + n) for n in (90, 33, 140, 5)]
    refs = [O.forward(cfg, w, t) for t in ts]
    free0 = eng.free_pages
    for rounds in range(2):                      # the second time through runs in pages and slots of the first
        seqs = [eng.seq_open() for _ in ts]
        outs, at = [[] for _ in ts], [0] * len(ts)
        sizes = [[40, 1, 1, 48], [2, 31], [64, 64, 3, 1, 1, 1, 6], [5]]
        step = 0
        while any(a < len(t) for a, t in zip(at, ts)):
            for i, t in enumerate(ts):
                if at[i] >= len(t) or step >= len(sizes[i]):
                    continue
                n = sizes[i][step]
                outs[i].append(eng.step(seqs[i], t[at[i]:at[i] + n], range(n)))
                at[i] += n
                if at[i] == len(t):
                    eng.seq_close(seqs[i])
            step += 1
        for o, r in zip(outs, refs):
            assert rel(np.concatenate(o), r) < F32_TOL
        assert eng.free_pages == free0
    eng.close()


# ---- attention: one key made to stand out, on both sides of a block's edge and at page borders ----
def stand_out(w, tok, H, G, D):
    """The last (unturned) coordinate of every head's key is large for token `tok` alone and the same coordinate of every query is constant,
    so a query's weight sits on token `tok` wherever it is in sight.  Channel 0 of the embedding tells the token apart."""
    w["embed"][:, 0] = -0.7; w["embed"][tok, 0] = 0.7
    p = "l0.mix."
    w[p + "k"][:] *= 0.3; w[p + "q"][:] *= 0.1; w[p + "k.b"][:] *= 0.1; w[p + "q.b"][:] *= 0.1
    for g in range(G):
        w[p + "k"][g * D + D - 1] = 0.0; w[p + "k"][g * D + D - 1, 0] = 1.0
    for h in range(H):
        w[p + "q"][h * D + D - 1] = 0.0; w[p + "q.b"][h * D + D - 1] = 2.0
    w[p + "q.norm"][:] = 1.0; w[p + "k.norm"][:] = 1.0


EDGES = [(64, 0), (64, 63), (64, 64), (64, 65), (64, 191), (100, 99), (100, 100), (100, 131), (100, 199), (33, 65), (33, 66), (300, 0), (300, 31), (300, 32), (300, 299), (None, 0), (None, 200), (7, 6), (7, 7)]


@pytest.mark.parametrize("size,where", EDGES)
def test_block_edges_show(tmp_path, size, where):
    """Token `where` draws the weight of every later query of its own block and of none after the block's end: a block that is one token
    off, or counted from a portion's start, changes the logits far beyond the tolerance."""
    a = att(heads=4, kv_heads=2, dim=16, vdim=16, scale=0.5, mask={"size": size} if size else None, rot={"dims": 4, "base": 100.0})
    cfg = md.fidatar_config(40, 48, [("attention", a, None)])
    n = 330
    t = toks(cfg, n, seed=3)
    t[t == 7] = 8
    t[where] = 7
    eng, w = build(tmp_path, cfg, max_tokens=400, tweak=lambda w: stand_out(w, 7, 4, 2, 16))
    ref = O.forward(cfg, w, t)
    t2 = t.copy(); t2[where] = 9
    change = rows(O.forward(cfg, w, t2), ref)
    last = min(n, (where // size + 1) * size) if size else n
    assert (change[where + 1:last] > 100 * F32_TOL).all() and (change[last:] == 0.0).all()
    if size and size > 1:                      # the oracle itself tells a block one token longer or shorter from the true one
        for other in (size - 1, size + 1):
            c2 = copy.deepcopy(cfg); c2["layers"][0]["mixer"]["mask"]["size"] = other
            assert rel(O.forward(c2, w, t), ref) > 100 * F32_TOL
    assert rel(whole(eng, t), ref) < F32_TOL
    assert rel(in_cuts(eng, t, [290] + [1] * 40), ref) < F32_TOL
    assert rel(in_cuts(eng, t, [max(1, where - 1)] + [1] * 60 + [n]), ref) < F32_TOL          # the block's edge (or the key) among single tokens
    assert rel(in_cuts(eng, t, [29, 2, 2, 31, 1, 1, 64, 130, 3, 4, 63]), ref) < F32_TOL
    if size:                                   # portions that end just before, at and just after the edge
        for first in (last - 1, last, last + 1):
            assert rel(in_cuts(eng, t, [first, 2, 3, n]), ref) < F32_TOL
    eng.close()


def test_decoding_over_many_blocks(tmp_path):
    """single tokens and short portions from the first token on, over the edges of blocks of several sizes at once"""
    cfg = md.fidatar_config(40, 48, [("attention", att(mask={"size": s}), None) for s in (3, 32, 47, 96, 5000)])
    eng, w = build(tmp_path, cfg, max_tokens=400)
    t = toks(cfg, 300, seed=3)
    ref = O.forward(cfg, w, t)
    for cuts in ([1] * 300, [2] * 150, [3, 4, 1, 2] * 30, [45, 4, 46, 1, 1, 4, 150, 3, 46]):
        assert rel(in_cuts(eng, t, cuts), ref) < F32_TOL, cuts[:4]
    eng.close()


def test_one_in_the_denominator_shows(tmp_path):
    """Scores far below zero leave nearly all of the weight to the one, which has no value; scores far above leave it none.  Through the key
    splits of a long decode too."""
    cfg = md.fidatar_config(40, 48, [("attention", att(heads=3, kv_heads=1, dim=16, vdim=16, scale=1.0, mask={"size": 150}, rot={"dims": 4, "base": 100.0}), None)])
    t = toks(cfg, 200, seed=9)
    size = {}
    for i, sign in enumerate((-1.0, 1.0, 0.02)):
        def tweak(w, sign=sign):               # one unturned coordinate of every query and key is large and constant: score = sign * constant
            for n, heads in (("q", 3), ("k", 1)):
                w["l0.mix." + n][:] *= 0.4; w["l0.mix." + n + ".b"][:] *= 0.4
                for h in range(heads):
                    w["l0.mix." + n][h * 16 + 15] = 0.0; w["l0.mix." + n + ".b"][h * 16 + 15] = 3.0 * (sign if n == "q" else 1.0)
                w["l0.mix." + n + ".norm"][:] = 1.0
        eng, w = build(tmp_path, cfg, tweak=tweak, name="s%d" % i)
        ref = O.forward(cfg, w, t)
        assert np.isfinite(ref).all()
        h = np.asarray(w["embed"], np.float64)[t] * cfg["embedding"]["scale"]
        y = O.attention(cfg["layers"][0]["mixer"], {k: np.asarray(v, np.float64) for k, v in w.items()}, "l0.mix.", h, 1e-5)
        size[sign] = np.abs(y).max()
        assert rel(whole(eng, t), ref) < F32_TOL
        assert rel(in_cuts(eng, t, [140] + [1] * 60), ref) < F32_TOL
        assert rel(in_cuts(eng, t, [2, 3] * 40), ref) < F32_TOL
        eng.close()
    assert size[-1.0] < 0.05 * size[1.0]


def test_rotation_norm_bias_and_scale_show(tmp_path):
    """The oracle tells each of the attention's parts from its absence on this model; the engine follows, far into a sequence."""
    sc = {"factor": 5.0, "original": 200, "fast": 6.0, "slow": 0.6}
    a = att(heads=4, kv_heads=2, dim=16, vdim=16, scale=0.9, mask={"size": 170}, rot={"dims": 12, "base": 50.0, "scaling": sc})
    cfg = md.fidatar_config(40, 48, [("attention", a, None)])
    eng, w = build(tmp_path, cfg)
    t = toks(cfg, 300, seed=3)
    ref = O.forward(cfg, w, t)
    rot = a["rot"]
    for change in ({"rot": {"dims": 0, "base": 50.0}}, {"rot": dict(rot, dims=10)}, {"rot": dict(rot, base=60.0)}, {"rot": {"dims": 12, "base": 50.0}}, {"rot": dict(rot, scaling=dict(sc, factor=5.5))},
                   {"rot": dict(rot, scaling=dict(sc, original=400))}, {"rot": dict(rot, scaling=dict(sc, fast=14.0))}, {"rot": dict(rot, scaling=dict(sc, slow=0.15))}, {"scale": 0.95}, {"mask": None}):
        other = copy.deepcopy(cfg); other["layers"][0]["mixer"].update(change)
        assert rel(O.forward(other, w, t), ref) > 100 * F32_TOL, change
    for name in ("q.b", "k.b", "v.b", "q.norm", "k.norm"):
        w2 = dict(w); w2["l0.mix." + name] = w["l0.mix." + name][::-1].copy()
        assert rel(O.forward(cfg, w2, t), ref) > 100 * F32_TOL, name
    u = np.random.default_rng(1).standard_normal((3, 2, 8))
    r = O.rotate_halves(u, {"dims": 4, "base": 100.0}, np.array([0.0, 1.0, 5.0]))
    z = (u[2, 1, 1] + 1j * u[2, 1, 3]) * np.exp(1j * 5 * 100.0 ** (-2.0 / 4))
    assert np.allclose([r[2, 1, 1], r[2, 1, 3]], [z.real, z.imag]) and np.array_equal(r[..., 4:], u[..., 4:]) and np.allclose(r[0], u[0])
    assert rel(whole(eng, t), ref) < F32_TOL
    assert rel(in_cuts(eng, t, [250] + [1] * 50), ref) < F32_TOL
    eng.close()


@pytest.mark.parametrize("scaling", [{"factor": 32.0, "original": 4096, "fast": 32.0, "slow": 1.0}, {"factor": 4.0, "original": 8, "fast": 1.0, "slow": 1.0}, {"factor": 0.5, "original": 1e6, "fast": 2.0, "slow": 1.0},
                                     {"factor": 3.0, "original": 3, "fast": 30.0, "slow": 20.0}])
def test_rotation_ramps(tmp_path, scaling):
    """a ramp inside the pairs, of no length, past the last pair and before the first"""
    check_alone(tmp_path, md.fidatar_config(40, 48, [("attention", att(dim=32, mask=None, rot={"dims": 32, "base": 10000.0, "scaling": scaling}), None)]))


# ---- the memory: a write that lasts hundreds of tokens, gates at their extremes, at and around the edges of the prefill's chunks ----
@pytest.mark.parametrize("where", [0, 3, 4, 63, 64, 65, 130])
def test_far_write_shows(tmp_path, where):
    """Nothing is forgotten and one token's input gate is open far wider than the others', so what it wrote is what later queries read."""
    cfg = md.fidatar_config(40, 48, [("mlstm", mem(heads=2, dim=12, vdim=8, gate_cap=30.0), None)])

    def tweak(w):
        w["embed"][:, 0] = -0.7; w["embed"][7, 0] = 0.7
        w["l0.mix.f"][:] *= 0.1; w["l0.mix.f.b"][:] = 16.0
        w["l0.mix.i"][:] *= 0.2; w["l0.mix.i"][:, 0] = 1.0; w["l0.mix.i.b"][:] = 0.0
    t = toks(cfg, 260, seed=3)
    t[t == 7] = 8
    t[where] = 7
    eng, w = build(tmp_path, cfg, max_tokens=300, tweak=tweak)
    ref = O.forward(cfg, w, t)
    t2 = t.copy(); t2[where] = 9
    assert rel(O.forward(cfg, w, t2)[-20:], ref[-20:]) > 100 * F32_TOL
    assert rel(whole(eng, t), ref) < F32_TOL
    assert rel(in_cuts(eng, t, [200] + [1] * 60), ref) < F32_TOL
    assert rel(in_cuts(eng, t, [where, 2, 5, 1, 64, 6, 3, 4, 260]), ref) < F32_TOL
    assert rel(in_cuts(eng, t, [where + 1, 3, 9, 2, 1, 33, 260]), ref) < F32_TOL
    eng.close()


@pytest.mark.parametrize("i_bias,f_bias,cap", [(0.0, 20.0, 25.0), (0.0, -20.0, 25.0), (-20.0, 3.0, 15.0), (20.0, 3.0, 15.0), (-9.0, -9.0, 12.0), (0.0, 0.0, 0.5), (40.0, 8.0, 60.0), (-40.0, 8.0, 45.0)])
def test_gate_extremes(tmp_path, i_bias, f_bias, cap):
    """forgetting within rounding of none and of all, writes that vanish beside the running maximum and writes that replace everything,
    gates at their caps, a cap below every gate"""
    cfg = md.fidatar_config(40, 48, [("mlstm", mem(gate_cap=cap), None)])

    def tweak(w):
        w["l0.mix.i.b"][:] += i_bias; w["l0.mix.f.b"][:] += f_bias
    eng, w = build(tmp_path, cfg, tweak=tweak)
    t = toks(cfg, 200)
    ref = O.forward(cfg, w, t)
    assert np.isfinite(ref).all()
    assert rel(whole(eng, t), ref) < F32_TOL
    assert rel(in_cuts(eng, t, [150] + [1] * 50), ref) < F32_TOL
    assert rel(in_cuts(eng, t, [7, 2, 6, 3, 5] * 9), ref) < F32_TOL
    eng.close()


def test_denominator_of_the_read_out_shows(tmp_path):
    """The norm of a head hides its scale unless the outputs are as small as the norm's own small number: there the denominator (its
    absolute value, the floor e^-m, the sum of the keys) decides.  The oracle tells each part from its absence."""
    cfg = md.fidatar_config(40, 48, [("mlstm", mem(heads=4, gate_cap=6.0), None)], eps=1e-3)

    def tweak(w):
        w["l0.mix.v"][:] *= 0.03; w["l0.mix.q"][:] *= 1.5
        w["l0.mix.i.b"][:] = [-4.0, 1.0, 3.0, 5.0]
    eng, w = build(tmp_path, cfg, tweak=tweak)
    t = toks(cfg, 200)
    ref = O.forward(cfg, w, t)
    plain = O.memory

    def changed(den):
        def memory(q, k, v, log_in, log_forget, state=None):
            T, H, D = q.shape
            out = np.zeros(v.shape)
            for a in range(H):
                S, n, m = np.zeros((D, v.shape[2])), np.zeros(D), 0.0
                for s in range(T):
                    new = max(log_forget[s, a] + m, log_in[s, a])
                    keep, write = np.exp(log_forget[s, a] + m - new), np.exp(log_in[s, a] - new)
                    S, n, m = keep * S + write * np.outer(k[s, a], v[s, a]), keep * n + write * k[s, a], new
                    out[s, a] = S.T @ q[s, a] / den(n @ q[s, a], m)
            return out, None
        return memory
    try:
        for den in (lambda z, m: 1.0, lambda z, m: max(z, np.exp(-m)), lambda z, m: abs(z) + 1e-6, lambda z, m: max(abs(z), 1.0), lambda z, m: np.exp(-m)):
            O.memory = changed(den)
            assert rel(O.forward(cfg, w, t), ref) > 100 * F32_TOL
        O.memory = changed(lambda z, m: max(abs(z), np.exp(-m)) + 1e-6)
        assert rel(O.forward(cfg, w, t), ref) < 1e-9
    finally:
        O.memory = plain
    assert rel(whole(eng, t), ref) < F32_TOL
    assert rel(in_cuts(eng, t, [1] * 200), ref) < F32_TOL
    assert rel(in_cuts(eng, t, [70, 2, 60, 3, 1, 64]), ref) < F32_TOL
    eng.close()


def test_silent_projections(tmp_path):
    """Queries, keys or values that vanish, an output that is zero for a whole head."""
    cfg = md.fidatar_config(40, 48, [("mlstm", MEM, None), ("attention", att(), None)])

    def tweak(w):
        w["l0.mix.k"][:20] = 0.0; w["l0.mix.v"][28:56] = 0.0; w["l0.mix.q"][40:] *= 1e-4
        w["l1.mix.q"][:20] = 0.0; w["l1.mix.q.b"][:20] = 0.0; w["l1.mix.k"][:] *= 1e-4; w["l1.mix.k.b"][:] = 0.0
    eng, w = build(tmp_path, cfg, tweak=tweak)
    t = toks(cfg, 60)
    ref = O.forward(cfg, w, t)
    assert np.isfinite(ref).all()
    assert rel(whole(eng, t), ref) < F32_TOL and rel(in_cuts(eng, t, [1] * 60), ref) < F32_TOL
    eng.close()


# ---- experts ----
def test_groups_of_experts_show(tmp_path):
    """The best experts of all often sit in groups that are not kept, and a group's second best counts: the oracle tells the choice from one
    without groups, with other groups and with the best score alone; weights are the scores themselves times the scale."""
    f = moe(12, 3, 4, 2, 1.7, 24)
    cfg = md.fidatar_config(50, 40, [("mlstm", mem(heads=2), f)])
    eng, w = build(tmp_path, cfg, keep=True)
    t = toks(cfg, 120)
    ref = O.forward(cfg, w, t)
    for count, keep in ((1, 1), (4, 1), (4, 3), (3, 2), (2, 1), (12, 6)):
        other = copy.deepcopy(cfg); other["layers"][0]["mlp"]["router"]["groups"] = {"count": count, "keep": keep}
        assert rel(O.forward(other, w, t), ref) > 100 * F32_TOL, (count, keep)
    for change in ({"scale": 1.6}, {"top": 2}):
        other = copy.deepcopy(cfg); other["layers"][0]["mlp"]["router"].update(change)
        assert rel(O.forward(other, w, t), ref) > 100 * F32_TOL
    h = np.random.default_rng(2).standard_normal((500, 40))
    wd = {k: np.asarray(v, np.float64) for k, v in w.items()}
    idx, wt = O.router(f, wd, "l0.mlp.", h)
    s = O.sigmoid(h @ wd["l0.mlp.router"].T)
    best = s.reshape(500, 4, 3).max(-1)
    alone = [set(np.argsort(-best[i])[:2]) != set(idx[i] // 3) and len(set(idx[i] // 3)) == 2 for i in range(500)]
    assert np.mean(alone) > 0.02          # the best score alone would keep other groups
    assert np.allclose(wt, 1.7 * np.take_along_axis(s, idx, -1)) and (np.diff(wt, axis=-1) <= 0).all()
    assert rel(whole(eng, t), ref) < F32_TOL
    assert rel(in_cuts(eng, t, [1] * 60 + [4] * 15), ref) < F32_TOL
    eng.close()


def test_bfloat16_layers(tmp_path):
    """one layer of each kind in bfloat16, routed experts included: every row within a few roundings"""
    for i, layer in enumerate((("attention", att(), dense(40)), ("mlstm", MEM, None), ("mlstm", MEM, MOE), ("attention", att(mask=None), moe(96, 6, 8, 3, 1.0, 12)))):
        cfg = md.fidatar_config(61, 72, [layer])
        eng, w = build(tmp_path, cfg, f32=False, name="b%d" % i)
        t = toks(cfg, 75)
        ref = O.forward(cfg, w, t)
        for got in (whole(eng, t), in_cuts(eng, t, [40, 2, 3] + [1] * 30)):
            r = rows(got, ref)
            assert np.mean(r > 0.01) < 0.03 and np.median(r) < 0.005
        eng.close()


# ---- embedding scale, the residual's factor, the norms of the sums, the cap of the logits ----
@pytest.mark.parametrize("kw", [{"alpha": 1.0}, {"alpha": 0.3, "scale": 1.0}, {"alpha": 4.0, "scale": 11.5}, {"softcap": None}, {"softcap": 2.0}, {"softcap": 300.0, "eps": 1e-6}, {"eps": 0.1}])
def test_model_constants(tmp_path, kw):
    layers = [("attention", att(), dense(20)), ("mlstm", MEM, MOE)]
    cfg = md.fidatar_config(40, 48, layers, **kw)
    eng, w = build(tmp_path, cfg)
    t = toks(cfg, 60)
    ref = O.forward(cfg, w, t)
    for key, value in (("postln_alpha", cfg["postln_alpha"] * 1.02), ("logit_softcap", (cfg.get("logit_softcap") or 5.0) * 0.98), ("embedding", {"scale": cfg["embedding"]["scale"] * 1.02}), ("norm", {"eps": cfg["norm"]["eps"] + 0.01})):
        if key == "logit_softcap" and cfg.get(key, 0) == 300.0:
            continue          # far above every logit
        assert rel(O.forward(dict(cfg, **{key: value}), w, t), ref) > 20 * F32_TOL, key
    assert rel(whole(eng, t), ref) < F32_TOL
    assert rel(in_cuts(eng, t, [3, 1, 20, 2, 34]), ref) < F32_TOL
    eng.close()


def test_long_prompt_splits_keys_in_decoding(tmp_path):
    """Short portions deal the key pages out to several blocks and merge; past 64 pages a block takes several of them; prompts longer than
    one portion of the engine's own; many chunks of the memory, more than one pass of its gates kernel."""
    cfg = md.fidatar_config(40, 48, [("attention", att(heads=3, kv_heads=1, mask=None), dense(24)), ("mlstm", MEM, None), ("attention", att(heads=3, kv_heads=1, mask={"size": 1500}), None)])
    eng, w = build(tmp_path, cfg, max_tokens=400)
    t = toks(cfg, 330, seed=6)
    ref = O.forward(cfg, w, t)
    assert rel(in_cuts(eng, t, [300] + [1] * 20 + [2, 3, 4, 1]), ref) < F32_TOL
    eng.close()
    t = toks(cfg, 2500, seed=7)
    ref = O.forward(cfg, w, t)
    for chunk in (None, 2400):
        eng, w = build(tmp_path, cfg, max_tokens=2600, name="l%d" % (chunk or 0), chunk=chunk)
        s = eng.seq_open()
        eng.step(s, t[:2400], [])
        got = [eng.step(s, t[2400 + i:2401 + i], [0]) for i in range(40)] + [eng.step(s, t[2440:2443], [0, 1, 2]), eng.step(s, t[2443:2500], range(57))]
        assert rel(np.concatenate(got), ref[2400:]) < F32_TOL
        eng.close()


def test_long_decoding(tmp_path):
    cfg = mixed_cfg()
    eng, w = build(tmp_path, cfg, max_tokens=700)
    t = toks(cfg, 650, seed=8)
    ref = O.forward(cfg, w, t)
    got = in_cuts(eng, t, [3] + [1] * 647)
    assert rel(got, ref) < 2 * F32_TOL
    eng.close()


def test_first_tokens_and_single_token_requests(tmp_path):
    cfg = mixed_cfg()
    eng, w = build(tmp_path, cfg)
    for n in (1, 2, 3, 5):
        t = toks(cfg, n, seed=20 + n)
        ref = O.forward(cfg, w, t)
        assert rel(whole(eng, t), ref) < F32_TOL
        assert rel(in_cuts(eng, t, [1] * n), ref) < F32_TOL
    t = toks(cfg, 9, seed=30)
    ref = O.forward(cfg, w, t)
    for _ in range(3):          # the same slot and pages again
        assert rel(in_cuts(eng, t, [1, 3, 5]), ref) < F32_TOL
    eng.close()


# ---- generation through the engine's own entry points ----
def test_greedy_generation(tmp_path):
    cfg = mixed_cfg(vocab=53)
    eng, w = build(tmp_path, cfg)
    prompt = toks(cfg, 17, seed=4)
    total = 60
    ids = np.zeros(total + 1, np.uint32); ids[:17] = prompt
    eng.decode_greedy(ids, 17, total)
    # the oracle follows the engine's ids and must agree on every choice whose margin is not a rounding matter
    ref = O.forward(cfg, w, ids[:total - 1])
    for pos in range(16, total - 1):
        top = np.sort(ref[pos])[-2:]
        if top[1] - top[0] > 1e-3:
            assert int(np.argmax(ref[pos])) == int(ids[pos + 1]), pos
    ids2 = np.zeros(total + 1, np.uint32); ids2[:17] = prompt
    for pos in range(total - 1):
        nxt = eng.next_greedy(ids2, pos, 1 if pos < 16 else 0)
        if pos >= 16:
            ids2[pos + 1] = nxt
    assert np.array_equal(ids[:total], ids2[:total])
    eng.close()
    # the generation command on the same folder
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    p = subprocess.run([sys.executable, "-m", "nano_b200.generate", "--model", str(tmp_path / "m"), "--prompt-ids", ",".join(str(int(x)) for x in prompt),
                        "--max-new", str(total - 17), "--dtype", "float32"], cwd=root, capture_output=True, text=True, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    assert [int(x) for x in p.stdout.split()] == [int(x) for x in ids[:total]]


def test_sampled_generation_and_penalty(tmp_path):
    """The device sampler and the repetition penalty on the implicit sequence."""
    cfg = mixed_cfg(vocab=80)
    eng, w = build(tmp_path, cfg)
    prompt = [5, 17, 3, 44]
    ids = np.zeros(32, np.uint32); ids[:4] = prompt
    for pos in range(3):
        eng.next_greedy(ids, pos, 1)
    tok, top6 = eng.next_sampled(ids, 3, 1.0, 0.8, 0.95, 0.01)
    ref = O.forward(cfg, w, prompt)[-1]
    assert top6[0] == int(np.argmax(ref)) and tok == top6[0]          # a coin near 0 takes the most probable token
    eng.forward(5, 0); eng.forward(17, 1)                             # position 0 starts over
    assert rel(eng.logits()[None, :], O.forward(cfg, w, [5, 17])[-1:]) < F32_TOL
    pen = O.forward(cfg, w, [5, 17, 3])[-1].copy()
    for i in (5, 17):
        pen[i] = pen[i] / 50.0 if pen[i] > 0 else pen[i] * 50.0
    ids[:3] = [5, 17, 3]
    assert eng.next_greedy(ids, 2, 0, 50.0) == int(np.argmax(pen))
    eng.close()


@pytest.mark.parametrize("kind,mixer,mlp", [("attention", att(rot={"dims": 22, "base": 10.0}), None), ("attention", att(kv_heads=4), None), ("attention", att(dim=300), None), ("attention", att(mask={"size": 0}), None),
                                            ("mlstm", mem(dim=600), None), ("mlstm", mem(gate_cap=0.0), None), ("mlstm", MEM, moe(12, 3, 5, 2)), ("mlstm", MEM, moe(12, 4, 4, 1)), ("mlstm", MEM, moe(12, 2, 3, 4))])
def test_bad_folders_are_refused(tmp_path, kind, mixer, mlp):
    """more turning coordinates than a head has; heads that the key/value heads do not divide; sizes without a kernel; an empty block; gates
    without a range; groups that the experts do not fill, too small for the choice, or more kept than there are"""
    cfg = md.fidatar_config(30, 32, [(kind, mixer, mlp)])
    w = md.fidatar_random(cfg)
    path = md.write_model_dir(str(tmp_path / "a"), cfg, w)
    with pytest.raises(E.NB200Error):
        E.Engine(path, 64)


def test_missing_tensor_is_named(tmp_path):
    cfg = md.fidatar_config(30, 32, [("attention", att(), MOE)])
    w = md.fidatar_random(cfg)
    del w["l0.mix.k.b"]
    with pytest.raises(E.NB200Error, match="l0.mix.k.b"):
        E.Engine(md.write_model_dir(str(tmp_path / "a"), cfg, w), 64)


def test_replay_command(tmp_path):
    """bin/trace_run on a Fidatar folder: portions, single tokens, a step that wants nothing, two requests one after the other."""
    cfg = no_close_calls(mixed_cfg())
    w = md.fidatar_random(cfg, 2)
    path = md.write_model_dir(str(tmp_path / "m"), cfg, w)
    a, b = toks(cfg, 70, seed=1), toks(cfg, 9, seed=2)
    ra, rb = O.forward(cfg, w, a), O.forward(cfg, w, b)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:40].tolist(), "want": [39, 3]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[40:42].tolist(), "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": a[42:43].tolist(), "want": [0]}], "end": []},
             {"step": 3, "entries": [{"id": "a", "tokens": a[43:70].tolist(), "want": [26]}], "end": ["a"]},
             {"step": 4, "entries": [{"id": "b", "tokens": b.tolist(), "want": [8]}], "end": ["b"]}]
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    for dtype, tol in (("float32", F32_TOL), ("bfloat16", 3 * BF16_TOL)):
        out = tmp_path / ("out_" + dtype)
        p = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", path, "--dtype", dtype, "--out", str(out), "--max-tokens", "128"],
                           input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=600)
        assert p.returncode == 0, p.stderr[-2000:]
        assert [l for l in p.stdout.split("\n") if l.startswith("done")] == ["done %d" % i for i in range(5)]
        V = cfg["vocab"]
        g0 = np.fromfile(out / "0.f32", "<f4").reshape(-1, V)
        assert rel(g0, ra[[39, 3]]) < tol
        assert not (out / "1.f32").exists()
        assert rel(np.fromfile(out / "2.f32", "<f4").reshape(-1, V), ra[[42]]) < tol
        assert rel(np.fromfile(out / "3.f32", "<f4").reshape(-1, V), ra[[69]]) < tol
        assert rel(np.fromfile(out / "4.f32", "<f4").reshape(-1, V), rb[[8]]) < tol
