"""Kadesun on the layered runtime against the plain restatement in tests/kadesun_oracle.py: every mechanism alone, prefill against
token-by-token decoding, portions of several sizes, interleaved requests, pages and slots used again, keys far away and at page
borders, the sink, the soft cap, the rotation, the norm over the whole projection, writes to the state that last or fade, the first
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

import kadesun_oracle as O

pytestmark = pytest.mark.gpu

LEFT = {"heads": 6, "kv_heads": 2, "dim": 20, "vdim": 12, "scale": 0.3, "softcap": 12.0, "rot": {"dims": 12, "base": 300.0}}
RIGHT = {"heads": 4, "kv_heads": 2, "dim": 12, "vdim": 20, "conv": 4}
DELTA = {"heads": 6, "kv_heads": 3, "dim": 24, "vdim": 20, "conv": 3}


def left(**kw):
    m = copy.deepcopy(LEFT)
    m.update(kw)
    return {k: v for k, v in m.items() if v is not None}


def par(l=None, r=None):
    return {"left": l or copy.deepcopy(LEFT), "right": dict(RIGHT, **(r or {}))}


def delta(**kw):
    return dict(DELTA, **kw)


def build(tmp_path, cfg, seed=0, f32=True, max_tokens=512, keep=False, chunk=None, name="m", tweak=None, **ranks):
    w = md.kadesun_random(cfg, seed, **ranks)
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


def check_alone(tmp_path, cfg, n=75, tweak=None, **ranks):
    eng, w = build(tmp_path, cfg, keep=True, tweak=tweak, **ranks)
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
    ("delta", DELTA),
    ("delta", delta(heads=1, kv_heads=1, dim=1, vdim=1, conv=2)),
    ("delta", delta(heads=3, kv_heads=3, dim=16, vdim=16, conv=1)),                 # no taps before the present one: no tail in the state
    ("delta", delta(heads=2, kv_heads=1, dim=33, vdim=7, conv=9)),                  # a convolution longer than a short portion; sizes no vector width divides
    ("delta", delta(heads=5, kv_heads=5, dim=64, vdim=40, conv=4)),
    ("delta", delta(heads=4, kv_heads=1, dim=128, vdim=72, conv=2)),
    ("delta", delta(heads=2, kv_heads=2, dim=130, vdim=150, conv=4)),               # the widest register tile; more value columns than a block's threads
    ("delta", delta(heads=1, kv_heads=1, dim=256, vdim=33, conv=4)),
    ("parallel", par()),
    ("parallel", par(left(heads=1, kv_heads=1, dim=2, vdim=1, rot={"dims": 2, "base": 5.0}), {"heads": 1, "kv_heads": 1, "dim": 1, "vdim": 1, "conv": 1})),
    ("parallel", par(left(heads=4, kv_heads=4, dim=16, vdim=16, rot={"dims": 16, "base": 1e4}), {"heads": 4, "kv_heads": 4, "dim": 16, "vdim": 16, "conv": 4})),      # one head per key/value head; sizes all equal
    ("parallel", par(left(heads=11, kv_heads=1, dim=7, vdim=5, rot={"dims": 2, "base": 9.0}), {"heads": 3, "kv_heads": 1, "dim": 9, "vdim": 13, "conv": 5})),          # more heads per key/value head than a block takes
    ("parallel", par(left(heads=6, kv_heads=3, dim=64, vdim=128, rot={"dims": 32, "base": 1e6}), {"heads": 2, "kv_heads": 2, "dim": 64, "vdim": 128, "conv": 4})),
    ("parallel", par(left(heads=2, kv_heads=1, dim=100, vdim=68, rot={"dims": 100, "base": 50.0}), {"heads": 2, "kv_heads": 1, "dim": 128, "vdim": 96, "conv": 3})),
    ("parallel", par(left(heads=2, kv_heads=2, dim=256, vdim=256, scale=0.06, rot={"dims": 64, "base": 100.0}), {"heads": 1, "kv_heads": 1, "dim": 200, "vdim": 24, "conv": 4})),
    ("parallel", par(left(softcap=None, rot=None))),                                # neither cap nor positions
]


# ---- each mechanism alone: one layer, no feed-forward, residual after the layer and logits; whole, token by token, portions ----
@pytest.mark.parametrize("kind,mixer", MIXERS)
def test_mixer_alone(tmp_path, kind, mixer):
    check_alone(tmp_path, md.kadesun_config(61, 72, [(kind, mixer, None)]))


@pytest.mark.parametrize("ranks", [(1, 1), (16, 16), (7, 40), (64, 3)])
def test_low_ranks(tmp_path, ranks):
    check_alone(tmp_path, md.kadesun_config(40, 48, [("parallel", par(), None)]), decay_rank=ranks[0], gate_rank=ranks[1])


@pytest.mark.parametrize("ff", [56, 7, 129, 1])
def test_feed_forward(tmp_path, ff):
    check_alone(tmp_path, md.kadesun_config(50, 40, [("delta", delta(heads=2, kv_heads=1), ff)]), n=40)


@pytest.mark.parametrize("width,vocab", [(50, 61), (37, 33), (130, 7), (1100, 20)])
def test_ragged_widths(tmp_path, width, vocab):
    """widths and vocabularies that no vector width divides, through every product of a layer"""
    cfg = md.kadesun_config(vocab, width, [("parallel", par(), 30), ("delta", DELTA, None), ("delta", delta(dim=10), 21)])
    eng, w = build(tmp_path, cfg)
    t = toks(cfg, 45)
    ref = O.forward(cfg, w, t)
    assert rel(whole(eng, t), ref) < F32_TOL
    assert rel(in_cuts(eng, t, [3, 1, 2, 4, 35]), ref) < F32_TOL
    eng.close()
    eng, w = build(tmp_path, cfg, f32=False, name="b")
    assert rel(whole(eng, t), ref) < BF16_TOL and rel(in_cuts(eng, t, [40, 1, 1, 3]), ref) < BF16_TOL
    eng.close()


def mixed_cfg(vocab=67):
    layers = [("delta", DELTA, None), ("parallel", par(), 40), ("parallel", par(left(heads=3, kv_heads=3, dim=8, rot={"dims": 4, "base": 40.0}), {"heads": 2, "kv_heads": 2}), None),
              ("delta", delta(heads=2, kv_heads=1, conv=5), 24), ("parallel", par(), 40)]
    return md.kadesun_config(vocab, 56, layers)


@pytest.mark.parametrize("order", ["d", "p", "pd", "dpd", "ddpp", "pDdP"])
def test_layer_order(tmp_path, order):
    """the residual after every layer; capitals carry a feed-forward"""
    layers = [("delta" if c in "dD" else "parallel", DELTA if c in "dD" else par(), 33 if c.isupper() else None) for c in order]
    cfg = md.kadesun_config(40, 48, layers)
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
    cfg = mixed_cfg()
    eng, w = build(tmp_path, cfg, f32=f32)
    t = toks(cfg, 150)
    ref = O.forward(cfg, w, t)
    tol = F32_TOL if f32 else BF16_TOL
    full = whole(eng, t)
    assert rel(full, ref) < tol
    for cuts in ([1] * 150, [2] * 75, [3, 2, 64, 5, 1, 1, 33, 2, 39], [100] + [1] * 50, [31, 1, 32, 33, 53], [7] * 22, [5, 6, 7, 8, 9, 10, 11, 12, 82], [149, 1], [4] * 38):
        got = in_cuts(eng, t, cuts)
        assert rel(got, ref) < tol, cuts[:4]
        assert rel(got, full) < tol, cuts[:4]
    eng.close()
    for chunk in (16, 5, 3):
        eng, _ = build(tmp_path, cfg, f32=f32, chunk=chunk, name="c%d" % chunk)       # chunks of the engine's own inside one step
        assert rel(whole(eng, t), ref) < tol
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


# ---- a far key among hundreds, where random weights would hide it: one key made to stand out, at and around page borders ----
def stand_out(w, tok, H, G, D):
    """Coordinate 0 of the residual is positive for token `tok` alone.  The last (unturned) coordinate of every head's key reads it with a
    large gain and the same coordinate of every query is constant, so a query's weight sits on token `tok` wherever it is in sight."""
    w["embed"][:, 0] = -3.0; w["embed"][tok, 0] = 3.0
    p = "l0.mix.left."
    w[p + "k"][:] *= 0.05; w[p + "q"][:] *= 0.05
    for g in range(G):
        w[p + "k"][g * D + D - 1] = 0.0; w[p + "k"][g * D + D - 1, 0] = 1.0
    for h in range(H):
        w[p + "q"][h * D + D - 1] = 0.0; w[p + "q"][h * D + D - 1, 0] = -1.0
    w["l0.mix.left.sink"][:] = -3.0


@pytest.mark.parametrize("where", [0, 31, 32, 33, 63, 64, 200])
def test_far_key_shows(tmp_path, where):
    """Queries hundreds of positions later put their weight on token `where`: losing that key or its value would change the logits far
    beyond the tolerance."""
    a = left(heads=4, kv_heads=2, dim=16, vdim=16, scale=0.5, softcap=9.0, rot={"dims": 4, "base": 100.0})
    cfg = md.kadesun_config(40, 48, [("parallel", par(a), None)])
    t = toks(cfg, 330, seed=3)
    t[t == 7] = 8
    t[where] = 7
    eng, w = build(tmp_path, cfg, max_tokens=400, tweak=lambda w: stand_out(w, 7, 4, 2, 16))
    ref = O.forward(cfg, w, t)
    t2 = t.copy(); t2[where] = 9
    r = copy.deepcopy(w); r["l0.mix.right.out"] = r["l0.mix.right.out"] * 0.0          # the attention branch alone: what a lost key does to it
    assert rel(O.forward(cfg, r, t2)[-20:], O.forward(cfg, r, t)[-20:]) > 100 * F32_TOL
    assert rel(whole(eng, t), ref) < F32_TOL
    assert rel(in_cuts(eng, t, [290] + [1] * 40), ref) < F32_TOL
    assert rel(in_cuts(eng, t, [29, 2, 2, 31, 1, 1, 64, 130, 3, 4, 63]), ref) < F32_TOL
    eng.close()


def test_sink_shows(tmp_path):
    """A large sink takes most of the weight, a very negative one none; each head has its own; a sink far above every score must not
    overflow.  The oracle tells them apart; the engine follows, also through the key splits of a long decode."""
    cfg = md.kadesun_config(40, 48, [("parallel", par(left(heads=3, kv_heads=1, dim=16, vdim=16, scale=0.5)), None)])
    t = toks(cfg, 200, seed=9)
    refs = []
    for i, sink in enumerate(([6.0, -30.0, 0.5], [0.0, 0.0, 0.0], [120.0, 3.0, -120.0])):
        def tweak(w, sink=sink):
            w["l0.mix.left.sink"][:] = np.asarray(sink, np.float32)
        eng, w = build(tmp_path, cfg, tweak=tweak, name="s%d" % i)
        ref = O.forward(cfg, w, t)
        refs.append(ref)
        assert np.isfinite(ref).all()
        assert rel(whole(eng, t), ref) < F32_TOL
        assert rel(in_cuts(eng, t, [150] + [1] * 50), ref) < F32_TOL
        assert rel(in_cuts(eng, t, [2, 3] * 40), ref) < F32_TOL
        eng.close()
    assert rel(refs[0], refs[1]) > 100 * F32_TOL and rel(refs[2], refs[1]) > 100 * F32_TOL


def test_cap_rotation_norm_and_gate_show(tmp_path):
    """The oracle tells each of the attention's parts from its absence on this model (large scores, so that the cap bites); the engine
    follows, far into a sequence."""
    a = left(heads=4, kv_heads=2, dim=16, vdim=16, scale=1.2, softcap=3.0, rot={"dims": 16, "base": 50.0})
    cfg = md.kadesun_config(40, 48, [("parallel", par(a), None)])
    eng, w = build(tmp_path, cfg)
    t = toks(cfg, 300, seed=3)
    ref = O.forward(cfg, w, t)
    for change in ({"softcap": None}, {"softcap": 3.2}, {"rot": {"dims": 0, "base": 50.0}}, {"rot": {"dims": 8, "base": 50.0}}, {"rot": {"dims": 16, "base": 60.0}}, {"scale": 1.25}):
        other = copy.deepcopy(cfg); other["layers"][0]["mixer"]["left"].update(change)
        assert rel(O.forward(other, w, t), ref) > 100 * F32_TOL, change
    w2 = dict(w); w2["l0.mix.left.g"] = w["l0.mix.left.g"][::-1]
    assert rel(O.forward(cfg, w2, t), ref) > 100 * F32_TOL
    q = t.astype(np.int64)
    h = np.asarray(w["embed"], np.float64)[q] @ np.asarray(w["l0.mix.left.q"], np.float64).T
    whole_norm = O.rms_norm(h, w["l0.mix.left.q.norm"], 1e-5).reshape(300, 4, 16)
    per_head = O.rms_norm(h.reshape(300, 4, 16), w["l0.mix.left.q.norm"].reshape(4, 16), 1e-5)
    assert np.abs(whole_norm - per_head).max() > 0.05          # the norm runs over the whole projection, not over each head
    u = np.random.default_rng(1).standard_normal((3, 2, 8))
    r = O.rotate_halves(u, {"dims": 4, "base": 100.0}, np.array([0.0, 1.0, 5.0]))
    z = (u[2, 1, 1] + 1j * u[2, 1, 3]) * np.exp(1j * 5 * 100.0 ** (-2.0 / 4))
    assert np.allclose([r[2, 1, 1], r[2, 1, 3]], [z.real, z.imag]) and np.array_equal(r[..., 4:], u[..., 4:]) and np.allclose(r[0], u[0])
    assert rel(whole(eng, t), ref) < F32_TOL
    assert rel(in_cuts(eng, t, [250] + [1] * 50), ref) < F32_TOL
    eng.close()


# ---- the state: a write that lasts hundreds of tokens, forgetting that is nearly complete, at and around the edges of the scan's chunks ----
@pytest.mark.parametrize("kind", ["delta", "parallel"])
@pytest.mark.parametrize("where", [0, 3, 4, 7, 8, 31, 130])
def test_far_write_shows(tmp_path, kind, where):
    """Nothing is forgotten by itself (decay rates near zero) and the keys of the other tokens are kept out of one direction, so what token
    `where` wrote there is still what later queries read."""
    cfg = md.kadesun_config(40, 48, [(kind, delta(heads=2, kv_heads=1, dim=12, vdim=8) if kind == "delta" else par(None, {"heads": 2, "kv_heads": 1, "dim": 12, "vdim": 8}), None)])
    p = "l0.mix." if kind == "delta" else "l0.mix.right."

    def tweak(w):
        w[p + "A_log"][:] = -12.0
        w["embed"][:, 0] = -3.0; w["embed"][7, 0] = 3.0
        for n in ("q", "k"):
            w[p + n + ".conv"][:, :-1] = 0.0; w[p + n + ".conv"][:, -1] = 1.0
            w[p + n][:] *= 0.3
            w[p + n][5] = 0.0
        w[p + "k"][5, 0] = 3.0          # silu keeps it large for token 7 and closes it for the others
        w[p + "q"][5, 0] = -1.0
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


@pytest.mark.parametrize("kind", ["delta", "parallel"])
@pytest.mark.parametrize("a_log,bias", [(-9.0, -6.0), (3.0, 3.0), (6.0, 6.0), (0.0, -9.0)])
def test_decay_extremes(tmp_path, kind, a_log, bias):
    """factors within rounding of one, and factors that are zero in single precision (their products inside a chunk as well)"""
    cfg = md.kadesun_config(40, 48, [(kind, DELTA if kind == "delta" else par(), None)])
    p = "l0.mix." if kind == "delta" else "l0.mix.right."

    def tweak(w):
        w[p + "A_log"][:] = a_log; w[p + "dt_bias"][:] = bias
    eng, w = build(tmp_path, cfg, tweak=tweak)
    t = toks(cfg, 200)
    ref = O.forward(cfg, w, t)
    assert np.isfinite(ref).all()
    assert rel(whole(eng, t), ref) < F32_TOL
    assert rel(in_cuts(eng, t, [150] + [1] * 50), ref) < F32_TOL
    assert rel(in_cuts(eng, t, [7, 2, 6, 3, 5] * 9), ref) < F32_TOL
    eng.close()


def test_silent_channels(tmp_path):
    """Projections that vanish: the unit vectors' own small number keeps them finite, a step size of nearly nothing writes nothing."""
    cfg = md.kadesun_config(40, 48, [("parallel", par(), None), ("delta", DELTA, None)])

    def tweak(w):
        w["l0.mix.right.k"][:] *= 1e-4; w["l0.mix.right.q"][:12] = 0.0
        w["l1.mix.k"][:] = 0.0; w["l1.mix.b"][0] = 0.0
    eng, w = build(tmp_path, cfg, tweak=tweak)
    t = toks(cfg, 60)
    ref = O.forward(cfg, w, t)
    assert np.isfinite(ref).all()
    assert rel(whole(eng, t), ref) < F32_TOL and rel(in_cuts(eng, t, [1] * 60), ref) < F32_TOL
    eng.close()


def test_long_prompt_splits_keys_in_decoding(tmp_path):
    """Short portions deal the key pages out to several blocks and merge; past 64 pages a block takes several of them."""
    cfg = md.kadesun_config(40, 48, [("parallel", par(left(heads=3, kv_heads=1)), 24)])
    eng, w = build(tmp_path, cfg, max_tokens=400)
    t = toks(cfg, 330, seed=6)
    ref = O.forward(cfg, w, t)
    assert rel(in_cuts(eng, t, [300] + [1] * 20 + [2, 3, 4, 1]), ref) < F32_TOL
    eng.close()
    eng, w = build(tmp_path, cfg, max_tokens=2300, name="l")
    t = toks(cfg, 2200, seed=7)
    s = eng.seq_open()
    eng.step(s, t[:2100], [])
    got = [eng.step(s, t[2100 + i:2101 + i], [0]) for i in range(40)] + [eng.step(s, t[2140:2143], [0, 1, 2]), eng.step(s, t[2143:2200], range(57))]
    ref = O.forward(cfg, w, t)
    assert rel(np.concatenate(got), ref[2100:]) < F32_TOL
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


@pytest.mark.parametrize("mixer", [("parallel", par(left(rot={"dims": 22, "base": 10.0}))), ("parallel", par(left(kv_heads=4))), ("delta", delta(kv_heads=4)),
                                   ("delta", delta(dim=300)), ("parallel", par(left(dim=300)))])
def test_bad_folders_are_refused(tmp_path, mixer):
    """more turning coordinates than a head has; heads that the key/value heads do not divide; sizes without a kernel"""
    cfg = md.kadesun_config(30, 32, [(mixer[0], mixer[1], None)])
    good = copy.deepcopy(cfg)
    m = good["layers"][0]["mixer"]
    for part in ([m] if mixer[0] == "delta" else [m["left"], m["right"]]):
        part["kv_heads"] = 1
    w = md.kadesun_random(good)
    path = md.write_model_dir(str(tmp_path / "a"), cfg, w)
    with pytest.raises(E.NB200Error):
        E.Engine(path, 64)


def test_missing_tensor_is_named(tmp_path):
    cfg = md.kadesun_config(30, 32, [("parallel", par(), 16)])
    w = md.kadesun_random(cfg)
    del w["l0.mix.right.a2"]
    with pytest.raises(E.NB200Error, match="l0.mix.right.a2"):
        E.Engine(md.write_model_dir(str(tmp_path / "a"), cfg, w), 64)


def test_replay_command(tmp_path):
    """bin/trace_run on a Kadesun folder: portions, single tokens, a step that wants nothing, two requests one after the other."""
    cfg = mixed_cfg()
    w = md.kadesun_random(cfg, 2)
    path = md.write_model_dir(str(tmp_path / "m"), cfg, w)
    a, b = toks(cfg, 70, seed=1), toks(cfg, 9, seed=2)
    ra, rb = O.forward(cfg, w, a), O.forward(cfg, w, b)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:40].tolist(), "want": [39, 3]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[40:42].tolist(), "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": a[42:43].tolist(), "want": [0]}], "end": []},
             {"step": 3, "entries": [{"id": "a", "tokens": a[43:70].tolist(), "want": [26]}], "end": ["a"]},
             {"step": 4, "entries": [{"id": "b", "tokens": b.tolist(), "want": [8]}], "end": ["b"]}]
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    for dtype, tol in (("float32", F32_TOL), ("bfloat16", BF16_TOL)):
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
