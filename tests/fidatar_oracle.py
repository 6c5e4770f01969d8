"""A plain, slow restatement of the Fidatar design in numpy (float64), one function per mechanism.  It shares no code with the engine:
it is what the engine's kernels are held against in tests/test_gpu_fidatar.py.

Fidatar: a decoder whose residual is normed AFTER every sum,  x <- norm(alpha x + sublayer(x)), the sublayer reading x itself.  Mixers
are "mlstm" (a matrix memory per head with exponential gates, kept in range by a running maximum) and "attention" (grouped-query softmax
attention inside fixed blocks of positions, a norm per query and key head, rescaled rotary positions, one added to the softmax
denominator).  Feed-forwards are squared-relu units, dense or as experts chosen by sigmoid scores inside the best groups.
"""
import math

import numpy as np


def rms_norm(u, w, eps):
    return u / np.sqrt((u ** 2).mean(-1, keepdims=True) + eps) * w


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def log_sigmoid(z):
    return -np.logaddexp(0.0, -z)


def relu_squared(z):
    return np.where(z > 0, z, 0.0) ** 2


def rotation_frequencies(rot):
    """(frequency of every turning pair, factor on cos and sin)"""
    dims, base = int(rot["dims"]), float(rot["base"])
    f = np.array([base ** (-2.0 * i / dims) for i in range(dims // 2)])
    sc = rot.get("scaling")
    if not sc:
        return f, 1.0

    def place(turns):          # the (fractional) coordinate that turns that often over the original length
        return dims * math.log(sc["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo, hi = max(math.floor(place(sc["fast"])), 0), min(math.ceil(place(sc["slow"])), dims - 1)
    out = np.empty_like(f)
    for i in range(dims // 2):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out[i] = f[i] / sc["factor"] * ramp + f[i] * (1.0 - ramp)
    return out, 0.1 * math.log(sc["factor"]) + 1.0


def rotate_halves(u, rot, positions):
    """u [T, heads, n]: coordinate i < dims/2 turns with coordinate i + dims/2; the rest pass"""
    f, amp = rotation_frequencies(rot)
    half = len(f)
    out = u.copy()
    for i in range(half):
        c, s = (amp * np.cos(positions * f[i]))[:, None], (amp * np.sin(positions * f[i]))[:, None]
        p, q = u[..., i], u[..., i + half]
        out[..., i] = p * c - q * s
        out[..., i + half] = q * c + p * s
    return out


def attention(m, w, p, h, eps):
    """position i sees the positions j <= i of its own block of mask.size positions"""
    T = h.shape[0]
    H, G, D, VD = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    size = m["mask"]["size"] if m.get("mask") else T + 1
    pos = np.arange(T, dtype=np.float64)
    q = (h @ w[p + "q"].T + w[p + "q.b"]).reshape(T, H, D)
    k = (h @ w[p + "k"].T + w[p + "k.b"]).reshape(T, G, D)
    v = (h @ w[p + "v"].T + w[p + "v.b"]).reshape(T, G, VD)
    q, k = rms_norm(q, w[p + "q.norm"], eps), rms_norm(k, w[p + "k.norm"], eps)
    if m.get("rot"):
        q, k = rotate_halves(q, m["rot"], pos), rotate_halves(k, m["rot"], pos)
    out = np.zeros((T, H, VD))
    for head in range(H):
        g = head // (H // G)
        for i in range(T):
            first = (i // size) * size
            s = (k[first:i + 1, g] @ q[i, head]) * m["scale"]
            top = max(s.max(), 0.0)
            e = np.exp(s - top)
            out[i, head] = (e / (math.exp(-top) + e.sum())) @ v[first:i + 1, g]
    return out.reshape(T, H * VD) @ w[p + "o"].T


def memory(q, k, v, log_in, log_forget, state=None):
    """q, k [T, H, D], v [T, H, VD], logs of the gates [T, H] -> outputs [T, H, VD] and the state (S [H, D, VD], n [H, D], m [H])"""
    T, H, D = q.shape
    S, n, m = (np.zeros((H, D, v.shape[2])), np.zeros((H, D)), np.zeros(H)) if state is None else [a.copy() for a in state]
    out = np.zeros(v.shape)
    for t in range(T):
        for a in range(H):
            new = max(log_forget[t, a] + m[a], log_in[t, a])
            keep, write = math.exp(log_forget[t, a] + m[a] - new), math.exp(log_in[t, a] - new)
            S[a] = keep * S[a] + write * np.outer(k[t, a], v[t, a])
            n[a] = keep * n[a] + write * k[t, a]
            m[a] = new
            out[t, a] = S[a].T @ q[t, a] / (max(abs(n[a] @ q[t, a]), math.exp(-new)) + 1e-6)
    return out, (S, n, m)


def mlstm(m, w, p, h, eps):
    T = h.shape[0]
    H, D, VD, cap = m["heads"], m["dim"], m["vdim"], m["gate_cap"]
    q = (h @ w[p + "q"].T).reshape(T, H, D) / math.sqrt(D)
    k = (h @ w[p + "k"].T).reshape(T, H, D)
    v = (h @ w[p + "v"].T).reshape(T, H, VD)
    log_in = cap * np.tanh((h @ w[p + "i"].T + w[p + "i.b"]) / cap)
    log_forget = log_sigmoid(cap * np.tanh((h @ w[p + "f"].T + w[p + "f.b"]) / cap))
    o, _ = memory(q, k, v, log_in, log_forget)
    o = rms_norm(o, 1.0, eps).reshape(T, H * VD)
    return (o * w[p + "norm"] * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def dense_ff(w, p, h):
    return relu_squared(h @ w[p + "up"].T) @ w[p + "down"].T


def router(f, w, p, h):
    """(chosen experts [T, top], best score first; their weights)"""
    r = f["router"]
    s = sigmoid(h @ w[p + "router"].T)
    NE, groups = r["experts"], r.get("groups") or {"count": 1, "keep": 1}
    size = NE // groups["count"]
    idx = np.zeros((h.shape[0], r["top"]), np.int64)
    for t in range(h.shape[0]):
        of_group = [np.sort(s[t, g * size:(g + 1) * size])[-2:].sum() for g in range(groups["count"])]
        best = sorted(range(groups["count"]), key=lambda g: (-of_group[g], g))[:groups["keep"]]
        open_ = [e for e in range(NE) if e // size in best]
        idx[t] = sorted(open_, key=lambda e: (-s[t, e], e))[:r["top"]]
    return idx, np.take_along_axis(s, idx, -1) * r.get("scale", 1.0)


def moe_ff(f, w, p, h):
    idx, wt = router(f, w, p, h)
    out = np.zeros((h.shape[0], w[p + "e0.down"].shape[0]))
    for t in range(h.shape[0]):
        for e, a in zip(idx[t], wt[t]):
            out[t] += a * dense_ff(w, p + f"e{e}.", h[t])
    return out


def forward(cfg, weights, tokens, trace=None):
    """logits [T, vocab] of a sequence from its start; trace (a list) receives the residual after every layer"""
    w = {k: np.asarray(v, np.float64) for k, v in weights.items()}
    eps, alpha = cfg["norm"]["eps"], cfg["postln_alpha"]
    x = w["embed"][np.asarray(tokens, np.int64)] * cfg["embedding"]["scale"]
    for i, L in enumerate(cfg["layers"]):
        p = f"l{i}."
        mix = {"attention": attention, "mlstm": mlstm}[L["type"]]
        x = rms_norm(alpha * x + mix(L["mixer"], w, p + "mix.", x, eps), w[p + "norm1"], eps)
        f = L.get("mlp")
        if f:
            y = moe_ff(f, w, p + "mlp.", x) if f["kind"] == "moe" else dense_ff(w, p + "mlp.", x)
            x = rms_norm(alpha * x + y, w[p + "norm2"], eps)
        if trace is not None:
            trace.append(x.copy())
    z = rms_norm(x, w["final.norm"], eps) @ w["head"].T
    cap = cfg.get("logit_softcap")
    return cap * np.tanh(z / cap) if cap else z
