"""A plain, slow restatement of the Kadesun design in numpy (float64), one function per mechanism.  It shares no code with the engine:
it is what the engine's kernels are held against in tests/test_gpu_kadesun.py.

Kadesun: a decoder whose sublayers read the residual itself and are normed on the way out,  x <- x + norm(sublayer(x)).  Mixers are
"delta" (a gated delta rule: a matrix state per head that forgets, is corrected towards the present value at the present key, and is
read by the query; one decay per head and token) and "parallel" (a grouped-query softmax attention and a gated delta rule with one
decay per key channel, side by side on the same input, each normed, then averaged).  The feed-forward is the gated silu unit.
"""
import math

import numpy as np


def rms_norm(u, w, eps):
    return u / np.sqrt((u ** 2).mean(-1, keepdims=True) + eps) * w


def unit(u):
    """unit vectors along the last axis"""
    return u / np.sqrt((u ** 2).sum(-1, keepdims=True) + 1e-6)


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, z)


def rotate_halves(u, rot, positions):
    """u [T, heads, n]: coordinate i < dims/2 turns with coordinate i + dims/2 by the angle positions * base^(-2i/dims); the rest pass"""
    dims = int(rot["dims"])
    half = dims // 2
    out = u.copy()
    for i in range(half):
        a = positions * float(rot["base"]) ** (-2.0 * i / dims)
        c, s = np.cos(a)[:, None], np.sin(a)[:, None]
        p, q = u[..., i], u[..., i + half]
        out[..., i] = p * c - q * s
        out[..., i + half] = q * c + p * s
    return out


def conv_silu(u, taps):
    """u [T, C], taps [C, K], the last tap is the present token's: causal, zeros before the start"""
    T, K = u.shape[0], taps.shape[1]
    out = np.zeros_like(u)
    for t in range(T):
        for j in range(K):
            src = t - (K - 1 - j)
            if src >= 0:
                out[t] += taps[:, j] * u[src]
    return silu(out)


def attention(m, w, p, h, eps):
    """causal grouped-query softmax attention; q and k normed over their whole projection before they are split into heads"""
    T = h.shape[0]
    H, G, D, VD = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    pos = np.arange(T, dtype=np.float64)
    q = rms_norm(h @ w[p + "q"].T, w[p + "q.norm"], eps).reshape(T, H, D)
    k = rms_norm(h @ w[p + "k"].T, w[p + "k.norm"], eps).reshape(T, G, D)
    v = (h @ w[p + "v"].T).reshape(T, G, VD)
    if m.get("rot"):
        q, k = rotate_halves(q, m["rot"], pos), rotate_halves(k, m["rot"], pos)
    gate = sigmoid(h @ w[p + "g"].T)
    out = np.zeros((T, H, VD))
    for head in range(H):
        g = head // (H // G)
        for i in range(T):
            s = (k[:i + 1, g] @ q[i, head]) * m["scale"]
            if m.get("softcap"):
                s = m["softcap"] * np.tanh(s / m["softcap"])
            sink = w[p + "sink"][head]
            mx = max(s.max(), sink)
            e = np.exp(s - mx)
            out[i, head] = (e / (e.sum() + math.exp(sink - mx))) @ v[:i + 1, g] * gate[i, head]
    return out.reshape(T, H * VD) @ w[p + "o"].T


def decay(m, w, p, h):
    """[T, H, D]: the factor every key channel's row of the state is multiplied by before a token's write"""
    T, H, D = h.shape[0], m["heads"], m["dim"]
    rate = np.exp(w[p + "A_log"])[None, :, None]
    if p + "a1" in w:
        z = (h @ w[p + "a1"].T @ w[p + "a2"].T + w[p + "dt_bias"]).reshape(T, H, D)
    else:
        z = np.repeat((h @ w[p + "a"].T + w[p + "dt_bias"])[:, :, None], D, axis=2)
    return np.exp(-rate * softplus(z))


def output_gate(m, w, p, h):
    T, H, VD = h.shape[0], m["heads"], m["vdim"]
    if p + "g1" in w:
        return sigmoid(h @ w[p + "g1"].T @ w[p + "g2"].T).reshape(T, H, VD)
    return silu(h @ w[p + "g"].T).reshape(T, H, VD)


def delta_recurrence(q, k, v, beta, g, state=None):
    """q, k [T, H, D], v [T, H, VD], beta [T, H], g [T, H, D] -> outputs [T, H, VD] and the state [H, D, VD]"""
    T, H, D = q.shape
    S = np.zeros((H, D, v.shape[2])) if state is None else state.copy()
    out = np.zeros(v.shape)
    for t in range(T):
        for a in range(H):
            S[a] *= g[t, a][:, None]
            u = beta[t, a] * (v[t, a] - S[a].T @ k[t, a])
            S[a] += np.outer(k[t, a], u)
            out[t, a] = S[a].T @ q[t, a]
    return out, S


def delta_rule(m, w, p, h, eps):
    T = h.shape[0]
    H, G, D, VD = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = unit(conv_silu(h @ w[p + "q"].T, w[p + "q.conv"]).reshape(T, G, D)) / math.sqrt(D)
    k = unit(conv_silu(h @ w[p + "k"].T, w[p + "k.conv"]).reshape(T, G, D))
    v = conv_silu(h @ w[p + "v"].T, w[p + "v.conv"]).reshape(T, H, VD)
    head = np.arange(H) // (H // G)
    o, _ = delta_recurrence(q[:, head], k[:, head], v, sigmoid(h @ w[p + "b"].T), decay(m, w, p, h))
    o = rms_norm(o, w[p + "norm"], eps) * output_gate(m, w, p, h)
    return o.reshape(T, H * VD) @ w[p + "o"].T


def parallel(m, w, p, h, eps):
    a = rms_norm(attention(m["left"], w, p + "left.", h, eps), w[p + "left.out"], eps)
    b = rms_norm(delta_rule(m["right"], w, p + "right.", h, eps), w[p + "right.out"], eps)
    return 0.5 * (a + b)


def dense_ff(w, p, h):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def forward(cfg, weights, tokens, trace=None):
    """logits [T, vocab] of a sequence from its start; trace (a list) receives the residual after every layer"""
    w = {k: np.asarray(v, np.float64) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][np.asarray(tokens, np.int64)]
    for i, L in enumerate(cfg["layers"]):
        p = f"l{i}."
        mix = {"delta": delta_rule, "parallel": parallel}[L["type"]]
        x = x + rms_norm(mix(L["mixer"], w, p + "mix.", x, eps), w[p + "norm1"], eps)
        if L.get("mlp"):
            x = x + rms_norm(dense_ff(w, p + "mlp.", x), w[p + "norm2"], eps)
        if trace is not None:
            trace.append(x.copy())
    return rms_norm(x, w["final.norm"], eps) @ w["head"].T
