"""A plain, slow implementation of the Kifunex design: numpy, float64, whole sequences, no cache, one function per
mechanism.  It shares no code with the library; the tests compare the engine against it.

A model is (config, tensors): ``config`` is the dictionary that config.json holds and ``tensors`` maps tensor names
to float64 arrays.  Linear weights are [out, in] and applied as W x.

    stream:     S copies x_1 .. x_S of the embedding's row; a sublayer f with its norm n and constants (a, b, M):
                y = f(n(sum_s a_s x_s));  x_t <- sum_s M[s, t] x_s + b_t y;  the end reads the sum of the copies
    norm:       tanh(alpha v) * w + b                                              no statistics
    mixer:      attention over a window, the values being the keys before their rotation
    ff:         experts chosen by sigmoid scores + a correction, weighted by the scores alone, and a shared expert
    weights_of: a layer that runs another layer's tensors again
"""
from __future__ import annotations

import numpy as np


def sigmoid(v):
    return np.where(v >= 0, 1.0 / (1.0 + np.exp(-np.abs(v))), np.exp(-np.abs(v)) / (1.0 + np.exp(-np.abs(v))))


def silu(v):
    return v * sigmoid(v)


def dynamic_tanh(v, t, name):
    return np.tanh(t[name + ".alpha"] * v) * t[name] + t[name + ".b"]


def gather_streams(x, weights):
    """x [T, S, width] -> [T, width]: the weighted sum over the copies that a sublayer reads."""
    return np.einsum("tsd,s->td", x, weights)


def spread_update(x, y, mix, out):
    """The copies after a sublayer: new copy ``to`` = sum over ``fr`` of mix[fr, to] x_fr, plus out[to] y."""
    new = np.zeros_like(x)
    count = x.shape[1]
    for to in range(count):
        for fr in range(count):
            new[:, to] += mix[fr, to] * x[:, fr]
        new[:, to] += out[to] * y
    return new


def rotation_frequencies(dims, base, scaling=None):
    """base^(-2i/dims), i < dims/2.  ``scaling`` {factor, low, high, original}: a frequency whose wavelength is below
    original/high stays, one above original/low is divided by factor, and in between the two are blended."""
    freq = []
    for i in range(dims // 2):
        f = float(base) ** (-2.0 * i / dims)
        if scaling:
            length = 2.0 * np.pi / f
            if length > scaling["original"] / scaling["low"]:
                f = f / scaling["factor"]
            elif not length < scaling["original"] / scaling["high"]:
                share = (scaling["original"] / length - scaling["low"]) / (scaling["high"] - scaling["low"])
                f = (1.0 - share) * f / scaling["factor"] + share * f
        freq.append(f)
    return np.array(freq)


def rotate_halves(v, positions, freq):
    """v [T, heads, dim]: with n frequencies, entry i < n of every head is paired with entry i + n and the pair is
    turned by position * freq[i].  Entries from 2n on stay."""
    out = v.copy()
    n = len(freq)
    angle = np.asarray(positions, dtype=np.float64)[:, None] * freq[None, :]
    cos, sin = np.cos(angle)[:, None, :], np.sin(angle)[:, None, :]
    a, b = v[..., :n], v[..., n:2 * n]
    out[..., :n] = a * cos - b * sin
    out[..., n:2 * n] = b * cos + a * sin
    return out


def windowed_attention(q, k, v, *, scale, window=None, positions=None):
    """q [R, H, dim] at ``positions`` (default: row r is position r) over k [T, G, dim], v [T, G, vdim]; the query at i
    sees j with 0 <= i - j < window (None: every j <= i)."""
    rows, heads = q.shape[0], q.shape[1]
    per = heads // k.shape[1]
    out = np.zeros((rows, heads, v.shape[2]))
    for r in range(rows):
        i = r if positions is None else int(positions[r])
        first = max(0, i - window + 1) if window else 0
        for g in range(k.shape[1]):
            heads_of = slice(g * per, (g + 1) * per)
            s = (q[r, heads_of] @ k[first:i + 1, g].T) * scale
            w = np.exp(s - s.max(axis=1, keepdims=True))
            out[r, heads_of] = (w / w.sum(axis=1, keepdims=True)) @ v[first:i + 1, g]
    return out


def attention_mixer(h, t, p, m):
    count = h.shape[0]
    q = (h @ t[p + "q"].T).reshape(count, m["heads"], m["dim"])
    k = (h @ t[p + "k"].T).reshape(count, m["kv_heads"], m["dim"])
    v = k.copy()                                        # the values: keys as projected, before the rotation
    rot = m.get("rot") or {}
    if rot.get("dims"):
        freq = rotation_frequencies(rot["dims"], rot["base"], rot.get("scaling"))
        q, k = rotate_halves(q, np.arange(count), freq), rotate_halves(k, np.arange(count), freq)
    o = windowed_attention(q, k, v, scale=m["scale"], window=(m.get("mask") or {}).get("size"))
    return o.reshape(count, -1) @ t[p + "o"].T


def gated_unit(h, t, p):
    return (silu(h @ t[p + "gate"].T) * (h @ t[p + "up"].T)) @ t[p + "down"].T


def choose_experts(scores, correction, top, scale):
    """scores [E]: the ``top`` largest of scores + correction (ties to the lower index); their weights are the scores
    without the correction, times scale, whatever their sum."""
    ids = np.argsort(-(scores + correction), kind="stable")[:top]
    return ids, scores[ids] * scale


def experts_ff(h, t, p, mlp, forced=None, routes=None):
    """``forced`` [T, top] replaces the choice (weights still from the scores); ``routes`` collects the choice."""
    r = mlp["router"]
    scale = r.get("scale", 1.0)
    scores = sigmoid(h @ t[p + "router"].T)
    out = np.zeros_like(h)
    chosen = np.zeros((h.shape[0], r["top"]), dtype=np.int64)
    for row in range(h.shape[0]):
        ids, weights = choose_experts(scores[row], t[p + "correction"], r["top"], scale)
        if forced is not None:
            ids = np.asarray(forced[row], dtype=np.int64)
            weights = scores[row][ids] * scale
        chosen[row] = ids
        for e, w in zip(ids, weights):
            out[row] += w * gated_unit(h[row], t, f"{p}e{int(e)}.")
    if routes is not None:
        routes.append(chosen)
    if mlp.get("shared"):
        out = out + gated_unit(h, t, p + "shared.")
    return out


def choice_margin(h, t, p, mlp):
    """Per row, the distance between the last choice score that won and the first that lost."""
    r = mlp["router"]
    if r["top"] >= r["experts"]:
        return np.full(h.shape[0], np.inf)
    ordered = -np.sort(-(sigmoid(h @ t[p + "router"].T) + t[p + "correction"]), axis=1)
    return ordered[:, r["top"] - 1] - ordered[:, r["top"]]


def owner(config, index):
    """The layer whose tensors layer ``index`` runs."""
    while config["layers"][index].get("weights_of") is not None:
        index = config["layers"][index]["weights_of"]
    return index


def forward(config, t, ids, streams=None, forced_routes=None, routes=None):
    """Logits [T, vocab]; ``streams`` (a list) gets the sum of the copies after every layer; ``forced_routes``: per
    layer with experts an array [T, top] of experts to use; ``routes`` receives every such layer's choice."""
    x = np.repeat(t["embed"][np.asarray(ids, dtype=np.int64)][:, None, :], config["streams"], axis=1)
    routed = 0
    for index, layer in enumerate(config["layers"]):
        p = f"l{owner(config, index)}."
        h = dynamic_tanh(gather_streams(x, t[p + "hc1.in"]), t, p + "norm1")
        x = spread_update(x, attention_mixer(h, t, p + "mix.", layer["mixer"]), t[p + "hc1.mix"], t[p + "hc1.out"])
        if layer.get("mlp"):
            h = dynamic_tanh(gather_streams(x, t[p + "hc2.in"]), t, p + "norm2")
            forced = forced_routes[routed] if forced_routes is not None else None
            routed += 1
            x = spread_update(x, experts_ff(h, t, p + "mlp.", layer["mlp"], forced, routes), t[p + "hc2.mix"], t[p + "hc2.out"])
        if streams is not None:
            streams.append(x.sum(axis=1))
    logits = dynamic_tanh(x.sum(axis=1), t, "final.norm") @ t["head"].T * config.get("logit_scale", 1.0)
    cap = config.get("logit_softcap")
    return cap * np.tanh(logits / cap) if cap else logits
