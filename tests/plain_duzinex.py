"""A plain, slow implementation of the Duzinex design: numpy, float64, whole sequences, no cache, one function per
mechanism.  It shares no code with the library; the tests compare the engine against it.

A model is (config, tensors): ``config`` is the dictionary that config.json holds and ``tensors`` maps tensor names
to float64 arrays.  Linear weights are [out, in] and applied as W x.

    layer:      x <- x + mixer(shift(n1(x)));  x <- x + ff(n2(x))
    norm:       tanh(alpha v) * w + b                                              no statistics
    shift:      h_t + (h_(t-1) - h_t) * s, h_(-1) = 0                             on what the mixer reads
    mixers:     attention (two maps over shared values, their weighted difference) | retention | mingru
    ff:         W_down act(W_up h), act a cubic of row-normed powers
    loop:       a stretch of layers several times; the embedding's rows are added before every pass but the first
"""
from __future__ import annotations

import numpy as np


def sigmoid(v):
    return np.where(v >= 0, 1.0 / (1.0 + np.exp(-np.abs(v))), np.exp(-np.abs(v)) / (1.0 + np.exp(-np.abs(v))))


def silu(v):
    return v * sigmoid(v)


def rms_divide(v, eps):
    return v / np.sqrt(np.mean(v * v, axis=-1, keepdims=True) + eps)


def dynamic_tanh(v, t, name):
    return np.tanh(t[name + ".alpha"] * v) * t[name] + t[name + ".b"]


def token_shift(h, share):
    """h [T, width]: every row moves towards the row before it, entry by entry; the first one towards zero."""
    before = np.concatenate([np.zeros((1, h.shape[1])), h[:-1]], axis=0)
    return h + (before - h) * share


def rotate_neighbours(v, positions, dims, base):
    """v [T, heads, dim]: entries 2i and 2i + 1 (i < dims/2) of every head are a pair, turned by position *
    base^(-2i/dims).  Entries from ``dims`` on stay."""
    out = v.copy()
    i = np.arange(dims // 2)
    angle = np.asarray(positions, dtype=np.float64)[:, None] * (base ** (-2.0 * i / dims))[None, :]
    cos, sin = np.cos(angle)[:, None, :], np.sin(angle)[:, None, :]
    a, b = v[..., 0:dims:2], v[..., 1:dims:2]
    out[..., 0:dims:2] = a * cos - b * sin
    out[..., 1:dims:2] = b * cos + a * sin
    return out


def visible(i, window, keep_first):
    """Positions that the query at i sees: the last ``window`` (None: all) and the first ``keep_first``."""
    j = np.arange(i + 1)
    return j if window is None else j[(i - j < window) | (j < keep_first)]


def map_attention(q, k, v, *, scale, window=None, keep_first=0, softcap=None, positions=None):
    """One map: q [R, H, dim] at ``positions`` (default: row r is position r) over k [T, G, dim], v [T, G, vdim]."""
    rows, heads = q.shape[0], q.shape[1]
    per = heads // k.shape[1]
    out = np.zeros((rows, heads, v.shape[2]))
    for r in range(rows):
        i = r if positions is None else int(positions[r])
        seen = visible(i, window, keep_first)
        for head in range(heads):
            g = head // per
            s = (k[seen, g] @ q[r, head]) * scale
            if softcap:
                s = softcap * np.tanh(s / softcap)
            w = np.exp(s - s.max())
            out[r, head] = (w / w.sum()) @ v[seen, g]
    return out


def lambda_of(lq1, lk1, lq2, lk2, diff):
    return np.exp(np.sum(lq1 * lk1)) - np.exp(np.sum(lq2 * lk2)) + diff


def difference_of_maps(a1, a2, lam, diff, eps):
    return rms_divide(a1 - lam * a2, eps) * (1.0 - diff)


def attention_mixer(h, t, p, m, eps):
    count = h.shape[0]
    heads, kv, dim, vdim = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ t[p + "q"].T + t[p + "q.b"]).reshape(count, heads * 2, dim)
    k = (h @ t[p + "k"].T + t[p + "k.b"]).reshape(count, kv * 2, dim)
    v = (h @ t[p + "v"].T + t[p + "v.b"]).reshape(count, kv, vdim)
    rot = m.get("rot") or {}
    if rot.get("dims"):
        q = rotate_neighbours(q, np.arange(count), rot["dims"], rot["base"])
        k = rotate_neighbours(k, np.arange(count), rot["dims"], rot["base"])
    mask = m.get("mask") or {}
    args = dict(scale=m["scale"], window=mask.get("size"), keep_first=mask.get("keep_first", 0), softcap=m.get("softcap"))
    a1 = map_attention(q[:, 0::2], k[:, 0::2], v, **args)
    a2 = map_attention(q[:, 1::2], k[:, 1::2], v, **args)
    lam = lambda_of(t[p + "lq1"], t[p + "lk1"], t[p + "lq2"], t[p + "lk2"], m["diff"])
    o = difference_of_maps(a1, a2, lam, m["diff"], eps)
    return o.reshape(count, heads * vdim) @ t[p + "o"].T + t[p + "o.b"]


def retention(q, k, v, decay):
    """q, k [T, heads, dim], v [T, heads, vdim], decay [heads].  Per head, from S = 0 [dim, vdim]:
    S <- decay S + k v^T;  o = S^T q."""
    count, heads, dim = q.shape
    out = np.zeros((count, heads, v.shape[2]))
    for head in range(heads):
        s = np.zeros((dim, v.shape[2]))
        for t in range(count):
            s = decay[head] * s + np.outer(k[t, head], v[t, head])
            out[t, head] = s.T @ q[t, head]
    return out


def retention_mixer(h, t, p, m, eps):
    count = h.shape[0]
    heads, dim, vdim = m["heads"], m["dim"], m["vdim"]
    q = (h @ t[p + "q"].T).reshape(count, heads, dim)
    k = (h @ t[p + "k"].T).reshape(count, heads, dim) * dim ** -0.5
    v = (h @ t[p + "v"].T).reshape(count, heads, vdim)
    o = rms_divide(retention(q, k, v, m["decay"]), eps).reshape(count, heads * vdim)
    return (o * silu(h @ t[p + "g"].T)) @ t[p + "o"].T


def min_gru(z, u):
    """z (in 0..1) and u [T, width]: S <- (1 - z) S + z cand from S = 0, cand = u + 1/2 or sigmoid(u) by u's sign."""
    cand = np.where(u >= 0, u + 0.5, sigmoid(u))
    out = np.zeros_like(u)
    s = np.zeros(u.shape[1])
    for t in range(u.shape[0]):
        s = (1.0 - z[t]) * s + z[t] * cand[t]
        out[t] = s
    return out


def min_gru_mixer(h, t, p):
    z = sigmoid(h @ t[p + "z"].T + t[p + "z.b"])
    u = h @ t[p + "x"].T + t[p + "x.b"]
    return (min_gru(z, u) * silu(h @ t[p + "g"].T)) @ t[p + "o"].T


def poly_norm(z, act, eps):
    a, b, c, e = act
    return a * rms_divide(z, eps) + b * rms_divide(z ** 2, eps) + c * rms_divide(z ** 3, eps) + e


def feed_forward(h, t, p, eps):
    return poly_norm(h @ t[p + "up"].T, t[p + "act"], eps) @ t[p + "down"].T


def run_order(config):
    """(layer, whether the embedding's rows are added first) of every run."""
    count = len(config["layers"])
    loop = config.get("loop")
    if not loop:
        return [(i, False) for i in range(count)]
    order = [(i, False) for i in range(loop["start"])]
    for turn in range(loop["times"]):
        order += [(i, turn > 0 and i == loop["start"]) for i in range(loop["start"], loop["stop"])]
    return order + [(i, False) for i in range(loop["stop"], count)]


def forward(config, t, ids, streams=None):
    """Logits [T, vocab]; ``streams`` (a list) gets the stream after every layer run."""
    eps = config["norm"]["eps"]
    embedded = t["embed"][np.asarray(ids, dtype=np.int64)] * config["embedding"]["scale"]
    x = embedded
    for index, again in run_order(config):
        layer, p = config["layers"][index], f"l{index}."
        if again:
            x = x + embedded
        h = token_shift(dynamic_tanh(x, t, p + "norm1"), t[p + "shift"])
        if layer["type"] == "attention":
            x = x + attention_mixer(h, t, p + "mix.", layer["mixer"], eps)
        elif layer["type"] == "retention":
            x = x + retention_mixer(h, t, p + "mix.", layer["mixer"], eps)
        else:
            x = x + min_gru_mixer(h, t, p + "mix.")
        if layer.get("mlp"):
            x = x + feed_forward(dynamic_tanh(x, t, p + "norm2"), t, p + "mlp.", eps)
        if streams is not None:
            streams.append(x.copy())
    return dynamic_tanh(x, t, "final.norm") @ t["embed"].T
