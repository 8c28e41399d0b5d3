"""Plain statement of the Suborax layer stack in numpy: one function per mechanism, whole sequences, nothing cached.

A model is (config dict, {name: array}); the names are those of the checkpoint. Every function works in the dtype of its
inputs, so the same code serves as a float64 yardstick. Shares nothing with the package under test."""
import math

import numpy as np


def silu(z):
    e = np.exp(-np.abs(z))
    return z * np.where(z >= 0, 1.0 / (1.0 + e), e / (1.0 + e)).astype(z.dtype)


def unit_rms(x, eps):
    """x over the root of (its mean square + eps), along the last axis."""
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + x.dtype.type(eps))


def norm(x, w, eps):
    """The stored weight is the difference from 1."""
    return unit_rms(x, eps) * (1 + w)


def frequencies(rot):
    """One per rotated pair. With `scaling`, wavelengths above original / low turn `factor` times slower, those below
    original / high stay, and between the two the share of the original frequency grows linearly in original / wavelength."""
    f = [rot["base"] ** (-2.0 * i / rot["dims"]) for i in range(rot["dims"] // 2)]
    sc = rot.get("scaling")
    if not sc:
        return f
    out = []
    for x in f:
        wave = 2.0 * math.pi / x
        if wave < sc["original"] / sc["high"]:
            out.append(x)
        elif wave > sc["original"] / sc["low"]:
            out.append(x / sc["factor"])
        else:
            keep = (sc["original"] / wave - sc["low"]) / (sc["high"] - sc["low"])
            out.append((1.0 - keep) * x / sc["factor"] + keep * x)
    return out


def rotate(x, pos, rot):
    """Half-split rotation of the first rot["dims"] of the last axis; x [T, heads, d], pos [T]."""
    half = rot["dims"] // 2
    a = pos.astype(x.dtype)[:, None, None] * np.array(frequencies(rot), x.dtype)
    c, s = np.cos(a), np.sin(a)
    u, v = x[..., :half], x[..., half:2 * half]
    return np.concatenate([u * c - v * s, v * c + u * s, x[..., 2 * half:]], -1)


def cap(z, limit):
    return z if limit is None else z.dtype.type(limit) * np.tanh(z / z.dtype.type(limit))


def scores(q, k, scale, softcap):
    """q, k [T, H, d] -> [H, T, T], -inf above the diagonal."""
    s = cap(np.einsum("ihd,jhd->hij", q, k) * q.dtype.type(scale), softcap)
    return np.where(np.tril(np.ones((len(q), len(q)), bool)), s, -np.inf)


def softmax_with_sink(s, sink):
    """s [H, T, T]; exp(sink[h]) joins the denominator of every row and has no column."""
    top = np.maximum(s.max(-1), sink[:, None])
    e = np.exp(s - top[..., None])
    return e / (e.sum(-1) + np.exp(sink[:, None] - top))[..., None]


def spread(x, heads):
    """[T, G, d] -> [T, heads, d]: blocks of heads / G consecutive heads share one of the G."""
    return np.repeat(x, heads // x.shape[1], axis=1)


def attention(h, m, w, eps):
    T, H, G = len(h), m["heads"], m["kv_heads"]
    pos = np.arange(T)
    q = (h @ w["q"].T).reshape(T, H, m["dim"])
    k = (h @ w["k"].T).reshape(T, G, m["dim"])
    v = (h @ w["v"].T).reshape(T, G, m["vdim"])
    q, k = (unit_rms(rotate(x, pos, m["rot"]), eps) for x in (q, k))
    p = softmax_with_sink(scores(q, spread(k, H), m["scale"], m.get("softcap")), w["sink"])
    o = np.einsum("hij,jhd->ihd", p, spread(v, H))
    return o.reshape(T, H * m["vdim"]) @ w["o"].T


def feed_forward(h, w):
    return (silu(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


def layer(x, cfg, i, weights):
    """The norm comes after each sum, and the sublayers read the stream as it is."""
    eps, alpha, spec, p = cfg["norm"]["eps"], x.dtype.type(cfg["postln_alpha"]), cfg["layers"][i], f"l{i}."
    sub = lambda part: {n[len(p + part):]: a for n, a in weights.items() if n.startswith(p + part)}
    x = norm(alpha * x + attention(x, spec["mixer"], sub("mix."), eps), weights[p + "norm1"], eps)
    if spec.get("mlp"):
        x = norm(alpha * x + feed_forward(x, sub("mlp.")), weights[p + "norm2"], eps)
    return x


def forward(cfg, weights, tokens, dtype=np.float64, trace=None):
    """Logits [T, vocab] of the whole sequence; `trace`, a list, gets the residual stream after every layer."""
    w = {n: a.astype(dtype) for n, a in weights.items()}
    x = w["embed"][np.asarray(tokens)] * dtype(cfg["embedding"]["scale"])
    for i in range(len(cfg["layers"])):
        x = layer(x, cfg, i, w)
        if trace is not None:
            trace.append(x)
    return norm(x, w["final.norm"], cfg["norm"]["eps"]) @ w["head"].T


def greedy(cfg, weights, prompt, n, dtype=np.float64):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(np.argmax(forward(cfg, weights, toks, dtype)[-1])))
    return toks[len(prompt):]
