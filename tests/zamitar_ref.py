"""Plain statement of the Zamitar layer stack in numpy: one function per mechanism, whole sequences, nothing cached.

A model is (config dict, {name: array}); the names are those of the checkpoint. Every function works in the dtype of its
inputs, so the same code serves as a float64 yardstick. Shares nothing with the package under test."""
import numpy as np


def sigmoid(z):
    return np.where(z >= 0, 1.0 / (1.0 + np.exp(-np.abs(z))), np.exp(-np.abs(z)) / (1.0 + np.exp(-np.abs(z)))).astype(z.dtype)


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.maximum(z, 0) + np.log1p(np.exp(-np.abs(z)))


def linear(x, w, b=None):
    y = x @ w.T
    return y if b is None else y + b


def layer_norm(x, w, eps):
    d = x - x.mean(-1, keepdims=True)
    return d / np.sqrt((d * d).mean(-1, keepdims=True) + x.dtype.type(eps)) * w


def rms_norm(x, w, eps):
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + x.dtype.type(eps)) * w


def unit_norm(x):
    return x / np.sqrt((x * x).sum(-1, keepdims=True) + x.dtype.type(1e-6))


def causal_conv(x, taps):
    """x [T, C], taps [C, n]: y[t] = sum_j taps[:, j] x[t - (n - 1) + j], zeros before the start."""
    n = taps.shape[1]
    pad = np.concatenate([np.zeros((n - 1, x.shape[1]), x.dtype), x])
    return sum(pad[j:j + len(x)] * taps[:, j] for j in range(n))


def rotate(x, pos, base, dims):
    """Half-split rotation of the first `dims` of the last axis; x [T, ..., d], pos [T]."""
    half = dims // 2
    f = np.array([float(base) ** (-2.0 * i / dims) for i in range(half)], x.dtype)
    ang = (pos.astype(x.dtype)[:, None] * f).reshape((len(pos),) + (1,) * (x.ndim - 2) + (half,))
    c, s = np.cos(ang), np.sin(ang)
    u, v = x[..., :half], x[..., half:dims]
    return np.concatenate([u * c - v * s, v * c + u * s, x[..., dims:]], -1)


def delta_rule(q, k, v, g, beta):
    """q, k, g [T, H, D], v [T, H, V], beta [T, H] -> o [T, H, V]; the state starts at zero."""
    T, H, D = q.shape
    S = np.zeros((H, D, v.shape[2]), q.dtype)
    out = np.empty_like(v)
    for t in range(T):
        S = g[t][:, :, None] * S
        u = beta[t][:, None] * (v[t] - np.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out[t] = np.einsum("hdv,hd->hv", S, q[t])
    return out


def channel_delta(h, m, w, eps):
    """m: the mixer's sizes; w: name -> array (without the layer's prefix)."""
    T, H, KH, D, V = len(h), m["heads"], m["kv_heads"], m["dim"], m["vdim"]

    def branch(name, n):
        return silu(causal_conv(linear(h, w[name]), w[name + ".conv"])).reshape(T, n, -1)

    q, k, v = branch("q", KH), branch("k", KH), branch("v", H)
    rep = [i // (H // KH) for i in range(H)]
    q = (unit_norm(q) * q.dtype.type(D ** -0.5))[:, rep]
    k = unit_norm(k)[:, rep]
    beta = sigmoid(linear(h, w["b"]))
    rate = softplus(linear(linear(h, w["a1"]), w["a2"]) + w["dt_bias"]).reshape(T, H, D)
    g = np.exp(-np.exp(w["A_log"])[:, None] * rate)
    o = rms_norm(delta_rule(q, k, v, g, beta), w["norm"], eps)
    o = o * sigmoid(linear(linear(h, w["g1"]), w["g2"])).reshape(T, H, V)
    return linear(o.reshape(T, H * V), w["o"])


def sink_attention(q, k, v, scale, sink):
    """q [T, H, d], k [T, H, d], v [T, H, dv], causal; sink [H] joins the denominator only."""
    T = len(q)
    s = np.einsum("ihd,jhd->hij", q, k) * q.dtype.type(scale)
    s = np.where(np.tril(np.ones((T, T), bool)), s, -np.inf)
    top = np.maximum(s.max(-1), sink[:, None])
    e = np.exp(s - top[..., None])
    p = e / (e.sum(-1) + np.exp(sink[:, None] - top))[..., None]
    return np.einsum("hij,jhd->ihd", p, v)


def latent_attention(h, m, w, eps):
    T, H, D, R, V, C = len(h), m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = np.arange(T)
    rot = m["rot"]
    q = linear(rms_norm(linear(h, w["dq"]), w["dq.norm"], eps), w["uq"]).reshape(T, H, D + R)
    ckv = linear(h, w["dkv"])
    c = rms_norm(ckv[:, :C], w["dkv.norm"], eps)
    kr = rotate(ckv[:, C:], pos, rot["base"], rot["dims"])
    k = np.concatenate([linear(c, w["uk"]).reshape(T, H, D), np.repeat(kr[:, None], H, 1)], -1)
    q = np.concatenate([q[..., :D], rotate(q[..., D:], pos, rot["base"], rot["dims"])], -1)
    v = linear(c, w["uv"]).reshape(T, H, V)
    o = sink_attention(q, k, v, m["scale"], w["sink"]).reshape(T, H * V)
    return linear(o * sigmoid(linear(h, w["g"])), w["o"])


MIXERS = {"channel_delta": channel_delta, "latent_attention": latent_attention}


def gated_mlp(h, w):
    return linear(silu(linear(h, w["gate"], w["gate.b"])) * linear(h, w["up"], w["up.b"]), w["down"], w["down.b"])


def layer(x, cfg, i, weights):
    eps, spec, p = cfg["norm"]["eps"], cfg["layers"][i], f"l{i}."
    sub = lambda part: {n[len(p + part):]: a for n, a in weights.items() if n.startswith(p + part)}
    h = layer_norm(x, weights[p + "norm1"], eps)
    y = MIXERS[spec["type"]](h, spec["mixer"], sub("mix."), eps) * weights[p + "ls1"]
    if spec.get("mlp"):
        y = y + gated_mlp(h, sub("mlp.")) * weights[p + "ls2"]
    return x + y


def layer_runs(cfg):
    """[(layer, pass or None if outside the loop, first layer of its pass)] in the order they run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None, False) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    runs = [(i, None, False) for i in range(a)]
    for t in range(loop["times"]):
        runs += [(i, t, i == a) for i in range(a, b)]
    return runs + [(i, None, False) for i in range(b, n)]


def forward(cfg, weights, tokens, dtype=np.float64, trace=None):
    """Logits [T, vocab] of the whole sequence; `trace`, a list, gets the residual stream after every layer run."""
    w = {n: (a if a.dtype.kind == "i" else a.astype(dtype)) for n, a in weights.items()}
    emb = w["embed"][np.asarray(tokens)] * dtype(cfg["embedding"]["scale"])
    x = emb
    for i, t, first in layer_runs(cfg):
        if first:
            if t > 0:
                x = x + emb
            x = x + w["loop.step"][t]
        x = layer(x, cfg, i, w)
        if trace is not None:
            trace.append(x)
    return layer_norm(x, w["final.norm"], cfg["norm"]["eps"]) @ w["embed"].T


def greedy(cfg, weights, prompt, n, dtype=np.float64):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(np.argmax(forward(cfg, weights, toks, dtype)[-1])))
    return toks[len(prompt):]
