"""CPU checks of the Zamitar reference and of what surrounds the device code: the reference's pieces against other ways to
write them, the reach of the comparison (a planted mistake must show), the checkpoint container, configuration errors, the
packed layout."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import zamitar_models as zm
import zamitar_ref as ref
from alice_llm_b200 import registry, stack
from alice_llm_b200.safetensors_file import SafetensorsError, SafetensorsFile, bf16_to_f32, f32_to_bf16, write_safetensors

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
RNG = np.random.default_rng


def test_delta_rule_single_step_and_decay():
    """From a zero state one write is read back as (k.q) beta v; an idle token (beta 0) scales it by the decays."""
    rng = RNG(0)
    q, k, g = (rng.standard_normal((2, 3, 5)) for _ in range(3))
    v = rng.standard_normal((2, 3, 4))
    beta = np.array([[0.3, 0.5, 1.0], [0.0, 0.0, 0.0]])
    o = ref.delta_rule(q, k, v, g, beta)
    assert np.allclose(o[0], np.einsum("hd,hd->h", k[0], q[0])[:, None] * beta[0][:, None] * v[0])
    assert np.allclose(o[1], np.einsum("hd,hd->h", g[1] * k[0], q[1])[:, None] * beta[0][:, None] * v[0])


def test_delta_rule_recalls_orthogonal_keys():
    """beta 1, no decay, orthonormal keys: every value comes back exactly, and a rewrite replaces it."""
    k = np.eye(4)[[0, 1, 2, 3, 1]][:, None]
    v = RNG(1).standard_normal((5, 1, 3))
    o = ref.delta_rule(k.copy(), k, v, np.ones_like(k), np.ones((5, 1)))
    assert np.allclose(o, v)
    q = np.broadcast_to(np.eye(4)[1], (5, 1, 4)).copy()
    assert np.allclose(ref.delta_rule(q, k, v, np.ones_like(k), np.ones((5, 1)))[4], v[4])


def test_sink_attention_equals_an_extra_key_of_value_zero():
    rng = RNG(2)
    q, k, v, sink = rng.standard_normal((6, 2, 5)), rng.standard_normal((6, 2, 5)), rng.standard_normal((6, 2, 3)), rng.standard_normal(2)
    got = ref.sink_attention(q, k, v, 0.4, sink)
    for i in range(6):
        for h in range(2):
            s = np.append(k[:i + 1, h] @ q[i, h] * 0.4, sink[h])
            p = np.exp(s - s.max())
            p /= p.sum()
            assert np.allclose(got[i, h], p[:-1] @ v[:i + 1, h])


def test_rotation_depends_on_distance_only_and_keeps_the_rest():
    rng = RNG(3)
    a, b = rng.standard_normal((1, 12)), rng.standard_normal((1, 12))
    dot = lambda p, s: float((ref.rotate(a, np.array([p]), 100.0, 8) * ref.rotate(b, np.array([s]), 100.0, 8)).sum())
    assert abs(dot(9, 4) - dot(105, 100)) < 1e-9 and abs(dot(9, 4) - dot(9, 5)) > 1e-3
    assert np.array_equal(ref.rotate(a, np.array([7]), 100.0, 8)[0, 8:], a[0, 8:])


def test_convolution_and_norms():
    x, w = RNG(4).standard_normal((7, 3)), RNG(5).standard_normal((3, 4))
    y = ref.causal_conv(x, w)
    for t in range(7):
        assert np.allclose(y[t], sum(w[:, 3 - j] * x[t - j] for j in range(4) if t >= j))
    h = ref.layer_norm(x, np.ones(3), 0.0)
    assert np.allclose(h.mean(1), 0) and np.allclose(h.var(1), 1)
    assert np.allclose((ref.rms_norm(x, np.ones(3), 0.0) ** 2).mean(1), 1)


def test_prefix_property():
    """Logits of a prefix do not depend on what follows."""
    w, toks = zm.floats(zm.weights(zm.MIXED)), RNG(6).integers(0, 131, 20)
    assert np.allclose(ref.forward(zm.MIXED, w, toks)[:9], ref.forward(zm.MIXED, w, toks[:9]), atol=1e-10)


def _forward_with(monkeypatch, cfg, w, toks, **patches):
    with monkeypatch.context() as m:
        for name, fn in patches.items():
            if name in ref.MIXERS:
                m.setitem(ref.MIXERS, name, fn)
            else:
                m.setattr(ref, name, fn)
        return ref.forward(cfg, w, toks)


def test_planted_mistakes_show_in_the_logits(monkeypatch):
    """What the device tests compare would notice each of these by more than their tolerances (1e-4 in 32 bits, 0.03 in bf16)."""
    cfg, toks = zm.MIXED, RNG(7).integers(0, 131, 60)
    w = zm.floats(zm.weights(cfg, peaky=3.0))
    good = ref.forward(cfg, w, toks)

    def worst(bad):
        return zm.row_errors(bad, good).max()

    def repeat_tiled(h, m, ww, eps):
        # key heads dealt out in turn instead of in blocks
        H, K, V = m["heads"], m["kv_heads"], m["vdim"]
        order = [i for k in range(K) for i in range(H) if i % K == k]
        ww = dict(ww)
        pick = lambda a, n: a.reshape(H, n, *a.shape[1:])[order].reshape(a.shape)
        for n in ("v", "v.conv", "g2"):
            ww[n] = pick(ww[n], V)
        for n in ("a2", "dt_bias"):
            ww[n] = pick(ww[n], m["dim"])
        ww["b"], ww["A_log"] = ww["b"][order], ww["A_log"][order]
        ww["o"] = ww["o"].reshape(-1, H, V)[:, order].reshape(ww["o"].shape)
        return ref.channel_delta(h, m, ww, eps)

    def read_before_write(q, k, v, g, beta):
        return ref_delta(q, k, v, g, beta) - np.einsum("thd,thd->th", k, q)[..., None] * _writes(q, k, v, g, beta)

    def _writes(q, k, v, g, beta):
        T, H, D = q.shape
        S, out = np.zeros((H, D, v.shape[2])), np.empty_like(v)
        for t in range(T):
            S = g[t][:, :, None] * S
            out[t] = beta[t][:, None] * (v[t] - np.einsum("hdv,hd->hv", S, k[t]))
            S = S + k[t][:, :, None] * out[t][:, None, :]
        return out

    ref_delta, ref_conv, ref_rot, ref_sink = ref.delta_rule, ref.causal_conv, ref.rotate, ref.sink_attention
    mistakes = {
        "no sink": dict(sink_attention=lambda q, k, v, s, sink: ref_sink(q, k, v, s, np.full_like(sink, -1e9))),
        "sink scaled": dict(sink_attention=lambda q, k, v, s, sink: ref_sink(q, k, v, s, sink * s)),
        "first key unseen": dict(sink_attention=lambda q, k, v, s, sink: np.concatenate([ref_sink(q, k, v, s, sink)[:1], ref_sink(q[1:], k[1:], v[1:], s, sink)])),
        "taps reversed": dict(causal_conv=lambda x, t: ref_conv(x, t[:, ::-1])),
        "convolution sees no past": dict(causal_conv=lambda x, t: x * t[:, -1]),
        "read before write": dict(delta_rule=read_before_write),
        "no decay": dict(delta_rule=lambda q, k, v, g, b: ref_delta(q, k, v, np.ones_like(g), b)),
        "one decay per head": dict(delta_rule=lambda q, k, v, g, b: ref_delta(q, k, v, np.broadcast_to(g.mean(-1, keepdims=True), g.shape), b)),
        "rotation off by one": dict(rotate=lambda x, p, base, d: ref_rot(x, p + (x.ndim == 3), base, d)),
        "key heads dealt in turn": dict(channel_delta=repeat_tiled),
    }
    for name, patch in mistakes.items():
        err = worst(_forward_with(monkeypatch, cfg, w, toks, **patch))
        assert err > 0.05, (name, err)
    no_emb = dict(w)
    no_emb["loop.step"] = np.zeros_like(w["loop.step"])
    assert worst(ref.forward(cfg, no_emb, toks)) > 0.1
    fewer = json.loads(json.dumps(cfg))
    fewer["loop"]["times"] = 2
    assert worst(ref.forward(fewer, w, toks)) > 0.1


def test_safetensors_round_trip_and_errors(tmp_path):
    p = str(tmp_path / "m.safetensors")
    t = {"a": f32_to_bf16(RNG(8).standard_normal((3, 5)).astype(np.float32)), "b": np.arange(4, dtype=np.int32), "c": np.float32([[1.5]])}
    write_safetensors(p, t)
    f = SafetensorsFile(p)
    assert set(f.names()) == {"a", "b", "c"} and all(np.array_equal(f.get(n), t[n]) and f.get(n).dtype == t[n].dtype for n in t)
    with pytest.raises(SafetensorsError, match="missing"):
        f.get("d")
    raw = open(p, "rb").read()
    for bad in (raw[:4], raw[:-1], b"\xff" * 8 + raw[8:], raw[:8] + b"x" + raw[9:], raw.replace(b'"I32"', b'"U32"')):
        q = str(tmp_path / "bad.safetensors")
        open(q, "wb").write(bad)
        with pytest.raises(SafetensorsError):
            SafetensorsFile(q)


def test_bf16_rounding_is_nearest_even():
    x = np.float32([1.0, 1.00390625, 1.01171875, -3.1415927, 1e-30])
    import torch
    assert np.array_equal(f32_to_bf16(x), torch.tensor(x).bfloat16().view(torch.int16).numpy().view(np.uint16))
    assert np.array_equal(bf16_to_f32(f32_to_bf16(bf16_to_f32(f32_to_bf16(x)))), bf16_to_f32(f32_to_bf16(x)))


def test_config_errors():
    good = zm.MIXED
    stack.StackConfig(good, 8)

    def bad(edit, match):
        c = json.loads(json.dumps(good))
        edit(c)
        with pytest.raises(stack.ConfigError, match=match):
            stack.StackConfig(c, 8)

    bad(lambda c: c["layers"][0].update(type="window_attention"), "window_attention")
    bad(lambda c: c["layers"][1]["mixer"].update(heads=5), "divide")
    bad(lambda c: c["layers"][0]["mixer"].pop("kv_rank"), "kv_rank")
    bad(lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7), "rotated")
    bad(lambda c: c["layers"][0]["mlp"].update(kind="experts"), "experts")
    bad(lambda c: c["loop"].update(stop=9), "loop")
    bad(lambda c: c.update(layers=[]), "layers")
    bad(lambda c: c.update(width=0), "width")


def test_tensor_shapes_are_checked():
    cfg = stack.StackConfig(zm.MIXED, 8)
    w = zm.weights(zm.MIXED)
    for name, change in (("l0.mix.uq", lambda a: a[:-1]), ("l1.mix.a2", lambda a: a[:, :-1]), ("l1.mix.q.conv", lambda a: a[:, 1:]),
                         ("l0.mlp.gate.b", lambda a: a[1:]), ("l3.ls1", None)):
        t = dict(w)
        if change:
            t[name] = change(t[name])
        else:
            del t[name]
        with pytest.raises(stack.ConfigError, match=name.replace(".", r"\.")):
            for i, L in enumerate(cfg.layers):
                stack.pack_layer(stack.Checkpoint(t), i, L, cfg)


@pytest.mark.parametrize("name", zm.MODELS)
def test_packed_layers_hold_every_weight(name):
    """Segments where the header says they are, zeros elsewhere."""
    d = zm.MODELS[name]
    cfg, w = stack.StackConfig(d, 8), zm.weights(d)
    for i, L in enumerate(cfg.layers):
        mats, vecs = stack.pack_layer(stack.Checkpoint(w), i, L, cfg)
        at, seen = 0, 0
        for n, rows in L.input_segments():
            seg = mats["in"][at:at + rows, :cfg.width]
            assert np.array_equal(seg, w[f"l{i}.mix.{n}"])
            seen += np.count_nonzero(seg)
            at += stack.pad(rows)
        assert np.count_nonzero(mats["in"]) == seen and all(s % 64 == 0 for s in mats["in"].shape)
        if L.ff:
            g = mats["gu"].reshape(-1, 2, 64, mats["gu"].shape[1])
            assert np.array_equal(g[:, 0].reshape(-1, g.shape[-1])[:L.ff, :cfg.width], w[f"l{i}.mlp.gate"])
            assert np.array_equal(g[:, 1].reshape(-1, g.shape[-1])[:L.ff, :cfg.width], w[f"l{i}.mlp.up"])
        if L.kind == stack.MIX_DELTA:
            dp = stack.delta_dim(L.dim)
            a2 = mats["a2"].reshape(L.heads, dp, -1)
            assert np.array_equal(a2[:, :L.dim, :L.decay_rank].reshape(L.heads * L.dim, -1), w[f"l{i}.mix.a2"])
            assert vecs["conv"].shape == (L.conv_taps, sum(stack.pad(r) for _, r in L.input_segments()[:3]))


def test_registry_refuses_unknown_architectures(tmp_path):
    (tmp_path / "config.json").write_text(json.dumps({"architecture": "Nothing"}))
    with pytest.raises(ValueError, match="Nothing"):
        registry.lookup(str(tmp_path))
    (tmp_path / "config.json").write_text(json.dumps({"architecture": "Zamitar"}))
    assert registry.lookup(str(tmp_path))[1] == "stack"


def test_trace_runner_without_a_device(tmp_path):
    """It fails at once, with the library's message, where there is no GPU."""
    import torch
    if torch.cuda.is_available():
        pytest.skip("a CUDA device is present")
    w = zm.weights(zm.ODD)
    write_safetensors(str(tmp_path / "model.safetensors"), w)
    (tmp_path / "config.json").write_text(json.dumps(zm.ODD))
    r = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path), "--out", str(tmp_path)], input="",
                       capture_output=True, text=True, timeout=600)
    assert r.returncode == 1 and "no CPU path" in r.stderr
