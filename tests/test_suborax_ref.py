"""CPU checks of the Suborax reference and of what surrounds the device code: the reference's pieces against other ways to write
them, the reach of the comparison (a planted mistake must show), configuration errors, the packed layout."""
import copy
import json
import math

import numpy as np
import pytest

import suborax_models as sm
import suborax_ref as ref
from alice_llm_b200 import registry, stack

RNG = np.random.default_rng


def test_softmax_with_sink_equals_an_extra_column():
    rng = RNG(0)
    s, sink = rng.standard_normal((2, 5, 5)) * 3, rng.standard_normal(2)
    s = np.where(np.tril(np.ones((5, 5), bool)), s, -np.inf)
    got = ref.softmax_with_sink(s, sink)
    for h in range(2):
        for i in range(5):
            e = np.exp(np.append(s[h, i], sink[h]))
            assert np.allclose(got[h, i], e[:-1] / e.sum())
    assert np.allclose(ref.softmax_with_sink(s, np.full(2, -np.inf)).sum(-1), 1)


def test_scores_are_capped_and_causal():
    rng = RNG(1)
    q, k = rng.standard_normal((6, 2, 4)) * 9, rng.standard_normal((6, 2, 4)) * 9
    s = ref.scores(q, k, 0.7, 5.0)
    for h in range(2):
        for i in range(6):
            for j in range(6):
                assert s[h, i, j] == -np.inf if j > i else abs(s[h, i, j] - 5 * math.tanh(float(q[i, h] @ k[j, h]) * 0.7 / 5)) < 1e-12
    assert np.abs(s[np.isfinite(s)]).max() <= 5 and np.abs(ref.scores(q, k, 0.7, None)[np.isfinite(s)]).max() > 5


def test_frequencies_at_the_edges_of_the_scaled_range():
    """Frequencies whose wavelengths lie on, inside and outside both edges; continuous across them."""
    sc = dict(factor=8.0, low=1.0, high=4.0, original=1000.0)

    def scaled(wave):
        # dims 4, so that the second pair has frequency base ** -0.5
        base = (wave / (2 * math.pi)) ** 2
        return ref.frequencies(dict(base=base, dims=4, scaling=sc))[1] * wave / (2 * math.pi)

    assert abs(scaled(249.0) - 1) < 1e-12 and abs(scaled(1001.0) - 1 / 8) < 1e-12
    assert abs(scaled(250.01) - 1) < 1e-3 and abs(scaled(999.9) - 1 / 8) < 1e-3
    assert abs(scaled(400.0) - ((1 - 0.5) / 8 + 0.5)) < 1e-12      # 1000 / 400 lies half way between 1 and 4
    assert ref.frequencies(dict(base=100.0, dims=4)) == [1.0, 0.1]


def test_rotation_depends_on_distance_only_and_keeps_the_rest():
    rng = RNG(2)
    a, b, rot = rng.standard_normal((1, 1, 12)), rng.standard_normal((1, 1, 12)), dict(base=100.0, dims=8, scaling=sm.scaling())
    dot = lambda p, s: float((ref.rotate(a, np.array([p]), rot) * ref.rotate(b, np.array([s]), rot)).sum())
    assert abs(dot(9, 4) - dot(105, 100)) < 1e-9 and abs(dot(9, 4) - dot(9, 5)) > 1e-3
    assert np.array_equal(ref.rotate(a, np.array([7]), rot)[..., 8:], a[..., 8:])
    assert np.allclose(ref.unit_rms(ref.rotate(a, np.array([7]), rot), 0.0), ref.rotate(ref.unit_rms(a, 0.0), np.array([7]), rot))


def test_norms_and_heads():
    x = RNG(3).standard_normal((7, 5))
    assert np.allclose((ref.unit_rms(x, 0.0) ** 2).mean(-1), 1)
    assert np.allclose(ref.unit_rms(np.zeros((1, 4)), 1e-3), 0) and np.allclose(ref.unit_rms(np.full((1, 4), 1e-2), 1e-4), 0.5 ** 0.5)
    assert np.allclose(ref.norm(x, np.zeros(5), 1e-3), ref.unit_rms(x, 1e-3))
    assert list(ref.spread(np.arange(3)[None, :, None], 6)[0, :, 0]) == [0, 0, 1, 1, 2, 2]


def test_prefix_property():
    """Logits of a prefix do not depend on what follows."""
    w, toks = sm.floats(sm.weights(sm.MIXED)), RNG(6).integers(0, 131, 20)
    assert np.allclose(ref.forward(sm.MIXED, w, toks)[:9], ref.forward(sm.MIXED, w, toks[:9]), atol=1e-10)


def test_planted_mistakes_show_in_the_logits(monkeypatch):
    """What the device tests compare would notice each of these by more than their tolerances (1e-4 in 32 bits, 0.03 in bf16)."""
    cfg, toks = sm.MIXED, RNG(7).integers(0, 131, 90)
    w = sm.floats(sm.weights(cfg))
    good = ref.forward(cfg, w, toks)
    r_rot, r_soft, r_scores, r_unit, r_freq, r_norm = ref.rotate, ref.softmax_with_sink, ref.scores, ref.unit_rms, ref.frequencies, ref.norm

    def first_key_unseen(q, k, scale, softcap):
        s = r_scores(q, k, scale, softcap)
        s[:, 1:, 0] = -np.inf
        return s

    def own_key_unseen(q, k, scale, softcap):
        s = r_scores(q, k, scale, softcap)
        i = np.arange(1, len(q))
        s[:, i, i] = -np.inf
        return s

    def interleaved(x, pos, rot):
        d, h = rot["dims"], rot["dims"] // 2
        order = np.concatenate([np.arange(0, d, 2), np.arange(1, d, 2)])
        y = r_rot(np.concatenate([x[..., order], x[..., d:]], -1), pos, rot)
        return np.concatenate([y[..., :d][..., np.argsort(order)], y[..., d:]], -1)

    mistakes = {
        "no sink": dict(softmax_with_sink=lambda s, sink: r_soft(s, np.full_like(sink, -np.inf))),
        "sink scaled": dict(softmax_with_sink=lambda s, sink: r_soft(s, sink * 0.5)),
        "sink capped": dict(softmax_with_sink=lambda s, sink: r_soft(s, ref.cap(sink, 1.0))),
        "sink counted twice": dict(softmax_with_sink=lambda s, sink: r_soft(s, sink + np.log(2.0))),
        "no cap": dict(cap=lambda z, limit: z),
        "cap clipped": dict(cap=lambda z, limit: np.clip(z, -limit, limit)),
        "scale inside the cap only": dict(scores=lambda q, k, scale, c: r_scores(q, k, scale, c) / scale),
        "first key unseen": dict(scores=first_key_unseen),
        "own key unseen": dict(scores=own_key_unseen),
        "queries off by one": dict(rotate=lambda x, p, rot: r_rot(x, p + (x.shape[1] % 2 == 0), rot)),
        "pairs side by side": dict(rotate=interleaved),
        "rotation of the whole head": dict(rotate=lambda x, p, rot: r_rot(x, p, dict(rot, dims=x.shape[2] // 2 * 2))),
        "frequencies not scaled": dict(frequencies=lambda rot: r_freq(dict(rot, scaling=None))),
        "heads dealt in turn": dict(spread=lambda x, heads: np.concatenate([x] * (heads // x.shape[1]), 1)),
        "queries and keys not normalised": dict(unit_rms=lambda x, eps: x if x.ndim == 3 else r_unit(x, eps)),
        "norm weight around one": dict(norm=lambda x, ww, eps: r_norm(x, ww - 1, eps)),
    }
    for name, patch in mistakes.items():
        with monkeypatch.context() as m:
            for k, fn in patch.items():
                m.setattr(ref, k, fn)
            err = sm.row_errors(ref.forward(cfg, w, toks), good).max()
        assert err > 0.05, (name, err)
    # the first norm takes the embedding's scale out again but for eps: only a large one shows it (GPU tests have such a model)
    big = dict(cfg, norm={"eps": 0.5})
    for name, a, b in (("alpha", cfg, dict(postln_alpha=1.0)), ("eps", cfg, big), ("embedding scale", big, dict(embedding={"scale": 0.2}))):
        err = sm.row_errors(ref.forward(dict(a, **b), w, toks), ref.forward(a, w, toks)).max()
        assert err > 0.05, (name, err)


def test_config_errors():
    stack.StackConfig(sm.MIXED, 8)

    def bad(edit, match):
        c = copy.deepcopy(sm.MIXED)
        edit(c)
        with pytest.raises(stack.ConfigError, match=match):
            stack.StackConfig(c, 8)

    mixer = lambda c: c["layers"][0]["mixer"]
    bad(lambda c: c.update(architecture="Other"), "Other")
    bad(lambda c: c["layers"][0].update(type="channel_delta"), "channel_delta")
    bad(lambda c: mixer(c).update(heads=5), "divide")
    bad(lambda c: mixer(c).pop("kv_heads"), "kv_heads")
    bad(lambda c: mixer(c).pop("rot"), "rot")
    bad(lambda c: mixer(c)["rot"].update(dims=7), "rotated")
    bad(lambda c: mixer(c)["rot"].update(dims=26), "rotated")
    bad(lambda c: mixer(c)["rot"]["scaling"].pop("low"), "low")
    bad(lambda c: mixer(c)["rot"]["scaling"].update(original=0), "original")
    bad(lambda c: mixer(c).update(softcap=-1.0), "softcap")
    bad(lambda c: c.pop("postln_alpha"), "postln_alpha")
    bad(lambda c: c["layers"][0]["mlp"].update(kind="experts"), "experts")


def test_a_family_refuses_what_it_does_not_have():
    import zamitar_models as zm
    c = copy.deepcopy(zm.MIXED)
    c["layers"][0] = copy.deepcopy(sm.MIXED["layers"][0])
    with pytest.raises(stack.ConfigError, match="'attention'"):
        stack.StackConfig(c, 8)


def test_tensor_shapes_are_checked():
    cfg, w = stack.StackConfig(sm.MIXED, 8), sm.weights(sm.MIXED)
    for name, change in (("l0.mix.q", lambda a: a[:-1]), ("l1.mix.v", lambda a: a[:, :-1]), ("l1.mix.sink", lambda a: a[1:]), ("l3.mix.o", lambda a: a[:, 1:]),
                         ("l0.mlp.down", lambda a: a[1:]), ("l3.norm2", None)):
        t = dict(w)
        if change:
            t[name] = change(t[name])
        else:
            del t[name]
        with pytest.raises(stack.ConfigError, match=name.replace(".", r"\.")):
            for i, L in enumerate(cfg.layers):
                stack.pack_layer(stack.Checkpoint(t), i, L, cfg)


@pytest.mark.parametrize("name", sm.MODELS)
def test_packed_layers_hold_every_weight(name):
    """Segments where the header says they are, zeros elsewhere; norm weights with their offset."""
    d = sm.MODELS[name]
    cfg, w = stack.StackConfig(d, 8), sm.weights(d)
    for i, L in enumerate(cfg.layers):
        mats, vecs = stack.pack_layer(stack.Checkpoint(w), i, L, cfg)
        at, seen = 0, 0
        for n, rows in L.input_segments():
            seg = mats["in"][at:at + rows, :cfg.width]
            assert np.array_equal(seg, w[f"l{i}.mix.{n}"])
            seen += np.count_nonzero(seg)
            at += stack.pad(rows)
        assert np.count_nonzero(mats["in"]) == seen and all(s % 64 == 0 for s in mats["in"].shape)
        f = sm.floats(w)
        assert np.array_equal(vecs["norm"], 1 + f[f"l{i}.norm1"]) and np.array_equal(vecs["sink"], f[f"l{i}.mix.sink"])
        assert ("norm2" in vecs) == bool(L.ff) and "ls1" not in vecs and "gate_bias" not in vecs
        if L.ff:
            assert np.array_equal(vecs["norm2"], 1 + f[f"l{i}.norm2"])


def test_registry_knows_the_architecture(tmp_path):
    (tmp_path / "config.json").write_text(json.dumps({"architecture": "Suborax"}))
    assert registry.lookup(str(tmp_path))[1] == "stack"
