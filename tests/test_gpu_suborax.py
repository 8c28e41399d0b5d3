"""Suborax models on the device against tests/suborax_ref.py (numpy, float64): every mechanism alone, whole prompts, portions,
decoding, reused cache rows, far keys, greedy generation, the trace runner. 32-bit models are held to 1e-4 of a row's spread, bf16
ones to 0.03; tests/test_suborax_ref.py shows that planted mistakes exceed both."""
import functools
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import suborax_models as sm
import suborax_ref as ref
import zamitar_models as zm
import zamitar_ref
from alice_llm_b200 import stack
from alice_llm_b200.gpu import AliceError, GpuEngine, GpuModel
from alice_llm_b200.registry import open_model
from alice_llm_b200.safetensors_file import f32_to_bf16, write_safetensors

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TOL = {"float32": 1e-4, "bfloat16": 3e-2}
DTYPES = list(TOL)


@pytest.fixture(scope="module")
def eng():
    e = GpuEngine(0)
    yield e
    e.close()


@functools.lru_cache(maxsize=None)
def case(name, n, seed=0):
    """(config, bf16 weights, tokens, float64 logits) of a named model."""
    cfg = sm.MODELS[name]
    w = sm.weights(cfg, seed)
    toks = np.random.default_rng(seed + 1).integers(0, cfg["vocab"], n)
    return cfg, w, toks, ref.forward(cfg, sm.floats(w), toks)


def close(got, want, dtype):
    err = sm.row_errors(got, want)
    assert err.max() <= TOL[dtype], (float(err.max()), int(err.argmax()))


def run_portions(m, toks, sizes):
    """All logits, with the tokens cut into portions of the given sizes (the last one repeats)."""
    out, at, i = [], 0, 0
    while at < len(toks):
        n = min(sizes[min(i, len(sizes) - 1)], len(toks) - at)
        out.append(m.forward_rows(toks[at:at + n], np.arange(n)))
        at += n
        i += 1
    return np.concatenate(out)


# ---- mechanisms alone -----------------------------------------------------------------------------------------------

A, one = sm.attention, lambda *layers, **kw: sm.config(list(layers), **kw)
ALONE = {
    "grouped heads": one(A(ff=0)),
    "a key head per query head": one(A(heads=4, kv_heads=4, ff=0)),
    "one key head": one(A(heads=6, kv_heads=1, ff=0)),
    "groups of twenty": one(A(heads=40, kv_heads=2, dim=16, vdim=16, ff=0)),
    "one head": one(A(heads=1, kv_heads=1, ff=0)),
    "values of odd width": one(A(heads=3, kv_heads=3, vdim=33, ff=0)),
    "dim 6, values of 3": one(A(heads=12, kv_heads=4, dim=6, vdim=3, rot=6, ff=0)),
    "64 / 64": one(A(dim=64, vdim=64, rot=64, scale=0.3, ff=0)),
    "64 / 128": one(A(dim=56, vdim=120, rot=24, scale=0.3, ff=0)),
    "128 / 128": one(A(dim=128, vdim=128, rot=64, scale=0.2, softcap=9.0, ff=0)),
    "128 / 16": one(A(dim=112, vdim=10, rot=112, scale=0.2, softcap=9.0, ff=0)),
    "192 / 128": one(A(dim=180, vdim=100, rot=64, scale=0.15, ff=0)),
    "256 / 256": one(A(dim=256, vdim=250, rot=64, scale=0.13, ff=0)),
    "beyond the tensor-core forms": one(A(dim=300, vdim=280, rot=300, scale=0.1, ff=0)),
    "keys of more than 256 alone": one(A(dim=264, vdim=24, rot=8, scale=0.1, ff=0)),
    "no rotation scaling": one(A(scaled=None, ff=0)),
    "all of the scaled range": one(A(dim=32, rot=32, base=10.0, scaled=sm.scaling(3.0, 1.0, 16.0, 90), ff=0)),
    "two rotated dimensions": one(A(rot=2, ff=0)),
    "no rotated dimensions": one(A(rot=0, ff=0)),
    "a cap far above the scores": one(A(softcap=300.0, ff=0)),
    "a cap three times the scores": one(A(dim=32, scale=0.25, softcap=24.0, ff=0)),
    "a cap of two thirds": one(A(dim=32, scale=0.25, softcap=16.0, ff=0)),
    "a cap among the scores": one(A(softcap=1.5, ff=0)),
    "no cap": one(A(softcap=None, ff=0)),
    "scores too large to go without a running maximum": one(A(dim=64, scale=1.2, softcap=None, ff=0)),
    "scale one": one(A(dim=16, scale=1.0, ff=0)),
    "feed-forward": one(A(heads=1, kv_heads=1, dim=8, vdim=8, rot=4, ff=200)),
    "alpha one, eps large": one(A(), alpha=1.0, eps=0.2, scale=0.3),
    "two layers without feed-forward": one(A(ff=0), A(heads=2, kv_heads=1, ff=0)),
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ALONE)
def test_each_mechanism_alone(eng, name, dtype):
    """Residual stream after every layer and logits; the prompt whole, in two portions, token by token."""
    cfg = ALONE[name]
    w, n = sm.weights(cfg, 3), 170
    toks = np.random.default_rng(4).integers(0, cfg["vocab"], n)
    want = []
    logits = ref.forward(cfg, sm.floats(w), toks, trace=want)
    m = GpuModel.load_stack(eng, (cfg, w), dtype=dtype, max_seq_len=n)
    m.trace(True)
    close(m.forward_rows(toks, np.arange(n)), logits, dtype)
    got = m.read_trace()
    assert got.shape == (len(want), n, cfg["width"]) == (m.config().layer_runs(), n, cfg["width"])
    for a, b in zip(got, want):
        assert np.abs(a - b).max() <= TOL[dtype] * np.abs(b).max()
    m.reset()
    close(run_portions(m, toks[:75], [74, 1]), logits[:75], dtype)
    assert np.abs(m.read_trace()[:, 0] - np.stack(want)[:, 74]).max() <= TOL[dtype] * np.abs(want).max()   # one token traced
    m.trace(False)
    m.reset()
    close(run_portions(m, toks, [3, 60, n]), logits, dtype)
    m.reset()
    close(run_portions(m, toks, [1]), logits, dtype)
    m.free()


# ---- whole models ----------------------------------------------------------------------------------------------------

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", [[300], [1], [2], [3], [4], [5], [64], [100, 2, 1, 65, 2, 2, 7], [1, 1, 1, 128, 129], [200, 1], [16, 15, 17, 31, 33, 2]], ids=str)
def test_portions(eng, sizes, dtype):
    cfg, w, toks, logits = case("mixed", 300)
    m = GpuModel.load_stack(eng, (cfg, w), dtype=dtype, max_seq_len=301)
    close(run_portions(m, toks, sizes), logits, dtype)
    assert m.position() == 300
    m.free()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sm.MODELS)
def test_models_prompt_then_long_decoding(eng, name, dtype):
    cfg, w, toks, logits = case(name, 260)
    m = GpuModel.load_stack(eng, (cfg, w), dtype=dtype, max_seq_len=260)
    close(m.forward_rows(toks, np.arange(260)), logits, dtype)
    m.reset()
    close(run_portions(m, toks, [40, 1]), logits, dtype)     # 220 tokens one by one
    m.reset()
    close(run_portions(m, toks, [90, 2, 3, 4, 2]), logits, dtype)
    m.free()


@pytest.mark.parametrize("dtype", DTYPES)
def test_prompt_longer_than_a_piece(eng, dtype):
    """More tokens than the model takes at once: the library cuts them (256 in 32 bits, 2048 in bf16). Then decoding over the
    many tiles and shares of that context."""
    cfg = one(A(heads=2, kv_heads=1, dim=8, vdim=8, rot=4, scale=1.2, ff=0), width=24, vocab=40)
    w, n = sm.weights(cfg, 8), 700 if dtype == "float32" else 2300
    toks = np.random.default_rng(9).integers(0, 40, n + 3)
    rows = np.array([0, 1, 255, 256, 257, 511, 512, 699] if dtype == "float32" else [0, 63, 64, 127, 128, 1000, 2047, 2048, 2049, 2299])
    want = ref.forward(cfg, sm.floats(w), toks)
    m = GpuModel.load_stack(eng, (cfg, w), dtype=dtype, max_seq_len=n + 3)
    close(m.forward_rows(toks[:n], rows), want[rows], dtype)
    close(run_portions(m, toks[n:], [1, 2]), want[n:], dtype)
    m.free()


@pytest.mark.parametrize("layer, n", [(A(heads=50, kv_heads=50, dim=250, vdim=256, rot=16, scale=0.15, ff=0), 290),
                                      (A(heads=75, kv_heads=75, dim=112, vdim=128, rot=16, scale=0.2, ff=0), 410),
                                      (A(heads=80, kv_heads=80, dim=24, vdim=20, rot=16, ff=0), 530)], ids=["256", "128", "32"])
def test_decoding_over_more_tiles_than_a_warp_has_room_for(eng, layer, n):
    cfg = one(layer, width=64, vocab=60)
    w = sm.weights(cfg, 5)
    toks = np.random.default_rng(6).integers(0, 60, n)
    want = ref.forward(cfg, sm.floats(w), toks, np.float32)
    m = GpuModel.load_stack(eng, (cfg, w), max_seq_len=n)
    close(run_portions(m, toks, [n - 40, 3] + [1] * 37), want, "bfloat16")
    m.free()


@pytest.mark.parametrize("dtype", DTYPES)
def test_more_rows_than_the_head_takes_at_once(eng, dtype):
    cfg, w, toks, logits = case("odd", 150)
    m = GpuModel.load_stack(eng, (cfg, w), dtype=dtype, max_seq_len=150)
    for rows in (np.arange(150), np.arange(0, 150, 2), np.array([149]), np.array([0, 149]), np.array([], int)):
        m.reset()
        got = m.forward_rows(toks, rows)
        assert got.shape == (len(rows), cfg["vocab"])
        if len(rows):
            close(got, logits[rows], dtype)
    m.free()


@pytest.mark.parametrize("dtype", DTYPES)
def test_state_is_given_back(eng, dtype):
    """A request after others gives the bits it gives on a fresh model; the others' lengths leave nothing behind."""
    cfg, w, toks, logits = case("mixed", 300)
    m = GpuModel.load_stack(eng, (cfg, w), dtype=dtype, max_seq_len=300)
    first = run_portions(m, toks[:90], [50, 3, 1])
    for n in (300, 1, 37):
        m.reset()
        run_portions(m, toks[::-1][:n], [33, 1, 2])
    m.reset()
    again = run_portions(m, toks[:90], [50, 3, 1])
    assert np.array_equal(first, again)
    close(again, logits[:90], dtype)
    m.free()


def test_models_of_two_families_on_one_engine_keep_apart(eng):
    """Steps of two models interleaved on one stream: each as if alone."""
    ca, wa, ta, la = case("mixed", 60)
    cb, wb, tb = zm.MIXED, zm.weights(zm.MIXED), np.random.default_rng(2).integers(0, 131, 60)
    lb = zamitar_ref.forward(cb, zm.floats(wb), tb)
    a, b = (GpuModel.load_stack(eng, (c, w), dtype="float32", max_seq_len=60) for c, w in ((ca, wa), (cb, wb)))
    ga, gb = [], []
    for i in range(0, 60, 4):
        ga.append(run_portions(a, ta[i:i + 4], [3, 1]))
        gb.append(run_portions(b, tb[i:i + 4], [1, 3]))
    close(np.concatenate(ga), la, "float32")
    close(np.concatenate(gb), lb, "float32")
    a.free(), b.free()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("key", [0, 1, 15, 16, 31, 32, 63, 64, 127, 128, 255, 256])
def test_far_key_is_seen(eng, monkeypatch, key, dtype):
    """One layer in which the query of the last tokens meets one key far away (at the edges of the tiles keys are read in) with
    a score that stands out: without that key the logits change by more than ten times the tolerance."""
    cfg = one(A(heads=4, kv_heads=2, dim=40, vdim=24, rot=8, scale=1.2, softcap=50.0, ff=0), width=64, vocab=90)
    w = sm.weights(cfg, 11)
    f = sm.floats(w)
    special, asks = 5, 6      # the token that is asked for and the one that asks
    n = key + 150
    toks = np.random.default_rng(12).integers(10, 90, n)
    toks[key], toks[-6:] = special, asks
    # what `asks` queries with is turned towards the unrotated part of the key of `special`
    k = (f["l0.mix.k"] @ f["embed"][special]).reshape(2, 40)
    k[:, :8] = 0
    x = f["embed"][asks]
    q = f["l0.mix.q"].reshape(4, 40, 64) + 30.0 * np.einsum("hd,c->hdc", np.repeat(k, 2, 0), x / (x @ x))
    w["l0.mix.q"] = f32_to_bf16(q.reshape(160, 64).astype(np.float32))
    f = sm.floats(w)
    want = ref.forward(cfg, f, toks)
    full = ref.scores

    def unseen(q, k, scale, softcap):
        s = full(q, k, scale, softcap)
        s[:, key + 1:, key] = -np.inf
        return s
    with monkeypatch.context() as p:
        p.setattr(ref, "scores", unseen)
        without = ref.forward(cfg, f, toks)
    assert sm.row_errors(without[-6:], want[-6:]).min() > 10 * TOL["bfloat16"]
    m = GpuModel.load_stack(eng, (cfg, w), dtype=dtype, max_seq_len=n)
    close(m.forward_rows(toks, np.arange(n - 6, n)), want[-6:], dtype)
    for sizes in ([key + 1, 100, 43, 1], [key + 1, 143, 2, 3, 1], [n - 1, 1]):
        m.reset()
        close(run_portions(m, toks, sizes)[-6:], want[-6:], dtype)
    m.free()


@pytest.mark.parametrize("dtype", DTYPES)
def test_own_key_and_the_next_one(eng, dtype):
    """Every token asks for the token behind it, which it must not see, and next for itself: a mask that is one off in either
    direction changes every row."""
    cfg = one(A(heads=2, kv_heads=1, dim=40, vdim=24, rot=0, scale=1.2, softcap=50.0, ff=0), width=64, vocab=300)
    w = sm.weights(cfg, 13)
    f = sm.floats(w)
    n = 290
    toks = np.arange(n)
    k = (f["embed"] @ f["l0.mix.k"].T)[:n]
    want_q = k.copy()
    want_q[:-1] += 1.5 * k[1:]
    solve = np.linalg.lstsq(f["embed"][:n].astype(np.float64), want_q.astype(np.float64), rcond=None)[0].T   # best linear map from token to query
    w["l0.mix.q"] = f32_to_bf16(np.concatenate([solve, solve]).astype(np.float32))
    want = ref.forward(cfg, sm.floats(w), toks)
    m = GpuModel.load_stack(eng, (cfg, w), dtype=dtype, max_seq_len=n)
    for sizes in ([n], [1], [2], [130, 1, 5]):
        m.reset()
        close(run_portions(m, toks, sizes), want, dtype)
    m.free()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sink", [-60.0, 12.0, 200.0])
def test_sinks_far_from_the_scores(eng, sink, dtype):
    """A sink that counts for nothing, one that takes most of the weight, one that takes all."""
    cfg = one(A(heads=4, kv_heads=2, ff=72), A(heads=4, kv_heads=1, ff=0, softcap=30.0, dim=64, scale=0.3))
    w = sm.weights(cfg, 14, sink=sink)
    toks = np.random.default_rng(15).integers(0, cfg["vocab"], 150)
    want = ref.forward(cfg, sm.floats(w), toks)
    assert np.isfinite(want).all()
    m = GpuModel.load_stack(eng, (cfg, w), dtype=dtype, max_seq_len=150)
    for sizes in ([150], [100, 1], [30, 2]):
        m.reset()
        close(run_portions(m, toks, sizes), want, dtype)
    m.free()


@pytest.mark.parametrize("dtype", DTYPES)
def test_first_tokens(eng, dtype):
    """Sequences of one to nine tokens, whole, in twos and one by one."""
    cfg, w, toks, logits = case("mixed", 300)
    m = GpuModel.load_stack(eng, (cfg, w), dtype=dtype, max_seq_len=300)
    for n in range(1, 10):
        for sizes in ([n], [1], [2]):
            m.reset()
            close(run_portions(m, toks[:n], sizes), logits[:n], dtype)
    m.free()


# ---- generation, limits ----------------------------------------------------------------------------------------------

@pytest.mark.parametrize("name", sm.MODELS)
def test_greedy_generation(eng, name):
    cfg, w, toks, _ = case(name, 260)
    m = GpuModel.load_stack(eng, (cfg, w), dtype="float32", max_seq_len=80)
    want = ref.greedy(cfg, sm.floats(w), toks[:20], 12)
    assert list(m.generate(toks[:20], 12)) == want
    m.reset()                                               # the captured step replayed on a new sequence
    assert list(m.generate(toks[:20], 12)) == want
    m.reset()
    assert list(m.generate(toks[:1], 5)) == ref.greedy(cfg, sm.floats(w), toks[:1], 5)
    m.free()


def test_greedy_generation_bf16_agrees_with_its_own_logits(eng):
    """The decode graph's tokens are the argmax of the logits the step calls give."""
    cfg, w, toks, _ = case("mixed", 300)
    m = GpuModel.load_stack(eng, (cfg, w), max_seq_len=120)
    got = [int(t) for t in m.generate(toks[:50], 30)]
    m.reset()
    m.forward_rows(toks[:49], [])
    tok = int(toks[49])
    for t in got:
        tok = int(np.argmax(m.forward_and_read(tok)))
        assert tok == t
    m.free()


@pytest.mark.parametrize("dtype", DTYPES)
def test_position_limits_and_going_back(eng, dtype):
    cfg, w, toks, logits = case("mixed", 300)
    m = GpuModel.load_stack(eng, (cfg, w), dtype=dtype, max_seq_len=40)
    m.forward_rows(toks[:30], [])
    with pytest.raises(AliceError, match="max_seq_len"):
        m.forward_rows(toks[:11], [])
    with pytest.raises(AliceError):
        m.forward_rows([cfg["vocab"]], [0])
    close(m.forward_rows(toks[30:40], [0, 9]), logits[[30, 39]], dtype)      # refused calls left the cache alone
    m.rollback_to(12)                                                        # rows are simply written again
    want = ref.forward(cfg, sm.floats(w), np.concatenate([toks[:12], toks[100:114]]))
    close(run_portions(m, toks[100:114], [9, 2, 1]), want[12:], dtype)
    m.free()


def test_weight_handles_of_the_wrong_shape_are_refused(eng):
    cfg, w = stack.StackConfig(sm.ODD, 16), sm.weights(sm.ODD)
    packed = [stack.pack_layer(stack.Checkpoint(w), i, L, cfg) for i, L in enumerate(cfg.layers)]
    embed = np.zeros((cfg.vocab_size, 64), np.uint16)
    with pytest.raises(AliceError, match="head"):
        stack.create(eng, cfg, packed, embed, np.ones(cfg.width, np.float32), None, True, embed[:-1])
    packed[1][0]["in"] = packed[1][0]["in"][:-1]
    with pytest.raises(AliceError, match="in must be"):
        stack.create(eng, cfg, packed, embed, np.ones(cfg.width, np.float32), None, True, embed)


# ---- from a folder ---------------------------------------------------------------------------------------------------

@pytest.mark.parametrize("dtype", DTYPES)
def test_trace_runner(tmp_path, dtype):
    cfg, w, toks, logits = case("mixed", 300)
    write_safetensors(str(tmp_path / "model.safetensors"), w)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    want = [0, 3, 99, 100, 119]
    steps, expect = [], {}
    for rid, cut in (("a", [120]), ("b", [100, 2, 1, 1, 16]), ("a", [1] * 6)):      # a name may come back once it has ended
        at = 0
        for i, n in enumerate(cut):
            rows = [p - at for p in want if at <= p < at + n]
            steps.append({"step": len(steps), "entries": [{"id": rid, "tokens": toks[at:at + n].tolist(), "want": rows}],
                          "end": [rid] if i + 1 == len(cut) else []})
            if rows:
                expect[len(steps) - 1] = logits[[at + r for r in rows]]
            at += n
    r = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", dtype, "--out", str(tmp_path),
                        "--max-tokens", "120"], input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [l for l in r.stdout.splitlines() if l.startswith("done ")] == [f"done {s['step']}" for s in steps]
    for n, want in expect.items():
        close(np.fromfile(tmp_path / f"{n}.f32", "<f4").reshape(want.shape), want, dtype)
    assert sorted(int(p.stem) for p in tmp_path.glob("*.f32")) == sorted(expect)


def test_open_model_from_a_folder(tmp_path, eng):
    cfg, w, toks, logits = case("odd", 150)
    write_safetensors(str(tmp_path / "model.safetensors"), w)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    m = open_model(str(tmp_path), engine=eng, dtype="float32", max_seq_len=150)
    assert m.vocab_size() == cfg["vocab"]
    close(m.forward_rows(toks[:10], np.arange(10)), logits[:10], "float32")
    m.free()
