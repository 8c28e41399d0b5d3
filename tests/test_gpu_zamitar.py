"""Zamitar models on the device against tests/zamitar_ref.py (numpy, float64): every mechanism alone, whole prompts, portions,
decoding, reused state, far keys, greedy generation, the trace runner. 32-bit models are held to 1e-4 of a row's spread, bf16
ones to 0.03; tests/test_zamitar_ref.py shows that planted mistakes exceed both."""
import functools
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import zamitar_models as zm
import zamitar_ref as ref
from alice_llm_b200 import stack
from alice_llm_b200.gpu import AliceError, GpuEngine, GpuModel, GpuQuantType
from alice_llm_b200.registry import open_model
from alice_llm_b200.safetensors_file import bf16_to_f32, f32_to_bf16, write_safetensors

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
def case(name, n, seed=0, peaky=3.0):
    """(config, bf16 weights, tokens, float64 logits) of a named model."""
    cfg = zm.MODELS[name]
    w = zm.weights(cfg, seed, peaky=peaky)
    toks = np.random.default_rng(seed + 1).integers(0, cfg["vocab"], n)
    return cfg, w, toks, ref.forward(cfg, zm.floats(w), toks)


def close(got, want, dtype):
    err = zm.row_errors(got, want)
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

ALONE = {
    "latent attention": zm.config([zm.latent(ff=0)]),
    "latent attention, many heads": zm.config([zm.latent(heads=40, dim=8, rot=8, vdim=8, ff=0)]),
    "latent attention, sizes without a tensor-core form": zm.config([zm.latent(heads=5, dim=7, rot=6, vdim=9, ff=0)]),
    "latent attention, 64 / 64": zm.config([zm.latent(heads=4, dim=32, rot=32, vdim=64, ff=0)]),
    "latent attention, 128 / 128": zm.config([zm.latent(heads=3, dim=72, rot=56, vdim=128, ff=0)]),
    "latent attention, 192 / 128": zm.config([zm.latent(heads=3, dim=128, rot=64, vdim=112, kv_rank=500, ff=0)]),
    "latent attention, 256 / 256": zm.config([zm.latent(heads=2, dim=200, rot=48, vdim=248, ff=0)]),
    "latent attention, a latent of 600": zm.config([zm.latent(heads=3, kv_rank=600, ff=0)]),
    "latent attention, wide rotated part": zm.config([zm.latent(heads=2, dim=8, rot=128, kv_rank=512, ff=0)]),
    "delta rule": zm.config([zm.delta(ff=0)]),
    "delta rule, one tap": zm.config([zm.delta(conv=1, ff=0)]),
    "delta rule, seven taps": zm.config([zm.delta(conv=7, ff=0)]),
    "delta rule, dim 32": zm.config([zm.delta(heads=2, kv_heads=2, dim=32, vdim=32, ff=0)]),
    "delta rule, dim 64": zm.config([zm.delta(heads=2, kv_heads=1, dim=64, vdim=96, ff=0)]),
    "delta rule, dim 128": zm.config([zm.delta(heads=2, kv_heads=1, dim=128, vdim=128, ff=0)]),
    "delta rule, dim 256": zm.config([zm.delta(heads=2, kv_heads=2, dim=256, vdim=256, ff=0)]),
    "delta rule, values wider than a cluster": zm.config([zm.delta(heads=1, kv_heads=1, dim=20, vdim=300, ff=0)]),
    "feed-forward": zm.config([zm.latent(heads=1, dim=8, rot=8, vdim=8, ff=200)]),
    "loop": zm.config([zm.latent(ff=0), zm.delta(ff=0)], loop=(0, 2, 2)),
    "loop of one pass": zm.config([zm.delta(ff=0), zm.latent(ff=0)], loop=(1, 2, 1)),
    "loop in the middle": zm.config([zm.delta(ff=0), zm.latent(ff=0), zm.delta(ff=0)], loop=(1, 2, 4)),
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ALONE)
def test_each_mechanism_alone(eng, name, dtype):
    """Residual stream after every layer run and logits, prompt and token by token."""
    cfg = ALONE[name]
    w = zm.weights(cfg, 3, peaky=2.0)
    toks = np.random.default_rng(4).integers(0, cfg["vocab"], 75)
    want = []
    logits = ref.forward(cfg, zm.floats(w), toks, trace=want)
    m = GpuModel.load_stack(eng, (cfg, w), dtype=dtype, max_seq_len=128)
    m.trace(True)
    close(m.forward_rows(toks, np.arange(75)), logits, dtype)
    got = m.read_trace()
    assert got.shape == (len(want), 75, cfg["width"]) == (m.config().layer_runs(), 75, cfg["width"])
    for a, b in zip(got, want):
        assert np.abs(a - b).max() <= TOL[dtype] * np.abs(b).max()
    m.trace(False)
    m.reset()
    close(run_portions(m, toks, [1]), logits, dtype)
    m.free()


# ---- whole models ----------------------------------------------------------------------------------------------------

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", [[300], [1], [2], [3], [5], [64], [100, 2, 1, 65, 2, 2, 7], [1, 1, 1, 128, 129], [200, 1]], ids=str)
def test_portions(eng, sizes, dtype):
    cfg, w, toks, logits = case("mixed", 300)
    m = GpuModel.load_stack(eng, (cfg, w), dtype=dtype, max_seq_len=301)
    close(run_portions(m, toks, sizes), logits, dtype)
    assert m.position() == 300
    m.free()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", zm.MODELS)
def test_models_prompt_then_long_decoding(eng, name, dtype):
    cfg, w, toks, logits = case(name, 260)
    m = GpuModel.load_stack(eng, (cfg, w), dtype=dtype, max_seq_len=260)
    close(m.forward_rows(toks, np.arange(260)), logits, dtype)
    m.reset()
    close(run_portions(m, toks, [40, 1]), logits, dtype)     # 220 tokens one by one
    m.free()


@pytest.mark.parametrize("dtype", DTYPES)
def test_prompt_longer_than_a_piece(eng, dtype):
    """More tokens than the model takes at once: the library cuts them (256 in 32 bits, 2048 in bf16)."""
    cfg = zm.config([zm.delta(heads=1, kv_heads=1, dim=8, vdim=8, ff=0), zm.latent(heads=1, dim=8, rot=8, vdim=8, ff=0)], width=24, vocab=40)
    w, n = zm.weights(cfg, 8, peaky=3.0), 700 if dtype == "float32" else 2300
    toks = np.random.default_rng(9).integers(0, 40, n)
    rows = np.array([0, 1, 255, 256, 257, 511, 512, 699] if dtype == "float32" else [0, 63, 64, 127, 128, 2047, 2048, 2049, 2299])
    want = ref.forward(cfg, zm.floats(w), toks)[rows]
    m = GpuModel.load_stack(eng, (cfg, w), dtype=dtype, max_seq_len=n)
    close(m.forward_rows(toks, rows), want, dtype)
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


def test_two_models_on_one_engine_keep_apart(eng):
    """Steps of two models interleaved on one stream: each as if alone."""
    (ca, wa, ta, la), (cb, wb, tb, lb) = case("mixed", 60), case("odd", 60)
    a, b = (GpuModel.load_stack(eng, (c, w), dtype="float32", max_seq_len=60) for c, w in ((ca, wa), (cb, wb)))
    ga, gb = [], []
    for i in range(0, 60, 4):
        ga.append(run_portions(a, ta[i:i + 4], [3, 1]))
        gb.append(run_portions(b, tb[i:i + 4], [1, 3]))
    close(np.concatenate(ga), la, "float32")
    close(np.concatenate(gb), lb, "float32")
    a.free(), b.free()


def drop_key(j, from_row):
    """sink_attention in which rows from `from_row` on do not see key j."""
    def fn(q, k, v, scale, sink):
        out = full(q, k, v, scale, sink)
        keep = np.arange(len(k)) != j
        for i in range(from_row, len(q)):
            n = i + 1
            kk, vv = k[:n][keep[:n]], v[:n][keep[:n]]
            qq = np.concatenate([np.zeros((len(kk) - 1,) + q.shape[1:]), q[i:i + 1]])
            out[i] = full(qq, kk, vv, scale, sink)[-1]
        return out
    full = ref.sink_attention
    return fn


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("key", [0, 1, 31, 32, 63, 64, 127, 128])
def test_far_key_is_seen(eng, monkeypatch, key, dtype):
    """One layer of attention in which the query of the last tokens meets one key far away (at the edges of the tiles keys are
    read in) with a score that stands out: without that key the logits change by more than ten times the tolerance."""
    cfg = zm.config([zm.latent(heads=2, dim=16, rot=8, vdim=16, ff=0)], width=64, vocab=90, scale=1.0)
    w = zm.weights(cfg, 11)
    f = zm.floats(w)
    special, asks = 5, 6      # the token that is asked for and the one that asks
    n = key + 150
    toks = np.random.default_rng(12).integers(10, 90, n)
    toks[key], toks[-3:] = special, asks
    # the query latent of `asks` is turned towards the key of `special` as the layer makes it
    x = f["embed"]
    h = ref.layer_norm(x.astype(np.float64), f["l0.norm1"], cfg["norm"]["eps"])
    c = ref.rms_norm(ref.linear(h[special], f["l0.mix.dkv"])[:56], f["l0.mix.dkv.norm"], cfg["norm"]["eps"])
    cq = ref.rms_norm(ref.linear(h[asks], f["l0.mix.dq"]), f["l0.mix.dq.norm"], cfg["norm"]["eps"])
    uq = f["l0.mix.uq"].reshape(2, 24, 40).copy()
    for hd in range(2):
        kk = f["l0.mix.uk"].reshape(2, 16, 56)[hd] @ c
        uq[hd, :16] += 60.0 * np.outer(kk / (kk @ kk), cq / (cq @ cq))
    w["l0.mix.uq"] = f32_to_bf16(uq.reshape(48, 40).astype(np.float32))
    f = zm.floats(w)
    want = ref.forward(cfg, f, toks)
    with monkeypatch.context() as p:
        p.setattr(ref, "sink_attention", drop_key(key, n - 3))
        without = ref.forward(cfg, f, toks)
    assert zm.row_errors(without[-3:], want[-3:]).min() > 10 * TOL["bfloat16"]
    m = GpuModel.load_stack(eng, (cfg, w), dtype=dtype, max_seq_len=n)
    close(m.forward_rows(toks, np.arange(n - 3, n)), want[-3:], dtype)
    m.reset()
    close(run_portions(m, toks, [key + 1, 100, 46, 1])[-3:], want[-3:], dtype)
    m.free()


@pytest.mark.parametrize("dtype", DTYPES)
def test_first_tokens(eng, dtype):
    """Sequences of one to nine tokens, whole and one by one: zeros before the start, a state that starts at zero."""
    cfg, w, toks, logits = case("mixed", 300)
    m = GpuModel.load_stack(eng, (cfg, w), dtype=dtype, max_seq_len=300)
    for n in range(1, 10):
        for sizes in ([n], [1], [2]):
            m.reset()
            close(run_portions(m, toks[:n], sizes), logits[:n], dtype)
    m.free()


# ---- generation, limits ----------------------------------------------------------------------------------------------

@pytest.mark.parametrize("name", zm.MODELS)
def test_greedy_generation(eng, name):
    cfg, w, toks, _ = case(name, 260)
    m = GpuModel.load_stack(eng, (cfg, w), dtype="float32", max_seq_len=80)
    want = ref.greedy(cfg, zm.floats(w), toks[:20], 12)
    assert list(m.generate(toks[:20], 12)) == want
    m.reset()                                               # the captured step replayed on a new sequence
    assert list(m.generate(toks[:20], 12)) == want
    m.reset()
    assert list(m.generate(toks[:1], 5)) == ref.greedy(cfg, zm.floats(w), toks[:1], 5)
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


def test_position_limits_and_rollback(eng):
    cfg, w, toks, logits = case("mixed", 300)
    m = GpuModel.load_stack(eng, (cfg, w), dtype="float32", max_seq_len=40)
    m.forward_rows(toks[:30], [])
    with pytest.raises(AliceError, match="max_seq_len"):
        m.forward_rows(toks[:11], [])
    with pytest.raises(AliceError, match="recurrent"):
        m.rollback_to(20)
    with pytest.raises(AliceError):
        m.forward_rows([cfg["vocab"]], [0])
    for rows in ([3], [1, 0], [0, 0]):
        with pytest.raises(AliceError):
            m.forward_rows(toks[30:33], rows)
    close(m.forward_rows(toks[30:40], [0, 9]), logits[[30, 39]], "float32")      # refused calls left the state alone
    m.free()
    cfg = ALONE["latent attention"]      # attention alone can go back: its rows are simply written again
    w = zm.weights(cfg)
    m = GpuModel.load_stack(eng, (cfg, w), dtype="float32", max_seq_len=40)
    m.forward_rows(toks[:30], [])
    m.rollback_to(12)
    close(m.forward_rows(toks[100:110], [9]), ref.forward(cfg, zm.floats(w), np.concatenate([toks[:12], toks[100:110]]))[-1:], "float32")
    with pytest.raises(AliceError, match="key / value"):
        m.kv_read(0, 0, 1)
    m.free()


def test_weight_handles_of_the_wrong_shape_are_refused(eng):
    cfg = stack.StackConfig(zm.ODD, 16)
    w = zm.weights(zm.ODD)
    packed = [stack.pack_layer(stack.Checkpoint(w), i, L, cfg) for i, L in enumerate(cfg.layers)]
    packed[1][0]["uk"] = packed[1][0]["uk"][:-1]
    embed = np.zeros((cfg.vocab_size, 64), np.uint16)
    with pytest.raises(AliceError, match="uk"):
        stack.create(eng, cfg, packed, embed, np.ones(cfg.width, np.float32), np.zeros((1, cfg.width), np.float32), True)


# ---- dense rows as a weight format -----------------------------------------------------------------------------------

def test_bf16_matvec_and_dequantize(eng):
    rng = np.random.default_rng(20)
    for rows, cols in ((1, 64), (77, 192), (1000, 4096), (5000, 1024)):
        w = f32_to_bf16(rng.standard_normal((rows, cols)).astype(np.float32))
        h = eng.upload_weights_typed(w.view(np.uint8), rows, cols, GpuQuantType.BF16)
        x = rng.standard_normal((3, cols)).astype(np.float32)
        xb, yb = eng.upload_f32(x), eng.alloc_f32(3 * rows)
        eng.matvec_dev(h, xb, yb, 3)
        got = eng.read_f32(yb).reshape(3, rows)
        eng.sync()
        want = x.astype(np.float64) @ bf16_to_f32(w).astype(np.float64).T
        assert np.abs(got - want).max() <= 2e-6 * np.abs(want).max() * cols ** 0.5
        assert np.array_equal(eng.dequantize(h).reshape(rows, cols), bf16_to_f32(w))
    h = eng.upload_weights_typed(np.zeros(2 * 40 * 4, np.uint8), 4, 40, GpuQuantType.BF16)
    with pytest.raises(AliceError):
        eng.matvec(h, np.zeros(40, np.float32))


# ---- from a folder ---------------------------------------------------------------------------------------------------

@pytest.mark.parametrize("dtype", DTYPES)
def test_trace_runner(tmp_path, dtype):
    cfg, w, toks, logits = case("mixed", 300)
    write_safetensors(str(tmp_path / "model.safetensors"), w)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    want = [0, 3, 99, 100, 119]
    steps, at, expect = [], 0, {}
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
