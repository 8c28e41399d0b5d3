"""Small random Zamitar models for the tests: configurations that differ in every size, and checkpoints whose values are
exact in bfloat16."""
import numpy as np

from alice_llm_b200.safetensors_file import bf16_to_f32, f32_to_bf16


def latent(heads=3, dim=16, rot=16, vdim=24, q_rank=40, kv_rank=56, scale=None, base=500.0, ff=72):
    return {"type": "latent_attention", "mlp": {"kind": "dense", "ff": ff} if ff else None,
            "mixer": dict(heads=heads, dim=dim, rot_dim=rot, vdim=vdim, q_rank=q_rank, kv_rank=kv_rank, scale=scale or (dim + rot) ** -0.5,
                          rot=dict(base=base, dims=rot))}


def delta(heads=4, kv_heads=2, dim=24, vdim=40, conv=4, ff=72):
    return {"type": "channel_delta", "mlp": {"kind": "dense", "ff": ff} if ff else None,
            "mixer": dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, conv=conv)}


def config(layers, width=80, vocab=131, eps=1e-5, scale=3.0, loop=None):
    return {"architecture": "Zamitar", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale}, "layers": layers,
            "loop": None if loop is None else dict(zip(("start", "stop", "times"), loop))}


def weights(cfg, seed=0, decay_rank=20, gate_rank=12, peaky=1.0):
    """{name: uint16 bfloat16 bits}. `peaky` scales the query projections of the attention: above 1 few keys stand out."""
    rng = np.random.default_rng(seed)
    w = {}

    def put(name, *shape, std=None, mean=0.0):
        std = std if std is not None else shape[-1] ** -0.5
        w[name] = f32_to_bf16((mean + std * rng.standard_normal(shape)).astype(np.float32))

    W = cfg["width"]
    put("embed", cfg["vocab"], W, std=0.5)
    put("final.norm", W, std=0.1, mean=1.0)
    if cfg["loop"]:
        put("loop.step", cfg["loop"]["times"], W, std=0.5)
    for i, L in enumerate(cfg["layers"]):
        m, p = L["mixer"], f"l{i}.mix."
        put(f"l{i}.norm1", W, std=0.1, mean=1.0)
        put(f"l{i}.ls1", W, std=0.2, mean=0.8)
        H, D, V = m["heads"], m["dim"], m["vdim"]
        if L["type"] == "latent_attention":
            R, Q, C = m["rot_dim"], m["q_rank"], m["kv_rank"]
            put(p + "dq", Q, W); put(p + "dq.norm", Q, std=0.1, mean=1.0)
            put(p + "uq", H * (D + R), Q, std=peaky * Q ** -0.5)
            put(p + "dkv", C + R, W); put(p + "dkv.norm", C, std=0.1, mean=1.0)
            put(p + "uk", H * D, C); put(p + "uv", H * V, C)
            put(p + "sink", H, std=1.0, mean=3.0)
            put(p + "g", H * V, W)
        else:
            K, n = m["kv_heads"], m["conv"]
            for t, rows in (("q", K * D), ("k", K * D), ("v", H * V)):
                put(p + t, rows, W)
                put(p + t + ".conv", rows, n, std=0.6)
            put(p + "b", H, W); put(p + "A_log", H, std=0.7, mean=-0.5); put(p + "norm", V, std=0.1, mean=1.0)
            put(p + "a1", decay_rank, W); put(p + "a2", H * D, decay_rank); put(p + "dt_bias", H * D, std=1.0, mean=-2.5)
            put(p + "g1", gate_rank, W); put(p + "g2", H * V, gate_rank)
        put(p + "o", W, H * V)
        if L["mlp"]:
            F, q = L["mlp"]["ff"], f"l{i}.mlp."
            for t, shape in (("gate", (F, W)), ("up", (F, W)), ("down", (W, F))):
                put(q + t, *shape)
                put(q + t + ".b", shape[0], std=0.3)
            put(f"l{i}.ls2", W, std=0.2, mean=0.7)
    return w


def floats(w):
    return {n: bf16_to_f32(a) for n, a in w.items()}


def row_errors(got, want):
    """Per row: root mean square of the difference (mean taken off) over that of the wanted row."""
    got, want = np.asarray(got, np.float64), np.asarray(want, np.float64)
    d = got - want
    d = d - d.mean(-1, keepdims=True)
    return np.sqrt((d * d).mean(-1)) / np.sqrt(((want - want.mean(-1, keepdims=True)) ** 2).mean(-1))


# Sizes chosen to differ from one another and to be no multiples of what the kernels tile by; the second has dimensions the
# tensor-core prefill does not take.
MIXED = config([latent(), delta(), delta(heads=3, kv_heads=3, dim=40, vdim=16, conv=2, ff=0), latent(heads=9, dim=8, rot=24, vdim=8, kv_rank=72, ff=48)],
               loop=(1, 3, 3))
ODD = config([delta(heads=6, kv_heads=2, dim=10, vdim=7, conv=3, ff=33), latent(heads=2, dim=6, rot=10, vdim=5, q_rank=9, kv_rank=11, ff=0),
              delta(heads=1, kv_heads=1, dim=33, vdim=65, conv=1)], width=50, vocab=77, eps=1e-3, scale=0.7, loop=(0, 3, 1))
WIDE = config([latent(heads=17, dim=64, rot=32, vdim=80, q_rank=200, kv_rank=320, ff=300), delta(heads=4, kv_heads=4, dim=96, vdim=130, ff=260),
               delta(heads=2, kv_heads=1, dim=130, vdim=64, conv=5, ff=100)], width=272, vocab=515)
MODELS = {"mixed": MIXED, "odd": ODD, "wide": WIDE}
