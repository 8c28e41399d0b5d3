"""Small random Suborax models for the tests: configurations that differ in every size, and checkpoints whose values are exact
in bfloat16."""
import numpy as np

from alice_llm_b200.safetensors_file import bf16_to_f32, f32_to_bf16


def scaling(factor=4.0, low=1.5, high=3.0, original=40):
    return dict(factor=factor, low=low, high=high, original=original)


def attention(heads=4, kv_heads=2, dim=24, vdim=40, rot=16, base=300.0, scale=0.5, softcap=6.0, ff=72, scaled=True):
    return {"type": "attention", "mlp": {"kind": "dense", "ff": ff} if ff else None,
            "mixer": dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, softcap=softcap,
                          rot=dict(base=base, dims=rot, scaling=scaling() if scaled is True else scaled or None))}


def config(layers, width=80, vocab=131, eps=1e-5, scale=0.8, alpha=1.7):
    return {"architecture": "Suborax", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale}, "postln_alpha": alpha,
            "layers": layers}


def weights(cfg, seed=0, sink=2.5):
    """{name: uint16 bfloat16 bits}."""
    rng = np.random.default_rng(seed)
    w = {}

    def put(name, *shape, std=None, mean=0.0):
        std = std if std is not None else shape[-1] ** -0.5
        w[name] = f32_to_bf16((mean + std * rng.standard_normal(shape)).astype(np.float32))

    W = cfg["width"]
    put("embed", cfg["vocab"], W, std=1.0)
    put("head", cfg["vocab"], W)
    put("final.norm", W, std=0.2)
    for i, L in enumerate(cfg["layers"]):
        m, p = L["mixer"], f"l{i}.mix."
        H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        put(f"l{i}.norm1", W, std=0.2)
        put(p + "q", H * D, W); put(p + "k", G * D, W); put(p + "v", G * V, W)
        put(p + "sink", H, std=1.0, mean=sink)
        put(p + "o", W, H * V, std=3.0 * (H * V) ** -0.5)
        if L["mlp"]:
            F, q = L["mlp"]["ff"], f"l{i}.mlp."
            put(q + "gate", F, W); put(q + "up", F, W); put(q + "down", W, F, std=2.0 * F ** -0.5)
            put(f"l{i}.norm2", W, std=0.2)
    return w


def floats(w):
    return {n: bf16_to_f32(a) for n, a in w.items()}


def row_errors(got, want):
    """Per row: root mean square of the difference (mean taken off) over that of the wanted row."""
    got, want = np.asarray(got, np.float64), np.asarray(want, np.float64)
    d = got - want
    d = d - d.mean(-1, keepdims=True)
    return np.sqrt((d * d).mean(-1)) / np.sqrt(((want - want.mean(-1, keepdims=True)) ** 2).mean(-1))


# Sizes chosen to differ from one another and to be no multiples of what the kernels tile by. "odd" has head sizes that are odd,
# one key head per query head, a layer without a feed-forward first, a large eps; "wide" groups above sixteen heads and larger sizes.
MIXED = config([attention(), attention(heads=6, kv_heads=1, dim=40, vdim=16, rot=40, softcap=3.0, ff=0), attention(heads=3, kv_heads=3, dim=8, vdim=56, rot=4, ff=48),
                attention(heads=10, kv_heads=5, dim=16, vdim=24, rot=10, base=50.0, scaled=None, ff=130)])
ODD = config([attention(heads=6, kv_heads=6, dim=7, vdim=9, rot=6, ff=0, softcap=20.0), attention(heads=5, kv_heads=1, dim=33, vdim=65, rot=2, scale=0.3, ff=33),
              attention(heads=4, kv_heads=2, dim=10, vdim=21, rot=10, softcap=1.0, ff=65, scaled=scaling(2.0, 1.0, 8.0, 100))], width=50, vocab=77, eps=0.3, scale=0.35, alpha=0.9)
WIDE = config([attention(heads=20, kv_heads=1, dim=64, vdim=72, rot=32, scale=0.2, ff=300), attention(heads=8, kv_heads=2, dim=128, vdim=128, rot=128, scale=0.15, softcap=12.0, ff=260),
               attention(heads=4, kv_heads=2, dim=200, vdim=130, rot=64, scale=0.12, ff=100)], width=272, vocab=515, scale=1.4, alpha=3.1)
MODELS = {"mixed": MIXED, "odd": ODD, "wide": WIDE}
