"""Layer-stack models: configuration, checkpoint layout, and the packing of a checkpoint's tensors into the matrices
``alice_stack_create`` takes (include/alice_cuda.h). A model is a list of layers, each with its own token mixer."""
from __future__ import annotations

import ctypes as C
import json
import os

import numpy as np

from . import _lib
from .safetensors_file import SafetensorsFile, bf16_to_f32

MIX_LATENT, MIX_DELTA, MIX_GROUPED = 1, 2, 3
BLOCK_PARALLEL, BLOCK_POST = 0, 1
NORM_LAYER, NORM_RMS = 0, 1
PAD = 64          # columns, and row segments of packed matrices, come in multiples of this


class Family:
    """What an architecture fixes, whatever its sizes."""

    def __init__(self, mixers, block, norm, norm_offset=0.0, mlp_bias=False, tied=True, unit_qk=False):
        self.mixers, self.block, self.norm = mixers, block, norm
        self.norm_offset = norm_offset      # added to stored norm weights
        self.mlp_bias = mlp_bias            # gate, up and down have biases
        self.tied = tied                    # the embedding table is the head
        self.unit_qk = unit_qk              # rotated queries and keys over their root mean square


FAMILIES = {
    "Zamitar": Family({"latent_attention": MIX_LATENT, "channel_delta": MIX_DELTA}, BLOCK_PARALLEL, NORM_LAYER, mlp_bias=True),
    "Suborax": Family({"attention": MIX_GROUPED}, BLOCK_POST, NORM_RMS, norm_offset=1.0, tied=False, unit_qk=True),
}


class ConfigError(ValueError):
    pass


def pad(n: int, m: int = PAD) -> int:
    return (n + m - 1) // m * m


def delta_dim(dim: int) -> int:
    """Key channels of a head as the recurrence keeps them."""
    for d in (64, 128, 256):
        if dim <= d:
            return d
    raise ConfigError(f"channel_delta: dim {dim} above 256")


def _size(d: dict, key: str, where: str, least: int = 1) -> int:
    if key not in d:
        raise ConfigError(f"{where}: {key} missing")
    v = d[key]
    if isinstance(v, bool) or not isinstance(v, int) or v < least:
        raise ConfigError(f"{where}: {key} = {v!r}")
    return v


def _number(d: dict, key: str, where: str) -> float:
    if key not in d or isinstance(d[key], bool) or not isinstance(d[key], (int, float)):
        raise ConfigError(f"{where}: {key} = {d.get(key)!r}")
    return float(d[key])


class LayerSpec:
    """One layer: mixer kind and sizes, feed-forward width (0 = none)."""

    SIZES = {MIX_LATENT: ("heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank"), MIX_DELTA: ("heads", "kv_heads", "dim", "vdim"),
             MIX_GROUPED: ("heads", "kv_heads", "dim", "vdim")}

    def __init__(self, d: dict, where: str, family: Family):
        kind = d.get("type")
        if kind not in family.mixers:
            raise ConfigError(f"{where}: mixer {kind!r} (known: {', '.join(family.mixers)})")
        self.kind, m = family.mixers[kind], d["mixer"]
        self.heads = self.kv_heads = self.dim = self.vdim = self.q_rank = self.kv_rank = self.rot_dim = self.rot_dims = 0
        self.conv_taps = self.decay_rank = self.gate_rank = 0
        self.scale = self.rot_base = 1.0
        self.softcap = self.rot_factor = self.rot_low = self.rot_high = self.rot_original = 0.0
        self.unit_qk = int(family.unit_qk)
        for key in self.SIZES[self.kind]:
            setattr(self, key, _size(m, key, where))
        if self.kind != MIX_DELTA:
            self.scale = _number(m, "scale", where)
            self._rotation(m.get("rot"), self.rot_dim if self.kind == MIX_LATENT else self.dim, where)
        else:
            self.conv_taps = _size(m, "conv", where)
        if self.kind == MIX_GROUPED and m.get("softcap") is not None:
            self.softcap = _number(m, "softcap", where)
            if self.softcap <= 0:
                raise ConfigError(f"{where}: softcap = {self.softcap}")
        if self.kind != MIX_LATENT and self.heads % self.kv_heads:
            raise ConfigError(f"{where}: {self.heads} heads do not divide over {self.kv_heads} key heads")
        self.ff = 0
        mlp = d.get("mlp")
        if mlp:
            if mlp.get("kind") != "dense":
                raise ConfigError(f"{where}: feed-forward {mlp.get('kind')!r} (known: dense)")
            self.ff = _size(mlp, "ff", where)

    def _rotation(self, rot, room: int, where: str):
        if not isinstance(rot, dict):
            raise ConfigError(f"{where}: rot = {rot!r}")
        self.rot_dims, self.rot_base = _size(rot, "dims", where, 0), _number(rot, "base", where)
        if self.rot_dims % 2 or self.rot_dims > room:
            raise ConfigError(f"{where}: {self.rot_dims} rotated dimensions of {room}")
        if self.rot_base <= 0:
            raise ConfigError(f"{where}: rot base = {self.rot_base}")
        if rot.get("scaling"):
            for key in ("factor", "low", "high", "original"):
                v = _number(rot["scaling"], key, f"{where}: rot scaling")
                if v <= 0:
                    raise ConfigError(f"{where}: rot scaling: {key} = {v}")
                setattr(self, "rot_" + key, v)

    # rows of the packed input projection: (tensor, rows), each starting at a multiple of PAD
    def input_segments(self):
        if self.kind == MIX_LATENT:
            return [("dq", self.q_rank), ("dkv", self.kv_rank + self.rot_dim), ("g", self.heads * self.vdim)]
        if self.kind == MIX_GROUPED:
            return [("q", self.heads * self.dim), ("k", self.kv_heads * self.dim), ("v", self.kv_heads * self.vdim)]
        return [("q", self.kv_heads * self.dim), ("k", self.kv_heads * self.dim), ("v", self.heads * self.vdim), ("b", self.heads),
                ("a1", self.decay_rank), ("g1", self.gate_rank)]

    def packed_shapes(self, width: int) -> dict:
        """name -> (rows, cols) of the matrices of this layer as the library takes them."""
        out = {"in": (sum(pad(r) for _, r in self.input_segments()), pad(width)), "o": (width, pad(self.heads * self.vdim))}
        if self.kind == MIX_LATENT:
            out["uq"] = (self.heads * (self.dim + self.rot_dim), pad(self.q_rank))
            out["uk"], out["uv"] = (self.heads * self.dim, pad(self.kv_rank)), (self.heads * self.vdim, pad(self.kv_rank))
        elif self.kind == MIX_DELTA:
            out["a2"] = (self.heads * delta_dim(self.dim), pad(self.decay_rank))
            out["g2"] = (self.heads * self.vdim, pad(self.gate_rank))
        if self.ff:
            out["gu"], out["down"] = (2 * pad(self.ff), pad(width)), (width, pad(self.ff))
        return out


class StackConfig:
    """config.json of a layer-stack model."""

    def __init__(self, d: dict, max_seq_len: int):
        where = "config"
        self.architecture = d.get("architecture")
        if self.architecture not in FAMILIES:
            raise ConfigError(f"config: architecture {self.architecture!r} (known: {', '.join(FAMILIES)})")
        self.family = FAMILIES[self.architecture]
        self.vocab_size, self.width = _size(d, "vocab", where), _size(d, "width", where)
        self.eps, self.embed_scale = _number(d["norm"], "eps", "norm"), _number(d["embedding"], "scale", "embedding")
        self.alpha = _number(d, "postln_alpha", where) if self.family.block == BLOCK_POST else 1.0
        self.layers = [LayerSpec(l, f"layer {i}", self.family) for i, l in enumerate(d["layers"])]
        if not self.layers:
            raise ConfigError("config: no layers")
        self.loop_start = self.loop_stop = self.loop_times = 0
        loop = d.get("loop")
        if loop:
            self.loop_start, self.loop_stop = _size(loop, "start", "loop", 0), _size(loop, "stop", "loop", 0)
            self.loop_times = _size(loop, "times", "loop")
            if not self.loop_start <= self.loop_stop <= len(self.layers):
                raise ConfigError(f"loop: layers {self.loop_start} .. {self.loop_stop} of {len(self.layers)}")
        self.max_seq_len = max_seq_len

    def layer_runs(self) -> int:
        return len(self.layers) + max(0, self.loop_times - 1) * (self.loop_stop - self.loop_start)


# ---- packing: bfloat16 as uint16 bits --------------------------------------------------------------------

def _rows(parts, cols: int) -> np.ndarray:
    """The parts one below the other, each padded to a multiple of PAD rows, all to `cols` columns."""
    out = np.zeros((sum(pad(len(p)) for p in parts), cols), np.uint16)
    at = 0
    for p in parts:
        out[at:at + len(p), :p.shape[1]] = p
        at += pad(len(p))
    return out


def _cols(m: np.ndarray, cols: int) -> np.ndarray:
    out = np.zeros((len(m), cols), np.uint16)
    out[:, :m.shape[1]] = m
    return out


def _interleave(gate: np.ndarray, up: np.ndarray, cols: int) -> np.ndarray:
    n = pad(len(gate))
    out = np.zeros((n // PAD, 2, PAD, cols), np.uint16)
    for i, m in enumerate((gate, up)):
        full = np.zeros((n, cols), np.uint16)
        full[:len(m), :m.shape[1]] = m
        out[:, i] = full.reshape(n // PAD, PAD, cols)
    return out.reshape(2 * n, cols)


def _vec(v, n: int) -> np.ndarray:
    out = np.zeros(n, np.float32)
    out[:len(v)] = v
    return out


class Checkpoint:
    """Named tensors with their shapes checked as they are taken."""

    def __init__(self, tensors: dict):
        self.tensors = tensors

    def raw(self, name, shape=None):
        if name not in self.tensors:
            raise ConfigError(f"tensor {name} missing")
        a = self.tensors[name]
        if shape is not None and tuple(a.shape) != tuple(shape):
            raise ConfigError(f"tensor {name} is {tuple(a.shape)}, expected {tuple(shape)}")
        return a

    def matrix(self, name, rows, cols):
        a = self.raw(name, (rows, cols))
        if a.dtype != np.uint16:
            raise ConfigError(f"tensor {name}: matrices are bfloat16")
        return a

    def floats(self, name, *shape):
        a = self.raw(name, shape)
        return bf16_to_f32(a) if a.dtype == np.uint16 else np.asarray(a, np.float32)


def pack_layer(ck: Checkpoint, i: int, L: LayerSpec, cfg: "StackConfig"):
    """-> ({matrix name: uint16 array}, {vector name: float32 array}); fills in the ranks only the tensors tell."""
    p, m, width, family = f"l{i}.", f"l{i}.mix.", cfg.width, cfg.family
    if L.kind == MIX_DELTA:
        L.decay_rank, L.gate_rank = len(ck.raw(m + "a1")), len(ck.raw(m + "g1"))
    shapes = L.packed_shapes(width)
    H, V = L.heads, L.vdim
    mats = {"in": _rows([ck.matrix(m + n, r, width) for n, r in L.input_segments()], pad(width)),
            "o": _cols(ck.matrix(m + "o", width, H * V), shapes["o"][1])}
    vecs = {"norm": ck.floats(p + "norm1", width) + np.float32(family.norm_offset)}
    if family.block == BLOCK_PARALLEL:
        vecs["ls1"] = ck.floats(p + "ls1", width)
    if L.kind == MIX_LATENT:
        for n, src in (("uq", L.q_rank), ("uk", L.kv_rank), ("uv", L.kv_rank)):
            mats[n] = _cols(ck.matrix(m + n, shapes[n][0], src), shapes[n][1])
        vecs.update(q_norm=ck.floats(m + "dq.norm", L.q_rank), kv_norm=ck.floats(m + "dkv.norm", L.kv_rank), sink=ck.floats(m + "sink", H))
    elif L.kind == MIX_GROUPED:
        vecs["sink"] = ck.floats(m + "sink", H)
    else:
        D, dp, K = L.dim, delta_dim(L.dim), L.conv_taps
        a2 = np.zeros((H, dp, L.decay_rank), np.uint16)
        a2[:, :D] = ck.matrix(m + "a2", H * D, L.decay_rank).reshape(H, D, L.decay_rank)
        mats["a2"] = _cols(a2.reshape(H * dp, L.decay_rank), shapes["a2"][1])
        mats["g2"] = _cols(ck.matrix(m + "g2", H * V, L.gate_rank), shapes["g2"][1])
        dt = np.zeros((H, dp), np.float32)
        dt[:, :D] = ck.floats(m + "dt_bias", H * D).reshape(H, D)
        convs = [ck.floats(m + f"{n}.conv", r, K) for n, r in L.input_segments()[:3]]
        conv = np.zeros((K, sum(pad(len(c)) for c in convs)), np.float32)
        at = 0
        for c in convs:
            conv[:, at:at + len(c)] = c.T
            at += pad(len(c))
        vecs.update(conv=conv, a_log=ck.floats(m + "A_log", H), dt_bias=dt, head_norm=ck.floats(m + "norm", V))
    if L.ff:
        q = f"l{i}.mlp."
        mats["gu"] = _interleave(ck.matrix(q + "gate", L.ff, width), ck.matrix(q + "up", L.ff, width), pad(width))
        mats["down"] = _cols(ck.matrix(q + "down", width, L.ff), shapes["down"][1])
        if family.block == BLOCK_POST:
            vecs["norm2"] = ck.floats(p + "norm2", width) + np.float32(family.norm_offset)
        else:
            vecs["ls2"] = ck.floats(p + "ls2", width)
        if family.mlp_bias:
            vecs.update(gate_bias=_vec(ck.floats(q + "gate.b", L.ff), pad(L.ff)), up_bias=_vec(ck.floats(q + "up.b", L.ff), pad(L.ff)),
                        down_bias=ck.floats(q + "down.b", width))
    for n, a in mats.items():
        assert a.shape == shapes[n], (n, a.shape, shapes[n])
    return mats, vecs


def create(engine, cfg: StackConfig, packed_layers, embed, final_norm, loop_step, exact: bool, head=None):
    """alice_stack_create over packed layers: [(matrices, vectors)]; a matrix is a uint16 array or a ready weight handle
    (head None: the embedding table).
    -> (handle, objects that must outlive it)."""
    from .gpu import GpuQuantType, GpuWeightBuffer
    keep = []

    def up(a):
        if not isinstance(a, GpuWeightBuffer):
            a = engine.upload_weights_typed(np.ascontiguousarray(a).view(np.uint8), a.shape[0], a.shape[1], GpuQuantType.BF16)
        keep.append(a)
        return a._h

    def vec(a):
        a = np.ascontiguousarray(a, np.float32)
        keep.append(a)
        return a.ctypes.data

    arr = (_lib.StackLayer * len(cfg.layers))()
    for spec, dst, (mats, vecs) in zip(cfg.layers, arr, packed_layers):
        dst.mixer = spec.kind
        for n in ("heads", "kv_heads", "dim", "vdim", "q_rank", "kv_rank", "rot_dim", "rot_dims", "conv_taps", "decay_rank", "gate_rank", "ff",
                  "unit_qk", "scale", "softcap", "rot_base", "rot_factor", "rot_low", "rot_high", "rot_original"):
            setattr(dst, n, getattr(spec, n))
        for n, a in mats.items():
            setattr(dst, n if n != "in" else "in_", up(a))
        for n, a in vecs.items():
            setattr(dst, n, vec(a))
    c = _lib.StackConfig(len(cfg.layers), cfg.width, cfg.vocab_size, cfg.max_seq_len, cfg.loop_start, cfg.loop_stop, cfg.loop_times, int(exact),
                         cfg.family.block, cfg.family.norm, cfg.eps, cfg.embed_scale, cfg.alpha, vec(loop_step) if cfg.loop_times else None,
                         None if head is None else up(head))
    h = C.c_void_p()
    _lib.check(engine._lib.alice_stack_create(engine._h, C.byref(c), arr, up(embed), C.c_void_p(vec(final_norm)), C.byref(h)))
    return h, keep


def load_tensors(engine, config: dict, tensors: dict, dtype: str = "bfloat16", max_seq_len: int = 4096):
    """-> (handle, StackConfig, objects to keep) of a model given as config.json's dict and {name: array}."""
    if dtype not in ("bfloat16", "float32"):
        raise ConfigError(f"dtype {dtype!r} (bfloat16 or float32)")
    cfg, ck = StackConfig(config, max_seq_len), Checkpoint(tensors)
    packed = [pack_layer(ck, i, L, cfg) for i, L in enumerate(cfg.layers)]
    embed = _cols(ck.matrix("embed", cfg.vocab_size, cfg.width), pad(cfg.width))
    step = ck.floats("loop.step", cfg.loop_times, cfg.width) if cfg.loop_times else None
    head = None if cfg.family.tied else _cols(ck.matrix("head", cfg.vocab_size, cfg.width), pad(cfg.width))
    final = ck.floats("final.norm", cfg.width) + np.float32(cfg.family.norm_offset)
    h, keep = create(engine, cfg, packed, embed, final, step, dtype == "float32", head)
    return h, cfg, keep


def load_dir(engine, path, dtype: str = "bfloat16", max_seq_len: int = 4096):
    """A folder with config.json and model.safetensors."""
    with open(os.path.join(path, "config.json")) as f:
        config = json.load(f)
    return load_tensors(engine, config, SafetensorsFile(os.path.join(path, "model.safetensors")).tensors, dtype, max_seq_len)
