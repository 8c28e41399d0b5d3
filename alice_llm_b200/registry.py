"""Which loader serves which architecture, and opening a model without knowing beforehand.

GGUF files name theirs in ``general.architecture`` (the reference's ModelArch, src/llama3.rs:74-236), checkpoint folders in
config.json's ``architecture``."""
from __future__ import annotations

import json
import os


def _llama(engine, path, dtype, max_seq_len):
    from .gpu import GpuModel
    if dtype != "bfloat16":
        raise ValueError("quantized GGUF models have no 32-bit mode")
    return GpuModel.load_gguf(engine, path, max_seq_len)


def _stack(engine, path, dtype, max_seq_len):
    from .gpu import GpuModel
    return GpuModel.load_stack(engine, path, dtype=dtype, max_seq_len=max_seq_len)


# architecture -> (loader, part of the native library it runs on)
ARCHITECTURES = {"llama": (_llama, "all"), "Zamitar": (_stack, "stack"), "Suborax": (_stack, "stack")}


def architecture_of(path) -> str:
    """The architecture a model folder or GGUF file declares."""
    if os.path.isdir(path):
        with open(os.path.join(path, "config.json")) as f:
            return str(json.load(f).get("architecture"))
    from .gguf_file import GgufFile
    return str(GgufFile.open(path).metadata.get("general.architecture", "llama"))


def lookup(path):
    arch = architecture_of(path)
    if arch not in ARCHITECTURES:
        raise ValueError(f"architecture {arch!r} is not supported (known: {', '.join(ARCHITECTURES)})")
    return ARCHITECTURES[arch]


def open_model(path, engine=None, dtype: str = "bfloat16", max_seq_len: int = 4096, device: int = 0):
    """-> GpuModel on `engine` (a new one on `device` if none is given)."""
    from . import _lib
    loader, part = lookup(path)
    if engine is None:
        _lib.prefer(part)
        from .gpu import GpuEngine
        engine = GpuEngine(device)
    return loader(engine, path, dtype, max_seq_len)
