"""Model registry: what a path holds -> the loader of its architecture -> a decoder session.  A folder with config.json
is looked up by its "architecture", a GGUF file by its general.architecture key."""
from __future__ import annotations

import json
import os

import emel_cpp_b200 as eb


def _metulix(backend, path, n_ctx, float32):
    from emel_cpp_b200 import metulix
    return metulix.load(backend, path, n_ctx=n_ctx or 4096, float32=float32)


def _sugonex(backend, path, n_ctx, float32):
    from emel_cpp_b200 import sugonex
    return sugonex.load(backend, path, n_ctx=n_ctx or 4096, float32=float32)


def _llama(backend, path, n_ctx, float32):
    from emel_cpp_b200 import gguf
    if float32:
        raise ValueError("block-quantized models run in their own formats")
    with gguf.File(path) as f:
        return gguf.load_llama(backend, f, n_ctx)


ARCHITECTURES = {"Metulix": _metulix, "Sugonex": _sugonex, "llama": _llama}


def architecture(path: str) -> str:
    if os.path.isdir(path):
        with open(os.path.join(path, "config.json")) as f:
            return json.load(f)["architecture"]
    from emel_cpp_b200 import gguf
    with gguf.File(path) as f:
        return f.get("general.architecture", "llama")


def load(backend: eb.Backend, path: str, n_ctx: int | None = None, float32: bool = False):
    """A decoder session of the model at `path`; n_ctx: token positions its sequences can hold (default: the model's)."""
    name = architecture(path)
    if name not in ARCHITECTURES:
        raise ValueError(f"unknown architecture {name!r} (known: {', '.join(sorted(ARCHITECTURES))})")
    return ARCHITECTURES[name](backend, path, n_ctx, float32)
