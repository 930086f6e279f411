"""Which class serves a model: a GGUF file by its `general.architecture`, a folder by the `architecture` of its config.json.

    engine = load_engine(path, gpu=None, dtype="bfloat16", slots=8)
    engine.generate([[1, 2, 3]], max_new=16)
"""
from __future__ import annotations

import json
import os
from typing import Callable, Dict

from .runtime import GpuContext, init_gpu

# architecture -> loader(path, **options) -> engine
FOLDERS: Dict[str, Callable] = {}
FILES: Dict[str, Callable] = {}


def folder_model(architecture: str):
    def put(f):
        FOLDERS[architecture] = f
        return f
    return put


def file_model(architecture: str):
    def put(f):
        FILES[architecture] = f
        return f
    return put


def _slot_engine(model, path, gpu=None, dtype="bfloat16", slots=1, capacity=0, step_rows=2048, portion=0, **_):
    from .engine import Engine

    return Engine(model.load(path, gpu or GpuContext(component="lm"), dtype=dtype, slots=slots, capacity=capacity, step_rows=step_rows), portion=portion)


@folder_model("Sonalorn")
def _sonalorn(path, **options):
    from .sonalorn import SonalornModel

    return _slot_engine(SonalornModel, path, **options)


@folder_model("Bubotar")
def _bubotar(path, **options):
    from .bubotar import BubotarModel

    return _slot_engine(BubotarModel, path, **options)


@file_model("llama")
def _llama(path, gpu=None, dtype="int8", slots=1, capacity=0, gguf=None, **_):
    from . import llama_gguf
    from .engine import LockstepEngine

    if dtype != "int8":
        raise ValueError("llama runs on the int8 path (dtype int8)")
    decoder, _gguf = llama_gguf.from_gguf(gguf if gguf is not None else path, gpu or init_gpu(), batch=slots, capacity=capacity or None)
    return LockstepEngine(decoder)


def load_engine(path: str, **options):
    """options: gpu, dtype, slots (sequences at once), capacity (positions of each), step_rows, portion."""
    if os.path.isdir(path):
        with open(os.path.join(path, "config.json")) as f:
            arch = json.load(f).get("architecture")
        if arch not in FOLDERS:
            raise ValueError(f"{path}: architecture {arch!r}; known: {', '.join(sorted(FOLDERS))}")
        options.setdefault("dtype", "bfloat16")
        return FOLDERS[arch](path, **options)
    from .gguf_file import GgufFile

    gpu = options.pop("gpu", None) or init_gpu()
    gguf = GgufFile.load(path, gpu)
    arch = gguf.get_metadata("general.architecture") or "llama"
    if arch not in FILES:
        raise ValueError(f"{path}: architecture {arch!r}; known: {', '.join(sorted(FILES))}")
    options.setdefault("dtype", "int8")
    return FILES[arch](path, gpu=gpu, gguf=gguf, **options)
