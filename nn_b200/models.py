"""Model registry: a path on disk -> a decoder ready to run.

A folder with config.json and model.safetensors is loaded by the entry named by config.json's
'architecture'; a GGUF file by the entry named by its general.architecture. Every loader returns an object
with the decoder interface (prefill / step / extend / state / generate / complete).
"""
from __future__ import annotations

import json
import os
from typing import Callable, Dict, Optional

from . import api

_FOLDERS: Dict[str, Callable] = {}
_GGUF: Dict[str, Callable] = {}


class UnknownArchitecture(api.TensorError):
    pass


def register_folder_model(name: str):
    """Decorator: loader(config, folder, backend, max_seq, act_dtype, **options) for config.json's 'architecture'."""
    def add(fn):
        _FOLDERS[name] = fn
        return fn
    return add


def register_gguf_model(name: str):
    """Decorator: loader(file, backend, max_seq, act_dtype, **options) for general.architecture."""
    def add(fn):
        _GGUF[name] = fn
        return fn
    return add


def architectures():
    return sorted(_FOLDERS) + sorted(_GGUF)


def load_model(path: str, backend: Optional[api.Backend] = None, *, max_seq: int, act_dtype: int = api.BF16, **options):
    if os.path.isdir(path):
        with open(os.path.join(path, "config.json")) as f:
            config = json.load(f)
        name = config.get("architecture")
        if name not in _FOLDERS:
            raise UnknownArchitecture(f"architecture {name!r} is not registered (have {', '.join(architectures())})")
        return _FOLDERS[name](config, path, backend, max_seq, act_dtype, **options)
    from . import gguf
    f = gguf.GgufFile.open(path, accept_standard_magic=True)
    name = f.architecture()
    if name not in _GGUF:
        raise UnknownArchitecture(f"architecture {name!r} is not registered (have {', '.join(architectures())})")
    return _GGUF[name](f, backend, max_seq, act_dtype, **options)


@register_folder_model("Sikivik")
def _sikivik(config, folder, backend, max_seq, act_dtype, **options):
    from . import sikivik
    return sikivik.load(config, os.path.join(folder, "model.safetensors"), backend, max_seq=max_seq, act_dtype=act_dtype, **options)


@register_folder_model("Rugesun")
def _rugesun(config, folder, backend, max_seq, act_dtype, **options):
    from . import rugesun
    return rugesun.load(config, os.path.join(folder, "model.safetensors"), backend, max_seq=max_seq, act_dtype=act_dtype, **options)


@register_gguf_model("qwen3")
def _qwen3(f, backend, max_seq, act_dtype, **options):
    from . import gguf
    return gguf.load_qwen3_decoder(f, backend, max_seq=max_seq, act_dtype=act_dtype, **options)[0]
