"""Which decoder serves a model: by `general.architecture` of a GGUF file, or by `architecture` of a folder's config.json.

    dec = load_model(Backend(), path, dtype="bfloat16")
"""
from __future__ import annotations

import json
import os
from typing import Callable

from .backend import ACT_FP32, ACT_INT8, Backend
from .decoder import Decoder


class UnknownModel(ValueError):
    pass


class UnsupportedDtype(ValueError):
    """No decoder of this architecture computes in the precision asked for."""


def _llama(backend: Backend, path: str, dtype: str, max_positions: int | None) -> Decoder:
    # Q8_0 weights: "bfloat16" is the serving default (int8 activation codes); "float32" the two-digit activations, whose products
    # are fp32-equivalent but not fp32 arithmetic, so it is not offered under that name
    from .llama import LlamaDecoder
    if dtype == "float32":
        raise UnsupportedDtype("the Q8_0 llama decoder has no 32-bit arithmetic; act_mode=ACT_FP32 is its closest mode")
    return LlamaDecoder.from_gguf(backend, path, act_mode=ACT_INT8, prompt_act_mode=ACT_FP32, max_positions=max_positions)


def _kipirax(backend: Backend, path: str, dtype: str, max_positions: int | None) -> Decoder:
    from .kipirax import KipiraxDecoder
    return KipiraxDecoder.load(backend, path, dtype=dtype, max_positions=max_positions)


def _sikivik(backend: Backend, path: str, dtype: str, max_positions: int | None) -> Decoder:
    from .sikivik import SikivikDecoder
    return SikivikDecoder.load(backend, path, dtype=dtype, max_positions=max_positions)


MODELS: dict[str, Callable[[Backend, str, str, "int | None"], Decoder]] = {"llama": _llama, "Kipirax": _kipirax, "Sikivik": _sikivik}


def architecture_of(path: str) -> str:
    if os.path.isdir(path):
        config = os.path.join(path, "config.json")
        if not os.path.exists(config):
            raise UnknownModel(f"{path}: no config.json")
        with open(config) as f:
            name = json.load(f).get("architecture")
    else:
        from . import gguf
        with gguf.GgufFile(path) as g:
            name = g.metadata.get("general.architecture")
    if name not in MODELS:
        raise UnknownModel(f"{path}: architecture {name!r} is not served; known: {', '.join(sorted(MODELS))}")
    return name


def load_model(backend: Backend, path: str, dtype: str = "bfloat16", max_positions: int | None = None) -> Decoder:
    """The model at `path`, resident and with its step graphs captured."""
    if dtype not in ("bfloat16", "float32"):
        raise UnsupportedDtype(f"dtype {dtype!r}")
    dec = MODELS[architecture_of(path)](backend, path, dtype, max_positions)
    dec.capture()
    return dec
