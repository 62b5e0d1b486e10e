"""Models by architecture.  ``load_model`` takes what a model is stored as — a GGUF file (GPT-2) or a
folder with ``config.json`` (its "architecture" names the class) — and returns a
:class:`caten_b200.model.Model`."""
from __future__ import annotations

import json
import os
from typing import Optional

from .model import Model
from .runtime import B200Runtime


def _gpt2(path: str, runtime: Optional[B200Runtime], **kw) -> Model:
    from .gpt2 import make_gpt2_from_gguf
    return make_gpt2_from_gguf(path, runtime, **kw)


def _binusun(path: str, runtime: Optional[B200Runtime], **kw) -> Model:
    from . import binusun
    return binusun.load(path, runtime, **kw)


def _goselix(path: str, runtime: Optional[B200Runtime], **kw) -> Model:
    from . import goselix
    return goselix.load(path, runtime, **kw)


ARCHITECTURES = {"gpt2": _gpt2, "Binusun": _binusun, "Goselix": _goselix}


def architecture_of(path: str) -> str:
    if os.path.isdir(path):
        with open(os.path.join(path, "config.json")) as f:
            return str(json.load(f).get("architecture"))
    from .gguf import load_gguf
    g = load_gguf(path)
    try:
        return str(g.metadata.get("general.architecture", "gpt2"))
    finally:
        g.close()


def load_model(path: str, runtime: Optional[B200Runtime] = None, **kw) -> Model:
    """``kw``: max_seq_len, batch, precision ("fp32", "bf16", "bf16x3") and what the class takes besides."""
    arch = architecture_of(path)
    if arch not in ARCHITECTURES:
        raise ValueError(f"unknown architecture {arch!r} (known: {', '.join(sorted(ARCHITECTURES))})")
    return ARCHITECTURES[arch](path, runtime, **kw)
