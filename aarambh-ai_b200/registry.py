"""Model registry: which loader serves a checkpoint.

A folder is recognised by the ``architecture`` its ``config.json`` names, a ``.gguf`` file by
its suffix.  A loader is a function ``load(path, dtype, max_tokens, max_seq_len)`` that
returns a ``DecoderModel``.
"""
from __future__ import annotations

import json
import os

import torch

from .model import DecoderModel

_ARCHITECTURES = {}


class UnknownModelError(ValueError):
    pass


def register(architecture: str):
    """Decorator: registers the loader of folders whose config.json names ``architecture``."""
    def add(loader):
        _ARCHITECTURES[architecture] = loader
        return loader
    return add


def architectures() -> list:
    return sorted(_ARCHITECTURES)


def loader_for(path: str):
    if path.endswith(".gguf"):
        from .gguf import load_gguf_model

        def load(path, dtype, max_tokens, max_seq_len):
            return load_gguf_model(path, dtype, max_tokens)  # the file holds its max_seq_len
        return load
    config = os.path.join(path, "config.json")
    if not os.path.isfile(config):
        raise UnknownModelError(f"{path} is neither a .gguf file nor a folder with a config.json")
    with open(config) as f:
        name = json.load(f).get("architecture")
    if name not in _ARCHITECTURES:
        raise UnknownModelError(f"architecture {name!r} is not registered (known: {', '.join(architectures())})")
    return _ARCHITECTURES[name]


def load_model(path: str, dtype: torch.dtype = torch.bfloat16, max_tokens: int = 512, max_seq_len: int = 4096) -> DecoderModel:
    """Loads a checkpoint onto the current GPU.  ``max_tokens`` bounds the tokens of one forward
    call, ``max_seq_len`` the positions of a sequence (where the checkpoint does not say)."""
    return loader_for(path)(path, dtype, max_tokens, max_seq_len)
