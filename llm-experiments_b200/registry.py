"""Model registry: which class serves a model folder, by the ``architecture`` of its ``config.json``.

A builder takes ``(ctx, config, weights, dtype, batch_size, max_tokens)`` - the parsed configuration, the checkpoint's tensors,
the storage type, the number of sequences held at a time and the most tokens of one - and returns an object with the interface
``generate_text`` drives (``ctx``, ``context``, ``cache``, ``prefill(tokens)``, ``decode_step(token)``).  Models that also take
prompts in portions have ``forward(entries)`` and ``release(slot)``.
"""
from __future__ import annotations

from typing import Callable, Dict

import torch

from . import checkpoint
from .types import GPUContext

_BUILDERS: Dict[str, Callable] = {}


def register_model(architecture: str):
    def wrap(builder):
        _BUILDERS[architecture] = builder
        return builder

    return wrap


def architectures():
    _import_models()
    return sorted(_BUILDERS)


def _import_models() -> None:
    from . import bamasun, gigezen, model  # noqa: F401  (they register themselves)


def build_model(ctx: GPUContext, config: dict, weights: Dict[str, torch.Tensor], dtype: torch.dtype = torch.bfloat16,
                batch_size: int = 1, max_tokens: int = 4096):
    _import_models()
    name = config.get("architecture")
    if name not in _BUILDERS:
        raise ValueError(f"unknown architecture {name!r}; known: {', '.join(sorted(_BUILDERS))}")
    return _BUILDERS[name](ctx, config, weights, dtype, batch_size, max_tokens)


def load_model(ctx: GPUContext, folder, dtype: torch.dtype = torch.bfloat16, batch_size: int = 1, max_tokens: int = 4096):
    """The model of a folder with ``config.json`` and ``model.safetensors``, on the context's device."""
    return build_model(ctx, checkpoint.read_config(folder), checkpoint.load_folder(folder), dtype, batch_size, max_tokens)
