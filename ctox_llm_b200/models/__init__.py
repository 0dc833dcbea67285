"""Model registry: a model folder's config.json names its architecture, the registry opens it.

    ex = open_model("folder", max_context_tokens=4096)      # loaded and warm
    for token in ex.generate(prompt, max_new_tokens=32): ...

An architecture module calls `register(name, opener)`; the opener gets (backend, folder, config,
dtype, max_context_tokens) and returns a loaded B200Executor.
"""
from __future__ import annotations

import json
import os
from typing import Callable, Dict, Optional

from .._native import CtoxError
from ..backend import B200Backend

INVALID_ARTIFACT, UNSUPPORTED_DTYPE, UNSUPPORTED_OPERATION = 2, 3, 4
DTYPES = ("bfloat16", "float32")
_OPENERS: Dict[str, Callable] = {}


def register(architecture: str, opener: Callable) -> None:
    _OPENERS[architecture] = opener


def architectures() -> list:
    return sorted(_OPENERS)


def read_config(folder: str) -> dict:
    with open(os.path.join(folder, "config.json")) as f:
        config = json.load(f)
    if not isinstance(config, dict) or config.get("architecture") not in _OPENERS:
        name = config.get("architecture") if isinstance(config, dict) else None
        raise CtoxError(UNSUPPORTED_OPERATION, f"architecture {name!r} is not one of {', '.join(architectures())}")
    return config


def open_model(folder: str, backend: Optional[B200Backend] = None, dtype: str = "bfloat16",
               max_context_tokens: int = 4096, **options):
    """Creates, loads and warms the executor of the model in `folder`. dtype "float32" runs everything
    in 32-bit. Further options go to the architecture's opener."""
    if dtype not in DTYPES:
        raise CtoxError(UNSUPPORTED_DTYPE, f"dtype {dtype!r} is not one of {', '.join(DTYPES)}")
    config = read_config(folder)
    backend = backend or B200Backend()
    executor = _OPENERS[config["architecture"]](backend, folder, config, dtype, max_context_tokens, **options)
    try:
        executor.warmup()
    except Exception:
        executor.unload()
        raise
    return executor


from . import lomelorn, qwen38, vasanex  # noqa: E402,F401  (they register themselves)
