"""Qwen3.8-27B-shaped hybrid models: a folder with config.json (the fields of ModelConfig) and
model.ctoxq (the packed container)."""
from __future__ import annotations

import os

from .. import _native as N
from ..artifact import CtoxqArtifact, load_into_executor
from ..executor import B200Executor, qwen38_27b_config
from . import register


def model_config(config: dict, dtype: str, max_context_tokens: int) -> N.ModelConfig:
    names = {n for n, _ in N.ModelConfig._fields_}
    fields = {k: v for k, v in config.items() if k in names}
    fields.update(kv_dtype=N.F32 if dtype == "float32" else N.BF16, max_context_tokens=max_context_tokens)
    return qwen38_27b_config(**fields)


def open_qwen38(backend, folder, config, dtype, max_context_tokens):
    ex = B200Executor(backend, model_config(config, dtype, max_context_tokens))
    art = CtoxqArtifact.open(os.path.join(folder, "model.ctoxq"))
    try:
        load_into_executor(art, ex, config.get("draft_token_ids"))
    finally:
        art.close()
    return ex


register("Qwen38", open_qwen38)
