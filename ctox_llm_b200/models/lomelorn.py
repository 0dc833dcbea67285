"""Lomelorn models: latent attention inside sliding windows, layer norms around every sublayer,
squared-relu feed-forwards, tanh-capped logits. The folder holds config.json (keys read below) and
model.safetensors (tensor names in load_weights)."""
from __future__ import annotations

import os

from .. import _native as N
from .._native import CtoxError
from ..backend import FusedMatVec
from ..executor import B200Executor, StackConfig
from ..safetensors import SafetensorsFile
from . import register

SHAPE, UNSUPPORTED_OPERATION = 1, 4
PAGE_TOKENS = 128


def layer_config(index: int, layer: dict) -> N.LayerConfig:
    if layer.get("type") != "latent_attention":
        raise CtoxError(UNSUPPORTED_OPERATION, f"layer {index}: mixer {layer.get('type')!r}")
    mixer, mlp = layer["mixer"], layer.get("mlp")
    if mlp is not None and mlp.get("kind") != "dense":
        raise CtoxError(UNSUPPORTED_OPERATION, f"layer {index}: feed-forward {mlp.get('kind')!r}")
    rot_dim = int(mixer["rot_dim"])
    if int(mixer["rot"]["dims"]) != rot_dim:
        raise CtoxError(SHAPE, f"layer {index}: the rotation covers {mixer['rot']['dims']} of {rot_dim} dimensions")
    window = int(mixer["mask"]["size"])
    if window < 1:
        raise CtoxError(SHAPE, f"layer {index}: a window of {window} tokens")
    source = mixer.get("kv_from")
    return N.LayerConfig(
        mixer=N.MIXER_LATENT_ATTENTION, heads=int(mixer["heads"]), dim=int(mixer["dim"]), rot_dim=rot_dim,
        vdim=int(mixer["vdim"]), q_rank=int(mixer["q_rank"]), kv_rank=int(mixer["kv_rank"]), window=window,
        rope_base=float(mixer["rot"]["base"]), score_scale=float(mixer["scale"]),
        kv_from=-1 if source is None else int(source),
        mlp=N.MLP_NONE if mlp is None else N.MLP_RELU2, ff=0 if mlp is None else int(mlp["ff"]))


def stack_config(config: dict, dtype: str, max_context_tokens: int, page_tokens: int = PAGE_TOKENS,
                 pass_tokens: int = 0) -> StackConfig:
    layers = [layer_config(i, layer) for i, layer in enumerate(config["layers"])]
    return StackConfig(
        vocab_size=int(config["vocab"]), hidden_size=int(config["width"]), layers=layers,
        norm_eps=float(config["norm"]["eps"]), logit_softcap=float(config.get("logit_softcap") or 0.0),
        max_context_tokens=max_context_tokens, kv_page_tokens=page_tokens,
        kv_dtype=N.F32 if dtype == "float32" else N.BF16, pass_tokens=pass_tokens)


def load_weights(weights: SafetensorsFile, ex: B200Executor) -> None:
    def matrix(layer, tensor, name):
        data, rows, columns = weights.bf16_matrix(name)
        ex.load_matrix(layer, tensor, FusedMatVec(N.BF16, data, rows, columns, None))

    def vector(layer, tensor, name):
        ex.load_vector(layer, tensor, weights.float_vector(name))

    matrix(N.LAYER_GLOBAL, N.T_EMBED, "embed")
    matrix(N.LAYER_GLOBAL, N.T_LM_HEAD, "head")
    vector(N.LAYER_GLOBAL, N.T_FINAL_NORM, "final.norm")
    for i, layer in enumerate(ex.config.layers):
        p = f"l{i}."
        vector(i, N.T_INPUT_NORM, p + "norm1")
        vector(i, N.T_MIX_OUT_NORM, p + "norm1b")
        matrix(i, N.T_Q_DOWN, p + "mix.dq")
        vector(i, N.T_Q_DOWN_NORM, p + "mix.dq.norm")
        matrix(i, N.T_Q_UP, p + "mix.uq")
        if layer.kv_from < 0:
            matrix(i, N.T_KV_DOWN, p + "mix.dkv")
            vector(i, N.T_KV_DOWN_NORM, p + "mix.dkv.norm")
        matrix(i, N.T_K_UP, p + "mix.uk")
        matrix(i, N.T_V_UP, p + "mix.uv")
        matrix(i, N.T_ATTN_O, p + "mix.o")
        if layer.mlp != N.MLP_NONE:
            vector(i, N.T_POST_NORM, p + "norm2")
            vector(i, N.T_MLP_OUT_NORM, p + "norm2b")
            matrix(i, N.T_MLP_UP, p + "mlp.up")
            matrix(i, N.T_MLP_DOWN, p + "mlp.down")


def open_lomelorn(backend, folder, config, dtype, max_context_tokens, **options):
    ex = B200Executor(backend, stack_config(config, dtype, max_context_tokens, **options))
    try:
        load_weights(SafetensorsFile(os.path.join(folder, "model.safetensors")), ex)
    except Exception:
        ex.unload()
        raise
    return ex


register("Lomelorn", open_lomelorn)
