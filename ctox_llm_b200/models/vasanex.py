"""Vasanex models: grouped attention with normed queries and keys, sliding windows, sinks and mixed values, and
matrix memories (mLSTM), in any order; clamped gated feed-forwards; tied logits. The folder holds config.json
(keys read below) and model.safetensors (tensor names in load_weights)."""
from __future__ import annotations

import os

import numpy as np

from .. import _native as N
from .._native import CtoxError
from ..backend import FusedMatVec
from ..executor import B200Executor, StackConfig
from ..safetensors import SafetensorsFile
from . import register

SHAPE, UNSUPPORTED_OPERATION = 1, 4
PAGE_TOKENS = 128
GLU_SLOPE = 1.702  # of the sigmoid in the feed-forward's gate


def feed_forward(index: int, mlp) -> dict:
    if mlp is None:
        return {"mlp": N.MLP_NONE}
    if mlp.get("kind") != "dense":
        raise CtoxError(UNSUPPORTED_OPERATION, f"layer {index}: feed-forward {mlp.get('kind')!r}")
    return {"mlp": N.MLP_CLAMPED_GLU, "ff": int(mlp["ff"]), "mlp_limit": float(mlp["limit"]), "mlp_slope": GLU_SLOPE}


def attention(index: int, mixer: dict) -> dict:
    window = int(mixer["mask"]["size"])
    if window < 1:
        raise CtoxError(SHAPE, f"layer {index}: a window of {window} tokens")
    options = N.ATTN_BIAS | N.ATTN_QK_NORM | N.ATTN_SINK | (N.ATTN_V_MIX if mixer.get("v_mix") else 0)
    return {"mixer": N.MIXER_GROUPED_ATTENTION, "kv_heads": int(mixer["kv_heads"]), "rot_dim": int(mixer["rot"]["dims"]),
            "rope_base": float(mixer["rot"]["base"]), "window": window, "score_scale": float(mixer["scale"]), "attn": options}


def matrix_memory(index: int, mixer: dict) -> dict:
    return {"mixer": N.MIXER_MATRIX_MEMORY, "gate_cap": float(mixer["gate_cap"])}


MIXERS = {"attention": attention, "mlstm": matrix_memory}


def layer_config(index: int, layer: dict) -> N.LayerConfig:
    if layer.get("type") not in MIXERS:
        raise CtoxError(UNSUPPORTED_OPERATION, f"layer {index}: mixer {layer.get('type')!r}")
    mixer = layer["mixer"]
    return N.LayerConfig(heads=int(mixer["heads"]), dim=int(mixer["dim"]), vdim=int(mixer["vdim"]), kv_from=-1,
                         **MIXERS[layer["type"]](index, mixer), **feed_forward(index, layer.get("mlp")))


def stack_config(config: dict, dtype: str, max_context_tokens: int, page_tokens: int = PAGE_TOKENS,
                 pass_tokens: int = 0) -> StackConfig:
    return StackConfig(
        vocab_size=int(config["vocab"]), hidden_size=int(config["width"]),
        layers=[layer_config(i, layer) for i, layer in enumerate(config["layers"])],
        norm_eps=float(config["norm"]["eps"]), logit_softcap=0.0, max_context_tokens=max_context_tokens,
        kv_page_tokens=page_tokens, kv_dtype=N.F32 if dtype == "float32" else N.BF16, pass_tokens=pass_tokens,
        norm=N.NORM_RMS, out_norms=False, tied_head=True, embed_scale=float(config["embedding"]["scale"]))


def load_weights(weights: SafetensorsFile, ex: B200Executor) -> None:
    def matrix(layer, tensor, name):
        data, rows, columns = weights.bf16_matrix(name)
        ex.load_matrix(layer, tensor, FusedMatVec(N.BF16, data, rows, columns, None))

    def vector(layer, tensor, name):
        ex.load_vector(layer, tensor, weights.float_vector(name))

    def norm(layer, tensor, name):  # stored around zero
        ex.load_vector(layer, tensor, np.float32(1.0) + weights.float_vector(name))

    matrix(N.LAYER_GLOBAL, N.T_EMBED, "embed")
    norm(N.LAYER_GLOBAL, N.T_FINAL_NORM, "final.norm")
    for i, layer in enumerate(ex.config.layers):
        p = f"l{i}."
        norm(i, N.T_INPUT_NORM, p + "norm1")
        matrix(i, N.T_MIX_Q, p + "mix.q")
        matrix(i, N.T_MIX_K, p + "mix.k")
        matrix(i, N.T_MIX_V, p + "mix.v")
        matrix(i, N.T_ATTN_O, p + "mix.o")
        if layer.mixer == N.MIXER_GROUPED_ATTENTION:
            vector(i, N.T_MIX_Q_BIAS, p + "mix.q.b")
            vector(i, N.T_MIX_K_BIAS, p + "mix.k.b")
            vector(i, N.T_MIX_V_BIAS, p + "mix.v.b")
            vector(i, N.T_MIX_O_BIAS, p + "mix.o.b")
            vector(i, N.T_Q_NORM, p + "mix.q.norm")
            vector(i, N.T_K_NORM, p + "mix.k.norm")
            vector(i, N.T_ATTN_SINK, p + "mix.sink")
            if layer.attn & N.ATTN_V_MIX and p + "mix.vmix" in weights.tensors:
                vector(i, N.T_V_MIX, p + "mix.vmix")
        else:
            matrix(i, N.T_MIX_GATE, p + "mix.g")
            vector(i, N.T_MIX_HEAD_NORM, p + "mix.norm")
            matrix(i, N.T_MEM_IN, p + "mix.i")
            vector(i, N.T_MEM_IN_BIAS, p + "mix.i.b")
            matrix(i, N.T_MEM_FORGET, p + "mix.f")
            vector(i, N.T_MEM_FORGET_BIAS, p + "mix.f.b")
        if layer.mlp != N.MLP_NONE:
            norm(i, N.T_POST_NORM, p + "norm2")
            matrix(i, N.T_MLP_GATE, p + "mlp.gate")
            matrix(i, N.T_MLP_UP, p + "mlp.up")
            matrix(i, N.T_MLP_DOWN, p + "mlp.down")


def open_vasanex(backend, folder, config, dtype, max_context_tokens, **options):
    ex = B200Executor(backend, stack_config(config, dtype, max_context_tokens, **options))
    try:
        load_weights(SafetensorsFile(os.path.join(folder, "model.safetensors")), ex)
    except Exception:
        ex.unload()
        raise
    return ex


register("Vasanex", open_vasanex)
