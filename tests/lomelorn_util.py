"""Small random Lomelorn models for the tests: configuration, weights, files."""
import json
import os

import numpy as np

from ctox_llm_b200.safetensors import write_safetensors


def bf16(x):
    """fp32 values rounded to bf16 (half up in magnitude), still as fp32."""
    u = (np.ascontiguousarray(x, np.float32).view(np.uint32) + 0x8000) & 0xFFFF0000
    return u.astype(np.uint32).view(np.float32)


def mixer(heads=3, dim=24, rot_dim=8, vdim=40, q_rank=36, kv_rank=56, window=11, base=1000.0, scale=None, kv_from=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
         "mask": {"size": window}, "rot": {"base": base, "dims": rot_dim},
         "scale": (dim + rot_dim) ** -0.5 if scale is None else scale}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return m


def layer(ff=100, **kw):
    return {"type": "latent_attention", "mixer": mixer(**kw), "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def model(layers, vocab=97, width=72, eps=1e-3, softcap=20.0, seed=0):
    """(config, tensors)."""
    config = {"architecture": "Lomelorn", "vocab": vocab, "width": width, "norm": {"eps": eps},
              "logit_softcap": softcap, "layers": layers}
    rng = np.random.default_rng(seed)

    def matrix(rows, cols, gain=1.0):
        return bf16(rng.standard_normal((rows, cols)) * gain / np.sqrt(cols))

    def norm(n):
        return bf16(1.0 + 0.2 * rng.standard_normal(n))

    t = {"embed": bf16(rng.standard_normal((vocab, width))), "final.norm": norm(width), "head": matrix(vocab, width, 4.0)}
    for i, spec in enumerate(layers):
        m, f = spec["mixer"], spec["mlp"]
        p = f"l{i}."
        t[p + "norm1"], t[p + "norm1b"] = norm(width), norm(width)
        t[p + "mix.dq"], t[p + "mix.dq.norm"] = matrix(m["q_rank"], width), norm(m["q_rank"])
        t[p + "mix.uq"] = matrix(m["heads"] * (m["dim"] + m["rot_dim"]), m["q_rank"], 2.0)
        if "kv_from" not in m:
            t[p + "mix.dkv"] = matrix(m["kv_rank"] + m["rot_dim"], width, 1.5)
            t[p + "mix.dkv.norm"] = norm(m["kv_rank"])
        t[p + "mix.uk"] = matrix(m["heads"] * m["dim"], m["kv_rank"])
        t[p + "mix.uv"] = matrix(m["heads"] * m["vdim"], m["kv_rank"])
        t[p + "mix.o"] = matrix(width, m["heads"] * m["vdim"])
        if f is not None:
            t[p + "norm2"], t[p + "norm2b"] = norm(width), norm(width)
            t[p + "mlp.up"], t[p + "mlp.down"] = matrix(f["ff"], width), matrix(width, f["ff"])
    return config, t


def write_model(folder, config, tensors):
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(config, f)
    write_safetensors(os.path.join(folder, "model.safetensors"),
                      {k: ("BF16", v.shape, (np.ascontiguousarray(v, np.float32).view(np.uint32) >> 16).astype(np.uint16))
                       for k, v in tensors.items()})
    return folder


def row_errors(got, want):
    """Per row: rms difference (mean taken off) over the rms of the whole expected array."""
    got, want = np.asarray(got, np.float64), np.asarray(want, np.float64)
    d = got - want
    d = d - d.mean(-1, keepdims=True)
    return np.sqrt((d * d).mean(-1)) / np.sqrt((want * want).mean())
