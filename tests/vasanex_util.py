"""Small random Vasanex models for the tests."""
import numpy as np

from lomelorn_util import bf16, row_errors, write_model  # noqa: F401  (shared helpers of the layer-stack tests)


def attention(heads=6, kv_heads=2, dim=24, vdim=40, window=11, base=900.0, rot=None, scale=None, v_mix=True, ff=72, limit=1.3):
    return {"type": "attention", "mlp": dense(ff, limit),
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": window},
                      "rot": {"base": base, "dims": dim // 4 * 2 if rot is None else rot},
                      "scale": dim ** -0.5 if scale is None else scale, "v_mix": v_mix}}


def mlstm(heads=3, dim=20, vdim=28, gate_cap=12.0, ff=None, limit=1.3):
    return {"type": "mlstm", "mlp": dense(ff, limit), "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": gate_cap}}


def dense(ff, limit):
    return None if ff is None else {"kind": "dense", "ff": ff, "limit": limit}


def model(layers, vocab=89, width=76, eps=1e-3, embed_scale=2.5, seed=0):
    """(config, tensors)."""
    config = {"architecture": "Vasanex", "vocab": vocab, "width": width, "norm": {"eps": eps},
              "embedding": {"scale": embed_scale}, "layers": layers}
    rng = np.random.default_rng(seed)

    def matrix(rows, cols, gain=1.0):
        return bf16(rng.standard_normal((rows, cols)) * gain / np.sqrt(cols))

    def vector(n, std, mean=0.0):
        return bf16(mean + std * rng.standard_normal(n))

    t = {"embed": matrix(vocab, width, 4.0), "final.norm": vector(width, 0.2)}
    for i, spec in enumerate(layers):
        m, p = spec["mixer"], f"l{i}.mix."
        H, dim, vdim = m["heads"], m["dim"], m["vdim"]
        t[f"l{i}.norm1"] = vector(width, 0.2)
        if spec["type"] == "attention":
            G = m["kv_heads"]
            for name, rows, norm in (("q", H * dim, True), ("k", G * dim, True), ("v", G * vdim, False)):
                t[p + name], t[p + name + ".b"] = matrix(rows, width), vector(rows, 0.3)
                if norm:
                    t[p + name + ".norm"] = vector(rows, 0.3, 1.5)
            t[p + "vmix"], t[p + "sink"] = vector(1, 0.1, 0.4).reshape(()), vector(H, 1.0)
            t[p + "o"], t[p + "o.b"] = matrix(width, H * vdim, 1.5), vector(width, 0.3)
        else:
            t[p + "q"], t[p + "k"], t[p + "v"] = matrix(H * dim, width), matrix(H * dim, width), matrix(H * vdim, width)
            t[p + "g"], t[p + "o"], t[p + "norm"] = matrix(H * vdim, width), matrix(width, H * vdim), vector(H * vdim, 0.2, 1.0)
            t[p + "i"], t[p + "i.b"] = matrix(H, width, 2.0), vector(H, 0.5, -0.5)
            t[p + "f"], t[p + "f.b"] = matrix(H, width, 1.0), vector(H, 0.5, 4.0)
        if spec["mlp"] is not None:
            ff = spec["mlp"]["ff"]
            t[f"l{i}.norm2"] = vector(width, 0.2)
            t[f"l{i}.mlp.gate"], t[f"l{i}.mlp.up"] = matrix(ff, width), matrix(ff, width)
            t[f"l{i}.mlp.down"] = matrix(width, ff)
    return config, t
