"""Plain float64 implementation of the Lomelorn design, one function per mechanism.

Slow and direct: every token looks at every key it may see, nothing is cached, nothing is fused or
absorbed. It shares no code with the package; the product's results are compared against it.
`tokens` of a sequence always start at position 0.
"""
import numpy as np


def layer_norm(x, w, eps):
    mean = x.mean(-1, keepdims=True)
    var = ((x - mean) ** 2).mean(-1, keepdims=True)
    return (x - mean) / np.sqrt(var + eps) * w


def rms_norm(x, w, eps):
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps) * w


def rotate_pairs(x, positions, base):
    """x [..., tokens, dims]: the pair (2i, 2i + 1) turned by position * base^(-2i / dims)."""
    dims = x.shape[-1]
    out = np.array(x)
    for i in range(dims // 2):
        angle = positions * base ** (-2.0 * i / dims)
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * np.cos(angle) - v * np.sin(angle)
        out[..., 2 * i + 1] = v * np.cos(angle) + u * np.sin(angle)
    return out


def visible(n, window):
    """[n, n]: query i sees key j."""
    i, j = np.arange(n)[:, None], np.arange(n)[None, :]
    return (j <= i) & (i - j < window)


def latent_queries(h, t, mixer, eps):
    """[heads, tokens, dim] unrotated part and [heads, tokens, rot_dim] rotated part."""
    H, dim, rot = mixer["heads"], mixer["dim"], mixer["rot_dim"]
    c_q = rms_norm(h @ t["dq"].T, t["dq.norm"], eps)
    q = (c_q @ t["uq"].T).reshape(len(h), H, dim + rot).transpose(1, 0, 2)
    return q[..., :dim], rotate_pairs(q[..., dim:], np.arange(len(h)), mixer["rot"]["base"])


def latent_keys(h, t, mixer, eps):
    """The latent [tokens, kv_rank] and the rotated key part [tokens, rot_dim] all heads share."""
    rank = mixer["kv_rank"]
    down = h @ t["dkv"].T
    c = rms_norm(down[:, :rank], t["dkv.norm"], eps)
    return c, rotate_pairs(down[:, rank:], np.arange(len(h)), mixer["rot"]["base"])


def latent_attention(h, t, mixer, eps, c, k_rot):
    H, dim, vdim = mixer["heads"], mixer["dim"], mixer["vdim"]
    q_plain, q_rot = latent_queries(h, t, mixer, eps)
    see = visible(len(h), mixer["mask"]["size"])
    heads = []
    for n in range(H):
        k = c @ t["uk"][n * dim:(n + 1) * dim].T
        v = c @ t["uv"][n * vdim:(n + 1) * vdim].T
        score = (q_plain[n] @ k.T + q_rot[n] @ k_rot.T) * mixer["scale"]
        score = np.where(see, score, -np.inf)
        p = np.exp(score - score.max(-1, keepdims=True))
        heads.append((p / p.sum(-1, keepdims=True)) @ v)
    return np.concatenate(heads, -1) @ t["o"].T


def feed_forward(h, up, down):
    return np.maximum(h @ up.T, 0.0) ** 2 @ down.T


def softcap(z, cap):
    return cap * np.tanh(z / cap)


def layer_tensors(tensors, l, part):
    prefix = f"l{l}.{part}."
    return {k[len(prefix):]: v for k, v in tensors.items() if k.startswith(prefix)}


def forward(config, tensors, tokens):
    """(logits [tokens, vocab], residual stream after every layer [layers, tokens, width])."""
    t = {k: np.asarray(v, np.float64) for k, v in tensors.items()}
    eps = config["norm"]["eps"]
    x = t["embed"][np.asarray(tokens)]
    kept, streams = {}, []
    for l, layer in enumerate(config["layers"]):
        mixer, mlp = layer["mixer"], layer["mlp"]
        mt = layer_tensors(t, l, "mix")
        h = layer_norm(x, t[f"l{l}.norm1"], eps)
        source = mixer.get("kv_from")
        if source is None:
            kept[l] = latent_keys(h, mt, mixer, eps)
        c, k_rot = kept[l if source is None else source]
        x = x + layer_norm(latent_attention(h, mt, mixer, eps, c, k_rot), t[f"l{l}.norm1b"], eps)
        if mlp is not None:
            ft = layer_tensors(t, l, "mlp")
            h = layer_norm(x, t[f"l{l}.norm2"], eps)
            x = x + layer_norm(feed_forward(h, ft["up"], ft["down"]), t[f"l{l}.norm2b"], eps)
        streams.append(x)
    logits = layer_norm(x, t["final.norm"], eps) @ t["head"].T
    return softcap(logits, config["logit_softcap"]), np.stack(streams)
