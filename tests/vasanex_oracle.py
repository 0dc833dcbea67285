"""Plain float64 implementation of the Vasanex design, one function per mechanism.

Slow and direct: every token looks at every key it may see, the recurrence runs token by token, nothing
is cached or fused. It shares no code with the package; the product's results are compared against it.
`tokens` of a sequence always start at position 0.
"""
import numpy as np


def rms(x, eps):
    """x over its root mean square (last axis)."""
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps)


def rms_norm(x, w, eps):
    return rms(x, eps) * w


def rms_norm_around_zero(x, w, eps):
    """The stored weight is the deviation from one."""
    return rms(x, eps) * (1.0 + w)


def sigmoid(z):
    return np.exp(-np.logaddexp(0.0, -z))


def logsigmoid(z):
    return -np.logaddexp(0.0, -z)


def rotate_halves(x, positions, dims, base):
    """x [tokens, heads, width]: dimension i of the first `dims` forms a pair with i + dims / 2, turned by
    position * base^(-2i / dims); the others pass."""
    out = np.array(x)
    for i in range(dims // 2):
        j = i + dims // 2
        angle = (positions * base ** (-2.0 * i / dims))[:, None]
        u, v = x[..., i], x[..., j]
        out[..., i] = u * np.cos(angle) - v * np.sin(angle)
        out[..., j] = v * np.cos(angle) + u * np.sin(angle)
    return out


def visible(n, window):
    """[n, n]: query i sees key j."""
    i, j = np.arange(n)[:, None], np.arange(n)[None, :]
    return (j <= i) & (i - j < window)


def sink_softmax(score, sink):
    """Softmax over the last axis with one more term exp(sink) in the denominator."""
    top = np.maximum(score.max(-1, keepdims=True), sink)
    p = np.exp(score - top)
    return p / (p.sum(-1, keepdims=True) + np.exp(sink - top))


def mix_values(v, first, amount):
    return (1.0 - amount) * v + amount * first


def queries_keys_values(h, t, m, eps):
    """Biased projections; queries and keys normed over the whole projection, then rotated."""
    n = len(h)
    positions = np.arange(n)
    q = rms_norm(h @ t["q"].T + t["q.b"], t["q.norm"], eps).reshape(n, m["heads"], m["dim"])
    k = rms_norm(h @ t["k"].T + t["k.b"], t["k.norm"], eps).reshape(n, m["kv_heads"], m["dim"])
    dims, base = m["rot"]["dims"], m["rot"]["base"]
    return rotate_halves(q, positions, dims, base), rotate_halves(k, positions, dims, base), h @ t["v"].T + t["v.b"]


def grouped_attention(q, k, v, m, sink):
    """q [n, H, dim], k [n, G, dim], v [n, G * vdim] -> [n, H * vdim]."""
    n, share = len(q), m["heads"] // m["kv_heads"]
    see = visible(n, m["mask"]["size"])
    v = v.reshape(n, m["kv_heads"], m["vdim"])
    heads = []
    for head in range(m["heads"]):
        score = np.where(see, q[:, head] @ k[:, head // share].T * m["scale"], -np.inf)
        heads.append(sink_softmax(score, sink[head]) @ v[:, head // share])
    return np.concatenate(heads, -1)


def attention(h, t, m, eps, first_values):
    """(mixer output, the layer's values before mixing). first_values: None where nothing is mixed in."""
    q, k, own = queries_keys_values(h, t, m, eps)
    v = own if first_values is None else mix_values(own, first_values, t["vmix"])
    return grouped_attention(q, k, v, m, t["sink"]) @ t["o"].T + t["o.b"], own


def soft_cap(z, cap):
    return cap * np.tanh(z / cap)


def log_gates(h, t, m):
    """Log input and log forget gate, [n, heads] each."""
    cap = m["gate_cap"]
    return soft_cap(h @ t["i"].T + t["i.b"], cap), logsigmoid(soft_cap(h @ t["f"].T + t["f.b"], cap))


def matrix_memory(q, k, v, i, f):
    """One head: q, k [n, dim], v [n, vdim], log gates [n] -> [n, vdim]."""
    S, n, m = np.zeros((q.shape[1], v.shape[1])), np.zeros(q.shape[1]), 0.0
    out = []
    for t in range(len(q)):
        top = max(f[t] + m, i[t])
        keep, take = np.exp(f[t] + m - top), np.exp(i[t] - top)
        S = keep * S + take * np.outer(k[t], v[t])
        n = keep * n + take * k[t]
        m = top
        out.append(S.T @ q[t] / (max(abs(n @ q[t]), np.exp(-m)) + 1e-6))
    return np.array(out)


def mlstm(h, t, m, eps):
    n, H, dim, vdim = len(h), m["heads"], m["dim"], m["vdim"]
    q = (h @ t["q"].T * dim ** -0.5).reshape(n, H, dim)
    k = (h @ t["k"].T).reshape(n, H, dim)
    v = (h @ t["v"].T).reshape(n, H, vdim)
    i, f = log_gates(h, t, m)
    o = [rms(matrix_memory(q[:, a], k[:, a], v[:, a], i[:, a], f[:, a]), eps) for a in range(H)]
    return (np.concatenate(o, -1) * t["norm"] * sigmoid(h @ t["g"].T)) @ t["o"].T


def feed_forward(h, gate, up, down, limit):
    g = np.minimum(h @ gate.T, limit)
    u = np.clip(h @ up.T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ down.T


def layer_tensors(tensors, l, part):
    prefix = f"l{l}.{part}."
    return {k[len(prefix):]: v for k, v in tensors.items() if k.startswith(prefix)}


def forward(config, tensors, tokens):
    """(logits [tokens, vocab], residual stream after every layer [layers, tokens, width])."""
    t = {k: np.asarray(v, np.float64) for k, v in tensors.items()}
    eps = config["norm"]["eps"]
    x = t["embed"][np.asarray(tokens)] * config["embedding"]["scale"]
    first, streams = None, []
    for l, layer in enumerate(config["layers"]):
        m, mlp = layer["mixer"], layer["mlp"]
        mt = layer_tensors(t, l, "mix")
        h = rms_norm_around_zero(x, t[f"l{l}.norm1"], eps)
        if layer["type"] == "mlstm":
            y = mlstm(h, mt, m, eps)
        else:
            y, own = attention(h, mt, m, eps, first if m["v_mix"] else None)
            if m["v_mix"] and first is None:
                first = own
        x = x + y
        if mlp is not None:
            ft = layer_tensors(t, l, "mlp")
            x = x + feed_forward(rms_norm_around_zero(x, t[f"l{l}.norm2"], eps), ft["gate"], ft["up"], ft["down"], mlp["limit"])
        streams.append(x)
    return rms_norm_around_zero(x, t["final.norm"], eps) @ t["embed"].T, np.stack(streams)
