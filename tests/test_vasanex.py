"""Vasanex without a GPU: the oracle's mechanisms against values worked out by hand, the configuration reader."""
import numpy as np
import pytest

import ctox_llm_b200 as ctox
from ctox_llm_b200 import _native as N
from ctox_llm_b200.models import vasanex
from ctox_llm_b200.safetensors import SafetensorsFile
import vasanex_oracle as oracle
from vasanex_util import attention, mlstm, model, write_model


# ---- the oracle, one mechanism at a time
def test_norm_weight_is_a_deviation_from_one():
    x = np.array([[3.0, 4.0]])  # mean square 12.5
    assert np.allclose(oracle.rms_norm_around_zero(x, np.array([0.0, -0.5]), 3.5), [[0.75, 0.5]])
    assert np.allclose(oracle.rms_norm(x, np.array([1.0, 2.0]), 3.5), [[0.75, 2.0]])


def test_rotation_pairs_the_halves_and_passes_the_rest():
    x = np.array([[[1.0, 0.0, 0.0, 2.0, 7.0]]])
    out = oracle.rotate_halves(x, np.array([np.pi / 2]), 4, 16.0)  # the second pair turns a quarter as fast
    c, s = np.cos(np.pi / 8), np.sin(np.pi / 8)
    assert np.allclose(out, [[[0.0, -2.0 * s, 1.0, 2.0 * c, 7.0]]])


def test_window_counts_the_token_itself():
    see = oracle.visible(5, 2)
    assert see.sum() == 9 and see[4, 4] and see[4, 3] and not see[4, 2] and not see[3, 4]


def test_sink_takes_weight_and_gives_nothing():
    assert np.allclose(oracle.sink_softmax(np.array([[0.0, -np.inf, 0.0]]), 0.0), [[1 / 3, 0, 1 / 3]])
    assert np.allclose(oracle.sink_softmax(np.array([[-800.0, -801.0]]), 0.0), 0.0)
    assert np.allclose(oracle.sink_softmax(np.array([[900.0]]), -5.0), 1.0)


def test_heads_share_keys_and_scale_leaves_the_sink_alone():
    m = attention(heads=4, kv_heads=2, dim=2, vdim=1, window=9, scale=0.5)["mixer"]
    q = np.ones((1, 4, 2))
    k = np.array([[[1.0, 1.0], [-1.0, -1.0]]])  # scores 1 and -1
    out = oracle.grouped_attention(q, k, np.array([[10.0, 20.0]]), m, np.array([0.0, 1.0, 0.0, -1.0]))
    e = np.e
    assert np.allclose(out, [[10 * e / (e + 1), 5.0, 20 / (1 + e), 10.0]])


def test_mixed_values():
    assert np.allclose(oracle.mix_values(np.array([4.0]), np.array([8.0]), 0.25), [5.0])


def test_first_layer_that_mixes_gives_its_values():
    layers = [attention(v_mix=False), attention(), mlstm(), attention()]
    config, t = model(layers, seed=1)
    base, _ = oracle.forward(config, t, range(12))
    for l, change in ((0, False), (1, False), (3, True)):
        u = {**t, f"l{l}.mix.vmix": np.float32(0.9)}
        assert (not np.allclose(oracle.forward(config, u, range(12))[0], base)) == change


def test_memory_of_one_token():
    """S = e^(i - m) k v^T: the output is v where |k . q| e^i is above one, and fades below."""
    q, k, v = np.array([[2.0]]), np.array([[3.0]]), np.array([[5.0, -1.0]])
    out = oracle.matrix_memory(q, k, v, np.array([0.0]), np.array([-1.0]))
    assert np.allclose(out, 6.0 * v / (6.0 + 1e-6))
    out = oracle.matrix_memory(q, k, v, np.array([-4.0]), np.array([-1.0]))  # the running maximum falls to -1
    take = np.exp(-3.0)
    assert np.allclose(out, take * 6.0 * v / (max(take * 6.0, np.e) + 1e-6))


def test_memory_forgets_and_adds():
    q, k = np.ones((2, 1)), np.ones((2, 1))
    v = np.array([[1.0], [0.0]])
    out = oracle.matrix_memory(q, k, v, np.array([0.0, 0.0]), np.array([-1.0, -1.0]))
    keep = np.exp(-1.0)
    assert np.allclose(out[1], keep / (keep + 1.0 + 1e-6))


def test_log_gates_are_capped():
    m = mlstm(heads=1, gate_cap=2.0)["mixer"]
    t = {"i": np.array([[1.0]]), "f": np.array([[1.0]]), "i.b": np.array([0.0]), "f.b": np.array([0.0])}
    i, f = oracle.log_gates(np.array([[1e3], [0.0]]), t, m)
    assert np.allclose(i[:, 0], [2.0, 0.0]) and np.allclose(f[:, 0], [-np.log1p(np.exp(-2.0)), -np.log(2.0)])


def test_feed_forward_clamps_both_parts():
    one = np.array([[1.0]])
    f = lambda g, u: oracle.feed_forward(np.array([[1.0]]), g * one, u * one, one, 2.0)[0, 0]
    s = lambda z: 1 / (1 + np.exp(-z))
    assert np.isclose(f(5.0, 9.0), 2 * s(3.404) * 3) and np.isclose(f(-5.0, -9.0), -5 * s(-8.51) * -1)


# ---- configuration, weights
def test_every_size_comes_from_the_configuration():
    config, _ = model([attention(heads=10, kv_heads=5, dim=14, vdim=7, window=13, base=77.5, rot=6, scale=0.3, ff=33, limit=2.5),
                       mlstm(heads=2, dim=9, vdim=11, gate_cap=3.5),
                       attention(v_mix=False, ff=None), mlstm(ff=15, limit=0.5)], vocab=11, width=18, eps=0.25, embed_scale=0.75)
    c = vasanex.stack_config(config, "float32", 100)
    assert (c.vocab_size, c.hidden_size, c.norm_eps, c.embed_scale, c.kv_dtype) == (11, 18, 0.25, 0.75, N.F32)
    assert (c.norm, c.out_norms, c.tied_head, c.logit_softcap) == (N.NORM_RMS, False, True, 0.0)
    a, b, x, y = c.layers
    assert (a.mixer, a.heads, a.kv_heads, a.dim, a.vdim, a.rot_dim, a.window) == (N.MIXER_GROUPED_ATTENTION, 10, 5, 14, 7, 6, 13)
    assert a.rope_base == 77.5 and abs(a.score_scale - 0.3) < 1e-7
    assert (a.mlp, a.ff, a.mlp_limit) == (N.MLP_CLAMPED_GLU, 33, 2.5) and abs(a.mlp_slope - 1.702) < 1e-6
    every = N.ATTN_BIAS | N.ATTN_QK_NORM | N.ATTN_SINK
    assert (a.attn, x.attn) == (every | N.ATTN_V_MIX, every) and (x.mlp, x.ff) == (N.MLP_NONE, 0)
    assert (b.mixer, b.heads, b.dim, b.vdim, b.gate_cap, b.mlp) == (N.MIXER_MATRIX_MEMORY, 2, 9, 11, 3.5, N.MLP_NONE)
    assert (y.mlp, y.ff, y.mlp_limit) == (N.MLP_CLAMPED_GLU, 15, 0.5)
    assert vasanex.stack_config(config, "bfloat16", 100).kv_dtype == N.BF16


@pytest.mark.parametrize("change", [lambda l: l.update(type="latent_attention"), lambda l: l["mlp"].update(kind="experts"),
                                    lambda l: l["mixer"]["mask"].update(size=0)])
def test_unknown_parts_are_refused(change):
    spec = attention()
    change(spec)
    with pytest.raises(ctox.CtoxError):
        vasanex.layer_config(0, spec)


class Recorder:
    """Stands in for the executor: what was loaded, by layer and tensor."""

    def __init__(self, config):
        self.config, self.got = config, {}

    def load_matrix(self, layer, tensor, op):
        self.got[layer, tensor] = np.asarray(op.weights).view("<u2").reshape(op.rows, op.columns)

    def load_vector(self, layer, tensor, values):
        self.got[layer, tensor] = values


def test_weights_go_where_they_belong(tmp_path):
    config, t = model([attention(), mlstm(ff=30), attention()], seed=2)
    del t["l0.mix.vmix"]  # unused in the first layer that mixes
    folder = write_model(str(tmp_path / "m"), config, t)
    ex = Recorder(vasanex.stack_config(config, "bfloat16", 64))
    vasanex.load_weights(SafetensorsFile(folder + "/model.safetensors"), ex)
    assert len(ex.got) == len(t)
    assert np.array_equal(ex.got[1, N.T_POST_NORM], np.float32(1) + t["l1.norm2"])
    assert np.array_equal(ex.got[2, N.T_Q_NORM], t["l2.mix.q.norm"]) and ex.got[2, N.T_V_MIX] == t["l2.mix.vmix"]
    assert ex.got[1, N.T_MEM_FORGET].shape == (3, 76) and (0, N.T_V_MIX) not in ex.got
