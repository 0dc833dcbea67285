"""Lomelorn without a GPU: the oracle's mechanisms against values worked out by hand, the file reader,
the configuration reader, the registry and the trace replay."""
import io
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import ctox_llm_b200 as ctox
from ctox_llm_b200 import _native as N
from ctox_llm_b200 import models, trace
from ctox_llm_b200.models import lomelorn
from ctox_llm_b200.safetensors import SafetensorsFile
import lomelorn_oracle as oracle
from lomelorn_util import layer, model, write_model

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


# ---- the oracle, one mechanism at a time
def test_layer_norm_takes_the_mean_off_and_puts_eps_inside_the_root():
    x = np.array([[1.0, 3.0]])  # mean 2, variance 1
    assert np.allclose(oracle.layer_norm(x, np.array([2.0, 4.0]), 3.0), [[-1.0, 2.0]])


def test_rms_norm_keeps_the_mean():
    assert np.allclose(oracle.rms_norm(np.array([[3.0, 4.0]]), np.array([1.0, 2.0]), 3.5), [[0.75, 2.0]])


def test_rotation_turns_neighbouring_pairs():
    x = np.array([[1.0, 0.0, 0.0, 2.0]])
    out = oracle.rotate_pairs(x, np.array([np.pi / 2]), 16.0)  # pair 1 turns a quarter as fast
    c, s = np.cos(np.pi / 8), np.sin(np.pi / 8)
    assert np.allclose(out, [[0.0, 1.0, -2.0 * s, 2.0 * c]])
    assert np.allclose(oracle.rotate_pairs(x, np.array([0.0]), 16.0), x)


def test_window_counts_the_token_itself():
    see = oracle.visible(5, 2)
    assert see.sum() == 9 and see[4, 4] and see[4, 3] and not see[4, 2] and not see[3, 4]
    assert np.array_equal(oracle.visible(5, 1), np.eye(5, dtype=bool))


def test_feed_forward_squares_the_positive_part():
    up, down = np.array([[1.0], [-1.0]]), np.array([[1.0, 10.0]])
    assert np.allclose(oracle.feed_forward(np.array([[3.0], [-2.0]]), up, down), [[9.0], [40.0]])


def test_softcap_bounds_and_keeps_small_values():
    assert np.allclose(oracle.softcap(np.array([1e-4, 1e9, -1e9]), 5.0), [1e-4, 5.0, -5.0])


def test_uniform_attention_averages_the_values_of_the_window():
    config, t = model([layer(heads=1, window=3, ff=None)], seed=3)
    t["l0.mix.uq"] = t["l0.mix.uq"] * 0  # every score 0
    m = config["layers"][0]["mixer"]
    h = np.random.default_rng(0).standard_normal((6, 72))
    mt = oracle.layer_tensors({k: np.asarray(v, np.float64) for k, v in t.items()}, 0, "mix")
    c, k_rot = oracle.latent_keys(h, mt, m, 1e-3)
    out = oracle.latent_attention(h, mt, m, 1e-3, c, k_rot)
    assert np.allclose(out[5], c[3:6].mean(0) @ mt["uv"].T @ mt["o"].T)


def test_shared_cache_layer_reads_the_named_layer():
    config, t = model([layer(), layer(kv_from=0), layer(kv_from=0, window=4)], seed=4)
    assert "l1.mix.dkv" not in t
    base, _ = oracle.forward(config, t, range(20))
    t["l0.mix.dkv"] = t["l0.mix.dkv"] * 1.5
    t["l0.mix.o"] = t["l0.mix.o"] * 0  # layer 0 adds nothing any more: a change can only come through the cache
    a, _ = oracle.forward(config, t, range(20))
    t["l0.mix.dkv"] = np.roll(t["l0.mix.dkv"], 1, axis=0)
    b, _ = oracle.forward(config, t, range(20))
    assert not np.allclose(a, base) and not np.allclose(a, b)


# ---- files, configuration, registry
def test_safetensors_round_trip_and_refusals(tmp_path):
    config, t = model([layer()])
    folder = write_model(str(tmp_path / "m"), config, t)
    f = SafetensorsFile(os.path.join(folder, "model.safetensors"))
    assert set(f.tensors) == set(t)
    data, rows, cols = f.bf16_matrix("l0.mix.uq")
    assert (rows, cols) == t["l0.mix.uq"].shape and data.nbytes == rows * cols * 2
    for name in ("embed", "final.norm"):
        assert np.array_equal(f.float_vector(name), t[name].reshape(-1))
    with pytest.raises(ctox.CtoxError):
        f.bf16_matrix("final.norm")
    with pytest.raises(ctox.CtoxError):
        f.raw("missing")
    broken = tmp_path / "broken.safetensors"
    blob = json.dumps({"a": {"dtype": "BF16", "shape": [4], "data_offsets": [0, 6]}}).encode()
    broken.write_bytes(len(blob).to_bytes(8, "little") + blob + b"\0" * 8)
    with pytest.raises(ctox.CtoxError):
        SafetensorsFile(str(broken))
    broken.write_bytes(b"\xff" * 16)
    with pytest.raises(ctox.CtoxError):
        SafetensorsFile(str(broken))


def test_every_size_comes_from_the_configuration():
    config, _ = model([layer(heads=5, dim=12, rot_dim=6, vdim=7, q_rank=9, kv_rank=10, window=13, base=77.5, scale=0.3),
                       layer(ff=None, kv_from=0, kv_rank=10, rot_dim=6, base=77.5)], vocab=11, width=18, eps=0.25, softcap=3.0)
    c = lomelorn.stack_config(config, "float32", 100)
    assert (c.vocab_size, c.hidden_size, c.norm_eps, c.logit_softcap, c.kv_dtype) == (11, 18, 0.25, 3.0, N.F32)
    a, b = c.layers
    assert (a.heads, a.dim, a.rot_dim, a.vdim, a.q_rank, a.kv_rank, a.window) == (5, 12, 6, 7, 9, 10, 13)
    assert a.rope_base == 77.5 and abs(a.score_scale - 0.3) < 1e-7 and a.kv_from == -1 and (a.mlp, a.ff) == (N.MLP_RELU2, 100)
    assert b.kv_from == 0 and (b.mlp, b.ff) == (N.MLP_NONE, 0)
    assert lomelorn.stack_config(config, "bfloat16", 100).kv_dtype == N.BF16


@pytest.mark.parametrize("change", [
    lambda l: l.update(type="recurrent"), lambda l: l["mlp"].update(kind="experts"),
    lambda l: l["mixer"]["rot"].update(dims=4), lambda l: l["mixer"]["mask"].update(size=0)])
def test_unknown_parts_are_refused(change):
    spec = layer()
    change(spec)
    with pytest.raises(ctox.CtoxError):
        lomelorn.layer_config(0, spec)


def test_registry_knows_the_architectures(tmp_path):
    assert models.architectures() == ["Lomelorn", "Qwen38", "Vasanex"]
    (tmp_path / "config.json").write_text(json.dumps({"architecture": "Other"}))
    with pytest.raises(ctox.CtoxError) as e:
        models.read_config(str(tmp_path))
    assert e.value.kind == "UnsupportedOperation"
    with pytest.raises(ctox.CtoxError):
        models.open_model(str(tmp_path), dtype="float16")


def test_struct_layouts_match_the_header(tmp_path):
    structs = {"ctox_layer_config": N.LayerConfig, "ctox_stack_config": N.StackConfigC}
    src = ['#include <stdio.h>', '#include <stddef.h>', '#include "ctox_b200.h"', 'int main(void){']
    want = []
    for name, s in structs.items():
        src.append(f'printf("%zu\\n", sizeof({name}));')
        want.append(__import__("ctypes").sizeof(s))
        for f in s._fields_:
            src.append(f'printf("%zu\\n", offsetof({name}, {f[0]}));')
            want.append(getattr(s, f[0]).offset)
    src.append(f'printf("%d\\n", (int)CTOX_T_MLP_GATE); return 0;}}')
    want.append(N.T_MLP_GATE)
    c, exe = tmp_path / "l.c", tmp_path / "l"
    c.write_text("\n".join(src))
    subprocess.check_call(["gcc", "-I", os.path.join(ROOT, "include"), str(c), "-o", str(exe)])
    assert [int(x) for x in subprocess.check_output([str(exe)]).split()] == want


# ---- trace replay and generation over a stand-in for the executor
class FakeExecutor:
    def __init__(self):
        self.calls = []

    def reset_session(self):
        self.calls.append("reset")

    def extend(self, tokens, want):
        self.calls.append(list(tokens))
        return np.array([[float(tokens[w]), -1.0] for w in want], dtype=np.float32).reshape(len(want), 2)

    def unload(self):
        self.calls.append("unload")


def test_trace_replay_writes_wanted_rows_and_resets_between_requests(tmp_path, monkeypatch):
    ex = FakeExecutor()
    monkeypatch.setattr(models, "open_model", lambda *a, **k: ex)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": [5, 6, 7], "want": [0, 2]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": [8], "want": []}], "end": ["a"]},
             {"step": 2, "entries": [{"id": "b", "tokens": [9], "want": [0]}], "end": ["b"]}]
    done = []
    trace.run("m", "bfloat16", str(tmp_path), 16, io.StringIO("\n".join(json.dumps(s) for s in steps)), done.append)
    assert done == [0, 1, 2]
    assert ex.calls == ["reset", [5, 6, 7], [8], "reset", [9], "unload"]
    assert np.array_equal(np.fromfile(tmp_path / "0.f32", "<f4"), [5, -1, 7, -1])
    assert not (tmp_path / "1.f32").exists() and np.array_equal(np.fromfile(tmp_path / "2.f32", "<f4"), [9, -1])
    steps = [dict(steps[0]), {"step": 1, "entries": [{"id": "b", "tokens": [8], "want": []}], "end": []}]
    with pytest.raises(RuntimeError):
        trace.run("m", "bfloat16", str(tmp_path), 16, io.StringIO("\n".join(json.dumps(s) for s in steps)), done.append)


def test_command_line_lists_the_models():
    out = subprocess.run([sys.executable, "-m", "ctox_llm_b200", "models"], cwd=ROOT, capture_output=True, text=True)
    assert out.returncode == 0 and out.stdout.split() == ["Lomelorn", "Qwen38", "Vasanex"]
