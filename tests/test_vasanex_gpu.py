"""Vasanex on the GPU against the plain implementation (vasanex_oracle.py), through the registry, the executor's
own calls and the command line."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import ctox_llm_b200 as ctox
from ctox_llm_b200 import _native as N
import vasanex_oracle as oracle
from vasanex_util import attention, bf16, mlstm, model, row_errors, write_model

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
# row_errors of the worst row and of the mean row
TOL = {"float32": 3e-5, "bfloat16": 6e-2}
MEAN = {"float32": 5e-6, "bfloat16": 1e-2}
PLANTED = 0.2  # least effect of a planted mistake that a test relies on
DTYPES = ["float32", "bfloat16"]


def close(got, want, dtype):
    e = row_errors(got, want)
    return e.max() < TOL[dtype] and e.mean() < MEAN[dtype]


@pytest.fixture(scope="module")
def be():
    b = ctox.B200Backend(0)
    yield b
    assert b.allocated_bytes() == 0
    b.close()


@pytest.fixture
def opened(be, tmp_path):
    """opened(config, tensors, dtype, **options) -> executor, unloaded afterwards."""
    live = []

    def make(config, tensors, dtype, context=1024, **options):
        folder = write_model(str(tmp_path / f"m{len(live)}"), config, tensors)
        ex = ctox.open_model(folder, backend=be, dtype=dtype, max_context_tokens=context, **options)
        live.append(ex)
        return ex

    yield make
    for ex in live:
        ex.unload()


def run(ex, tokens, cuts=()):
    """Logits of every token with the sequence cut at the given places."""
    ex.reset_session()
    edges = [0] + list(cuts) + [len(tokens)]
    return np.concatenate([ex.extend(tokens[a:b], range(b - a)) for a, b in zip(edges, edges[1:])])


def tokens_of(n, vocab, seed=0):
    return [int(t) for t in np.random.default_rng(seed).integers(0, vocab, n)]


# Sizes that are nobody's: odd widths, head sizes that are no multiple of 16, layers that differ in everything, layers
# with and without feed-forward and mixed values in any place, more value than key dimensions and the reverse.
MODELS = {
    "mixed": lambda: model([mlstm(ff=50), attention(v_mix=False, ff=None, heads=4, kv_heads=4, dim=10, vdim=6, window=5, rot=10),
                            attention(window=29), mlstm(heads=1, dim=33, vdim=7, gate_cap=1.5, ff=31, limit=0.4),
                            attention(heads=5, kv_heads=1, dim=48, vdim=80, window=70, rot=2, base=55.0, scale=0.4, ff=None),
                            attention(heads=8, kv_heads=2, dim=8, vdim=40, window=1, limit=7.0)], seed=1),
    "memories": lambda: model([mlstm(heads=2, dim=64, vdim=128), mlstm(heads=5, dim=16, vdim=16, ff=40), mlstm(heads=1, dim=7, vdim=300),
                               mlstm(heads=3, dim=96, vdim=80)], vocab=131, width=120, seed=2),
    "smallest": lambda: model([attention(heads=1, kv_heads=1, dim=2, vdim=1, rot=2, ff=1), mlstm(heads=1, dim=1, vdim=1, ff=1)],
                              vocab=13, width=5, seed=3),
    "wide": lambda: model([attention(heads=16, kv_heads=4, dim=64, vdim=128, window=150, rot=32, ff=500),
                           mlstm(heads=4, dim=128, vdim=256),
                           attention(heads=12, kv_heads=4, dim=128, vdim=128, window=90, rot=128, base=1e6, scale=0.05, ff=None),
                           mlstm(heads=2, dim=256, vdim=192, ff=300)], vocab=1000, width=384, seed=4),
    "wide_heads": lambda: model([attention(heads=4, kv_heads=2, dim=256, vdim=256, window=130, rot=64), mlstm(heads=2, dim=40, vdim=512)],
                                seed=5),
    "short_passes_only": lambda: model([attention(heads=2, kv_heads=1, dim=320, vdim=272, window=40), mlstm(heads=2, dim=272, vdim=20)],
                                       seed=6),
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(MODELS))
def test_whole_prompt_portions_and_single_tokens(opened, name, dtype):
    config, t = MODELS[name]()
    tokens = tokens_of(300, config["vocab"])
    want, streams = oracle.forward(config, t, tokens)
    ex = opened(config, t, dtype)
    ex.keep_streams()
    whole = run(ex, tokens)
    assert close(whole, want, dtype)
    for l in range(len(config["layers"])):
        assert close(ex.last_stream(l, 0, len(tokens)), streams[l], dtype)
    # portions of 2, 3, ... tokens, around the pass, chunk and page sizes, then one by one
    cuts = np.cumsum([2, 3, 4, 5, 7, 8, 9, 2, 16, 17, 63, 2, 127, 2]).tolist()
    portions = run(ex, tokens, cuts + list(range(cuts[-1] + 4, len(tokens))))
    assert close(portions, want, dtype)
    single = run(ex, tokens[:60], range(1, 60))
    assert close(single, want[:60], dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_passes_of_every_short_length(opened, dtype):
    config, t = MODELS["mixed"]()
    tokens = tokens_of(70, config["vocab"], 5)
    want, _ = oracle.forward(config, t, tokens)
    ex = opened(config, t, dtype)
    for m in range(1, 12):
        assert close(run(ex, tokens, range(m, 70, m)), want, dtype), m


def test_portions_around_the_chunk_length(opened):
    config, t = MODELS["memories"]()
    tokens = tokens_of(520, config["vocab"], 6)
    want, _ = oracle.forward(config, t, tokens)
    ex = opened(config, t, "bfloat16")
    for size in (127, 128, 129, 255, 256, 257):
        assert close(run(ex, tokens, range(size, 520, size)), want, "bfloat16"), size
    ex = opened(config, t, "bfloat16", context=4500, pass_tokens=2200)  # more than 2048 tokens in a pass
    tokens = tokens_of(2300, config["vocab"], 7)
    want, _ = oracle.forward(config, t, tokens)
    assert close(run(ex, tokens), want, "bfloat16")


@pytest.mark.parametrize("size", [1000, 130, 70, 37])
def test_many_prompts_give_the_same_bits(be, size):
    grouped = dict(mixer=N.MIXER_GROUPED_ATTENTION, heads=12, kv_heads=3, dim=64, vdim=128, rot_dim=32, rope_base=1e4, window=200,
                   kv_from=-1, score_scale=0.3, attn=15, mlp=N.MLP_CLAMPED_GLU, ff=512, mlp_limit=3.0, mlp_slope=1.702)
    memory = dict(mixer=N.MIXER_MATRIX_MEMORY, heads=4, dim=128, vdim=192, kv_from=-1, gate_cap=15.0, mlp=N.MLP_NONE)
    ex = ctox.B200Executor(be, ctox.StackConfig(vocab_size=1000, hidden_size=512, norm_eps=1e-6, logit_softcap=0.0,
                                                layers=[N.LayerConfig(**x) for x in (grouped, memory, grouped, memory)],
                                                max_context_tokens=3100, norm=N.NORM_RMS, out_norms=False, tied_head=True))
    ex.fill_synthetic(0)
    ex.warmup()
    tokens, first = tokens_of(3000, 1000, 1), None
    for _ in range(20):
        ex.reset_session()
        for a in range(0, 3000, size):
            ex.extend(tokens[a:a + size])
        for token in tokens[:3]:
            ex.extend([token])
        hidden = ex.last_hidden()
        first = hidden if first is None else first
        assert np.isfinite(hidden).all() and np.array_equal(hidden, first)
    ex.unload()


# ---- mechanisms on their own
def check_all(opened, config, t, n=150, seed=0):
    """Whole, in portions and token by token, in both modes."""
    tokens = tokens_of(n, config["vocab"], seed)
    want, _ = oracle.forward(config, t, tokens)
    for dtype in DTYPES:
        ex = opened(config, t, dtype)
        for cuts in ((), (n // 3, n // 3 + 2, n // 2), range(1, n)):
            assert close(run(ex, tokens, cuts), want, dtype), (dtype, cuts)
    return tokens, want


def test_query_and_key_norms_run_over_the_whole_projection(opened):
    """Heads of very different size: a norm per head would give all the same size."""
    config, t = model([attention(heads=4, kv_heads=2, ff=None, window=40)], seed=11)
    for name, heads in (("q", 4), ("k", 2)):
        size = np.repeat(np.geomspace(0.05, 2.0, heads), 24)
        t[f"l0.mix.{name}"], t[f"l0.mix.{name}.b"] = bf16(t[f"l0.mix.{name}"] * 30 * size[:, None]), bf16(t[f"l0.mix.{name}.b"] * 30 * size)
    check_all(opened, config, t)


def test_rotation_covers_the_first_dimensions_only(opened):
    """Queries and keys are nearly the same for all tokens (biases), so distances decide."""
    config, t = model([attention(heads=3, kv_heads=1, dim=40, rot=24, base=31.0, ff=None, window=60, scale=0.4)], seed=13)
    for name in ("q", "k"):
        t[f"l0.mix.{name}"] = bf16(t[f"l0.mix.{name}"] * 0.1)
        t[f"l0.mix.{name}.b"] = bf16(t[f"l0.mix.{name}.b"] * 10)
    tokens, want = check_all(opened, config, t)
    for change in ({"dims": 24, "base": 62.0}, {"dims": 32, "base": 31.0}):
        spec = attention(heads=3, kv_heads=1, dim=40, ff=None, window=60, scale=0.4)
        spec["mixer"]["rot"] = change
        off, _ = oracle.forward({**config, "layers": [spec]}, t, tokens)
        assert row_errors(off, want)[60:].mean() > 0.05  # another rotation would show


def test_sinks(opened):
    config, t = model([attention(ff=None, window=9, scale=0.02)], seed=14)  # flat scores
    t["l0.mix.sink"] = bf16(np.array([-30.0, 0.0, 2.0, 5.0, 20.0, 90.0]))
    tokens, want = check_all(opened, config, t)
    off, _ = oracle.forward(config, {**t, "l0.mix.sink": t["l0.mix.sink"] * 0 - 1e9}, tokens)
    assert row_errors(off, want).mean() > PLANTED


def test_sinks_above_and_below_large_scores(opened):
    config, t = model([attention(ff=None, window=30, scale=9.0)], seed=15)
    t["l0.mix.sink"] = bf16(np.array([-200.0, -50.0, 0.0, 60.0, 150.0, 300.0]))
    for name in "qk":  # unit-sized so that scores reach hundreds; 16-bit errors would be amplified
        t[f"l0.mix.{name}.norm"] = bf16(t[f"l0.mix.{name}.norm"] * 0 + 1)
    tokens = tokens_of(100, config["vocab"])
    want, _ = oracle.forward(config, t, tokens)
    ex = opened(config, t, "float32")
    for cuts in ((), range(1, 100)):
        assert row_errors(run(ex, tokens, cuts), want).max() < 5e-4
    got = run(opened(config, t, "bfloat16"), tokens)
    assert np.isfinite(got).all()


def test_values_are_mixed_before_they_are_cached(opened):
    config, t = model([attention(ff=None, v_mix=False, window=20), attention(ff=None, window=20), mlstm(),
                       attention(heads=4, kv_heads=1, vdim=80, ff=None, window=20), attention(ff=None, v_mix=False, heads=2, kv_heads=2),
                       attention(window=20)], seed=16)
    for l, amount in ((0, 0.7), (1, -3.0), (3, 0.6), (4, 5.0), (5, 1.25)):
        t[f"l{l}.mix.vmix"] = bf16(np.float32(amount)).reshape(())
    check_all(opened, config, t)


def test_biases(opened):
    config, t = model([attention(ff=None, window=20)], seed=17)
    for name in ("q.b", "k.b", "v.b", "o.b"):
        t[f"l0.mix.{name}"] = bf16(t[f"l0.mix.{name}"] * 8)
    check_all(opened, config, t)


@pytest.mark.parametrize("limit", [0.05, 1.0, 50.0])
def test_feed_forward_limits(opened, limit):
    config, t = model([attention(window=20, limit=limit), mlstm(ff=55, limit=limit)], seed=18)
    for l in (0, 1):
        for name in ("gate", "up"):
            t[f"l{l}.mlp.{name}"] = bf16(t[f"l{l}.mlp.{name}"] * 3)
    check_all(opened, config, t, n=60)


def test_eps_and_embedding_scale(opened):
    for eps, scale in ((0.8, 0.25), (1e-6, 9.0)):
        config, t = model([attention(window=20), mlstm(ff=30)], eps=eps, embed_scale=scale, seed=19)
        check_all(opened, config, t, n=60)


def test_gates_over_their_whole_range(opened):
    """Tokens that keep nothing, tokens that change nothing, tokens that outweigh all before."""
    for cap in (0.7, 15.0):
        config, t = model([mlstm(heads=4, dim=32, vdim=48, gate_cap=cap)], seed=20)
        rng = np.random.default_rng(1)
        t["l0.mix.i"] = bf16(rng.standard_normal((4, 76)) * [[0.1], [0.5], [1.0], [1.0]])
        t["l0.mix.f"] = bf16(rng.standard_normal((4, 76)) * [[0.1], [0.5], [1.0], [1.0]])
        t["l0.mix.f.b"] = bf16(np.array([9.0, 3.0, 0.0, 6.0]))
        check_all(opened, config, t, n=290)


# ---- something far away that stands out
def test_memory_of_a_far_token(opened):
    """One token is written into the memory hundreds of times stronger than any other, and kept."""
    config, t = model([mlstm(heads=2, dim=32, vdim=48, gate_cap=15.0)], seed=21)
    T = {k: np.asarray(v, np.float64) for k, v in t.items()}
    h = oracle.rms_norm_around_zero(T["embed"] * 2.5, T["l0.norm1"], 1e-3)
    key = 7
    t["l0.mix.i"] = bf16(np.stack([h[key] / (h[key] @ h[key]) * 14] * 2))
    t["l0.mix.i.b"], t["l0.mix.f.b"] = bf16(np.full(2, -6.0)), bf16(np.full(2, 13.0))
    t["l0.mix.f"] = t["l0.mix.f"] * 0
    filler = [v for v in range(config["vocab"]) if v != key]
    for dtype in DTYPES:
        ex = opened(config, t, dtype)
        for key_at in (0, 1, 7, 8, 126, 127, 128, 129, 255, 256):
            tokens = [filler[i] for i in np.random.default_rng(key_at).integers(0, len(filler), 620)]
            tokens[key_at] = key
            want, _ = oracle.forward(config, t, tokens)
            without, _ = oracle.forward(config, t, tokens[:key_at] + [filler[0]] + tokens[key_at + 1:])
            assert row_errors(without, want)[key_at:].mean() > PLANTED
            for cuts in ((), (key_at + 1, key_at + 2), (key_at + 1, 600, 601), range(60, 620, 37)):
                # a query nearly orthogonal to the kept key amplifies rounding (the same rows as when the projections
                # are rounded in the plain implementation)
                e = row_errors(run(ex, tokens, cuts), want)
                assert e.max() < 6 * TOL[dtype] and e.mean() < MEAN[dtype], (key_at, cuts)


def standing_out(window, seed=22):
    """A model without rotation effects whose scores depend on the tokens alone, a query token and the key token that
    outweighs every other by far in the first head."""
    spec = attention(heads=2, kv_heads=1, ff=None, window=window, rot=2, base=1.0, scale=1.0)
    config, t = model([spec], seed=seed)
    t["l0.mix.q.norm"] = t["l0.mix.q.norm"].copy()
    t["l0.mix.q.norm"].reshape(2, 24)[:, :2] = 0  # what is rotated counts nothing
    T = {k: np.asarray(v, np.float64) for k, v in t.items()}
    m, mt = spec["mixer"], oracle.layer_tensors(T, 0, "mix")
    h = oracle.rms_norm_around_zero(T["embed"] * 2.5, T["l0.norm1"], 1e-3)
    q, k, _ = oracle.queries_keys_values(h, mt, m, 1e-3)
    score = q[:, 0] @ k[:, 0].T
    ranked = np.sort(score, -1)
    query = int(np.argmax(ranked[:, -1] - ranked[:, -2]))
    key = int(np.argmax(score[query]))
    m["scale"] = float(np.float32(12.0 / (ranked[query, -1] - ranked[query, -2])))
    t["l0.mix.sink"] = bf16(np.array([score[query, key] * m["scale"] - 12.0, 0.0]))
    t["l0.mix.o"] = bf16(t["l0.mix.o"] * 3)
    filler = [v for v in range(config["vocab"]) if v not in (query, key)]
    return config, t, query, key, filler


def place(n, query_at, key_at, query, key, filler, seed):
    tokens = [filler[i] for i in np.random.default_rng(seed).integers(0, len(filler), n)]
    tokens[query_at], tokens[key_at] = query, key
    return tokens


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window", [2, 33, 64, 127, 128, 129, 200])
def test_keys_at_the_edge_of_the_window(opened, window, dtype):
    config, t, query, key, filler = standing_out(window)
    ex = opened(config, t, dtype)
    for query_at in (window + 3, 255, 256, 383, 400):
        for distance in (window - 1, window):  # the last one seen, the first one not seen
            if query_at < distance:
                continue
            tokens = place(query_at + 2, query_at, query_at - distance, query, key, filler, seed=query_at)
            want, _ = oracle.forward(config, t, tokens)
            config["layers"][0]["mixer"]["mask"]["size"] = window + (1 if distance == window else -1)
            wrong, _ = oracle.forward(config, t, tokens)
            config["layers"][0]["mixer"]["mask"]["size"] = window
            assert row_errors(wrong, want)[query_at] > PLANTED  # a window one token off would show
            for cuts in ((), (query_at - 1,), (query_at, query_at + 1), (max(1, query_at - 70),)):
                got = run(ex, tokens, cuts)
                assert row_errors(got, want)[query_at] < TOL[dtype] * 2, (query_at, distance, cuts)


@pytest.mark.parametrize("dtype", DTYPES)
def test_far_keys_at_page_and_tile_borders(opened, dtype):
    config, t, query, key, filler = standing_out(700)
    ex = opened(config, t, dtype)
    for key_at in (0, 1, 63, 64, 127, 128, 129, 255, 256):
        tokens = place(620, 600, key_at, query, key, filler, seed=key_at)
        want, _ = oracle.forward(config, t, tokens)
        without, _ = oracle.forward(config, t, tokens[:key_at] + [filler[0]] + tokens[key_at + 1:])
        assert row_errors(without, want)[600] > PLANTED
        for cuts in ((), (600, 601), (key_at + 1, 598)):
            assert row_errors(run(ex, tokens, cuts), want)[600] < TOL[dtype] * 2, (key_at, cuts)


@pytest.mark.parametrize("dtype", DTYPES)
def test_first_tokens(opened, dtype):
    config, t = MODELS["wide"]()
    ex = opened(config, t, dtype)
    for n in (1, 2, 3, 8, 9, 10, 17):
        tokens = tokens_of(n, config["vocab"], n)
        want, _ = oracle.forward(config, t, tokens)
        assert close(run(ex, tokens), want, dtype)
        assert close(run(ex, tokens, range(1, n)), want, dtype)


# ---- cache pages, states and sessions
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("pages,pass_tokens", [(128, 64), (128, 130), (16, 0), (24, 0)])
def test_pages_are_used_again_when_the_window_has_passed(opened, dtype, pages, pass_tokens):
    config, t = model([attention(window=40), mlstm(), attention(window=9), attention(window=61)], seed=30)
    ex = opened(config, t, dtype, context=1500, page_tokens=pages, pass_tokens=pass_tokens)
    session = ex.allocations()["session_bytes"]
    tokens = tokens_of(900, config["vocab"], 1)
    want, _ = oracle.forward(config, t, tokens)
    assert close(run(ex, tokens), want, dtype)
    assert close(run(ex, tokens, list(range(37, 600, 37)) + list(range(700, 900))), want, dtype)
    assert ex.allocations()["session_bytes"] == session


@pytest.mark.parametrize("dtype", DTYPES)
def test_requests_one_after_the_other_do_not_see_each_other(opened, dtype):
    config, t = MODELS["mixed"]()
    ex = opened(config, t, dtype, context=400, pass_tokens=64)
    requests = [tokens_of(n, config["vocab"], n) for n in (300, 1, 33, 7, 129, 2)]
    alone = []
    for r in requests:
        fresh = opened(config, t, dtype, context=400, pass_tokens=64)
        alone.append(run(fresh, r, (len(r) // 2,) if len(r) > 1 else ()))
    for k in (0, 1, 2, 3, 4, 5, 0, 3):
        r = requests[k]
        assert np.array_equal(run(ex, r, (len(r) // 2,) if len(r) > 1 else ()), alone[k])


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding(opened, dtype):
    config, t = MODELS["mixed"]()
    tokens = tokens_of(560, config["vocab"], 9)
    want, _ = oracle.forward(config, t, tokens)
    got = run(opened(config, t, dtype), tokens, [50] + list(range(51, 560)))
    assert close(got, want, dtype)


# ---- generation
def oracle_greedy(config, t, prompt, n):
    seq = list(prompt)
    for _ in range(n):
        logits, _ = oracle.forward(config, t, seq)
        seq.append(int(np.argmax(logits[-1])))
    return seq[len(prompt):]


def test_greedy_generation_is_the_oracles(opened):
    config, t = MODELS["mixed"]()
    for prompt in ([4], tokens_of(37, config["vocab"], 3)):
        want = oracle_greedy(config, t, prompt, 24)
        assert list(opened(config, t, "float32").generate(prompt, 24)) == want
        # in 16 bits every token must be the best one up to rounding, given the tokens before it
        got = list(opened(config, t, "bfloat16").generate(prompt, 24))
        logits, _ = oracle.forward(config, t, list(prompt) + got)
        for i, token in enumerate(got):
            row = logits[len(prompt) - 1 + i]
            assert row[token] > row.max() - 2 * TOL["bfloat16"] * np.sqrt((logits ** 2).mean())


def test_sampling_and_selection(opened):
    config, t = MODELS["mixed"]()
    prompt = tokens_of(12, config["vocab"], 8)
    ex = opened(config, t, "float32")
    greedy = list(ex.generate(prompt, 10))
    assert list(ex.generate(prompt, 10, temperature=0.7, top_k=1)) == greedy
    a = list(ex.generate(prompt, 16, temperature=9.0, seed=5))
    assert a == list(ex.generate(prompt, 16, temperature=9.0, seed=5)) and a != list(ex.generate(prompt, 16, temperature=9.0, seed=6))


def test_decode_reports_logits_and_hidden_state(opened):
    config, t = MODELS["mixed"]()
    prompt = tokens_of(20, config["vocab"], 2)
    ex = opened(config, t, "float32")
    ex.keep_logits(True)
    ex.prefill(prompt)
    blk = ex.decode(prompt[-1], mtp_enabled=False)
    logits, streams = oracle.forward(config, t, prompt)
    assert close(ex.last_logits(0)[None], logits[-1:], "float32") and blk.token_id == int(np.argmax(logits[-1]))
    final = oracle.rms_norm_around_zero(streams[-1][-1], np.asarray(t["final.norm"], np.float64), config["norm"]["eps"])
    assert np.abs(ex.last_hidden() - final).max() < 1e-3 and ex.position() == 20


def test_command_line_generates(tmp_path):
    config, t = MODELS["mixed"]()
    folder = write_model(str(tmp_path / "m"), config, t)
    out = subprocess.run([sys.executable, "-m", "ctox_llm_b200", "generate", "--model", folder, "--tokens", "3,1,4", "--max-new", "6",
                          "--dtype", "float32"], cwd=ROOT, capture_output=True, text=True)
    assert out.returncode == 0, out.stderr[-2000:]
    assert [int(x) for x in out.stdout.split()] == oracle_greedy(config, t, [3, 1, 4], 6)


def test_trace_runner_process(tmp_path):
    config, t = MODELS["mixed"]()
    folder = write_model(str(tmp_path / "m"), config, t)
    tokens = tokens_of(45, config["vocab"], 6)
    want, _ = oracle.forward(config, t, tokens)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": tokens[:40], "want": list(range(40))}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": tokens[40:], "want": [0, 4]}], "end": ["a"]},
             {"step": 2, "entries": [{"id": "b", "tokens": tokens[:1], "want": [0]}], "end": ["b"]}]
    for dtype in DTYPES:
        out = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", dtype, "--out", str(tmp_path),
                              "--max-tokens", "45"], input="\n".join(json.dumps(s) for s in steps), capture_output=True, text=True)
        assert out.returncode == 0, out.stderr[-2000:]
        assert out.stdout.split("\n")[:3] == ["done 0", "done 1", "done 2"]
        rows = [np.fromfile(tmp_path / f"{i}.f32", "<f4").reshape(-1, config["vocab"]) for i in range(3)]
        assert close(np.concatenate(rows), want[list(range(40)) + [40, 44, 0]], dtype)


def test_dependent_launch_overlap_changes_no_bit(tmp_path):
    """The same calls with every launch serialised (CTOX_PDL=0) give the same bits: nothing that runs ahead of its
    dependency wait reads what is still being written."""
    config, t = MODELS["wide"]()
    folder = write_model(str(tmp_path / "m"), config, t)
    code = ("import sys, numpy as np; sys.path.insert(0, %r); import ctox_llm_b200 as c\n"
            "ex = c.open_model(%r, dtype=sys.argv[1], max_context_tokens=512, pass_tokens=160)\n"
            "t = [int(x) for x in np.random.default_rng(1).integers(0, 1000, 330)]\n"
            "out = [ex.extend(t[:300], range(0, 300, 7)), ex.extend(t[300:305], range(5))]\n"
            "out += [ex.extend(t[i:i + 1], [0]) for i in range(305, 330)]\n"
            "np.save(sys.argv[2], np.concatenate(out))\n" % (ROOT, folder))
    for dtype in DTYPES:
        files = []
        for pdl in ("1", "0"):
            files.append(str(tmp_path / f"{dtype}{pdl}.npy"))
            subprocess.run([sys.executable, "-c", code, dtype, files[-1]], check=True, env={**os.environ, "CTOX_PDL": pdl})
        assert np.array_equal(np.load(files[0]), np.load(files[1]))


# ---- refusals
def test_refusals(be, opened):
    config, t = MODELS["mixed"]()
    for bad in (attention(heads=5, kv_heads=2), attention(rot=7), attention(rot=26, dim=24), attention(vdim=44), mlstm(gate_cap=0.0)):
        c, tt = model([attention(), bad])
        with pytest.raises(ctox.CtoxError) as e:
            opened(c, tt, "bfloat16")
        assert e.value.kind == "Shape"
    for missing in ("l2.mix.q.b", "l4.mix.vmix", "l3.mix.f", "l0.mix.norm", "l5.mlp.gate", "final.norm"):
        short = dict(t)
        del short[missing]
        with pytest.raises(ctox.CtoxError):
            opened(config, short, "bfloat16")
    ex = opened(config, t, "bfloat16", context=64)
    for tensor in (N.T_LM_HEAD, N.T_Q_DOWN, N.T_ATTN_QKV):
        with pytest.raises(ctox.CtoxError):
            ex.load_vector(0, tensor, np.zeros(4, np.float32))
    assert run(ex, [1, 2]).shape == (2, config["vocab"])
    assert be.device_error() == 0
