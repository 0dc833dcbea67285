"""Lomelorn on the GPU against the plain implementation (lomelorn_oracle.py), through the registry, the
executor's own calls and the command line."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import ctox_llm_b200 as ctox
from ctox_llm_b200 import _native as N
import lomelorn_oracle as oracle
from lomelorn_util import bf16, layer, model, row_errors, write_model

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
# row_errors of a single row. In 16 bits a layer norm of a small sublayer output amplifies the rounding of
# single rows (the same rows as when the operands are rounded in the plain implementation): close() bounds
# the worst row loosely and the mean tightly.
TOL = {"float32": 2e-5, "bfloat16": 0.1}
ROW = {"float32": 2e-5, "bfloat16": 5e-2}  # a row that does not suffer from it
MEAN = {"float32": 1e-5, "bfloat16": 1e-2}
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


# Sizes that are nobody's: odd widths, dims that are no multiple of 16, layers that differ in everything,
# several readers of one cache with other windows, a layer without a feed-forward, a window of one token.
MODELS = {
    "mixed": lambda: model([layer(), layer(heads=2, dim=40, vdim=24, q_rank=50, ff=None, kv_from=0, window=29, scale=0.4),
                            layer(heads=1, dim=7, rot_dim=6, vdim=9, q_rank=5, kv_rank=11, window=1, base=5e4, ff=33),
                            layer(kv_from=0, window=3, heads=4, ff=77)], seed=1),
    "one_head": lambda: model([layer(heads=1, dim=1, rot_dim=2, vdim=1, q_rank=1, kv_rank=2, ff=1)], vocab=13, width=5, seed=2),
    "wide": lambda: model([layer(heads=16, dim=64, rot_dim=32, vdim=96, q_rank=200, kv_rank=264, window=150, ff=700),
                           layer(heads=20, dim=48, rot_dim=32, vdim=64, q_rank=96, kv_rank=264, window=70, ff=512, kv_from=0)],
                          vocab=1000, width=384, seed=3),
    "rank_512": lambda: model([layer(heads=12, dim=128, rot_dim=64, vdim=128, q_rank=256, kv_rank=512, window=90, ff=320)],
                              vocab=300, width=256, seed=4),
    "rank_768": lambda: model([layer(heads=3, dim=32, rot_dim=16, vdim=144, q_rank=64, kv_rank=768, window=40)], seed=5),
    "rank_1100": lambda: model([layer(heads=2, dim=16, rot_dim=16, vdim=32, q_rank=64, kv_rank=1100, window=40)], seed=6),
    "vdim_272": lambda: model([layer(heads=2, dim=32, rot_dim=16, vdim=272, window=40)], seed=7),
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(MODELS))
def test_whole_prompt_portions_and_single_tokens(opened, name, dtype):
    config, t = MODELS[name]()
    tokens = tokens_of(230, config["vocab"])
    want, streams = oracle.forward(config, t, tokens)
    ex = opened(config, t, dtype)
    ex.keep_streams()
    whole = run(ex, tokens)
    assert close(whole, want, dtype)
    for l in range(len(config["layers"])):
        assert close(ex.last_stream(l, 0, len(tokens)), streams[l], dtype)
    # portions of 2, 3, ... tokens, around the pass and page sizes, then one by one
    cuts = np.cumsum([2, 3, 4, 5, 7, 8, 9, 2, 16, 17, 63, 2]).tolist()
    portions = run(ex, tokens, cuts + list(range(cuts[-1] + 40, len(tokens))))
    assert close(portions, want, dtype)
    single = run(ex, tokens[:60], range(1, 60))
    assert close(single, want[:60], dtype)


def test_portions_of_a_tile_again_and_again(opened):
    """Few key tiles per pass and many passes: the last products of a tile row are the ones just issued."""
    config, t = model([layer(heads=10, dim=32, rot_dim=16, vdim=80, window=100), layer(heads=6, dim=64, rot_dim=32, vdim=48, window=60)],
                      seed=8)
    tokens = tokens_of(700, config["vocab"], 4)
    want, _ = oracle.forward(config, t, tokens)
    ex = opened(config, t, "bfloat16")
    first = None
    for size in (64, 63, 37, 130) * 5:
        got = run(ex, tokens, range(size, 700, size))
        assert close(got, want, "bfloat16"), size
        if size == 64:
            first = got if first is None else first
            assert np.array_equal(got, first)


@pytest.mark.parametrize("heads,dim,rot_dim,vdim,window,size", [(16, 128, 64, 128, 4096, 1000), (6, 32, 32, 112, 90, 1000),
                                                                (6, 32, 32, 112, 90, 70), (10, 64, 32, 48, 300, 500)])
def test_many_prompts_give_the_same_bits(be, heads, dim, rot_dim, vdim, window, size):
    spec = dict(rope_base=1e4, mixer=N.MIXER_LATENT_ATTENTION, heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, q_rank=256,
                kv_rank=128, window=window, kv_from=-1, score_scale=3 * (dim + rot_dim) ** -0.5, mlp=N.MLP_RELU2, ff=512)
    ex = ctox.B200Executor(be, ctox.StackConfig(vocab_size=1000, hidden_size=512, norm_eps=1e-6, logit_softcap=30.0,
                                                layers=[N.LayerConfig(**spec) for _ in range(3)], max_context_tokens=3100))
    ex.fill_synthetic(0)
    ex.warmup()
    tokens, first = tokens_of(3000, 1000, 1), None
    for _ in range(40):
        ex.reset_session()
        for a in range(0, 3000, size):
            ex.extend(tokens[a:a + size])
        hidden = ex.last_hidden()
        first = hidden if first is None else first
        assert np.array_equal(hidden, first)
    ex.unload()


@pytest.mark.parametrize("dtype", DTYPES)
def test_passes_of_every_short_length(opened, dtype):
    config, t = MODELS["mixed"]()
    tokens = tokens_of(70, config["vocab"], 5)
    want, _ = oracle.forward(config, t, tokens)
    ex = opened(config, t, dtype)
    for m in range(1, 12):
        assert close(run(ex, tokens, range(m, 70, m)), want, dtype), m


# ---- mechanisms on their own
def test_normed_query_latent_and_its_weight(opened):
    config, t = model([layer(ff=None)], seed=11)
    t["l0.mix.dq"] = bf16(t["l0.mix.dq"] * 64)  # without the norm the scores would be 64 times larger
    t["l0.mix.dq.norm"] = bf16(t["l0.mix.dq.norm"] * np.linspace(0.1, 3.0, 36))
    tokens = tokens_of(40, config["vocab"])
    want, _ = oracle.forward(config, t, tokens)
    for dtype in DTYPES:
        assert close(run(opened(config, t, dtype), tokens), want, dtype)


def test_normed_key_latent_leaves_the_rotated_part_alone(opened):
    config, t = model([layer(ff=None)], seed=12)
    t["l0.mix.dkv"] = bf16(t["l0.mix.dkv"] * np.r_[np.full(56, 20.0), np.full(8, 3.0)][:, None])
    tokens = tokens_of(40, config["vocab"])
    want, _ = oracle.forward(config, t, tokens)
    for dtype in DTYPES:
        assert close(run(opened(config, t, dtype), tokens), want, dtype)


def test_rotation_alone_decides(opened):
    """Unrotated keys are zero: scores depend on the rotated part and on the distance only."""
    config, t = model([layer(ff=None, rot_dim=24, kv_rank=40, base=37.0, window=60, scale=0.5)], seed=13)
    t["l0.mix.uk"] = t["l0.mix.uk"] * 0
    tokens = tokens_of(120, config["vocab"])
    want, _ = oracle.forward(config, t, tokens)
    off, _ = oracle.forward({**config, "layers": [layer(ff=None, rot_dim=24, kv_rank=40, base=74.0, window=60, scale=0.5)]},
                            t, tokens)
    assert row_errors(off, want)[60:].mean() > PLANTED  # another base would show
    for dtype in DTYPES:
        ex = opened(config, t, dtype)
        assert close(run(ex, tokens), want, dtype)
        assert close(run(ex, tokens, range(1, 120)), want, dtype)


def test_softcap_is_applied_once_and_everywhere(opened):
    config, t = model([layer(ff=None)], softcap=1.5, seed=14)
    tokens = tokens_of(30, config["vocab"])
    want, _ = oracle.forward(config, t, tokens)
    assert np.abs(want).max() > 1.4
    for dtype in DTYPES:
        ex = opened(config, t, dtype)
        for cuts in ((), (1, 2, 5)):
            assert close(run(ex, tokens, cuts), want, dtype)


def test_norm_eps_is_used_in_every_norm(opened):
    config, t = model([layer()], eps=0.5, seed=15)
    tokens = tokens_of(30, config["vocab"])
    want, _ = oracle.forward(config, t, tokens)
    for dtype in DTYPES:
        ex = opened(config, t, dtype)
        for cuts in ((), range(1, 30)):
            assert close(run(ex, tokens, cuts), want, dtype)


# ---- a key that stands out
def standing_out(window, heads=2, seed=20, layers=1, kv_from=None):
    """A model whose scores depend on the tokens alone (no rotated keys), a query token and the key token
    that outweighs every other token by far in its first layer's first head."""
    specs = [layer(heads=heads, ff=None, window=window, scale=1.0)]
    config, t = model(specs, seed=seed)
    t["l0.mix.dkv"][56:] = 0
    T = {k: np.asarray(v, np.float64) for k, v in t.items()}
    mt = oracle.layer_tensors(T, 0, "mix")
    h = oracle.layer_norm(T["embed"], T["l0.norm1"], 1e-3)
    m = specs[0]["mixer"]
    q, _ = oracle.latent_queries(h, mt, m, 1e-3)
    c, _ = oracle.latent_keys(h, mt, m, 1e-3)
    score = q[0] @ (c @ mt["uk"][:24].T).T
    ranked = np.sort(score, -1)
    query = int(np.argmax(ranked[:, -1] - ranked[:, -2]))
    key = int(np.argmax(score[query]))
    m["scale"] = float(np.float32(12.0 / (ranked[query, -1] - ranked[query, -2])))
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
                assert row_errors(got, want)[query_at] < ROW[dtype], (query_at, distance, cuts)


@pytest.mark.parametrize("dtype", DTYPES)
def test_far_keys_at_page_and_tile_borders(opened, dtype):
    config, t, query, key, filler = standing_out(700)
    ex = opened(config, t, dtype)
    for key_at in (0, 1, 63, 64, 127, 128, 129, 255, 256):
        tokens = place(620, 600, key_at, query, key, filler, seed=key_at)
        want, _ = oracle.forward(config, t, tokens)
        lost = list(tokens)
        lost[key_at] = filler[0]
        without, _ = oracle.forward(config, t, lost)
        assert row_errors(without, want)[600] > PLANTED
        for cuts in ((), (600, 601), (key_at + 1, 598)):
            assert row_errors(run(ex, tokens, cuts), want)[600] < ROW[dtype], (key_at, cuts)


@pytest.mark.parametrize("dtype", DTYPES)
def test_first_tokens(opened, dtype):
    config, t = MODELS["wide"]()
    ex = opened(config, t, dtype)
    for n in (1, 2, 3, 8, 9, 10, 17):
        tokens = tokens_of(n, config["vocab"], n)
        want, _ = oracle.forward(config, t, tokens)
        assert close(run(ex, tokens), want, dtype)
        assert close(run(ex, tokens, range(1, n)), want, dtype)


# ---- cache pages and sessions
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("pages,pass_tokens", [(128, 64), (128, 130), (16, 0), (24, 0)])
def test_pages_are_used_again_when_the_window_has_passed(opened, dtype, pages, pass_tokens):
    """The cache is a ring of pages: far fewer slots than tokens. (Pages that are no whole tiles allow
    short passes only.)"""
    config, t = model([layer(window=40), layer(window=61, kv_from=0), layer(window=9)], seed=30)
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
        got = run(ex, r, (len(r) // 2,) if len(r) > 1 else ())
        assert np.array_equal(got, alone[k])


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding(opened, dtype):
    config, t = MODELS["mixed"]()
    tokens = tokens_of(560, config["vocab"], 9)
    want, _ = oracle.forward(config, t, tokens)
    ex = opened(config, t, dtype)
    got = run(ex, tokens, [50] + list(range(51, 560)))
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
        ex = opened(config, t, "bfloat16")
        got = list(ex.generate(prompt, 24))
        logits, _ = oracle.forward(config, t, list(prompt) + got)
        for i, token in enumerate(got):
            row = logits[len(prompt) - 1 + i]
            assert row[token] > row.max() - TOL["bfloat16"] * np.sqrt((logits ** 2).mean())


def test_sampling_and_selection(opened):
    config, t = MODELS["mixed"]()
    prompt = tokens_of(12, config["vocab"], 8)
    ex = opened(config, t, "float32")
    greedy = list(ex.generate(prompt, 10))
    assert list(ex.generate(prompt, 10, temperature=0.7, top_k=1)) == greedy
    a = list(ex.generate(prompt, 16, temperature=2.0, seed=5))
    assert a == list(ex.generate(prompt, 16, temperature=2.0, seed=5)) and a != list(ex.generate(prompt, 16, temperature=2.0, seed=6))
    assert list(ex.generate(prompt, 10, stop_tokens=[greedy[3]]))[-1] == greedy[3]
    # the distribution of the first sampled token
    logits, _ = oracle.forward(config, t, prompt)
    p = np.exp((logits[-1] - logits[-1].max()) / 3.0)
    p /= p.sum()
    seen = np.zeros(config["vocab"])
    for s in range(1500):
        seen[next(iter(ex.generate(prompt, 1, temperature=3.0, seed=s)))] += 1
    assert 0.5 * np.abs(seen / seen.sum() - p).sum() < 0.15


def test_decode_reports_logits_and_hidden_state(opened):
    config, t = MODELS["mixed"]()
    prompt = tokens_of(20, config["vocab"], 2)
    ex = opened(config, t, "float32")
    ex.keep_logits(True)
    ex.prefill(prompt)
    blk = ex.decode(prompt[-1], mtp_enabled=False)
    logits, streams = oracle.forward(config, t, prompt)
    assert close(ex.last_logits(0)[None], logits[-1:], "float32") and blk.token_id == int(np.argmax(logits[-1]))
    final = oracle.layer_norm(streams[-1][-1], np.asarray(t["final.norm"], np.float64), config["norm"]["eps"])
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
    out = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", "float32", "--out", str(tmp_path),
                          "--max-tokens", "45"], input="\n".join(json.dumps(s) for s in steps), capture_output=True, text=True)
    assert out.returncode == 0, out.stderr[-2000:]
    assert out.stdout.split("\n")[:3] == ["done 0", "done 1", "done 2"]
    rows = [np.fromfile(tmp_path / f"{i}.f32", "<f4").reshape(-1, config["vocab"]) for i in range(3)]
    got = np.concatenate(rows)
    assert close(got, want[list(range(40)) + [40, 44, 0]], "float32")


def test_dependent_launch_overlap_changes_no_bit(tmp_path):
    """The same calls with every launch serialised (CTOX_PDL=0) give the same bits: nothing that runs ahead
    of its dependency wait reads what is still being written."""
    config, t = MODELS["wide"]()
    folder = write_model(str(tmp_path / "m"), config, t)
    code = ("import sys, numpy as np; sys.path.insert(0, %r); import ctox_llm_b200 as c\n"
            "ex = c.open_model(%r, dtype=sys.argv[1], max_context_tokens=512, pass_tokens=96)\n"
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
def test_refusals(be, opened, tmp_path):
    config, t = MODELS["mixed"]()
    ex = opened(config, t, "bfloat16", context=64)
    for tokens, want in (([config["vocab"]], []), ([1] * 60, []), ([1, 2], [2]), ([1, 2], [1, 0])):
        with pytest.raises(ctox.CtoxError) as e:
            ex.extend(tokens, want)
        assert e.value.kind == "Shape"
    with pytest.raises(ctox.CtoxError):
        ex.decode(1, mtp_enabled=True)
    with pytest.raises(ctox.CtoxError):  # a hybrid model's tensor
        ex.load_vector(0, N.T_A_LOG, np.zeros(4, np.float32))
    token = ctox.CancellationToken()
    token.cancel()
    with pytest.raises(ctox.CtoxError) as e:
        ex.extend([1, 2], [], token)
    assert e.value.kind == "Cancelled"
    assert run(ex, [1, 2]).shape == (2, config["vocab"])  # still usable
    for bad in (layer(kv_from=0, kv_rank=40), layer(kv_from=0, rot_dim=6), layer(kv_from=0, base=3.0), layer(kv_from=1),
                layer(kv_from=5)):
        c, tt = model([layer(), bad])
        with pytest.raises(ctox.CtoxError) as e:
            opened(c, tt, "bfloat16")
        assert e.value.kind == "Shape"
    short = dict(t)
    del short["l1.mix.uv"]
    with pytest.raises(ctox.CtoxError):
        opened(config, short, "bfloat16")
    assert be.device_error() == 0
