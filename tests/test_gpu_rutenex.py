"""Rutenex on the GPU against the plain numpy statement (oracle/rutenex.py): each mechanism, prompts against decoding,
portions of any size, sequences one after the other, keys at the edge of the window, sizes off every grid, and generation
through the engine's own loop.  FP32 engines run everything in 32-bit; BF16 engines keep BF16 weights, FP16 cache rows and
16-bit tensor-core operands (activations as hi + lo pairs)."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

from oracle import rutenex as R
from rutenex_util import ODD, SMALL, bf16_bits, engine, error, mixer, model, portions, tokens

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TOL = {"float32": 4e-6, "bfloat16": 3e-3}
DTYPES = sorted(TOL)


@pytest.fixture(scope="module")
def E():
    import torch
    if not torch.cuda.is_available():
        pytest.skip("needs a GPU")
    from lighterpp_b200 import engine
    return engine


@pytest.fixture(scope="module")
def small():
    W = R.random_weights(SMALL, 1)
    toks = tokens(SMALL, 150, 1)
    return W, toks, R.forward(SMALL, W, toks)


def check(got, want, dtype, slack=1.0):
    e = error(got, want)
    print(f"{dtype}: {e:.2e}")
    assert e <= TOL[dtype] * slack, (e, TOL[dtype])
    return e


# ------------------------------------------------------------------ whole prompts, decoding, portions

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", [[150], [1], [2], [3, 1, 64, 2, 65], [63, 1, 1, 80], [5]], ids=str)
def test_portions(E, small, dtype, sizes):
    W, toks, want = small
    e = engine(E, SMALL, W, dtype)
    got = portions(e, toks, sizes)
    check(got, want, dtype)
    e.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_wanted_places_only(E, small, dtype):
    """Logits of some places of a portion, none of others; a portion without any leaves the cache as one with."""
    W, toks, want = small
    e = engine(E, SMALL, W, dtype)
    a = e.extend(toks[:100], 0, [0, 63, 64, 99])
    e.extend(toks[100:130], 100)
    b = e.extend(toks[130:], 130, [0, 19])
    check(np.concatenate([a, b]), want[[0, 63, 64, 99, 130, 149]], dtype)
    for bad in ([3, 3], [4, 2], [20], [-1]):
        with pytest.raises(E.LppError):
            e.extend(toks[130:], 130, bad)
    with pytest.raises(E.LppError):
        e.extend([SMALL["vocab"]], 0)
    with pytest.raises(E.LppError):
        e.extend(toks[:2], 255)
    e.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_sequences_one_after_the_other(E, small, dtype):
    """The cache is used again: what an earlier, longer sequence left never shows, to the last bit."""
    W, toks, want = small
    e = engine(E, SMALL, W, dtype)
    first = portions(e, toks[:40], [17, 1, 22])
    portions(e, tokens(SMALL, 200, 9), [64, 3])
    again = portions(e, toks[:40], [17, 1, 22])
    assert np.array_equal(first, again)
    check(again, want[:40], dtype)
    e.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding_passes_the_window_over_decoded_tokens(E, dtype):
    cfg = model([(mixer(window=21), 64), (mixer(window=70, kv_rank=64), 64)], width=64)
    W, toks = R.random_weights(cfg, 3), tokens(cfg, 420, 3)
    want = R.forward(cfg, W, toks)
    e = engine(E, cfg, W, dtype, seq_len=420)
    e.extend(toks[:5], 0)
    got = np.stack([e.step_logits(int(t), 5 + i) for i, t in enumerate(toks[5:])])
    check(got, want[5:], dtype)
    e.close()


@pytest.mark.parametrize("n", [1, 2, 3, 16, 17])
def test_first_tokens(E, small, n):
    W, toks, want = small
    for dtype in DTYPES:
        e = engine(E, SMALL, W, dtype, seq_len=n)  # the cache is exactly as long as the sequence
        check(portions(e, toks[:n], [n]), want[:n], dtype)
        check(portions(e, toks[:n], [1]), want[:n], dtype)
        e.close()


# ------------------------------------------------------------------ mechanisms

@pytest.mark.parametrize("dtype", DTYPES)
def test_cache_rows(E, small, dtype):
    """What a token leaves behind in the first layer, written by the prompt path and by the step: latent normed, key part
    rotated (YaRN), for near and far positions."""
    W, toks, _ = small
    e = engine(E, SMALL, W, dtype)
    e.extend(toks[:100], 0)
    for i in range(100, 150):
        e.step_logits(int(toks[i]), i)
    x = R.layer_norm(W["embed"][toks].astype(np.float64), W["l0.norm1"], W["l0.norm1.b"], 1e-5)
    c, k = R.latent_split(x, {n: a.astype(np.float64) for n, a in W.items()}, "l0.mix.", SMALL["layers"][0]["mixer"], 1e-5, np.arange(150))
    want = np.concatenate([c, k], axis=1)
    got = np.stack([e.latent_read(0, p) for p in range(150)])
    assert np.abs(got - want).max() <= (2e-5 if dtype == "float32" else 4e-3) * np.abs(want).max()
    with pytest.raises(E.LppError):
        e.kv_prefill(0, np.zeros((1, 1, 8), np.float32), np.zeros((1, 1, 8), np.float32), 1)
    e.close()


@pytest.mark.parametrize("rot", [dict(base=7.0, scaling=False), dict(base=40.0, factor=8.0, original=200, fast=16.0, slow=0.5),
                                 dict(base=1e6, factor=1.5, original=2048, fast=32.0, slow=1.0), dict(base=30.0, dims=4, factor=2.0),
                                 dict(base=30.0, dims=0, scaling=False), dict(base=50.0, original=5, fast=1.0, slow=1.0)], ids=str)
def test_rotations(E, rot):
    """Plain and stretched rotations, only a part of the rotated dimensions turning, none, and a ramp of zero length."""
    cfg = model([(mixer(rot_dim=12, window=0, scale=0.6, **rot), 0)], width=64)
    W, toks = R.random_weights(cfg, 4), tokens(cfg, 180, 4)
    want = R.forward(cfg, W, toks)
    for dtype in DTYPES:
        e = engine(E, cfg, W, dtype)
        check(portions(e, toks, [90, 1, 1, 60]), want, dtype)
        e.close()


def test_layer_norm_with_a_large_mean_and_a_large_epsilon(E):
    cfg = model([(mixer(), 40)], eps=0.4)
    W = R.random_weights(cfg, 6)
    W["embed"] = R.bf16_round(W["embed"] + 25.0)
    toks = tokens(cfg, 30, 6)
    want = R.forward(cfg, W, toks)
    want -= want.mean(axis=1, keepdims=True)  # 25 times the sum of the last norm's rows: the same in every logit
    for dtype in DTYPES:
        e = engine(E, cfg, W, dtype)
        got = portions(e, toks, [12, 1, 17])
        check(got - got.mean(axis=1, keepdims=True), want, dtype, 25.0 if dtype == "float32" else 2.0)  # the mean is 25 times the spread
        e.close()


@pytest.mark.parametrize("width", [2056, 4104, 8200])
def test_wide_rows(E, width):
    """Norms of rows that no longer fit the registers of one pass."""
    cfg = model([(mixer(heads=2, dim=8, vdim=8, kv_rank=16), 24)], width=width, vocab=33)
    W, toks = R.random_weights(cfg, 7), tokens(cfg, 9, 7)
    want = R.forward(cfg, W, toks)
    for dtype in DTYPES:
        e = engine(E, cfg, W, dtype, seq_len=16)
        check(portions(e, toks, [5, 1]), want, dtype)
        e.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_sizes_off_every_grid(E, dtype):
    W, toks = R.random_weights(ODD, 2), tokens(ODD, 140, 2)
    want = R.forward(ODD, W, toks)
    e = engine(E, ODD, W, dtype)
    check(portions(e, toks, [70, 1, 2, 3, 40, 1]), want, dtype, 1.5)
    e.close()


@pytest.mark.parametrize("width,ff", [(71, 300), (130, 700)])
def test_padding_of_narrow_rows_stays_zero(E, width, ff):
    """Residual products cut along K whose rows are narrower than the row pitch: partial sums of the padding are zero too."""
    cfg = model([(mixer(heads=9, vdim=24), ff), (mixer(), ff)], width=width)
    W, toks = R.random_weights(cfg, ff), tokens(cfg, 100, ff)
    e = engine(E, cfg, W, "bfloat16")
    check(portions(e, toks, [70, 2, 28]), R.forward(cfg, W, toks), "bfloat16")
    e.close()


@pytest.mark.parametrize("heads,kv_rank,rot_dim,window", [(4, 96, 16, 30), (16, 200, 8, 100), (12, 512, 64, 150), (24, 128, 16, 20),
                                                          (33, 256, 32, 64), (20, 448, 64, 0), (3, 640, 16, 90), (17, 8, 2, 65)])
def test_attention_instantiations(E, heads, kv_rank, rot_dim, window):
    """Every tensor-core tile shape (query rows of one and of several tokens, latent widths, several key splits) and a
    latent too wide for it, against the CUDA-core kernel and the oracle."""
    cfg = model([(mixer(heads=heads, dim=16, rot_dim=rot_dim, vdim=12, kv_rank=kv_rank, window=window, scale=0.7), 32)], width=128, vocab=64)
    W, toks = R.random_weights(cfg, heads), tokens(cfg, 230, heads)
    want = R.forward(cfg, W, toks)
    for flags in (0, E.FLAG_LATENT_CUDA_CORES):
        e = engine(E, cfg, W, "bfloat16", flags=flags)
        check(portions(e, toks, [130, 1, 1, 1, 64, 30, 1]), want, "bfloat16")
        e.close()


@pytest.mark.parametrize("flags", ["FLAG_GEMV_LDG", "FLAG_NO_GRAPH", "FLAG_NO_PDL", "FLAG_NO_PREFILL_GEMM"])
def test_engine_flags(E, small, flags):
    W, toks, want = small
    for dtype in DTYPES:
        e = engine(E, SMALL, W, dtype, flags=getattr(E, flags))
        check(portions(e, toks[:60], [40, 1]), want[:60], dtype)
        e.close()


# ------------------------------------------------------------------ keys far away and at the edges of the window

def needle_model(window):
    """One layer in which every query looks for one token: queries come from the norm's large bias and point along that
    token's latent, so its key stands out by several units of score wherever it is visible."""
    cfg = model([(mixer(heads=2, dim=32, rot_dim=4, vdim=24, kv_rank=32, window=window, scale=1.0, scaling=False), 0)], width=64, vocab=80)
    W = R.random_weights(cfg, 12)
    W["l0.norm1.b"] = R.bf16_round(3.0 * np.sign(np.random.default_rng(5).standard_normal(64)))
    m, b = cfg["layers"][0]["mixer"], W["l0.norm1.b"].astype(np.float64)
    W["l0.mix.q"] = np.zeros_like(W["l0.mix.q"])
    h = R.layer_norm(W["embed"].astype(np.float64), W["l0.norm1"], W["l0.norm1.b"], 1e-5)
    c, _ = R.latent_split(h, W, "l0.mix.", m, 1e-5, np.zeros(80))
    for a in range(2):
        keys = c @ W["l0.mix.uk"][32 * a:32 * a + 32].T.astype(np.float64)
        away = keys[79] - keys[:79].mean(axis=0)
        W["l0.mix.q"][36 * a:36 * a + 32] = R.bf16_round(np.outer(9.0 * away / (away @ away), b / (b @ b)))
    W["l0.mix.uv"] *= 4
    return cfg, W


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window", [1, 2, 16, 63, 64, 65, 100, 130])
def test_needle_at_the_edge_of_the_window(E, dtype, window):
    cfg, W = needle_model(window)
    n = 2 * window + 150
    for at in (0, 1, 62, 63, 64, 100):
        toks = np.random.default_rng(at).integers(0, 79, n).astype(np.int32)
        toks[at] = 79
        inside, outside = at + window - 1, at + window
        spots = sorted({at, min(at + 1, n - 1), max(at, inside - 1), inside, outside, outside + 1})
        want = R.forward(cfg, W, toks)
        toks_without = toks.copy()
        toks_without[at] = 0
        without = R.forward(cfg, W, toks_without)
        if window > 1:
            assert error(without[inside], want[inside]) > 0.15  # the needle's weight is in these logits
        assert error(without[outside], want[outside]) < 1e-12
        e = engine(E, cfg, W, dtype, seq_len=n)
        check(e.extend(toks[:outside + 2], 0, spots), want[spots], dtype)              # all in one portion
        e.extend(toks[:at + 1], 0)                                                     # the needle ends a portion
        if outside - 2 > at + 1:
            e.extend(toks[at + 1:outside - 2], at + 1)
        start = max(at + 1, outside - 2)
        got = np.stack([e.step_logits(int(toks[p]), p) for p in range(start, outside + 2)])  # decoding across the edge
        check(got, want[start:outside + 2], dtype)
        e.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n,seq_len", [(700, 700), (700, 9000), (2500, 2500)])
def test_far_key_without_a_window(E, dtype, n, seq_len):
    """Splits that meet in a cluster, splits left apart (a long cache), and more keys than splits of the smallest size."""
    cfg, W = needle_model(0)
    toks = np.random.default_rng(0).integers(0, 79, n).astype(np.int32)
    toks[3] = 79
    want = R.forward(cfg, W, toks)
    e = engine(E, cfg, W, dtype, seq_len=seq_len)
    e.extend(toks[:n - 60], 0)
    check(e.extend(toks[n - 60:n - 10], n - 60, range(50)), want[n - 60:n - 10], dtype)
    check(np.stack([e.step_logits(int(toks[p]), p) for p in range(n - 10, n)]), want[n - 10:], dtype)
    e.close()


# ------------------------------------------------------------------ generation and programs

@pytest.mark.parametrize("dtype", DTYPES)
def test_greedy_generation(E, small, dtype):
    """Every token the device-resident loop picks is the best of the oracle's logits for its own prefix (ties within
    the tolerance); the same tokens come out of one step call per token."""
    from lighterpp_b200.session import Session
    W, toks, _ = small
    e = engine(E, SMALL, W, dtype)
    s = Session(e)
    prompt = [int(t) for t in toks[:75]]
    out = s.generate(prompt, 60)
    assert s.generate(prompt, 60) == out
    lg = R.forward(SMALL, W, prompt + out)
    for i, t in enumerate(out):
        row = lg[len(prompt) - 1 + i]
        assert row.max() - row[t] <= 8 * TOL[dtype] * np.sqrt((row ** 2).mean()), i
    e.extend(prompt[:-1], 0)
    tok, got = prompt[-1], []
    for i in range(60):
        tok = e.forward(tok, len(prompt) - 1 + i)
        got.append(tok)
    assert got == out
    sampled = s.generate(prompt, 40, temperature=0.9, penalty=1.1, seed=3)
    assert sampled == s.generate(prompt, 40, temperature=0.9, penalty=1.1, seed=3) and sampled != out[:40]
    e.close()


def test_programs(E, small, tmp_path):
    """The command line and the trace replayer on a model folder."""
    W, toks, want = small
    folder = str(tmp_path / "model")
    R.write_model(folder, SMALL, W)
    from lighterpp_b200.models import load_engine
    from lighterpp_b200.session import Session
    prompt = [int(t) for t in toks[:20]]
    eng = load_engine(folder)
    expect = Session(eng).generate(prompt, 12)
    eng.close()
    r = subprocess.run([sys.executable, "-m", "lighterpp_b200", "generate", "--model", folder, "--prompt", ",".join(map(str, prompt)), "-n", "12"],
                       cwd=ROOT, capture_output=True, text=True, timeout=120)
    assert r.returncode == 0, r.stderr
    assert [int(t) for t in r.stdout.split(",")] == expect
    steps, cuts = [], [0, 40, 41, 43, 110, 150]
    for i, (a, b) in enumerate(zip(cuts, cuts[1:])):
        steps.append({"step": i, "entries": [{"id": "x", "tokens": toks[a:b].tolist(), "want": [] if i == 2 else [b - a - 1, 0]}],
                      "end": ["x"] if b == 150 else []})
    steps.append({"step": 9, "entries": [{"id": "y", "tokens": toks[:7].tolist(), "want": [6]}], "end": ["y"]})
    for dtype in DTYPES:
        out = tmp_path / dtype
        out.mkdir()
        r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", dtype, "--out", str(out), "--max-tokens", "150"],
                           input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=120)
        assert r.returncode == 0, r.stderr
        assert r.stdout.split("\n")[:-1] == [f"done {s['step']}" for s in steps]
        assert sorted(os.listdir(out)) == ["0.f32", "1.f32", "3.f32", "4.f32", "9.f32"]
        for i, (a, b) in enumerate(zip(cuts, cuts[1:])):
            if i != 2:
                check(np.fromfile(out / f"{i}.f32", dtype="<f4").reshape(2, -1), want[[b - 1, a]], dtype)
        check(np.fromfile(out / "9.f32", dtype="<f4"), want[6], dtype)


def test_incomplete_and_wrong_uploads_are_refused(E, small):
    from rutenex_util import configured
    W, _, _ = small
    e = E.Engine(configured(SMALL, 16), "bf16", "f16")
    with pytest.raises(E.LppError, match="was never uploaded"):
        e.finalize()
    with pytest.raises(E.LppError, match="does not belong"):
        e.upload("wq", np.zeros((4, 4), np.float32), 0)
    with pytest.raises(E.LppError, match="no feed-forward"):
        e.upload("w1", bf16_bits(W["l0.mlp.gate"]), 1)
    e.close()
    c = configured(SMALL, 16)
    c.layers[0].mixer.rot_dim = 7
    with pytest.raises(E.LppError, match="rotation"):
        E.Engine(c, "bf16", "f16")
    with pytest.raises(E.LppError, match="BF16 / F16"):
        E.Engine(configured(SMALL, 16), "f16", "f16")


def test_portions_with_logits_on_the_grouped_query_engine(E):
    """lpp_extend serves the reference's own architecture too: batched portions against one step per token."""
    from lighterpp_b200 import synth
    c, dt, tied, seed, T = synth.named("tiny-gqa-f16")
    toks = synth.prompt_tokens(c.vocab_size, 90, seed)
    a, b = E.Engine(c, dt, "f16"), E.Engine(c, dt, "f16")
    for e in (a, b):
        e.load_weights(T)
    got = np.concatenate([a.extend(toks[:70], 0, [0, 5, 63, 64, 69]), a.extend(toks[70:71], 70, [0]), a.extend(toks[71:90], 71, [18])])
    want = np.stack([b.step_logits(int(t), p) for p, t in enumerate(toks)])[[0, 5, 63, 64, 69, 70, 89]]
    assert np.abs(got - want).max() < 2e-3 * max(1.0, np.abs(want).max())
    a.close()
    b.close()
