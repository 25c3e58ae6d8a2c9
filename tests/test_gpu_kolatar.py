"""Kolatar on the GPU against the plain numpy statement (oracle/kolatar.py): each mechanism, prompts against decoding, portions
of any size, sequences one after the other, keys and states far back and at the edge of a window, sizes off every grid, loops,
and generation through the engine's own loop.  FP32 engines run everything in 32-bit; BF16 engines keep BF16 weights, FP16
cache rows, an FP32 recurrent state and 16-bit tensor-core operands (activations as hi + lo pairs)."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

from kolatar_util import ODD, SMALL, attention, mamba, model
from oracle import kolatar as K
from rutenex_util import configured, engine, error, portions, tokens

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
    W = K.random_weights(SMALL, 1)
    toks = tokens(SMALL, 150, 1)
    return W, toks, K.forward(SMALL, W, toks)


def check(got, want, dtype, slack=1.0):
    e = error(got, want)
    print(f"{dtype}: {e:.2e}")
    assert e <= TOL[dtype] * slack, (e, TOL[dtype])
    return e


def check_model(E, cfg, n, sizes, seed=0, dtypes=DTYPES, slack=1.0, W=None, toks=None, **kw):
    W = K.random_weights(cfg, seed) if W is None else W
    toks = tokens(cfg, n, seed) if toks is None else toks
    want = K.forward(cfg, W, toks)
    for dtype in dtypes:
        e = engine(E, cfg, W, dtype, seq_len=n, **kw)
        check(portions(e, toks, sizes), want, dtype, slack)
        e.close()


# ------------------------------------------------------------------ whole prompts, decoding, portions

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", [[150], [1], [2], [3, 1, 64, 2, 65], [63, 1, 1, 80], [5], [4, 2, 3]], ids=str)
def test_portions(E, small, dtype, sizes):
    W, toks, want = small
    e = engine(E, SMALL, W, dtype)
    check(portions(e, toks, sizes), want, dtype)
    e.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_wanted_places_only(E, small, dtype):
    """Logits of some places of a portion, none of others; a portion without any leaves cache and state as one with."""
    W, toks, want = small
    e = engine(E, SMALL, W, dtype)
    a = e.extend(toks[:100], 0, [0, 63, 64, 99])
    e.extend(toks[100:130], 100)
    b = e.extend(toks[130:], 130, [0, 19])
    check(np.concatenate([a, b]), want[[0, 63, 64, 99, 130, 149]], dtype)
    e.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_sequences_one_after_the_other(E, small, dtype):
    """Cache and state are used again: what an earlier, longer sequence left never shows, to the last bit."""
    W, toks, want = small
    e = engine(E, SMALL, W, dtype)
    first = portions(e, toks[:40], [17, 1, 22])
    portions(e, tokens(SMALL, 200, 9), [64, 3])
    again = portions(e, toks[:40], [17, 1, 22])
    assert np.array_equal(first, again)
    check(again, want[:40], dtype)
    portions(e, tokens(SMALL, 70, 10), [70])
    check(portions(e, toks[:9], [1]), want[:9], dtype)  # a new sequence that starts with single tokens
    e.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_recurrent_state_only_goes_on(E, small, dtype):
    """A position that is neither 0 nor the next one is refused and leaves the sequence as it was; a profile run ends it."""
    W, toks, want = small
    e = engine(E, SMALL, W, dtype)
    e.extend(toks[:50], 0)
    for bad in (49, 51, 1):
        with pytest.raises(E.LppError, match="stands at position 50"):
            e.extend(toks[50:60], bad)
        with pytest.raises(E.LppError, match="stands at position 50"):
            e.step_logits(int(toks[50]), bad)
        with pytest.raises(E.LppError, match="stands at position 50"):
            e.decode(int(toks[50]), bad, 3)
    check(e.extend(toks[50:60], 50, range(10)), want[50:60], dtype)
    check(e.step_logits(int(toks[60]), 60), want[60], dtype)
    e.profile_step(20, 1)
    with pytest.raises(E.LppError, match="start at position 0"):
        e.extend(toks[61:70], 61)
    check(portions(e, toks[:70], [66, 1]), want[:70], dtype)
    e.profile_kind(3, "scan", 1)
    with pytest.raises(E.LppError, match="start at position 0"):
        e.step_logits(0, 70)
    for bad in ([3, 3], [4, 2], [20], [-1]):
        with pytest.raises(E.LppError):
            e.extend(toks[:10], 0, bad)
    with pytest.raises(E.LppError):
        e.extend([SMALL["vocab"]], 0)
    e.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding_passes_the_window_over_decoded_tokens(E, dtype):
    cfg = model([(mamba(inner=64), 0), (attention(window=21), 64), (attention(window=70, heads=2, kv_heads=1, dim=40, rot=16), 64)], width=64, loop=(0, 2, 2))
    W, toks = K.random_weights(cfg, 3), tokens(cfg, 420, 3)
    want = K.forward(cfg, W, toks)
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


# ------------------------------------------------------------------ selective scan

@pytest.mark.parametrize("state,conv,dt_rank,inner", [(1, 1, 1, 33), (16, 2, 8, 64), (17, 3, 9, 70), (32, 4, 33, 128), (33, 5, 61, 48), (64, 4, 16, 36),
                                                      (65, 7, 130, 20), (128, 4, 40, 96), (129, 2, 5, 30), (300, 9, 12, 14), (16, 4, 700, 40), (1000, 4, 1024, 9)])
def test_scan_instantiations(E, state, conv, dt_rank, inner):
    """Every number of lanes and pieces per channel, every form of the convolution, step ranks up to one whose rows do not fit
    shared memory together, portions shorter than the convolution."""
    cfg = model([(mamba(inner, state, conv, dt_rank), 0), (mamba(inner + 3, state, conv, dt_rank), 40)], width=64, vocab=96)
    check_model(E, cfg, 140, [66, 1, 2, 3, 1, 1, 40], seed=state)


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_token_far_back_is_remembered(E, dtype):
    """States that forget a thousandth of a step's size, and one token whose steps are a thousand times those of the others:
    it shows 600 tokens later, the same after prompts and after decoding."""
    cfg = model([(mamba(inner=48, state=8), 0)], width=64, vocab=90)
    W = K.random_weights(cfg, 5)
    W["l0.mix.A_log"] = K.bf16_round(np.full_like(W["l0.mix.A_log"], np.log(0.001)))
    h = K.rms_norm(W["embed"].astype(np.float64) * cfg["embedding"]["scale"], W["l0.norm1"], 1e-5)
    W["l0.mix.in"][0] = K.bf16_round(14 * h[89] / (h[89] @ h[89]))  # channel 0 sees the token
    W["l0.mix.conv"] = np.eye(1, 4, 3, dtype=np.float32).repeat(48, axis=0)
    W["l0.mix.x"][:6] = 0
    W["l0.mix.x"][0, 0] = 1                                            # and sets everybody's step
    W["l0.mix.dt"] = np.eye(1, 6, 0, dtype=np.float32).repeat(48, axis=0)
    W["l0.mix.dt.b"] = np.full(48, -6, np.float32)
    toks = tokens(cfg, 640, 5) % 89
    other = toks.copy()
    toks[0] = 89
    want = K.forward(cfg, W, toks)
    assert error(K.forward(cfg, W, other)[600:], want[600:]) > 20 * TOL[dtype]
    e = engine(E, cfg, W, dtype, seq_len=640)
    got = portions(e, toks, [64, 64, 64, 1, 2, 200, 200, 1])
    check(got, want, dtype, 10.0 if dtype == "float32" else 1.0)  # some rows are small differences
    assert error(got[600:], K.forward(cfg, W, other)[600:]) > 15 * TOL[dtype]
    e.close()


def test_fast_and_slow_decays_and_large_steps(E):
    """Decays from none to total, on both sides of where their difference from 1 changes its form; step sizes in the linear
    part of the softplus and far below it."""
    cfg = model([(mamba(inner=64, state=16), 0)], width=64, vocab=90)
    W = K.random_weights(cfg, 6)
    W["l0.mix.A_log"] = K.bf16_round(np.linspace(-9, 5, 64 * 16).reshape(64, 16))
    W["l0.mix.dt.b"] = K.bf16_round(np.linspace(-12, 9, 64)[np.random.default_rng(0).permutation(64)])
    check_model(E, cfg, 200, [130, 1, 1, 60], W=W, seed=6, slack=2.0)


@pytest.mark.parametrize("dtype", DTYPES)
def test_convolution_across_portions(E, dtype):
    """A strong oldest tap: what a portion's first tokens take from the ones before it stands out."""
    cfg = model([(mamba(inner=48, conv=5), 0)], width=64, vocab=90)
    W = K.random_weights(cfg, 7)
    W["l0.mix.conv"][:, 0] = K.bf16_round(3 * np.ones(48))
    toks = tokens(cfg, 90, 7)
    want = K.forward(cfg, W, toks)
    for sizes in ([90], [1], [2], [3], [4], [5], [64, 2, 2, 1, 1, 20], [1, 2, 1, 70, 1]):
        e = engine(E, cfg, W, dtype, seq_len=90)
        check(portions(e, toks, sizes), want, dtype)
        e.close()


# ------------------------------------------------------------------ attention

@pytest.mark.parametrize("rot", [dict(rot=12, base=7.0, scaling=False), dict(rot=24, base=40.0, factor=8.0, original=200, fast=16.0, slow=0.5),
                                 dict(rot=20, base=1e6, factor=1.5, original=2048, fast=32.0, slow=1.0), dict(rot=2, base=30.0, factor=2.0),
                                 dict(rot=0, scaling=False), dict(rot=16, base=50.0, original=5, fast=1.0, slow=1.0)], ids=str)
def test_rotations(E, rot):
    """Plain and stretched rotations of all, some and none of the dimensions, and a ramp of zero length."""
    check_model(E, model([(attention(window=0, scale=0.4, **rot), 0)], width=64), 180, [90, 1, 1, 60], seed=4)


@pytest.mark.parametrize("softcap", [0, 0.3, 5.0, 50.0])
def test_score_caps(E, softcap):
    cfg = model([(attention(window=40, scale=1.5, softcap=softcap), 0)], width=64)
    check_model(E, cfg, 120, [70, 1, 2, 40, 1], seed=8)


@pytest.mark.parametrize("heads,kv_heads,dim,rot,window", [(8, 8, 64, 16, 30), (8, 2, 64, 64, 150), (32, 8, 32, 8, 0), (33, 1, 16, 4, 100), (20, 4, 128, 32, 70),
                                                           (4, 4, 200, 40, 130), (3, 1, 512, 2, 64), (2, 1, 600, 30, 90), (12, 6, 10, 10, 65), (1, 1, 1, 0, 2)])
def test_attention_instantiations(E, heads, kv_heads, dim, rot, window):
    """Every tensor-core tile shape, groups of many and of one head, several key splits, a head too wide for the tensor cores,
    against the CUDA-core kernel and the oracle."""
    cfg = model([(attention(heads, kv_heads, dim, rot, window, softcap=4.0, scale=0.7 * dim ** -0.5), 32)], width=128, vocab=64)
    W, toks = K.random_weights(cfg, heads), tokens(cfg, 230, heads)
    want = K.forward(cfg, W, toks)
    for flags in (0, E.FLAG_LATENT_CUDA_CORES):
        e = engine(E, cfg, W, "bfloat16", flags=flags)
        check(portions(e, toks, [130, 1, 1, 1, 64, 30, 1]), want, "bfloat16")
        e.close()


def needle_model(window, kv_heads=2):
    """One attention layer in which every query looks for one token: queries are a bias along that token's key, in the
    dimensions that do not turn, so the token stands out by several units of score wherever it is visible."""
    cfg = model([(attention(heads=4, kv_heads=kv_heads, dim=36, rot=4, window=window, scale=1.0, softcap=25.0, scaling=False), 0)], width=64, vocab=80, logit=1.0)
    W = K.random_weights(cfg, 12)
    h = K.rms_norm(W["embed"].astype(np.float64) * cfg["embedding"]["scale"], W["l0.norm1"], 1e-5)
    k = (h @ W["l0.mix.k"].T.astype(np.float64)).reshape(80, kv_heads, 36)
    W["l0.mix.q"] *= 0
    b = np.zeros((4, 36))
    for a in range(4):
        keys = k[:, a // (4 // kv_heads), 4:]
        away = keys[79] - keys[:79].mean(axis=0)
        b[a, 4:] = 10.0 * away / (away @ away)
    W["l0.mix.q.b"] = K.bf16_round(b.reshape(-1))
    W["l0.mix.o"] = K.bf16_round(W["l0.mix.o"] * 4)
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
        want = K.forward(cfg, W, toks)
        toks_without = toks.copy()
        toks_without[at] = 0
        without = K.forward(cfg, W, toks_without)
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
    cfg, W = needle_model(0, kv_heads=1)
    toks = np.random.default_rng(0).integers(0, 79, n).astype(np.int32)
    toks[3] = 79
    want = K.forward(cfg, W, toks)
    e = engine(E, cfg, W, dtype, seq_len=seq_len)
    e.extend(toks[:n - 60], 0)
    check(e.extend(toks[n - 60:n - 10], n - 60, range(50)), want[n - 60:n - 10], dtype)
    check(np.stack([e.step_logits(int(toks[p]), p) for p in range(n - 10, n)]), want[n - 10:], dtype)
    e.close()


# ------------------------------------------------------------------ order of layers, sizes, constants

@pytest.mark.parametrize("loop", [(0, 0, 1), (0, 1, 1), (0, 3, 2), (1, 2, 5), (2, 3, 3), (0, 2, 4)], ids=str)
def test_loops(E, loop):
    """No loop, one pass, loops at the start, in the middle and at the end, around each mixer: every pass has its own state."""
    cfg = model([(mamba(inner=40), 0), (attention(window=12), 0), (mamba(inner=24, conv=3), 56)], width=64, loop=loop)
    check_model(E, cfg, 80, [41, 1, 2, 30, 1], seed=sum(loop))


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_loop_is_its_layers_written_out(E, dtype):
    """All kinds of mixers in one model: two passes of a loop without vectors of its own give what the same layers give
    when they are listed twice."""
    from lighterpp_b200.formats import LatentMixer, Layer, LayeredConfig, Loop, MambaMixer, Rotation, SharedKvMixer
    from lighterpp_b200.models import PRECISIONS
    rot = Rotation(8, 300.0)
    kinds = [Layer(MambaMixer(56, 12, 4, 5)), Layer(LatentMixer(2, 16, 8, 12, 24, 0.2, rot, 9), 40, "gelu_tanh"),
             Layer(SharedKvMixer(4, 2, 20, 0.3, rot, 11, 3.0, True, True), 48), Layer(SharedKvMixer(2, 2, 16, 0.3, rot), 0)]
    D, V = 64, 70

    def shapes(y):
        m = y.mixer
        s = {"rms_att": (D,)}
        if isinstance(m, MambaMixer):
            s.update(scan_in=(2 * m.inner, D), scan_conv=(m.inner, m.conv), scan_conv_b=(m.inner,), scan_low=(m.dt_rank + 2 * m.state, m.inner),
                     scan_dt=(m.inner, m.dt_rank), scan_dt_b=(m.inner,), scan_a_log=(m.inner, m.state), scan_d=(m.inner,), wo=(D, m.inner))
        elif isinstance(m, LatentMixer):
            s.update(lat_q=(m.heads * (m.dim + m.rot_dim), D), lat_dkv=(m.kv_rank + m.rot_dim, D), lat_norm=(m.kv_rank,), lat_uk=(m.heads * m.dim, m.kv_rank),
                     lat_uv=(m.heads * m.vdim, m.kv_rank), lat_g=(m.heads, D), wo=(D, m.heads * m.vdim))
        else:
            s.update(wq=(m.heads * m.dim, D), wk=(m.kv_heads * m.dim, D), wo=(D, m.heads * m.dim))
            if m.bias:
                s.update(wq_b=(m.heads * m.dim,), wk_b=(m.kv_heads * m.dim,), wo_b=(D,))
            if m.gate:
                s.update(wg=(m.heads * m.dim, D))
        if y.ff:
            s.update(rms_ffn=(D,), w1=(y.ff, D), w3=(y.ff, D), w2=(D, y.ff))
        return s
    rng = np.random.default_rng(3)
    draw = lambda shape: (rng.standard_normal(shape) / (np.sqrt(shape[1]) if len(shape) > 1 else 4)).astype(np.float32)
    layer_w = [{n: draw(s) for n, s in shapes(y).items()} for y in kinds]
    common = {"tok_emb": draw((V, D)) * 4, "rms_final": np.ones(D, np.float32)}
    toks = np.random.default_rng(4).integers(0, V, 90)
    got = []
    for cfg, order in ((LayeredConfig(D, V, 90, kinds, loop=Loop(0, 4, 2)), range(4)), (LayeredConfig(D, V, 90, kinds * 2), [0, 1, 2, 3] * 2)):
        e = E.Engine(cfg, *PRECISIONS[dtype])
        for n, a in common.items():
            e.upload(n, a)
        if cfg.loop:
            e.upload("loop_step", np.zeros((2, D), np.float32))
        for l, k in enumerate(order):
            for n, a in layer_w[k].items():
                e.upload(n, a, l)
        e.finalize()
        got.append(portions(e, toks, [66, 1, 1, 22]))
        e.close()
    assert np.array_equal(got[0], got[1]) and np.abs(got[0]).max() > 0.1


@pytest.mark.parametrize("dtype", DTYPES)
def test_sizes_off_every_grid(E, dtype):
    check_model(E, ODD, 140, [70, 1, 2, 3, 40, 1], seed=2, dtypes=[dtype], slack=1.5)


@pytest.mark.parametrize("width", [2056, 4104, 8200])
def test_wide_rows(E, width):
    """Norms of rows that no longer fit the registers of one pass."""
    cfg = model([(mamba(inner=32), 0), (attention(heads=2, kv_heads=1, dim=8, rot=4), 24)], width=width, vocab=33, loop=(0, 1, 2))
    check_model(E, cfg, 9, [5, 1], seed=7)


@pytest.mark.parametrize("emb,logit,eps", [(1.0, 1.0, 1e-5), (40.0, 0.01, 1e-6), (0.02, 30.0, 0.5)])
def test_scales_and_epsilon(E, emb, logit, eps):
    cfg = model([(mamba(), 0), (attention(), 40)], eps=eps, emb=emb, logit=logit, loop=(1, 2, 2))
    W = K.random_weights(cfg, 9)
    W["embed"] = K.bf16_round(np.random.default_rng(1).standard_normal(W["embed"].shape))  # of unit size before the factor
    check_model(E, cfg, 40, [30, 1], W=W)


@pytest.mark.parametrize("flags", ["FLAG_GEMV_LDG", "FLAG_NO_GRAPH", "FLAG_NO_PDL", "FLAG_NO_PREFILL_GEMM"])
def test_engine_flags(E, small, flags):
    W, toks, want = small
    for dtype in DTYPES:
        e = engine(E, SMALL, W, dtype, flags=getattr(E, flags))
        check(portions(e, toks[:60], [40, 1]), want[:60], dtype)
        e.close()


def test_many_rows_for_few_multiprocessors(E):
    """More row pairs per warp of the input product than its epilogue holds together."""
    cfg = model([(mamba(inner=10000, state=4, dt_rank=4), 0), (attention(heads=150, kv_heads=75, dim=64, rot=8), 0)], width=64, vocab=40)
    check_model(E, cfg, 12, [6, 1], seed=3)


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
    lg = K.forward(SMALL, W, prompt + out)
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
    assert len(s.generate(prompt[:1], 5)) == 5
    e.close()


def test_programs(E, small, tmp_path):
    """The command line and the trace replayer on a model folder."""
    W, toks, want = small
    folder = str(tmp_path / "model")
    K.write_model(folder, SMALL, W)
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
        for i, (a, b) in enumerate(zip(cuts, cuts[1:])):
            if i != 2:
                check(np.fromfile(out / f"{i}.f32", dtype="<f4").reshape(2, -1), want[[b - 1, a]], dtype)
        check(np.fromfile(out / "9.f32", dtype="<f4"), want[6], dtype)


def test_incomplete_and_wrong_descriptions_are_refused(E, small):
    W, _, _ = small
    e = E.Engine(configured(SMALL, 16), "bf16", "f16")
    with pytest.raises(E.LppError, match="was never uploaded"):
        e.finalize()
    for name, layer in (("wq", 0), ("scan_in", 1), ("lat_q", 1), ("wv", 1), ("norm1_b", 0)):
        with pytest.raises(E.LppError):
            e.upload(name, np.zeros((4, 4), np.float32), layer)
    with pytest.raises(E.LppError, match="keeps no latents"):
        E._check(e.lib.lpp_latent_read(e.h, 0, 0, np.zeros(8, np.float32).ctypes.data_as(E.C.POINTER(E.C.c_float))), "lpp_latent_read")
    e.close()
    for change in (lambda c: setattr(c.layers[1].mixer, "kv_heads", 3), lambda c: setattr(c.layers[1].mixer.rotation, "dims", 26),
                   lambda c: setattr(c.layers[1].mixer.rotation, "dims", 7), lambda c: setattr(c.layers[0].mixer, "state", 2000),
                   lambda c: setattr(c.layers[0].mixer, "conv", 0), lambda c: setattr(c.loop, "stop", 6), lambda c: setattr(c.loop, "times", 0)):
        c = configured(SMALL, 16)
        change(c)
        with pytest.raises(E.LppError):
            E.Engine(c, "bf16", "f16")
