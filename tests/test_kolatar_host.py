"""Kolatar on the CPU: the oracle's own mechanisms against hand-worked cases, the configuration and weight readers, and that
faults of the kind the GPU suite is there for move the logits far beyond its tolerances."""
import json
import math

import numpy as np
import pytest

from kolatar_util import ODD, SMALL, attention, mamba, model
from lighterpp_b200 import models
from lighterpp_b200.formats import MambaMixer, SharedKvMixer
from oracle import kolatar as K
from rutenex_util import error, tokens


# ------------------------------------------------------------------ mechanisms by hand

def test_convolution_by_hand():
    x = np.array([[1.0, 10.0], [2.0, 20.0], [3.0, 30.0]])
    w = np.array([[0.5, 2.0, 1.0], [0.0, -1.0, 3.0]])  # last column: the current token
    y = K.causal_conv(x, w, np.array([100.0, 0.0]))
    assert y[:, 0].tolist() == [101.0, 100 + 2 + 2 * 1, 100 + 3 + 2 * 2 + 0.5 * 1]
    assert y[:, 1].tolist() == [30.0, 60 - 10, 90 - 20]


def test_scan_by_hand():
    # one channel, two elements; exp(dt A) = 1/2 and 1/4 at dt = 1
    A = -np.array([[math.log(2), math.log(4)]])
    x, dt = np.array([[3.0], [5.0]]), np.array([[1.0], [1.0]])
    B, C = np.array([[1.0, 2.0], [1.0, 0.0]]), np.array([[1.0, 1.0], [1.0, 10.0]])
    y = K.selective_scan(x, dt, A, B, C, np.array([0.1]))
    # states: (3, 6), then (3/2 + 5, 6/4)
    assert np.allclose(y[:, 0], [9 + 0.3, 6.5 + 15 + 0.5])
    # a step of size zero leaves the state alone
    s = np.array([[7.0, 8.0]])
    K.selective_scan(np.array([[1.0]]), np.zeros((1, 1)), A, B[:1], C[:1], np.zeros(1), s)
    assert s.tolist() == [[7.0, 8.0]]


def test_softplus_and_silu():
    assert np.allclose(K.softplus(np.array([0.0, 100.0, -100.0])), [math.log(2), 100.0, math.exp(-100)])
    assert np.allclose(K.silu(np.array([0.0, 2.0])), [0.0, 2 / (1 + math.exp(-2))])


def test_capped_scores():
    s = np.array([0.0, 0.01, 3.0, 1e6, -1e6])
    assert np.allclose(K.capped(s, 2.0), [0.0, 0.01, 2 * math.tanh(1.5), 2.0, -2.0], atol=1e-6)
    assert np.array_equal(K.capped(s, None), s)


def test_values_are_the_unrotated_keys():
    """One visible key only (window 1): the result is that key's projection before rotation, times the gate."""
    m = attention(heads=2, kv_heads=1, dim=4, rot=4, window=1)["mixer"]
    rng = np.random.default_rng(0)
    W = {"q": rng.standard_normal((8, 6)), "q.b": rng.standard_normal(8), "k": rng.standard_normal((4, 6)), "k.b": rng.standard_normal(4),
         "g": rng.standard_normal((8, 6)), "o": np.eye(8), "o.b": np.zeros(8)}
    h = rng.standard_normal((5, 6))
    k = h @ W["k"].T + W["k.b"]
    assert np.allclose(K.gated_attention(h, W, "", m), np.concatenate([k, k], axis=1) * K.sigmoid(h @ W["g"].T))


def test_order_of_layers():
    cfg = model([(mamba(), 0)] * 4, loop=(1, 3, 2))
    assert K.layer_order(cfg) == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (3, None)]
    assert K.layer_order(model([(mamba(), 0)] * 2, loop=(0, 1, 1))) == [(0, 0), (1, None)]


# ------------------------------------------------------------------ readers

def test_configuration_reads_every_size_and_constant():
    c = models.ARCHITECTURES["Kolatar"].configure(ODD, 77)
    assert (c.dim, c.vocab_size, c.seq_len, c.n_layers, c.norm, c.norm_eps, c.emb_scale, c.logit_scale) == (71, 131, 77, 6, "rms", 0.02, 0.3, 11.0)
    assert (c.loop.start, c.loop.stop, c.loop.times) == (0, 2, 3)
    for y, want in zip(c.layers, ODD["layers"]):
        w, m = want["mixer"], y.mixer
        assert y.ff == (want["mlp"]["ff"] if want["mlp"] else 0) and y.act == "silu"
        if want["type"] == "mamba1":
            assert isinstance(m, MambaMixer) and vars(m) == w
            continue
        assert isinstance(m, SharedKvMixer) and m.bias and m.gate
        assert (m.heads, m.kv_heads, m.dim, m.scale, m.window, m.softcap) == (
            w["heads"], w["kv_heads"], w["dim"], w["scale"], w["mask"]["size"], w.get("softcap", 0.0))
        assert (m.rotation.dims, m.rotation.base) == (w["rot"]["dims"], w["rot"]["base"])
        assert vars(m.rotation.yarn) == {k: float(w["rot"]["scaling"][k]) for k in ("factor", "original", "fast", "slow")}
    plain = models.ARCHITECTURES["Kolatar"].configure(model([(attention(window=0, scaling=False, softcap=0), 8)]), 8)
    assert plain.layers[0].mixer.window == 0 and plain.layers[0].mixer.rotation.yarn is None and plain.layers[0].mixer.softcap == 0.0
    for cfg in (ODD, SMALL):
        assert {n: s for _, _, n, s in models.kolatar_tensors(models.kolatar_config(cfg, 8))} == K.tensor_shapes(cfg)


def test_unknown_designs_are_refused():
    for change in (lambda c: c["layers"][1].update(type="mamba9"), lambda c: c["layers"][0]["mlp"].update(kind="sparse"),
                   lambda c: c["layers"][0]["mixer"].update(vdim=7)):
        bad = json.loads(json.dumps(ODD))
        change(bad)
        with pytest.raises(ValueError):
            models.ARCHITECTURES["Kolatar"].configure(bad, 8)


# ------------------------------------------------------------------ faults show

EDGE = model([(mamba(), 0), (attention(window=11, scale=0.9, softcap=2.0), 64), (mamba(inner=64, state=20), 0), (attention(window=6, scale=0.9, heads=6, kv_heads=3), 0)],
             width=64, vocab=97, loop=(0, 3, 2))


def run_with(monkeypatch, cfg=EDGE, weights=None, **patches):
    W = K.random_weights(EDGE, 8)
    W.update(weights(W) if weights else {})
    for name, fn in patches.items():
        monkeypatch.setattr(K, name, fn)
    return K.forward(cfg, W, tokens(EDGE, 40))


def changed(path, value):
    cfg = json.loads(json.dumps(EDGE))
    at = cfg
    for key in path[:-1]:
        at = at[key]
    at[path[-1]] = value
    return cfg


def zeroed(part):
    return lambda W: {k: v * 0 for k, v in W.items() if part in k}


CONFIG_FAULTS = {"window one longer": (["layers", 1, "mixer", "mask", "size"], 12), "window one shorter": (["layers", 1, "mixer", "mask", "size"], 10),
                 "no cap": (["layers", 1, "mixer", "softcap"], None), "no stretching": (["layers", 1, "mixer", "rot", "scaling"], None),
                 "embedding not scaled": (["embedding", "scale"], 1.0), "logits not scaled": (["logit_scale"], 1.0),
                 "one pass too few": (["loop", "times"], 1), "loop one layer longer": (["loop", "stop"], 4)}
WEIGHT_FAULTS = {"no query bias": ".q.b", "no key bias": ".k.b", "no output bias": ".o.b", "no loop vector": "loop.step", "no convolution bias": "conv.b",
                 "no step bias": "dt.b", "no skip": "mix.D", "decay without exp(A_log)": "A_log", "gate at one half": ".mix.g"}


@pytest.mark.parametrize("fault", sorted(CONFIG_FAULTS))
def test_configuration_faults_are_visible_in_the_logits(fault, monkeypatch):
    assert error(run_with(monkeypatch, changed(*CONFIG_FAULTS[fault])), run_with(monkeypatch)) > 0.03


@pytest.mark.parametrize("fault", sorted(WEIGHT_FAULTS))
def test_weight_faults_are_visible_in_the_logits(fault, monkeypatch):
    assert error(run_with(monkeypatch, weights=zeroed(WEIGHT_FAULTS[fault])), run_with(monkeypatch)) > 0.03


def scan_cut_every_eight(x, dt, A, B, C, D, state=None):
    return np.concatenate([K_scan(x[i:i + 8], dt[i:i + 8], A, B[i:i + 8], C[i:i + 8], D) for i in range(0, len(x), 8)])


def conv_cut_every_eight(x, w, b):
    return np.concatenate([K_conv(x[i:i + 8], w, b) for i in range(0, len(x), 8)])


def rotated_values(h, W, pre, m, positions=None):
    n, G, d = h.shape[0], m["kv_heads"], m["dim"]
    pos = np.arange(n)
    k = K.rotate((h @ W[pre + "k"].T + W[pre + "k.b"]).reshape(n, G, d), pos, m["rot"])
    q = K.rotate((h @ W[pre + "q"].T + W[pre + "q.b"]).reshape(n, m["heads"], d), pos, m["rot"])
    vis = K.window_mask(n, m["mask"]["size"])
    out = [K.softmax_attend(K.capped(q[:, a] @ k[:, a // (m["heads"] // G)].T * m["scale"], m["softcap"]), vis, k[:, a // (m["heads"] // G)])
           for a in range(m["heads"])]
    return (np.concatenate(out, axis=1) * K.sigmoid(h @ W[pre + "g"].T)) @ W[pre + "o"].T + W[pre + "o.b"]


K_scan, K_conv = K.selective_scan, K.causal_conv
CODE_FAULTS = {
    "state lost between portions": dict(selective_scan=scan_cut_every_eight),
    "convolution inputs lost between portions": dict(causal_conv=conv_cut_every_eight),
    "taps reversed": dict(causal_conv=lambda x, w, b: K_conv(x, w[:, ::-1], b)),
    "convolution one token late": dict(causal_conv=lambda x, w, b: K_conv(np.concatenate([x[:1] * 0, x[:-1]]), w, b)),
    "values rotated": dict(gated_attention=rotated_values),
    "relu for silu": dict(silu=lambda z: np.maximum(z, 0)),
    "norm by the sum of squares": dict(rms_norm=lambda x, w, eps: x / np.sqrt((x * x).sum(axis=-1, keepdims=True) + eps) * w),
}


@pytest.mark.parametrize("fault", sorted(CODE_FAULTS))
def test_code_faults_are_visible_in_the_logits(fault, monkeypatch):
    good = run_with(monkeypatch)
    assert error(run_with(monkeypatch, **CODE_FAULTS[fault]), good) > 0.03
