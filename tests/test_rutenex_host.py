"""Rutenex on the CPU: the oracle's own mechanisms against hand-worked cases, the configuration and weight readers, the
session's bookkeeping, and that the edge tests of the GPU suite can see the faults they are there for."""
import json
import math
import os

import numpy as np
import pytest

from lighterpp_b200 import models
from lighterpp_b200.formats import read_safetensors
from lighterpp_b200.session import Session
from oracle import rutenex as R
from rutenex_util import ODD, SMALL, error, mixer, model, tokens


def test_layer_norm_and_rms_norm_by_hand():
    x = np.array([[1.0, 3.0]])
    assert np.allclose(R.layer_norm(x, np.array([2.0, 2.0]), np.array([0.5, -0.5]), 3.0), [[-1 + 0.5, 1 - 0.5]])  # (x - 2) / sqrt(1 + 3)
    assert np.allclose(R.rms_norm(x, np.array([1.0, 2.0]), 4.0), [[1 / 3, 6 / 3]])                               # x / sqrt(5 + 4)


def test_rotation_by_hand():
    rot = {"base": 4.0, "dims": 4}
    assert np.allclose(R.rotation_frequencies(rot), [1.0, 0.5])
    x = np.array([[1.0, 0.0, 0.0, 2.0, 7.0, 8.0]])
    y = R.rotate(x, np.array([3]), rot)
    assert np.allclose(y[0], [math.cos(3), math.sin(3), -2 * math.sin(1.5), 2 * math.cos(1.5), 7.0, 8.0])  # the last two do not turn
    # scores depend on the distance only
    rng = np.random.default_rng(0)
    q, k = rng.standard_normal((1, 4)), rng.standard_normal((1, 4))
    dots = [float((R.rotate(q, np.array([p + 5]), rot) @ R.rotate(k, np.array([p]), rot).T)[0, 0]) for p in (0, 9, 40)]
    assert np.allclose(dots, dots[0])


def test_yarn_blend_by_hand():
    # dims 8, base 10: border(t) = 8 ln(100 / (2 pi t)) / (2 ln 10); fast 4 -> 2.4 -> 2, slow 1 -> 4.8 -> 5
    rot = {"base": 10.0, "dims": 8, "scaling": {"factor": 4.0, "original": 100, "fast": 4.0, "slow": 1.0}}
    plain = [10 ** (-i / 4) for i in range(4)]
    want = [plain[0], plain[1], plain[2], plain[3] * (1 - 1 / 3) + plain[3] / 4 / 3]
    assert np.allclose(R.rotation_frequencies(rot), want)
    assert math.isclose(R.rotation_magnitude(rot), 0.1 * math.log(4) + 1)
    y = R.rotate(np.array([[1.0] + [0.0] * 8]), np.array([0]), rot)
    assert math.isclose(y[0, 0], R.rotation_magnitude(rot))


def test_window_mask_by_hand():
    m = R.window_mask(5, 2)
    assert m.astype(int).tolist() == [[1, 0, 0, 0, 0], [1, 1, 0, 0, 0], [0, 1, 1, 0, 0], [0, 0, 1, 1, 0], [0, 0, 0, 1, 1]]
    assert R.window_mask(4, None).sum() == 10


def test_gelu_form():
    z = np.array([-3.0, -0.5, 0.0, 0.7, 2.0])
    exact = 0.5 * z * (1 + np.array([math.erf(v / math.sqrt(2)) for v in z]))
    assert np.abs(R.gelu_tanh(z) - exact).max() < 1e-3 and R.gelu_tanh(z)[2] == 0.0


def test_configuration_reads_every_size_and_constant():
    c = models.ARCHITECTURES["Rutenex"].configure(ODD, 77)
    assert (c.dim, c.vocab_size, c.seq_len, c.n_layers, c.norm, c.norm_eps) == (71, 131, 77, 3, "layer", 0.02)
    for y, want in zip(c.layers, ODD["layers"]):
        m, w = y.mixer, want["mixer"]
        assert (m.heads, m.dim, m.rot_dim, m.vdim, m.kv_rank, m.window, m.scale) == (
            w["heads"], w["dim"], w["rot_dim"], w["vdim"], w["kv_rank"], w["mask"]["size"], w["scale"])
        assert (m.rotation.dims, m.rotation.base) == (w["rot"]["dims"], w["rot"]["base"])
        s = w["rot"]["scaling"]
        assert vars(m.rotation.yarn) == {k: float(s[k]) for k in ("factor", "original", "fast", "slow")}
        assert y.ff == (want["mlp"]["ff"] if want["mlp"] else 0) and y.act == "gelu_tanh"
    plain = models.ARCHITECTURES["Rutenex"].configure(model([(mixer(window=0, scaling=False), 8)]), 8)
    assert plain.layers[0].mixer.window == 0 and plain.layers[0].mixer.rotation.yarn is None
    assert {n: s for _, _, n, s in models.rutenex_tensors(c)} == R.tensor_shapes(ODD)


def test_unknown_designs_are_refused(tmp_path):
    bad = json.loads(json.dumps(SMALL))
    bad["layers"][1]["type"] = "something_else"
    with pytest.raises(ValueError, match="something_else"):
        models.ARCHITECTURES["Rutenex"].configure(bad, 8)
    with open(tmp_path / "config.json", "w") as f:
        json.dump({**SMALL, "architecture": "Nobody"}, f)
    with pytest.raises(ValueError, match="Nobody"):
        models.read_config(str(tmp_path), 8)


def test_safetensors_reader(tmp_path):
    W = R.random_weights(SMALL, 5)
    R.write_model(str(tmp_path), SMALL, W)
    T = read_safetensors(os.path.join(tmp_path, "model.safetensors"))
    assert set(T) == set(W)
    for n, a in W.items():
        assert T[n].dtype == np.uint16 and T[n].shape == a.shape
        assert np.array_equal((T[n].astype(np.uint32) << 16).view(np.float32), a)
    with open(tmp_path / "cut.safetensors", "wb") as f:
        f.write(open(tmp_path / "model.safetensors", "rb").read()[:-2])
    with pytest.raises(ValueError, match="does not fit"):
        read_safetensors(str(tmp_path / "cut.safetensors"))


class FakeEngine:
    """Records what a session asks for; logits are the token's index."""

    def __init__(self, seq_len=10):
        self.cfg = type("C", (), {"seq_len": seq_len, "vocab_size": 3})()
        self.calls = []

    def extend(self, toks, start, want):
        self.calls.append((list(toks), start, list(want)))
        return np.array([[w] * 3 for w in want], dtype=np.float32).reshape(len(want), 3)

    def decode(self, first, pos, n, *a):
        self.calls.append(("decode", first, pos, n))
        return np.arange(n), 0.0


def test_session_positions_owners_and_capacity():
    e = FakeEngine()
    s = Session(e)
    assert s.extend("a", [1, 2, 3], [2, 0, 2])[:, 0].tolist() == [2, 0, 2]
    s.extend("a", [4])
    assert e.calls == [([1, 2, 3], 0, [0, 2]), ([4], 3, [])]
    with pytest.raises(RuntimeError, match="one sequence"):
        s.extend("b", [1])
    with pytest.raises(ValueError, match="exceed"):
        s.extend("a", [0] * 7)
    s.end("b")  # not the owner: nothing happens
    assert s.owner == "a" and s.length == 4
    s.end("a")
    s.extend("b", [9, 9])
    assert e.calls[-1] == ([9, 9], 0, [])
    s.end("b")
    assert s.generate([5, 6, 7], 4) == [0, 1, 2, 3] and e.calls[-2:] == [([5, 6], 0, []), ("decode", 7, 2, 4)]
    assert s.generate([5], 2) == [0, 1] and s.owner is None
    with pytest.raises(ValueError):
        s.generate([1] * 8, 4)


EDGE = model([(mixer(window=11, scale=1.5), 64), (mixer(window=6, scale=1.5), 0)], width=64, vocab=97)


@pytest.mark.parametrize("fault", ["window +1", "window -1", "no gate", "no yarn", "magnitude", "key not rotated", "latent not normed",
                                   "silu", "mean kept", "no bias"])
def test_faults_are_visible_in_the_logits(fault, monkeypatch):
    """A fault planted in the oracle moves the logits far beyond what the GPU tests tolerate (1e-2 in BF16)."""
    W, toks = R.random_weights(EDGE, 8), tokens(EDGE, 40)
    good = R.forward(EDGE, W, toks)
    cfg = json.loads(json.dumps(EDGE))
    m = cfg["layers"][0]["mixer"]
    W2 = dict(W)
    if fault.startswith("window"):
        m["mask"]["size"] += int(fault.split()[1])
    elif fault == "no gate":
        W2 = {k: (v * 0 if k == "l0.mix.g" else v) for k, v in W.items()}
    elif fault == "no yarn":
        del m["rot"]["scaling"]
    elif fault == "magnitude":
        monkeypatch.setattr(R, "rotation_magnitude", lambda rot: 1.0)
    elif fault == "key not rotated":
        monkeypatch.setattr(R, "latent_split", lambda h, W, pre, m, eps, pos: (
            R.rms_norm((h @ W[pre + "dkv"].T)[:, :m["kv_rank"]], W[pre + "dkv.norm"], eps), (h @ W[pre + "dkv"].T)[:, m["kv_rank"]:]))
    elif fault == "latent not normed":
        monkeypatch.setattr(R, "rms_norm", lambda x, w, eps: x * w)
    elif fault == "silu":
        monkeypatch.setattr(R, "gelu_tanh", lambda z: z * R.sigmoid(z))
    elif fault == "mean kept":
        monkeypatch.setattr(R, "layer_norm", lambda x, w, b, eps: x / np.sqrt((x * x).mean(-1, keepdims=True) + eps) * w + b)
    elif fault == "no bias":
        W2 = {k: (v * 0 if k.endswith(".b") else v) for k, v in W.items()}
    assert error(R.forward(cfg, W2, toks), good) > 0.05
