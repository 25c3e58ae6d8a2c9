"""Plain, slow numpy statement of the Kolatar decoder (selective-scan layers, attention whose values are its unrotated keys
under a sliding window with capped scores and an element-wise output gate, a group of layers that runs several times),
one function per mechanism, used only to check the CUDA engine.

Everything runs in one floating type (``dtype``, double by default) and without a cache: a whole sequence goes through a
layer at once; the scan walks the tokens one by one, the convolution is written out tap by tap, attention looks visible
keys up in a boolean matrix.  Nothing here is shared with the package under test; mechanisms that the Rutenex statement
already has (norm, rotation, mask) come from there.

A model is ``cfg`` (the decoded config.json) plus ``W``, a dict of numpy arrays by tensor name.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import numpy as np

from oracle.rutenex import bf16_round, rms_norm, rotate, sigmoid, softmax_attend, window_mask, write_model  # noqa: F401


# ------------------------------------------------------------------ mechanisms

def silu(z: np.ndarray) -> np.ndarray:
    return z * sigmoid(z)


def softplus(z: np.ndarray) -> np.ndarray:
    return np.maximum(z, 0) + np.log1p(np.exp(-np.abs(z)))


def causal_conv(x: np.ndarray, weight: np.ndarray, bias: np.ndarray) -> np.ndarray:
    """x [tokens, channels], weight [channels, taps]: the last tap is the current token, zeros before the first."""
    taps = weight.shape[1]
    out = np.tile(bias, (x.shape[0], 1)).astype(x.dtype)
    for t in range(x.shape[0]):
        for back in range(min(taps, t + 1)):
            out[t] += weight[:, taps - 1 - back] * x[t - back]
    return out


def selective_scan(x: np.ndarray, dt: np.ndarray, A: np.ndarray, B: np.ndarray, C: np.ndarray, D: np.ndarray,
                   state: Optional[np.ndarray] = None) -> np.ndarray:
    """x, dt [tokens, channels]; A [channels, n]; B, C [tokens, n].  ``state`` [channels, n] is updated in place."""
    s = np.zeros_like(A) if state is None else state
    y = np.empty_like(x)
    for t in range(x.shape[0]):
        s[...] = np.exp(dt[t][:, None] * A) * s + (dt[t] * x[t])[:, None] * B[t][None, :]
        y[t] = s @ C[t] + D * x[t]
    return y


def mamba_mixer(h: np.ndarray, W: Dict[str, np.ndarray], pre: str, m: dict) -> np.ndarray:
    inner, n, r = m["inner"], m["state"], m["dt_rank"]
    xz = h @ W[pre + "in"].T
    x = silu(causal_conv(xz[:, :inner], W[pre + "conv"], W[pre + "conv.b"]))
    low = x @ W[pre + "x"].T
    dt = softplus(low[:, :r] @ W[pre + "dt"].T + W[pre + "dt.b"])
    y = selective_scan(x, dt, -np.exp(W[pre + "A_log"]), low[:, r:r + n], low[:, r + n:], W[pre + "D"])
    return (y * silu(xz[:, inner:])) @ W[pre + "o"].T


def capped(scores: np.ndarray, cap: Optional[float]) -> np.ndarray:
    return cap * np.tanh(scores / cap) if cap else scores


def gated_attention(h: np.ndarray, W: Dict[str, np.ndarray], pre: str, m: dict, positions: Optional[np.ndarray] = None) -> np.ndarray:
    n = h.shape[0]
    pos = np.arange(n) if positions is None else positions
    H, G, d = m["heads"], m["kv_heads"], m["dim"]
    q = (h @ W[pre + "q"].T + W[pre + "q.b"]).reshape(n, H, d)
    k = (h @ W[pre + "k"].T + W[pre + "k.b"]).reshape(n, G, d)
    q_turned, k_turned = rotate(q, pos, m["rot"]), rotate(k, pos, m["rot"])
    vis = window_mask(n, (m.get("mask") or {}).get("size"))
    heads = []
    for a in range(H):
        b = a // (H // G)
        s = capped((q_turned[:, a] @ k_turned[:, b].T) * h.dtype.type(m["scale"]), m.get("softcap"))
        heads.append(softmax_attend(s, vis, k[:, b]))
    return (np.concatenate(heads, axis=1) * sigmoid(h @ W[pre + "g"].T)) @ W[pre + "o"].T + W[pre + "o.b"]


def dense_feed_forward(h: np.ndarray, W: Dict[str, np.ndarray], pre: str) -> np.ndarray:
    return (silu(h @ W[pre + "gate"].T) * (h @ W[pre + "up"].T)) @ W[pre + "down"].T


def layer_order(cfg: dict) -> list:
    """(layer, pass or None) in the order of execution; the pass number marks the first layer of a pass only."""
    lo, hi, times = cfg["loop"]["start"], cfg["loop"]["stop"], cfg["loop"]["times"]
    order = [(i, None) for i in range(lo)]
    for t in range(times):
        order += [(i, t if i == lo else None) for i in range(lo, hi)]
    return order + [(i, None) for i in range(hi, len(cfg["layers"]))]


# ------------------------------------------------------------------ the model

def forward(cfg: dict, W: Dict[str, np.ndarray], tokens, dtype=np.float64, trace: Optional[List[np.ndarray]] = None) -> np.ndarray:
    """Logits [tokens, vocab] of one sequence; ``trace`` collects the residual stream after every layer run."""
    W = {k: np.asarray(v, dtype=dtype) for k, v in W.items()}
    eps = cfg["norm"]["eps"]
    x = W["embed"][np.asarray(tokens)] * dtype(cfg["embedding"]["scale"])
    for i, begins in layer_order(cfg):
        layer, p = cfg["layers"][i], f"l{i}."
        if begins is not None:
            x = x + W["loop.step"][begins]
        h = rms_norm(x, W[p + "norm1"], eps)
        if layer["type"] == "mamba1":
            x = x + mamba_mixer(h, W, p + "mix.", layer["mixer"])
        elif layer["type"] == "attention":
            x = x + gated_attention(h, W, p + "mix.", layer["mixer"])
        else:
            raise ValueError(layer["type"])
        if layer.get("mlp"):
            if layer["mlp"]["kind"] != "dense":
                raise ValueError(layer["mlp"]["kind"])
            x = x + dense_feed_forward(rms_norm(x, W[p + "norm2"], eps), W, p + "mlp.")
        if trace is not None:
            trace.append(x.copy())
    return rms_norm(x, W["final.norm"], eps) @ W["head"].T * dtype(cfg["logit_scale"])


# ------------------------------------------------------------------ random models

def tensor_shapes(cfg: dict) -> Dict[str, tuple]:
    D, V = cfg["width"], cfg["vocab"]
    s = {"embed": (V, D), "loop.step": (cfg["loop"]["times"], D)}
    for i, layer in enumerate(cfg["layers"]):
        m, p = layer["mixer"], f"l{i}."
        s[p + "norm1"] = (D,)
        if layer["type"] == "mamba1":
            E, N, R = m["inner"], m["state"], m["dt_rank"]
            s.update({p + "mix.in": (2 * E, D), p + "mix.conv": (E, m["conv"]), p + "mix.conv.b": (E,), p + "mix.x": (R + 2 * N, E),
                      p + "mix.dt": (E, R), p + "mix.dt.b": (E,), p + "mix.A_log": (E, N), p + "mix.D": (E,), p + "mix.o": (D, E)})
        else:
            q, k = m["heads"] * m["dim"], m["kv_heads"] * m["dim"]
            s.update({p + "mix.q": (q, D), p + "mix.q.b": (q,), p + "mix.k": (k, D), p + "mix.k.b": (k,), p + "mix.g": (q, D),
                      p + "mix.o": (D, q), p + "mix.o.b": (D,)})
        if layer.get("mlp"):
            F = layer["mlp"]["ff"]
            s.update({p + "norm2": (D,), p + "mlp.gate": (F, D), p + "mlp.up": (F, D), p + "mlp.down": (D, F)})
    s.update({"final.norm": (D,), "head": (V, D)})
    return s


def random_weights(cfg: dict, seed: int) -> Dict[str, np.ndarray]:
    """bfloat16-valued float32 tensors: unit-gain matrices, norm weights near 1, biases and loop vectors of moderate size,
    step sizes around 0.1 and decays that keep a state for a few to a hundred tokens."""
    rng = np.random.default_rng(seed)
    W = {}
    for name, shape in tensor_shapes(cfg).items():
        a = rng.standard_normal(shape)
        if name.endswith("dt.b"):
            a = -2.0 + 0.7 * a
        elif name.endswith("A_log"):
            a = np.log(rng.uniform(0.1, 4.0, shape))
        elif name.endswith(".b"):
            a = 0.3 * a
        elif name.endswith("loop.step"):
            a = 0.5 * a
        elif name.endswith(".conv"):
            a = a / math.sqrt(shape[1])
        elif len(shape) == 1:
            a = 1.0 + 0.1 * a
        elif name == "embed":
            a = a / cfg["embedding"]["scale"]
        else:
            a = a / math.sqrt(shape[1])
        W[name] = bf16_round(a)
    return W
