"""Plain, slow numpy statement of the Rutenex decoder (latent attention under a sliding window, layer norms, gated
GELU feed-forward), one function per mechanism, used only to check the CUDA engine.

Everything runs in one floating type (``dtype``, double by default) and without a cache: a whole sequence goes
through a layer at once, every query row looks its visible keys up in a boolean matrix, keys and values are
expanded per head.  Nothing here is shared with the package under test.

A model is ``cfg`` (the decoded config.json) plus ``W``, a dict of numpy arrays by tensor name.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import numpy as np


# ------------------------------------------------------------------ mechanisms

def layer_norm(x: np.ndarray, weight: np.ndarray, bias: np.ndarray, eps: float) -> np.ndarray:
    centred = x - x.mean(axis=-1, keepdims=True)
    var = (centred * centred).mean(axis=-1, keepdims=True)
    return centred / np.sqrt(var + eps) * weight + bias


def rms_norm(x: np.ndarray, weight: np.ndarray, eps: float) -> np.ndarray:
    return x / np.sqrt((x * x).mean(axis=-1, keepdims=True) + eps) * weight


def rotation_frequencies(rot: dict) -> np.ndarray:
    """Angle per position of every rotated pair; with ``scaling`` the slow pairs are stretched by its factor and the
    fast ones kept, with a linear blend between the two border pairs."""
    dims, base = rot["dims"], float(rot["base"])
    freqs = []
    sc = rot.get("scaling")
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        if sc:
            def border(turns):
                return dims * math.log(sc["original"] / (2 * math.pi * turns)) / (2 * math.log(base))
            lo = max(math.floor(border(sc["fast"])), 0)
            hi = min(math.ceil(border(sc["slow"])), dims - 1)
            blend = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
            f = f / sc["factor"] * blend + f * (1 - blend)
        freqs.append(f)
    return np.array(freqs, dtype=np.float64)


def rotation_magnitude(rot: dict) -> float:
    sc = rot.get("scaling")
    return 0.1 * math.log(sc["factor"]) + 1.0 if sc else 1.0


def rotate(x: np.ndarray, positions: np.ndarray, rot: dict) -> np.ndarray:
    """x [tokens, ..., n]: the first rot.dims of the last axis turn pairwise (neighbours form a pair)."""
    out = np.array(x, copy=True)
    mag = rotation_magnitude(rot)
    for i, f in enumerate(rotation_frequencies(rot)):
        shape = (len(positions),) + (1,) * (x.ndim - 2)
        ang = positions.astype(np.float64) * f
        c = (np.cos(ang) * mag).reshape(shape).astype(x.dtype)
        s = (np.sin(ang) * mag).reshape(shape).astype(x.dtype)
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * c - v * s
        out[..., 2 * i + 1] = v * c + u * s
    return out


def window_mask(n: int, size: Optional[int]) -> np.ndarray:
    """visible[i, j]: key j is at or before query i and at most size - 1 tokens back (no limit when size is None)."""
    i, j = np.arange(n)[:, None], np.arange(n)[None, :]
    vis = j <= i
    return vis if not size else vis & (i - j < size)


def softmax_attend(scores: np.ndarray, visible: np.ndarray, values: np.ndarray) -> np.ndarray:
    """scores [q, k], values [k, v] of one head."""
    s = np.where(visible, scores, -np.inf)
    p = np.exp(s - s.max(axis=1, keepdims=True))
    return (p / p.sum(axis=1, keepdims=True)) @ values


def sigmoid(x: np.ndarray) -> np.ndarray:
    return 1.0 / (1.0 + np.exp(-x))


def gelu_tanh(z: np.ndarray) -> np.ndarray:
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def latent_split(h: np.ndarray, W: Dict[str, np.ndarray], pre: str, m: dict, eps: float, positions: np.ndarray):
    """The two things a token leaves behind: its normed latent and its rotated key part."""
    r = m["kv_rank"]
    d = h @ W[pre + "dkv"].T
    return rms_norm(d[:, :r], W[pre + "dkv.norm"], eps), rotate(d[:, r:], positions, m["rot"])


def latent_attention(h: np.ndarray, W: Dict[str, np.ndarray], pre: str, m: dict, eps: float,
                     positions: Optional[np.ndarray] = None) -> np.ndarray:
    n = h.shape[0]
    pos = np.arange(n) if positions is None else positions
    H, dn, dr, dv = m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    q = (h @ W[pre + "q"].T).reshape(n, H, dn + dr)
    q_plain, q_turn = q[:, :, :dn], rotate(q[:, :, dn:], pos, m["rot"])
    c, k_turn = latent_split(h, W, pre, m, eps, pos)
    k_plain = (c @ W[pre + "uk"].T).reshape(n, H, dn)
    value = (c @ W[pre + "uv"].T).reshape(n, H, dv)
    gate = sigmoid(h @ W[pre + "g"].T)
    vis = window_mask(n, (m.get("mask") or {}).get("size"))
    heads = []
    for a in range(H):
        scores = (q_plain[:, a] @ k_plain[:, a].T + q_turn[:, a] @ k_turn.T) * h.dtype.type(m["scale"])
        heads.append(softmax_attend(scores, vis, value[:, a]) * gate[:, a:a + 1])
    return np.concatenate(heads, axis=1) @ W[pre + "o"].T


def dense_feed_forward(h: np.ndarray, W: Dict[str, np.ndarray], pre: str) -> np.ndarray:
    return (gelu_tanh(h @ W[pre + "gate"].T) * (h @ W[pre + "up"].T)) @ W[pre + "down"].T


# ------------------------------------------------------------------ the model

def forward(cfg: dict, W: Dict[str, np.ndarray], tokens, dtype=np.float64, trace: Optional[List[np.ndarray]] = None
            ) -> np.ndarray:
    """Logits [tokens, vocab] of one sequence; ``trace`` collects the residual stream after every layer."""
    W = {k: np.asarray(v, dtype=dtype) for k, v in W.items()}
    eps = cfg["norm"]["eps"]
    x = W["embed"][np.asarray(tokens)]
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        if layer["type"] != "latent_attention":
            raise ValueError(layer["type"])
        x = x + latent_attention(layer_norm(x, W[p + "norm1"], W[p + "norm1.b"], eps), W, p + "mix.", layer["mixer"], eps)
        if layer.get("mlp"):
            if layer["mlp"]["kind"] != "dense":
                raise ValueError(layer["mlp"]["kind"])
            x = x + dense_feed_forward(layer_norm(x, W[p + "norm2"], W[p + "norm2.b"], eps), W, p + "mlp.")
        if trace is not None:
            trace.append(x.copy())
    return layer_norm(x, W["final.norm"], W["final.norm.b"], eps) @ W["embed"].T


# ------------------------------------------------------------------ random models

def tensor_shapes(cfg: dict) -> Dict[str, tuple]:
    D, V = cfg["width"], cfg["vocab"]
    s = {"embed": (V, D)}
    for i, layer in enumerate(cfg["layers"]):
        m, p = layer["mixer"], f"l{i}."
        H, qd = m["heads"], m["dim"] + m["rot_dim"]
        s.update({p + "norm1": (D,), p + "norm1.b": (D,), p + "mix.q": (H * qd, D),
                  p + "mix.dkv": (m["kv_rank"] + m["rot_dim"], D), p + "mix.dkv.norm": (m["kv_rank"],),
                  p + "mix.uk": (H * m["dim"], m["kv_rank"]), p + "mix.uv": (H * m["vdim"], m["kv_rank"]),
                  p + "mix.g": (H, D), p + "mix.o": (D, H * m["vdim"])})
        if layer.get("mlp"):
            F = layer["mlp"]["ff"]
            s.update({p + "norm2": (D,), p + "norm2.b": (D,), p + "mlp.gate": (F, D), p + "mlp.up": (F, D),
                      p + "mlp.down": (D, F)})
    s.update({"final.norm": (D,), "final.norm.b": (D,)})
    return s


def bf16_round(a: np.ndarray) -> np.ndarray:
    """Nearest bfloat16 (ties to even), as float32."""
    u = np.ascontiguousarray(a, dtype=np.float32).view(np.uint32).astype(np.uint64)
    u = (u + 0x7FFF + ((u >> 16) & 1)) & 0xFFFF0000
    return u.astype(np.uint32).view(np.float32)


def random_weights(cfg: dict, seed: int) -> Dict[str, np.ndarray]:
    """bfloat16-valued float32 tensors: unit-gain matrices, norm weights near 1, small biases, unit-size embedding rows
    scaled so that logits are of order one."""
    rng = np.random.default_rng(seed)
    W = {}
    for name, shape in tensor_shapes(cfg).items():
        a = rng.standard_normal(shape)
        if name.endswith(".b"):
            a = 0.1 * a
        elif len(shape) == 1:
            a = 1.0 + 0.1 * a
        elif name != "embed":
            a = a / math.sqrt(shape[1])
        else:
            a = a / math.sqrt(shape[1]) * 4.0
        W[name] = bf16_round(a)
    return W


def write_model(folder: str, cfg: dict, W: Dict[str, np.ndarray]) -> None:
    """config.json and a bfloat16 model.safetensors, written from the file format's description."""
    import json
    import os
    import struct
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    head, blobs, off = {}, [], 0
    for name, a in W.items():
        raw = (np.ascontiguousarray(a, dtype=np.float32).view(np.uint32) >> 16).astype("<u2").tobytes()
        head[name] = {"dtype": "BF16", "shape": list(a.shape), "data_offsets": [off, off + len(raw)]}
        blobs.append(raw)
        off += len(raw)
    text = json.dumps(head).encode()
    with open(os.path.join(folder, "model.safetensors"), "wb") as f:
        f.write(struct.pack("<Q", len(text)) + text + b"".join(blobs))
