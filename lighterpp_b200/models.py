"""Model registry: which architectures the engine serves, how their configuration reads and which of their tensors goes
where.

A model is a file the reference knows (llama2.c ``.bin``, GGUF) or a folder with ``config.json`` and
``model.safetensors``.  A folder's ``architecture`` key picks an entry of ``ARCHITECTURES``: a function that turns the
decoded config.json into a ``LayeredConfig`` and one that lists (engine tensor, layer, file tensor, shape).
"""
from __future__ import annotations

import json
import os
from typing import Callable, Dict, Iterator, NamedTuple, Tuple

import numpy as np

from .engine import Engine
from .formats import (Layer, LatentMixer, LayeredConfig, Loop, MambaMixer, Rotation, SharedKvMixer, Yarn, load_model, read_safetensors)

TensorRow = Tuple[str, int, str, Tuple[int, ...]]


class Architecture(NamedTuple):
    configure: Callable[[dict, int], LayeredConfig]
    tensors: Callable[[LayeredConfig], Iterator[TensorRow]]


# ------------------------------------------------------------------ Rutenex: latent attention layers under layer norms

def _rotation(rot: dict) -> Rotation:
    s = rot.get("scaling")
    yarn = Yarn(float(s["factor"]), float(s["original"]), float(s["fast"]), float(s["slow"])) if s else None
    return Rotation(int(rot["dims"]), float(rot["base"]), yarn)


def _feed_forward(i: int, y: dict) -> int:
    mlp = y.get("mlp")
    if mlp and mlp["kind"] != "dense":
        raise ValueError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
    return int(mlp["ff"]) if mlp else 0


def _feed_forward_tensors(i: int, y: Layer, dim: int) -> Iterator[TensorRow]:
    if y.ff:
        yield "rms_ffn", i, f"l{i}.norm2", (dim,)
        yield "w1", i, f"l{i}.mlp.gate", (y.ff, dim)
        yield "w3", i, f"l{i}.mlp.up", (y.ff, dim)
        yield "w2", i, f"l{i}.mlp.down", (dim, y.ff)


def rutenex_config(cfg: dict, seq_len: int) -> LayeredConfig:
    layers = []
    for i, y in enumerate(cfg["layers"]):
        if y["type"] != "latent_attention":
            raise ValueError(f"layer {i}: unknown mixer {y['type']!r}")
        m, mask = y["mixer"], y["mixer"].get("mask") or {}
        layers.append(Layer(LatentMixer(int(m["heads"]), int(m["dim"]), int(m["rot_dim"]), int(m["vdim"]), int(m["kv_rank"]),
                                        float(m["scale"]), _rotation(m["rot"]), int(mask.get("size") or 0)),
                            _feed_forward(i, y), "gelu_tanh"))
    return LayeredConfig(int(cfg["width"]), int(cfg["vocab"]), seq_len, layers, "layer", float(cfg["norm"]["eps"]))


def rutenex_tensors(c: LayeredConfig) -> Iterator[TensorRow]:
    D = c.dim
    yield "tok_emb", 0, "embed", (c.vocab_size, D)
    for i, y in enumerate(c.layers):
        p, m = f"l{i}.", y.mixer
        yield "rms_att", i, p + "norm1", (D,)
        yield "norm1_b", i, p + "norm1.b", (D,)
        yield "lat_q", i, p + "mix.q", (m.heads * (m.dim + m.rot_dim), D)
        yield "lat_dkv", i, p + "mix.dkv", (m.kv_rank + m.rot_dim, D)
        yield "lat_norm", i, p + "mix.dkv.norm", (m.kv_rank,)
        yield "lat_uk", i, p + "mix.uk", (m.heads * m.dim, m.kv_rank)
        yield "lat_uv", i, p + "mix.uv", (m.heads * m.vdim, m.kv_rank)
        yield "lat_g", i, p + "mix.g", (m.heads, D)
        yield "wo", i, p + "mix.o", (D, m.heads * m.vdim)
        yield from _feed_forward_tensors(i, y, D)
        if y.ff:
            yield "norm2_b", i, p + "norm2.b", (D,)
    yield "rms_final", 0, "final.norm", (D,)
    yield "norm_final_b", 0, "final.norm.b", (D,)


# ------------------------------------------------------------------ Kolatar: selective-scan and key-is-value attention layers,
# some of which run several times

def kolatar_config(cfg: dict, seq_len: int) -> LayeredConfig:
    layers = []
    for i, y in enumerate(cfg["layers"]):
        m = y["mixer"]
        if y["type"] == "mamba1":
            mixer = MambaMixer(int(m["inner"]), int(m["state"]), int(m["conv"]), int(m["dt_rank"]))
        elif y["type"] == "attention":
            if int(m.get("vdim", m["dim"])) != int(m["dim"]):
                raise ValueError(f"layer {i}: values of {m['vdim']} dimensions cannot be keys of {m['dim']}")
            mixer = SharedKvMixer(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), float(m["scale"]), _rotation(m["rot"]),
                                  int((m.get("mask") or {}).get("size") or 0), float(m.get("softcap") or 0.0), bias=True, gate=True)
        else:
            raise ValueError(f"layer {i}: unknown mixer {y['type']!r}")
        layers.append(Layer(mixer, _feed_forward(i, y), "silu"))
    loop = cfg.get("loop")
    return LayeredConfig(int(cfg["width"]), int(cfg["vocab"]), seq_len, layers, "rms", float(cfg["norm"]["eps"]),
                         float(cfg["embedding"]["scale"]), float(cfg["logit_scale"]),
                         Loop(int(loop["start"]), int(loop["stop"]), int(loop["times"])) if loop else None)


def kolatar_tensors(c: LayeredConfig) -> Iterator[TensorRow]:
    D = c.dim
    yield "tok_emb", 0, "embed", (c.vocab_size, D)
    if c.loop and c.loop.stop > c.loop.start:
        yield "loop_step", 0, "loop.step", (c.loop.times, D)
    for i, y in enumerate(c.layers):
        p, m = f"l{i}.mix.", y.mixer
        yield "rms_att", i, f"l{i}.norm1", (D,)
        if isinstance(m, MambaMixer):
            yield "scan_in", i, p + "in", (2 * m.inner, D)
            yield "scan_conv", i, p + "conv", (m.inner, m.conv)
            yield "scan_conv_b", i, p + "conv.b", (m.inner,)
            yield "scan_low", i, p + "x", (m.dt_rank + 2 * m.state, m.inner)
            yield "scan_dt", i, p + "dt", (m.inner, m.dt_rank)
            yield "scan_dt_b", i, p + "dt.b", (m.inner,)
            yield "scan_a_log", i, p + "A_log", (m.inner, m.state)
            yield "scan_d", i, p + "D", (m.inner,)
            yield "wo", i, p + "o", (D, m.inner)
        else:
            q, k = m.heads * m.dim, m.kv_heads * m.dim
            yield "wq", i, p + "q", (q, D)
            yield "wq_b", i, p + "q.b", (q,)
            yield "wk", i, p + "k", (k, D)
            yield "wk_b", i, p + "k.b", (k,)
            yield "wg", i, p + "g", (q, D)
            yield "wo", i, p + "o", (D, q)
            yield "wo_b", i, p + "o.b", (D,)
        yield from _feed_forward_tensors(i, y, D)
    yield "rms_final", 0, "final.norm", (D,)
    yield "w_cls", 0, "head", (c.vocab_size, D)


ARCHITECTURES: Dict[str, Architecture] = {"Kolatar": Architecture(kolatar_config, kolatar_tensors),
                                          "Rutenex": Architecture(rutenex_config, rutenex_tensors)}

# weight / cache types of the two precisions a model folder is served in
PRECISIONS = {"bfloat16": ("bf16", "f16"), "float32": ("f32", "f32")}
DEFAULT_CONTEXT = 4096


def read_config(folder: str, seq_len: int) -> Tuple[Architecture, LayeredConfig]:
    with open(os.path.join(folder, "config.json")) as f:
        cfg = json.load(f)
    name = cfg.get("architecture")
    if name not in ARCHITECTURES:
        raise ValueError(f"{folder}: unknown architecture {name!r} (known: {', '.join(sorted(ARCHITECTURES))})")
    arch = ARCHITECTURES[name]
    return arch, arch.configure(cfg, seq_len)


def load_folder(folder: str, dtype: str = "bfloat16", seq_len: int = DEFAULT_CONTEXT, **kw) -> Engine:
    arch, c = read_config(folder, seq_len)
    tensors = read_safetensors(os.path.join(folder, "model.safetensors"))
    wd, kd = PRECISIONS[dtype]
    rows = list(arch.tensors(c))
    for _, _, name, shape in rows:  # all of it before the first byte goes to the device
        if name not in tensors:
            raise ValueError(f"{folder}: missing tensor {name}")
        if tuple(tensors[name].shape) != shape:
            raise ValueError(f"{folder}: tensor {name} has shape {tensors[name].shape}, expected {shape}")
    eng = Engine(c, wd, kd, **kw)
    try:
        for ours, layer, name, _ in rows:
            eng.upload(ours, tensors[name], layer)
        eng.finalize()
    except Exception:
        eng.close()
        raise
    return eng


def load_engine(path: str, dtype: str = "", seq_len: int = 0, **kw) -> Engine:
    """Any model the registry or the reference's loaders know.  ``dtype`` ("bfloat16" / "float32") and ``seq_len`` (cache
    positions) apply to model folders; files carry both themselves."""
    if os.path.isdir(path):
        return load_folder(path, dtype or "bfloat16", seq_len or DEFAULT_CONTEXT, **kw)
    cfg, tensors = load_model(path)
    wd = "f16" if tensors["wq"].dtype == np.float16 else "f32"
    if dtype and dtype != {"f16": "float16", "f32": "float32"}[wd]:
        raise ValueError(f"{path} holds {wd} weights, not {dtype}")
    kw.setdefault("kv_dtype", "f16" if wd == "f16" else "f32")
    eng = Engine(cfg, wd, **kw)
    eng.load_weights(tensors)
    return eng
