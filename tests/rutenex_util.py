"""Configurations and comparisons shared by the Rutenex tests (CPU and GPU)."""
import numpy as np

from oracle import rutenex as R


def mixer(heads=4, dim=24, rot_dim=8, vdim=20, kv_rank=48, window=9, base=500.0, dims=None, scaling=True, scale=None,
          factor=4.0, original=64, fast=8.0, slow=1.0):
    rot = {"base": base, "dims": rot_dim if dims is None else dims}
    if scaling:
        rot["scaling"] = {"factor": factor, "original": original, "fast": fast, "slow": slow}
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "rot": rot,
         "scale": scale if scale is not None else (dim + rot_dim) ** -0.5}
    if window:
        m["mask"] = {"size": window}
    return m


def model(layers, width=96, vocab=203, eps=1e-5):
    return {"architecture": "Rutenex", "width": width, "vocab": vocab, "norm": {"eps": eps},
            "layers": [{"type": "latent_attention", "mixer": m, "mlp": {"kind": "dense", "ff": ff} if ff else None} for m, ff in layers]}


SMALL = model([(mixer(), 80), (mixer(window=5, heads=2, dim=32), 0), (mixer(window=14, base=90.0, scaling=False), 112)])
# nothing even, nothing equal, nothing shared between layers
ODD = model([(mixer(heads=3, dim=21, rot_dim=6, vdim=13, kv_rank=37, window=7), 51), (mixer(heads=1, dim=5, rot_dim=10, vdim=1, kv_rank=9, window=1), 0),
             (mixer(heads=5, dim=1, rot_dim=2, vdim=7, kv_rank=70, window=33, base=3.0), 1)], width=71, vocab=131, eps=0.02)


def tokens(cfg, n, seed=0):
    return np.random.default_rng([seed, n]).integers(0, cfg["vocab"], n).astype(np.int32)


def error(got, want):
    """Root mean square of the difference over that of the expected logits, per row; the worst row."""
    got, want = np.atleast_2d(got), np.atleast_2d(want)
    assert np.isfinite(got).all()
    return float((np.sqrt(((got - want) ** 2).mean(axis=1)) / np.sqrt((want ** 2).mean(axis=1))).max())


def configured(cfg, seq_len):
    from lighterpp_b200.models import ARCHITECTURES
    return ARCHITECTURES[cfg["architecture"]].configure(cfg, seq_len)


def bf16_bits(a):
    return (np.ascontiguousarray(a, dtype=np.float32).view(np.uint32) >> 16).astype(np.uint16)


def engine(E, cfg, W, dtype="float32", seq_len=256, **kw):
    from lighterpp_b200.models import ARCHITECTURES, PRECISIONS
    c = configured(cfg, seq_len)
    e = E.Engine(c, *PRECISIONS[dtype], **kw)
    for ours, layer, name, shape in ARCHITECTURES[cfg["architecture"]].tensors(c):
        assert W[name].shape == shape, (name, W[name].shape, shape)
        e.upload(ours, bf16_bits(W[name]), layer)
    e.finalize()
    return e


def portions(e, toks, sizes, start=0):
    """Logits of every token, fed in portions of the given sizes (the last one repeats)."""
    out, at, i = [], 0, 0
    while at < len(toks):
        n = min(sizes[min(i, len(sizes) - 1)], len(toks) - at)
        out.append(e.extend(toks[at:at + n], start + at, range(n)))
        at, i = at + n, i + 1
    return np.concatenate(out)
