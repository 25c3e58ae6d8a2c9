"""Configurations shared by the Kolatar tests (CPU and GPU)."""


def mamba(inner=80, state=16, conv=4, dt_rank=6):
    return {"type": "mamba1", "mixer": {"inner": inner, "state": state, "conv": conv, "dt_rank": dt_rank}}


def attention(heads=4, kv_heads=2, dim=24, rot=8, window=9, softcap=6.0, base=500.0, scaling=True, scale=None, factor=4.0, original=64,
              fast=8.0, slow=1.0):
    r = {"base": base, "dims": rot}
    if scaling:
        r["scaling"] = {"factor": factor, "original": original, "fast": fast, "slow": slow}
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "rot": r, "scale": scale if scale is not None else dim ** -0.5}
    if softcap:
        m["softcap"] = softcap
    if window:
        m["mask"] = {"size": window}
    return {"type": "attention", "mixer": m}


def model(layers, width=96, vocab=203, eps=1e-5, loop=(0, 0, 1), emb=3.5, logit=1.7):
    """layers: (mixer, feed-forward width or 0)"""
    return {"architecture": "Kolatar", "width": width, "vocab": vocab, "norm": {"eps": eps}, "embedding": {"scale": emb}, "logit_scale": logit,
            "loop": dict(zip(("start", "stop", "times"), loop)),
            "layers": [dict(m, mlp={"kind": "dense", "ff": ff} if ff else None) for m, ff in layers]}


# both mixers with and without a feed-forward, the loop in the middle and around both of them
SMALL = model([(mamba(), 0), (attention(), 88), (mamba(inner=64, state=24, conv=3, dt_rank=12), 72), (attention(heads=6, kv_heads=6, dim=16, window=5), 0),
               (mamba(conv=2), 0)], loop=(1, 4, 2))
# nothing even where it may be odd, nothing equal, nothing shared between layers
ODD = model([(attention(heads=6, kv_heads=2, dim=21, rot=6, window=7), 51), (mamba(inner=37, state=5, conv=2, dt_rank=3), 0),
             (attention(heads=1, kv_heads=1, dim=5, rot=4, window=1, softcap=0.7), 0), (mamba(inner=131, state=19, conv=6, dt_rank=13), 1),
             (attention(heads=9, kv_heads=3, dim=2, rot=2, window=33, base=3.0, softcap=0), 0), (mamba(inner=1, state=1, conv=1, dt_rank=1), 7)],
            width=71, vocab=131, eps=0.02, loop=(0, 2, 3), emb=0.3, logit=11.0)
