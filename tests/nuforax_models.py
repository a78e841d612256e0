"""Small random Nuforax models for the tests."""
import numpy as np

import nuforax_plain as npl
import sonuzen_plain as sp
from sonuzen_models import distance                             # noqa: F401  (one measure for all designs)


def rotation(dims, base=10000.0, factor=4.0, original=64, fast=8.0, slow=0.5):
    r = {"dims": dims, "base": base}
    if factor:
        r["scaling"] = {"factor": factor, "original": original, "fast": fast, "slow": slow}
    return r


def latent(heads, dim, rot_dim, vdim, kv_rank, size, ff=None, kv_from=None, scale=None, rot=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "mask": {"size": size}, "rot": rot or rotation(rot_dim),
         "scale": scale or 1.3 * (dim + rot_dim) ** -0.5}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def mamba2(heads, vdim, state, groups, conv, norm_groups, ff=None):
    return {"type": "mamba2", "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def config(width, vocab, layers, buckets=97, mul_prev=31, mul_cur=11, spread=2.0, eps=1e-5):
    """spread: of the logits, roughly"""
    scale = round(width ** 0.5 / spread, 3)
    return {"architecture": "Nuforax", "width": width, "vocab": vocab, "layers": layers, "norm": {"eps": eps},
            "embedding": {"scale": scale, "bigram": {"buckets": buckets, "mul_prev": mul_prev, "mul_cur": mul_cur}}}


FAST = rotation(8, base=500.0, factor=2.5, original=40, fast=4.0, slow=0.25)
CONFIGS = {
    # every branch once: shared caches (one read twice, with other windows, heads and sizes), both mixers with and without feed-forward
    "mixed": config(72, 101, [latent(3, 24, 8, 40, 48, 20, ff=56), mamba2(6, 20, 24, 2, 3, 3, ff=40), latent(5, 16, 8, 24, 48, 33, kv_from=0),
                              latent(4, 32, 16, 16, 72, 9, scale=0.4), mamba2(4, 32, 16, 4, 5, 1), latent(2, 40, 8, 32, 48, 64, ff=72, kv_from=0)], eps=3e-4),
    "one_rotation_each": config(96, 300, [latent(4, 16, 8, 16, 32, 17, ff=64, rot=FAST), latent(2, 24, 12, 24, 40, 90, rot=rotation(12, factor=None)),
                                          latent(4, 16, 8, 32, 32, 70, ff=48, kv_from=0, rot=FAST)], buckets=1, mul_prev=0, mul_cur=3, spread=3.0),
    "recurrent": config(64, 77, [mamba2(8, 16, 40, 1, 4, 8, ff=96), mamba2(3, 40, 130, 3, 2, 1, ff=32), mamba2(10, 12, 64, 5, 1, 2)], mul_prev=4000000007, mul_cur=4294967295),
    "odd_sizes": config(76, 63, [latent(3, 20, 6, 12, 36, 5, ff=44), latent(7, 13, 6, 9, 36, 1, kv_from=0), mamba2(5, 9, 11, 5, 7, 3, ff=28), latent(2, 30, 2, 22, 20, 40, ff=12)],
                        buckets=63, spread=1.2),
    "wide": config(200, 150, [latent(9, 128, 64, 128, 264, 100, ff=136), mamba2(4, 64, 128, 2, 4, 2, ff=64), latent(17, 64, 16, 48, 264, 150, rot=rotation(16)),
                              latent(2, 192, 64, 200, 264, 31, kv_from=0, ff=72)]),
}


def tensors(cfg, seed):
    """Weights as a model folder holds them (all on the bfloat16 grid)."""
    rng = np.random.default_rng(seed)
    W, V = cfg["width"], cfg["vocab"]
    t = {}

    def matrix(name, rows, cols, gain=1.0):
        t[name] = sp.bf16_round(rng.standard_normal((rows, cols)).astype(np.float32) * (gain * cols ** -0.5))

    def vector(name, *shape, mean=0.0, spread=0.3):
        t[name] = sp.bf16_round((mean + spread * rng.standard_normal(shape)).astype(np.float32))

    matrix("embed", V, W, gain=W ** 0.5 / cfg["embedding"]["scale"])            # spread 1 in the stream
    matrix("bigram", cfg["embedding"]["bigram"]["buckets"] + 1, W, gain=0.6 * W ** 0.5)
    for i, l in enumerate(cfg["layers"]):
        p, m = f"l{i}.", l["mixer"]
        mix = p + "mix."
        vector(p + "norm1", W, mean=0.7)
        if l["type"] == "latent_attention":
            H = m["heads"]
            matrix(mix + "q", H * (m["dim"] + m["rot_dim"]), W)
            if m.get("kv_from") is None:
                matrix(mix + "dkv", m["kv_rank"] + m["rot_dim"], W)
                vector(mix + "dkv.norm", m["kv_rank"], mean=1.0)
            matrix(mix + "uk", H * m["dim"], m["kv_rank"])
            matrix(mix + "uv", H * m["vdim"], m["kv_rank"])
            vector(mix + "sink", H, mean=2.5, spread=1.0)
            matrix(mix + "o", W, H * m["vdim"])
        else:
            inner, bc = m["heads"] * m["vdim"], 2 * m["groups"] * m["state"]
            matrix(mix + "in", 2 * inner + bc + m["heads"], W)
            vector(mix + "conv", inner + bc, m["conv"], spread=0.6)
            vector(mix + "conv.b", inner + bc, spread=0.2)
            vector(mix + "dt_bias", m["heads"], mean=-1.0, spread=1.5)
            vector(mix + "A_log", m["heads"], mean=-1.5, spread=1.5)            # slow and fast decays
            vector(mix + "D", m["heads"], mean=0.5, spread=0.5)
            vector(mix + "norm", inner, mean=1.0)
            matrix(mix + "o", W, inner)
        if l["mlp"]:
            vector(p + "norm2", W, mean=0.7)
            matrix(p + "mlp.up", l["mlp"]["ff"], W)
            matrix(p + "mlp.down", W, l["mlp"]["ff"])
    vector("final.norm", W, mean=1.0)
    return t


def write(folder, name, seed=1):
    cfg = CONFIGS[name] if isinstance(name, str) else name
    t = tensors(cfg, seed)
    sp.write_model(folder, cfg, t)
    return cfg, t


def plain(cfg, t):
    return npl.Plain(cfg, t)


def rounding(cfg, t, tokens):
    """What rounding to bfloat16 alone does to each position's logits: the largest distance of a few roundings.  (A sublayer's output is
    normed before it is added, so a position whose output happens to be small is far more sensitive than the others.)"""
    want, worst = plain(cfg, t).forward(tokens), 0.0
    for shift in (0.0, 1e-3, -1e-3):
        rounded = npl.Plain(cfg, t, operands=lambda a: sp.bf16_round((a * (1 + shift)).astype(np.float32)).astype(np.float64) / (1 + shift))
        worst = np.maximum(worst, distance(rounded.forward(tokens), want))
    return worst
