"""Small random Sonuzen models for the tests."""
import numpy as np

import sonuzen_plain as sp


def attention(heads, kv_heads, dim, vdim, scale=None, mlp=None):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale or dim ** -0.5}, "mlp": mlp}


def mingru(width, mlp=None):
    return {"type": "mingru", "mixer": {"width": width}, "mlp": mlp}


def moe(ff, experts, top):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def config(width, vocab, layers, loop=None, taps=4, eps=1e-5, residual_mult=0.4, logit_scale=0.5):
    return {"architecture": "Sonuzen", "width": width, "vocab": vocab, "layers": layers, "loop": loop, "canon": {"taps": taps}, "norm": {"eps": eps},
            "residual_mult": residual_mult, "logit_scale": logit_scale}


CONFIGS = {
    # every branch once: layers before, in and after the loop, layers without feed-forward, unequal sizes everywhere
    "mixed": config(72, 101, [mingru(40, moe(48, 3, 1)), attention(6, 2, 24, 40, 0.31, moe(56, 5, 2)), mingru(88), attention(4, 4, 32, 16, 0.2),
                              attention(3, 1, 48, 24, mlp=moe(40, 4, 3))],
                    loop={"start": 1, "stop": 3, "times": 3}, taps=3, eps=2e-4, residual_mult=0.55, logit_scale=1.7),
    "no_loop": config(128, 77, [attention(8, 1, 64, 128, mlp=moe(96, 6, 2)), mingru(136, moe(64, 2, 2))], loop=None, taps=6),
    "looped": config(96, 300, [attention(2, 1, 80, 48, mlp=moe(32, 7, 3)), mingru(64, moe(24, 4, 2))], loop={"start": 0, "stop": 2, "times": 2}, taps=2,
                     residual_mult=1.0, logit_scale=0.25),
    "one_tap": config(64, 50, [mingru(64, moe(40, 3, 2)), attention(5, 1, 16, 16)], loop={"start": 1, "stop": 2, "times": 1}, taps=1),
    "odd_sizes": config(76, 63, [attention(3, 3, 20, 12, mlp=moe(44, 3, 2)), mingru(36, moe(28, 3, 1))], loop={"start": 1, "stop": 2, "times": 2}, taps=5),
}


def tensors(cfg, seed):
    """Weights as a model folder holds them (matrices on the bfloat16 grid)."""
    rng = np.random.default_rng(seed)
    W, V, taps = cfg["width"], cfg["vocab"], cfg["canon"]["taps"]
    t = {}

    def matrix(name, rows, cols, gain=1.0):
        t[name] = sp.bf16_round(rng.standard_normal((rows, cols)).astype(np.float32) * (gain * cols ** -0.5))

    def vector(name, *shape, mean=0.0, spread=0.3):
        t[name] = sp.bf16_round((mean + spread * rng.standard_normal(shape)).astype(np.float32))

    matrix("embed", V, W, gain=W ** 0.5)
    if cfg.get("loop"):
        vector("loop.step", cfg["loop"]["times"], W, spread=0.5)
    for i, l in enumerate(cfg["layers"]):
        p, m = f"l{i}.", l["mixer"]
        for n in ("norm1", "norm1b") + (("norm2", "norm2b") if l["mlp"] else ()):
            vector(p + n, W)
        vector(p + "canon1", W, taps, spread=0.4)
        if l["type"] == "attention":
            matrix(p + "mix.q", m["heads"] * m["dim"], W)
            matrix(p + "mix.k", m["kv_heads"] * m["dim"], W)
            matrix(p + "mix.v", m["kv_heads"] * m["vdim"], W)
            vector(p + "mix.q.norm", m["dim"], mean=1.5)
            vector(p + "mix.k.norm", m["dim"], mean=1.5)
            t[p + "mix.r1"] = sp.bf16_round(rng.uniform(0.05, 0.6, m["heads"]).astype(np.float32))
            t[p + "mix.r2"] = sp.bf16_round(rng.uniform(0.02, 1.5, m["heads"]).astype(np.float32))
            matrix(p + "mix.o", W, m["heads"] * m["vdim"])
        else:
            for n in "zxg":
                matrix(p + "mix." + n, m["width"], W, gain=2.0)
            vector(p + "mix.z.b", m["width"], mean=-1.5, spread=1.5)       # slow gates: the state reaches far back
            vector(p + "mix.x.b", m["width"], spread=0.5)
            matrix(p + "mix.o", W, m["width"])
        if l["mlp"]:
            vector(p + "canon2", W, taps, spread=0.4)
            ff, n, top = l["mlp"]["expert"]["ff"], l["mlp"]["router"]["experts"], l["mlp"]["router"]["top"]
            for e in range(n):
                matrix(f"{p}mlp.e{e}.gate", ff, W)
                matrix(f"{p}mlp.e{e}.up", ff, W)
                matrix(f"{p}mlp.e{e}.down", W, ff)
            t[p + "mlp.table"] = np.stack([rng.permutation(n)[:top] for _ in range(V)]).astype(np.int32)
    vector("final.norm", W)
    matrix("head", V, W)
    return t


def write(folder, name, seed=1):
    cfg = CONFIGS[name] if isinstance(name, str) else name
    t = tensors(cfg, seed)
    sp.write_model(folder, cfg, t)
    return cfg, t


def distance(got, want):
    """Per row: rms of the difference without its mean, relative to the rms of the wanted logits without theirs."""
    d = np.asarray(got, np.float64) - want
    d -= d.mean(axis=-1, keepdims=True)
    w = want - want.mean(axis=-1, keepdims=True)
    return np.sqrt((d ** 2).mean(axis=-1) / (w ** 2).mean())


def plain(cfg, t):
    return sp.Plain(cfg, t)
