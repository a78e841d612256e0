"""A slow, plain implementation of the Sonuzen decoder in numpy, one function per mechanism.

Written from the equations of the design and sharing no code with the product path; everything
is computed in `dtype` (float64 unless a test says otherwise), one whole sequence at a time, with
no cache: position i of the result depends on tokens 0 .. i only because each mechanism is causal.

Shapes: a sequence is [T][width]; weights are a dict name -> array as stored in the model folder.
"""
import json
import os

import numpy as np

SAFETENSOR_DTYPES = {"BF16": 2, "F32": 4, "I32": 4}


def bf16_round(a):
    """Nearest bfloat16 (ties to even) of a float32 array, as float32."""
    u = np.ascontiguousarray(a, np.float32).view(np.uint32).astype(np.uint64)
    u = (u + 0x7FFF + ((u >> 16) & 1)) & 0xFFFF0000
    return u.astype(np.uint32).view(np.float32)


def bf16_bits(a):
    return (bf16_round(a).view(np.uint32) >> 16).astype(np.uint16)


def read_safetensors(path):
    out = {}
    with open(path, "rb") as f:
        n = int.from_bytes(f.read(8), "little")
        head = json.loads(f.read(n))
        data = f.read()
    for name, t in head.items():
        if name == "__metadata__":
            continue
        lo, hi = t["data_offsets"]
        raw = data[lo:hi]
        if t["dtype"] == "BF16":
            a = (np.frombuffer(raw, np.uint16).astype(np.uint32) << 16).view(np.float32)
        elif t["dtype"] == "F32":
            a = np.frombuffer(raw, np.float32)
        else:
            assert t["dtype"] == "I32", t
            a = np.frombuffer(raw, np.int32)
        out[name] = a.reshape(t["shape"])
    return out


def write_safetensors(path, tensors):
    """float arrays as bfloat16, integer arrays as int32."""
    head, blobs, at = {}, [], 0
    for name, a in tensors.items():
        if np.issubdtype(a.dtype, np.integer):
            raw, dt = np.ascontiguousarray(a, np.int32).tobytes(), "I32"
        else:
            raw, dt = bf16_bits(a).tobytes(), "BF16"
        head[name] = {"dtype": dt, "shape": list(a.shape), "data_offsets": [at, at + len(raw)]}
        blobs.append(raw)
        at += len(raw)
    text = json.dumps(head).encode()
    with open(path, "wb") as f:
        f.write(len(text).to_bytes(8, "little"))
        f.write(text)
        for b in blobs:
            f.write(b)


def write_model(folder, config, tensors):
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(config, f, indent=1)
    write_safetensors(os.path.join(folder, "model.safetensors"), tensors)


# ---- mechanisms ----------------------------------------------------------------------------

def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def rms(x, eps):
    return np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def norm_one_plus(x, w, eps):
    return x / rms(x, eps) * (1.0 + w)


def norm_plain(x, w, eps):
    return x / rms(x, eps) * w


def causal_conv(h, w):
    """w: [width][taps]; output t = sum_j w[:, j] h[t - taps + 1 + j], zeros before the start."""
    T, taps = h.shape[0], w.shape[1]
    padded = np.concatenate([np.zeros((taps - 1, h.shape[1]), h.dtype), h])
    return sum(padded[j:j + T] * w[:, j] for j in range(taps))


def min_gru(z, u, gate_in):
    """S_t = (1 - z) S_(t-1) + z c(u), S_(-1) = 0; returns S * silu(gate)."""
    z = sigmoid(z)
    cand = np.where(u >= 0, u + 0.5, sigmoid(u))
    S = np.zeros(z.shape[1], z.dtype)
    out = np.empty_like(z)
    for t in range(z.shape[0]):
        S = (1.0 - z[t]) * S + z[t] * cand[t]
        out[t] = S
    return out * silu(gate_in)


def distance_bias(r1, r2, T):
    d = np.arange(T)[:, None] - np.arange(T)[None, :]
    return r1[:, None, None] * np.log1p(r2[:, None, None] * np.maximum(d, 0))


def sink_softmax(s, mask):
    """exp(s_j) / (1 + sum exp(s_j)) over the positions the mask keeps."""
    s = np.where(mask, s, -np.inf)
    m = np.maximum(s.max(axis=-1, keepdims=True), 0.0)
    e = np.exp(s - m)
    return e / (np.exp(-m) + e.sum(axis=-1, keepdims=True))


def attention(q, k, v, r1, r2, scale):
    """q [T][H][dim], k [T][G][dim], v [T][G][vdim] (q and k already normalised) -> [T][H * vdim]."""
    T, H = q.shape[:2]
    G = k.shape[1]
    kk, vv = np.repeat(k, H // G, axis=1), np.repeat(v, H // G, axis=1)
    s = np.einsum("ihd,jhd->hij", q, kk) * scale - distance_bias(r1, r2, T)
    p = sink_softmax(s, np.tril(np.ones((T, T), bool)))
    return np.einsum("hij,jhd->ihd", p, vv).reshape(T, -1)


def expert(x, gate, up, down):
    return (silu(x @ gate.T) * (x @ up.T)) @ down.T


def table_moe(x, tokens, table, experts):
    """experts: list of (gate, up, down); every chosen expert counts 1 / top."""
    out = np.zeros_like(x)
    top = table.shape[1]
    for t, tok in enumerate(tokens):
        for e in table[tok]:
            out[t] += expert(x[t:t + 1], *experts[e])[0] / top
    return out


# ---- the model -----------------------------------------------------------------------------

def layer_order(config):
    """(layer, pass or None) in execution order; a pass number marks the layer that begins the pass."""
    n = len(config["layers"])
    loop = config.get("loop") or {"start": 0, "stop": 0, "times": 0}
    order = [(i, None) for i in range(loop["start"])]
    for t in range(loop["times"]):
        order += [(i, t if i == loop["start"] else None) for i in range(loop["start"], loop["stop"])]
    return order + [(i, None) for i in range(loop["stop"] if loop["times"] else loop["start"], n)]


class Plain:
    def __init__(self, config, tensors, dtype=np.float64):
        self.c, self.dtype = config, dtype
        self.w = {k: (a if np.issubdtype(a.dtype, np.integer) else a.astype(dtype)) for k, a in tensors.items()}
        self.eps = config["norm"]["eps"]

    @classmethod
    def load(cls, folder, dtype=np.float64):
        with open(os.path.join(folder, "config.json")) as f:
            config = json.load(f)
        return cls(config, read_safetensors(os.path.join(folder, "model.safetensors")), dtype)

    def mixer(self, i, h):
        spec, w, p = self.c["layers"][i], self.w, f"l{i}.mix."
        m = spec["mixer"]
        if spec["type"] == "mingru":
            y = min_gru(h @ w[p + "z"].T + w[p + "z.b"], h @ w[p + "x"].T + w[p + "x.b"], h @ w[p + "g"].T)
            return y @ w[p + "o"].T
        assert spec["type"] == "attention"
        T, H, G = h.shape[0], m["heads"], m["kv_heads"]
        q = norm_plain((h @ w[p + "q"].T).reshape(T, H, m["dim"]), w[p + "q.norm"], self.eps)
        k = norm_plain((h @ w[p + "k"].T).reshape(T, G, m["dim"]), w[p + "k.norm"], self.eps)
        v = (h @ w[p + "v"].T).reshape(T, G, m["vdim"])
        return attention(q, k, v, w[p + "r1"], w[p + "r2"], m["scale"]) @ w[p + "o"].T

    def feed_forward(self, i, h, tokens):
        w, p = self.w, f"l{i}.mlp."
        n = self.c["layers"][i]["mlp"]["router"]["experts"]
        return table_moe(h, tokens, w[p + "table"], [tuple(w[f"{p}e{e}.{s}"] for s in ("gate", "up", "down")) for e in range(n)])

    def layer(self, i, x, tokens):
        w, m = self.w, self.c["residual_mult"]
        h = norm_one_plus(x, w[f"l{i}.norm1"], self.eps)
        h = h + causal_conv(h, w[f"l{i}.canon1"])
        x = x + m * norm_one_plus(self.mixer(i, h), w[f"l{i}.norm1b"], self.eps)
        if self.c["layers"][i]["mlp"] is not None:
            h = norm_one_plus(x, w[f"l{i}.norm2"], self.eps)
            h = h + causal_conv(h, w[f"l{i}.canon2"])
            x = x + m * norm_one_plus(self.feed_forward(i, h, tokens), w[f"l{i}.norm2b"], self.eps)
        return x

    def forward(self, tokens, layers=None):
        """Logits [T][vocab]; `layers`, when given, collects the residual stream after every layer run."""
        x = self.w["embed"][np.asarray(tokens)]
        for i, begins in layer_order(self.c):
            if begins is not None:
                x = x + self.w["loop.step"][begins]
            x = self.layer(i, x, tokens)
            if layers is not None:
                layers.append(x.copy())
        return norm_one_plus(x, self.w["final.norm"], self.eps) @ self.w["head"].T * self.c["logit_scale"]
