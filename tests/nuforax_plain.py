"""A slow, plain implementation of the Nuforax decoder in numpy, one function per mechanism.

Written from the equations of the design and sharing no code with the product path; everything is computed in `dtype`
(float64 unless a test says otherwise), one whole sequence at a time, with no cache and no carried state.

Shapes: a sequence is [T][width]; weights are a dict name -> array as stored in the model folder.
"""
import json
import math
import os

import numpy as np

from sonuzen_plain import causal_conv, norm_plain, read_safetensors, silu


# ---- mechanisms ----------------------------------------------------------------------------

def bigram_rows(tokens, buckets, mul_prev, mul_cur):
    """Row of the pair table for every token; the first token of a sequence has the last row to itself."""
    rows = [buckets]
    for prev, cur in zip(tokens[:-1], tokens[1:]):
        rows.append((int(prev) * mul_prev + int(cur) * mul_cur) % buckets)
    return np.array(rows)


def yarn(dims, base, scaling=None):
    """Frequencies of the dims / 2 pairs and the factor of cos and sin."""
    f = np.array([base ** (-2.0 * i / dims) for i in range(dims // 2)])
    if not scaling:
        return f, 1.0
    def turn(t):
        return dims * math.log(scaling["original"] / (2 * math.pi * t)) / (2 * math.log(base))
    lo, hi = max(math.floor(turn(scaling["fast"])), 0), min(math.ceil(turn(scaling["slow"])), dims - 1)
    ramp = np.clip((np.arange(dims // 2) - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return f / scaling["factor"] * ramp + f * (1 - ramp), 0.1 * math.log(scaling["factor"]) + 1.0


def rotate(x, positions, freqs, mult):
    """x [T][...][n]: pairs (2 i, 2 i + 1) of the leading 2 * len(freqs) values turn by position * freqs[i]."""
    n = 2 * len(freqs)
    a = (positions[:, None] * freqs).reshape(len(positions), *([1] * (x.ndim - 2)), len(freqs))
    c, s = np.cos(a) * mult, np.sin(a) * mult
    out = x.copy()
    u, v = x[..., 0:n:2], x[..., 1:n:2]
    out[..., 0:n:2] = u * c - v * s
    out[..., 1:n:2] = v * c + u * s
    return out


def window_mask(T, size):
    d = np.arange(T)[:, None] - np.arange(T)[None, :]
    return (d >= 0) & (d < size)


def sink_weights(s, mask, sink):
    """s [H][T][T]; exp(s_ij) / (exp(sink_h) + sum_j exp(s_ij)) over the keys of the mask."""
    s = np.where(mask, s, -np.inf)
    m = np.maximum(s.max(axis=-1, keepdims=True), sink[:, None, None])
    e = np.exp(s - m)
    return e / (np.exp(sink[:, None, None] - m) + e.sum(axis=-1, keepdims=True))


def latent_attention(q, c, k_rot, uk, uv, sink, scale, size):
    """q [T][H][dim + rot] (rotated part last, turned already), c [T][rank], k_rot [T][rot] (turned already),
    uk [H * dim][rank], uv [H * vdim][rank] -> [T][H * vdim]."""
    T, H = q.shape[:2]
    dim, vdim = uk.shape[0] // H, uv.shape[0] // H
    k, v = (c @ uk.T).reshape(T, H, dim), (c @ uv.T).reshape(T, H, vdim)
    s = (np.einsum("ihd,jhd->hij", q[..., :dim], k) + np.einsum("ihd,jd->hij", q[..., dim:], k_rot)) * scale
    p = sink_weights(s, window_mask(T, size), sink)
    return np.einsum("hij,jhd->ihd", p, v).reshape(T, -1)


def softplus(z):
    return np.logaddexp(0.0, z)


def state_space(x, B, C, dt, A_log, D):
    """x [T][H][P], B and C [T][G][N], dt [T][H] (after softplus): S_t = exp(-exp(A_log) dt) S_(t-1) + dt B x^T,
    y = C S + D x, S_(-1) = 0 -> [T][H][P]."""
    T, H, P = x.shape
    G, N = B.shape[1:]
    S = np.zeros((H, N, P), x.dtype)
    y = np.empty_like(x)
    for t in range(T):
        b, c = np.repeat(B[t], H // G, axis=0), np.repeat(C[t], H // G, axis=0)
        S = np.exp(-np.exp(A_log) * dt[t])[:, None, None] * S + (dt[t][:, None] * b)[:, :, None] * x[t][:, None, :]
        y[t] = np.einsum("hn,hnp->hp", c, S) + D[:, None] * x[t]
    return y


def gated_group_norm(y, z, w, parts, eps):
    g = y * silu(z)
    T, n = g.shape
    return norm_plain(g.reshape(T, parts, n // parts), 1.0, eps).reshape(T, n) * w


def relu_squared(z):
    return np.maximum(z, 0.0) ** 2


# ---- the model -----------------------------------------------------------------------------

class Plain:
    def __init__(self, config, tensors, dtype=np.float64, operands=lambda a: a):
        """operands: applied to what enters a matrix product and to what a cache holds (rounding, to see what it causes)."""
        self.c, self.dtype, self.op = config, dtype, operands
        self.w = {k: (a if np.issubdtype(a.dtype, np.integer) else a.astype(dtype)) for k, a in tensors.items()}
        self.eps = config["norm"]["eps"]

    @classmethod
    def load(cls, folder, dtype=np.float64):
        with open(os.path.join(folder, "config.json")) as f:
            config = json.load(f)
        return cls(config, read_safetensors(os.path.join(folder, "model.safetensors")), dtype)

    def embed(self, tokens):
        e = self.c["embedding"]
        b = e["bigram"]
        return self.w["embed"][np.asarray(tokens)] * e["scale"] + self.w["bigram"][bigram_rows(tokens, b["buckets"], b["mul_prev"], b["mul_cur"])]

    def attention(self, i, h, kept):
        w, m, p = self.w, self.c["layers"][i]["mixer"], f"l{i}.mix."
        op, T, H, pos = self.op, h.shape[0], m["heads"], np.arange(h.shape[0]).astype(self.dtype)
        freqs, mult = yarn(m["rot"]["dims"], m["rot"]["base"], m["rot"].get("scaling"))
        freqs = freqs.astype(self.dtype)
        q = (h @ w[p + "q"].T).reshape(T, H, m["dim"] + m["rot_dim"])
        q = np.concatenate([q[..., :m["dim"]], rotate(q[..., m["dim"]:], pos, freqs, mult)], axis=-1)
        if m.get("kv_from") is None:
            d = h @ w[p + "dkv"].T
            kept[i] = op(norm_plain(d[:, :m["kv_rank"]], w[p + "dkv.norm"], self.eps)), op(rotate(d[:, m["kv_rank"]:], pos, freqs, mult))
        c, k_rot = kept[m.get("kv_from") if m.get("kv_from") is not None else i]
        y = latent_attention(op(q), c, k_rot, w[p + "uk"], w[p + "uv"], w[p + "sink"], m["scale"], m["mask"]["size"])
        return op(y) @ w[p + "o"].T

    def mamba2(self, i, h):
        w, m, p = self.w, self.c["layers"][i]["mixer"], f"l{i}.mix."
        T, H, P, N, G = h.shape[0], m["heads"], m["vdim"], m["state"], m["groups"]
        inner = H * P
        z, xbc, dt = np.split(h @ w[p + "in"].T, [inner, 2 * inner + 2 * G * N], axis=1)
        xbc = silu(causal_conv(xbc, w[p + "conv"]) + w[p + "conv.b"])
        x, B, C = np.split(xbc, [inner, inner + G * N], axis=1)
        y = state_space(x.reshape(T, H, P), B.reshape(T, G, N), C.reshape(T, G, N), softplus(dt + w[p + "dt_bias"]), w[p + "A_log"], w[p + "D"])
        return self.op(gated_group_norm(y.reshape(T, inner), z, w[p + "norm"], m["norm_groups"], self.eps)) @ w[p + "o"].T

    def layer(self, i, x, kept):
        w, spec = self.w, self.c["layers"][i]
        h = self.op(x)
        y = self.attention(i, h, kept) if spec["type"] == "latent_attention" else self.mamba2(i, h)
        x = x + norm_plain(y, w[f"l{i}.norm1"], self.eps)
        if spec["mlp"] is not None:
            y = self.op(relu_squared(self.op(x) @ w[f"l{i}.mlp.up"].T)) @ w[f"l{i}.mlp.down"].T
            x = x + norm_plain(y, w[f"l{i}.norm2"], self.eps)
        return x

    def forward(self, tokens, layers=None):
        """Logits [T][vocab]; `layers`, when given, collects the residual stream after every layer."""
        x, kept = self.embed(list(tokens)), {}
        for i in range(len(self.c["layers"])):
            x = self.layer(i, x, kept)
            if layers is not None:
                layers.append(x.copy())
        return self.op(norm_plain(x, self.w["final.norm"], self.eps)) @ self.w["embed"].T
