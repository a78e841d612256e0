"""Throughput of Nuforax models beside Sonuzen models of equal size (bench.py --workload nuforax-*).

Random bfloat16 weights in layers of a real model's size; the Sonuzen model has the same width, depth, number of heads and active
feed-forward weights.  Measured: decoding (device-fed greedy tokens after a prompt), prompts, and every kernel alone, as for the
Sonuzen workloads (bench_sonuzen.py, bench_models.py).
"""
import ctypes as C
import json
import os
import sys
import time

import numpy as np

import bench_models
import bench_sonuzen
from bench_models import CONTEXT, STEP, VOCAB

SIZES = {
    # width, heads of 128 + 64 rotated, latent of 512, heads of 64 and groups of the state spaces, feed-forward width, layers
    "nuforax-1024": dict(width=1024, heads=8, ssm_heads=32, groups=2, ff=3072, layers=8),
    "nuforax-2048": dict(width=2048, heads=16, ssm_heads=64, groups=4, ff=8448, layers=8),
    "nuforax-4096": dict(width=4096, heads=32, ssm_heads=128, groups=8, ff=16512, layers=4),
}
DIM, ROT, VDIM, RANK, WINDOW = 128, 64, 128, 512, 1024
P, N, TAPS = 64, 128, 4


def config(z):
    """Of four layers: attention, a state space, attention, attention over the third's cache."""
    mlp = {"kind": "dense", "ff": z["ff"]}
    layers = []
    for i in range(z["layers"]):
        if i % 4 == 1:
            layers.append({"type": "mamba2", "mlp": mlp, "mixer": {"heads": z["ssm_heads"], "vdim": P, "state": N, "groups": z["groups"], "conv": TAPS, "norm_groups": z["groups"]}})
            continue
        m = {"heads": z["heads"], "dim": DIM, "rot_dim": ROT, "vdim": VDIM, "kv_rank": RANK, "mask": {"size": WINDOW}, "scale": (DIM + ROT) ** -0.5,
             "rot": {"dims": ROT, "base": 10000.0, "scaling": {"factor": 4.0, "original": 4096, "fast": 32.0, "slow": 1.0}}}
        if i % 4 == 3:
            m["kv_from"] = i - 1
        layers.append({"type": "latent_attention", "mlp": mlp, "mixer": m})
    return {"architecture": "Nuforax", "width": z["width"], "vocab": VOCAB, "layers": layers, "norm": {"eps": 1e-5},
            "embedding": {"scale": z["width"] ** 0.5, "bigram": {"buckets": 20011, "mul_prev": 41, "mul_cur": 13}}}


def tensor_shapes(cfg):
    W = cfg["width"]
    shapes = {"embed": (VOCAB, W), "bigram": (cfg["embedding"]["bigram"]["buckets"] + 1, W), "final.norm": (W,)}
    for i, l in enumerate(cfg["layers"]):
        p, m, mix = f"l{i}.", l["mixer"], f"l{i}.mix."
        shapes[p + "norm1"] = shapes[p + "norm2"] = (W,)
        if l["type"] == "latent_attention":
            H = m["heads"]
            shapes[mix + "q"], shapes[mix + "uk"], shapes[mix + "uv"] = (H * (DIM + ROT), W), (H * DIM, RANK), (H * VDIM, RANK)
            shapes[mix + "sink"], shapes[mix + "o"] = (H,), (W, H * VDIM)
            if "kv_from" not in m:
                shapes[mix + "dkv"], shapes[mix + "dkv.norm"] = (RANK + ROT, W), (RANK,)
        else:
            H, inner, bc = m["heads"], m["heads"] * P, 2 * m["groups"] * N
            shapes[mix + "in"], shapes[mix + "o"], shapes[mix + "norm"] = (2 * inner + bc + H, W), (W, inner), (inner,)
            shapes[mix + "conv"], shapes[mix + "conv.b"] = (inner + bc, TAPS), (inner + bc,)
            shapes[mix + "dt_bias"] = shapes[mix + "A_log"] = shapes[mix + "D"] = (H,)
        shapes[p + "mlp.up"], shapes[p + "mlp.down"] = (l["mlp"]["ff"], W), (W, l["mlp"]["ff"])
    return shapes


def active_bytes(cfg):
    """Weight bytes that one decoded token reads (the embedding table is the output matrix)."""
    return sum(2 * int(np.prod(s)) for n, s in tensor_shapes(cfg).items() if n != "bigram")


def kernel_times(pkg, torch, z, peaks):
    W, H, ff, G, SH = z["width"], z["heads"], z["ff"], z["groups"], z["ssm_heads"]
    inner, bc = SH * P, 2 * G * N
    raw_ssm, q_rows, prompt = 2 * inner + bc + SH, H * (DIM + ROT), f"prompt of {STEP}"
    with pkg.Context(0) as gpu:
        bench = bench_models.Kernels(pkg, torch, gpu, peaks)
        lib, h, rng, ring, f32, b16 = bench.lib, bench.h, bench.rng, bench.ring, bench.f32, bench.b16

        def add(phase, name, launch, nbytes, flops=0.0):
            bench.add("nuforax", phase, name, launch, nbytes, flops)
        pos = gpu.upload(np.array([CONTEXT - 1] * 4, np.uint32))
        pos_prompt = gpu.upload(np.array([CONTEXT - STEP] * 4, np.uint32))
        ids = gpu.upload(rng.integers(0, VOCAB, 4096).astype(np.uint32))
        # -- products ------------------------------------------------------------------------
        widest = max(W, inner, ff, H * VDIM)
        x1, xT = f32(1, widest), b16(STEP, widest)
        out = gpu.zeros(STEP * max(W, raw_ssm, q_rows + RANK + ROT, ff) * 4)
        for name, r, k, act in (("input projections (attention)", q_rows + RANK + ROT, W, 0), ("input projections (attention, shared cache)", q_rows, W, 0),
                                ("output projection (attention)", W, H * VDIM, 0), ("input projection (state space)", raw_ssm, W, 0), ("output projection (state space)", W, inner, 0),
                                ("up + squared ReLU", ff, W, 1), ("down", W, ff, 0)):
            w, d = ring(r * k * 2)
            add("decode", name, lambda i: lib.lv_gemv_bf16(h, out, r, w(i), r, k, k, x1, k, 1, 1.0, act), r * k * 2)
            t = pkg.TYPE_BF16 if act else pkg.TYPE_F32
            add(prompt, name, lambda i: lib.lv_gemm_bf16(h, out, t, r, w(i), r, k, k, xT, k, STEP, 1.0, act), r * k * 2 + STEP * (k * 2 + r * (2 if act else 4)), 2.0 * r * k * STEP)
            gpu.free(d)
        w, d = ring(VOCAB * W * 2)
        head = gpu.zeros(VOCAB * 4)
        add("decode", "output head", lambda i: lib.lv_gemv_bf16(h, head, VOCAB, w(i), VOCAB, W, W, x1, W, 1, 1.0, 0), VOCAB * W * 2)
        # -- norms and embedding -----------------------------------------------------------------
        xa, xb, y, vec = f32(STEP, W), gpu.zeros(STEP * W * 4), f32(STEP, W), f32(W)

        def nc(n, first):
            a = pkg.NormConvArgs(pos=pos.value, eps=1e-5, mult=1.0, x_out=xb.value, out=out.value, out_type=pkg.TYPE_F32 if n == 1 else pkg.TYPE_BF16, out_ld=W, width=W, batch=n, plain_w=1)
            if first:
                a.embed, a.embed_ld, a.vocab, a.token_log, a.embed_scale, a.pos = d.value, W, VOCAB, ids.value, 3.0, pos_prompt.value
                a.pair_embed, a.pair_ld, a.pair_buckets, a.pair_mul_prev, a.pair_mul_cur = d.value, W, 20011, 41, 13
            else:
                a.x, a.y, a.y_rows, a.post_w = xa.value, y.value, 1, vec.value
            return C.byref(a)
        for n, phase in ((1, "decode"), (STEP, prompt)):
            add(phase, "embedding of a token and its pair", lambda i: lib.lv_norm_conv(h, nc(n, True)), n * W * (4 + 4 + (4 if n == 1 else 2)))
            add(phase, "norm and residual", lambda i: lib.lv_norm_conv(h, nc(n, False)), n * W * (12 + (4 if n == 1 else 2)))
        gpu.free(d)
        # -- attention ---------------------------------------------------------------------------
        freqs, mults = gpu.upload(np.geomspace(1, 1e-4, ROT // 2)), f32(ROT // 2)
        angles = gpu.zeros(STEP * ROT * 4)
        for n, phase in ((1, "decode"), (STEP, prompt)):
            add(phase, "rotary table, once per step", lambda i: lib.lv_rotary_table(h, angles, freqs, mults, ROT // 2, pos_prompt, n), n * ROT * 4)
        cache, sink, raw = b16(2048, RANK + ROT), f32(H), f32(STEP, q_rows + RANK + ROT)
        w, d = ring(H * (DIM + VDIM) * RANK * 2)
        norm = f32(RANK)

        def latent(i, n, own):
            return pkg.LatentArgs(q=raw.value, q_ld=q_rows + RANK + ROT, dkv=pkg.offset(raw, q_rows * 4).value if own else None, dkv_ld=q_rows + RANK + ROT, heads=H, dim=DIM, rot=ROT,
                                  vdim=VDIM, kv_rank=RANK, scale=0.05, eps=1e-5, kv_norm=norm.value, angles=angles.value, angle_ld=ROT, angle_pairs=ROT // 2, w=w(i).value, w_ld=RANK,
                                  sink=sink.value, window=WINDOW, cache=cache.value, cache_type=pkg.TYPE_BF16, ctx_rows=2048, pos=(pos if n == 1 else pos_prompt).value, out=out.value,
                                  out_type=pkg.TYPE_F32 if n == 1 else pkg.TYPE_BF16, out_ld=H * VDIM)
        sizes = {n: lib.lv_latent_scratch_bytes(h, C.byref(latent(0, n, True)), n, 2048) for n in (1, STEP)}
        scratch = gpu.zeros(max(sizes.values()))
        mat = H * (DIM + VDIM) * RANK * 2
        add("decode", f"latent attention, {CONTEXT} keys", lambda i: lib.lv_latent_attention(h, C.byref(latent(i, 1, True)), scratch, sizes[1], 1, 2048), mat + CONTEXT * (RANK + ROT) * 2)
        pairs = STEP * (CONTEXT - STEP) + STEP * STEP / 2
        add(prompt, f"latent attention, {CONTEXT} keys", lambda i: lib.lv_latent_attention(h, C.byref(latent(i, STEP, True)), scratch, sizes[STEP], STEP, 2048),
            mat + CONTEXT * (RANK + ROT) * 2 + STEP * (q_rows * 4 + H * VDIM * 2), 2.0 * CONTEXT * H * (DIM + VDIM) * RANK + 2.0 * (DIM + ROT + VDIM) * H * pairs)
        kv = gpu.zeros(2048 * H * (DIM + VDIM) * 2)
        add(prompt, "keys and values of the window (part of it)", lambda i: lib.lv_gemm_bf16_window(h, kv, pkg.TYPE_BF16, H * (DIM + VDIM), w(i), H * (DIM + VDIM), RANK, RANK, cache, RANK + ROT,
                                                                                                  2048, pos_prompt, STEP, WINDOW, STEP + WINDOW - 1),
            mat + CONTEXT * (RANK + H * (DIM + VDIM)) * 2, 2.0 * CONTEXT * H * (DIM + VDIM) * RANK)
        gpu.free(d)
        # -- state space -------------------------------------------------------------------------
        raw, conv, vec, heads = f32(STEP, raw_ssm), f32(TAPS, inner + bc), f32(max(inner, inner + bc)), f32(SH)
        states = max(3, int(300e6 // (inner * N * 4)))               # decoding reads another state every time
        S, hist = gpu.zeros(states * inner * N * 4), f32(TAPS, inner + bc)

        def ssm(i, n):
            return pkg.SsmArgs(raw=raw.value, raw_ld=raw_ssm, heads=SH, vdim=P, state=N, groups=G, taps=TAPS, conv_w=conv.value, conv_b=vec.value, dt_bias=heads.value, A_log=heads.value,
                               D=heads.value, norm_w=vec.value, norm_groups=G, eps=1e-5, history=hist.value, S=pkg.offset(S, (i % states) * inner * N * 4).value, pos=pos.value,
                               out=out.value, out_type=pkg.TYPE_F32 if n == 1 else pkg.TYPE_BF16, out_ld=inner)
        sizes = {n: lib.lv_ssm_scratch_bytes(C.byref(ssm(0, n)), n) for n in (1, STEP)}
        scratch2 = gpu.zeros(max(sizes.values()))
        for n, phase in ((1, "decode"), (STEP, prompt)):
            add(phase, "state space", lambda i: lib.lv_ssm(h, C.byref(ssm(i, n)), scratch2, sizes[n], n), 2 * inner * N * 4 + n * (raw_ssm * 4 + inner * (4 if n == 1 else 2)))
    return bench.rows


def run(pkg, args, model_dir, peaks, clocks, out):
    import torch
    z = SIZES[args.workload]
    args.steps = min(args.steps, 64)
    kernels = pkg.load_kernels()
    os.makedirs(model_dir, exist_ok=True)
    cfg, path = config(z), os.path.join(model_dir, args.workload)
    other = args.workload.replace("nuforax", "sonuzen")
    z_other, path_other = bench_sonuzen.SIZES[other], os.path.join(model_dir, other)
    t0 = time.time()
    if not os.path.exists(path + ".done"):
        bench_models.write_folder(path, cfg, tensor_shapes(cfg))
        open(path + ".done", "w").close()
    if not os.path.exists(path_other + ".done"):
        bench_sonuzen.write_folder(path_other, z_other)
        open(path_other + ".done", "w").close()
    print(f"[bench] model folders after {time.time() - t0:.1f} s", file=sys.stderr)
    clocks.start()
    line = {"metric": "nuforax decode tokens/s", "unit": "tokens/s", "n_gpus": 1, "steps": args.steps, "warmup": args.warmup, "higher_is_better": True,
            "data": "synthetic", "dtype": "bf16",
            "config": dict(z, model=args.workload, vocab=VOCAB, dim=DIM, rot_dim=ROT, vdim=VDIM, kv_rank=RANK, window=WINDOW, state=N, ssm_vdim=P, taps=TAPS,
                           l2="weights of a token and kernel rings exceed L2")}
    for name, p, nbytes in (("nuforax", path, active_bytes(cfg)), ("sonuzen", path_other, bench_sonuzen.active_bytes(z_other, bench_sonuzen.config(z_other)["layers"]))):
        m = bench_models.model_times(pkg, torch, p, 4096, STEP, args, kernels)
        sec = m["decode"]["ms_per_token"] * 1e-3
        m["decode"]["weight_bytes_per_token"] = nbytes
        m["decode"]["frac_of_hbm"] = nbytes / sec / (peaks["hbm_gbs"] * 1e9)
        m["prompt"]["TFLOP/s"] = (nbytes - VOCAB * z["width"] * 2) * m["prompt"]["tokens"] / (m["prompt"]["ms"] * 1e-3) / 1e12      # 2 per weight of 2 bytes, head left out
        line[name] = m
    line["kernels"] = kernel_times(pkg, torch, z, peaks) + bench_sonuzen.kernel_times(pkg, torch, z_other, peaks, llama=False)
    line["clocks"] = clocks.stop()
    decode = line["nuforax"]["decode"]
    line["value"] = decode["tokens_per_s"]
    line["ms_per_step"] = decode["ms_per_token"]
    line["gpu_launches"] = decode["launches_per_token"] * args.steps
    line["e2e"] = {"value": decode["e2e_tokens_per_s"], "unit": "tokens/s", "h2d_bytes_per_step": 4, "d2h_bytes_per_step": 4}
    print(json.dumps(line), file=out, flush=True)
