"""Throughput of Sonuzen models beside LLaMA models of equal size (bench.py --workload sonuzen-*).

Random bfloat16 weights in layers of a real model's size; the LLaMA model (q4_0 and q8_0) has the same width, depth, number
of heads and active feed-forward width.  Measured: decoding (device-fed greedy tokens after a prompt), prompts, and every
kernel alone.  A kernel's launches are replayed from one CUDA graph, each reading another copy of its weights from a ring
larger than the 126 MB L2; `roofline` is the larger of bytes / measured copy bandwidth and FLOPs / measured dense bfloat16 rate,
`frac` is roofline time / measured time.
"""
import ctypes as C
import json
import os
import sys
import time

import numpy as np

import bench_models
from bench_models import CONTEXT, STEP, VOCAB

SIZES = {
    # width, query heads of 128, key/value heads, recurrent width, experts, expert width, experts of a token, layers
    "sonuzen-1024": dict(width=1024, heads=8, kv_heads=2, gru=1536, experts=16, ff=512, top=4, layers=8),
    "sonuzen-2048": dict(width=2048, heads=16, kv_heads=4, gru=2560, experts=16, ff=1408, top=4, layers=8),
    "sonuzen-4096": dict(width=4096, heads=32, kv_heads=8, gru=4096, experts=8, ff=5504, top=2, layers=4),
}
DIM, TAPS = 128, 4


def config(z):
    mlp = {"kind": "moe", "expert": {"ff": z["ff"]}, "router": {"experts": z["experts"], "top": z["top"]}}
    attn = {"type": "attention", "mixer": {"heads": z["heads"], "kv_heads": z["kv_heads"], "dim": DIM, "vdim": DIM, "scale": DIM ** -0.5}, "mlp": mlp}
    gru = {"type": "mingru", "mixer": {"width": z["gru"]}, "mlp": mlp}
    return {"architecture": "Sonuzen", "width": z["width"], "vocab": VOCAB, "layers": [gru if i % 4 == 1 else attn for i in range(z["layers"])], "loop": None,
            "canon": {"taps": TAPS}, "norm": {"eps": 1e-5}, "residual_mult": 0.5, "logit_scale": 1.0}


def write_folder(path, z):
    """config.json and a safetensors file of that design with random weights (matrices repeat one random slab)."""
    cfg, rng = config(z), np.random.default_rng(7)
    shapes = {"embed": (VOCAB, z["width"]), "head": (VOCAB, z["width"]), "final.norm": (z["width"],)}
    W = z["width"]
    for i, l in enumerate(cfg["layers"]):
        p, m = f"l{i}.", l["mixer"]
        for n in ("norm1", "norm1b", "norm2", "norm2b"):
            shapes[p + n] = (W,)
        shapes[p + "canon1"] = shapes[p + "canon2"] = (W, TAPS)
        if l["type"] == "attention":
            shapes[p + "mix.q"], shapes[p + "mix.k"], shapes[p + "mix.v"] = (z["heads"] * DIM, W), (z["kv_heads"] * DIM, W), (z["kv_heads"] * DIM, W)
            shapes[p + "mix.q.norm"] = shapes[p + "mix.k.norm"] = (DIM,)
            shapes[p + "mix.r1"] = shapes[p + "mix.r2"] = (z["heads"],)
            shapes[p + "mix.o"] = (W, z["heads"] * DIM)
        else:
            for n in "zxg":
                shapes[p + "mix." + n] = (z["gru"], W)
            shapes[p + "mix.z.b"] = shapes[p + "mix.x.b"] = (z["gru"],)
            shapes[p + "mix.o"] = (W, z["gru"])
        for e in range(z["experts"]):
            shapes[f"{p}mlp.e{e}.gate"] = shapes[f"{p}mlp.e{e}.up"] = (z["ff"], W)
            shapes[f"{p}mlp.e{e}.down"] = (W, z["ff"])
        shapes[p + "mlp.table"] = (VOCAB, z["top"])
    tables = {n: rng.random((VOCAB, z["experts"])).argsort(axis=1)[:, :z["top"]] for n in shapes if n.endswith("table")}
    bench_models.write_folder(path, cfg, shapes, tables)


def active_bytes(z, layers):
    """bfloat16 weight bytes that one decoded token reads."""
    W, total = z["width"], VOCAB * z["width"] * 2 + z["width"] * 2
    for l in layers:
        if l["type"] == "attention":
            total += 2 * W * ((2 * z["heads"] + 2 * z["kv_heads"]) * DIM)
        else:
            total += 2 * W * 4 * z["gru"]
        total += 2 * 3 * W * z["ff"] * z["top"]
    return total


def kernel_times(pkg, torch, z, peaks, llama=True):
    """Every kernel of a layer alone and, with `llama`, its LLaMA counterpart of equal size -> list of rows."""
    W, H, G, gru, ff, top, E = z["width"], z["heads"], z["kv_heads"], z["gru"], z["ff"], z["top"], z["experts"]
    with pkg.Context(0) as gpu:
        bench = bench_models.Kernels(pkg, torch, gpu, peaks)
        lib, h, rng, ring, f32, b16, add = bench.lib, bench.h, bench.rng, bench.ring, bench.f32, bench.b16, bench.add
        pos = gpu.upload(np.array([CONTEXT - 1] * 4, np.uint32))
        pos_prompt = gpu.upload(np.array([CONTEXT - STEP] * 4, np.uint32))
        zero = gpu.upload(np.zeros(4, np.uint32))
        ids = gpu.upload(rng.integers(0, VOCAB, 4096).astype(np.uint32))
        table = gpu.upload(rng.random((VOCAB, E)).argsort(axis=1)[:, :top].astype(np.uint32))
        raw_n = (H + 2 * G) * DIM
        # -- products ------------------------------------------------------------------------
        x1, xT = f32(1, max(W, gru, H * DIM)), b16(STEP * top, max(W, gru, ff, H * DIM))
        out = gpu.zeros(max(STEP * top * max(W, raw_n, 3 * gru, ff), STEP * VOCAB // 8) * 4)
        for name, r, k in (("input projections (attention)", raw_n, W), ("output projection (attention)", W, H * DIM), ("output projection (recurrent)", W, gru)):
            w, d = ring(r * k * 2)
            add("sonuzen", "decode", name, lambda i: lib.lv_gemv_bf16(h, out, r, w(i), r, k, k, x1, k, 1, 1.0, 0), r * k * 2)
            add("sonuzen", f"prompt of {STEP}", name, lambda i: lib.lv_gemm_bf16(h, out, pkg.TYPE_F32, r, w(i), r, k, k, xT, k, STEP, 1.0, 0),
                r * k * 2 + STEP * (k * 2 + r * 4), 2.0 * r * k * STEP)
            gpu.free(d)
        w, d = ring(3 * gru * W * 2)
        bias, state = f32(gru), f32(gru)
        each = gru * W * 2
        add("sonuzen", "decode", "input projections + recurrence", lambda i: lib.lv_gemv_bf16_mingru(
            h, out, w(i), pkg.offset(w(i), each), pkg.offset(w(i), 2 * each), W, gru, W, bias, bias, x1, state, pos), 3 * each)
        add("sonuzen", f"prompt of {STEP}", "input projections (recurrent)", lambda i: lib.lv_gemm_bf16(h, out, pkg.TYPE_F32, 3 * gru, w(i), 3 * gru, W, W, xT, W, STEP, 1.0, 0),
            3 * each + STEP * (W * 2 + 3 * gru * 4), 6.0 * gru * W * STEP)
        gpu.free(d)
        w, d = ring(VOCAB * W * 2)
        add("sonuzen", "decode", "output head", lambda i: lib.lv_gemv_bf16(h, out, VOCAB, w(i), VOCAB, W, W, x1, W, 1, 1.0, 0), VOCAB * W * 2)
        gpu.free(d)
        # -- experts -------------------------------------------------------------------------
        w, d = ring(E * ff * W * 2 * 3)
        mat = E * ff * W * 2

        def expert(i, down):
            a = pkg.ExpertArgs(experts=E, top=top, vocab=VOCAB, table=table.value, token_log=ids.value, pos=pos.value)
            if down:
                a.w0, a.ld, a.rows, a.cols = pkg.offset(w(i), 2 * mat).value, ff, W, ff
            else:
                a.w0, a.w1, a.ld, a.rows, a.cols = w(i).value, pkg.offset(w(i), mat).value, W, ff, W
            return C.byref(a)
        act = f32(top, ff)
        add("sonuzen", "decode", "expert gate/up + SiLU", lambda i: lib.lv_gemv_bf16_expert_gate_up(h, out, ff, expert(i, 0), x1, W, 1), 2 * top * ff * W * 2)
        add("sonuzen", "decode", "expert down", lambda i: lib.lv_gemv_bf16_expert_down(h, out, W, expert(i, 1), act, ff, 1), top * ff * W * 2)
        max_tiles = lib.lv_expert_max_tiles(STEP, top, E)
        index, tiles = gpu.zeros(STEP * top * 4), gpu.zeros(max_tiles * 12)
        job = np.zeros(1, np.dtype([("table", "u8"), ("experts", "u4"), ("top", "u4"), ("index", "u8"), ("tiles", "u8"), ("max_tiles", "u4"), ("unused", "u4")]))
        job[0] = (table.value, E, top, index.value, tiles.value, max_tiles, 0)
        dj = gpu.upload(job)
        add("sonuzen", f"prompt of {STEP}", "expert routing", lambda i: lib.lv_expert_route(h, dj, 1, E, ids, zero, VOCAB, STEP), STEP * top * 12)
        add("sonuzen", f"prompt of {STEP}", "expert gate/up + SiLU", lambda i: lib.lv_gemm_bf16_expert_gate_up(h, out, ff, expert(i, 0), tiles, xT, W, STEP),
            2 * mat + STEP * top * (W + ff) * 2, 4.0 * STEP * top * ff * W)
        add("sonuzen", f"prompt of {STEP}", "expert down", lambda i: lib.lv_gemm_bf16_expert_down(h, out, W, expert(i, 1), tiles, xT, ff, STEP),
            mat + STEP * top * (ff * 2 + W * 4), 2.0 * STEP * top * ff * W)
        gpu.free(d)
        # -- norm / residual / convolution ------------------------------------------------------
        xa, xb, y, vec, conv, hist = f32(STEP, W), gpu.zeros(STEP * W * 4), f32(STEP * top, W), f32(W), f32(TAPS, W), f32(TAPS - 1, W)
        factor = gpu.zeros(STEP * 4)

        def nc(n, rows_per_token):
            a = pkg.NormConvArgs(x=xa.value, pos=pos.value, y=y.value, y_rows=rows_per_token, y_index=index.value if rows_per_token > 1 else None, mult=0.5, eps=1e-5,
                                 post_w=vec.value, x_out=xb.value, row_factor=factor.value, pre_w=vec.value, conv_w=conv.value, history=hist.value, taps=TAPS, out=out.value,
                                 out_type=pkg.TYPE_F32 if n == 1 else pkg.TYPE_BF16, out_ld=W, width=W, batch=n)
            return C.byref(a)
        add("sonuzen", "decode", "norm, residual, norm, convolution", lambda i: lib.lv_norm_conv(h, nc(1, 1)), (4 * W + 2 * TAPS * W + 4 * W) * 4)
        add("sonuzen", f"prompt of {STEP}", "norm, residual, norm, convolution", lambda i: lib.lv_norm_conv(h, nc(STEP, 1)), STEP * W * 14)
        add("sonuzen", f"prompt of {STEP}", "the same after experts", lambda i: lib.lv_norm_conv(h, nc(STEP, top)), STEP * W * (10 + 4 * top))
        # -- attention and recurrence over a prompt ------------------------------------------------
        kc, vc = b16(G * 2048, DIM), b16(G * 2048, DIM)
        hv, qn = f32(H), f32(DIM)
        qkv = f32(STEP, raw_n)

        def gqa(n):
            a = pkg.GqaArgs(qkv=qkv.value, qkv_ld=raw_n, heads=H, kv_heads=G, dim=DIM, vdim=DIM, scale=DIM ** -0.5, eps=1e-5, q_norm=qn.value, k_norm=qn.value,
                            r1=habs.value, r2=habs.value, sink=1, k_cache=kc.value, v_cache=vc.value, cache_type=pkg.TYPE_BF16, ctx_rows=2048,
                            pos=(pos if n == 1 else pos_prompt).value, out=out.value, out_type=pkg.TYPE_F32 if n == 1 else pkg.TYPE_BF16, out_ld=H * DIM)
            return a
        habs = gpu.upload(np.abs(rng.standard_normal(H)).astype(np.float32) * 0.3)
        nbytes = lib.lv_gqa_scratch_bytes(h, C.byref(gqa(1)), STEP, 2048)
        scratch = gpu.zeros(nbytes)
        add("sonuzen", "decode", f"attention, {CONTEXT} keys", lambda i: lib.lv_attention_gqa(h, C.byref(gqa(1)), scratch, nbytes, 1, CONTEXT, 1), 2 * CONTEXT * G * DIM * 2)
        add("sonuzen", f"prompt of {STEP}", "key norm + append", lambda i: lib.lv_qk_norm_append(h, C.byref(gqa(STEP)), STEP), STEP * 2 * G * DIM * 6)
        pairs = STEP * (CONTEXT - STEP) + STEP * STEP / 2
        add("sonuzen", f"prompt of {STEP}", f"attention, {CONTEXT} keys", lambda i: lib.lv_attention_gqa(h, C.byref(gqa(STEP)), scratch, nbytes, STEP, CONTEXT, 0),
            2 * CONTEXT * G * DIM * 2 + STEP * H * DIM * 6, 4.0 * DIM * H * pairs)
        rawz = f32(STEP, 3 * gru)
        add("sonuzen", f"prompt of {STEP}", "recurrence scan", lambda i: lib.lv_mingru_scan(h, out, pkg.TYPE_BF16, gru, rawz, 3 * gru, gru, bias, bias, state, pos, STEP), STEP * gru * 14)
        if not llama:
            return bench.rows
        # -- LLaMA of equal size ----------------------------------------------------------------
        act_ff = ff * top
        llama_ff = (act_ff + 255) // 256 * 256
        norm = f32(W)
        x64 = f32(64, llama_ff)
        rope = gpu.alloc(2048 * DIM * 4)
        pkg.check(lib.lv_rope_table_build(h, rope, 2048, DIM))
        lk, lv_ = gpu.zeros(2048 * W * 2), gpu.zeros(2048 * W * 2)
        lscratch = gpu.zeros(lib.lv_attention_scratch_bytes(W // DIM, DIM, 2048, 64))
        split = gpu.alloc(lib.lv_act_split_bytes(max(W, llama_ff), 64))
        for wt, bpb in ((pkg.TYPE_Q4_0, 18), (pkg.TYPE_Q8_0, 34)):
            name = "llama q4_0" if bpb == 18 else "llama q8_0"
            size = lambda r, k: r * k // 32 * bpb

            def quant(r, k, n):
                w, d = ring(n * size(r, k))
                return w, d
            for label, r, k, n in (("input projections (attention)", W, W, 3), ("output projection (attention)", W, W, 1), ("gate/up + SiLU", llama_ff, W, 2), ("down", W, llama_ff, 1),
                                   ("output head", VOCAB, W, 1)):
                w, d = quant(r, k, n)
                s = size(r, k)
                if n == 3:
                    one = lambda i: lib.lv_norm_qkv_kvappend(h, out, lk, lv_, w(i), pkg.offset(w(i), s), pkg.offset(w(i), 2 * s), wt, x64, norm, pos, W, W, 1, 2048)
                    many = lambda i: lib.lv_gemm_tc_qkv_kvappend(h, out, lk, lv_, w(i), pkg.offset(w(i), s), pkg.offset(w(i), 2 * s), wt, split, pos, W, W, 64, 2048)
                elif n == 2:
                    one = lambda i: lib.lv_norm_gate_up_silu(h, out, w(i), pkg.offset(w(i), s), wt, x64, norm, r, k, 1)
                    many = lambda i: lib.lv_gemm_tc_silu(h, out, w(i), pkg.offset(w(i), s), wt, split, r, k, 64)
                elif label == "output head":
                    one, many = (lambda i: lib.lv_norm_gemv(h, out, w(i), wt, x64, norm, r, k, 1)), None
                else:
                    one = lambda i: lib.lv_gemv(h, out, w(i), wt, x64, r, k, 1, 1)
                    many = lambda i: lib.lv_gemm_tc(h, out, w(i), wt, split, r, k, 64, 1)
                add(name, "decode", label, lambda i: one(i), n * s)
                if many:
                    pkg.check(lib.lv_act_split_f16(h, split, x64, None, k, 64))
                    add(name, "prompt of 64", label, lambda i: many(i), n * s + 64 * (k + n * r) * 4, 2.0 * n * r * k * 64)
                gpu.free(d)
        add("llama", "decode", f"attention, {CONTEXT} keys", lambda i: lib.lv_attention_fused(h, out, x64, lk, lv_, pos, rope, lscratch, W // DIM, DIM, 1024, 1), 2 * CONTEXT * W * 2)
        pos64 = gpu.upload(np.array([CONTEXT - 64] * 4, np.uint32))
        add("llama", "prompt of 64", f"attention, {CONTEXT} keys", lambda i: lib.lv_attention_fused(h, out, x64, lk, lv_, pos64, rope, lscratch, W // DIM, DIM, 1024, 64),
            2 * CONTEXT * W * 2 + 64 * W * 8, 4.0 * W * 64 * (CONTEXT - 32))
        add("llama", "decode", "norm", lambda i: lib.lv_norm_f32(h, out, x64, norm, W, 1), 3 * W * 4)
        add("llama", "prompt of 64", "norm + activation split", lambda i: lib.lv_act_split_f16(h, split, x64, norm, W, 64), 64 * W * 8)
    return bench.rows


def run(pkg, args, model_dir, peaks, clocks, out):
    import torch
    z = SIZES[args.workload]
    args.steps = min(args.steps, 64)
    kernels = pkg.load_kernels()
    os.makedirs(model_dir, exist_ok=True)
    path = os.path.join(model_dir, args.workload)
    if not os.path.exists(path + ".done"):
        t0 = time.time()
        write_folder(path, z)
        open(path + ".done", "w").close()
        print(f"[bench] wrote {path} in {time.time() - t0:.1f} s", file=sys.stderr)
    clocks.start()
    line = {"metric": "sonuzen decode tokens/s", "unit": "tokens/s", "n_gpus": 1, "steps": args.steps, "warmup": args.warmup, "higher_is_better": True,
            "data": "synthetic", "dtype": "bf16", "config": dict(z, model=args.workload, vocab=VOCAB, head_dim=DIM, taps=TAPS, l2="weights of a token and kernel rings exceed L2")}
    ours = bench_models.model_times(pkg, torch, path, 4096, STEP, args, kernels)
    nbytes = active_bytes(z, config(z)["layers"])
    sec = ours["decode"]["ms_per_token"] * 1e-3
    ours["decode"]["weight_bytes_per_token"] = nbytes
    ours["decode"]["frac_of_hbm"] = nbytes / sec / (peaks["hbm_gbs"] * 1e9)
    flops = (nbytes - VOCAB * z["width"] * 2) * ours["prompt"]["tokens"]             # 2 per weight of 2 bytes, head left out
    ours["prompt"]["TFLOP/s"] = flops / (ours["prompt"]["ms"] * 1e-3) / 1e12
    line["sonuzen"] = ours
    ff = (z["ff"] * z["top"] + 255) // 256 * 256
    for wt, name, bpb in ((pkg.TYPE_Q4_0, "llama_q4_0", 18), (pkg.TYPE_Q8_0, "llama_q8_0", 34)):
        p = os.path.join(model_dir, f"llama_{z['width']}_L{z['layers']}_{name}.ggjt")
        if not os.path.exists(p):
            if not pkg.load_host().llava_synth_write(os.fsencode(p), z["width"], z["width"] // DIM, z["layers"], ff, VOCAB, wt, 1234, 0):
                raise RuntimeError("cannot write " + p)
        m = bench_models.model_times(pkg, torch, p, 0, 64, args, kernels)
        b = (z["layers"] * (4 * z["width"] ** 2 + 3 * ff * z["width"]) + VOCAB * z["width"]) * bpb // 32
        m["decode"]["weight_bytes_per_token"] = b
        m["decode"]["frac_of_hbm"] = b / (m["decode"]["ms_per_token"] * 1e-3) / (peaks["hbm_gbs"] * 1e9)
        line[name] = m
    line["kernels"] = kernel_times(pkg, torch, z, peaks)
    line["clocks"] = clocks.stop()
    line["value"] = ours["decode"]["tokens_per_s"]
    line["ms_per_step"] = ours["decode"]["ms_per_token"]
    line["gpu_launches"] = ours["decode"]["launches_per_token"] * args.steps
    line["e2e"] = {"value": ours["decode"]["e2e_tokens_per_s"], "unit": "tokens/s", "h2d_bytes_per_step": 4, "d2h_bytes_per_step": 4}
    print(json.dumps(line), file=out, flush=True)
