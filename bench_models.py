"""Pieces of the model workloads of bench.py: writing random model folders, timing kernels from graphs, decoding and prompts of a model."""
import ctypes as C
import json
import os
import time

import numpy as np

VOCAB, CONTEXT, PROMPT, STEP = 32000, 1024, 2048, 512


def write_folder(path, cfg, shapes, tables=None):
    """config.json and a safetensors file with random bfloat16 tensors of the given shapes (matrices repeat one random slab); `tables`
    holds the int32 tensors."""
    rng, tables = np.random.default_rng(7), tables or {}
    head, at = {}, 0
    for name, s in shapes.items():
        n = int(np.prod(s)) * (4 if name in tables else 2)
        head[name] = {"dtype": "I32" if name in tables else "BF16", "shape": list(s), "data_offsets": [at, at + n]}
        at += n
    text = json.dumps(head).encode()
    slab = (rng.standard_normal(1 << 22).astype(np.float32) * 0.02).view(np.uint32) >> 16
    slab = slab.astype(np.uint16)
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    with open(os.path.join(path, "model.safetensors"), "wb") as f:
        f.write(len(text).to_bytes(8, "little") + text)
        for name, s in shapes.items():
            if name in tables:
                f.write(tables[name].astype(np.int32).tobytes())
                continue
            n, off = int(np.prod(s)), int(rng.integers(0, 1 << 20))
            while n:
                k = min(n, slab.size - off)
                f.write(slab[off:off + k].tobytes())
                n -= k
                off = 0


class Timer:
    def __init__(self, pkg, gpu, torch):
        self.pkg, self.gpu, self.torch, self.lib, self.h = pkg, gpu, torch, gpu.lib, gpu.handle
        self.stream = torch.cuda.ExternalStream(self.lib.lv_ctx_stream(self.h), device=0)

    def __call__(self, launch, iters=40):
        """Seconds per launch; launch(i) enqueues the i-th one."""
        pkg, lib, h, torch = self.pkg, self.lib, self.h, self.torch
        for i in range(3):
            launch(i)
        self.gpu.sync()
        graph = C.c_void_p()
        pkg.check(lib.lv_graph_begin_capture(h))
        for i in range(iters):
            launch(i)
        pkg.check(lib.lv_graph_end_capture(h, C.byref(graph)))
        best = []
        for _ in range(4):
            e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            e0.record(self.stream)
            pkg.check(lib.lv_graph_launch(h, graph))
            e1.record(self.stream)
            self.gpu.sync()
            best.append(e0.elapsed_time(e1) * 1e-3 / iters)
        pkg.check(lib.lv_graph_destroy(graph))
        return sorted(best[1:])[1]


class Kernels:
    """Kernels of a layer alone -> rows of a table.  A kernel's launches read a ring of weight copies larger than the 126 MB L2; `frac` is
    max(bytes / measured copy bandwidth, FLOPs / measured dense bfloat16 rate) / time."""

    def __init__(self, pkg, torch, gpu, peaks):
        self.pkg, self.gpu, self.lib, self.h = pkg, gpu, gpu.lib, gpu.handle
        self.t, self.rng, self.rows = Timer(pkg, gpu, torch), np.random.default_rng(3), []
        self.hbm, self.tflops = peaks["hbm_gbs"] * 1e9, peaks["bf16_tflops"] * 1e12

    def ring(self, nbytes):
        """copies of a random block of nbytes, more than 400 MB together"""
        n = max(3, int(400e6 // nbytes) + 1)
        stride = (nbytes + 255) // 256 * 256
        d = self.gpu.alloc(n * stride)
        slab = ((self.rng.standard_normal(1 << 20).astype(np.float32) * 0.02).view(np.uint32) >> 16).astype(np.uint16)
        host = np.resize(slab, nbytes // 2 + 1)
        for i in range(n):
            self.pkg.check(self.lib.lv_upload(self.h, self.pkg.offset(d, i * stride), host.ctypes.data_as(C.c_void_p), nbytes))
        return lambda i: self.pkg.offset(d, (i % n) * stride), d

    def add(self, model, phase, name, launch, nbytes, flops=0.0):
        """launch(i) enqueues the i-th launch and returns its status"""
        sec = self.t(lambda i: self.pkg.check(launch(i)))
        roof = max(nbytes / self.hbm, flops / self.tflops)
        self.rows.append({"model": model, "phase": phase, "kernel": name, "us": round(sec * 1e6, 2), "GB/s": round(nbytes / sec / 1e9),
                          "TFLOP/s": round(flops / sec / 1e12, 1), "frac": round(roof / sec, 3)})

    def f32(self, *s):
        return self.gpu.upload(self.rng.standard_normal(s).astype(np.float32))

    def b16(self, *s):
        return self.gpu.upload(((self.rng.standard_normal(s).astype(np.float32)).view(np.uint32) >> 16).astype(np.uint16))


def model_times(pkg, torch, path, max_context, prompt_step, args, kernels):
    """Decoding and prompt throughput of one model."""
    ctx = pkg.HostContext(path, 0)
    lv = C.c_void_p(ctx.lib.llava_context_lv(ctx.handle))
    stream = torch.cuda.ExternalStream(kernels.lv_ctx_stream(lv), device=0)
    tokens = [int(x) for x in np.random.default_rng(4321).integers(3, VOCAB, PROMPT)]

    def timed_prompt(n):
        s = ctx.session(max_context)
        s.set_deterministic(True)
        assert s.set_max_batch(prompt_step)
        best = []
        for _ in range(4):                                        # the first pass records the steps
            s.rewind(0)
            for x in tokens[:n]:
                assert s.push_token(x)
            pkg.check(kernels.lv_stream_sync(lv, 0))
            e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            e0.record(stream)
            assert s.start_next_token_prediction()
            e1.record(stream)
            tok = s.finish_next_token_prediction()
            best.append(e0.elapsed_time(e1) * 1e-3)
        return s, tok, sorted(best[1:])[1]

    s, _, sec = timed_prompt(PROMPT if max_context > PROMPT else 1984)
    s.close()
    n_prompt = PROMPT if max_context > PROMPT else 1984
    prompt = {"tokens": n_prompt, "step": prompt_step, "ms": sec * 1e3, "tokens_per_s": n_prompt / sec}
    s, tok, _ = timed_prompt(CONTEXT - args.steps // 2 - args.warmup - 2)
    assert s.push_token(tok)
    s.generate_greedy_on_device(args.warmup)
    runs = []
    start = len(s.tokens())
    e2e = []
    for _ in range(3):
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        e0.record(stream)
        s.enqueue_greedy_on_device(args.steps)
        e1.record(stream)
        s.collect_greedy_on_device()
        runs.append(e0.elapsed_time(e1) * 1e-3 / args.steps)
    launches = s.step_kernel_launches()
    for _ in range(2):                                            # through the public calls, host in the loop
        t0 = time.perf_counter()
        for _ in range(args.steps):
            tok = s.predict_next_token()
            assert s.push_token(tok)
        e2e.append((time.perf_counter() - t0) / args.steps)
    sec = sorted(runs)[1]
    decode = {"context": [start, start + 3 * args.steps], "ms_per_token": sec * 1e3, "tokens_per_s": 1 / sec, "e2e_tokens_per_s": 1 / min(e2e), "launches_per_token": launches}
    s.close()
    ctx.close()
    return {"prompt": prompt, "decode": decode}
