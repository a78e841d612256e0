"""Sonuzen models end to end on the GPU: the session, its caches and states, the command line, the trace runner and the
server against the plain implementation (float64)."""
import json
import os
import struct
import subprocess

import numpy as np
import pytest

import sonuzen_models as sm
import sonuzen_plain as sp
from conftest import ROOT, load_pkg
from hybrid_harness import LIMIT, Model, cached_models, feed, frame_records, greedy

pytestmark = pytest.mark.gpu
pkg = load_pkg()


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    yield from cached_models(sm, tmp_path_factory)


CUTS = {"whole": [150], "token by token": [1] * 150, "pairs": [2] * 75, "sizes": [1, 2, 3, 61, 1, 1, 2, 64, 5, 10], "prompt and decoding": [131] + [1] * 19}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(sm.CONFIGS))
def test_logits_do_not_depend_on_the_portions(models, name, dtype):
    m = models(name)
    tokens = m.tokens(150)
    want = m.plain.forward(tokens)
    for cuts in CUTS.values():
        s = m.session(dtype)
        far = sm.distance(feed(s, m, tokens, cuts), want)
        s.close()
        assert far.max() < LIMIT[dtype], (cuts[:4], int(far.argmax()), far.max())


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_steps_shorter_than_the_prompt(models, dtype):
    """A portion that exceeds the step size is evaluated in several recorded steps."""
    m = models("mixed")
    tokens = m.tokens(100, 5)
    want = m.plain.forward(tokens)
    for batch in (1, 2, 7, 33):
        s = m.session(dtype)
        assert s.set_max_batch(batch)
        assert sm.distance(feed(s, m, tokens, [90, 1, 9]), want).max() < LIMIT[dtype]
        s.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_interleaved_requests_and_reused_memory(models, dtype):
    """Requests of unequal length that take turns, end and make room for others give what each gives alone."""
    m = models("mixed")
    requests = [m.tokens(n, 10 + n) for n in (3, 90, 41, 1, 130)]
    want = [m.plain.forward(r) for r in requests]
    live, done = {}, {}
    order = [0, 1, 2, 1, 0, 2, 3, 1, 4, 2, 4]
    rng = np.random.default_rng(2)
    turn = 0
    while len(done) < len(requests):
        i = order[turn % len(order)]
        turn += 1
        if i in done:
            continue
        s, at, rows = live.setdefault(i, (m.session(dtype), 0, []))
        n = min(int(rng.integers(1, 40)), len(requests[i]) - at)
        for t in requests[i][at:at + n]:
            s.push_token(t)
        rows.append(s.evaluate_pending(range(at, at + n), m.vocab))
        live[i] = (s, at + n, rows)
        if at + n == len(requests[i]):
            s.close()
            done[i] = np.concatenate(rows)
    for i, r in done.items():
        assert sm.distance(r, want[i]).max() < LIMIT[dtype], i


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_rewound_sessions_start_over(models, dtype):
    m = models("looped")
    a, b = m.tokens(60, 1), m.tokens(30, 2)
    s = m.session(dtype)
    feed(s, m, a, [50, 10])
    s.rewind(20)
    assert s.tokens() == a[:20] and s.tokens_in_gpu() == 0        # a recurrent state cannot be taken back: evaluated again
    for t in b:
        s.push_token(t)
    got = s.evaluate_pending(range(20, 50), m.vocab)
    assert sm.distance(got, m.plain.forward(a[:20] + b)[20:]).max() < LIMIT[dtype]
    s.rewind(0)
    assert sm.distance(feed(s, m, b, [1, 29]), m.plain.forward(b)).max() < LIMIT[dtype]
    assert s.set_text("".join(f"<{t}>" for t in b + a[:5]))        # shares all that is evaluated: continues from there
    assert s.tokens_in_gpu() == 30
    assert sm.distance(s.evaluate_pending([34], m.vocab), m.plain.forward(b + a[:5])[-1:]).max() < LIMIT[dtype]
    assert s.set_text(f"<{b[0]}><{b[1]}>") and s.tokens_in_gpu() == 0
    s.close()


def test_greedy_generation_three_ways(models):
    m = models("no_loop")
    prompt = m.tokens(23, 8)
    want, lead = greedy(m.plain, prompt, 40)
    assert lead > 1e-4                                            # no ties that rounding could decide
    s = m.session("float32")
    for t in prompt:
        s.push_token(t)
    got = []
    for _ in range(40):
        got.append(s.predict_next_token())
        assert s.push_token(got[-1])
    assert got == want
    s.close()
    s = m.session("float32")
    for t in prompt:
        s.push_token(t)
    first = s.predict_next_token()
    s.push_token(first)
    assert [first] + s.generate_greedy_on_device(39) == want
    s.close()
    ids = os.path.join(m.path, "ids.txt")
    with open(ids, "w") as f:
        f.write(" ".join(map(str, prompt)))
    for extra in ([], ["--on-device"], ["--prompt-batch", "8"], ["--context", "4096"]):
        out = subprocess.run([os.path.join(ROOT, "llama-vulkan_b200", "vulkan_llama"), "-m", m.path, "--greedy", "--tokens", ids, "--n-predict", "40",
                              "--dtype", "float32"] + extra, capture_output=True, text=True, timeout=120)
        assert out.returncode == 0, out.stderr
        assert out.stdout.strip() == "".join(f"<{t}>" for t in want)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding(models, dtype):
    """Several hundred tokens generated on the device, checked in one piece against the plain implementation."""
    m = models("mixed")
    prompt, n = m.tokens(5, 3), 400
    s = m.session(dtype)
    for t in prompt:
        s.push_token(t)
    s.push_token(s.predict_next_token())
    s.generate_greedy_on_device(n)
    tokens = s.tokens()
    assert len(tokens) == len(prompt) + 1 + n
    z = m.plain.forward(tokens)
    chosen = z[np.arange(len(prompt) - 1, len(tokens) - 1), tokens[len(prompt):]]
    behind = (z[len(prompt) - 1:-1].max(axis=1) - chosen) / np.abs(z).max()
    assert behind.max() < LIMIT[dtype]                            # every choice is the largest logit up to rounding
    got = s.evaluate_pending([len(tokens) - 1], m.vocab)
    assert sm.distance(got, z[-1:]).max() < LIMIT[dtype]
    s.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_session_longer_than_the_default(tmp_path, dtype):
    cfg = sm.config(64, 40, [sm.attention(4, 2, 32, 32, mlp=sm.moe(32, 2, 1)), sm.mingru(32)], taps=4)
    m = Model(tmp_path, cfg, sm)
    tokens = m.tokens(2500)
    want = m.plain.forward(tokens)
    s = m.session(dtype, 2600)
    got = feed(s, m, tokens, [2047, 2, 1, 430, 18, 1, 1])
    assert sm.distance(got, want).max() < LIMIT[dtype]
    s.close()
    with pytest.raises(RuntimeError):
        m.session(dtype, 1 << 30)
    s = m.session(dtype)                                           # the default holds 2048 tokens
    for t in tokens[:2048]:
        assert s.push_token(t)
    assert not s.push_token(tokens[2048])
    s.close()
    m.close()


def test_sampled_generation_is_reproducible(models):
    m = models("looped")
    prompt = m.tokens(12, 4)

    def run(seed):
        s = m.ctx("bfloat16").session()
        s.set_seed(seed)
        for t in prompt:
            s.push_token(t)
        out = []
        for _ in range(30):
            out.append(s.predict_next_token())
            assert out[-1] < m.vocab and s.push_token(out[-1])
        s.close()
        return out
    assert run(7) == run(7) != run(8)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_snapshot_and_restore(models, dtype, tmp_path):
    m = models("mixed")
    tokens = m.tokens(80, 21)
    want = m.plain.forward(tokens)
    s = m.session(dtype)
    feed(s, m, tokens[:50], [49, 1])
    path = str(tmp_path / "state")
    assert s.snapshot(path) == 0
    s.close()
    t = m.session(dtype, 300)                                      # another capacity
    assert t.restore(path) == 0
    assert t.tokens() == tokens[:50] and t.tokens_in_gpu() == 50
    for x in tokens[50:]:
        t.push_token(x)
    assert sm.distance(t.evaluate_pending(range(50, 80), m.vocab), want[50:]).max() < LIMIT[dtype]
    with open(path, "ab") as f:
        f.write(b"x")
    assert t.restore(path) != 0
    t.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("n", [1, 30])
def test_frames_hold_the_stream_after_every_layer_run(models, dtype, n, tmp_path):
    m = models("mixed")
    tokens, layers = m.tokens(n, 6), []
    m.plain.forward(tokens, layers)
    s = m.session(dtype)
    assert s.set_options(1) == 0
    for t in tokens:
        s.push_token(t)
    s.predict_next_token()
    path = str(tmp_path / "frame")
    assert s.save_frame(path) == 0
    s.close()
    seen = frame_records(path)
    assert [k for k, _ in seen] == [f"step.run.{i:04d}.residual" for i in range(len(layers))]
    for (name, got), want in zip(seen, layers):
        err = np.linalg.norm(got[:n] - want) / np.linalg.norm(want)
        assert err < (1e-5 if dtype == "float32" else 2e-2), (name, err)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_runner(models, dtype, tmp_path):
    m = models("one_tap")
    a, b = m.tokens(40, 1), m.tokens(9, 2)
    steps = [("a", a[:30], [0, 7, 29], []), ("b", b[:1], [0], []), ("a", a[30:31], [], []), ("b", b[1:], [7, 2], ["b"]), ("a", a[31:], [8], ["a"]), ("b", a[:3], [2], ["b"])]
    text = "".join(json.dumps({"step": i, "entries": [{"id": r, "tokens": t, "want": w}], "end": e}) + "\n" for i, (r, t, w, e) in enumerate(steps))
    run = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", m.path, "--dtype", dtype, "--out", str(tmp_path), "--max-tokens", "50"],
                         input=text, capture_output=True, text=True, timeout=300)
    assert run.returncode == 0, run.stderr
    assert [x for x in run.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(len(steps))]
    pa, pb, pc = m.plain.forward(a), m.plain.forward(b), m.plain.forward(a[:3])
    want = {0: pa[[0, 7, 29]], 1: pb[[0]], 3: pb[[8, 3]], 4: pa[[39]], 5: pc[[2]]}
    assert sorted(os.listdir(tmp_path)) == [f"{i}.f32" for i in sorted(want)]
    for i, w in want.items():
        got = np.fromfile(tmp_path / f"{i}.f32", np.float32).reshape(-1, m.vocab)
        assert sm.distance(got, w).max() < LIMIT[dtype]
    bad = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", m.path, "--dtype", dtype, "--out", str(tmp_path), "--max-tokens", "50"],
                         input=json.dumps({"step": 0, "entries": [{"id": "x", "tokens": [m.vocab], "want": []}], "end": []}) + "\n",
                         capture_output=True, text=True, timeout=300)
    assert bad.returncode == 1


def test_the_server_serves_the_model(models):
    m = models("no_loop")
    prompt = m.tokens(9, 3)
    want, lead = greedy(m.plain, prompt, 6)
    assert lead > 1e-4
    C = pkg.Client
    with pkg.Server(m.ctx("float32"), deterministic=True) as server:
        clients = [C(server.port) for _ in range(2)]
        for c in clients:
            op, data = c.call(C.NEW_SESSION)
            c.sid = struct.unpack("<I", data[:4])[0]
            for t in prompt:
                c.call(C.ADD_TOKEN, struct.pack("<II", c.sid, t))
        for c in clients:
            got = []
            for _ in range(6):
                op, data = c.call(C.TICK, struct.pack("<I", c.sid))
                assert op == C.NEW_TOKEN
                got.append(struct.unpack("<III", data)[1])
            assert got == want
            c.call(C.KILL_SESSION, struct.pack("<I", c.sid))
            c.close()


def test_sessions_of_this_design_do_not_form_groups(models):
    m = models("no_loop")
    a, b = m.session("bfloat16"), m.session("bfloat16")
    with pytest.raises(RuntimeError):
        pkg.SessionGroup(m.ctx("bfloat16"), [a, b])
    a.close()
    b.close()


@pytest.mark.parametrize("damage", ["missing", "shape", "type"])
def test_damaged_folders_are_refused(tmp_path, damage):
    cfg = sm.CONFIGS["one_tap"]
    t = sm.tensors(cfg, 1)
    if damage == "missing":
        del t["l1.mix.r2"]
    elif damage == "shape":
        t["l0.mix.o"] = t["l0.mix.o"][:, :-1]
    else:
        t["l0.mlp.table"] = t["l0.mlp.table"].astype(np.float32)
    sp.write_model(str(tmp_path), cfg, t)
    with pytest.raises(RuntimeError):
        pkg.HostContext(str(tmp_path), 0)
