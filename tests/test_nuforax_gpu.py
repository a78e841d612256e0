"""Nuforax models end to end on the GPU: the session, its caches and states, the command line, the trace runner and the server
against the plain implementation (float64)."""
import copy
import json
import os
import struct
import subprocess

import numpy as np
import pytest

import nuforax_models as nm
import sonuzen_plain as sp
from conftest import ROOT, load_pkg
from hybrid_harness import LIMIT, Model, cached_models, feed, frame_records, greedy

pytestmark = pytest.mark.gpu
pkg = load_pkg()
DTYPES = ["float32", "bfloat16"]


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    yield from cached_models(nm, tmp_path_factory)


def check(m, dtype, tokens, rows, got, want=None):
    """Logits of `rows` of a sequence against the plain ones; sensitive positions of bfloat16 get what rounding alone makes of them."""
    want = m.plain.forward(tokens) if want is None else want
    far, limit = nm.distance(got, want[rows]), np.full(len(rows), LIMIT[dtype])
    if dtype == "bfloat16" and far.max() >= LIMIT[dtype]:
        limit = np.maximum(limit, 3 * nm.rounding(m.cfg, m.plain.w, tokens)[rows])
    assert (far < limit).all(), (int((far / limit).argmax()), far[(far / limit).argmax()], (far / limit).max())
    assert np.median(far) < LIMIT[dtype] / 2


CUTS = {"whole": [170], "token by token": [1] * 170, "pairs": [2] * 85, "sizes": [1, 2, 3, 61, 1, 1, 2, 64, 5, 30], "prompt and decoding": [141] + [1] * 29,
        "threes to sixes": [3, 4, 5, 6] * 9 + [8]}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(nm.CONFIGS))
def test_logits_do_not_depend_on_the_portions(models, name, dtype):
    m = models(name)
    tokens = m.tokens(170)
    want = m.plain.forward(tokens)
    for cuts in CUTS.values():
        s = m.session(dtype)
        check(m, dtype, tokens, range(170), feed(s, m, tokens, cuts), want)
        s.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_steps_shorter_than_the_prompt(models, dtype):
    """A portion that exceeds the step size is evaluated in several recorded steps; the step size changes while a session lives."""
    m = models("mixed")
    tokens = m.tokens(100, 5)
    want = m.plain.forward(tokens)
    for batch in (1, 2, 7, 33):
        s = m.session(dtype)
        assert s.set_max_batch(batch)
        check(m, dtype, tokens, range(80), feed(s, m, tokens[:80], [70, 1, 9]), want)
        assert s.set_max_batch(batch + 5)                         # new step buffers: the token before the next one is still known
        for t in tokens[80:]:
            s.push_token(t)
        check(m, dtype, tokens, range(80, 100), s.evaluate_pending(range(80, 100), m.vocab), want)
        s.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_interleaved_requests_and_reused_memory(models, dtype):
    """Requests of unequal length that take turns, end and make room for others give what each gives alone."""
    m = models("mixed")
    requests = [m.tokens(n, 10 + n) for n in (3, 90, 41, 1, 130)]
    live, done = {}, {}
    rng = np.random.default_rng(2)
    turn = 0
    while len(done) < len(requests):
        i = [0, 1, 2, 1, 0, 2, 3, 1, 4, 2, 4][turn % 11]
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
        check(m, dtype, requests[i], range(len(r)), r)


@pytest.mark.parametrize("dtype", DTYPES)
def test_rewound_sessions_start_over(models, dtype):
    m = models("mixed")
    a, b = m.tokens(60, 1), m.tokens(30, 2)
    s = m.session(dtype)
    feed(s, m, a, [50, 10])
    s.rewind(20)
    assert s.tokens() == a[:20] and s.tokens_in_gpu() == 0
    for t in b:
        s.push_token(t)
    got = s.evaluate_pending(range(20, 50), m.vocab)
    check(m, dtype, a[:20] + b, range(20, 50), got)
    s.rewind(0)
    check(m, dtype, b, range(30), feed(s, m, b, [1, 29]))
    s.close()


def edge_model(folder, size):
    """A single attention layer of nearly equal weights and no sink to speak of: every key of the window has its part in every output."""
    cfg = nm.config(48, 64, [nm.latent(2, 16, 4, 16, 24, size, scale=0.02)], mul_prev=0, mul_cur=1)
    m = Model(folder, cfg, nm)
    t = dict(m.plain.w)
    t["l0.mix.sink"] = np.full(2, -20.0)
    sp.write_model(m.path, cfg, {k: v.astype(np.float32) for k, v in t.items()})
    m.plain = nm.plain(cfg, t)
    return m


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("size", [1, 2, 15, 64, 65])
def test_a_change_outside_the_window_changes_nothing(tmp_path, dtype, size):
    """Token 40 differs: the positions up to size - 1 later see it, those after do not, in a prompt, in portions and decoded."""
    m = edge_model(tmp_path, size)
    a = m.tokens(150, 3)
    b = list(a)
    b[40] = (a[40] + 17) % m.vocab
    want = m.plain.forward(a)
    for cuts in ([150], [41 + size // 2, 1, 1, 109 - 2 - size // 2], [30] + [1] * 120):
        s, r = m.session(dtype), m.session(dtype)
        za, zb = feed(s, m, a, cuts), feed(r, m, b, cuts)
        s.close()
        r.close()
        check(m, dtype, a, range(150), za, want)
        same = np.abs(za - zb).max(axis=1) == 0
        assert same[:40].all() and not same[40:40 + size].any() and same[40 + size:].all()
    m.close()


def test_greedy_generation_three_ways(models):
    m = models("mixed")
    for seed in range(20):
        prompt = m.tokens(23, seed)
        want, lead = greedy(m.plain, prompt, 40)
        if lead > 1e-4:                                           # no ties that rounding could decide
            break
    assert lead > 1e-4
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


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mixed", "recurrent"])
def test_long_decoding(models, dtype, name):
    """Several hundred tokens generated on the device, checked in one piece against the plain implementation."""
    m = models(name)
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
    assert behind.max() < 2 * LIMIT[dtype]                        # every choice is the largest logit up to rounding
    got = s.evaluate_pending([len(tokens) - 1], m.vocab)
    check(m, dtype, tokens, range(len(tokens) - 1, len(tokens)), got, z)
    s.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_session_longer_than_the_default(tmp_path, dtype):
    cfg = nm.config(64, 40, [nm.latent(4, 32, 8, 24, 40, 700), nm.mamba2(4, 16, 24, 2, 4, 2, ff=48), nm.latent(2, 16, 8, 16, 40, 1300, kv_from=0)])
    m = Model(tmp_path, cfg, nm)
    tokens = m.tokens(2500)
    want = m.plain.forward(tokens)
    s = m.session(dtype, 2600)
    got = feed(s, m, tokens, [2047, 2, 1, 430, 18, 1, 1])
    check(m, dtype, tokens, range(2500), got, want)
    s.close()
    m.close()


def test_sampled_generation_is_reproducible(models):
    m = models("odd_sizes")
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


@pytest.mark.parametrize("dtype", DTYPES)
def test_snapshot_and_restore(models, dtype, tmp_path):
    m = models("mixed")
    tokens = m.tokens(80, 21)
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
    check(m, dtype, tokens, range(50, 80), t.evaluate_pending(range(50, 80), m.vocab))      # (the first of them pairs with a restored token)
    with open(path, "ab") as f:
        f.write(b"x")
    assert t.restore(path) != 0
    t.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n", [1, 30])
def test_frames_hold_the_stream_after_every_layer(models, dtype, n, tmp_path):
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


@pytest.mark.parametrize("dtype", DTYPES)
def test_trace_runner(models, dtype, tmp_path):
    m = models("odd_sizes")
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
        assert nm.distance(got, w).max() < LIMIT[dtype]


def test_the_server_serves_the_model(models):
    m = models("one_rotation_each")
    for seed in range(20):
        prompt = m.tokens(9, seed)
        want, lead = greedy(m.plain, prompt, 6)
        if lead > 1e-4:
            break
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


@pytest.mark.parametrize("damage", ["missing", "shape", "type", "pairs"])
def test_damaged_folders_are_refused(tmp_path, damage):
    cfg = copy.deepcopy(nm.CONFIGS["odd_sizes"])
    t = nm.tensors(cfg, 1)
    if damage == "missing":
        del t["l2.mix.A_log"]
    elif damage == "shape":
        t["l0.mix.uv"] = t["l0.mix.uv"][:, :-1]
    elif damage == "type":
        t["l0.mix.uk"] = t["l0.mix.uk"].astype(np.int32)
    else:
        t["bigram"] = t["bigram"][:-1]                             # without the row of first tokens
    sp.write_model(str(tmp_path), cfg, t)
    with pytest.raises(RuntimeError):
        pkg.HostContext(str(tmp_path), 0)
