"""Sessions of model folders against the plain implementations: shared by the tests of the designs."""
import struct

import numpy as np

from conftest import load_pkg

pkg = load_pkg()
LIMIT = {"float32": 3e-5, "bfloat16": 3e-2}


class Model:
    """A small random model on disk; `design` is the module that draws it (CONFIGS, write, plain)."""

    def __init__(self, folder, name, design, seed=1):
        self.path = str(folder)
        self.cfg, t = design.write(self.path, name, seed)
        self.vocab = self.cfg["vocab"]
        self.plain = design.plain(self.cfg, t)
        self.open = {}

    def ctx(self, dtype):
        if dtype not in self.open:
            self.open[dtype] = pkg.HostContext(self.path, 0, dtype=dtype)
        return self.open[dtype]

    def tokens(self, n, seed=0):
        return [int(x) for x in np.random.default_rng(seed).integers(0, self.vocab, n)]

    def session(self, dtype, max_context=0):
        s = self.ctx(dtype).session(max_context)
        s.set_deterministic(True)
        return s

    def close(self):
        for c in self.open.values():
            c.close()
        self.open = {}


def cached_models(design, tmp_path_factory):
    """name -> Model, made once; a generator for a module's fixture."""
    made = {}

    def get(name):
        if name not in made:
            made[name] = Model(tmp_path_factory.mktemp(name), name, design)
        return made[name]
    yield get
    for m in made.values():
        m.close()


def feed(s, m, tokens, cuts):
    """Evaluates `tokens` in portions; logits of every token."""
    out, at = [], 0
    for n in cuts:
        for t in tokens[at:at + n]:
            assert s.push_token(t)
        out.append(s.evaluate_pending(range(at, at + n), m.vocab))
        at += n
    assert at == len(tokens)
    return np.concatenate(out)


def greedy(plain, prompt, n):
    """Greedy tokens of the plain implementation and how far each winner is ahead of the runner-up."""
    tokens, lead = list(prompt), []
    for _ in range(n):
        z = plain.forward(tokens)[-1]
        top = np.sort(z)[-2:]
        lead.append((top[1] - top[0]) / np.abs(z).max())
        tokens.append(int(z.argmax()))
    return tokens[len(prompt):], min(lead)


def frame_records(path):
    """(name, array) of a saved trace frame."""
    with open(path, "rb") as f:
        data, at, seen = f.read(), 0, []
    while at < len(data):
        cols, rows, _ = struct.unpack_from("<III", data, at)
        name = data[at + 12:data.index(b"\0", at + 12)].decode()
        at += (12 + len(name) + 1 + 31) & ~31
        seen.append((name, np.frombuffer(data, np.float32, cols * rows, at).reshape(rows, cols)))
        at += 4 * cols * rows
    return seen
