"""Nuforax on the CPU: configurations that are refused, and the plain implementation itself."""
import copy

import numpy as np
import pytest

import nuforax_models as nm
import nuforax_plain as npl
from conftest import load_pkg
from test_model_folder import refused

pkg = load_pkg()


def test_the_registry_knows_the_design(tmp_path):
    nm.write(str(tmp_path), "mixed")
    ctx = pkg.HostContext(str(tmp_path), None)
    assert ctx.architecture() == "Nuforax"
    ctx.close()


@pytest.mark.parametrize("change", [
    lambda c: c.pop("embedding"), lambda c: c["embedding"].pop("bigram"), lambda c: c["embedding"].pop("scale"), lambda c: c["embedding"]["bigram"].update(buckets=0),
    lambda c: c["layers"][0]["mixer"].pop("mask"), lambda c: c["layers"][0]["mixer"]["mask"].update(size=0), lambda c: c["layers"][0]["mixer"].pop("rot"),
    lambda c: c["layers"][0]["mixer"]["rot"].update(dims=10), lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7), lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].pop("slow"),
    lambda c: c["layers"][2]["mixer"].update(kv_from=1), lambda c: c["layers"][2]["mixer"].update(kv_from=3), lambda c: c["layers"][2]["mixer"].update(kv_from=2),
    lambda c: c["layers"][2]["mixer"].update(kv_rank=40), lambda c: c["layers"][2]["mixer"]["rot"].update(base=77.0), lambda c: c["layers"][5]["mixer"].update(kv_from=2),
    lambda c: c["layers"][1]["mixer"].update(groups=4), lambda c: c["layers"][1]["mixer"].update(norm_groups=7), lambda c: c["layers"][1]["mixer"].pop("conv"),
    lambda c: c["layers"][1]["mixer"].update(state=300), lambda c: c["layers"][0]["mixer"].update(kv_rank=2000), lambda c: c["layers"][0]["mlp"].update(kind="moe"),
    lambda c: c["layers"][0]["mlp"].pop("ff"), lambda c: c["layers"][0].update(type="attention"), lambda c: c.update(layers=[])])
def test_bad_configurations_are_refused(tmp_path, change):
    cfg = copy.deepcopy(nm.CONFIGS["mixed"])
    change(cfg)
    assert refused(str(tmp_path), cfg)


@pytest.mark.parametrize("name", list(nm.CONFIGS))
def test_the_plain_implementation_is_causal(name):
    cfg = nm.CONFIGS[name]
    p = nm.plain(cfg, nm.tensors(cfg, 3))
    tokens = np.random.default_rng(0).integers(0, cfg["vocab"], 20)
    a = p.forward(tokens)
    other = tokens.copy()
    other[13:] = (other[13:] + 1) % cfg["vocab"]
    b = p.forward(other)
    assert np.allclose(a[:13], b[:13]) and not np.allclose(a[13:], b[13:], atol=1e-3)
    assert np.allclose(p.forward(tokens[:7]), a[:7])


def test_frequencies_between_both_ends_of_the_ramp():
    plain, one = npl.yarn(32, 10000.0)
    scaled, mult = npl.yarn(32, 10000.0, {"factor": 8.0, "original": 256, "fast": 16.0, "slow": 1.0})
    ratio = scaled / plain
    assert one == 1.0 and abs(mult - (0.1 * np.log(8.0) + 1)) < 1e-12
    assert ratio[0] == 1 and np.isclose(ratio[-1], 1 / 8) and (np.diff(ratio) <= 0).all() and ((ratio > 1 / 8 + 1e-6) & (ratio < 1 - 1e-6)).sum() >= 3
    turns = 256 * plain / (2 * np.pi)                                # within the original length
    assert (ratio[turns > 16 * 1.8] == 1).all() and np.allclose(ratio[turns < 1 / 1.8], 1 / 8)


def test_rotation_depends_on_the_distance_only():
    rng = np.random.default_rng(1)
    f, _ = npl.yarn(8, 100.0)
    q, k = rng.standard_normal((2, 1, 10))
    score = lambda i, j: (npl.rotate(q, np.array([float(i)]), f, 1.0) * npl.rotate(k, np.array([float(j)]), f, 1.0)).sum()
    assert np.isclose(score(9, 4), score(105, 100)) and not np.isclose(score(9, 4), score(9, 5))


def test_planted_mistakes_show_in_the_plain_logits(monkeypatch):
    """The test models are sensitive: every mechanism that is left out or shifted moves the logits hundreds of times the 32-bit limit."""
    cfg = nm.CONFIGS["mixed"]
    t = nm.tensors(cfg, 1)
    tokens = [int(x) for x in np.random.default_rng(1).integers(0, cfg["vocab"], 150)]
    want = nm.plain(cfg, t).forward(tokens)

    def moved(change=None, patch=None, config=None):
        w, c = {k: v.copy() for k, v in t.items()}, copy.deepcopy(cfg)
        if change:
            change(w)
        if config:
            config(c)
        with monkeypatch.context() as m:
            if patch:
                m.setattr(npl, *patch)
            z = nm.plain(c, w).forward(tokens)
        return np.median(nm.distance(z[100:], want[100:]))

    mixer = lambda c, i: c["layers"][i]["mixer"]
    assert moved() == 0
    assert moved(patch=("window_mask", lambda T, size, f=npl.window_mask: f(T, size + 1))) > 0.01
    assert moved(patch=("window_mask", lambda T, size, f=npl.window_mask: f(T, size - 1))) > 0.01
    for i in (0, 2, 3, 5):
        assert moved(config=lambda c: mixer(c, i)["mask"].update(size=mixer(c, i)["mask"]["size"] + 1)) > 3e-4
        assert moved(lambda w: w[f"l{i}.mix.sink"].fill(-50)) > 5e-4
        assert moved(config=lambda c: mixer(c, i).update(scale=mixer(c, i)["scale"] * 1.1)) > 0.003
    assert moved(patch=("rotate", lambda x, p, f, mult, g=npl.rotate: g(x, p, f, 1.0))) > 0.003
    assert moved(patch=("rotate", lambda x, p, f, mult, g=npl.rotate: g(x, p + (x.ndim == 3), f, mult))) > 0.003      # queries one position on
    assert moved(patch=("yarn", lambda d, b, s=None, g=npl.yarn: (g(d, b)[0], g(d, b, s)[1]))) > 0.003
    assert moved(patch=("bigram_rows", lambda tok, b, p, c, g=npl.bigram_rows: g(tok, b, c, p))) > 0.1
    assert moved(patch=("bigram_rows", lambda tok, b, p, c, g=npl.bigram_rows: np.array([b] + [b] * (len(tok) - 1)))) > 0.1
    assert moved(patch=("relu_squared", lambda z: np.maximum(z, 0))) > 0.1
    assert moved(patch=("gated_group_norm", lambda y, z, w, parts, eps, g=npl.gated_group_norm: g(y, z, w, 1, eps))) > 0.003
    assert moved(lambda w: w["l1.mix.D"].fill(0)) > 0.01
    assert moved(lambda w: w["l1.mix.conv"].__setitem__((slice(None), 0), 0)) > 0.01
    assert moved(lambda w: w["l4.mix.A_log"].fill(3)) > 0.01                          # a state that is lost after a token
    assert moved(lambda w: w["l1.mix.dt_bias"].fill(0)) > 0.01
