"""Model folders on the CPU: reading, the vocabulary of ids, the architecture registry, and the plain implementation itself."""
import copy
import json
import os
import subprocess

import numpy as np
import pytest

import sonuzen_models as sm
import sonuzen_plain as sp
from conftest import ROOT, load_pkg

pkg = load_pkg()


def test_header_and_id_vocabulary(tmp_path):
    sm.write(str(tmp_path), "mixed")
    ctx = pkg.HostContext(str(tmp_path), None)                     # the model only, no device
    assert ctx.architecture() == "Sonuzen"
    ctx.close()
    out = subprocess.run([os.path.join(ROOT, "llama-vulkan_b200", "vulkan_llama"), "-m", str(tmp_path), "--print_header"], capture_output=True, text=True)
    assert out.returncode == 0 and "Sonuzen" in out.stdout and "101" in out.stdout


def test_ggjt_files_stay_with_their_architecture(tmp_path):
    path = str(tmp_path / "tiny.ggjt")
    pkg.write_synthetic_model(path, "7b", n_layers=1, vocab=320)
    ctx = pkg.HostContext(path, None)
    assert ctx.architecture().startswith("LLaMA")
    ctx.close()


def refused(folder, cfg, tensors=None):
    sp.write_model(folder, cfg, tensors if tensors is not None else {"embed": np.zeros((2, 2), np.float32)})
    lib = pkg.load_host()
    h = lib.llava_context_open_model_only(os.fsencode(folder))
    if h:
        lib.llava_context_close(h)
        h = lib.llava_context_open(os.fsencode(folder), 0)          # the configuration is checked before a device is looked for
        assert not h
    return True


@pytest.mark.parametrize("change", [
    lambda c: c.update(architecture="Unheard"), lambda c: c.pop("vocab"), lambda c: c.pop("norm"), lambda c: c["canon"].pop("taps"),
    lambda c: c["layers"][1]["mixer"].update(kv_heads=4), lambda c: c["layers"][0].update(type="unknown"), lambda c: c["layers"][1]["mixer"].pop("scale"),
    lambda c: c["layers"][0]["mlp"]["router"].update(top=9), lambda c: c["loop"].update(stop=9), lambda c: c["layers"][0]["mlp"].update(kind="dense"),
    lambda c: c.update(layers=[])])
def test_bad_configurations_are_refused(tmp_path, change):
    cfg = copy.deepcopy(sm.CONFIGS["mixed"])
    change(cfg)
    assert refused(str(tmp_path), cfg)


@pytest.mark.parametrize("text", ["{", '{"architecture": "Sonuzen"', "[1, 2", '{"a": 01x}', '{"a": "\\q"}', "", '{"a": 1} x', "[" * 500])
def test_broken_json_is_refused(tmp_path, text):
    sm.write(str(tmp_path), "one_tap")
    (tmp_path / "config.json").write_text(text)
    assert not pkg.load_host().llava_context_open_model_only(os.fsencode(str(tmp_path)))


@pytest.mark.parametrize("damage", ["header length", "offsets", "dtype", "short"])
def test_broken_safetensors_are_refused(tmp_path, damage):
    sm.write(str(tmp_path), "one_tap")
    path = tmp_path / "model.safetensors"
    raw = path.read_bytes()
    n = int.from_bytes(raw[:8], "little")
    head = json.loads(raw[8:8 + n])
    if damage == "header length":
        raw = (1 << 60).to_bytes(8, "little") + raw[8:]
    elif damage == "short":
        raw = raw[:5]
    else:
        if damage == "offsets":
            head["embed"]["data_offsets"][1] += 1 << 30
        else:
            head["embed"]["dtype"] = "F8"
        text = json.dumps(head).encode()
        raw = len(text).to_bytes(8, "little") + text + raw[8 + n:]
    path.write_bytes(raw)
    assert not pkg.load_host().llava_context_open_model_only(os.fsencode(str(tmp_path)))


@pytest.mark.parametrize("name", list(sm.CONFIGS))
def test_the_plain_implementation_is_causal(name):
    cfg = sm.CONFIGS[name]
    p = sp.Plain(cfg, sm.tensors(cfg, 3))
    tokens = np.random.default_rng(0).integers(0, cfg["vocab"], 20)
    a = p.forward(tokens)
    other = tokens.copy()
    other[13:] = (other[13:] + 1) % cfg["vocab"]
    b = p.forward(other)
    assert np.allclose(a[:13], b[:13]) and not np.allclose(a[13:], b[13:], atol=1e-3)
    assert np.allclose(p.forward(tokens[:7]), a[:7])


def test_planted_mistakes_show_in_the_plain_logits():
    """The test models are sensitive: leaving out a mechanism moves the logits hundreds of times the 32-bit limit."""
    cfg = sm.CONFIGS["mixed"]
    t = sm.tensors(cfg, 1)
    tokens = np.random.default_rng(1).integers(0, cfg["vocab"], 150)
    want = sp.Plain(cfg, t).forward(tokens)

    def moved(change=None, patch=None):
        w = {k: v.copy() for k, v in t.items()}
        if change:
            change(w)
        p = sp.Plain(cfg, w)
        if patch:
            patch(p)
        return np.median(sm.distance(p.forward(tokens)[100:], want[100:]))

    def without_sink(p):
        p.mixer_plain = p.mixer
        def mixer(i, h):
            keep = sp.sink_softmax
            sp.sink_softmax = lambda s, mask: (lambda e: e / e.sum(-1, keepdims=True))(np.exp(np.where(mask, s, -np.inf) - np.where(mask, s, -np.inf).max(-1, keepdims=True)))
            try:
                return p.mixer_plain(i, h)
            finally:
                sp.sink_softmax = keep
        p.mixer = mixer

    assert moved() == 0
    assert moved(lambda w: w["l1.mix.r1"].fill(0)) > 0.03                              # distance bias
    assert moved(lambda w: w["l0.canon1"].fill(0)) > 0.1                               # convolution
    assert moved(lambda w: w["l4.canon2"].fill(0)) > 0.03
    assert moved(lambda w: w["loop.step"].__setitem__(2, w["loop.step"][1])) > 0.03      # the vector of a pass
    assert moved(lambda w: w["l4.mlp.table"].__setitem__(slice(None), (w["l4.mlp.table"] + 1) % 4)) > 0.1
    assert moved(patch=without_sink) > 0.01
