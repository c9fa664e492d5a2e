"""Sozopel, what needs no GPU: the model registry, folder checks, slot bookkeeping of trace replay, and the plain
restatement's own consistency (a whole sequence against the same sequence cut off at every length)."""
import json

import numpy as np
import pytest
import sozopel_oracle as ora
from tenzo_b200 import build, load_library, synth
from tenzo_b200.trace import Replay

CFG = {"vocab": 40, "width": 24, "max_positions": 30, "norm": {"eps": 1e-5}, "canon": {"taps": 3}, "layers": [
    {"type": "wkv", "mlp": None, "mixer": {"heads": 2, "dim": 6}},
    {"type": "parallel", "mlp": {"kind": "dense", "ff": 20}, "mixer": {
        "left": {"heads": 2, "kv_heads": 1, "dim": 8, "vdim": 4, "conv": 2, "mask": {"size": 5}, "scale": 0.3},
        "right": {"heads": 1, "dim": 6, "vdim": 10, "tau": 3.0}}},
    {"type": "retention", "mlp": None, "mixer": {"heads": 2, "dim": 4, "vdim": 7, "decay": [0.9, 0.99]}}]}


def test_registry_names_match_the_build():
    lib = load_library()
    names, i = [], 0
    while lib.tenzo_ext_architecture(i) is not None:
        names.append(lib.tenzo_ext_architecture(i).decode())
        i += 1
    assert sorted(names) == sorted(build.ARCHITECTURES)
    assert lib.tenzo_ext_architecture(-1) is None
    assert set(build.ARCHITECTURES.values()) == set(build.FAMILIES)
    assert sorted(build.SOURCES) == sorted(p.name for p in build.CSRC.glob("*.cu"))


def test_weight_files_round_trip(tmp_path):
    W = synth.write_sozopel(tmp_path, CFG, rank=3, seed=1)
    back = ora.read_safetensors(tmp_path / "model.safetensors")
    assert set(W) == set(back) and all(np.array_equal(W[n].astype(np.float64), back[n]) for n in W)
    assert json.loads((tmp_path / "config.json").read_text())["architecture"] == "Sozopel"
    assert back["l0.norm1"].shape == ()


def test_oracle_is_causal(tmp_path):
    W = {n: a.astype(np.float64) for n, a in synth.write_sozopel(tmp_path, CFG, rank=3, seed=2).items()}
    tokens = np.random.default_rng(0).integers(0, 40, 25)
    whole = ora.forward(CFG, W, tokens)
    for n in (1, 2, 7, 24):
        assert np.allclose(ora.forward(CFG, W, tokens[:n]), whole[:n], atol=1e-10)


def test_oracle_window_and_sink():
    q = k = np.ones((6, 1, 4))
    v = np.arange(6.0)[:, None, None] * np.ones((6, 1, 2))
    out = ora.window_attention(q, k, v, 100.0, 2)          # scores so high that the sink vanishes: the last two, biased by distance
    b = np.exp(-2.0 ** -8)
    assert np.allclose(out[5, 0], (5 + 4 * b) / (1 + b))
    assert np.allclose(ora.window_attention(0 * q, k, v, 1.0, 1)[3, 0], 1.5)    # score 0 against the unit sink


class FakeEngine:
    """Counts tokens per slot; a logit row is (tokens seen so far, slot)."""
    batch = 2

    def __init__(self):
        self.n = [0, 0]

    def reset_seq(self, s):
        self.n[s] = 0

    def forward(self, tokens, want, seq=0):
        base = self.n[seq]
        self.n[seq] += len(tokens)
        return np.array([[base + w, seq] for w in want], np.float32).reshape(len(want), 2)


def test_replay_slots():
    e = FakeEngine()
    r = Replay(e)
    a = r.step({"step": 0, "entries": [{"id": "a", "tokens": [1, 2, 3], "want": [2, 0]}, {"id": "b", "tokens": [4], "want": [0]}], "end": []})
    assert a[:, 0].tolist() == [2, 0, 0] and a[0, 1] != a[2, 1]
    assert r.step({"step": 1, "entries": [{"id": "a", "tokens": [1], "want": []}], "end": ["a"]}) is None
    c = r.step({"step": 2, "entries": [{"id": "c", "tokens": [5, 6], "want": [1]}, {"id": "b", "tokens": [7], "want": [0]}], "end": ["c", "b"]})
    assert c[:, 0].tolist() == [1, 1]
    with pytest.raises(RuntimeError, match="slots"):
        r.step({"step": 3, "entries": [{"id": x, "tokens": [1], "want": []} for x in "xyz"], "end": []})
