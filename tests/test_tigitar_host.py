"""Tigitar, what needs no GPU: folders, the argument structs against the C header, and the plain restatement's own consistency
(its mechanisms against small cases worked out another way, a whole sequence against the same one cut off)."""
import ctypes as C
import json
import subprocess
from pathlib import Path

import numpy as np
import pytest
import tigitar_oracle as ora
from tenzo_b200 import abi, load_library, synth

ROOT = Path(__file__).resolve().parents[1]
LATENT = {"heads": 2, "dim": 6, "rot_dim": 4, "vdim": 5, "kv_rank": 12, "mask": {"size": 5}, "rot": {"base": 50.0, "dims": 4}, "scale": 0.4}
CFG = {"vocab": 40, "width": 24, "norm": {"eps": 1e-5}, "logit_softcap": 6.0, "layers": [
    {"type": "latent_attention", "mlp": {"kind": "dense", "ff": 20}, "mixer": LATENT},
    {"type": "delta", "mlp": {"kind": "moe", "expert": {"ff": 9}, "router": {"experts": 5, "top": 2}}, "mixer": {"heads": 4, "kv_heads": 2, "dim": 6, "vdim": 7, "conv": 3}},
    {"type": "latent_attention", "mlp": None, "mixer": dict(LATENT, heads=3, kv_from=0, mask={"size": 11})}]}


def weights(folder, cfg=CFG, seed=1):
    return {n: a.astype(np.float64) for n, a in synth.write_tigitar(folder, cfg, seed=seed).items()}


def test_weight_files_round_trip(tmp_path):
    W = weights(tmp_path)
    back = ora.read_safetensors(tmp_path / "model.safetensors")
    assert set(W) == set(back) and all(np.array_equal(W[n], back[n]) for n in W)
    assert json.loads((tmp_path / "config.json").read_text())["architecture"] == "Tigitar"
    assert "l2.mix.dkv" not in W and "l2.norm2" not in W and "l1.mlp.e4.down" in W


def test_argument_structs_have_the_size_of_the_header(tmp_path):
    names = {"rows": "tenzo_rows_args", "gemm": "tenzo_gemm_args", "window_attention": "tenzo_window_attention_args", "linear_scan": "tenzo_scan_args",
             "delta_rule": "tenzo_delta_args", "latent_attention": "tenzo_latent_attention_args", "route": "tenzo_route_args"}
    assert set(names) == set(abi.STRUCT_CALLS)
    fields = [(n, f) for n in names for f, _ in abi.STRUCT_CALLS[n]._fields_]
    src = tmp_path / "probe.c"
    src.write_text('#include <stddef.h>\n#include <stdio.h>\n#include "tenzo_kernels.h"\nint main(){' +
                   "".join(f'printf("%zu\\n",sizeof({t}));' for t in names.values()) +
                   "".join(f'printf("%zu\\n",offsetof({names[n]},{f}));' for n, f in fields) + "return 0;}")
    subprocess.run(["gcc", "-I", str(ROOT / "include"), str(src), "-o", str(tmp_path / "probe")], check=True)
    out = [int(v) for v in subprocess.run([str(tmp_path / "probe")], capture_output=True, text=True, check=True).stdout.split()]
    assert out == [C.sizeof(abi.STRUCT_CALLS[n]) for n in names] + [getattr(abi.STRUCT_CALLS[n], f).offset for n, f in fields]


def test_kernel_calls_reject_bad_arguments_without_a_device():
    lib = load_library()
    for name in ("delta_rule", "latent_attention", "route"):
        assert getattr(lib, "tenzo_cuda_" + name)(None, None) == abi.ERR_INVALID
    a = abi.DeltaArgs(M=1, heads=3, kv_heads=2, dim=8, vdim=8, taps=1)
    assert lib.tenzo_cuda_delta_rule(C.byref(a), None) == -1
    b = abi.LatentAttentionArgs(M=1, heads=1, dim=8, rot=3, vdim=8, rank=8, window=1, ring=1)
    assert lib.tenzo_cuda_latent_attention(C.byref(b), None) == -1
    r = abi.RouteArgs(M=1, experts=2, top=3)
    assert lib.tenzo_cuda_route(C.byref(r), None) == -1
    assert lib.tenzo_cuda_delta_rule_work_floats(9, 4, 2, 33, 17) == 2 * 2 * 16 * 64 + 2 * 4 * 8 * 24 + 2 * 4 * 144 + 9 * 4 * 17


def test_oracle_is_causal(tmp_path):
    W = weights(tmp_path)
    tokens = np.random.default_rng(0).integers(0, 40, 25)
    whole = ora.forward(CFG, W, tokens)
    for n in (1, 2, 7, 24):
        assert np.allclose(ora.forward(CFG, W, tokens[:n]), whole[:n], atol=1e-10)


def test_oracle_delta_rule():
    """With full steps and unit keys the state answers a key with the value last stored under it, decayed since."""
    k = np.eye(3)[[0, 1, 0, 2]][:, None]
    v = np.arange(8.0).reshape(4, 1, 2)
    g = np.full((4, 1), 0.5)
    one = np.ones((4, 1))
    out = ora.delta_recurrence(k, k, v, g, one)
    assert np.allclose(out[:, 0], v[:, 0])
    probe = np.eye(3)[[0, 0, 0, 1]][:, None]                    # asks for key 0, later for key 1 stored at row 1
    out = ora.delta_recurrence(probe, k, v, g, one)
    assert np.allclose(out[1, 0], 0.5 * v[0, 0]) and np.allclose(out[2, 0], v[2, 0]) and np.allclose(out[3, 0], 0.25 * v[1, 0])
    assert np.allclose(ora.delta_recurrence(k, k, v, g, 0 * one), 0)


def test_oracle_rotation_is_relative():
    rng = np.random.default_rng(0)
    a, b = rng.standard_normal((2, 8))
    dot = lambda p, q: ora.rotate_halves(a[None], [p], 30.0)[0] @ ora.rotate_halves(b[None], [q], 30.0)[0]
    assert np.isclose(dot(5, 2), dot(105, 102)) and not np.isclose(dot(5, 2), dot(5, 3))
    turned = ora.rotate_halves(np.array([[1.0, 0, 0, 0]]), [1], 30.0)[0]
    assert np.allclose(turned, [np.cos(1), 0, np.sin(1), 0])


def test_oracle_window_and_routing():
    p = ora.window_softmax(np.zeros((6, 6)), 2)
    assert np.allclose(p[5], [0, 0, 0, 0, 0.5, 0.5]) and np.allclose(p[0], [1, 0, 0, 0, 0, 0])
    chosen, w = ora.route(np.array([[0.0, 3.0, 1.0]]), np.array([0.9, 0.0, 0.0]), 2)
    assert chosen.tolist() == [[0, 1]] and np.allclose(w, [[0.5, ora.sigmoid(3.0)]])


def test_weights_of_a_borrowed_cache_matter(tmp_path):
    """The borrowing layer reads layer 0's latents: changing them changes what it adds."""
    W = weights(tmp_path)
    tokens = np.random.default_rng(1).integers(0, 40, 12)
    layers, moved = [], []
    ora.forward(CFG, W, tokens, layers)
    ora.forward(CFG, dict(W, **{"l0.mix.dkv.norm": 2 * W["l0.mix.dkv.norm"], "l0.mix.o": 0 * W["l0.mix.o"]}), tokens, moved)
    ora.forward(CFG, dict(W, **{"l0.mix.o": 0 * W["l0.mix.o"]}), tokens, base := [])
    assert np.allclose(moved[1], base[1]) and not np.allclose(moved[2], base[2])


def test_a_broken_configuration_is_refused_before_any_work(tmp_path):
    import torch
    if torch.cuda.is_available():
        pytest.skip("a GPU is present: tests of whole folders cover this there")
    from tenzo_b200.engine import Engine
    weights(tmp_path)
    with pytest.raises(RuntimeError, match="no CPU path"):
        Engine.open(tmp_path)
