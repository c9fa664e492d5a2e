"""Sozopel on the GPU against the plain NumPy restatement (sozopel_oracle.py): every mechanism alone through its flat kernel
call, then models of several shapes through the engine - whole prompts, portions, decoding, slots, generation, traces."""
import json
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest
import sozopel_oracle as ora
import torch
from tenzo_b200 import abi, kernels, synth
from tenzo_b200.engine import Engine

pytestmark = pytest.mark.gpu
ROOT = Path(__file__).resolve().parents[1]
DT = {0: torch.bfloat16, 1: torch.float32}


def dev(a, dtype=torch.float32):
    return torch.from_numpy(np.array(a, np.float32)).to("cuda", dtype)


def host(t):
    return t.float().cpu().numpy().astype(np.float64)


def as_stored(a, f32):
    """What the storage type makes of an array."""
    return np.asarray(a, np.float64) if f32 else ora.bf16_to_f64(ora.f32_to_bf16(np.asarray(a, np.float32)))


def rel(got, want):
    return float(np.sqrt(np.mean((got - want) ** 2)) / (np.sqrt(np.mean(np.asarray(want) ** 2)) + 1e-30))


@pytest.fixture(autouse=True)
def _lib(cuda_lib):
    return cuda_lib


# ---- matrix products --------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("f32", [0, 1])
@pytest.mark.parametrize("M,N,K", [(1, 37, 72), (2, 130, 2500), (7, 64, 200), (11, 200, 64), (16, 128, 64), (40, 257, 328), (130, 100, 1100), (300, 513, 200)])
def test_gemm(f32, M, N, K):
    rng = np.random.default_rng(M * N + K)
    ld = (K + 63) // 64 * 64
    a, w = np.zeros((M, ld)), np.zeros((N, ld))
    a[:, :K], w[:, :K] = as_stored(rng.standard_normal((M, K)), f32), as_stored(rng.standard_normal((N, K)), 0)
    want = a @ w.T
    ws = kernels.gemm_workspace()
    common = dict(a=dev(a, DT[f32]), w=dev(w, torch.bfloat16), M=M, N=N, ld_k=ld, f32=f32, workspace=ws, workspace_bytes=ws.numel(), seg_end=[N] + [0] * 7)
    for _ in range(2):                                    # the split-K counters are ready for a second launch
        c = torch.full((M, N + 3), 7.0, device="cuda")
        kernels.gemm(c=c, ld_c=N + 3, **common)
        assert rel(host(c)[:, :N], want) < 2e-6
        assert bool((c[:, N:] == 7.0).all())
    c = torch.zeros((M, N), dtype=DT[f32], device="cuda")
    kernels.gemm(c=c, ld_c=N, epilogue=1, act_pos=0.9, act_neg=1.3, **{**common, "a": common["a"] * 0.1})
    z = (host(common["a"] * 0.1)) @ w.T
    y = np.where(z > 0, 0.9 * z * z, 1.3 * (np.expm1(np.minimum(z, 0)) - z)) + 0.5 * z
    assert rel(host(c), y) < (3e-6 if f32 else 3e-3)
    assert kernels.load_library().tenzo_cuda_gemm_take_timeouts() == 0


@pytest.mark.parametrize("f32", [0, 1])
@pytest.mark.parametrize("M", [1, 5, 33])
def test_gemm_segments_read_their_own_matrix(f32, M):
    rng = np.random.default_rng(M)
    ends, ld = [128, 384, 400], 128
    a = as_stored(rng.standard_normal((3, M, ld)), f32)
    w = as_stored(rng.standard_normal((ends[-1], ld)), 0)
    want = np.concatenate([a[s] @ w[lo:hi].T for s, (lo, hi) in enumerate(zip([0] + ends[:-1], ends))], axis=1)
    ws = kernels.gemm_workspace()
    c = torch.zeros((M, ends[-1]), device="cuda")
    kernels.gemm(a=dev(a, DT[f32]), w=dev(w, torch.bfloat16), M=M, N=ends[-1], ld_k=ld, n_seg=3, seg_end=ends + [0] * 5, a_seg_stride=M * ld,
                 c=c, ld_c=ends[-1], f32=f32, workspace=ws, workspace_bytes=ws.numel())
    assert rel(host(c), want) < 2e-6


# ---- rows -----------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("width,taps,mixes", [(72, 4, 0), (200, 1, 2), (1030, 3, 5), (64, 6, 0)])
@pytest.mark.parametrize("cuts", [[29], [1] * 29, [2, 2, 9, 16]])
def test_rows(width, taps, mixes, cuts):
    """Residual update from two normed addends, norm, convolution, mixes - cut anyhow, one row at a time as decode rows."""
    T, eps = 29, 1e-4
    rng = np.random.default_rng(width)
    x, y0, y1 = (rng.standard_normal((T, width)) for _ in range(3))
    w0, w1 = rng.standard_normal((2, width))
    cw, mu = rng.standard_normal((width, taps)), rng.standard_normal((max(mixes, 1), width))
    xo = x + 0.5 * (ora.over_rms(y0, eps) * w0 + ora.over_rms(y1, eps) * w1)
    u = ora.over_rms(xo, eps) * 1.7
    y = u + ora.causal_conv(u, cw)
    prev = np.concatenate([np.zeros((1, width)), y[:-1]])
    want = np.stack([y + (prev - y) * m for m in mu]) if mixes else y[None]
    state = torch.zeros(taps * width, device="cuda")      # tail rows, then the previous row
    got, got_x, at = np.zeros_like(want), np.zeros_like(xo), 0
    for n in cuts:
        sl = slice(at, at + n)
        stage = state if n == 1 else torch.zeros_like(state)
        out, x_out = torch.zeros((max(mixes, 1), n, width), device="cuda"), torch.zeros((n, width), device="cuda")
        kernels.rows(x_in=dev(x[sl]), y0=dev(y0[sl]), y1=dev(y1[sl]), w0=dev(w0), w1=dev(w1), ld_y=width, x_out=x_out, width=width, M=n, eps=eps,
                     gain=1.7, conv_w=dev(cw.T.copy()), taps=taps, tail_in=state, tail_out=stage, mu=dev(mu) if mixes else None, n_mix=mixes,
                     prev_in=state[(taps - 1) * width:], prev_out=stage[(taps - 1) * width:], seq_stride=0, decode=int(n == 1), out=out,
                     ld_out=width, row_inv=torch.empty(n, device="cuda"), f32=1)
        torch.cuda.synchronize()
        state = stage
        got[:, sl], got_x[sl] = host(out), host(x_out)
        at += n
    assert rel(got_x, xo) < 1e-6 and rel(got, want) < 2e-6


# ---- attention --------------------------------------------------------------------------------------------------------------
class Attention:
    """The attention kernel with its carried state over one sequence."""

    def __init__(self, f32, heads, kv, dim, vdim, taps, window, ring, scale, rng, slope_base=8.0, sink=1.0):
        self.__dict__.update(locals())
        up8 = lambda v: (v + 7) // 8 * 8
        self.ch = (heads * dim, kv * dim, kv * vdim)
        self.conv = [rng.standard_normal((c, taps)) * 0.5 + 0.3 for c in self.ch]
        self.tail = torch.zeros(max(1, (taps - 1) * sum(self.ch)), device="cuda")
        self.rk = torch.zeros((kv, ring, up8(dim)), dtype=DT[f32], device="cuda")
        self.rv = torch.zeros((kv, ring, up8(vdim)), dtype=DT[f32], device="cuda")
        self.pos, self.up8 = 0, up8

    def run(self, qkv):
        M, n = len(qkv), sum(self.ch)
        x = dev(qkv)
        out = torch.zeros((M, self.heads * self.vdim), dtype=DT[self.f32], device="cuda")
        lin = [torch.zeros(s, dtype=DT[self.f32], device="cuda") for s in
               ((M, self.heads, self.up8(self.dim)), (self.kv, self.ring + M, self.up8(self.dim)), (self.kv, self.ring + M, self.up8(self.vdim)))]
        stage = self.tail if M == 1 else torch.zeros_like(self.tail)
        o = np.cumsum((0,) + self.ch)
        cw = [dev(c.T.copy()) for c in self.conv]
        pos = torch.tensor([self.pos], dtype=torch.int32, device="cuda")
        kernels.window_attention(q=x, k=x[:, o[1]:], v=x[:, o[2]:], ld=n, conv_q=cw[0], conv_k=cw[1], conv_v=cw[2], taps=self.taps, tail_in=self.tail,
                                 tail_out=stage, heads=self.heads, kv_heads=self.kv, dim=self.dim, vdim=self.vdim, scale=self.scale,
                                 slope_base=self.slope_base, sink=self.sink, window=self.window, ring=self.ring, ring_k=self.rk, ring_v=self.rv,
                                 pos=pos, pos0=self.pos, M=M, decode=int(M == 1), out=out, ld_out=self.heads * self.vdim, lin_q=lin[0], lin_k=lin[1],
                                 lin_v=lin[2], f32=self.f32)
        torch.cuda.synchronize()
        self.tail = stage
        self.pos += M
        return host(out)

    def want(self, qkv):
        o = np.cumsum((0,) + self.ch)
        q, k, v = (as_stored(ora.causal_conv(qkv[:, a:b], w.astype(np.float32).astype(np.float64)), self.f32) for a, b, w in zip(o[:-1], o[1:], self.conv))
        T = len(qkv)
        return ora.window_attention(q.reshape(T, self.heads, -1), k.reshape(T, self.kv, -1), v.reshape(T, self.kv, -1), self.scale, self.window).reshape(T, -1)


SHAPES = [(4, 2, 64, 64, 3, 24), (6, 2, 40, 72, 2, 17), (8, 1, 36, 20, 1, 64), (3, 3, 128, 128, 4, 1), (10, 1, 32, 128, 3, 300), (2, 1, 256, 256, 3, 33), (4, 4, 96, 64, 3, 5000)]


@pytest.mark.parametrize("f32", [0, 1])
@pytest.mark.parametrize("heads,kv,dim,vdim,taps,window", SHAPES)
def test_window_attention(f32, heads, kv, dim, vdim, taps, window):
    T = 400
    rng = np.random.default_rng(heads * dim + window)
    qkv = rng.standard_normal((T, heads * dim + kv * (dim + vdim))).astype(np.float32).astype(np.float64)
    for cuts in ([T], [2, 100, 1, 1, 7, 64, 2] + [1] * 60 + [163], [37] + [1] * 20 + [3, 2, 130, 208]):
        att = Attention(f32, heads, kv, dim, vdim, taps, window, min(window, 1024), dim ** -0.5, np.random.default_rng(7))
        want = att.want(qkv)
        got = np.concatenate([att.run(part) for part in np.split(qkv, np.cumsum(cuts)[:-1])])
        assert rel(got, want) < (3e-6 if f32 else 6e-3), cuts
        assert np.abs(got - want).max() < (3e-5 if f32 else 6e-2), cuts


@pytest.mark.parametrize("f32", [0, 1])
@pytest.mark.parametrize("decode", [False, True])
@pytest.mark.parametrize("window", [8, 33, 64, 129])
def test_window_edge_shows(f32, decode, window):
    """One key matches one query so strongly that it takes all the weight when it is inside the window - at the last place
    inside, and at the first place outside."""
    rng = np.random.default_rng(window)
    dim = vdim = 64
    for back in (window - 1, window):
        T, at = window + 40, window + 30                  # the query's row
        qkv = 0.1 * rng.standard_normal((T, 3 * dim))
        d = rng.standard_normal(dim)
        d /= np.linalg.norm(d)
        qkv[at, :dim] = 20 * d
        qkv[at - back, dim:2 * dim] = 20 * d
        qkv[at - back, 2 * dim:] = 5.0
        att = Attention(f32, 1, 1, dim, vdim, 1, window, window, 1.0, rng)
        att.conv = [np.ones((c, 1)) for c in att.ch]
        got = np.concatenate([att.run(qkv[:at])] + [att.run(qkv[i:i + 1]) for i in range(at, T)] if decode else [att.run(qkv[:5]), att.run(qkv[5:])])
        want = att.want(qkv)
        assert (want[at].mean() > 4.5) == (back < window)   # the case discriminates
        assert np.abs(got - want).max() < (2e-4 if f32 else 4e-2)


def test_sink_and_bias_are_parameters():
    rng = np.random.default_rng(0)
    qkv = rng.standard_normal((50, 3 * 32)).astype(np.float32).astype(np.float64)
    att = Attention(1, 1, 1, 32, 32, 1, 12, 12, 0.2, rng, slope_base=0.0, sink=0.0)
    att.conv = [np.ones((c, 1)) for c in att.ch]
    q, k, v = np.split(qkv, 3, axis=1)
    dist = np.arange(50)[:, None] - np.arange(50)[None, :]
    s = np.where((dist >= 0) & (dist < 12), 0.2 * q @ k.T, -np.inf)
    p = np.exp(s - s.max(1, keepdims=True))
    want = p @ v / p.sum(1, keepdims=True)
    got = np.concatenate([att.run(qkv[:30])] + [att.run(qkv[i:i + 1]) for i in range(30, 50)])
    assert rel(got, want) < 3e-6


# ---- recurrences ------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("kind,bonus,norm", [(0, False, None), (1, False, "shared"), (2, True, "head"), (2, False, "head"), (0, True, "shared")])
@pytest.mark.parametrize("heads,dim,vdim", [(3, 32, 64), (2, 20, 50), (1, 64, 128), (2, 100, 36), (1, 256, 256), (5, 1, 3)])
def test_linear_scan(kind, bonus, norm, heads, dim, vdim):
    T, rank, tau, eps = 150, 5, 4.0, 1e-4
    rng = np.random.default_rng(heads * dim + vdim + kind)
    n, nv = heads * dim, heads * vdim
    x = rng.standard_normal((T, 2 * n + 2 * nv + rank)).astype(np.float32).astype(np.float64)
    off = np.cumsum([0, n, n, nv, nv, rank])
    q, k, v, g, low = (x[:, a:b] for a, b in zip(off[:-1], off[1:]))
    up, bias = as_stored(rng.standard_normal((n, rank)) * 0.5, 0), rng.standard_normal(n).astype(np.float32).astype(np.float64) - 1.0
    decay_h = rng.uniform(0.8, 1.0, heads).astype(np.float32).astype(np.float64)
    u = rng.standard_normal(n).astype(np.float32).astype(np.float64)
    gain = rng.standard_normal(vdim if norm == "shared" else nv).astype(np.float32).astype(np.float64)
    z = (np.tanh(low) if kind == 2 else low) @ up.T + bias
    w = {0: np.repeat(np.broadcast_to(decay_h, (T, heads)), dim, axis=1), 1: np.exp(-np.logaddexp(0, -z) / tau), 2: np.exp(-np.exp(z))}[kind]
    hd = lambda a: a.reshape(T, heads, -1)
    o = ora.over_rms(ora.linear_recurrence(hd(q) * 0.5, hd(k) * 0.7, hd(v), hd(w), u.reshape(heads, dim) if bonus else None), eps)
    o = o * gain.reshape(1, -1, vdim) if norm else o
    want = o.reshape(T, nv) * ora.silu(g)
    ldv = (vdim + 3) // 4 * 4
    fixed = dict(ld=x.shape[1], q_scale=0.5, k_scale=0.7, heads=heads, dim=dim, vdim=vdim, decay_kind=kind, decay=dev(decay_h), up=dev(np.pad(up, ((0, 0), (0, -rank % 8))), torch.bfloat16),
                 bias=dev(bias), rank=rank, tau=tau, bonus=dev(u) if bonus else None, norm=dev(gain) if norm else None, norm_per_head=int(norm == "head"),
                 eps=eps, ld_out=nv, f32=1)
    for cuts in ([T], [1] * 30 + [2, 118], [64, 2, 3, 1, 70, 10]):
        state = torch.zeros((heads, dim, ldv), device="cuda")
        got = []
        for part in np.split(x, np.cumsum(cuts)[:-1]):
            M = len(part)
            d = dev(part)
            out = torch.zeros((M, nv), device="cuda")
            kernels.linear_scan(q=d, k=d[:, off[1]:], v=d[:, off[2]:], g=d[:, off[3]:], low=d[:, off[4]:], state=state, M=M, decode=int(M == 1), out=out,
                                w_rows=torch.zeros((M, n), device="cuda"), o_rows=torch.zeros((M, nv), device="cuda"),
                                part=kernels.linear_scan_part(M, heads, dim, vdim), **fixed)
            got.append(host(out))
        assert rel(np.concatenate(got), want) < 2e-5, cuts


# ---- models -------------------------------------------------------------------------------------------------------------------
def parallel(lh, lkv, ld, lvd, conv, size, rh, rd, rvd, tau, ff, scale=None):
    return {"type": "parallel", "mlp": ff and {"kind": "dense", "ff": ff},
            "mixer": {"left": {"heads": lh, "kv_heads": lkv, "dim": ld, "vdim": lvd, "conv": conv, "mask": {"size": size}, "scale": scale or ld ** -0.5},
                      "right": {"heads": rh, "dim": rd, "vdim": rvd, "tau": tau}}}


def retention(heads, dim, vdim, ff=None, decay=None):
    return {"type": "retention", "mlp": ff and {"kind": "dense", "ff": ff},
            "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay or [1 - 2.0 ** -(3 + i) for i in range(heads)]}}


def wkv(heads, dim, ff=None):
    return {"type": "wkv", "mlp": ff and {"kind": "dense", "ff": ff}, "mixer": {"heads": heads, "dim": dim}}


def config(layers, width=96, vocab=210, taps=4, eps=1e-5, n_pos=600):
    return {"vocab": vocab, "width": width, "max_positions": n_pos, "norm": {"eps": eps}, "canon": {"taps": taps}, "layers": layers}


MODELS = {
    "attention_beside_gla": (config([parallel(4, 2, 24, 32, 3, 19, 3, 20, 28, 8.0, 130)]), 7),
    "retention": (config([retention(3, 20, 44), retention(2, 32, 16, ff=72)], width=80), 4),
    "time_mixing": (config([wkv(3, 24), wkv(2, 48, ff=333), wkv(1, 20, ff=140)], width=72, taps=3), 12),
    "mixed": (config([wkv(4, 16, ff=96), parallel(6, 3, 16, 48, 2, 31, 2, 40, 24, 20.0, None), retention(2, 24, 40), parallel(5, 1, 32, 16, 4, 70, 1, 16, 64, 5.0, 200)],
                     width=120, vocab=301, taps=2, eps=1e-3), 9),
    "no_reach_back": (config([parallel(2, 2, 16, 16, 1, 1, 2, 16, 16, 1.0, 64), wkv(1, 40), retention(1, 12, 20)], width=64, taps=1), 1),
}


@pytest.fixture(scope="module")
def model(tmp_path_factory):
    made = {}

    def get(name):
        if name not in made:
            cfg, rank = MODELS[name]
            folder = tmp_path_factory.mktemp(name)
            W = {n: a.astype(np.float64) for n, a in synth.write_sozopel(folder, cfg, rank=rank, seed=len(name)).items()}
            tokens = np.random.default_rng(3).integers(0, cfg["vocab"], 260)
            made[name] = folder, cfg, W, tokens, ora.forward(cfg, W, tokens)
        return made[name]

    return get


LIMIT = {"float32": 5e-5, "bfloat16": 6e-2}


def close(got, want, compute):
    d = got - want
    err = np.sqrt(np.mean(d * d, axis=-1)) / np.sqrt(np.mean(want * want))
    assert err.max() < LIMIT[compute], (err.max(), int(err.argmax()))


def feed(e, tokens, cuts, seq=0):
    out, at = [], 0
    for n in cuts:
        out.append(e.forward(tokens[at:at + n], range(n), seq=seq))
        at += n
    assert at == len(tokens)
    return np.concatenate(out)


@pytest.mark.parametrize("compute", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", MODELS)
def test_prompts_portions_and_decoding_give_the_same_logits(model, name, compute):
    folder, cfg, W, tokens, want = model(name)
    with Engine.open(folder, compute=compute) as e:
        assert e.config.hidden_size == cfg["width"] and e.config.vocab_size == cfg["vocab"] and e.config.max_seq_len == cfg["max_positions"]
        for cuts in ([260], [200] + [1] * 60, [2] * 9 + [3, 1, 64, 15, 1, 1, 2, 60, 80, 15], [1] * 40 + [2, 100, 7, 111]):
            close(feed(e, tokens, cuts), want, compute)
            assert e.seq_len() == 260
            e.reset()                                       # the same slot again, with other leftovers every time
        e.prefill_chunk(tokens[:150])
        close(e.forward(tokens[150:151], [0]), want[150:151], compute)
        assert rel(e.read_buffer(15).astype(np.float64), want[150]) < LIMIT[compute]


@pytest.mark.parametrize("compute", ["float32", "bfloat16"])
def test_residual_after_every_layer(model, compute, tmp_path):
    folder, cfg, W, tokens, _ = model("mixed")
    layers = []
    ora.forward(cfg, W, tokens[:40], layers)
    for n in range(1, len(cfg["layers"]) + 1):
        d = tmp_path / str(n)
        d.mkdir()
        (d / "config.json").write_text(json.dumps(dict(cfg, architecture="Sozopel", layers=cfg["layers"][:n])))
        (d / "model.safetensors").symlink_to(folder / "model.safetensors")
        with Engine.open(d, compute=compute) as e:
            e.prefill_chunk(tokens[:30])
            assert rel(e.read_buffer(0), layers[n - 1][29]) < LIMIT[compute]
            for i in range(30, 40):
                e.prefill_token(tokens[i])
                assert rel(e.read_buffer(0), layers[n - 1][i]) < LIMIT[compute]


def test_one_layer_of_a_step(model):
    """run_layer on a given residual: the first layer of a fresh sequence, then the second on what it left."""
    folder, cfg, W, tokens, _ = model("mixed")
    layers = []
    ora.forward(cfg, W, tokens[:1], layers)
    with Engine.open(folder, compute="float32") as e:
        e.write_x(W["embed"][tokens[0]] + W["pos"][0])
        for l in range(len(layers)):
            e.run_layer(l)
            assert rel(e.read_buffer(0), layers[l][0]) < LIMIT["float32"]


@pytest.mark.parametrize("compute", ["float32", "bfloat16"])
def test_slots_are_independent_and_reusable(model, compute):
    """Unequal requests side by side, then batched decoding of all slots, then one slot given back and taken by another."""
    folder, cfg, W, tokens, want = model("mixed")
    lens = [5, 90, 1, 33]
    other = np.random.default_rng(9).integers(0, cfg["vocab"], 60)
    other_want = ora.forward(cfg, W, other)
    with Engine.open(folder, compute=compute, batch=4) as e:
        for s, n in enumerate(lens):
            close(feed(e, tokens[:n], [n], seq=s), want[:n], compute)
        for i in range(12):
            e.generate_steps([tokens[n + i] for n in lens])
            for s, n in enumerate(lens):
                close(e.read_buffer(15, seq=s)[None], want[n + i:n + i + 1], compute)
        e.reset_seq(1)
        close(feed(e, other, [20, 2, 38], seq=1), other_want, compute)
        at = lens[3] + 12
        close(e.forward(tokens[at:at + 2], [0, 1], seq=3), want[at:at + 2], compute)      # untouched by its neighbours


def test_wide_batches_take_the_tensor_cores(model):
    folder, cfg, W, tokens, want = model("mixed")
    with Engine.open(folder, batch=40) as e:
        for s in range(40):
            e.forward(tokens[:s + 1], seq=s)
        for i in range(6):
            e.generate_steps([tokens[s + 1 + i] for s in range(40)])
        got = np.stack([e.read_buffer(15, seq=s) for s in range(40)])
        close(got, want[np.arange(40) + 6], "bfloat16")


def test_long_decoding(model):
    folder, cfg, W, _, _ = model("attention_beside_gla")
    tokens = np.random.default_rng(11).integers(0, cfg["vocab"], 600)
    want = ora.forward(cfg, W, tokens)
    with Engine.open(folder, compute="float32") as e:
        close(feed(e, tokens, [3] + [1] * 597), want, "float32")
        with pytest.raises(RuntimeError, match="max_seq_len"):
            e.forward([0])                                  # every learned position is used up


@pytest.mark.parametrize("use_graph,use_pdl", [(1, 1), (1, 0), (0, 1), (0, 0)])
def test_greedy_generation(model, use_graph, use_pdl):
    folder, cfg, W, tokens, _ = model("mixed")
    prompt = tokens[:21].tolist()
    want = ora.greedy(cfg, W, prompt, 24)
    with Engine.open(folder, compute="float32", use_graph=use_graph, use_pdl=use_pdl) as e:
        assert e.generate(prompt, 24) == want
        e.reset()
        e.prefill_chunk(prompt[:-1])
        assert e.decode_greedy([prompt[-1]], 24)[:, 0].tolist() == want      # tokens fed back on the device
        e.reset()
        sampled = e.generate(prompt, 8, abi.TenzoSampling(0.8, 0.9, 10, 1.1))
        assert all(0 <= t < cfg["vocab"] for t in sampled)
        assert e.kernel_launches() > 0


def test_a_state_cannot_be_cut_back(model):
    folder, cfg, W, tokens, _ = model("retention")
    with Engine.open(folder) as e:
        e.prefill_chunk(tokens[:10])
        with pytest.raises(RuntimeError, match="recurrent state"):
            e.set_seq_len(0, 4)
        e.set_seq_len(0, 0)
        assert e.seq_len() == 0
        with pytest.raises(RuntimeError, match="token id"):
            e.forward([cfg["vocab"]])
        with pytest.raises(RuntimeError, match="BitNet"):
            e.kv_export(0, 0, 0)


@pytest.mark.parametrize("compute", ["float32", "bfloat16"])
def test_far_tokens_show(tmp_path, compute):
    """Slow decays, and keys and values that favour one direction of the input: an early token that lies along it is felt
    hundreds of tokens later, and the model with it and without it are told apart."""
    cfg = config([retention(2, 32, 32, decay=[0.9995, 0.999])], width=64, vocab=50, taps=2)

    def change(t):
        d = t["embed"][7] / np.linalg.norm(t["embed"][7])
        t["embed"][8:] -= 0.9 * np.outer(t["embed"][8:] @ d, d)
        k, v = t["l0.mix.k"], t["l0.mix.v"]
        t["l0.mix.k"] = 0.1 * k + 12 * np.outer(k @ d, d)
        t["l0.mix.v"] = v + 4 * np.outer(v @ d, d)

    W = {n: a.astype(np.float64) for n, a in synth.write_sozopel(tmp_path, cfg, seed=5, change=change).items()}
    moved = np.random.default_rng(2).integers(8, 50, 500)
    tokens = moved.copy()
    tokens[20] = 7
    want, without = ora.forward(cfg, W, tokens), ora.forward(cfg, W, moved)
    felt = rel(without[300:], want[300:])
    assert felt > 0.05
    with Engine.open(tmp_path, compute=compute) as e:
        got = feed(e, tokens, [100, 2, 65, 300] + [1] * 33)
        assert rel(got[300:], want[300:]) < (2e-5 if compute == "float32" else felt / 4)
        e.reset()
        got = feed(e, moved, [500])
        assert rel(got[300:], without[300:]) < (2e-5 if compute == "float32" else felt / 4)


def test_broken_folders_are_reported(tmp_path, model):
    folder, cfg, *_ = model("retention")
    for broken in (tmp_path / "nowhere", tmp_path_with(tmp_path, "{")):
        with pytest.raises(RuntimeError, match="config.json"):
            Engine.open(broken)
    with pytest.raises(RuntimeError, match="no model of this library"):
        Engine.open(tmp_path_with(tmp_path, json.dumps({"architecture": "Unknown"})))
    bad = dict(cfg, architecture="Sozopel", width=cfg["width"] + 8)
    d = tmp_path_with(tmp_path, json.dumps(bad))
    (d / "model.safetensors").symlink_to(folder / "model.safetensors")
    with pytest.raises(RuntimeError, match="shape"):
        Engine.open(d)
    bad = dict(cfg, architecture="Sozopel", layers=[dict(cfg["layers"][0], type="other")])
    d2 = tmp_path_with(tmp_path, json.dumps(bad), "b")
    (d2 / "model.safetensors").symlink_to(folder / "model.safetensors")
    with pytest.raises(RuntimeError, match="unknown type"):
        Engine.open(d2)


def tmp_path_with(tmp_path, text, name="a"):
    d = tmp_path / name
    d.mkdir(exist_ok=True)
    (d / "config.json").write_text(text)
    return d


# ---- trace replay ----------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("compute", ["float32", "bfloat16"])
def test_trace_replay(model, compute, tmp_path):
    folder, cfg, W, tokens, want = model("mixed")
    steps = [{"step": 0, "entries": [{"id": "p", "tokens": tokens[:50].tolist(), "want": [0, 49, 7]}], "end": []},
             {"step": 1, "entries": [{"id": "p", "tokens": tokens[50:52].tolist(), "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "p", "tokens": tokens[52:53].tolist(), "want": [0]}], "end": ["p"]},
             {"step": 3, "entries": [{"id": "q", "tokens": tokens[:4].tolist(), "want": [3]}], "end": ["q"]}]
    r = subprocess.run([str(ROOT / "bin" / "trace_run"), "--model", str(folder), "--dtype", compute, "--out", str(tmp_path), "--max-tokens", "64"],
                       input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(4)]
    read = lambda i: np.fromfile(tmp_path / f"{i}.f32", "<f4").reshape(-1, cfg["vocab"])
    close(read(0), want[[0, 49, 7]], compute)
    close(read(2), want[[52]], compute)
    close(read(3), want[[3]], compute)
    assert not (tmp_path / "1.f32").exists()


def test_command_line_generates(model):
    folder, cfg, W, tokens, _ = model("mixed")
    prompt = tokens[:9].tolist()
    r = subprocess.run([sys.executable, "-m", "tenzo_b200", "generate", "--model", str(folder), "--dtype", "float32", "--n", "6", "--tokens",
                        ",".join(map(str, prompt))], capture_output=True, text=True, timeout=300, cwd=ROOT)
    assert r.returncode == 0, r.stderr
    assert [int(t) for t in r.stdout.split()] == ora.greedy(cfg, W, prompt, 6)
