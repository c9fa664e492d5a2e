"""Tigitar on the GPU against the plain NumPy restatement (tigitar_oracle.py): every mechanism alone through its flat kernel
call, then models of several shapes through the engine - whole prompts, portions, decoding, slots, generation, traces."""
import json
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest
import tigitar_oracle as ora
import torch
from tenzo_b200 import abi, kernels, synth
from tenzo_b200.engine import Engine

pytestmark = pytest.mark.gpu
ROOT = Path(__file__).resolve().parents[1]
DT = {0: torch.bfloat16, 1: torch.float32}


def dev(a, dtype=torch.float32):
    return torch.from_numpy(np.array(a, np.float32)).to("cuda", dtype)


def ints(*shape):
    return torch.zeros(shape, dtype=torch.int32, device="cuda")


def host(t):
    return t.float().cpu().numpy().astype(np.float64)


def as_stored(a, f32):
    """What the storage type makes of an array."""
    return np.asarray(a, np.float64) if f32 else ora.bf16_to_f64(ora.f32_to_bf16(np.asarray(a, np.float32)))


def as_f32(a):
    return np.asarray(a, np.float32).astype(np.float64)


def rel(got, want):
    return float(np.sqrt(np.mean((got - want) ** 2)) / (np.sqrt(np.mean(np.asarray(want) ** 2)) + 1e-30))


def up(v, m):
    return (v + m - 1) // m * m


@pytest.fixture(autouse=True)
def _lib(cuda_lib):
    yield cuda_lib
    assert cuda_lib.tenzo_cuda_gemm_take_timeouts() == 0


# ---- matrix products: epilogues, segments of equal size, groups ----------------------------------------------------------
def padded(a, ld):
    out = np.zeros((a.shape[0], ld))
    out[:, :a.shape[1]] = a
    return out


@pytest.mark.parametrize("f32", [0, 1])
@pytest.mark.parametrize("M,N,K", [(1, 38, 72), (6, 130, 200), (13, 40, 64), (16, 128, 64), (45, 258, 328), (300, 514, 200)])
def test_gemm_epilogues(f32, M, N, K):
    rng = np.random.default_rng(M * N + K)
    a, w = as_stored(rng.standard_normal((M, K)), f32), as_stored(rng.standard_normal((N, K)) * K ** -0.5, 0)
    z, ld, ws = a @ w.T, up(K, 64), kernels.gemm_workspace()
    base = dict(a=dev(padded(a, ld), DT[f32]), w=dev(padded(w, ld), torch.bfloat16), M=M, N=N, ld_k=ld, seg_end=[N] + [0] * 7, f32=f32, workspace=ws, workspace_bytes=ws.numel())
    limit = 3e-6 if f32 else 3e-3
    for epilogue, act in ((2, ora.relu), (3, ora.silu)):
        c = torch.full((M, N // 2 + 2), 7.0, dtype=DT[f32], device="cuda")
        kernels.gemm(c=c, ld_c=N // 2 + 2, epilogue=epilogue, **base)
        assert rel(host(c)[:, :N // 2], act(z[:, 0::2]) * z[:, 1::2]) < limit
        assert bool((c[:, N // 2:] == 7.0).all())
    c = torch.zeros((M, N), dtype=DT[f32], device="cuda")
    kernels.gemm(c=c, ld_c=N, epilogue=4, **base)
    assert rel(host(c), z) < limit
    c = torch.zeros((M, N), device="cuda")
    kernels.gemm(c=c, ld_c=N, epilogue=5, cap=1.3, **base)
    assert rel(host(c), ora.soft_cap(z, 1.3)) < 3e-6


@pytest.mark.parametrize("f32", [0, 1])
@pytest.mark.parametrize("M,rows,n", [(1, 24, 3), (5, 40, 12), (33, 24, 5), (20, 128, 11), (300, 256, 2)])
def test_gemm_segments_of_equal_size(f32, M, rows, n):
    rng = np.random.default_rng(M + rows)
    a, w, ws = as_stored(rng.standard_normal((n, M, 64)), f32), as_stored(rng.standard_normal((n * rows, 64)), 0), kernels.gemm_workspace()
    want = np.concatenate([a[s] @ w[s * rows:(s + 1) * rows].T for s in range(n)], axis=1)
    c = torch.zeros((M, n * rows), device="cuda")
    kernels.gemm(a=dev(a, DT[f32]), w=dev(w, torch.bfloat16), M=M, N=n * rows, ld_k=64, seg_rows=rows, a_seg_stride=M * 64, c=c, ld_c=n * rows, f32=f32,
                 workspace=ws, workspace_bytes=ws.numel())
    assert rel(host(c), want) < 2e-6


@pytest.mark.parametrize("f32", [0, 1])
@pytest.mark.parametrize("experts,top,M,N,K", [(8, 3, 1, 40, 72), (5, 1, 9, 130, 64), (6, 6, 3, 38, 200), (40, 2, 33, 260, 136), (4, 2, 700, 130, 128), (3, 1, 500, 64, 64)])
def test_routed_products(f32, experts, top, M, N, K):
    """Routing, the two grouped products and the weighted sum of a row kernel, against every expert on every row."""
    rng = np.random.default_rng(experts * M + N)
    ff = N // 2
    h, logits = as_stored(rng.standard_normal((M, K)), f32), as_f32(rng.standard_normal((M, experts)) * 2)
    corr = as_f32(rng.standard_normal(experts) * 0.3)
    logits[:, experts // 2] = -30.0                                 # an expert that nobody takes while there are others
    gate, upw = as_stored(rng.standard_normal((2, experts, ff, K)) * K ** -0.5, 0)
    down = as_stored(rng.standard_normal((experts, K, ff)) * ff ** -0.5, 0)
    chosen, weights = ora.route(logits, corr, top)
    ld_k, ld_f, ws, pairs = up(K, 64), up(ff, 64), kernels.gemm_workspace(), M * top
    w1 = np.zeros((experts, 2 * ff, ld_k))
    w1[:, 0::2, :K], w1[:, 1::2, :K] = gate, upw
    w2 = np.zeros((experts, K, ld_f))
    w2[:, :, :ff] = down
    r = dict(chosen=ints(M, top), weight=torch.zeros(M, top, device="cuda"), slot=ints(M, top), row_of=ints(pairs), group_off=ints(experts + 1))
    kernels.route(logits=dev(logits), ld=experts, correction=dev(corr), experts=experts, top=top, M=M, **r)
    assert np.array_equal(r["chosen"].cpu().numpy(), chosen) and rel(host(r["weight"]), weights) < 1e-6
    off = r["group_off"].cpu().numpy()
    assert off.tolist() == [int((chosen < e).sum()) for e in range(experts + 1)]
    order = [(m, j) for e in range(experts) for m in range(M) for j in range(top) if chosen[m, j] == e]
    assert r["row_of"].cpu().tolist() == [m for m, _ in order]
    slot = r["slot"].cpu().numpy()
    assert [slot[m, j] for m, j in order] == list(range(pairs))
    common = dict(M=pairs, group_off=r["group_off"], n_group=experts, f32=f32, workspace=ws, workspace_bytes=ws.numel())
    act = torch.zeros((pairs, ld_f), dtype=DT[f32], device="cuda")
    kernels.gemm(a=dev(padded(h, ld_k), DT[f32]), w=dev(w1, torch.bfloat16), N=2 * ff, ld_k=ld_k, epilogue=3, c=act, ld_c=ld_f, a_index=r["row_of"], a_rows=M,
                 a_gather=torch.zeros((pairs, ld_k), dtype=torch.bfloat16, device="cuda"), **common)
    ye = torch.zeros((pairs, K), device="cuda")
    kernels.gemm(a=act, w=dev(w2, torch.bfloat16), N=K, ld_k=ld_f, c=ye, ld_c=K, **common)
    x, w0 = rng.standard_normal((M, K)), rng.standard_normal(K)
    out, x_out, gain = torch.zeros((M, K), device="cuda"), torch.zeros((M, K), device="cuda"), rng.standard_normal(K)
    for normed in (0, 1):
        kernels.rows(x_in=dev(x), y0=ye, ld_y=K, w0=dev(w0) if normed else None, y_slot=r["slot"], y_weight=r["weight"], n_y=top, x_out=x_out, width=K, M=M, eps=1e-5,
                     gain_w=dev(gain), out=out, ld_out=K, f32=1)
        y = np.zeros((M, K))
        for e in range(experts):
            y += np.where(chosen == e, weights, 0).sum(1, keepdims=True) * ora.glu(h, gate[e], upw[e], down[e], ora.silu)
        want = x + (ora.over_rms(y, 1e-5) * w0 if normed else y)
        assert rel(host(x_out), want) < (3e-6 if f32 else 4e-3)
        assert rel(host(out), ora.over_rms(want, 1e-5) * gain) < (3e-6 if f32 else 4e-3)


def test_route_ties_and_corrections():
    """Equal choice scores go to the lower index; a correction moves the choice and leaves the weight alone."""
    z = np.zeros((2, 5))
    z[1] = [0, 1, 2, 3, 4]
    corr = np.array([0, 0, 0.9, 0, 0])
    r = dict(chosen=ints(2, 2), weight=torch.zeros(2, 2, device="cuda"), slot=ints(2, 2), row_of=ints(4), group_off=ints(6))
    kernels.route(logits=dev(z), ld=5, correction=dev(corr), experts=5, top=2, M=2, **r)
    assert r["chosen"].cpu().tolist() == [[2, 0], [2, 4]]
    assert np.allclose(host(r["weight"]), [[0.5, 0.5], [ora.sigmoid(2.0), ora.sigmoid(4.0)]], atol=1e-6)


# ---- rows -----------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("M,width,decode", [(1, 72, 1), (5, 1030, 1), (19, 200, 0), (3, 4100, 0), (2, 4100, 1)])
def test_rows_with_a_normed_addend(M, width, decode):
    rng = np.random.default_rng(width)
    x, y, w0, gain = rng.standard_normal((M, width)), rng.standard_normal((M, width)), rng.standard_normal(width), rng.standard_normal(width)
    out, x_out = torch.zeros((M, width), device="cuda"), torch.zeros((M, width), device="cuda")
    kernels.rows(x_in=dev(x), y0=dev(y), ld_y=width, w0=dev(w0), x_out=x_out, width=width, M=M, eps=1e-3, gain=0.5, gain_w=dev(gain), decode=decode, out=out, ld_out=width,
                 row_inv=torch.empty(M, device="cuda"), f32=1)
    want = x + ora.over_rms(y, 1e-3) * w0
    assert rel(host(x_out), want) < 1e-6 and rel(host(out), ora.over_rms(want, 1e-3) * gain * 0.5) < 2e-6
    emb = as_stored(rng.standard_normal((9, width)), 0)
    tok = np.arange(M) * 2 % 9
    kernels.rows(tokens=torch.from_numpy(tok.astype(np.int32)).cuda(), embed=dev(emb, torch.bfloat16), vocab=9, x_out=x_out, width=width, M=M, eps=1e-3, gain_w=dev(gain),
                 decode=decode, out=out, ld_out=width, row_inv=torch.empty(M, device="cuda"), f32=1)
    assert rel(host(x_out), emb[tok]) == 0 and rel(host(out), ora.over_rms(emb[tok], 1e-3) * gain) < 2e-6


# ---- delta rule ---------------------------------------------------------------------------------------------------------------
class Delta:
    """The delta rule's kernels with their carried state over one sequence."""

    def __init__(self, f32, heads, kv, dim, vdim, taps, rng, spread=1.0):
        self.__dict__.update(locals())
        self.nk, self.nv = kv * dim, heads * vdim
        self.conv = [as_f32(rng.standard_normal((c, taps)) * 0.5 + 0.3) for c in (self.nk, self.nk, self.nv)]
        self.a_log, self.dt, self.norm = as_f32(spread * rng.standard_normal(heads) - 2), as_f32(rng.standard_normal(heads)), as_f32(rng.standard_normal(vdim))
        self.off = np.cumsum([0, self.nk, self.nk, self.nv, self.nv, heads, heads])
        self.eps, self.q_scale = 1e-4, dim ** -0.5
        self.reset()

    def reset(self):
        self.state = torch.zeros((self.heads, self.dim, up(self.vdim, 4)), device="cuda")
        self.tail = torch.zeros((self.taps, 2 * self.nk + self.nv), device="cuda")
        self.pos = 0

    def run(self, x, decode=None):
        M, o = len(x), self.off
        d = dev(x)
        out = torch.zeros((M, self.nv), dtype=DT[self.f32], device="cuda")
        part = lambda i: d[:, o[i]:]
        cw = [dev(c.T.copy()) for c in self.conv]
        kernels.delta_rule(q=d, k=part(1), v=part(2), g=part(3), a=part(4), b=part(5), ld=d.shape[1], conv_q=cw[0], conv_k=cw[1], conv_v=cw[2], taps=self.taps,
                           tail=self.tail, heads=self.heads, kv_heads=self.kv, dim=self.dim, vdim=self.vdim, q_scale=self.q_scale, a_log=dev(self.a_log),
                           dt_bias=dev(self.dt), norm=dev(self.norm), eps=self.eps, state=self.state, pos=torch.tensor([self.pos], dtype=torch.int32, device="cuda"),
                           pos0=self.pos, M=M, decode=int(M == 1) if decode is None else decode, out=out, ld_out=self.nv,
                           work=kernels.delta_rule_work(M, self.heads, self.kv, self.dim, self.vdim), f32=self.f32)
        torch.cuda.synchronize()
        self.pos += M
        return host(out)

    def want(self, x):
        T, H, o = len(x), self.heads, self.off
        q, k, v = (ora.silu(ora.causal_conv(x[:, a:b], w)) for a, b, w in zip(o[:3], o[1:4], self.conv))
        hd = lambda u, n: u.reshape(T, n, -1)
        q, k = (np.repeat(ora.unit_vectors(hd(u, self.kv)), H // self.kv, axis=1) for u in (q, k))
        y = ora.delta_recurrence(q * self.q_scale, k, hd(v, H), ora.head_decay(x[:, o[4]:o[5]], self.a_log, self.dt), ora.sigmoid(x[:, o[5]:]))
        y = ora.over_rms(y, self.eps) * self.norm
        return y.reshape(T, -1) * ora.silu(x[:, o[3]:o[4]])


DELTA = [(4, 2, 64, 64, 4), (3, 3, 32, 48, 2), (6, 2, 20, 50, 3), (2, 1, 100, 128, 1), (4, 1, 128, 36, 5), (1, 1, 256, 256, 4), (3, 1, 1, 3, 7), (10, 10, 8, 20, 16)]


@pytest.mark.parametrize("heads,kv,dim,vdim,taps", DELTA)
def test_delta_rule(heads, kv, dim, vdim, taps):
    T = 150
    rng = np.random.default_rng(heads * dim + vdim)
    x = as_f32(rng.standard_normal((T, 2 * kv * dim + 2 * heads * vdim + 2 * heads)))
    d = Delta(1, heads, kv, dim, vdim, taps, rng)
    want = d.want(x)
    for cuts in ([T], [1] * 40 + [2, 108], [64, 2, 3, 1, 1, 7, 8, 9, 45, 10], [2] * 10 + [1] * 3 + [127]):
        got = np.concatenate([d.run(part) for part in np.split(x, np.cumsum(cuts)[:-1])])
        assert rel(got, want) < 2e-5, cuts
        d.reset()
    got = np.concatenate([d.run(x[:5], decode=0)] + [d.run(x[5:6], decode=0)] + [d.run(x[6:])])      # one row as a chunk
    assert rel(got, want) < 2e-5
    low = Delta(0, heads, kv, dim, vdim, taps, np.random.default_rng(0))
    assert rel(low.run(x), low.want(x)) < 4e-3


def test_delta_rule_decays_of_any_size():
    """Rows that forget everything beside rows that forget nothing, inside one block of rows."""
    rng = np.random.default_rng(4)
    x = as_f32(rng.standard_normal((90, 2 * 32 + 2 * 64 + 4)))
    x[::7, -4:-2] = 400.0                                       # decay of exp(-400 e^a_log): the state is gone
    x[3::5, -4:-2] = -60.0                                      # and of 1
    x[4::9, -2:] = 50.0                                         # full steps
    d = Delta(1, 2, 1, 32, 32, 2, rng)
    d.a_log = np.array([1.0, -1.0])
    want = d.want(x)
    for cuts in ([90], [1] * 20 + [70], [13, 20, 2, 55]):
        assert rel(np.concatenate([d.run(part) for part in np.split(x, np.cumsum(cuts)[:-1])]), want) < 2e-5
        d.reset()


@pytest.mark.parametrize("f32", [0, 1])
def test_delta_rule_slots_side_by_side(f32):
    """Decode rows of several sequences at different positions, each against its own history."""
    rng = np.random.default_rng(8)
    B, heads, kv, dim, vdim, taps = 5, 4, 2, 24, 40, 4
    one = Delta(f32, heads, kv, dim, vdim, taps, rng)
    xs = [as_f32(rng.standard_normal((n + 6, one.off[-1]))) for n in (0, 1, 3, 20, 9)]
    state = torch.zeros((B,) + tuple(one.state.shape), device="cuda")
    tail = torch.zeros((B,) + tuple(one.tail.shape), device="cuda")
    for s, x in enumerate(xs):
        one.reset()
        if len(x) > 6:
            one.run(x[:-6], decode=0)
        state[s], tail[s] = one.state, one.tail
    want = [one.want(x)[-6:] for x in xs]
    cw, o = [dev(c.T.copy()) for c in one.conv], one.off
    for i in range(6):
        d = dev(np.stack([x[len(x) - 6 + i] for x in xs]))
        out = torch.zeros((B, one.nv), dtype=DT[f32], device="cuda")
        kernels.delta_rule(q=d, k=d[:, o[1]:], v=d[:, o[2]:], g=d[:, o[3]:], a=d[:, o[4]:], b=d[:, o[5]:], ld=d.shape[1], conv_q=cw[0], conv_k=cw[1], conv_v=cw[2],
                           taps=taps, tail=tail, tail_seq_stride=tail[0].numel(), heads=heads, kv_heads=kv, dim=dim, vdim=vdim, q_scale=one.q_scale, a_log=dev(one.a_log),
                           dt_bias=dev(one.dt), norm=dev(one.norm), eps=one.eps, state=state, state_seq_stride=state[0].numel(),
                           pos=torch.tensor([len(x) - 6 + i for x in xs], dtype=torch.int32, device="cuda"), M=B, decode=1, out=out, ld_out=one.nv, f32=f32)
        assert rel(host(out), np.stack([w[i] for w in want])) < (2e-5 if f32 else 4e-3)


# ---- latent attention -------------------------------------------------------------------------------------------------------
class Latent:
    """Latent attention with its cache over one sequence; `readers` are further sets of heads that borrow the cache."""

    def __init__(self, f32, heads, dim, rot, vdim, rank, window, rng, ring=None, base=1000.0, owner=None, scale=None):
        self.__dict__.update(locals())
        self.ring = ring or (owner.ring if owner else window)
        self.scale = scale or (dim + rot) ** -0.5
        self.d8, self.r8, self.v8, self.ld = up(dim, 8), up(rot, 8), up(vdim, 8), up(rank, 64)
        self.uk, self.uv = (as_stored(rng.standard_normal((heads, n, rank)) * rank ** -0.5, 0) for n in (dim, vdim))
        w = np.zeros((heads * (self.d8 + self.v8), self.ld))
        for h in range(heads):
            w[h * self.d8:h * self.d8 + dim, :rank] = self.uk[h]
            w[heads * self.d8 + h * self.v8:][:vdim, :rank] = self.uv[h]
        self.w = dev(w, torch.bfloat16)
        if owner:
            self.norm, self.rc, self.rr, self.lin = owner.norm, owner.rc, owner.rr, owner.lin
        else:
            self.norm = as_f32(1 + 0.2 * rng.standard_normal(rank))
            self.rc, self.rr = (torch.zeros((self.ring, n), dtype=DT[f32], device="cuda") for n in (self.ld, self.r8))
            self.lin = {}
        self.freq = torch.from_numpy(base ** (-2.0 * np.arange(rot // 2) / rot)).cuda()
        self.ws, self.pos = kernels.gemm_workspace(), 0

    def run(self, q, dkv, decode=None):
        M, H, dt = len(q), self.heads, DT[self.f32]
        x = dev(np.concatenate([q, dkv], axis=1))
        buf = lambda *s: torch.zeros(s, dtype=dt, device="cuda")
        out = buf(M, H * self.v8)
        if self.owner is None:
            self.lin["c"], self.lin["r"] = buf(M + self.ring, self.ld), buf(M + self.ring, self.r8)
        kernels.latent_attention(q=x, dkv=None if self.owner else x[:, q.shape[1]:], ld=x.shape[1], norm=dev(self.norm), eps=1e-5, freq=self.freq, heads=H, dim=self.dim,
                                 rot=self.rot, vdim=self.vdim, rank=self.rank, scale=self.scale, window=self.window, w_kv=self.w, ring_c=self.rc, ring_r=self.rr, ring=self.ring,
                                 pos=torch.tensor([self.pos], dtype=torch.int32, device="cuda"), pos0=self.pos, M=M, decode=int(M == 1) if decode is None else decode, out=out,
                                 ld_out=H * self.v8, lin_q=buf(M, H, self.d8 + self.r8), lin_c=self.lin["c"], lin_r=self.lin["r"],
                                 kv=buf(M + self.window, H * (self.d8 + self.v8)), q_abs=torch.zeros((M, H, self.ld), device="cuda"), lat=buf(H, M, self.ld),
                                 workspace=self.ws, workspace_bytes=self.ws.numel(), f32=self.f32)
        torch.cuda.synchronize()
        self.pos += M
        y = host(out).reshape(M, H, self.v8)
        assert not y[:, :, self.vdim:].any()
        return y[:, :, :self.vdim].reshape(M, -1)

    def want(self, q, dkv):
        T, H = len(q), self.heads
        q = q.reshape(T, H, -1)
        c = as_stored(ora.over_rms(dkv[:, :self.rank], 1e-5) * self.norm, self.f32)
        k = as_stored(ora.rotate_halves(dkv[:, self.rank:], range(T), self.base), self.f32)
        return ora.latent_attention(q[:, :, :self.dim], ora.rotate_halves(q[:, :, self.dim:], range(T), self.base), c, k, self.uk, self.uv, self.scale, self.window).reshape(T, -1)


LATENT = [(4, 24, 16, 40, 72, 19), (1, 40, 6, 20, 64, 1), (20, 16, 8, 16, 130, 64), (3, 128, 64, 128, 512, 33), (17, 36, 10, 128, 256, 200), (2, 100, 32, 72, 700, 50),
          (5, 200, 100, 256, 96, 7), (6, 64, 32, 64, 192, 300)]


@pytest.mark.parametrize("f32", [0, 1])
@pytest.mark.parametrize("heads,dim,rot,vdim,rank,window", LATENT)
def test_latent_attention(f32, heads, dim, rot, vdim, rank, window):
    T = 400
    rng = np.random.default_rng(heads * dim + window)
    q, dkv = as_f32(rng.standard_normal((T, heads * (dim + rot)))), as_f32(rng.standard_normal((T, rank + rot)))
    for cuts in ([T], [2, 100, 1, 1, 7, 64, 2] + [1] * 60 + [163], [37] + [1] * 20 + [3, 2, 130, 208]):
        att = Latent(f32, heads, dim, rot, vdim, rank, window, np.random.default_rng(7))
        want = att.want(q, dkv)
        at = np.cumsum(cuts)[:-1]
        got = np.concatenate([att.run(*part) for part in zip(np.split(q, at), np.split(dkv, at))])
        assert rel(got, want) < (3e-6 if f32 else 8e-3), cuts
        assert np.abs(got - want).max() < (3e-5 if f32 else 8e-2), cuts


@pytest.mark.parametrize("f32", [0, 1])
@pytest.mark.parametrize("B,heads,dim,rot,vdim,rank,window", [(2, 3, 20, 4, 16, 72, 5), (15, 4, 100, 10, 24, 130, 40), (70, 2, 128, 64, 128, 512, 33)])
def test_latent_attention_of_sequences_side_by_side(f32, B, heads, dim, rot, vdim, rank, window):
    """Decode rows of several sequences at different positions, each against its own history."""
    rng = np.random.default_rng(B)
    one = Latent(f32, heads, dim, rot, vdim, rank, window, rng)
    xs = [(as_f32(rng.standard_normal((n + 2, heads * (dim + rot)))), as_f32(rng.standard_normal((n + 2, rank + rot)))) for n in rng.integers(0, 3 * window, B)]
    rc, rr = (torch.zeros((B,) + tuple(t.shape), dtype=DT[f32], device="cuda") for t in (one.rc, one.rr))
    for s, (q, dkv) in enumerate(xs):
        one.pos = 0
        one.rc.zero_(), one.rr.zero_()
        if len(q) > 2:
            one.run(q[:-2], dkv[:-2], decode=0)
        rc[s], rr[s] = one.rc, one.rr
    want = np.stack([one.want(q, dkv)[-2:] for q, dkv in xs])
    got = []
    for i in range(2):
        x = dev(np.stack([np.concatenate([q[len(q) - 2 + i], dkv[len(q) - 2 + i]]) for q, dkv in xs]))
        out = torch.zeros((B, heads * one.v8), dtype=DT[f32], device="cuda")
        kernels.latent_attention(q=x, dkv=x[:, heads * (dim + rot):], ld=x.shape[1], norm=dev(one.norm), eps=1e-5, freq=one.freq, heads=heads, dim=dim, rot=rot, vdim=vdim, rank=rank,
                                 scale=one.scale, window=window, w_kv=one.w, ring_c=rc, ring_r=rr, ring=window, ring_c_stride=rc[0].numel(), ring_r_stride=rr[0].numel(),
                                 pos=torch.tensor([len(q) - 2 + i for q, _ in xs], dtype=torch.int32, device="cuda"), M=B, decode=1, out=out, ld_out=heads * one.v8,
                                 q_abs=torch.zeros((B, heads, one.ld), device="cuda"), lat=torch.zeros((heads, B, one.ld), dtype=DT[f32], device="cuda"), workspace=one.ws,
                                 workspace_bytes=one.ws.numel(), f32=f32)
        got.append(host(out).reshape(B, heads, one.v8)[:, :, :vdim].reshape(B, -1))
    assert rel(np.stack(got, axis=1), want) < (3e-6 if f32 else 8e-3)


@pytest.mark.parametrize("f32", [0, 1])
@pytest.mark.parametrize("windows", [(9, 40), (40, 9), (70, 70), (1, 130)])
def test_a_borrowed_latent_cache(f32, windows):
    """A second set of heads with a window of its own reads the rows that the first one left; the ring serves the wider window."""
    T, rank, rot = 300, 80, 12
    rng = np.random.default_rng(windows[0])
    own = Latent(f32, 3, 20, rot, 16, rank, windows[0], rng, ring=max(windows))
    other = Latent(f32, 5, 32, rot, 24, rank, windows[1], rng, owner=own)
    q1, q2, dkv = (as_f32(rng.standard_normal((T, n))) for n in (3 * 32, 5 * 44, rank + rot))
    a, b, at = [], [], 0
    for n in [50, 2, 1, 1, 3, 64] + [1] * 90 + [80, 9]:
        a.append(own.run(q1[at:at + n], dkv[at:at + n]))
        b.append(other.run(q2[at:at + n], dkv[at:at + n]))
        at += n
    assert at == T
    limit = 3e-6 if f32 else 8e-3
    assert rel(np.concatenate(a), own.want(q1, dkv)) < limit and rel(np.concatenate(b), other.want(q2, dkv)) < limit


@pytest.mark.parametrize("f32", [0, 1])
@pytest.mark.parametrize("decode", [False, True])
@pytest.mark.parametrize("window", [1, 8, 33, 64, 129])
def test_latent_window_edge_shows(f32, decode, window):
    """One key matches one query so strongly that it takes all the weight when it is inside the window - at the last place
    inside, and at the first place outside."""
    rng = np.random.default_rng(window)
    dim, rot, rank, vdim = 64, 2, 64, 64
    for back in (window - 1, window):
        T, at = window + 40, window + 30                  # the query's row
        q, dkv = 0.1 * rng.standard_normal((T, dim + rot)), rng.standard_normal((T, rank + rot))
        d = rng.standard_normal(rank)
        d /= np.linalg.norm(d)
        dkv[:, :rank] -= np.outer(dkv[:, :rank] @ d, d)
        dkv[:, rank:] = 0
        dkv[at - back, :rank] = 20 * d
        q[at, :dim] = 60 * d
        att = Latent(f32, 1, dim, rot, vdim, rank, window, rng, scale=1.0)
        att.norm = np.ones(rank)
        att.uk[0] = np.eye(rank)
        att.uv[0] = as_stored(3 * np.outer(np.ones(vdim), d), 0)
        att.w[:64] = dev(att.uk[0], torch.bfloat16)
        att.w[64:] = dev(att.uv[0], torch.bfloat16)
        q, dkv = as_f32(q), as_f32(dkv)
        parts = [(0, at)] + [(i, i + 1) for i in range(at, T)] if decode else [(0, 5), (5, T)]
        got = np.concatenate([att.run(q[a:b], dkv[a:b]) for a, b in parts])
        want = att.want(q, dkv)
        assert (want[at].mean() > 10) == (back < window)   # the case discriminates
        assert np.abs(got - want).max() < (2e-4 if f32 else 0.1)


def test_rotation_far_out():
    """Angles of a late position are as exact as those of an early one: a single key turned away by its distance alone."""
    rng = np.random.default_rng(1)
    att = Latent(1, 1, 8, 64, 8, 64, 4, rng, base=10000.0)
    att.pos = 700_001
    q, dkv = as_f32(rng.standard_normal((6, 72))), as_f32(rng.standard_normal((6, 128)))
    got = np.concatenate([att.run(q[:3], dkv[:3]), att.run(q[3:4], dkv[3:4]), att.run(q[4:], dkv[4:])])
    near = Latent(1, 1, 8, 64, 8, 64, 4, np.random.default_rng(1), base=10000.0)
    want = near.want(q, dkv)
    # the cache in front of position 700001 is zero here, so rows whose window reaches it differ; the last three do not
    assert rel(got[3:], want[3:]) < 5e-6


# ---- models -------------------------------------------------------------------------------------------------------------------
def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def delta(heads, kv, dim, vdim, conv, mlp=None):
    return {"type": "delta", "mlp": mlp, "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "conv": conv}}


def latent(heads, dim, rot, vdim, rank, size, mlp=None, base=500.0, scale=None, kv_from=None):
    mix = {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "mask": {"size": size}, "rot": {"base": base, "dims": rot},
           "scale": scale or (dim + rot) ** -0.5}
    return {"type": "latent_attention", "mlp": mlp, "mixer": dict(mix, kv_from=kv_from) if kv_from is not None else mix}


def config(layers, width=96, vocab=210, eps=1e-5, cap=9.0):
    return {"vocab": vocab, "width": width, "norm": {"eps": eps}, "logit_softcap": cap, "layers": layers}


MODELS = {
    "delta_alone": config([delta(6, 3, 20, 28, 3), delta(2, 2, 40, 32, 1, dense(100))], width=80),
    "latent_alone": config([latent(4, 24, 16, 20, 72, 19, dense(130)), latent(3, 32, 8, 40, 40, 33)], width=72),
    "experts": config([delta(2, 1, 32, 32, 2, moe(6, 2, 40)), delta(1, 1, 16, 48, 4, moe(9, 1, 24)), latent(2, 16, 8, 16, 24, 12, moe(3, 3, 70))], width=64),
    "mixed": config([latent(3, 20, 12, 36, 80, 21, moe(7, 3, 48), base=900.0), delta(4, 2, 24, 40, 4, dense(150)), latent(5, 16, 12, 24, 80, 47, dense(90), kv_from=0, base=900.0),
                     delta(3, 3, 36, 12, 3, moe(12, 4, 20)), latent(2, 28, 6, 16, 56, 30, None), latent(4, 12, 12, 8, 80, 9, moe(5, 1, 33), kv_from=0, base=900.0),
                     delta(8, 2, 16, 16, 2, None)], width=120, vocab=301, eps=1e-3, cap=4.0),
    "wide_heads": config([delta(2, 1, 128, 128, 4, dense(300)), latent(2, 128, 64, 128, 512, 128, moe(16, 4, 64)), latent(17, 16, 64, 16, 512, 40, None, kv_from=1)], width=256),
    "one_of_each": config([delta(1, 1, 8, 8, 1, moe(1, 1, 16)), latent(1, 8, 2, 8, 16, 1, dense(16))], width=40, vocab=33),
}


def clear_choices(tensors):
    """Corrections far apart: which experts a token takes does not hang on rounding (how much of them still does)."""
    for n in tensors:
        if n.endswith(".correction"):
            tensors[n] = 2.0 * np.random.default_rng(len(n) + int(n[1:n.index(".")])).permutation(len(tensors[n])).astype(np.float32)


@pytest.fixture(scope="module")
def model(tmp_path_factory):
    """Folder, configuration, weights, tokens and expected logits. A close choice of experts that bf16 rounding flips moves
    every later row, so the models that run in bf16 have clear choices."""
    made = {}

    def get(name, compute="float32"):
        key = name, compute
        if key not in made:
            cfg = MODELS[name]
            folder = tmp_path_factory.mktemp(name)
            change = clear_choices if compute == "bfloat16" else None
            W = {n: a.astype(np.float64) for n, a in synth.write_tigitar(folder, cfg, seed=len(name), change=change).items()}
            tokens = np.random.default_rng(3).integers(0, cfg["vocab"], 260)
            made[key] = folder, cfg, W, tokens, ora.forward(cfg, W, tokens)
        return made[key]

    return get


LIMIT = {"float32": 1e-4, "bfloat16": 5e-2}


def close(got, want, compute):
    """Root mean square errors against the logits' own size: over all rows, and (a head's output is divided by its own size,
    which is small at some positions and lets rounding show there) three times that for a single row."""
    d = got - want
    err = np.sqrt(np.mean(d * d, axis=-1)) / np.sqrt(np.mean(want * want))
    assert np.sqrt(np.mean(err * err)) < LIMIT[compute] and err.max() < 3 * LIMIT[compute], (err.max(), int(err.argmax()))


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
    folder, cfg, W, tokens, want = model(name, compute)
    with Engine.open(folder, compute=compute) as e:
        assert e.config.hidden_size == cfg["width"] and e.config.vocab_size == cfg["vocab"]
        for cuts in ([260], [200] + [1] * 60, [2] * 9 + [3, 1, 64, 15, 1, 1, 2, 60, 80, 15], [1] * 40 + [2, 100, 7, 111]):
            close(feed(e, tokens, cuts), want, compute)
            assert e.seq_len() == 260
            e.reset()                                       # the same slot again, with other leftovers every time


@pytest.mark.parametrize("compute", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["mixed", "wide_heads"])
def test_residual_after_every_layer(model, name, compute, tmp_path):
    folder, cfg, W, tokens, _ = model(name, compute)
    layers = []
    ora.forward(cfg, W, tokens[:40], layers)
    for n in range(1, len(cfg["layers"]) + 1):
        d = tmp_path / str(n)
        d.mkdir()
        (d / "config.json").write_text(json.dumps(dict(cfg, architecture="Tigitar", layers=cfg["layers"][:n])))
        (d / "model.safetensors").symlink_to(folder / "model.safetensors")
        with Engine.open(d, compute=compute) as e:
            e.prefill_chunk(tokens[:30])
            assert rel(e.read_buffer(0), layers[n - 1][29]) < 2 * LIMIT[compute]
            for i in range(30, 40):
                e.prefill_token(tokens[i])
                assert rel(e.read_buffer(0), layers[n - 1][i]) < 2 * LIMIT[compute]


def test_one_layer_of_a_step(model):
    folder, cfg, W, tokens, _ = model("mixed")
    layers = []
    ora.forward(cfg, W, tokens[:1], layers)
    with Engine.open(folder, compute="float32") as e:
        e.write_x(W["embed"][tokens[0]])
        for l in range(len(layers)):
            e.run_layer(l)
            assert rel(e.read_buffer(0), layers[l][0]) < LIMIT["float32"]


@pytest.mark.parametrize("compute", ["float32", "bfloat16"])
def test_slots_are_independent_and_reusable(model, compute):
    """Unequal requests side by side, then batched decoding of all slots, then one slot given back and taken by another."""
    folder, cfg, W, tokens, want = model("mixed", compute)
    lens = [5, 90, 1, 33]
    other = np.random.default_rng(9).integers(0, cfg["vocab"], 60)
    other_want = ora.forward(cfg, W, other)
    with Engine.open(folder, compute=compute, batch=4) as e:
        for s, n in enumerate(lens):
            close(feed(e, tokens[:n], [n], seq=s), want[:n], compute)
        got, expect = [], []
        for i in range(12):
            e.generate_steps([tokens[n + i] for n in lens])
            got += [e.read_buffer(15, seq=s) for s in range(4)]
            expect += [want[n + i] for n in lens]
        close(np.stack(got), np.stack(expect), compute)
        e.reset_seq(1)
        close(feed(e, other, [20, 2, 38], seq=1), other_want, compute)
        at = lens[3] + 12
        close(e.forward(tokens[at:at + 8], range(8), seq=3), want[at:at + 8], compute)      # untouched by its neighbours


@pytest.mark.parametrize("name", ["mixed", "wide_heads"])
def test_wide_batches_take_the_tensor_cores(model, name):
    folder, cfg, W, tokens, want = model(name, "bfloat16")
    with Engine.open(folder, batch=40) as e:
        for s in range(40):
            e.forward(tokens[:s + 1], seq=s)
        for i in range(6):
            e.generate_steps([tokens[s + 1 + i] for s in range(40)])
        got = np.stack([e.read_buffer(15, seq=s) for s in range(40)])
        close(got, want[np.arange(40) + 6], "bfloat16")


def test_long_decoding(model):
    folder, cfg, W, _, _ = model("mixed")
    tokens = np.random.default_rng(11).integers(0, cfg["vocab"], 700)
    want = ora.forward(cfg, W, tokens)
    with Engine.open(folder, compute="float32") as e:
        close(feed(e, tokens, [3] + [1] * 697), want, "float32")


def test_a_prompt_longer_than_a_chunk(model):
    """Prompts of more than 4096 tokens go through in several portions."""
    folder, cfg, W, _, _ = model("latent_alone")
    tokens = np.random.default_rng(12).integers(0, cfg["vocab"], 4200)
    want = ora.forward(cfg, W, tokens[-120:])               # two windows of 19 and 33: the last rows see no further back than that
    with Engine.open(folder, compute="float32") as e:
        got = e.forward(tokens, range(4100, 4200))
        # rotation is relative, so the same keys at other positions give the same scores
        close(got[60:], want[80:], "float32")


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


def test_batched_greedy_generation(model):
    """Requests of unequal length decoded together on the device give what each gives alone."""
    folder, cfg, W, tokens, _ = model("mixed")
    prompts = [tokens[a:b].tolist() for a, b in ((0, 4), (10, 60), (100, 102))]
    want = [ora.greedy(cfg, W, p, 10) for p in prompts]
    with Engine.open(folder, compute="float32", batch=3) as e:
        for s, p in enumerate(prompts):
            e.forward(p[:-1], seq=s)
        assert e.decode_greedy([p[-1] for p in prompts], 10).T.tolist() == want


@pytest.mark.parametrize("compute", ["float32", "bfloat16"])
def test_far_tokens_show(tmp_path, compute):
    """Slow decays, and keys and values that favour one direction of the input: an early token that lies along it is felt
    hundreds of tokens later, and the model with it and without it are told apart."""
    cfg = config([delta(2, 1, 32, 32, 2)], width=64, vocab=50)

    def change(t):
        d = t["embed"][7] / np.linalg.norm(t["embed"][7])
        t["embed"][8:] -= 0.98 * np.outer(t["embed"][8:] @ d, d)
        t["l0.mix.A_log"][:] = -9.0                              # decays of exp(-1e-4 softplus)
        t["l0.mix.q"] = 0.2 * t["l0.mix.q"]
        t["l0.mix.q.conv"][:] = [0, 1]
        t["l0.mix.k.conv"][:] = [0, 1]
        key = np.abs(np.random.default_rng(0).standard_normal(32)) * 3
        t["l0.mix.k"] = 0.3 * t["l0.mix.k"] + np.outer(key, d) * 4
        t["l0.mix.q"] += np.outer(key, t["embed"][9] / np.linalg.norm(t["embed"][9]))
        t["l0.mix.v"] = t["l0.mix.v"] + 6 * np.outer(np.abs(np.random.default_rng(1).standard_normal(64)), d)

    W = {n: a.astype(np.float64) for n, a in synth.write_tigitar(tmp_path, cfg, seed=5, change=change).items()}
    moved = np.random.default_rng(2).integers(8, 50, 400)
    moved[250::10] = 9                                           # a token that asks along the marked direction
    tokens = moved.copy()
    tokens[20] = 7
    want, without = ora.forward(cfg, W, tokens), ora.forward(cfg, W, moved)
    felt = rel(without[250::10], want[250::10])
    assert felt > 0.05
    with Engine.open(tmp_path, compute=compute) as e:
        for t, w in ((tokens, want), (moved, without)):
            got = feed(e, t, [100, 2, 65, 200] + [1] * 33)
            assert rel(got[250::10], w[250::10]) < (3e-5 if compute == "float32" else felt / 4)
            e.reset()


def folder_with(path, text):
    path.mkdir(exist_ok=True)
    (path / "config.json").write_text(text)
    return path


def test_broken_folders_are_reported(tmp_path, model):
    folder, cfg, *_ = model("mixed")

    def refused(name, match, **change):
        d = folder_with(tmp_path / name, json.dumps(dict(cfg, architecture="Tigitar", **change)))
        (d / "model.safetensors").symlink_to(folder / "model.safetensors")
        with pytest.raises(RuntimeError, match=match):
            Engine.open(d)

    edit = lambda i, f: [f(json.loads(json.dumps(l))) if i == j else l for j, l in enumerate(cfg["layers"])]
    refused("width", "shape", width=cfg["width"] + 8)
    refused("type", "unknown type", layers=edit(1, lambda l: dict(l, type="other")))
    refused("mlp", "unknown feed-forward", layers=edit(1, lambda l: dict(l, mlp={"kind": "other"})))
    refused("from", "kv_from", layers=edit(2, lambda l: dict(l, mixer=dict(l["mixer"], kv_from=1))))
    refused("later", "kv_from", layers=edit(2, lambda l: dict(l, mixer=dict(l["mixer"], kv_from=4))))
    refused("rot", "rotated", layers=edit(2, lambda l: dict(l, mixer=dict(l["mixer"], rot={"base": 900.0, "dims": 6}))))
    refused("top", "experts per token", layers=edit(0, lambda l: dict(l, mlp=moe(7, 8, 48))))
    refused("cap", "positive", logit_softcap=0)


def test_a_state_cannot_be_cut_back(model):
    folder, cfg, W, tokens, _ = model("mixed")
    with Engine.open(folder) as e:
        e.prefill_chunk(tokens[:10])
        with pytest.raises(RuntimeError, match="recurrent state"):
            e.set_seq_len(0, 4)
        e.set_seq_len(0, 0)
        with pytest.raises(RuntimeError, match="token id"):
            e.forward([cfg["vocab"]])


# ---- command line ----------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("compute", ["float32", "bfloat16"])
def test_trace_replay(model, compute, tmp_path):
    folder, cfg, W, tokens, want = model("latent_alone")
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
    folder, cfg, W, tokens, _ = model("experts")
    prompt = tokens[:9].tolist()
    r = subprocess.run([sys.executable, "-m", "tenzo_b200", "generate", "--model", str(folder), "--dtype", "float32", "--n", "6", "--tokens",
                        ",".join(map(str, prompt))], capture_output=True, text=True, timeout=300, cwd=ROOT)
    assert r.returncode == 0, r.stderr
    assert [int(t) for t in r.stdout.split()] == ora.greedy(cfg, W, prompt, 6)
