"""`bench.py --workload sozopel`: the Sozopel hybrid decoder beside BitNet at equal size.

Models of 8 layers with random weights at three widths (vocabulary 32768, the feed-forward of the BitNet shape of that
width in both): prompt throughput (one 2048-token chunk), decode throughput of one sequence and of 64. Then every kernel
of the new design alone, at the largest width, against its roofline, and the like kernel of BitNet against its own:
inputs rotate over more than the L2 cache, one CUDA graph per measurement, CUDA events around its replays.
"""
from __future__ import annotations

import json
import tempfile
import time
from pathlib import Path

import numpy as np

from . import synth

SIZES = {1024: 2816, 2048: 5632, 2560: 6912}             # width -> feed-forward
LAYERS, VOCAB, CHUNK, BATCH, WINDOW = 8, 32768, 2048, 64, 1024
FP32_TFLOPS = 148 * 128 * 2 * 1.9e9 / 1e12                # FMA units at 1.9 GHz (no measured peak of the plain pipeline)


def _peaks():
    p = Path(__file__).resolve().parents[1] / "MEASURED_PEAKS.json"
    if p.exists():
        d = json.loads(p.read_text())
        return float(d["hbm_gbs"]) * 1e9, float(d["bf16_tflops"]) * 1e12, "measured"
    return 6650e9, 1590e12, "fallback"


def sozopel_config(width: int, ff: int) -> dict:
    heads = width // 128
    left = {"heads": heads, "kv_heads": max(1, heads // 4), "dim": 128, "vdim": 128, "conv": 4, "mask": {"size": WINDOW}, "scale": 128 ** -0.5}
    mlp = {"kind": "dense", "ff": ff}
    par = {"type": "parallel", "mixer": {"left": left, "right": {"heads": heads, "dim": 64, "vdim": 128, "tau": 16.0}}, "mlp": mlp}
    ret = {"type": "retention", "mixer": {"heads": heads, "dim": 64, "vdim": 128, "decay": [1 - 2.0 ** -(5 + i % 8) for i in range(heads)]}, "mlp": mlp}
    wkv = {"type": "wkv", "mixer": {"heads": width // 64, "dim": 64}, "mlp": mlp}
    return {"vocab": VOCAB, "width": width, "max_positions": 16384, "norm": {"eps": 1e-5}, "canon": {"taps": 4}, "layers": [par, wkv, ret, par, wkv, ret, par, wkv]}


def bitnet_config(width: int, ff: int) -> dict:
    heads = width // 128
    kv = next(k for k in range(max(1, heads // 4), heads + 1) if heads % k == 0 and heads // k in (1, 2, 4, 8))
    return dict(hidden_size=width, num_q_heads=heads, num_kv_heads=kv, head_dim=128, num_layers=LAYERS, ffn_dim=ff, vocab_size=VOCAB, max_seq_len=4096)


def _median(f, n=5):
    return float(np.median([f() for _ in range(n)]))


def _engine_numbers(one, many, reset, steps):
    """Milliseconds of a prompt chunk and of a decode step at batch 1 and BATCH."""
    prompt = synth.prompt_tokens(1, CHUNK, VOCAB)

    def prefill():
        reset(one)
        one.synchronize()
        t0 = time.perf_counter()
        one.prefill_chunk(prompt)
        one.synchronize()
        wall = (time.perf_counter() - t0) * 1e3
        ms = one.last_device_ms()
        return ms if 0 < ms < wall else wall

    prefill()
    pf = _median(prefill)

    def decode(e):
        first = synth.prompt_tokens(2, e.batch, VOCAB)
        e.decode_greedy(first, 8)

        def run():
            e.decode_greedy(first, steps)
            return e.last_device_ms() / steps
        return _median(run)

    d1, db = decode(one), decode(many)
    return {"prefill_tok_s": CHUNK / pf * 1e3, "prefill_ms": pf, "decode_b1_tok_s": 1e3 / d1, "decode_b1_ms": d1,
            f"decode_b{BATCH}_tok_s": BATCH * 1e3 / db, f"decode_b{BATCH}_ms": db}


def _models(width, ff, steps):
    from .engine import Engine
    out = {}
    cfg = sozopel_config(width, ff)
    with tempfile.TemporaryDirectory() as d:
        synth.write_sozopel_pooled(d, cfg, rank=64, seed=0)
        with Engine.open(d) as one, Engine.open(d, batch=BATCH) as many:
            out["sozopel"] = _engine_numbers(one, many, lambda e: e.reset(), steps)
    n_w = sum(int(np.prod(s)) for n, (s, _, _) in synth.sozopel_tensors(cfg, 64).items() if n not in ("embed", "pos"))
    out["sozopel"]["weight_bytes"] = 2 * n_w
    m = synth.SyntheticModel(bitnet_config(width, ff), seed=0)
    with Engine(m.config_struct()).load_synthetic(m) as one, Engine(m.config_struct(), batch=BATCH).load_synthetic(m) as many:
        many.kv_fill_random(CHUNK, seed=0)
        out["bitnet"] = _engine_numbers(one, many, lambda e: e.reset(), steps)
    out["bitnet"]["weight_bytes"] = m.weight_bytes_per_token()
    hbm = _peaks()[0]
    for v in out.values():
        v["decode_b1_hbm_frac"] = v["weight_bytes"] / (v["decode_b1_ms"] * 1e-3) / hbm
    return out


def _time(calls, iters=20):
    """Microseconds per call: `calls` (distinct buffers) captured back to back in one graph."""
    import torch
    st = torch.cuda.Stream()
    with torch.cuda.stream(st):
        for c in calls:
            c()
        st.synchronize()
        graph = torch.cuda.CUDAGraph()
        with torch.cuda.graph(graph, stream=st):
            for c in calls:
                c()
        for _ in range(3):
            graph.replay()
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        st.synchronize()
        e0.record(st)
        for _ in range(iters):
            graph.replay()
        e1.record(st)
        st.synchronize()
    return e0.elapsed_time(e1) * 1e3 / iters / len(calls)


def _kernels(width, ff, only=None):
    import torch
    from . import kernels as K
    hbm, tc, _ = _peaks()
    g = torch.Generator(device="cuda").manual_seed(0)
    rnd = lambda *s, dt=torch.float32: torch.randn(*s, generator=g, device="cuda").to(dt)
    bf = torch.bfloat16
    rows = []

    def add(name, us, nbytes, flops=0, flop_peak=tc, like=None):
        floor = max(nbytes / hbm, flops / flop_peak if flops else 0) * 1e6
        rows.append({"kernel": name, "us": round(us, 2), "roofline_us": round(floor, 2), "frac": round(floor / us, 3),
                     "bound": "memory" if not flops or nbytes / hbm > flops / flop_peak else "math", **({"like": like} if like else {})})

    want = lambda n: only is None or n in only
    heads, kv = width // 128, max(1, width // 512)
    ws = K.gemm_workspace()
    gk = dict(workspace=ws, workspace_bytes=ws.numel())
    if want("gemm"):
        n_rot = 8
        w = [rnd(ff, width, dt=bf) for _ in range(n_rot)]
        w8 = [torch.randint(0, 81, (ff * width // 4,), generator=g, device="cuda") for _ in range(n_rot)]
        table = torch.from_numpy(synth._BYTE81).cuda()
        w8 = [table[i].contiguous() for i in w8]
        for M in (1, BATCH, CHUNK):
            x, c = rnd(M, width, dt=bf), torch.empty(M, ff, device="cuda")
            us = _time([lambda w=w_: K.gemm(a=x, w=w, M=M, N=ff, ld_k=width, seg_end=[ff] + [0] * 7, c=c, ld_c=ff, use_pdl=int(M < 100), **gk) for w_ in w])
            add(f"gemm {ff}x{width}, {M} rows", us, 2 * ff * width + M * (2 * width + 4 * ff), 2 * M * ff * width)
            xf = rnd(M, width)
            wsp = torch.empty(K.load_library().tenzo_cuda_tl1_gemv_workspace_bytes(max(M, 2), width), dtype=torch.uint8, device="cuda")
            us = _time([lambda w=w_: K.tl1_gemv(xf, w, ff // 64, width, [0.02], out=c, use_pdl=M < 100, workspace=wsp) for w_ in w8])
            add(f"BitNet tl1 {ff}x{width}, {M} rows", us, ff * width // 4 + M * (4 * width + 4 * ff), 2 * M * ff * width, 2 * tc, like=f"gemm {ff}x{width}, {M} rows")
        del w, w8
    if want("head"):
        w = [rnd(VOCAB, width, dt=bf) for _ in range(2)]
        x, c = rnd(1, width, dt=bf), torch.empty(1, VOCAB, device="cuda")
        add(f"head {VOCAB}x{width}, 1 row", _time([lambda w=w_: K.gemm(a=x, w=w, M=1, N=VOCAB, ld_k=width, seg_end=[VOCAB] + [0] * 7, c=c, ld_c=VOCAB, use_pdl=1, **gk) for w_ in w]),
            2 * VOCAB * width + 4 * VOCAB)
        w = [torch.randint(-127, 128, (VOCAB, width), generator=g, device="cuda", dtype=torch.int8) for _ in range(3)]
        sc, xf, arg = torch.rand(VOCAB, device="cuda") * 0.01, rnd(1, width), torch.zeros(1, dtype=torch.int32, device="cuda")
        add(f"BitNet head {VOCAB}x{width}, 1 row", _time([lambda w=w_: K.lm_head_i8_static(xf, w, sc, argmax=arg, use_pdl=True) for w_ in w]), VOCAB * width + 4 * VOCAB,
            like=f"head {VOCAB}x{width}, 1 row")
        del w
    if want("attention"):
        n_ch = (heads + 2 * kv) * 128
        cw = [torch.ones(4, n, device="cuda") * 0.25 for n in (heads * 128, kv * 128, kv * 128)]
        for B, win in ((1, WINDOW), (BATCH, WINDOW), (BATCH, 4096)):
            n_rot = max(1, int(2.6e8 / (B * kv * win * 512)) + 1) if B > 1 else 32
            x, out = rnd(B, n_ch), torch.empty(B, heads * 128, dtype=bf, device="cuda")
            rk, rv = [rnd(B, kv, win, 128, dt=bf) for _ in range(n_rot)], [rnd(B, kv, win, 128, dt=bf) for _ in range(n_rot)]
            tail = torch.zeros(B, 3 * n_ch, device="cuda")
            pos = torch.full((B,), win + 5, dtype=torch.int32, device="cuda")
            us = _time([lambda a=a, b=b: K.window_attention(q=x, k=x[:, heads * 128:], v=x[:, (heads + kv) * 128:], ld=n_ch, conv_q=cw[0], conv_k=cw[1], conv_v=cw[2], taps=4,
                        tail_in=tail, tail_out=tail, tail_seq_stride=3 * n_ch, heads=heads, kv_heads=kv, dim=128, vdim=128, scale=0.09, window=win, ring=win, ring_k=a, ring_v=b,
                        ring_k_stride=kv * win * 128, ring_v_stride=kv * win * 128, pos=pos, M=B, decode=1, out=out, ld_out=heads * 128, use_pdl=1) for a, b in zip(rk, rv)])
            add(f"window attention decode, {B} x {win} keys", us, B * kv * win * 512)
            del rk, rv
            i8 = lambda: torch.randint(-127, 128, (B, 1, kv, win, 128), generator=g, device="cuda", dtype=torch.int8)
            n_rot = 2 * n_rot if B > 1 else n_rot
            ck, cv = [i8() for _ in range(n_rot)], [i8() for _ in range(n_rot)]
            sk = torch.rand(B, 1, kv, win, device="cuda") * 0.03
            q, k1, v1 = rnd(B, heads * 128), rnd(B, kv * 128), rnd(B, kv * 128)
            p8 = torch.full((B,), win - 1, dtype=torch.int32, device="cuda")
            us = _time([lambda a=a, b=b: K.attention_int8(q, k1, v1, a, b, sk, sk, p8, layer=0, n_q=heads, n_kv=kv, max_seq=win, max_len=win) for a, b in zip(ck, cv)])
            add(f"BitNet attention decode, {B} x {win} keys", us, B * kv * win * 264, like=f"window attention decode, {B} x {win} keys")
            del ck, cv
        M = CHUNK
        x, out = rnd(M, n_ch), torch.empty(M, heads * 128, dtype=bf, device="cuda")
        rk, rv = rnd(kv, WINDOW, 128, dt=bf), rnd(kv, WINDOW, 128, dt=bf)
        lin = [torch.empty(M, heads, 128, dtype=bf, device="cuda")] + [torch.empty(kv, WINDOW + M, 128, dtype=bf, device="cuda") for _ in range(2)]
        tail, stage = torch.zeros(3 * n_ch, device="cuda"), torch.zeros(3 * n_ch, device="cuda")
        us = _time([lambda: K.window_attention(q=x, k=x[:, heads * 128:], v=x[:, (heads + kv) * 128:], ld=n_ch, conv_q=cw[0], conv_k=cw[1], conv_v=cw[2], taps=4, tail_in=tail,
                    tail_out=stage, heads=heads, kv_heads=kv, dim=128, vdim=128, scale=0.09, window=WINDOW, ring=WINDOW, ring_k=rk, ring_v=rv, pos0=4096, M=M, decode=0, out=out,
                    ld_out=heads * 128, lin_q=lin[0], lin_k=lin[1], lin_v=lin[2])])
        add(f"window attention chunk (prepare, ring, attention), {M} rows, window {WINDOW}", us, 4 * M * n_ch * 2, 4 * M * WINDOW * heads * 128)
        shared = lambda t: t.as_strided(t.shape, (0,) + t.stride()[1:])      # every query row reads the one sequence's cache
        ck, cv = (shared(torch.randint(-127, 128, (1, 1, kv, M, 128), generator=g, device="cuda", dtype=torch.int8)) for _ in range(2))
        sk = shared(torch.rand(1, 1, kv, M, device="cuda") * 0.03)
        q, k1 = rnd(M, heads * 128), rnd(M, kv * 128)
        p8 = torch.arange(M, dtype=torch.int32, device="cuda")
        us = _time([lambda: K.attention_int8(q, k1, k1, ck, cv, sk, sk, p8, layer=0, n_q=heads, n_kv=kv, max_seq=M, max_len=M, append=False, tiles=2)], iters=3)
        add(f"BitNet attention chunk, {M} rows (mean {M // 2} keys)", us, 4 * M * heads * 128 * 2, 4 * M * (M // 2) * heads * 128,
            like=f"window attention chunk (prepare, ring, attention), {M} rows, window {WINDOW}")
    if want("scan"):
        sh, dim, vd, rank = heads, 64, 128, 64
        n, nv = sh * dim, sh * vd
        for kind, name in ((0, "retention"), (1, "gated"), (2, "time mixing")):
            up, bias, dec = rnd(n, rank, dt=bf), rnd(n), torch.full((sh,), 0.98, device="cuda")
            fixed = dict(heads=sh, dim=dim, vdim=vd, decay_kind=kind, decay=dec, up=up, bias=bias, rank=rank, tau=16.0, bonus=bias if kind == 2 else None, eps=1e-5, ld_out=nv)
            for B in (1, BATCH):
                ld = 2 * n + 2 * nv + rank
                x, out = rnd(B, ld), torch.empty(B, nv, dtype=bf, device="cuda")
                n_rot = int(2.6e8 / (B * n * vd * 8)) + 1 if B > 1 else 64
                st = [torch.zeros(B, n * vd, device="cuda") for _ in range(n_rot)]
                us = _time([lambda s=s: K.linear_scan(q=x, k=x[:, n:], v=x[:, 2 * n:], g=x[:, 2 * n + nv:], low=x[:, 2 * n + 2 * nv:], ld=ld, state=s, state_seq_stride=n * vd, M=B,
                            decode=1, out=out, use_pdl=1, **fixed) for s in st])
                add(f"scan decode ({name}), {B} sequences", us, 2 * B * n * vd * 4 + B * ld * 4)
                del st
            M = CHUNK
            x, out, st = rnd(M, ld), torch.empty(M, nv, dtype=bf, device="cuda"), torch.zeros(n * vd, device="cuda")
            wr, orow, part = torch.empty(M, n, device="cuda"), torch.empty(M, nv, device="cuda"), K.linear_scan_part(M, sh, dim, vd)
            us = _time([lambda: K.linear_scan(q=x, k=x[:, n:], v=x[:, 2 * n:], g=x[:, 2 * n + nv:], low=x[:, 2 * n + 2 * nv:], ld=ld, state=st, M=M, decode=0, out=out, w_rows=wr,
                        o_rows=orow, part=part, **fixed)])
            add(f"scan chunk ({name}), {M} rows", us, M * (ld + nv) * 4, M * n * vd * 6, FP32_TFLOPS * 1e12)
    if want("rows"):
        for M, dec in ((1, 1), (BATCH, 1), (CHUNK, 0)):
            n_rot = 8 if M == CHUNK else 1
            xs = [rnd(M, width) for _ in range(n_rot)]
            y, xo, out = rnd(M, width), torch.empty(M, width, device="cuda"), torch.empty(M, width, dtype=bf, device="cuda")
            inv = torch.empty(M, device="cuda")
            cw, tail = rnd(4, width), torch.zeros(M if dec else 2, 3 * width, device="cuda")
            us = _time([lambda x=x_: K.rows(x_in=x, y0=y, ld_y=width, x_out=xo, width=width, M=M, eps=1e-5, conv_w=cw, taps=4, tail_in=tail, tail_out=tail if dec else tail[1],
                        seq_stride=3 * width, decode=dec, row_inv=inv, out=out, ld_out=width, use_pdl=dec) for x_ in xs])
            add(f"rows (residual, norm, convolution), {M} rows", us, M * width * 14)
            us = _time([lambda x=x_: K.rmsnorm_quant(x, want_y=False) for x_ in xs])
            add(f"BitNet norm + quantiser, {M} rows", us, M * width * 5, like=f"rows (residual, norm, convolution), {M} rows")
    return rows


def run(args):
    import torch
    torch.cuda.set_device(0)
    _, _, src = _peaks()
    steps = min(args.steps, 64)
    import bench
    sampler = bench.ClockSampler(0).start()
    sampler.mark()
    sizes = {f"width {w}, ff {f}": _models(w, f, steps) for w, f in SIZES.items()}
    width = max(SIZES)
    kernels = _kernels(width, SIZES[width])
    clocks = sampler.stop()
    big = sizes[f"width {width}, ff {SIZES[width]}"]["sozopel"]
    print(json.dumps({
        "metric": "sozopel_decode_tokens_per_second_batch1", "value": big["decode_b1_tok_s"], "unit": "tok/s", "n_gpus": 1, "steps": steps, "warmup": 8,
        "ms_per_step": big["decode_b1_ms"], "higher_is_better": True, "scaling": "weak", "vs_baseline": None, "dtype": "bf16", "data": "synthetic",
        "config": {"workload": f"sozopel: {LAYERS} layers (attention beside gated linear attention, time mixing, retention, each with a feed-forward), vocabulary {VOCAB}, "
                               f"window {WINDOW}; prompt {CHUNK} tokens; random weights", "l2": "weights of a step larger than L2; kernels rotate over more than L2"},
        "sizes": sizes, "kernels": kernels, "peak_source": src, "clocks": clocks}), flush=True)
