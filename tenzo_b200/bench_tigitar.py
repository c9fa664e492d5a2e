"""`bench.py --workload tigitar`: the Tigitar decoder beside Sozopel, the library's nearest other design, at equal size.

Models of 8 layers with random weights at three widths (vocabulary 32768, the same feed-forward width: the experts a token
takes add up to it): prompt throughput (one 2048-token chunk), decode throughput of one sequence and of 64. Then every
kernel of the design alone, at the largest width, against its roofline, and the like kernel of Sozopel against its own:
inputs rotate over more than the L2 cache, one CUDA graph per measurement, CUDA events around its replays.
"""
from __future__ import annotations

import json
import tempfile

import numpy as np

from . import synth
from .bench_hybrid import BATCH, CHUNK, FP32_TFLOPS, LAYERS, SIZES, VOCAB, WINDOW, _engine_numbers, _peaks, _time, sozopel_config

EXPERTS, TOP, RANK, ROT = 16, 4, 512, 64


def tigitar_config(width: int, ff: int) -> dict:
    heads = width // 128
    kv = next(k for k in range(max(1, heads // 2), heads + 1) if heads % k == 0)
    mix_d = {"heads": heads, "kv_heads": kv, "dim": 128, "vdim": 128, "conv": 4}
    mix_l = {"heads": heads, "dim": 128, "rot_dim": ROT, "vdim": 128, "kv_rank": RANK, "mask": {"size": WINDOW}, "rot": {"base": 10000.0, "dims": ROT},
             "scale": (128 + ROT) ** -0.5}
    dense, moe = {"kind": "dense", "ff": ff}, {"kind": "moe", "expert": {"ff": ff // TOP}, "router": {"experts": EXPERTS, "top": TOP}}
    d = lambda mlp: {"type": "delta", "mixer": mix_d, "mlp": mlp}
    a = lambda mlp, **kw: {"type": "latent_attention", "mixer": dict(mix_l, **kw), "mlp": mlp}
    return {"vocab": VOCAB, "width": width, "norm": {"eps": 1e-5}, "logit_softcap": 30.0,
            "layers": [d(dense), a(moe), d(dense), d(moe), a(dense, kv_from=1), d(dense), d(moe), a(dense)]}


def _weights_read(cfg: dict, spec: dict) -> int:
    """Bytes of weights that one token reads: everything but the embedding, and of the experts those it takes."""
    total = 0
    for name, (shape, _, _) in spec.items():
        n = 2 * int(np.prod(shape))
        if name == "embed":
            continue
        if ".mlp.e" in name:
            r = cfg["layers"][int(name[1:name.index(".")])]["mlp"]["router"]
            n = n * r["top"] // r["experts"]
        total += n
    return total


def _models(width, ff, steps):
    from .engine import Engine
    out = {}
    cfg, soz = tigitar_config(width, ff), sozopel_config(width, ff)
    for name, write, read in (("tigitar", lambda d: synth.write_tigitar_pooled(d, cfg, seed=0), _weights_read(cfg, synth.tigitar_tensors(cfg))),
                              ("sozopel", lambda d: synth.write_sozopel_pooled(d, soz, rank=64, seed=0),
                               sum(2 * int(np.prod(s)) for n, (s, _, _) in synth.sozopel_tensors(soz, 64).items() if n not in ("embed", "pos")))):
        with tempfile.TemporaryDirectory() as d:
            write(d)
            with Engine.open(d) as one:
                res = _engine_numbers(one, one, lambda e: e.reset(), steps)
            with Engine.open(d, batch=BATCH) as many:
                first = synth.prompt_tokens(2, BATCH, VOCAB)
                many.decode_greedy(first, WINDOW)              # every window is full
                runs = []
                for _ in range(5):
                    many.decode_greedy(first, steps)
                    runs.append(many.last_device_ms() / steps)
                ms = float(np.median(runs))
        res = {k: v for k, v in res.items() if "decode_b64" not in k}
        out[name] = {**res, f"decode_b{BATCH}_tok_s": BATCH * 1e3 / ms, f"decode_b{BATCH}_ms": ms, "weight_bytes": read,
                     "decode_b1_hbm_frac": read / (res["decode_b1_ms"] * 1e-3) / _peaks()[0]}
    return out


def _kernels(width, ff, only=None):
    import torch
    from . import kernels as K
    hbm, tc, _ = _peaks()
    g = torch.Generator(device="cuda").manual_seed(0)
    rnd = lambda *s, dt=torch.float32: torch.randn(*s, generator=g, device="cuda").to(dt)
    bf = torch.bfloat16
    zeros = lambda *s, dt=bf: torch.zeros(s, dtype=dt, device="cuda")
    rows, heads = [], width // 128
    cfg = tigitar_config(width, ff)

    def add(name, us, nbytes, flops=0, flop_peak=tc, like=None):
        floor = max(nbytes / hbm, flops / flop_peak if flops else 0) * 1e6
        rows.append({"kernel": name, "us": round(us, 2), "roofline_us": round(floor, 2), "frac": round(floor / us, 4),
                     "bound": "memory" if not flops or nbytes / hbm > flops / flop_peak else "math", **({"like": like} if like else {})})

    want = lambda n: only is None or n in only
    ws = K.gemm_workspace()
    gk = dict(workspace=ws, workspace_bytes=ws.numel())
    fe = ff // TOP
    if want("ff"):
        n_rot = 4
        up, down = [rnd(2 * ff, width, dt=bf) for _ in range(n_rot)], [rnd(width, ff, dt=bf) for _ in range(n_rot)]
        for M in (1, BATCH, CHUNK):
            x, act, y, wide = rnd(M, width, dt=bf), zeros(M, ff), zeros(M, width, dt=torch.float32), zeros(M, 2 * ff, dt=torch.float32)
            pdl = int(M < 100)
            plain = lambda a, w, c, n, k, **kw: K.gemm(a=a, w=w, M=M, N=n, ld_k=k, seg_end=[n] + [0] * 7, c=c, use_pdl=pdl, **{**gk, **kw})
            us = _time([lambda w=w: plain(x, w, act, 2 * ff, width, epilogue=2, ld_c=ff) for w in up])
            add(f"gated product 2x{ff}x{width}, {M} rows", us, 4 * ff * width + M * (2 * width + 2 * ff), 4 * M * ff * width)
            us = _time([lambda w=w: plain(x, w, wide, 2 * ff, width, ld_c=2 * ff) for w in up])
            add(f"Sozopel product 2x{ff}x{width}, {M} rows", us, 4 * ff * width + M * (2 * width + 8 * ff), 4 * M * ff * width, like=f"gated product 2x{ff}x{width}, {M} rows")

            def both(w1, w2):
                plain(x, w1, act, 2 * ff, width, epilogue=2, ld_c=ff)
                plain(act, w2, y, width, ff, ld_c=width)
            us = _time([lambda a=a, b=b: both(a, b) for a, b in zip(up, down)])
            add(f"dense feed-forward, {M} rows", us, 6 * ff * width + M * (6 * width + 4 * ff), 6 * M * ff * width)
        del up, down
        n_rot = 2
        up, down = [rnd(EXPERTS, 2 * fe, width, dt=bf) for _ in range(n_rot)], [rnd(EXPERTS, width, fe, dt=bf) for _ in range(n_rot)]
        for M in (1, BATCH, CHUNK):
            P, pdl = M * TOP, int(M < 100)
            x, act, ye, z = rnd(M, width, dt=bf), zeros(P, fe), zeros(P, width, dt=torch.float32), rnd(M, EXPERTS)
            i32 = lambda *s: zeros(*s, dt=torch.int32)
            # one token after another for the few-row case: other experts every time
            zs = [rnd(M, EXPERTS) for _ in range(8 if M == 1 else 1)]
            r = dict(chosen=i32(M, TOP), weight=zeros(M, TOP, dt=torch.float32), slot=i32(M, TOP), row_of=i32(P), group_off=i32(EXPERTS + 1))
            gather, corr = zeros(P, width), zeros(EXPERTS, dt=torch.float32)
            gg = dict(M=P, group_off=r["group_off"], n_group=EXPERTS, use_pdl=pdl, **gk)

            def routed(w1, w2, z):
                K.route(logits=z, ld=EXPERTS, correction=corr, experts=EXPERTS, top=TOP, M=M, use_pdl=pdl, **r)
                K.gemm(a=x, w=w1, N=2 * fe, ld_k=width, epilogue=3, c=act, ld_c=fe, a_index=r["row_of"], a_rows=M, a_gather=gather, **gg)
                K.gemm(a=act, w=w2, N=width, ld_k=fe, c=ye, ld_c=width, **gg)
            calls = [lambda a=a, b=b, z=z: routed(a, b, z) for z in zs for a, b in zip(up, down)]
            us = _time(calls)
            used = len({int(e) for z_ in zs[:1] for e in z_.topk(TOP, dim=1).indices.flatten().tolist()})
            add(f"routed feed-forward ({TOP} of {EXPERTS} experts), {M} rows", us, used * 6 * fe * width + P * (6 * width + 4 * fe), 6 * P * fe * width,
                like=f"dense feed-forward, {M} rows")
            us = _time([lambda: K.route(logits=z, ld=EXPERTS, correction=corr, experts=EXPERTS, top=TOP, M=M, use_pdl=pdl, **r)] * 4)
            add(f"route alone, {M} rows", us, M * EXPERTS * 4 + P * 20)
        del up, down
    if want("attention"):
        m = cfg["layers"][1]["mixer"]
        d8, r8, v8, rank = 128, ROT, 128, RANK
        nw = 8
        w = [rnd(heads * (d8 + v8), rank, dt=bf) * 0.05 for _ in range(nw)]
        ld = heads * (d8 + r8) + rank + r8
        freq = torch.from_numpy(m["rot"]["base"] ** (-2.0 * np.arange(ROT // 2) / ROT)).cuda()
        norm = torch.ones(rank, device="cuda")
        fixed = dict(ld=ld, norm=norm, eps=1e-5, freq=freq, heads=heads, dim=d8, rot=r8, vdim=v8, rank=rank, scale=m["scale"], **gk)
        kv = max(1, heads // 4)
        n_ch = (heads + 2 * kv) * 128
        cw = [torch.ones(4, n, device="cuda") * 0.25 for n in (heads * 128, kv * 128, kv * 128)]
        for B, win in ((1, WINDOW), (BATCH, WINDOW), (BATCH, 4096)):
            n_rot = max(1, int(2.6e8 / (B * win * (rank + r8) * 2)) + 1) if B > 1 else 32
            rc, rr = [rnd(B, win, rank, dt=bf) for _ in range(n_rot)], [rnd(B, win, r8, dt=bf) for _ in range(n_rot)]
            x, out, qa, lat = rnd(B, ld), zeros(B, heads * v8), zeros(B, heads, rank, dt=torch.float32), zeros(heads, B, rank)
            pos = torch.full((B,), win + 5, dtype=torch.int32, device="cuda")
            us = _time([lambda i=i: K.latent_attention(q=x, dkv=x[:, heads * (d8 + r8):], window=win, w_kv=w[i % nw], ring_c=rc[i % n_rot], ring_r=rr[i % n_rot], ring=win,
                        ring_c_stride=win * rank, ring_r_stride=win * r8, pos=pos, M=B, decode=1, out=out, ld_out=heads * v8, q_abs=qa, lat=lat, use_pdl=1, **fixed)
                        for i in range(max(n_rot, nw))])
            add(f"latent attention decode (absorb, attend, values), {B} x {win} keys", us, B * win * (rank + r8) * 2 + heads * (d8 + v8) * rank * 2)
            del rc, rr
            n_rot = max(1, int(2.6e8 / (B * kv * win * 512)) + 1) if B > 1 else 32
            xs, o2 = rnd(B, n_ch), zeros(B, heads * 128)
            rk, rv = [rnd(B, kv, win, 128, dt=bf) for _ in range(n_rot)], [rnd(B, kv, win, 128, dt=bf) for _ in range(n_rot)]
            tail = torch.zeros(B, 3 * n_ch, device="cuda")
            us = _time([lambda a=a, b=b: K.window_attention(q=xs, k=xs[:, heads * 128:], v=xs[:, (heads + kv) * 128:], ld=n_ch, conv_q=cw[0], conv_k=cw[1], conv_v=cw[2], taps=4,
                        tail_in=tail, tail_out=tail, tail_seq_stride=3 * n_ch, heads=heads, kv_heads=kv, dim=128, vdim=128, scale=0.09, window=win, ring=win, ring_k=a, ring_v=b,
                        ring_k_stride=kv * win * 128, ring_v_stride=kv * win * 128, pos=pos, M=B, decode=1, out=o2, ld_out=heads * 128, use_pdl=1) for a, b in zip(rk, rv)])
            add(f"Sozopel window attention decode, {B} x {win} keys", us, B * kv * win * 512, like=f"latent attention decode (absorb, attend, values), {B} x {win} keys")
            del rk, rv
        M, pos0 = CHUNK, 4096
        x, out = rnd(M, ld), zeros(M, heads * v8)
        rc, rr = rnd(WINDOW, rank, dt=bf), rnd(WINDOW, r8, dt=bf)
        lin = dict(lin_q=zeros(M, heads, d8 + r8), lin_c=zeros(M + WINDOW, rank), lin_r=zeros(M + WINDOW, r8), kv=zeros(M + WINDOW, heads * (d8 + v8)))
        us = _time([lambda w_=w_: K.latent_attention(q=x, dkv=x[:, heads * (d8 + r8):], window=WINDOW, w_kv=w_, ring_c=rc, ring_r=rr, ring=WINDOW, pos0=pos0, M=M, decode=0,
                    out=out, ld_out=heads * v8, **lin, **fixed) for w_ in w[:2]])
        T = M + WINDOW - 1
        add(f"latent attention chunk (rows, ring, expansion, attention), {M} rows, window {WINDOW}", us, 4 * M * ld + 2 * M * heads * v8,
            2 * T * rank * heads * (d8 + v8) + 2 * M * WINDOW * heads * (d8 + r8 + v8))
        xs, o2 = rnd(M, n_ch), zeros(M, heads * 128)
        rk, rv = rnd(kv, WINDOW, 128, dt=bf), rnd(kv, WINDOW, 128, dt=bf)
        l3 = [zeros(M, heads, 128)] + [zeros(kv, WINDOW + M, 128) for _ in range(2)]
        tail, stage = torch.zeros(3 * n_ch, device="cuda"), torch.zeros(3 * n_ch, device="cuda")
        us = _time([lambda: K.window_attention(q=xs, k=xs[:, heads * 128:], v=xs[:, (heads + kv) * 128:], ld=n_ch, conv_q=cw[0], conv_k=cw[1], conv_v=cw[2], taps=4, tail_in=tail,
                    tail_out=stage, heads=heads, kv_heads=kv, dim=128, vdim=128, scale=0.09, window=WINDOW, ring=WINDOW, ring_k=rk, ring_v=rv, pos0=pos0, M=M, decode=0, out=o2,
                    ld_out=heads * 128, lin_q=l3[0], lin_k=l3[1], lin_v=l3[2])])
        add(f"Sozopel window attention chunk, {M} rows, window {WINDOW}", us, 4 * M * n_ch * 2, 4 * M * WINDOW * heads * 128,
            like=f"latent attention chunk (rows, ring, expansion, attention), {M} rows, window {WINDOW}")
    if want("delta"):
        for dim in (128, 64):
            vd, kvh = 128, cfg["layers"][0]["mixer"]["kv_heads"]
            nk, nv = kvh * dim, heads * vd
            off = np.cumsum([0, nk, nk, nv, nv, heads, heads])
            ld, n_ch = int((off[-1] + 3) // 4 * 4), 2 * nk + nv
            cw = [torch.ones(4, n, device="cuda") * 0.25 for n in (nk, nk, nv)]
            hv = dict(a_log=torch.full((heads,), -2.0, device="cuda"), dt_bias=torch.zeros(heads, device="cuda"), norm=torch.ones(vd, device="cuda"))
            split = lambda x: dict(q=x, k=x[:, off[1]:], v=x[:, off[2]:], g=x[:, off[3]:], a=x[:, off[4]:], b=x[:, off[5]:])
            fixed = dict(ld=ld, conv_q=cw[0], conv_k=cw[1], conv_v=cw[2], taps=4, heads=heads, kv_heads=kvh, dim=dim, vdim=vd, q_scale=dim ** -0.5, eps=1e-5, ld_out=nv, **hv)
            sn, rk = heads * dim, 64
            up, bias = rnd(sn, rk, dt=bf), rnd(sn)
            soz = dict(heads=heads, dim=dim, vdim=vd, decay_kind=1, up=up, bias=bias, rank=rk, tau=16.0, eps=1e-5, ld_out=nv)
            sl = 2 * sn + 2 * nv + rk
            cut = lambda x: dict(q=x, k=x[:, sn:], v=x[:, 2 * sn:], g=x[:, 2 * sn + nv:], low=x[:, 2 * sn + 2 * nv:], ld=sl)
            for B in (1, BATCH):
                x, out = rnd(B, ld), zeros(B, nv)
                n_rot = int(2.6e8 / (B * sn * vd * 8)) + 1 if B > 1 else 32
                st, tail = [torch.zeros(B, sn * vd, device="cuda") for _ in range(n_rot)], torch.zeros(B, 4 * n_ch, device="cuda")
                pos = torch.full((B,), 100, dtype=torch.int32, device="cuda")
                us = _time([lambda s=s: K.delta_rule(**split(x), tail=tail, tail_seq_stride=4 * n_ch, state=s, state_seq_stride=sn * vd, pos=pos, M=B, decode=1, out=out, use_pdl=1,
                            **fixed) for s in st])
                add(f"delta decode, {B} sequences, dim {dim}", us, 2 * B * sn * vd * 4 + B * ld * 4)
                xs = rnd(B, sl)
                us = _time([lambda s=s: K.linear_scan(**cut(xs), state=s, state_seq_stride=sn * vd, M=B, decode=1, out=out, use_pdl=1, **soz) for s in st])
                add(f"Sozopel scan decode (gated), {B} sequences, dim {dim}", us, 2 * B * sn * vd * 4 + B * sl * 4, like=f"delta decode, {B} sequences, dim {dim}")
                del st
            M = CHUNK
            x, out, st, tail = rnd(M, ld), zeros(M, nv), torch.zeros(sn * vd, device="cuda"), torch.zeros(4 * n_ch, device="cuda")
            work = K.delta_rule_work(M, heads, kvh, dim, vd)
            us = _time([lambda: K.delta_rule(**split(x), tail=tail, state=st, M=M, decode=0, out=out, work=work, **fixed)])
            add(f"delta chunk, {M} rows, dim {dim}", us, M * (ld + nv) * 4, M * sn * vd * 8, FP32_TFLOPS * 1e12)
            xs, wr, orow, part = rnd(M, sl), torch.empty(M, sn, device="cuda"), torch.empty(M, nv, device="cuda"), K.linear_scan_part(M, heads, dim, vd)
            us = _time([lambda: K.linear_scan(**cut(xs), state=st, M=M, decode=0, out=out, w_rows=wr, o_rows=orow, part=part, **soz)])
            add(f"Sozopel scan chunk (gated), {M} rows, dim {dim}", us, M * (sl + nv) * 4, M * sn * vd * 6, FP32_TFLOPS * 1e12, like=f"delta chunk, {M} rows, dim {dim}")
    if want("rows"):
        for M, dec in ((1, 1), (BATCH, 1), (CHUNK, 0)):
            n_rot = 8 if M == CHUNK else 1
            xs = [rnd(M, width) for _ in range(n_rot)]
            y, xo, out, inv = rnd(M, width), torch.empty(M, width, device="cuda"), zeros(M, width), torch.empty(M, device="cuda")
            w0, gw, cw, tail = rnd(width), rnd(width), rnd(4, width), torch.zeros(M if dec else 2, 3 * width, device="cuda")
            us = _time([lambda x=x: K.rows(x_in=x, y0=y, ld_y=width, w0=w0, x_out=xo, width=width, M=M, eps=1e-5, gain_w=gw, decode=dec, row_inv=inv, out=out, ld_out=width,
                        use_pdl=dec) for x in xs])
            add(f"rows (normed addend, residual, norm), {M} rows", us, M * width * 14)
            us = _time([lambda x=x: K.rows(x_in=x, y0=y, ld_y=width, x_out=xo, width=width, M=M, eps=1e-5, conv_w=cw, taps=4, tail_in=tail, tail_out=tail if dec else tail[1],
                        seq_stride=3 * width, decode=dec, row_inv=inv, out=out, ld_out=width, use_pdl=dec) for x in xs])
            add(f"Sozopel rows (residual, norm, convolution), {M} rows", us, M * width * 14, like=f"rows (normed addend, residual, norm), {M} rows")
            ye = rnd(M * TOP, width)
            slot, wt = torch.randperm(M * TOP, device="cuda").to(torch.int32), torch.rand(M * TOP, device="cuda")
            us = _time([lambda x=x: K.rows(x_in=x, y0=ye, ld_y=width, w0=w0, y_slot=slot, y_weight=wt, n_y=TOP, x_out=xo, width=width, M=M, eps=1e-5, gain_w=gw, decode=dec, row_inv=inv,
                        out=out, ld_out=width, use_pdl=dec) for x in xs])
            add(f"rows (sum of {TOP} experts, residual, norm), {M} rows", us, M * width * (10 + 4 * TOP), like=None)
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
    big = sizes[f"width {width}, ff {SIZES[width]}"]["tigitar"]
    print(json.dumps({
        "metric": "tigitar_decode_tokens_per_second_batch1", "value": big["decode_b1_tok_s"], "unit": "tok/s", "n_gpus": 1, "steps": steps, "warmup": 8,
        "ms_per_step": big["decode_b1_ms"], "higher_is_better": True, "scaling": "weak", "vs_baseline": None, "dtype": "bf16", "data": "synthetic",
        "config": {"workload": f"tigitar: {LAYERS} layers (5 delta rule, 3 latent attention of which one borrows its cache; 3 with {TOP} of {EXPERTS} experts), vocabulary {VOCAB}, "
                               f"window {WINDOW}; prompt {CHUNK} tokens; random weights", "l2": "weights of a step larger than L2; kernels rotate over more than L2"},
        "sizes": sizes, "kernels": kernels, "peak_source": src, "clocks": clocks}), flush=True)
