"""Vokepel layers (attention with learned sinks beside a gated recurrence, talking heads over keys that are values, squared ReLU)
next to the closest existing model: prompt and decode throughput through the engine beside the Kipolix-shaped model (windowed
attention and retention, SwiGLU, one residual stream) of equal width, heads, windows and feed-forward parameters, and every kernel
of the design against its roofline next to the like kernel.

    python bench.py --vokepel [--steps K --warmup W]

A size is a few layers of a real model's shape with random weights. Timing and rooflines as in bench_hybrid: CUDA events,
buffers that together exceed L2, measured copy bandwidth and bf16 rate. Arithmetic is what the equations need: the second term of
the softmax weights does not count, and the mixing of the heads' scores counts at the rate of the tensor cores.
"""
from __future__ import annotations

import json
from dataclasses import replace

import torch

from .bench_hybrid import Timer, _copies, engine_numbers
from .utils.roofline import load_measured_peaks

SIZES = {
    # the layers of llama3-8b; half its width; many heads of 64
    "w4096-h32": dict(width=4096, ff=21504, heads=32, kv_heads=8, dim=128, window=4096, t_heads=32, t_kv=8, t_dim=128, t_window=1024, gru=4096),
    "w2048-h16": dict(width=2048, ff=12288, heads=16, kv_heads=4, dim=128, window=2048, t_heads=16, t_kv=4, t_dim=128, t_window=512, gru=2048),
    "w2048-h32": dict(width=2048, ff=12288, heads=32, kv_heads=8, dim=64, window=2048, t_heads=32, t_kv=8, t_dim=64, t_window=1024, gru=2048),
}
VOCAB = 32000
LAYERS = 8


def _configs(name: str):
    from .models.config import _kipolix_preset, _vokepel_preset

    z = SIZES[name]
    vok = _vokepel_preset("vokepel-" + name, vocab=VOCAB, pattern="pt" * (LAYERS // 2), **z)
    kip = _kipolix_preset("kipolix-" + name, vocab=VOCAB, pattern="ar" * (LAYERS // 2), width=z["width"], ff=z["ff"] * 2 // 3, heads=z["heads"],
                          kv_heads=z["kv_heads"], dim=z["dim"], window=z["window"], keep_first=0, r_heads=z["heads"], r_dim=z["dim"],
                          r_vdim=z["dim"], streams=0)
    return vok, kip


def kernel_numbers(vok, kip, peaks: dict, timer: Timer, batch: int, ctx: int, m: int, only: str = "") -> list:
    """One row per kernel: name, microseconds, roofline microseconds, fraction of the roofline. `only`: names that contain it."""
    from . import ops
    from .models.hybrid import talk_head, talk_pass, tc_head
    from .ops import hybrid as hops

    dev = torch.device("cuda", 0)
    bf = dict(dtype=torch.bfloat16, device=dev)
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=dev)
    bw, fl = peaks["hbm_gbs"] * 1e3, peaks["bf16_tflops"] * 1e6        # bytes / us, flops / us
    rows = []

    def add(name, calls_of, nbytes, flops=0.0):
        if only not in name:
            return
        n = _copies(nbytes)
        us = timer([calls_of(i) for i in range(n)])
        roof = max(nbytes / bw, flops / fl)
        rows.append({"kernel": name, "us": round(us, 2), "roofline_us": round(roof, 2), "fraction": round(roof / us, 3)})
        torch.cuda.empty_cache()

    part = lambda mc, k: next(p for L in mc.layers for p in L.mixer.parts if p.kind == k)
    att, talk, gru = part(vok, "attention"), part(vok, "talking_attention"), part(vok, "min_gru")
    katt, ret = part(kip, "attention"), part(kip, "retention")
    d, rot, none = vok.d_model, hops.Rotary(att.rot, dev), hops.Rotary(None, dev)
    H, G, D, P = talk.heads, talk.kv_heads, talk.dim, talk_head(talk)
    mats = dict(talk=torch.eye(H, device=dev), bias=torch.zeros(H, talk.window, device=dev))
    for M in (batch, m):
        tag = f"[{M} rows]"
        ones, zeros, one = torch.ones(d, device=dev), torch.zeros(d, device=dev), torch.ones(1, device=dev)
        pages = M // 16 + 1
        pos, slots = torch.arange(M, dtype=torch.int32, device=dev), torch.arange(M, device=dev)

        def bn(i, M=M):
            x, y, h = torch.randn(M, d, device=dev), torch.randn(M, d, device=dev), torch.empty(M, d, **bf)
            return lambda: hops.branch_norm(x, M, norm_w=[ones], h=[h], eps=1e-5, branches=[(y, None, 0.5, False)])
        add("branch_norm " + tag, bn, M * d * (8 + 4 + 2))

        def sp(i, M=M):
            x, y, h = torch.randn(M, d, device=dev), torch.randn(M, d, device=dev), torch.empty(M, 3 * d, **bf)
            emb, tok = torch.randn(1000, d, **bf), torch.randint(0, 1000, (M,), dtype=torch.int32, device=dev)
            return lambda: hops.branch_norm(x, M, norm_w=(), h=(), eps=1e-5, branches=[(y, None, 0.5, False)], split=h, split_off=d, x0_tokens=tok,
                                            embed=emb)
        add("branch_norm, operand of a pass's entry " + tag, sp, M * d * (8 + 4 + 6 + 2))

        def sn(i, M=M):
            x, y, h = torch.randn(M, 1, d, device=dev), torch.randn(M, d, device=dev), torch.empty(M, d, **bf)
            return lambda: hops.stream_norm(x, M, norm_w=zeros, eps=1e-5, h=h, y=y, mix=one, out_w=one, in_w=one)
        add("stream_norm (Kipolix) " + tag, sn, M * d * (8 + 8 + 2))

        def heads(a, q_norm, tied, i, M=M):
            dp = P if tied else tc_head(a)
            W = (a.heads + a.kv_heads) * a.dim + (0 if tied else a.kv_heads * a.vdim)
            proj, q, kc = torch.randn(M, W, **bf), torch.zeros(M, a.heads * dp, **bf), torch.zeros(pages, a.kv_heads, 16, dp, **bf)
            kw = dict(k_rms=torch.zeros(pages, 16, device=dev)) if tied else dict(v_cache=torch.zeros_like(kc))
            if q_norm:
                kw["q_norm"] = torch.ones(a.heads * a.dim, device=dev)
                if not tied:
                    kw["k_norm"] = torch.ones(a.kv_heads * a.dim, device=dev)
            return lambda: hops.heads(proj, M, h=a.heads, g=a.kv_heads, d=a.dim, e=a.dim, rot=none if tied else hops_rot(a), positions=pos, q_out=q,
                                      q_hd=dp, k_cache=kc, slots=slots, **kw)
        rots = {}

        def hops_rot(a):
            if a.rot not in rots:
                rots[a.rot] = hops.Rotary(a.rot, dev)
            return rots[a.rot]
        wid = lambda a, v: (a.heads + a.kv_heads) * a.dim + v * a.kv_heads * a.dim
        add("heads, rotation " + tag, lambda i: heads(att, False, False, i), 4 * M * wid(att, 1))
        add("heads, norms, keys that are values " + tag, lambda i: heads(talk, True, True, i), 4 * M * wid(talk, 0))
        add("heads, norms and rotation (Kipolix) " + tag, lambda i: heads(katt, True, False, i), 4 * M * wid(katt, 1))

    # decode attention
    nb_seq, splits = ctx // 16, 16
    lens = i32([ctx] * batch)

    def plan(hk):
        per_sm = 12 if hk >= 4 else 4
        want = max(1, min(splits, -(-per_sm * 148 // (batch * hk))))
        return i32([(max(4, -(-nb_seq // want)) + 3) // 4 * 4])

    def dec(a, i, sinks):
        dp = tc_head(a)
        kc, vc = torch.zeros(batch * nb_seq, a.kv_heads, 16, dp, **bf), torch.zeros(batch * nb_seq, a.kv_heads, 16, dp, **bf)
        bt = torch.randperm(batch * nb_seq, device=dev).to(torch.int32).view(batch, nb_seq)
        q, out = torch.randn(batch, a.heads, dp, **bf), torch.empty(batch, a.heads * a.vdim, **bf)
        po, pm = torch.empty(batch * a.heads * splits * dp, device=dev), torch.empty(batch * a.heads * splits * 2, device=dev)
        kw = dict(sinks=torch.zeros(a.heads, device=dev), out_gain=0.5) if sinks else {}
        pps = plan(att.kv_heads)
        return lambda: ops.paged_decode(q, kc, vc, bt, lens, pps, po, pm, out, batch=batch, max_splits=splits, window=a.window, scale=0.1,
                                        out_d=a.vdim, exact_p=True, **kw)

    def tdec(i):
        c, r = torch.zeros(batch * nb_seq, G, 16, P, **bf), torch.zeros(batch * nb_seq, 16, device=dev)
        bt = torch.randperm(batch * nb_seq, device=dev).to(torch.int32).view(batch, nb_seq)
        q, out, gate = torch.randn(batch, H * P, **bf), torch.empty(batch, H * D, **bf), torch.randn(batch, H * D, **bf)
        po, pm = torch.empty(batch * H * splits * P, device=dev), torch.empty(batch * H * splits * 2, device=dev)
        return lambda: hops.talk_decode(q, c, r, bt, lens, rows=batch, h=H, d=D, window=talk.window, scale=0.1, cap=30.0, gate=gate, out=out,
                                        part_o=po, part_ml=pm, max_splits=splits, **mats)
    vis = lambda w: min(ctx, w + 16) if w else ctx
    add(f"paged_decode, window and sinks [{batch} x {vis(att.window)} keys]", lambda i: dec(att, i, True),
        batch * vis(att.window) * att.kv_heads * att.dim * 4)
    add(f"talk_decode [{batch} x {vis(talk.window)} keys]", tdec, batch * vis(talk.window) * (G * D * 2 + 4) + batch * 8 * H * D)
    add(f"paged_decode, window (Kipolix) [{batch} x {vis(katt.window)} keys]", lambda i: dec(katt, i, False),
        batch * vis(katt.window) * katt.kv_heads * katt.dim * 4)
    short = replace(katt, window=talk.window, heads=H, kv_heads=G, dim=D, vdim=D)
    add(f"paged_decode, the talking heads' window and sizes (Kipolix) [{batch} x {vis(talk.window)} keys]", lambda i: dec(short, i, False),
        batch * vis(talk.window) * G * D * 4)

    # prompt attention: m tokens in sequences of L
    L = 2048
    ns = m // L
    tiles = [(s, t * 128) for s in range(ns) for t in range(L // 128)]
    ts, tq = i32([t[0] for t in tiles]), i32([t[1] for t in tiles])
    qs, ql = i32([s * L for s in range(ns)]), i32([L] * ns)
    bt = torch.arange(m // 16, dtype=torch.int32, device=dev).view(ns, L // 16)
    pairs = lambda w: sum(min(i + 1, w) for i in range(L)) * ns

    def pre(a, i, sinks):
        dp = tc_head(a)
        kc, vc = torch.randn(m // 16, a.kv_heads, 16, dp, **bf), torch.randn(m // 16, a.kv_heads, 16, dp, **bf)
        q, out = torch.randn(m, a.heads, dp, **bf), torch.empty(m, a.heads * a.vdim, **bf)
        kw = dict(sinks=torch.zeros(a.heads, device=dev), out_gain=0.5) if sinks else {}
        return lambda: ops.paged_prefill(q, kc, vc, bt, ts, tq, qs, ql, ql, out, n_tiles=len(tiles), window=a.window, scale=0.1, out_d=a.vdim,
                                         exact_p=True, **kw)

    def tpre(i):
        c, r = torch.randn(m // 16, G, 16, P, **bf), torch.ones(m // 16, 16, device=dev)
        q, out, gate = torch.randn(m, H * P, **bf), torch.empty(m, H * D, **bf), torch.randn(m, H * D, **bf)
        span = hops.talk_span(talk.window, L)
        step = talk_pass(len(tiles), H * 128 * span)
        ws = torch.empty(step * H * 128 * span, device=dev)

        def call():
            for t0 in range(0, len(tiles), step):
                hops.talk_prefill(q, c, r, bt, ts[t0:], tq[t0:], qs, ql, ql, n_tiles=min(step, len(tiles) - t0), h=H, d=D, window=talk.window,
                                  scale=0.1, cap=30.0, gate=gate, out=out, scores=ws, span=span, **mats)
        return call
    flops = lambda a, w: 4.0 * pairs(w) * a.heads * a.dim
    add(f"paged_prefill, window and sinks [{m} tokens of {L}]", lambda i: pre(att, i, True), m * att.heads * 4 * att.dim, flops(att, att.window))
    add(f"talk_prefill [{m} tokens of {L}]", tpre, m * H * 6 * D, flops(talk, talk.window) + 2.0 * pairs(talk.window) * H * H)
    add(f"paged_prefill, window (Kipolix) [{m} tokens of {L}]", lambda i: pre(katt, i, False), m * katt.heads * 4 * katt.dim, flops(katt, katt.window))
    add(f"paged_prefill, the talking heads' window and sizes (Kipolix) [{m} tokens of {L}]", lambda i: pre(short, i, False), m * H * 4 * D,
        flops(talk, talk.window))

    # recurrences
    N = gru.width_p
    bias = torch.zeros(2 * N, device=dev)
    sl, ps = torch.arange(batch, dtype=torch.int32, device=dev), i32([100] * batch)

    def gd(i):
        proj, st, out = torch.randn(batch, 3 * N, **bf), torch.zeros(batch, N, device=dev), torch.empty(batch, N, **bf)
        return lambda: hops.gru_decode(proj, batch, bias=bias, gain=0.5, state=st, row_slots=sl, positions=ps, out=out)
    add(f"gru_decode [{batch} x {N}]", gd, batch * N * (6 + 8 + 2))
    rh, rd, rv = ret.heads, ret.dim, ret.vdim
    pw, rrot, WR = hops.decay_powers(ret.decay, dev), hops.Rotary(ret.rot, dev), ret.in_width

    def rdec(i):
        proj, st, out = torch.randn(batch, WR, **bf), torch.zeros(batch, rh, rd, rv, device=dev), torch.empty(batch, rh * rv, **bf)
        return lambda: hops.retention_decode(proj, batch, h=rh, d=rd, e=rv, decay_pow=pw, rot=rrot, k_scale=0.1, eps=1e-5, state=st,
                                             row_slots=sl, positions=ps, out=out)
    add(f"retention_decode (Kipolix) [{batch} x {rh} states of {rd} x {rv}]", rdec, batch * (rh * rd * rv * 8 + 2 * (WR + rh * rv)))
    sq = torch.arange(ns, dtype=torch.int32, device=dev)
    gws = torch.empty(hops.gru_ws_elems(N, len(tiles)), device=dev)

    def gp(i):
        proj, st, out = torch.randn(m, 3 * N, **bf), torch.zeros(ns, N, device=dev), torch.empty(m, N, **bf)
        return lambda: hops.gru_prefill(proj, m, bias=bias, gain=0.5, state=st, seq_slots=sq, tile_seq=ts, tile_q0=tq, q_start=qs, q_lens=ql,
                                        ctx_lens=ql, n_tiles=len(tiles), ws=gws, out=out)
    add(f"gru_prefill [{m} tokens of {L}, {N} channels]", gp, m * N * 8)
    qr, kr = torch.randn(rh, m, rd, device=dev), torch.randn(rh, m, rd, device=dev)
    rws = torch.empty(2 * len(tiles) * rh * rd * rv, device=dev)

    def rp(i):
        proj, st, out = torch.randn(m, WR, **bf), torch.zeros(ns, rh, rd, rv, device=dev), torch.empty(m, rh * rv, **bf)
        return lambda: hops.retention_prefill(proj, m, h=rh, d=rd, e=rv, decay_pow=pw, eps=1e-5, state=st, seq_slots=sq, tile_seq=ts, tile_q0=tq,
                                              q_start=qs, q_lens=ql, ctx_lens=ql, n_tiles=len(tiles), n_seqs=ns, q_rot=qr, k_rot=kr, ws=rws, out=out)
    C = hops.retention_chunk()
    add(f"retention_prefill (Kipolix) [{m} tokens of {L}, {rh} heads {rd} x {rv}]", rp,
        m * rh * (2 * rd * 4 + 3 * rv * 2) + 4.0 * (m // C) * rh * rd * rv * 4, m * rh * (4.0 * rd * rv + (C + 1.0) * (rd + rv)))

    # feed-forward
    ff, kff = vok.layers[0].mlp.ff, kip.layers[0].mlp.ff
    for M in (batch, m):
        def up(i, M=M):
            x, w, o = torch.randn(M, d, **bf), ops.tile_weight(torch.randn(ff, d, **bf)), torch.empty(M, ff, **bf)
            sh = dict(bn=ops.pick_bn(ff, (M + 127) // 128))
            return lambda: ops.gemm(x, w, out=o, act=2, **sh)
        add(f"gemm up, squared ReLU [{M} rows, {d} -> {ff}]", up, 2 * (ff * d + M * (d + ff)), 2.0 * M * ff * d)

        def gu(i, M=M):
            x, w, o = torch.randn(M, d, **bf), ops.tile_weight(torch.randn(2 * kff, d, **bf)), torch.empty(M, kff, **bf)
            sh = dict(bn=ops.pick_bn(2 * kff, (M + 127) // 128))
            return lambda: ops.gemm(x, w, out=o, epi=ops.EPI_SWIGLU_BF16, **sh)
        add(f"gemm gate|up, SwiGLU (Kipolix) [{M} rows, {d} -> {2 * kff}]", gu, 2 * (2 * kff * d + M * (d + kff)), 4.0 * M * kff * d)
    return rows


def run(args, clocks) -> None:
    """`clocks`: bench.py's nvidia-smi sampler."""
    torch.cuda.set_device(0)
    peaks = load_measured_peaks()
    timer = Timer(max(3, args.warmup), max(20, args.steps))
    out = {"bench": "vokepel beside kipolix", "data": "random tokens, random weights", "layers": LAYERS,
           "peaks": {k: peaks.get(k) for k in ("hbm_gbs", "bf16_tflops")}, "sizes": {}}
    clocks.start()
    for name in [args.vokepel_size] if args.vokepel_size else list(SIZES):
        vok, kip = _configs(name)
        res = {"vokepel_params_m": round(vok.n_params() / 1e6), "kipolix_params_m": round(kip.n_params() / 1e6), "engine": []}
        for batch, prompt in ((1, 2048), (32, 2048), (128, 2048)):
            row = {"batch": batch, "prompt": prompt}
            for key, mc in (("vokepel", vok), ("kipolix", kip)):
                row[key] = engine_numbers(replace(mc), batch=batch, prompt=prompt, warmup=max(3, args.warmup), steps=args.steps)
                torch.cuda.empty_cache()
            res["engine"].append(row)
        res["kernels"] = kernel_numbers(vok, kip, peaks, timer, batch=64, ctx=4096, m=8192)
        out["sizes"][name] = res
        torch.cuda.empty_cache()
    out["clocks"] = clocks.stop()
    print(json.dumps(out), flush=True)
