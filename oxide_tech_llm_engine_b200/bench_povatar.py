"""Povatar layers (attention and a state-space mixer side by side, a mixture of experts beside them) next to the
closest existing models: prompt and decode throughput through the engine beside the Mixtral-shaped model of
equal width, heads, experts and expert parameters, and every kernel of the design against its roofline next to
the like kernel (Llama / Mixtral attention, norm, dispatch and expert products; retention for the recurrence).

    python bench.py --povatar [--steps K --warmup W]

A size is a few layers of a real model's shape with random weights. Timing and rooflines as in bench_hybrid:
CUDA events, buffers that together exceed L2, measured copy bandwidth and bf16 rate.
"""
from __future__ import annotations

import json
from dataclasses import replace

import torch

from .bench_hybrid import Timer, _copies, engine_numbers
from .utils.roofline import load_measured_peaks

SIZES = {
    # 64 small experts; few large experts; heads of 64 with a narrower state
    "w2048-e64": dict(width=2048, n_layers=8, heads=16, kv_heads=4, dim=128, chunk=8192, s_heads=64, s_vdim=64, state=128, groups=8,
                      ff=1536, experts=64, top=8),
    "w4096-e8": dict(width=4096, n_layers=4, heads=32, kv_heads=8, dim=128, chunk=8192, s_heads=128, s_vdim=64, state=128, groups=8,
                     ff=10752, experts=8, top=2),
    "w1536-e32": dict(width=1536, n_layers=8, heads=24, kv_heads=6, dim=64, chunk=1024, s_heads=48, s_vdim=64, state=64, groups=1,
                      ff=768, experts=32, top=4),
}
VOCAB = 32000


def _configs(name: str, layers: int = 0):
    from .models.config import ModelConfig, _povatar_preset

    z = dict(SIZES[name])
    if layers:
        z["n_layers"] = layers
    pov = _povatar_preset("povatar-" + name, vocab=VOCAB, **z)
    mix = ModelConfig(name="mixtral-" + name, arch="mixtral", n_layers=z["n_layers"], d_model=z["width"], n_heads=z["heads"],
                      n_kv_heads=z["kv_heads"], head_dim=z["dim"], ffn_dim=z["ff"] * 2 // 3, vocab_size=VOCAB, max_ctx=1 << 17,
                      n_experts=z["experts"], n_experts_used=z["top"])
    return pov, mix


def kernel_numbers(pov, mix, peaks: dict, timer: Timer, batch: int, ctx: int, m: int) -> list:
    """One row per kernel: name, microseconds, roofline microseconds, fraction of the roofline."""
    from . import ops
    from .ops import hybrid as hops

    dev = torch.device("cuda", 0)
    bf = dict(dtype=torch.bfloat16, device=dev)
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=dev)
    bw, fl = peaks["hbm_gbs"] * 1e3, peaks["bf16_tflops"] * 1e6        # bytes / us, flops / us
    rows = []

    def add(name, calls_of, nbytes, flops=0.0, launches=1):
        n = _copies(nbytes)
        us = timer([calls_of(i) for i in range(n)])
        roof = max(nbytes / bw, flops / fl)
        rows.append({"kernel": name, "us": round(us, 2), "roofline_us": round(roof, 2), "fraction": round(roof / us, 3)})
        torch.cuda.empty_cache()

    L0 = pov.layers[0]
    att, ssd, moe = L0.mixer.left, L0.mixer.right, L0.mlp
    d, E, top, ff = pov.d_model, moe.experts, moe.top, moe.ff
    P = 64 if max(att.dim, att.vdim) <= 64 else 128
    W = att.heads * att.dim + att.kv_heads * (att.dim + att.vdim)
    Wp = (W + 63) // 64 * 64 + ssd.width_p
    rot = hops.Rotary(att.rot, dev)
    D, Hq, Hk = mix.head_dim, mix.n_heads, mix.n_kv_heads
    for M in (batch, m):
        tag = f"[{M} rows]"
        ones, one32 = torch.ones(d, device=dev), torch.ones(d, **bf)
        pages = M // 16 + 1
        pos, slots = torch.arange(M, dtype=torch.int32, device=dev), torch.arange(M, device=dev)

        def bn(i, M=M):
            x, ys = torch.randn(M, d, device=dev), [torch.randn(M, d, device=dev) for _ in range(2)]
            er, h = torch.randn(M * top, d, **bf), [torch.empty(M, d, **bf) for _ in range(2)]
            sl, wt = torch.randperm(M * top, device=dev).to(torch.int32), torch.rand(M * top, device=dev)
            return lambda: hops.branch_norm(x, M, norm_w=[ones, ones], h=h, eps=1e-5, branches=[(y, ones, 0.5, False) for y in ys],
                                            experts=(er, sl, wt, top))
        add("branch_norm " + tag, bn, M * d * (8 + 8 + 2 * top + 4))

        def fn(i, M=M):
            acc, res, out = torch.randn(M, d, device=dev), torch.zeros(M, d, **bf), torch.empty(M, d, **bf)
            return lambda: ops.finalize_norm(rows=M, n=d, acc=acc, residual_in=res, residual_out=res, norm_w=one32,
                                             out_ptrs=[out.data_ptr()], device=dev)
        add("finalize_norm (Mixtral) " + tag, fn, M * d * (8 + 4 + 2))

        def hd(i, M=M):
            proj, q = torch.randn(M, Wp, **bf), torch.empty(M, att.heads * P, **bf)
            kc, vc = torch.zeros(pages, att.kv_heads, 16, P, **bf), torch.zeros(pages, att.kv_heads, 16, P, **bf)
            return lambda: hops.heads(proj, M, h=att.heads, g=att.kv_heads, d=att.dim, e=att.vdim, rot=rot, positions=pos, q_out=q,
                                      q_hd=P, k_cache=kc, v_cache=vc, slots=slots)
        add("heads " + tag, hd, 4 * M * W)
        inv = torch.ones(D // 2, device=dev)

        def qr(i, M=M):
            proj, q = torch.randn(M, (Hq + 2 * Hk) * D, **bf), torch.empty(M, Hq * D, **bf)
            kc, vc = torch.zeros(pages, Hk, 16, D, **bf), torch.zeros(pages, Hk, 16, D, **bf)
            return lambda: ops.qkv_rope_append(qkv_bf16=proj, positions=pos, slot_mapping=slots, inv_freq=inv, q_out=q, k_cache=kc,
                                               v_cache=vc, m=M, hq=Hq, hkv=Hk, d=D)
        add("qkv_rope_append (Mixtral) " + tag, qr, 4 * M * (Hq + 2 * Hk) * D)

        nw = torch.ones(ssd.inner, device=dev)

        def gn(i, M=M):
            y, proj, out = torch.randn(M, ssd.inner, **bf), torch.randn(M, ssd.width_p, **bf), torch.empty(M, ssd.inner, **bf)
            return lambda: hops.gated_norm(y, proj, M, h=ssd.heads, e=ssd.vdim, ep=ssd.vdim_p, groups=ssd.norm_groups, w=nw, eps=1e-5,
                                           out=out)
        if ssd.vdim == ssd.vdim_p:
            add("gated_norm " + tag, gn, M * ssd.inner * 6)

        # router and placement of the chosen rows
        router = torch.randn((E + 63) // 64 * 64, d, **bf) * d ** -0.5
        counts = torch.zeros(E, dtype=torch.int32, device=dev)
        wt, ex, sl = torch.zeros(M * top, device=dev), torch.zeros(M * top, dtype=torch.int32, device=dev), torch.zeros(
            M * top, dtype=torch.int32, device=dev)
        m_tiles = min(E, M * top) if M <= 128 else (M * top + 127 * E) // 128
        n_rows = max(E * 128, m_tiles * 128)
        kw = dict(e=E, top=top, weight=wt, expert=ex, slot=sl)

        def route(h, xs, logits, M=M):
            counts.zero_()
            if M <= 128:
                hops.moe_route(h, router[:E], M, mode=1, counts=counts, xs=xs, **kw)
            else:
                ops.gemm(h, router, out=logits, epi=ops.EPI_STORE_F32, bn=64)
                hops.moe_route(h, router[:E], M, mode=2, logits=logits, counts=counts, **kw)
                hops.moe_scatter(h, M, e=E, top=top, expert=ex, slot=sl, counts=counts, xs=xs)

        def mr(i, M=M):
            h, xs, lg = torch.randn(M, d, **bf), torch.empty(n_rows, d, **bf), torch.empty(M, router.shape[0], device=dev)
            return lambda: route(h, xs, lg)
        add("router and placement " + tag, mr, M * d * 2 * (1 + top) + E * d * 2, 2.0 * M * E * d)
        if E <= 64 and top <= 8:
            cap = max(M, 128)
            meta = torch.zeros(E * cap * 4, dtype=torch.int32, device=dev)

            def fm(i, M=M):
                acc, res, slab = torch.randn(M, d, device=dev), torch.zeros(M, d, **bf), torch.empty(E, cap, d, **bf)

                def call():
                    counts.zero_()
                    ops.finalize_norm(rows=M, n=d, acc=acc, residual_in=res, residual_out=res, norm_w=one32, router_w=router[:E],
                                      top_k=top, experts_per_rank=E, slab_ptrs=[slab.data_ptr()], meta_ptrs=[meta.data_ptr()],
                                      cnt_ptrs=[counts.data_ptr()], cap=cap, device=dev)
                return call
            add("finalize_norm with router and dispatch (Mixtral) " + tag, fm, M * d * (8 + 4 + 2 * top) + E * d * 2, 2.0 * M * E * d)

        # expert products on the rows of one routed step
        h = torch.randn(M, d, **bf)
        xs = torch.zeros(n_rows, d, **bf)
        route(h, xs, torch.empty(M, router.shape[0], device=dev))
        active = int((counts > 0).sum())
        pairs = M * top
        flops = 2.0 * pairs * d * ff
        nb = active * d * ff * 2 + pairs * (d + ff) * 2
        reps = 1 if E * d * ff * 2 > 300e6 else 2
        ups, downs = [torch.randn(E, ff, d, **bf) for _ in range(reps)], [torch.randn(E, d, ff, **bf) for _ in range(reps)]
        act, out = torch.zeros(n_rows, ff, **bf), torch.zeros(n_rows, d, **bf)
        if M <= 128:
            v = lambda t: t[:E * 128].view(E, 128, -1)
        else:
            v = lambda t: t[:m_tiles * 128]
        bnw = lambda n: next((b for b in (256, 128) if m_tiles * ((n + b - 1) // b) >= 148), 64)
        add(f"expert up, squared ReLU [{M} rows x {top}]", lambda i: (lambda: ops.gemm(
            v(xs), ups[i % reps], out=v(act), group_counts=counts, m_tiles=m_tiles, act=2, bn=bnw(ff))), nb, flops)
        add(f"expert down [{M} rows x {top}]", lambda i: (lambda: ops.gemm(
            v(act), downs[i % reps], out=v(out), group_counts=counts, m_tiles=m_tiles, bn=bnw(d))), nb, flops)
        fm_ = mix.ffn_dim
        cap = max(M, 128)
        gus, dws = [torch.randn(E, 2 * fm_, d, **bf) for _ in range(reps)], [torch.randn(E, d, fm_, **bf) for _ in range(reps)]
        slab, acts, acc = torch.zeros(E, cap, d, **bf), torch.zeros(E, cap, fm_, **bf), torch.zeros(M, d, device=dev)
        # where each slab row goes back to
        meta = torch.zeros(E, cap, 4, dtype=torch.int32, device=dev)
        meta[..., 1] = torch.randint(0, M, (E, cap), device=dev)
        add(f"expert gate and up, SwiGLU (Mixtral) [{M} rows x {top}]", lambda i: (lambda: ops.gemm(
            slab, gus[i % reps], out=acts, epi=ops.EPI_SWIGLU_BF16, group_counts=counts, m_tiles=(M * top + 127) // 128 + E, bn=128)),
            active * 2 * d * fm_ * 2 + pairs * (d + fm_) * 2, 4.0 * pairs * d * fm_)
        add(f"expert down, combine (Mixtral) [{M} rows x {top}]", lambda i: (lambda: ops.gemm(
            acts, dws[i % reps], epi=ops.EPI_RED_F32, dst_ptrs=[acc.data_ptr()], group_counts=counts, row_meta=meta,
            m_tiles=(M * top + 127) // 128 + E, bn=128)), active * d * fm_ * 2 + pairs * (fm_ * 2 + d * 4), 2.0 * pairs * d * fm_)
        del ups, downs, gus, dws, slab, acts, act, out, xs
        torch.cuda.empty_cache()

    nb_seq = ctx // 16
    splits = 16

    def dec(hq, hk, D, P, chunk, sink, exact):
        kc, vc = torch.zeros(batch * nb_seq, hk, 16, P, **bf), torch.zeros(batch * nb_seq, hk, 16, P, **bf)
        bt = torch.randperm(batch * nb_seq, device=dev).to(torch.int32).view(batch, nb_seq)
        q, out = torch.randn(batch, hq, P, **bf), torch.empty(batch, hq * D, **bf)
        po, pm = torch.empty(batch * hq * splits * P, device=dev), torch.empty(batch * hq * splits * 2, device=dev)
        per_sm = 12 if hk >= 4 else 4
        want = max(1, min(splits, -(-per_sm * 148 // (batch * hk))))
        pps = i32([(max(4, -(-nb_seq // want)) + 3) // 4 * 4])
        lens = i32([ctx] * batch)
        return lambda: ops.paged_decode(q, kc, vc, bt, lens, pps, po, pm, out, batch=batch, max_splits=splits, scale=0.1, out_d=D,
                                        exact_p=exact, chunk=chunk, sink=sink)
    vis = ctx - (ctx - 1) // att.chunk * att.chunk
    add(f"paged_decode, chunks and sink [{batch} x {vis} keys]", lambda i: dec(att.heads, att.kv_heads, att.vdim, P, att.chunk, 0.0, True),
        batch * vis * att.kv_heads * (att.dim + att.vdim) * 2)
    add(f"paged_decode (Mixtral) [{batch} x {ctx} keys]", lambda i: dec(Hq, Hk, D, D, 0, float("-inf"), False), batch * ctx * Hk * D * 4)

    L = 2048
    ns = m // L
    tiles = [(s, t * 128) for s in range(ns) for t in range(L // 128)]
    ts, tq = i32([t[0] for t in tiles]), i32([t[1] for t in tiles])
    qs, ql = i32([s * L for s in range(ns)]), i32([L] * ns)

    def pre(hq, hk, D, P, chunk, sink, exact):
        kc, vc = torch.randn(m // 16, hk, 16, P, **bf), torch.randn(m // 16, hk, 16, P, **bf)
        bt = torch.arange(m // 16, dtype=torch.int32, device=dev).view(ns, L // 16)
        q, out = torch.randn(m, hq, P, **bf), torch.empty(m, hq * D, **bf)
        return lambda: ops.paged_prefill(q, kc, vc, bt, ts, tq, qs, ql, ql, out, n_tiles=len(tiles), scale=0.1, out_d=D, exact_p=exact,
                                         chunk=chunk, sink=sink)
    pairs = sum(i % att.chunk + 1 for i in range(L)) * ns
    add(f"paged_prefill, chunks and sink [{m} tokens of {L}]",
        lambda i: pre(att.heads, att.kv_heads, att.vdim, P, att.chunk, 0.0, True), m * att.heads * 4 * att.dim,
        2.0 * pairs * att.heads * (att.dim + att.vdim))
    add(f"paged_prefill (Mixtral) [{m} tokens of {L}]", lambda i: pre(Hq, Hk, D, D, 0, float("-inf"), False), m * Hq * 4 * D,
        4.0 * (L * (L + 1) // 2 * ns) * Hq * D)

    # state-space layer, and retention with states of the same shape
    h, G, N, V = ssd.heads, ssd.groups, ssd.state_p, ssd.vdim_p
    ch = ssd.channels_p
    w = (torch.randn(ch, ssd.taps, device=dev), torch.zeros(ch, device=dev), torch.zeros(h, device=dev), torch.zeros(h, device=dev),
         torch.ones(h, device=dev))

    def sd(i):
        proj, st = torch.randn(batch, (ssd.width_p + 7) // 8 * 8, **bf), torch.zeros(batch, h, N, V, device=dev)
        cv, y = torch.zeros(batch, ssd.taps, ch, device=dev), torch.empty(batch, h * V, **bf)
        sl, ps = torch.arange(batch, dtype=torch.int32, device=dev), i32([100] * batch)
        return lambda: hops.ssd_decode(proj, batch, h=h, g=G, w=w, state=st, conv_state=cv, row_slots=sl, positions=ps, y=y)
    add(f"ssd_decode [{batch} x {h} states of {N} x {V}]", sd,
        batch * (h * N * V * 8 + 2 * (ch + h * V) + 4 * ch * (ssd.taps + 1)))
    pw, nrot = hops.decay_powers([0.99] * h, dev), hops.Rotary(None, dev)

    def rd(i):
        proj, st, out = torch.randn(batch, 2 * h * (N + V), **bf), torch.zeros(batch, h, N, V, device=dev), torch.empty(batch, h * V, **bf)
        sl, ps = torch.arange(batch, dtype=torch.int32, device=dev), i32([100] * batch)
        return lambda: hops.retention_decode(proj, batch, h=h, d=N, e=V, decay_pow=pw, rot=nrot, k_scale=1.0, eps=1e-5, state=st,
                                             row_slots=sl, positions=ps, out=out)
    add(f"retention_decode [{batch} x {h} states of {N} x {V}]", rd, batch * (h * N * V * 8 + 2 * (2 * h * (N + V) + h * V)))

    for mm, nseq in ((m, ns), (L, 1)):
        tl = tiles[:mm // 128]
        sq = torch.arange(nseq, dtype=torch.int32, device=dev)
        u, y = torch.empty(mm, ch, **bf), torch.empty(mm, h * V, **bf)
        seg = hops.ssd_segment(h, V, len(tl), nseq)
        sws = torch.empty(hops.ssd_ws_elems(h, V, N, len(tl)), device=dev) if seg else None

        def sp(i):
            proj = torch.randn(mm, (ssd.width_p + 7) // 8 * 8, **bf)
            st, cv = torch.zeros(nseq, h, N, V, device=dev), torch.zeros(nseq, ssd.taps, ch, device=dev)
            return lambda: hops.ssd_prefill(proj, mm, h=h, g=G, w=w, state=st, conv_state=cv, seq_slots=sq, tile_seq=ts, tile_q0=tq,
                                            q_start=qs, q_lens=ql, ctx_lens=ql, n_tiles=len(tl), n_seqs=nseq, u=u, y=y, runs=True,
                                            segment=seg, ws=sws)
        C = 64
        # the projection in, the convolved channels out and in again, y out, the states of the sequences; the run form's
        # arithmetic (for retention its inputs, output and states; neither counts the states between chunks or segments)
        add(f"ssd convolution and runs [{mm} tokens of {L}, {h} heads {N} x {V}]", sp, mm * 2 * (3 * ch + h * V) + nseq * h * N * V * 8,
            mm * (h * (4.0 * N * V + (C + 1) * V) + G * (C + 1) * N))
        qr_, kr_ = torch.randn(h, mm, N, device=dev), torch.randn(h, mm, N, device=dev)
        ws = torch.empty(2 * len(tl) * h * N * V, device=dev)
        proj, out = torch.randn(mm, 2 * h * (N + V), **bf), torch.empty(mm, h * V, **bf)

        def rp(i):
            st = torch.zeros(nseq, h, N, V, device=dev)
            return lambda: hops.retention_prefill(proj, mm, h=h, d=N, e=V, decay_pow=pw, eps=1e-5, state=st, seq_slots=sq, tile_seq=ts,
                                                  tile_q0=tq, q_start=qs, q_lens=ql, ctx_lens=ql, n_tiles=len(tl), n_seqs=nseq,
                                                  q_rot=qr_, k_rot=kr_, ws=ws, out=out)
        add(f"retention_prefill [{mm} tokens of {L}, {h} heads {N} x {V}]", rp, mm * h * (2 * N * 4 + 3 * V * 2) + nseq * h * N * V * 8,
            mm * h * (4.0 * N * V + (C + 1) * (N + V)))
    return rows


def run(args, clocks) -> None:
    """`clocks`: bench.py's nvidia-smi sampler."""
    torch.cuda.set_device(0)
    peaks = load_measured_peaks()
    timer = Timer(max(3, args.warmup), max(20, args.steps))
    out = {"bench": "povatar beside mixtral", "data": "random tokens, random weights",
           "peaks": {k: peaks.get(k) for k in ("hbm_gbs", "bf16_tflops")}, "sizes": {}}
    clocks.start()
    for name in [args.povatar_size] if args.povatar_size else list(SIZES):
        pov, mix = _configs(name, args.layers)
        res = {"povatar_params_m": round(pov.n_params() / 1e6), "mixtral_params_m": round(mix.n_params() / 1e6), "layers": pov.n_layers,
               "engine": []}
        for batch, prompt in ((1, 2048), (32, 2048), (128, 2048)):
            row = {"batch": batch, "prompt": prompt}
            for key, mc in (("povatar", pov), ("mixtral", mix)):
                row[key] = engine_numbers(replace(mc), batch=batch, prompt=prompt, warmup=max(3, args.warmup), steps=args.steps)
                torch.cuda.empty_cache()
            res["engine"].append(row)
        res["kernels"] = kernel_numbers(pov, mix, peaks, timer, batch=64, ctx=4096, m=8192)
        out["sizes"][name] = res
        torch.cuda.empty_cache()
    out["clocks"] = clocks.stop()
    print(json.dumps(out), flush=True)
