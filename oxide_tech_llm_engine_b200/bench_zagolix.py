"""Zagolix layers (differential attention, latent attention with shared latents, matrix memory, gated experts behind a
grouped sigmoid router) next to the closest existing models: prompt and decode throughput through the engine beside the
Mixtral-shaped model of equal width, experts and expert size, and every kernel of the design against its roofline next to
the like kernel (Mixtral's attention, norm, dispatch and expert products; retention for the recurrence).

    python bench.py --zagolix [--steps K --warmup W]

A size is a few layers of a real model's shape with random weights. Timing and rooflines as in bench_hybrid: CUDA events,
buffers that together exceed L2, measured copy bandwidth and bf16 rate. Arithmetic is what the equations need: the zeros
beside the keys of the other map, the second term of the softmax weights and the terms of 32-bit operands do not count.
"""
from __future__ import annotations

import json
from dataclasses import replace

import torch

from .bench_hybrid import Timer, _copies, engine_numbers
from .utils.roofline import load_measured_peaks

SIZES = {
    # 64 small experts and 16 heads over latents of 512 + 64; 40 narrow heads over 256 + 32; few large experts and 32 heads
    "w2048-e64": dict(width=2048, pattern="alsm" * 2, ff=8192, heads=16, kv_heads=4, dim=64, l_heads=16, l_dim=128, rot=64, l_vdim=128,
                      q_rank=1536, kv_rank=512, m_heads=4, m_dim=256, m_vdim=512, e_ff=1408, experts=64, top=6, groups=8, keep=4),
    "w2560-e32": dict(width=2560, pattern="alsm" * 2, ff=6400, heads=20, kv_heads=4, dim=64, l_heads=40, l_dim=64, rot=32, l_vdim=64,
                      q_rank=768, kv_rank=256, m_heads=10, m_dim=128, m_vdim=256, e_ff=1280, experts=32, top=4, groups=4, keep=2),
    "w4096-e8": dict(width=4096, pattern="alsm", ff=14336, heads=32, kv_heads=8, dim=64, l_heads=32, l_dim=128, rot=64, l_vdim=128,
                     q_rank=1536, kv_rank=512, m_heads=8, m_dim=256, m_vdim=512, e_ff=7168, experts=8, top=2, groups=2, keep=1),
}
VOCAB = 32000


def _configs(name: str):
    from .models.config import ModelConfig, _zagolix_preset

    z = SIZES[name]
    zag = _zagolix_preset("zagolix-" + name, vocab=VOCAB, **z)
    mix = ModelConfig(name="mixtral-" + name, arch="mixtral", n_layers=len(z["pattern"]), d_model=z["width"], n_heads=z["width"] // 128,
                      n_kv_heads=4 if z["width"] % 1024 else z["kv_heads"], head_dim=128, ffn_dim=z["e_ff"], vocab_size=VOCAB,
                      max_ctx=1 << 17, n_experts=z["experts"], n_experts_used=z["top"])
    return zag, mix


def kernel_numbers(zag, mix, peaks: dict, timer: Timer, batch: int, ctx: int, m: int) -> list:
    """One row per kernel: name, microseconds, roofline microseconds, fraction of the roofline."""
    from . import ops
    from .models.hybrid import latent_layout, tc_head
    from .ops import hybrid as hops

    dev = torch.device("cuda", 0)
    bf = dict(dtype=torch.bfloat16, device=dev)
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=dev)
    bw, fl = peaks["hbm_gbs"] * 1e3, peaks["bf16_tflops"] * 1e6        # bytes / us, flops / us
    rows = []

    def add(name, calls_of, nbytes, flops=0.0):
        n = _copies(nbytes)
        us = timer([calls_of(i) for i in range(n)])
        roof = max(nbytes / bw, flops / fl)
        rows.append({"kernel": name, "us": round(us, 2), "roofline_us": round(roof, 2), "fraction": round(roof / us, 3)})
        torch.cuda.empty_cache()

    kind = lambda k: next(L for L in zag.layers if L.mixer.kind == k)
    att, lat, mem = (kind(k).mixer for k in ("attention", "latent_attention", "mlstm"))
    moe = kind("mlstm").mlp
    d, E, top, ff = zag.d_model, moe.experts, moe.top, moe.ff
    D, Hq, Hk = mix.head_dim, mix.n_heads, mix.n_kv_heads
    nq, P = att.heads * 2, tc_head(att)
    H, R, T, cp = lat.heads, lat.kv_rank, lat.rot_dim, lat.cache_row
    dk, dv, at = latent_layout(lat)
    rot, none = hops.Rotary(lat.rot, dev), hops.Rotary(None, dev)
    for M in (batch, m):
        tag = f"[{M} rows]"
        ones, one32 = torch.ones(d, device=dev), torch.ones(d, **bf)
        pages = M // 16 + 1
        pos, slots = torch.arange(M, dtype=torch.int32, device=dev), torch.arange(M, device=dev)

        def bn(i, M=M, experts=False):
            x, y = torch.randn(M, d, device=dev), torch.randn(M, d, device=dev)
            er, h = torch.randn(M * top if experts else 1, d, **bf), torch.empty(M, d, **bf)
            sl, wt = torch.randperm(M * top, device=dev).to(torch.int32), torch.rand(M * top, device=dev)
            kw = dict(branches=[(None, ones, 1.0, False)], experts=(er, sl, wt, top)) if experts else dict(branches=[(y, ones, 1.0, False)])
            return lambda: hops.branch_norm(x, M, norm_w=[ones], h=[h], eps=1e-5, **kw)
        add("branch_norm " + tag, bn, M * d * (8 + 4 + 2))
        add("branch_norm of the expert rows " + tag, lambda i: bn(i, experts=True), M * d * (8 + 2 * top + 2))

        def fn(i, M=M):
            acc, res, out = torch.randn(M, d, device=dev), torch.zeros(M, d, **bf), torch.empty(M, d, **bf)
            return lambda: ops.finalize_norm(rows=M, n=d, acc=acc, residual_in=res, residual_out=res, norm_w=one32,
                                             out_ptrs=[out.data_ptr()], device=dev)
        add("finalize_norm (Mixtral) " + tag, fn, M * d * (8 + 4 + 2))

        W = att.in_width
        bias = torch.zeros(W, device=dev)

        def hd(i, M=M):
            proj, q = torch.randn(M, W, **bf), torch.zeros(M, nq * P, **bf)
            kc, vc = torch.zeros(pages, att.kv_heads, 16, P, **bf), torch.zeros(pages, att.kv_heads, 16, P, **bf)
            return lambda: hops.heads(proj, M, h=nq, g=att.kv_heads * 2, d=att.dim, e=att.vdim, rot=none, positions=pos, q_out=q, q_hd=P,
                                      k_cache=kc, v_cache=vc, slots=slots, maps=2, bias=bias, temp_coef=0.1, temp_every=64.0)
        add("heads, two maps " + tag, hd, 4 * M * W)
        Wl = lat.in_width

        def lr(i, M=M):
            proj, q, c = torch.randn(M, (Wl + 63) // 64 * 64, **bf), torch.empty(M, lat.q_rank, **bf), torch.zeros(pages, 1, 16, cp, **bf)
            qn, kn = torch.ones(lat.q_rank, device=dev), torch.ones(R, device=dev)
            return lambda: hops.latent_rows(proj, M, q_rank=lat.q_rank, q_norm=qn, q_out=q, positions=pos, eps=1e-5, kv_col=lat.kv_col,
                                            kv_rank=R, kv_norm=kn, cache=c, slots=slots, rot=rot)
        add("latent_rows " + tag, lr, 4 * M * Wl)

        def hr(i, M=M):
            q = torch.randn(M, H * dk, **bf)
            return lambda: hops.heads(q, M, h=H, g=0, d=T, e=4, rot=rot, positions=pos, q_out=q, q_hd=dk, q_pd=dk)
        add("heads, rotated part of latent queries " + tag, hr, 4 * M * H * T)
        inv = torch.ones(D // 2, device=dev)

        def qr(i, M=M):
            proj, q = torch.randn(M, (Hq + 2 * Hk) * D, **bf), torch.empty(M, Hq * D, **bf)
            kc, vc = torch.zeros(pages, Hk, 16, D, **bf), torch.zeros(pages, Hk, 16, D, **bf)
            return lambda: ops.qkv_rope_append(qkv_bf16=proj, positions=pos, slot_mapping=slots, inv_freq=inv, q_out=q, k_cache=kc,
                                               v_cache=vc, m=M, hq=Hq, hkv=Hk, d=D)
        add("qkv_rope_append (Mixtral) " + tag, qr, 4 * M * (Hq + 2 * Hk) * D)

        # router and placement of the chosen rows
        router = torch.randn((E + 63) // 64 * 64, d, **bf) * d ** -0.5
        counts = torch.zeros(E, dtype=torch.int32, device=dev)
        wt, ex, sl = torch.zeros(M * top, device=dev), torch.zeros(M * top, dtype=torch.int32, device=dev), torch.zeros(
            M * top, dtype=torch.int32, device=dev)
        m_tiles = min(E, M * top) if M <= 128 else (M * top + 127 * E) // 128
        n_rows = max(E * 128, m_tiles * 128)

        def route(h, xs, logits, M=M, like=False):
            counts.zero_()
            kw = dict(e=E, top=top, weight=wt, expert=ex, slot=sl)
            if not like:
                kw.update(softmax=False, groups=moe.groups, keep=moe.keep)
            if M <= 128:
                hops.moe_route(h, router[:E], M, mode=1, counts=counts, xs=xs, **kw)
            else:
                ops.gemm(h, router, out=logits, epi=ops.EPI_STORE_F32, bn=64)
                hops.moe_route(h, router[:E], M, mode=2, logits=logits, counts=counts, **kw)
                hops.moe_scatter(h, M, e=E, top=top, expert=ex, slot=sl, counts=counts, xs=xs)

        def mr(i, M=M, like=False):
            h, xs, lg = torch.randn(M, d, **bf), torch.empty(n_rows, d, **bf), torch.empty(M, router.shape[0], device=dev)
            return lambda: route(h, xs, lg, like=like)
        add("router with groups and placement " + tag, mr, M * d * 2 * (1 + top) + E * d * 2, 2.0 * M * E * d)
        add("router and placement (Povatar) " + tag, lambda i: mr(i, like=True), M * d * 2 * (1 + top) + E * d * 2, 2.0 * M * E * d)

        # expert products on the rows of one routed step
        h = torch.randn(M, d, **bf)
        xs = torch.zeros(n_rows, d, **bf)
        route(h, xs, torch.empty(M, router.shape[0], device=dev))
        active, pairs = int((counts > 0).sum()), M * top
        reps = 1 if E * d * ff * 2 > 300e6 else 2
        gus, dws = [torch.randn(E, 2 * ff, d, **bf) for _ in range(reps)], [torch.randn(E, d, ff, **bf) for _ in range(reps)]
        act, out = torch.zeros(n_rows, ff, **bf), torch.zeros(n_rows, d, **bf)
        v = (lambda t: t[:E * 128].view(E, 128, -1)) if M <= 128 else (lambda t: t[:m_tiles * 128])
        width = lambda n, whole: next((b for b in (256, 128) if (not whole or n % b == 0) and m_tiles * ((n + b - 1) // b) >= 148), 64)
        up_b, up_f = active * 2 * d * ff * 2 + pairs * (d + ff) * 2, 4.0 * pairs * d * ff
        dn_b, dn_f = active * d * ff * 2 + pairs * (d + ff) * 2, 2.0 * pairs * d * ff
        add(f"expert gate and up, SwiGLU [{M} rows x {top}]", lambda i: (lambda: ops.gemm(
            v(xs), gus[i % reps], out=v(act), epi=ops.EPI_SWIGLU_BF16, group_counts=counts, m_tiles=m_tiles, bn=width(2 * ff, True))), up_b, up_f)
        add(f"expert down [{M} rows x {top}]", lambda i: (lambda: ops.gemm(
            v(act), dws[i % reps], out=v(out), group_counts=counts, m_tiles=m_tiles, bn=width(d, False))), dn_b, dn_f)
        cap = max(M, 128)
        if E * cap * d * 2 < 20e9:
            slab, acts, acc = torch.zeros(E, cap, d, **bf), torch.zeros(E, cap, ff, **bf), torch.zeros(M, d, device=dev)
            meta = torch.zeros(E, cap, 4, dtype=torch.int32, device=dev)      # where each slab row goes back to
            meta[..., 1] = torch.randint(0, M, (E, cap), device=dev)
            mt = (M * top + 127) // 128 + E
            add(f"expert gate and up, SwiGLU (Mixtral) [{M} rows x {top}]", lambda i: (lambda: ops.gemm(
                slab, gus[i % reps], out=acts, epi=ops.EPI_SWIGLU_BF16, group_counts=counts, m_tiles=mt, bn=128)), up_b, up_f)
            add(f"expert down, combine (Mixtral) [{M} rows x {top}]", lambda i: (lambda: ops.gemm(
                acts, dws[i % reps], epi=ops.EPI_RED_F32, dst_ptrs=[acc.data_ptr()], group_counts=counts, row_meta=meta, m_tiles=mt,
                bn=128)), dn_b, dn_f)
            del slab, acts, acc, meta
        del gus, dws, act, out, xs
        torch.cuda.empty_cache()

    # decode attention: `batch` sequences of `ctx` tokens
    nb_seq, splits = ctx // 16, 16
    bt = torch.randperm(batch * nb_seq, device=dev).to(torch.int32).view(batch, nb_seq)
    lens = i32([ctx] * batch)

    def split_pages(hk):
        want = max(1, min(splits, -(-(12 if hk >= 4 else 4) * 148 // (batch * hk))))
        return i32([(max(4, -(-nb_seq // want)) + 3) // 4 * 4])

    def dec(hq, hk, P, od, exact, diff=()):
        kc, vc = torch.zeros(batch * nb_seq, hk, 16, P, **bf), torch.zeros(batch * nb_seq, hk, 16, P, **bf)
        q, out = torch.randn(batch, hq, P, **bf), torch.empty(batch, hq * P, **bf)
        po, pm = torch.empty(batch * hq * splits * P, device=dev), torch.empty(batch * hq * splits * 2, device=dev)
        pps = split_pages(hk)
        return lambda: ops.paged_decode(q, kc, vc, bt, lens, pps, po, pm, out, batch=batch, max_splits=splits, scale=0.1, out_d=od,
                                        exact_p=exact, diff=diff)
    add(f"paged_decode, two maps and their difference [{batch} x {ctx} keys]", lambda i: dec(nq, att.kv_heads, P, att.vdim, True, (0.4, 0.5, 1e-5)),
        batch * ctx * att.cache_values * 2, 2.0 * batch * ctx * nq * (att.dim + att.vdim))

    def ld(i):
        c = torch.zeros(batch * nb_seq, 1, 16, cp, **bf)
        q, out = torch.randn(batch, H, cp, **bf), torch.empty(batch, H * R, **bf)
        po, pm = torch.empty(batch * H * splits * R, device=dev), torch.empty(batch * H * splits * 2, device=dev)
        return lambda: hops.latent_decode(q, c, bt, lens, po, pm, out, rows=batch, kv_rank=R, max_splits=splits, scale=0.1, o_hd=R)
    add(f"latent_decode [{batch} x {ctx} keys, {H} heads, {R} + {T}]", ld, batch * ctx * (R + T) * 2, 2.0 * batch * ctx * H * (2 * R + T))
    add(f"paged_decode (Mixtral) [{batch} x {ctx} keys]", lambda i: dec(Hq, Hk, D, D, False), batch * ctx * Hk * D * 4)

    def ph(i, up):
        q, c, o = torch.randn(batch, H, dk, **bf), torch.randn(batch, H, cp, **bf), torch.empty(batch, H, lat.vdim, **bf)
        x, w, y = ((q[:, :, at:at + lat.dim], torch.randn(H, R, lat.dim, **bf), c[:, :, :R]) if up
                   else (c[:, :, :R], torch.randn(H, lat.vdim, R, **bf), o))
        return lambda: ops.gemm(x.transpose(0, 1), w, out=y.transpose(0, 1), bn=64)
    add(f"queries times W_uk [{batch} rows, {H} heads]", lambda i: ph(i, True), 2 * H * (R * lat.dim + batch * (R + lat.dim)))
    add(f"latents times W_uv [{batch} rows, {H} heads]", lambda i: ph(i, False), 2 * H * (R * lat.vdim + batch * (R + lat.vdim)))

    # prompt attention: m tokens in sequences of 2048
    L = 2048
    ns = m // L
    tiles = [(s, t * 128) for s in range(ns) for t in range(L // 128)]
    ts, tq = i32([t[0] for t in tiles]), i32([t[1] for t in tiles])
    qs, ql = i32([s * L for s in range(ns)]), i32([L] * ns)
    pbt = torch.arange(m // 16, dtype=torch.int32, device=dev).view(ns, L // 16)
    pairs = L * (L + 1) // 2 * ns

    def pre(hq, hk, P, od, exact, f32):
        kc, vc = torch.randn(m // 16, hk, 16, P, **bf), torch.randn(m // 16, hk, 16, P, **bf)
        q, out = torch.randn(m, hq, P, **bf), torch.empty(m, hq * od, dtype=torch.float32 if f32 else torch.bfloat16, device=dev)
        return lambda: ops.paged_prefill(q, kc, vc, pbt, ts, tq, qs, ql, ql, out, n_tiles=len(tiles), scale=0.1, out_d=od, exact_p=exact)
    add(f"paged_prefill, two maps [{m} tokens of {L}]", lambda i: pre(nq, att.kv_heads, P, att.vdim, True, True), m * nq * (2 * att.dim + 4 * att.vdim),
        2.0 * pairs * nq * (att.dim + att.vdim))

    def dn(i):
        a, o = torch.randn(m, nq * att.vdim, device=dev), torch.empty(m, att.out_dim, **bf)
        return lambda: hops.diff_norm(a, m, h=att.heads, e=att.vdim, lam=0.4, gain=0.5, eps=1e-5, out=o)
    add(f"diff_norm [{m} rows]", dn, m * (nq * 4 + att.heads * 2) * att.vdim)

    def lg(i):
        c, o = torch.randn(m // 16, 1, 16, cp, **bf), torch.empty(m, cp, **bf)
        return lambda: hops.latent_gather(c, pbt, ql, qs, seq0=0, n_seqs=ns, max_pages=L // 16, out=o)
    add(f"latent_gather [{m} rows]", lg, 4 * m * cp)
    wkv = ops.tile_weight(torch.randn(H * (dk + dv), cp, **bf))

    def kv(i):
        x, o = torch.randn(m, cp, **bf), torch.empty(m, H * (dk + dv), **bf)
        return lambda: ops.gemm(x, wkv, out=o)
    # what the equations need: W_uk and W_uv of every latent
    add(f"keys and values of all heads from latents [{m} rows]", kv, m * 2 * (cp + H * (lat.dim + lat.vdim)), 2.0 * m * H * R * (lat.dim + lat.vdim))

    def pr(i):
        q, x, o = torch.randn(m, H, dk, **bf), torch.randn(m, H * (dk + dv), **bf), torch.empty(m, H * lat.vdim, **bf)
        return lambda: hops.prefill_rows(q, x, ts, tq, qs, ql, ql, qs, o, dk=dk, dv=dv, g=H, n_tiles=len(tiles), scale=0.1, out_d=lat.vdim)
    add(f"prefill_rows [{m} tokens of {L}, {H} heads {lat.dim} + {T}, {lat.vdim}]", pr, m * H * 2 * (2 * (lat.dim + T) + 2 * lat.vdim),
        2.0 * pairs * H * (lat.dim + T + lat.vdim))
    add(f"paged_prefill (Mixtral) [{m} tokens of {L}]", lambda i: pre(Hq, Hk, D, D, False, False), m * Hq * 4 * D, 4.0 * pairs * Hq * D)

    # matrix memory, and retention with states of the same size
    h, N, V = mem.heads, mem.dim, mem.vdim
    WM = mem.in_width
    zw = torch.zeros((2 * h + 63) // 64 * 64, d, **bf)
    kw = dict(h=h, d=N, e=V, z_bias=torch.zeros(2 * h, device=dev), cap=15.0, eps=1e-5, norm_w=torch.ones(h * V, device=dev))

    def md(i):
        proj, hid, o = torch.randn(batch, WM, **bf), torch.randn(batch, d, **bf), torch.empty(batch, h * V, **bf)
        st, sm = torch.zeros(batch, h, N * V + N, device=dev), torch.zeros(batch, h, device=dev)
        sl, ps = torch.arange(batch, dtype=torch.int32, device=dev), i32([100] * batch)
        return lambda: hops.memory_decode(proj, batch, hidden=hid, z_w=zw, state=st, state_m=sm, row_slots=sl, positions=ps, out=o, **kw)
    add(f"memory_decode [{batch} x {h} states of {N} x {V}]", md, batch * (h * (N * V + N) * 8 + 2 * (WM + h * V + d)))
    rh, rv = (h, V) if V <= 256 else (h * V // 256, 256)          # value sizes that retention takes
    pw = hops.decay_powers([0.99] * rh, dev)
    WR = 2 * rh * (N + rv)

    def rd(i):
        proj, st, out = torch.randn(batch, WR, **bf), torch.zeros(batch, rh, N, rv, device=dev), torch.empty(batch, rh * rv, **bf)
        sl, ps = torch.arange(batch, dtype=torch.int32, device=dev), i32([100] * batch)
        return lambda: hops.retention_decode(proj, batch, h=rh, d=N, e=rv, decay_pow=pw, rot=none, k_scale=1.0, eps=1e-5, state=st,
                                             row_slots=sl, positions=ps, out=out)
    add(f"retention_decode [{batch} x {rh} states of {N} x {rv}]", rd, batch * (rh * N * rv * 8 + 2 * (WR + rh * rv)))
    C = hops.memory_chunk()
    for mm, nseq in ((m, ns), (L, 1)):
        tl = len(tiles) * mm // m
        sq = torch.arange(nseq, dtype=torch.int32, device=dev)
        z = torch.randn(mm, zw.shape[0], device=dev)
        ws = torch.empty(hops.memory_ws_elems(h, N, V, tl), device=dev)

        def mp(i):
            proj, o = torch.randn(mm, WM, **bf), torch.empty(mm, h * V, **bf)
            st, sm = torch.zeros(nseq, h, N * V + N, device=dev), torch.zeros(nseq, h, device=dev)
            return lambda: hops.memory_prefill(proj, mm, z=z, state=st, state_m=sm, seq_slots=sq, tile_seq=ts, tile_q0=tq, q_start=qs, q_lens=ql,
                                               ctx_lens=ql, n_tiles=tl, n_seqs=nseq, ws=ws, chunks=True, out=o, **kw)
        work = lambda h, E: mm * h * (4.0 * N * E + (C + 1) * (N + E))
        add(f"memory_prefill [{mm} tokens of {L}, {h} heads {N} x {V}]", mp, mm * h * 2 * (2 * N + 3 * V) + nseq * h * N * V * 8, work(h, V))
        qr_, kr_ = torch.randn(rh, mm, N, device=dev), torch.randn(rh, mm, N, device=dev)
        rws = torch.empty(2 * tl * rh * N * rv, device=dev)
        proj, out = torch.randn(mm, WR, **bf), torch.empty(mm, rh * rv, **bf)

        def rp(i):
            st = torch.zeros(nseq, rh, N, rv, device=dev)
            return lambda: hops.retention_prefill(proj, mm, h=rh, d=N, e=rv, decay_pow=pw, eps=1e-5, state=st, seq_slots=sq, tile_seq=ts,
                                                  tile_q0=tq, q_start=qs, q_lens=ql, ctx_lens=ql, n_tiles=tl, n_seqs=nseq, q_rot=qr_,
                                                  k_rot=kr_, ws=rws, out=out)
        add(f"retention_prefill [{mm} tokens of {L}, {rh} heads {N} x {rv}]", rp, mm * rh * (2 * N * 4 + 3 * rv * 2) + nseq * rh * N * rv * 8,
            work(rh, rv))
    return rows


def run(args, clocks) -> None:
    """`clocks`: bench.py's nvidia-smi sampler."""
    torch.cuda.set_device(0)
    peaks = load_measured_peaks()
    timer = Timer(max(3, args.warmup), max(20, args.steps))
    out = {"bench": "zagolix beside mixtral", "data": "random tokens, random weights",
           "peaks": {k: peaks.get(k) for k in ("hbm_gbs", "bf16_tflops")}, "sizes": {}}
    clocks.start()
    for name in [args.zagolix_size] if args.zagolix_size else list(SIZES):
        zag, mix = _configs(name)
        res = {"zagolix_params_m": round(zag.n_params() / 1e6), "mixtral_params_m": round(mix.n_params() / 1e6), "layers": zag.n_layers,
               "engine": []}
        for batch, prompt in ((1, 2048), (32, 2048), (128, 2048)):
            row = {"batch": batch, "prompt": prompt}
            for key, mc in (("zagolix", zag), ("mixtral", mix)):
                row[key] = engine_numbers(replace(mc), batch=batch, prompt=prompt, warmup=max(3, args.warmup), steps=args.steps)
                torch.cuda.empty_cache()
            res["engine"].append(row)
        res["kernels"] = kernel_numbers(zag, mix, peaks, timer, batch=64, ctx=4096, m=8192)
        out["sizes"][name] = res
        torch.cuda.empty_cache()
    out["clocks"] = clocks.stop()
    print(json.dumps(out), flush=True)
