"""Layer-list decoders (Kipolix) beside the Llama-family model of equal size: prompt and decode throughput
through the engine, and every kernel of the new design against its roofline next to the like kernel.

    python bench.py --kipolix [--steps K --warmup W]

Each size is a few layers of a real model's shape with random weights: attention and retention layers
alternate, the Llama model has the same width, FFN, heads and layer count. Engine numbers are CUDA-event
times of whole `LLMEngine.step()` calls. Kernel times are CUDA events over calls that rotate through
buffers larger than L2; a kernel's roofline is its algorithmic bytes at the measured copy bandwidth, or
its arithmetic at the measured bf16 rate where that takes longer.
"""
from __future__ import annotations

import json
import os
from dataclasses import replace

import numpy as np
import torch

SIZES = {
    # the layers of llama3-8b; heads of 64 at a 1B width; heads of 96 (padded to the 128-wide kernels)
    "w4096-h128": dict(width=4096, ff=14336, heads=32, kv_heads=8, dim=128, r_heads=32, r_dim=128, r_vdim=128, window=4096),
    "w2048-h64": dict(width=2048, ff=8192, heads=32, kv_heads=8, dim=64, r_heads=16, r_dim=64, r_vdim=128, window=1024),
    "w3072-h96": dict(width=3072, ff=8192, heads=32, kv_heads=32, dim=96, r_heads=12, r_dim=128, r_vdim=256, window=2048),
}
VOCAB = 32000


def _configs(name: str, layers: int):
    from .models.config import ModelConfig, _kipolix_preset

    z = SIZES[name]
    kip = _kipolix_preset("kipolix-" + name, vocab=VOCAB, pattern="ar" * (layers // 2), keep_first=16, streams=2, buckets=30011, **z)
    hd = z["dim"] if z["dim"] in (64, 128) else 128
    heads = z["heads"] if hd == z["dim"] else z["heads"] * z["dim"] // hd       # head sizes the Llama kernels take
    kv = max(1, min(z["kv_heads"], heads))
    lla = ModelConfig(name="llama-" + name, n_layers=layers, d_model=z["width"], n_heads=heads, n_kv_heads=kv, head_dim=hd,
                      ffn_dim=z["ff"], vocab_size=VOCAB, max_ctx=1 << 17)
    return kip, lla


def _engine(mc, batch: int, prompt: int, steps: int, chunk: int):
    from .config import EngineConfig
    from .engine.engine import LLMEngine

    ctx = (prompt + steps + 64 + 15) // 16 * 16
    cfg = EngineConfig(model=mc.name, ctx_size=ctx, max_num_seqs=batch, max_num_batched_tokens=chunk, sla_budget=False,
                       chunk_max=chunk, enable_radix=False, graph_buckets=(batch,), num_kv_blocks=batch * ctx // 16 + 16)
    return LLMEngine(cfg, mc, random_init=True)


def _time_steps(eng, n: int) -> float:
    """Milliseconds per engine step by CUDA events."""
    a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    torch.cuda.synchronize()
    a.record()
    for _ in range(n):
        eng.step()
    b.record()
    torch.cuda.synchronize()
    return a.elapsed_time(b) / n


def engine_numbers(mc, *, batch: int, prompt: int, warmup: int, steps: int) -> dict:
    from .sampling_params import SamplingParams

    chunk = 8192
    budget = warmup + steps + 16 + batch * prompt // chunk      # early requests decode while others prefill
    eng = _engine(mc, batch, prompt, budget, chunk)
    rng = np.random.default_rng(0)
    sp = SamplingParams(greedy=True, max_tokens=budget, ignore_eos=True)

    def submit():
        for _ in range(batch):
            eng.add_request(rng.integers(0, mc.vocab_size, size=prompt).tolist(), sp)

    submit()                                # first pass: lazy initialisation, buffers
    for _ in range(3):
        eng.step()
    for r in list(eng.requests):
        eng.cancel(r)
        eng.requests.pop(r)
    submit()
    full = batch * prompt // chunk          # steps made of whole chunks of prompt tokens
    n_pre = max(1, min(full, 8))
    t_pre = _time_steps(eng, n_pre)
    while True:                             # until every request decodes
        before = eng.stats["prefill_tokens"]
        eng.step()
        if eng.stats["prefill_tokens"] == before:
            break
    for _ in range(warmup):
        eng.step()
    t_dec = _time_steps(eng, steps)
    eng.check_device_status()
    eng.close()
    pre = min(chunk, batch * prompt) / t_pre * 1e3
    return {"prefill_tok_s": round(pre), "prefill_ms_per_step": round(t_pre, 3), "decode_tok_s": round(batch / t_dec * 1e3),
            "decode_ms_per_step": round(t_dec, 4)}


# ------------------------------------------------------------------------------------------ kernels
class Timer:
    def __init__(self, warmup: int, steps: int):
        self.warmup, self.steps = warmup, steps

    def __call__(self, calls: list) -> float:
        """Microseconds per call; `calls` run round robin over buffers that together exceed L2."""
        for i in range(max(self.warmup, len(calls))):
            calls[i % len(calls)]()
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        torch.cuda.synchronize()
        a.record()
        for i in range(self.steps):
            calls[i % len(calls)]()
        b.record()
        torch.cuda.synchronize()
        return a.elapsed_time(b) / self.steps * 1e3


def _copies(bytes_per_call: float) -> int:
    return int(min(64, max(1, -(-300e6 // max(1.0, bytes_per_call)))))


def kernel_numbers(kip, lla, peaks: dict, timer: Timer, batch: int, ctx: int, m: int) -> list:
    """One row per kernel: [name, what it is compared with, us, roofline us, fraction of roofline]."""
    from . import ops
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

    d = kip.d_model
    att = next(L.mixer for L in kip.layers if L.mixer.kind == "attention")
    ret = next(L.mixer for L in kip.layers if L.mixer.kind == "retention")
    S = kip.streams
    for M in (batch, m):
        tag = f"[{M} rows]"
        nb = M * d * (8 * S + 8 + 2)
        w = torch.zeros(d, device=dev)
        one, mix = torch.ones(S, device=dev), torch.eye(S, device=dev)

        def sn(i, M=M):
            x, y, h = torch.randn(M, S, d, device=dev), torch.randn(M, d, device=dev), torch.empty(M, d, **bf)
            return lambda: hops.stream_norm(x, M, norm_w=w, eps=1e-5, h=h, y=y, mix=mix, out_w=one, in_w=one)
        add("stream_norm " + tag, sn, nb)
        wb = torch.ones(d, **bf)

        def fn(i, M=M):
            acc, res, out = torch.randn(M, d, device=dev), torch.zeros(M, d, **bf), torch.empty(M, d, **bf)
            return lambda: ops.finalize_norm(rows=M, n=d, acc=acc, residual_in=res, residual_out=res, norm_w=wb,
                                             out_ptrs=[out.data_ptr()], device=dev)
        add("finalize_norm (Llama) " + tag, fn, M * d * (8 + 4 + 2))

        pages = M // 16 + 1
        P = 64 if max(att.dim, att.vdim) <= 64 else 128
        W = att.heads * att.dim + att.kv_heads * (att.dim + att.vdim)
        rot = hops.Rotary(att.rot, dev)
        qn, kn = torch.ones(att.heads * att.dim, device=dev), torch.ones(att.kv_heads * att.dim, device=dev)
        pos, slots = torch.arange(M, dtype=torch.int32, device=dev), torch.arange(M, device=dev)

        def hd(i, M=M):
            proj, q = torch.randn(M, W, **bf), torch.empty(M, att.heads * P, **bf)
            kc, vc = torch.zeros(pages, att.kv_heads, 16, P, **bf), torch.zeros(pages, att.kv_heads, 16, P, **bf)
            return lambda: hops.heads(proj, M, h=att.heads, g=att.kv_heads, d=att.dim, e=att.vdim, rot=rot, positions=pos, q_out=q,
                                      q_hd=P, q_norm=qn, k_norm=kn, k_cache=kc, v_cache=vc, slots=slots)
        add("heads " + tag, hd, 4 * M * W)
        D, Hq, Hk = lla.head_dim, lla.n_heads, lla.n_kv_heads
        inv = torch.ones(D // 2, device=dev)

        def qr(i, M=M):
            proj, q = torch.randn(M, (Hq + 2 * Hk) * D, **bf), torch.empty(M, Hq * D, **bf)
            kc, vc = torch.zeros(pages, Hk, 16, D, **bf), torch.zeros(pages, Hk, 16, D, **bf)
            return lambda: ops.qkv_rope_append(qkv_bf16=proj, positions=pos, slot_mapping=slots, inv_freq=inv, q_out=q, k_cache=kc,
                                               v_cache=vc, m=M, hq=Hq, hkv=Hk, d=D)
        add("qkv_rope_append (Llama) " + tag, qr, 4 * M * (Hq + 2 * Hk) * D)

    # decode attention: `batch` sequences of `ctx` tokens, and the windowed form of the new design
    nb_seq = ctx // 16
    vis = min(ctx, att.window + 16) if att.window else ctx
    splits = 16

    def dec(hq, hk, D, P, window, keep, exact, real):
        kc, vc = torch.zeros(batch * nb_seq, hk, 16, P, **bf), torch.zeros(batch * nb_seq, hk, 16, P, **bf)
        bt = torch.randperm(batch * nb_seq, device=dev).to(torch.int32).view(batch, nb_seq)
        q = torch.randn(batch, hq, P, **bf)
        out = torch.empty(batch, hq * D, **bf)
        po, pm = torch.empty(batch * hq * splits * P, device=dev), torch.empty(batch * hq * splits * 2, device=dev)
        per_sm = 12 if hk >= 4 else 4
        want = max(1, min(splits, -(-per_sm * 148 // (batch * hk))))
        pps = i32([(max(4, -(-nb_seq // want)) + 3) // 4 * 4])
        lens = i32([ctx] * batch)
        return lambda: ops.paged_decode(q, kc, vc, bt, lens, pps, po, pm, out, batch=batch, max_splits=splits, window=window,
                                        keep_first=keep, scale=0.1, out_d=D if real else 0, exact_p=exact)
    P = 64 if max(att.dim, att.vdim) <= 64 else 128
    add(f"paged_decode, window + kept first [{batch} x {vis} keys]",
        lambda i: dec(att.heads, att.kv_heads, att.vdim, P, att.window, att.keep_first, True, True),
        batch * vis * att.kv_heads * (att.dim + att.vdim) * 2)
    add(f"paged_decode (Llama) [{batch} x {ctx} keys]",
        lambda i: dec(lla.n_heads, lla.n_kv_heads, lla.head_dim, lla.head_dim, 0, 0, False, False),
        batch * ctx * lla.n_kv_heads * lla.head_dim * 4)

    # prompt attention: m tokens in sequences of 2048
    L = 2048
    ns = m // L
    tiles = [(s, t * 128) for s in range(ns) for t in range(L // 128)]
    ts, tq = i32([t[0] for t in tiles]), i32([t[1] for t in tiles])
    qs, ql = i32([s * L for s in range(ns)]), i32([L] * ns)

    def pre(hq, hk, D, P, window, keep, exact, real):
        kc, vc = torch.randn(m // 16, hk, 16, P, **bf), torch.randn(m // 16, hk, 16, P, **bf)
        bt = torch.arange(m // 16, dtype=torch.int32, device=dev).view(ns, L // 16)
        q, out = torch.randn(m, hq, P, **bf), torch.empty(m, hq * D, **bf)
        return lambda: ops.paged_prefill(q, kc, vc, bt, ts, tq, qs, ql, ql, out, n_tiles=len(tiles), window=window, keep_first=keep,
                                         scale=0.1, out_d=D if real else 0, exact_p=exact)
    win = att.window or L
    pairs = sum(min(i + 1, win + min(att.keep_first, max(0, i + 1 - win))) for i in range(L)) * ns
    add(f"paged_prefill, window + kept first [{m} tokens of {L}]",
        lambda i: pre(att.heads, att.kv_heads, att.vdim, P, att.window, att.keep_first, True, True),
        m * att.heads * 4 * att.dim, 2.0 * pairs * att.heads * (att.dim + att.vdim))
    add(f"paged_prefill (Llama) [{m} tokens of {L}]",
        lambda i: pre(lla.n_heads, lla.n_kv_heads, lla.head_dim, lla.head_dim, 0, 0, False, False),
        m * lla.n_heads * 4 * lla.head_dim, 4.0 * (L * (L + 1) // 2 * ns) * lla.n_heads * lla.head_dim)

    # retention: the state stream of a decode step, the chunks of a prompt step
    h, D, E = ret.heads, ret.dim, ret.vdim
    pw = hops.decay_powers(ret.decay, dev)
    rrot = hops.Rotary(ret.rot, dev)
    WR = 2 * h * (D + E)

    def rd(i):
        proj, st, out = torch.randn(batch, WR, **bf), torch.zeros(batch, h, D, E, device=dev), torch.empty(batch, h * E, **bf)
        sl, ps = torch.arange(batch, dtype=torch.int32, device=dev), i32([100] * batch)
        return lambda: hops.retention_decode(proj, batch, h=h, d=D, e=E, decay_pow=pw, rot=rrot, k_scale=D ** -0.5, eps=1e-5, state=st,
                                             row_slots=sl, positions=ps, out=out)
    add(f"retention_decode [{batch} x {h} states of {D} x {E}]", rd, batch * (h * D * E * 8 + 2 * (WR + h * E)))
    C = hops.retention_chunk()
    qr_, kr_ = torch.randn(h, m, D, device=dev), torch.randn(h, m, D, device=dev)
    ws = torch.empty(2 * len(tiles) * h * D * E, device=dev)
    sl = torch.arange(ns, dtype=torch.int32, device=dev)
    proj = torch.randn(m, WR, **bf)
    pos = torch.arange(m, dtype=torch.int32, device=dev)

    def rh(i):
        return lambda: hops.heads(proj, m, h=h, g=h, d=D, e=E, rot=rrot, positions=pos, q_out=qr_, q_hd=D, k_out=kr_, k_scale=0.1)
    add(f"heads, dense fp32 q and k [{m} rows]", rh, m * 2 * h * D * 6)

    def rp(i):
        st, out = torch.zeros(ns, h, D, E, device=dev), torch.empty(m, h * E, **bf)
        return lambda: hops.retention_prefill(proj, m, h=h, d=D, e=E, decay_pow=pw, eps=1e-5, state=st, seq_slots=sl, tile_seq=ts,
                                              tile_q0=tq, q_start=qs, q_lens=ql, ctx_lens=ql, n_tiles=len(tiles), n_seqs=ns,
                                              q_rot=qr_, k_rot=kr_, ws=ws, out=out)
    n_ch = m // C
    # bytes of the chunked form: q, k, v, gate in, o out, chunk states written, scanned (read + write) and read
    nbytes = m * h * (2 * D * 4 + 3 * E * 2) + 4.0 * n_ch * h * D * E * 4
    flops = m * h * (4.0 * D * E + 2.0 * (C + 1) / 2 * (D + E))
    add(f"retention_prefill [{m} tokens of {L}, {h} heads {D} x {E}]", rp, nbytes, flops)
    return rows


def run(args, clocks) -> None:
    """`clocks`: bench.py's nvidia-smi sampler."""
    from .utils.roofline import load_measured_peaks

    torch.cuda.set_device(0)
    try:
        peaks = json.load(open(os.path.join(os.path.dirname(os.path.dirname(os.path.abspath(__file__))), "MEASURED_PEAKS.json")))
    except OSError:
        peaks = load_measured_peaks()
    timer = Timer(max(3, args.warmup), max(20, args.steps))
    out = {"bench": "kipolix beside llama", "layers": args.layers or 8, "data": "random tokens, random weights", "peaks": {
        k: peaks.get(k) for k in ("hbm_gbs", "bf16_tflops")}, "sizes": {}}
    clocks.start()
    names = [args.kipolix_size] if args.kipolix_size else list(SIZES)
    for name in names:
        kip, lla = _configs(name, out["layers"])
        res = {"kipolix_params_m": round(kip.n_params() / 1e6), "llama_params_m": round(lla.n_params() / 1e6), "engine": []}
        for batch, prompt in ((1, 2048), (32, 2048), (128, 2048)):
            row = {"batch": batch, "prompt": prompt}
            for key, mc in (("kipolix", kip), ("llama", lla)):
                row[key] = engine_numbers(replace(mc), batch=batch, prompt=prompt, warmup=max(3, args.warmup), steps=args.steps)
                torch.cuda.empty_cache()
            res["engine"].append(row)
        res["kernels"] = kernel_numbers(kip, lla, peaks, timer, batch=64, ctx=4096, m=8192)
        out["sizes"][name] = res
        torch.cuda.empty_cache()
    out["clocks"] = clocks.stop()
    print(json.dumps(out), flush=True)
