"""Kernels and serving of Vokepel models on the GPU against the plain implementation: every mechanism alone, then whole models in
32-bit (sharp) and bf16."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import hybrid_models as hm
import hybrid_oracle as plain
import vokepel_models as vm
import vokepel_oracle as oracle
from oxide_tech_llm_engine_b200.sampling_params import SamplingParams
from test_gpu_hybrid import gen, paged, rel
from test_gpu_povatar import b16, i32
from test_gpu_zagolix import chunk, row_errors, toks

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DEV = "cuda"


@pytest.fixture(scope="module")
def H():
    from oxide_tech_llm_engine_b200.ops import hybrid

    return hybrid


@pytest.fixture(autouse=True)
def no_device_error():
    yield
    from oxide_tech_llm_engine_b200 import ops

    torch.cuda.synchronize()
    ops.check_status(torch.device("cuda", 0))


# ---------------------------------------------------------------- residual stream
@pytest.mark.parametrize("dtype,tol", [(torch.float32, 3e-6), (torch.bfloat16, 6e-3)])
@pytest.mark.parametrize("N,rows", [(64, 3), (200, 700), (76, 5), (4096, 300), (4096, 4), (9000, 2), (33, 6)])
def test_stream_that_a_product_replaces_and_operand_rows(H, N, rows, dtype, tol):
    g = gen(N + rows)
    off, eps, bf = (N + 63) // 64 * 64, 1e-3, dtype == torch.bfloat16
    c = lambda t: t.to(DEV)
    emb, tok = torch.randn(40, N, generator=g).to(dtype), torch.randint(0, 40, (rows,), generator=g, dtype=torch.int32)
    x0, y, base, nw = torch.randn(rows, N, generator=g), torch.randn(rows, off, generator=g), torch.randn(N, generator=g), torch.randn(N, generator=g)
    x, acc = c(x0).clone(), c(y).clone()
    parts = 3 if bf else 2
    ent = torch.full((rows, parts * off), 7.0, dtype=dtype, device=DEV)

    def operand(stream):
        """x as the rows have it (two terms in bf16), and what the other columns hold."""
        v = ent.view(rows, parts, off).cpu()
        assert torch.equal(v[:, -1, :N], emb[tok.long()]) and bool((v[:, :, N:] == 7).all())
        if bf:
            assert torch.equal(v[:, 0, :N], stream.to(dtype).cpu())
            return v[:, 0, :N].double() + v[:, 1, :N].double()
        return v[:, 0, :N].double()

    # the embedding itself, then the stream with a branch
    H.branch_norm(x, rows, norm_w=(), h=(), eps=eps, tokens=c(tok), embed=c(emb), branches=[(acc, None, 1.0, False)], split=ent, split_off=off, x0_tokens=c(tok))
    assert torch.equal(operand(emb[tok.long()].float()), emb[tok.long()].double())
    x.copy_(c(x0))
    H.branch_norm(x, rows, norm_w=(), h=(), eps=eps, branches=[(acc, None, 0.3, True)], embed=c(emb), split=ent, split_off=off, x0_tokens=c(tok))
    want = x0.double() + 0.3 * y[:, :N].double()
    assert rel(x, want) < 1e-6 and rel(operand(x), want) < (2e-5 if bf else 1e-6) and float(acc[:, :N].abs().max()) == 0
    # a product's rows and a vector take the place of the stream
    h = torch.zeros(rows, off, dtype=dtype, device=DEV)
    H.branch_norm(x, rows, norm_w=[c(nw)], h=[h], eps=eps, branches=[(c(y), None, 1.0, False)], base=c(base))
    want = y[:, :N].double() + base.double()
    assert rel(x, want) < 1e-6 and rel(h[:, :N], plain.rms(want, eps) * nw) < tol


# ---------------------------------------------------------------- heads whose keys are values
@pytest.mark.parametrize("dtype,proj_dtype,tol", [(torch.float32, torch.float32, 3e-6), (torch.bfloat16, torch.bfloat16, 6e-3),
                                                  (torch.bfloat16, torch.float32, 6e-3)])
@pytest.mark.parametrize("heads,G,D,rows", [(6, 3, 40, 5), (32, 8, 128, 5), (1, 1, 4, 5), (5, 5, 7, 5), (4, 1, 64, 700)])
def test_keys_are_kept_before_their_norm(H, heads, G, D, rows, dtype, proj_dtype, tol):
    g = gen(D + rows)
    W, ld = (heads + G) * D, ((heads + G) * D + 15) // 16 * 16 + 32
    proj = torch.zeros(rows, ld)
    proj[:, :W] = b16(torch.randn(rows, W, generator=g))
    qn, kn = 1 + 0.2 * torch.randn(heads * D, generator=g), 1 + 0.2 * torch.randn(G, D, generator=g)
    P, pages = D + 8, rows // 16 + 3
    kc, kr = torch.zeros(pages, G, 16, P, dtype=dtype, device=DEV), torch.zeros(pages, 16, device=DEV)
    q = torch.zeros(rows, heads * P, dtype=dtype, device=DEV)
    slots = torch.randperm(pages * 16, generator=g)[:rows]
    slots[1] = -1
    wq = qn * kn.repeat_interleave(heads // G, 0).reshape(-1)
    H.heads(proj.to(proj_dtype).to(DEV), rows, h=heads, g=G, d=D, e=D, rot=H.Rotary(None, DEV), positions=i32(list(range(rows))), q_out=q, q_hd=P,
            q_norm=wq.to(DEV), eps=1e-3, k_cache=kc, slots=slots.to(DEV), k_rms=kr)
    p64 = proj.double()
    want = plain.rms(p64[:, :heads * D], 1e-3) * wq
    assert rel(q.view(rows, heads, P)[:, :, :D].reshape(rows, -1), want) < tol and float(q.view(rows, heads, P)[:, :, D:].abs().max()) == 0
    k = p64[:, heads * D:W]
    used = torch.zeros(pages * 16, dtype=torch.bool)
    for t in range(rows):
        s = int(slots[t])
        if s >= 0:
            used[s] = True
            assert torch.equal(kc[s // 16, :, s % 16, :D].cpu().double(), k[t].view(G, D))
            assert abs(float(kr[s // 16, s % 16]) * float(torch.sqrt((k[t] ** 2).mean() + 1e-3)) - 1) < 1e-6
    assert float(kr.view(-1).cpu()[~used].abs().max()) == 0


# ---------------------------------------------------------------- talking heads
class Talk:
    """Random talking heads over T positions; keys are the values times one number per position."""

    def __init__(self, heads, G, D, T, seed, window, cap=8.0, scale=None):
        g = gen(seed)
        self.heads, self.G, self.D, self.T, self.window, self.cap = heads, G, D, T, window, cap
        self.q, self.v = b16(torch.randn(T, heads, D, generator=g)), b16(torch.randn(T, G, D, generator=g))
        self.rms, self.gate = 0.5 + torch.rand(T, generator=g), b16(torch.randn(T, heads * D, generator=g))
        self.talk = b16(0.8 * torch.eye(heads) + 0.5 * torch.randn(heads, heads, generator=g) / heads ** 0.5)
        self.r1, self.r2 = 0.5 + 0.5 * torch.randn(heads, generator=g), 0.3 * torch.rand(heads, generator=g)
        self.scale = 1.5 * D ** -0.5 if scale is None else scale

    def want(self):
        o = oracle
        q, v, r = self.q.double(), self.v.double(), self.rms.double()[:, None, None]
        s = o.raw_scores(q, v * r, self.scale)
        if self.cap:
            s = o.cap(s, self.cap)
        s = o.talk(s - o.distance_bias(self.T, self.r1.double(), self.r2.double()), self.talk.double())
        a = o.values_of(o.masked_softmax(s, self.window or self.T), v)
        return a * o.sigmoid(self.gate.double()).view(self.T, self.heads, self.D)

    def run(self, H, path, mode, lens=None, max_splits=8, gate_f32=False):
        """Every position (or those before `lens`) as a decode row of its own, or the last `mode` positions as one portion. Unused
        places of the cache hold large values."""
        heads, G, D, T = self.heads, self.G, self.D, self.T
        dt = torch.float32 if path == "f32" else torch.bfloat16
        DP = (64 if D <= 64 else 128) if path == "tc" else (D + 7) // 8 * 8
        cache, _, bt = paged(self.v, self.v, DP, DP, dt, T)
        rms = torch.full((cache.shape[0], 16), 3.0)
        rms[bt[torch.arange(T) // 16].long(), torch.arange(T) % 16] = self.rms
        q = torch.zeros(T, heads * DP, dtype=dt, device=DEV)
        q.view(T, heads, DP)[:, :, :D] = self.q.to(DEV)
        far = self.window or 16 * len(bt)
        tk = self.talk.to(DEV)
        kw = dict(h=heads, d=D, window=self.window, scale=self.scale, cap=self.cap, talk=tk, bias=H.talk_bias(tk, self.r1.to(DEV), self.r2.to(DEV), far))
        gate = self.gate.to(torch.float32 if path == "f32" or gate_f32 else dt).to(DEV)
        if mode == "decode":
            at = torch.tensor(range(T) if lens is None else [n - 1 for n in lens])
            n = len(at)
            out = torch.full((n, heads * D), float("nan"), dtype=dt, device=DEV)
            parts = {}
            if path == "tc":
                assert H.talk_decode_ok(heads, G, DP)
                parts = dict(part_o=torch.full((n * heads * max_splits * DP,), float("nan"), device=DEV),
                             part_ml=torch.full((n * heads * max_splits * 2,), float("nan"), device=DEV), max_splits=max_splits)
            H.talk_decode(q[at].contiguous(), cache, rms.to(DEV), bt[None].repeat(n, 1).to(DEV), (at + 1).to(torch.int32).to(DEV), rows=n,
                          gate=gate[at].contiguous(), out=out, **kw, **parts)
            return out.view(n, heads, D)
        tiles, a = chunk(mode, T)
        out = torch.full((mode, heads * D), float("nan"), dtype=dt, device=DEV)
        ws = {}
        if path == "tc":
            assert H.talk_prefill_ok(heads, DP)
            span = H.talk_span(self.window, T)
            ws = dict(scores=torch.full((tiles * heads * 128 * span,), float("nan"), device=DEV), span=span)
        H.talk_prefill(q[T - mode:].contiguous(), cache, rms.to(DEV), bt[None].contiguous().to(DEV), n_tiles=tiles, gate=gate[T - mode:].contiguous(),
                       out=out, **a, **kw, **ws)
        return out.view(mode, heads, D)


TALK_TOL = {"tc": 6e-3, "bf16": 6e-3, "f32": 2e-5}


@pytest.mark.parametrize("path", ["tc", "bf16", "f32"])
@pytest.mark.parametrize("heads,G,D,T,window", [(6, 2, 64, 300, 41), (5, 1, 40, 270, 16), (32, 8, 128, 150, 97), (9, 3, 96, 333, 0), (1, 1, 4, 129, 1),
                                                (16, 16, 64, 200, 130), (24, 3, 20, 140, 33), (17, 1, 128, 130, 64), (2, 2, 128, 700, 500)])
def test_talking_heads(H, path, heads, G, D, T, window):
    t = Talk(heads, G, D, T, T + heads, window)
    want = t.want()
    for mode in ("decode", T, 2, 67, 129):
        if path == "tc" and mode != "decode" and heads > 32:
            continue
        got = t.run(H, path, mode)
        assert rel(got, want if mode == "decode" else want[T - mode:]) < TALK_TOL[path], mode


def test_head_counts_that_only_the_decode_kernel_takes(H):
    for heads, G, D in ((40, 8, 64), (64, 4, 128), (33, 11, 32), (64, 1, 64), (48, 16, 128)):
        t = Talk(heads, G, D, 170, heads, 70)
        assert H.talk_decode_ok(heads, G, 64 if D <= 64 else 128) and not H.talk_prefill_ok(heads, 64)
        want = t.want()
        assert rel(t.run(H, "tc", "decode"), want) < TALK_TOL["tc"]
        assert rel(t.run(H, "bf16", 40), want[130:]) < TALK_TOL["bf16"]


@pytest.mark.parametrize("heads,G,D,window", [(32, 8, 128, 0), (6, 2, 64, 300), (12, 1, 96, 0), (20, 10, 64, 700)])
def test_few_long_sequences_in_many_splits(H, heads, G, D, window):
    t = Talk(heads, G, D, 900, D, window)
    lens = [900, 17, 431, 1, 899, 16]
    want = t.want()[[n - 1 for n in lens]]
    for splits in (1, 3, 16):
        assert rel(t.run(H, "tc", "decode", lens, splits, gate_f32=splits == 3), want) < TALK_TOL["tc"], splits


@pytest.mark.parametrize("path", ["tc", "f32"])
@pytest.mark.parametrize("window", [32, 45, 112, 0])
def test_one_key_that_stands_out_at_every_edge(H, path, window):
    """Every 50th position outweighs all others: rows see it exactly as long as it is in their window, across pages, blocks and
    tiles; without a cap."""
    t = Talk(4, 2, 32, 400, 3, window, cap=0.0)
    t.q[:, :, 0] = 4.0
    t.v[:, :, 0] = -0.5
    t.v[::50, :, 0] = 6.0
    t.talk = b16(torch.eye(4) + 0.1)
    want = t.want()
    for mode in ("decode", 400, 131, 2):
        assert rel(t.run(H, path, mode), want if mode == "decode" else want[400 - mode:]) < TALK_TOL[path], mode


@pytest.mark.parametrize("path", ["tc", "f32"])
@pytest.mark.parametrize("rising", [True, False])
def test_scores_that_grow_or_shrink_by_hundreds(H, path, rising):
    """The reference of the softmax moves again and again (or never after the first page)."""
    t = Talk(10, 2, 64, 350, 5, 0, cap=0.0, scale=1.0)
    ramp = torch.linspace(0, 400, 350)
    t.q[:, :, 0] = 1.0
    t.v[:, :, 0] = b16(ramp if rising else ramp.flip(0))[:, None]
    t.rms[:] = 1.0
    t.talk = b16(torch.eye(10) + 0.02)
    want = t.want()
    for mode in ("decode", 350, 77):
        assert rel(t.run(H, path, mode), want if mode == "decode" else want[350 - mode:]) < 2 * TALK_TOL[path], mode


def test_a_head_that_speaks_for_another(H):
    """A matrix that exchanges heads, one that silences a head (its softmax is then even), and one of large entries."""
    for change in ("exchange", "silence", "large"):
        t = Talk(6, 3, 48, 200, 9, 60)
        t.talk = {"exchange": torch.eye(6)[[3, 4, 5, 0, 1, 2]], "silence": torch.diag(torch.tensor([1.0, 0, 1, 1, 0, 1])), "large": 40 * t.talk}[change]
        if change == "large":
            t.cap = 0.5
        want = t.want()
        for path in ("tc", "f32"):
            assert rel(t.run(H, path, "decode"), want) < TALK_TOL[path] and rel(t.run(H, path, 90), want[110:]) < TALK_TOL[path], (change, path)


def test_ragged_batch_of_prompt_tiles(H):
    """Portions of several sequences with pasts of their own in one launch, against each alone."""
    ts = [Talk(12, 4, 64, n, n, 50) for n in (300, 40, 129, 2)]
    news = [200, 40, 1, 2]
    for t in ts[1:]:
        t.talk, t.r1, t.r2, t.scale = ts[0].talk, ts[0].r1, ts[0].r2, ts[0].scale
    pages = [(t.T + 15) // 16 for t in ts]
    cache, rms = torch.full((sum(pages) + 2, 4, 16, 64), 9.0), torch.full((sum(pages) + 2, 16), 2.0)
    perm, tables, at = torch.randperm(sum(pages) + 2, generator=gen(1)), torch.zeros(4, max(pages), dtype=torch.int32), 0
    for i, t in enumerate(ts):
        tables[i, :pages[i]] = perm[at:at + pages[i]].to(torch.int32)
        at += pages[i]
        for j in range(t.T):
            cache[tables[i, j // 16], :, j % 16], rms[tables[i, j // 16], j % 16] = t.v[j], t.rms[j]
    tile = [(i, 128 * k) for i, n in enumerate(news) for k in range(-(-n // 128))]
    start = np.cumsum([3] + news)          # rows of other requests come first
    M = int(start[-1])
    q, gate, out = (torch.zeros(M, 768, dtype=torch.bfloat16, device=DEV) for _ in range(3))
    for i, (t, n) in enumerate(zip(ts, news)):
        q[start[i]:start[i + 1]] = t.q[t.T - n:].reshape(n, -1).to(DEV).to(torch.bfloat16)
        gate[start[i]:start[i + 1]] = t.gate[t.T - n:].to(DEV).to(torch.bfloat16)
    span, tk = H.talk_span(50, 300), ts[0].talk.to(DEV)
    H.talk_prefill(q, cache.to(torch.bfloat16).to(DEV), rms.to(DEV), tables.to(DEV), i32([x[0] for x in tile]), i32([x[1] for x in tile]),
                   i32(start[:4].tolist()), i32(news), i32([t.T for t in ts]), n_tiles=len(tile), h=12, d=64, window=50, scale=ts[0].scale,
                   cap=8.0, talk=tk, bias=H.talk_bias(tk, ts[0].r1.to(DEV), ts[0].r2.to(DEV), 50), gate=gate, out=out,
                   scores=torch.full((len(tile) * 12 * 128 * span,), float("nan"), device=DEV), span=span)
    assert float(out[:3].abs().max()) == 0
    for i, (t, n) in enumerate(zip(ts, news)):
        assert rel(out[start[i]:start[i + 1]].view(n, 12, 64), t.want()[t.T - n:]) < TALK_TOL["tc"], i


# ---------------------------------------------------------------- sinks
@pytest.mark.parametrize("path", ["tc", "bf16", "f32"])
@pytest.mark.parametrize("heads,G,D,E,window", [(6, 2, 64, 64, 33), (4, 1, 24, 40, 0), (8, 8, 128, 128, 96)])
def test_a_sink_per_head(H, path, heads, G, D, E, window):
    from oxide_tech_llm_engine_b200 import ops

    T, gain = 200, 0.7
    g = gen(heads)
    q, k, v = (b16(torch.randn(T, n, d, generator=g)) for n, d in ((heads, D), (G, D), (G, E)))
    sinks = torch.linspace(-3, 9, heads)        # from nothing to nearly all of the weight
    want = gain * oracle.values_of(oracle.masked_softmax(oracle.raw_scores(q.double(), k.double(), 0.2), window or T, sinks.double()), v.double())
    dt = torch.float32 if path == "f32" else torch.bfloat16
    DP, EP = (64 if max(D, E) <= 64 else 128,) * 2 if path == "tc" else (D, E)
    kc, vc, bt = paged(k, v, DP, EP, dt, T)
    qp = torch.zeros(T, heads, DP, dtype=dt, device=DEV)
    qp[:, :, :D] = q.to(DEV)
    tables, lens = bt[None].repeat(T, 1).contiguous().to(DEV), i32(list(range(1, T + 1)))
    kw, own = dict(window=window, keep_first=0, scale=0.2, sinks=sinks.to(DEV), out_gain=gain), dict(h=heads, d=D, e=E)
    out = torch.zeros(T, heads * E + 8, dtype=dt, device=DEV)[:, :heads * E]       # rows of a wider buffer
    if path == "tc":
        po, pm = torch.empty(T * heads * 4 * DP, device=DEV), torch.empty(T * heads * 4 * 2, device=DEV)
        ops.paged_decode(qp, kc, vc, tables, lens, i32([4]), po, pm, out, batch=T, max_splits=4, out_d=E, exact_p=True, **kw)
    else:
        H.row_attention(qp.view(T, -1), DP, kc, vc, tables, n=T, seq_lens=lens, out=out, **own, **kw)
    assert rel(out.reshape(T, heads, E), want) < TALK_TOL[path]
    n = 150
    tiles, a = chunk(n, T)
    out = torch.zeros(n, heads * E + 8, dtype=dt, device=DEV)[:, :heads * E]
    if path == "tc":
        ops.paged_prefill(qp[T - n:].contiguous(), kc, vc, tables[:1], *a.values(), out, n_tiles=tiles, out_d=E, exact_p=True, **kw)
    else:
        H.row_attention(qp[T - n:].reshape(n, -1), DP, kc, vc, tables[:1], n=tiles, out=out, **own, **kw, **a)
    assert rel(out.reshape(n, heads, E), want[T - n:]) < TALK_TOL[path]


# ---------------------------------------------------------------- gated recurrence
def gru_inputs(N, T, seed, z_mean=-2.0):
    g = gen(seed)
    return b16(torch.randn(T, 3 * N, generator=g)), torch.cat([z_mean + torch.randn(N, generator=g), 0.3 * torch.randn(N, generator=g)])


def gru_want(proj, bias, gain, state=None):
    N = proj.shape[1] // 3
    p, b = proj.double(), bias.double()
    s = oracle.gru(oracle.sigmoid(p[:, :N] + b[:N]), oracle.candidate(p[:, N:2 * N] + b[N:]), state)
    return s * oracle.silu(p[:, 2 * N:]) * gain, s[-1]


@pytest.mark.parametrize("form,tol", [("f32", 2e-6), ("bf16", 5e-3), ("bf16-f32-rows", 5e-3)])
@pytest.mark.parametrize("N,T", [(16, 300), (272, 700), (1040, 260), (8, 33)])
def test_recurrence_in_portions(H, form, tol, N, T):
    proj, bias = gru_inputs(N, T, N)
    want, last = gru_want(proj, bias, 0.6)
    dt = torch.float32 if form == "f32" else torch.bfloat16
    rows = proj.to(torch.bfloat16 if form == "bf16" else torch.float32).to(DEV)
    for cuts in ([T], [2, 1, 1, 130, 31, 1, 64], [1] * 20 + [128]):
        state = torch.full((3, N), 50.0, device=DEV)        # a slot that was used before
        out, at = torch.full((T, N + 8), 3.0, dtype=dt, device=DEV), 0
        ws = torch.full((H.gru_ws_elems(N, T // 128 + 2),), float("nan"), device=DEV)
        cuts = list(cuts)
        while at < T:
            n = min(cuts.pop(0) if cuts else T, T - at)
            kw = dict(bias=bias.to(DEV), gain=0.6, state=state, out=out[at:])
            if n == 1:
                H.gru_decode(rows[at:], 1, row_slots=i32([1]), positions=i32([at]), **kw)
            else:
                tiles, a = chunk(n, at + n)
                H.gru_prefill(rows[at:], n, seq_slots=i32([1]), n_tiles=tiles, ws=ws, **a, **kw)
            at += n
        assert rel(out[:, :N], want) < tol and rel(state[1], last) < (2e-6 if form == "f32" else 2e-5)
        assert bool((out[:, N:] == 3).all()) and bool((state[[0, 2]] == 50).all())


def test_states_that_keep_thousands_of_tokens_stay_sharp(H):
    """Update gates of 1/3000 on average: rounding must not add up over the tokens that a state keeps."""
    N, T = 64, 6000
    proj, bias = gru_inputs(N, T, 1, z_mean=-8.0)
    want, last = gru_want(proj, bias, 1.0)
    for step in (T, 1):
        state, out = torch.zeros(1, N, device=DEV), torch.zeros(T, N, device=DEV)
        kw = dict(bias=bias.to(DEV), gain=1.0, state=state)
        rows = proj.to(DEV)
        if step == T:
            tiles, a = chunk(T, T)
            H.gru_prefill(rows, T, seq_slots=i32([0]), n_tiles=tiles, ws=torch.empty(H.gru_ws_elems(N, tiles), device=DEV), out=out, **a, **kw)
        else:
            slot, pos = i32([0]), torch.arange(T, dtype=torch.int32, device=DEV)
            for t in range(T):
                H.gru_decode(rows[t:], 1, row_slots=slot, positions=pos[t:], out=out[t:], **kw)
        assert rel(out, want) < 3e-6 and rel(state[0], last) < 3e-6


def test_gates_at_their_ends(H):
    """Gates that are shut or open to the last bit, and candidates of both branches."""
    proj = torch.zeros(40, 3 * 8)
    proj[:, :8] = torch.tensor([-200.0, -60, -20, 0, 20, 60, 200, 3])
    proj[:, 8:16] = torch.linspace(-150, 150, 40)[:, None]
    proj[:, 16:] = torch.tensor([100.0, -100, 1, 2, 3, -1, -2, 0])
    want, last = gru_want(proj, torch.zeros(16), 1.0)
    for dt, tol in ((torch.float32, 2e-6), (torch.bfloat16, 6e-3)):
        state, out = torch.zeros(1, 8, device=DEV), torch.zeros(40, 8, dtype=dt, device=DEV)
        tiles, a = chunk(40, 40)
        H.gru_prefill(proj.to(dt).to(DEV), 40, bias=torch.zeros(16, device=DEV), gain=1.0, state=state, seq_slots=i32([0]), n_tiles=tiles,
                      ws=torch.empty(H.gru_ws_elems(8, tiles), device=DEV), out=out, **a)
        w = gru_want(proj.to(dt), torch.zeros(16), 1.0)[0]
        assert bool(torch.isfinite(out).all()) and rel(out, w) < tol
    assert bool(torch.isfinite(last).all())


def test_ragged_batch_of_recurrences(H):
    """Prompts with and without a past beside decode rows and padding rows, slots in any order."""
    N, lens, past = 48, [129, 2, 300, 64], [0, 7, 0, 100]
    ps = [gru_inputs(N, n + k, n)[0] for n, k in zip(lens, past)]
    bias = gru_inputs(N, 4, 9)[1]
    slots, state = [4, 0, 5, 2], torch.full((6, N), 30.0, device=DEV)
    for p, k, s in zip(ps, past, slots):
        if k:
            state[s] = gru_want(p[:k], bias, 1.0)[1].float().to(DEV)
    start = np.cumsum([0] + lens)
    rows = torch.cat([p[k:] for p, k in zip(ps, past)]).to(torch.bfloat16).to(DEV)
    tile = [(i, 128 * j) for i, n in enumerate(lens) for j in range(-(-n // 128))]
    out = torch.zeros(len(rows), N, dtype=torch.bfloat16, device=DEV)
    H.gru_prefill(rows, len(rows), bias=bias.to(DEV), gain=1.0, state=state, seq_slots=i32(slots), tile_seq=i32([t[0] for t in tile]),
                  tile_q0=i32([t[1] for t in tile]), q_start=i32(start[:4].tolist()), q_lens=i32(lens), ctx_lens=i32([n + k for n, k in zip(lens, past)]),
                  n_tiles=len(tile), ws=torch.full((H.gru_ws_elems(N, len(tile)),), float("nan"), device=DEV), out=out)
    nxt = gru_inputs(N, 6, 77)[0]
    o1 = torch.full((6, N), 3.0, dtype=torch.bfloat16, device=DEV)
    H.gru_decode(nxt.to(torch.bfloat16).to(DEV), 6, bias=bias.to(DEV), gain=1.0, state=state, row_slots=i32([2, -1, 4, 0, 1, 5]),
                 positions=i32([164, 5, 129, 9, 0, 300]), out=o1)
    for i, (p, k, s, row) in enumerate(zip(ps, past, slots, (2, 3, 5, 0))):
        want, last = gru_want(torch.cat([p, nxt[row:row + 1]]), bias, 1.0)
        assert rel(out[start[i]:start[i + 1]], want[k:-1]) < 6e-3 and rel(o1[row], want[-1]) < 6e-3 and rel(state[s], last) < 2e-5, i
    assert bool((o1[1] == 3).all()) and bool((state[3] == 30).all())
    assert rel(o1[4], gru_want(nxt[4:5], bias, 1.0)[0][0]) < 6e-3          # a first token: the slot's old state does not count


# ---------------------------------------------------------------- feed-forward and logits
@pytest.mark.parametrize("M", [1, 2, 5, 129, 300])
def test_squared_relu_of_a_dense_product(M):
    from oxide_tech_llm_engine_b200 import ops

    g = gen(M)
    x, w = torch.randn(M, 192, generator=g).to(torch.bfloat16), (torch.randn(320, 192, generator=g) * 192 ** -0.5).to(torch.bfloat16)
    want = torch.relu(x.double() @ w.double().T).square()
    out = torch.zeros(M, 320, dtype=torch.bfloat16, device=DEV)
    ops.gemm(x.to(DEV), w.to(DEV), out=out, act=2)
    assert rel(out, want) < 5e-3
    if M <= 8:
        out.zero_()
        ops.gemv(x.to(DEV), w.to(DEV), out, act=2)
        assert rel(out, want) < 5e-3


def test_squared_relu_in_32_bit(H):
    u = torch.randn(7, 36, generator=gen(1))
    out = torch.zeros(7, 40, device=DEV)
    H.glu_f32(u.to(DEV), out, 7, 36, 2)
    assert rel(out[:, :36], torch.relu(u.double()).square()) < 1e-6 and float(out[:, 36:].abs().max()) == 0


# ---------------------------------------------------------------- whole models
def rounding(c, w, t, draws=4):
    """How far 16-bit storage of what enters the products moves each row of logits: the plain implementation with relative noise
    of that size on the normed rows, queries, keys, values, read-outs and activations; the largest of a few draws."""
    names = ("rms", "raw_scores", "values_of", "gru", "candidate", "silu", "sigmoid", "feed_forward")
    kept, want, worst = {n: getattr(oracle, n) for n in names}, oracle.forward(c, w, t).numpy(), 0.0
    for seed in range(draws):
        g = gen(seed)
        noisy = lambda x: x * (1 + 2.0 ** -9 * (2 * torch.rand(x.shape, generator=g, dtype=x.dtype) - 1))
        try:
            oracle.rms = lambda x, eps: noisy(kept["rms"](noisy(x), eps))
            oracle.raw_scores = lambda q, k, s: kept["raw_scores"](noisy(q), noisy(k), s)
            oracle.values_of = lambda p, v: noisy(kept["values_of"](p, noisy(v)))
            oracle.gru = lambda z, x, s=None: noisy(kept["gru"](z, x, s))
            oracle.candidate, oracle.silu = lambda u: kept["candidate"](noisy(u)), lambda z: noisy(kept["silu"](noisy(z)))
            oracle.sigmoid = lambda z: kept["sigmoid"](noisy(z))
            oracle.feed_forward = lambda z, p, h: noisy(torch.relu(h @ z[p + "up"].T).square()) @ z[p + "down"].T
            worst = np.maximum(worst, row_errors(oracle.forward(c, w, t).numpy(), want))
        finally:
            for n in names:
                setattr(oracle, n, kept[n])
    return want, worst


class Expected:
    """Logits of the plain implementation and what rounding allows each row."""

    def __init__(self, c, w, tokens, dtype):
        self.dtype = dtype
        if dtype == "float32":
            self.want = oracle.forward(c, w, tokens).numpy()
        else:
            self.want, self.noise = rounding(c, w, tokens)

    def wrong(self, got, at=slice(None)):
        """Rows outside their limits, with their errors."""
        e = row_errors(got, self.want[at])
        limit = 1e-4 if self.dtype == "float32" else 0.008 + 4 * self.noise[at]
        return [(i, float(e[i])) for i in np.flatnonzero(e > limit)]


@pytest.mark.parametrize("name", list(vm.CONFIGS))
def test_prompts_portions_and_batches_equal_the_plain_implementation(name):
    c = vm.CONFIGS[name]
    w = vm.weights(c, 2)
    eng = hm.engine(c, w, dtype="float32", live=3, blocks=56)
    seqs = [toks(n, c["vocab"], n) for n in (1, 45, 150, 2, 97, 290, 33, 128)]
    want = [Expected(c, w, t, "float32") for t in seqs]
    for t, x in zip(seqs, want):
        assert not x.wrong(hm.feed_all(eng, 0, t, []))
        assert not x.wrong(hm.feed_all(eng, 0, t, [2, 3, 1, 1, 17, 2, 64]))
    for seed in (1, 2):
        for got, x in zip(hm.interleaved(eng, seqs, seed), want):
            assert not x.wrong(got)
    assert eng.sched.num_free_blocks() == 56
    eng.close()


@pytest.mark.parametrize("name", list(vm.CONFIGS))
def test_bf16_prompts_portions_and_batches(name):
    c = vm.CONFIGS[name]
    w = vm.weights(c, 3)
    eng = hm.engine(c, w, live=3, blocks=64)
    t = toks(330, c["vocab"], 7)
    x = Expected(c, w, t, "bfloat16")
    assert np.median(x.noise) < 0.03
    for n, cuts in ((330, []), (330, [2, 3, 1, 1, 17, 2, 64, 100]), (300, [40] + [1] * 260), (129, [128])):
        assert not x.wrong(hm.feed_all(eng, 0, t[:n], cuts), slice(0, n)), (n, cuts)
    lens = [200, 3, 77, 129, 64, 1]
    for got, n in zip(hm.interleaved(eng, [t[:n] for n in lens], 5), lens):
        assert not x.wrong(got, slice(0, n))
    eng.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding_token_by_token(dtype):
    c = vm.CONFIGS["mixed"]
    w = vm.weights(c, 2)
    eng = hm.engine(c, w, dtype=dtype, live=2, blocks=48)
    t = toks(300, c["vocab"], 5)
    assert not Expected(c, w, t, dtype).wrong(hm.feed_all(eng, 0, t, [1] * 300))
    assert eng.stats["graph_replays"] > 250
    eng.close()


def test_prompt_tiles_in_several_passes(monkeypatch):
    from oxide_tech_llm_engine_b200.models import hybrid

    monkeypatch.setattr(hybrid, "TALK_SCORE_BYTES", 1)
    c = vm.CONFIGS["talk"]
    w = vm.weights(c, 5)
    eng = hm.engine(c, w, live=4, blocks=96)
    seqs = [toks(n, c["vocab"], n) for n in (150, 40, 33, 290)]
    cut = (100, 20, 30, 2)
    first = eng.feed([(i, t[:n], [n - 1]) for i, (t, n) in enumerate(zip(seqs, cut))])
    rest = eng.feed([(i, t[n:], [len(t) - n - 1]) for i, (t, n) in enumerate(zip(seqs, cut))])
    for i, (t, n) in enumerate(zip(seqs, cut)):
        x = Expected(c, w, t, "bfloat16")
        assert not x.wrong(first[i:i + 1], [n - 1]) and not x.wrong(rest[i:i + 1], [len(t) - 1])
    eng.close()


@pytest.mark.parametrize("name", ["mixed", "pair"])
def test_layer_outputs_follow_every_layer_run(name):
    c = vm.CONFIGS[name]
    w = vm.weights(c, 2)
    eng = hm.engine(c, w, dtype="float32")
    t = toks(37, c["vocab"], 8)
    seen = {}
    eng.model.layer_hook = lambda i, x: seen.__setitem__(i, x.cpu().clone())
    eng.feed([(0, t, [])])
    _, want = oracle.forward(c, w, t, want_layers=True)
    assert sorted(seen) == list(range(len(want)))
    for i, x in enumerate(want):
        assert rel(seen[i], x) < 2e-5
    eng.close()


@pytest.mark.parametrize("burst", [0, 6])
@pytest.mark.parametrize("name", ["mixed", "ones", "talk"])
def test_greedy_generation_through_the_engine(name, burst):
    """32-bit, so that the tokens are the plain implementation's: chunked prompts, a pool and slots that are short, graph
    replays, decode bursts."""
    c = vm.CONFIGS[name]
    w = vm.weights(c, 4)
    eng = hm.engine(c, w, dtype="float32", live=3, blocks=14, tokens=40, chunk_min=4, chunk_max=32, sla_budget=False, decode_burst=burst)
    prompts = [toks(n, c["vocab"], 70 + n) for n in (3, 60, 41, 17, 1)]
    if burst:
        prompts = prompts[2:]
    outs = eng.generate(prompts, SamplingParams(greedy=True, max_tokens=30, ignore_eos=True))
    for p, o in zip(prompts, outs):
        lg = oracle.forward(c, w, p + o[:-1]).numpy()[len(p) - 1:]
        assert len(o) == 30 and (lg.max(-1) - lg[np.arange(30), o]).max() < 1e-3 * lg.std()
    assert eng.stats["graph_replays"] > 0 and (not burst or eng.stats.get("burst_steps", 0) > 0)
    assert eng.sched.num_free_blocks() == 14
    eng.close()


def test_sampling_in_bf16_and_the_server_facing_entry_point():
    c = vm.CONFIGS["mixed"]
    w = vm.weights(c, 4)
    eng = hm.engine(c, w, live=3, blocks=40, tokens=64, speculative="ngram", chunk_max=64)
    assert eng._drafter is None              # a state cannot be cut back
    prompts = [toks(n, c["vocab"], n) for n in (20, 33, 150)]
    outs = eng.generate(prompts, SamplingParams(greedy=True, max_tokens=20, ignore_eos=True))
    for p, o in zip(prompts, outs):
        lg = oracle.forward(c, w, p + o[:-1]).numpy()[len(p) - 1:]
        assert (lg.max(-1) - lg[np.arange(20), o]).max() < 0.2 * lg.std()
    s = eng.generate(prompts, SamplingParams(temperature=0.8, top_k=20, top_p=0.9, seed=1, max_tokens=8, ignore_eos=True))
    assert all(len(x) == 8 and 0 <= min(x) and max(x) < c["vocab"] for x in s)
    eng.close()


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_trace_replay_program(tmp_path, dtype):
    c = vm.CONFIGS["mixed"]
    w = vm.weights(c, 6)
    hm.write_model(tmp_path / "m", c, w)
    t = toks(170, c["vocab"], 3)
    want = Expected(c, w, t, dtype)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": t[:150], "want": [0, 149]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": t[150:151], "want": []}, {"id": "b", "tokens": t[:2], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "b", "tokens": t[2:40], "want": [37]}, {"id": "a", "tokens": t[151:], "want": [18]}],
              "end": ["a", "b"]},
             {"step": 3, "entries": [{"id": "a", "tokens": t[:20], "want": [19]}], "end": ["a"]}]
    r = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path / "m"), "--dtype", dtype, "--out",
                        str(tmp_path / "out"), "--max-tokens", "256"], input="".join(json.dumps(s) + "\n" for s in steps), text=True,
                       capture_output=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    read = lambda n: np.fromfile(tmp_path / "out" / f"{n}.f32", dtype="<f4").reshape(-1, c["vocab"])
    assert not want.wrong(read(0), [0, 149]) and not (tmp_path / "out" / "1.f32").exists()
    assert not want.wrong(read(2), [39, 169]) and not want.wrong(read(3), [19])
