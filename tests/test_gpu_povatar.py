"""Kernels and serving of Povatar models on the GPU against the plain implementation: every mechanism alone, then whole
models in 32-bit (sharp) and bf16."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import hybrid_models as hm
import hybrid_oracle as plain
import povatar_models as pm
import povatar_oracle as oracle
from oxide_tech_llm_engine_b200.sampling_params import SamplingParams
from test_gpu_hybrid import gen, rel, run_attention

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


def b16(t):
    return t.to(torch.bfloat16).float()


def i32(x):
    return torch.tensor(x, dtype=torch.int32, device=DEV)


# ---------------------------------------------------------------- residual branches and norms
@pytest.mark.parametrize("dtype,tol", [(torch.float32, 3e-6), (torch.bfloat16, 6e-3)])
@pytest.mark.parametrize("N,rows,top", [(64, 3, 2), (200, 700, 3), (76, 5, 1), (2048, 330, 8), (4096, 4, 4), (3072, 400, 2), (8192, 3, 5),
                                        (9000, 2, 3), (130, 9, 0)])
def test_branch_norm(H, N, rows, top, dtype, tol):
    g = gen(N + rows)
    vocab, ld, eps = 50, (N + 63) // 64 * 64, 1e-3
    c = lambda t: t.to(DEV)
    emb = torch.randn(vocab, N, generator=g).to(dtype)
    tok = torch.randint(0, vocab, (rows,), generator=g, dtype=torch.int32)
    n1, n2, wa, wb = (1 + 0.3 * torch.randn(N, generator=g) for _ in range(4))
    x = torch.full((rows, N), float("nan"), device=DEV)
    h, h2 = (torch.zeros(rows, ld, dtype=dtype, device=DEV) for _ in range(2))
    ys = [torch.full((rows, ld), 7.0, device=DEV) for _ in range(2)]
    acc = torch.ones(rows, 12, device=DEV)
    H.branch_norm(x, rows, norm_w=[c(n1), c(n2)], h=[h, h2], eps=eps, tokens=c(tok), embed=c(emb), embed_scale=11.5, clear=acc,
                  branches=[(ys[0], c(wa), 0.5, True), (ys[1], c(wb), 0.5, False)])
    xs = emb[tok.long()].double() * 11.5
    assert rel(x, xs) < 1e-6 and rel(h[:, :N], plain.rms(xs, eps) * n1) < tol and rel(h2[:, :N], plain.rms(xs, eps) * n2) < tol
    assert float(acc.abs().max()) == 0 and float(ys[0][:, :N].abs().max()) == 0 and bool((ys[1] == 7).all())
    assert ld == N or float(h[:, N:].abs().max()) == 0
    # the sum of a layer: both branches by their norms, one plain with its gain, and the chosen rows (one of them missing)
    a, b = torch.randn(rows, N, generator=g), 3 * torch.randn(rows, N, generator=g)
    ys[0][:, :N], ys[1][:, :N] = c(a), c(b)
    er = torch.randn(rows * top + 5, ld, generator=g).to(dtype)
    slot = torch.randperm(rows * top + 5, generator=g)[:rows * top].to(torch.int32)
    wt = torch.rand(rows * top, generator=g)
    if top > 1:
        slot[1] = -1
    ex = (c(er), c(slot), c(wt), top) if top else None
    H.branch_norm(x, rows, norm_w=[c(n2), c(n1)], h=[h, h2], eps=eps, branches=[(ys[0], c(wa), 0.5, True), (ys[1], None, 0.25, False)],
                  experts=ex)
    e = torch.zeros(rows, N, dtype=torch.float64)
    for i in range(rows * top):
        if slot[i] >= 0:
            e[i // top] += wt[i].double() * er[slot[i], :N].double()
    xs = xs + 0.5 * plain.rms(a.double(), eps) * wa + 0.25 * b.double() + e
    assert rel(x, xs) < 3e-6 and rel(h[:, :N], plain.rms(xs, eps) * n2) < tol and rel(h2[:, :N], plain.rms(xs, eps) * n1) < tol
    assert float(ys[0][:, :N].abs().max()) == 0 and rel(ys[1][:, :N], b) == 0
    # the last one: only the mapped rows, x stays
    rmap = torch.full((rows,), -1, dtype=torch.int32)
    rmap[rows - 1] = 0
    before, out = x.clone(), torch.zeros(1, ld, dtype=dtype, device=DEV)
    H.branch_norm(x, rows, norm_w=[c(n1)], h=[out], eps=eps, branches=[(ys[1], c(wb), 2.0, False)], row_map=c(rmap), store_x=False)
    xs = xs + 2.0 * plain.rms(b.double(), eps) * wb
    assert torch.equal(x, before) and rel(out[0, :N], plain.rms(xs, eps)[-1] * n1) < tol


# ---------------------------------------------------------------- scaled rotation
@pytest.mark.parametrize("dtype,tol", [(torch.float32, 3e-6), (torch.bfloat16, 4e-3)])
@pytest.mark.parametrize("D,dims,base,sc", [(64, 16, 20000.0, (5.0, 512, 16.0, 1.0)), (40, 24, 300.0, (8.0, 64, 3.0, 0.5)), (128, 128, 1e6, (40.0, 4096, 32.0, 1.0)),
                                            (33, 6, 100.0, None)])
def test_scaled_rotation_of_the_half_layout(H, D, dims, base, sc, dtype, tol):
    from oxide_tech_llm_engine_b200.models.layer_spec import RotarySpec, YarnSpec

    g = gen(D)
    T, heads, G, E = 6, 3, 1, 32
    proj = b16(torch.randn(T, heads * D + G * (D + E), generator=g))
    pos = torch.tensor([0, 1, 63, 777, 30011, 262143], dtype=torch.int32)
    kc, vc = torch.zeros(1, G, 16, D, dtype=dtype, device=DEV), torch.zeros(1, G, 16, E, dtype=dtype, device=DEV)
    q = torch.zeros(T, heads * D, dtype=dtype, device=DEV)
    H.heads(proj.to(dtype).to(DEV), T, h=heads, g=G, d=D, e=E, rot=H.Rotary(RotarySpec(dims, base, False, YarnSpec(*sc) if sc else None), DEV),
            positions=pos.to(DEV), q_out=q, q_hd=D, k_cache=kc, v_cache=vc, slots=torch.arange(T, device=DEV))
    f, gain = oracle.yarn_frequencies(base, dims, dict(zip(("factor", "original", "fast", "slow"), sc)) if sc else None)
    p = proj.double()
    want_q = oracle.rotate_half(p[:, :heads * D].view(T, heads, D), pos, f, gain)
    want_k = oracle.rotate_half(p[:, heads * D:(heads + G) * D].view(T, G, D), pos, f, gain)
    assert rel(q.view(T, heads, D), want_q) < tol and rel(kc[0, :, :T].transpose(0, 1), want_k) < tol


# ---------------------------------------------------------------- chunks and the sink
@pytest.mark.parametrize("path", ["tc", "bf16", "f32"])
@pytest.mark.parametrize("heads,G,D,E,T,chunk", [(4, 2, 64, 64, 300, 44), (3, 1, 48, 96, 420, 129), (2, 2, 96, 32, 200, 16), (8, 1, 128, 128, 530, 256),
                                                 (2, 1, 80, 72, 150, 1), (4, 4, 32, 40, 270, 0), (12, 1, 64, 24, 260, 100)])
def test_attention_sees_its_chunk_and_nothing_else(H, path, heads, G, D, E, T, chunk):
    g = gen(T + D)
    q, k, v = b16(torch.randn(T, heads, D, generator=g)), b16(torch.randn(T, G, D, generator=g)), b16(torch.randn(T, G, E, generator=g))
    scale = 1.3 * D ** -0.5
    tol = 2e-5 if path == "f32" else 5e-3
    want = oracle.chunk_attention(q.double(), k.double(), v.double(), scale, chunk)
    for mode in ("decode", T, T // 2 + 1, 2):
        got = run_attention(H, path, q, k, v, scale, 0, 0, mode, chunk=chunk, sink=0.0)
        lo = 0 if mode == "decode" else T - mode
        assert rel(got[lo:], want[lo:]) < tol, mode


@pytest.mark.parametrize("path", ["tc", "f32"])
def test_one_standing_out_key_at_every_chunk_edge(H, path):
    """A key that would take nearly all the weight is placed just inside and just outside every edge."""
    heads, G, D, E, T, chunk = 2, 1, 64, 48, 290, 50
    g = gen(3)
    q, k0, v = b16(torch.randn(T, heads, D, generator=g)), b16(torch.randn(T, G, D, generator=g) * 0.1), b16(torch.randn(T, G, E, generator=g))
    q[:, 1] = q[:, 0]
    for i in (0, 49, 50, 51, 99, 100, 127, 128, 149, 150, T - 1):
        for j in {i // chunk * chunk + d for d in (-2, -1, 0, 1)} | {i - 1, i, 15, 16, 127, 128}:
            if not 0 <= j <= i:
                continue
            k = k0.clone()
            k[j, 0] = b16(2.0 * q[i, 0])
            want = oracle.chunk_attention(q.double(), k.double(), v.double(), 0.2, chunk)
            for mode in ("decode", T):
                got = run_attention(H, path, q, k, v, 0.2, 0, 0, mode, chunk=chunk, sink=0.0)
                assert rel(got[i], want[i]) < (2e-5 if path == "f32" else 5e-3), (i, j, mode)
            hit = float((want[i, 0] - v[j, 0]).abs().max()) < 0.05
            assert hit == oracle.same_chunk(i, j, chunk), (i, j)      # the case is sharp


@pytest.mark.parametrize("path", ["tc", "f32"])
@pytest.mark.parametrize("level", [-4.0, 0.0, 3.0, 60.0])
def test_the_sink_takes_its_share(H, path, level):
    """All scores near `level`: the sink (score 0) takes nearly everything, a countable part, or nothing. Other sinks scale."""
    heads, G, D, E, T = 2, 2, 64, 64, 40
    g = gen(5)
    k = b16(0.01 * torch.randn(T, G, D, generator=g))
    q = b16(0.01 * torch.randn(T, heads, D, generator=g))
    q[..., 0], k[..., 0] = 8.0, level / 8.0
    v = 1 + 0.1 * torch.rand(T, G, E, generator=g)
    k, v = b16(k), b16(v)
    for sink in (0.0, 1.5):
        want = oracle.chunk_attention(q.double(), k.double(), v.double(), 1.0, 9, sink=False)
        for i in range(T):
            s = torch.einsum("hd,jhd->hj", q[i].double(), k[i // 9 * 9:i + 1].double())
            want[i] *= (torch.sigmoid(torch.logsumexp(s, -1) - sink))[:, None]
        for mode in ("decode", T):
            got = run_attention(H, path, q, k, v, 1.0, 0, 0, mode, chunk=9, sink=sink)
            assert rel(got, want) < (2e-5 if path == "f32" else 6e-3), (sink, mode)
    got = run_attention(H, path, q, k, v, 1.0, 0, 0, T, chunk=9)             # none
    assert rel(got, oracle.chunk_attention(q.double(), k.double(), v.double(), 1.0, 9, sink=False)) < 6e-3


# ---------------------------------------------------------------- state-space layer
def pad16(n):
    return (n + 15) // 16 * 16


class Ssd:
    """A state-space layer's weights and inputs in the device's padded layout, run in portions."""

    def __init__(self, H, h, E, N, G, taps, T, seed, proj_dtype, scale_dt=0.5):
        g = gen(seed)
        self.ops, self.h, self.E, self.N, self.G, self.taps, self.T = H, h, E, N, G, taps, T
        self.EP, self.NP = pad16(E), pad16(N)
        inner, gn = h * E, G * N
        self.xbc = b16(torch.randn(T, inner + 2 * gn, generator=g))
        self.dt = b16(torch.randn(T, h, generator=g) * scale_dt)
        self.conv, self.conv_b = 0.6 * torch.randn(inner + 2 * gn, taps, generator=g), 0.2 * torch.randn(inner + 2 * gn, generator=g)
        self.bias, self.A, self.D = -1.5 + 0.5 * torch.randn(h, generator=g), -2.5 + 1.5 * torch.randn(h, generator=g), torch.randn(h, generator=g)
        self.proj_dtype = proj_dtype

    def channels(self, t):
        """[.., inner + 2 G N] -> padded channels."""
        x, b, c = t.split([self.h * self.E, self.G * self.N, self.G * self.N], -1)
        pad = lambda u, n, k, kp: torch.nn.functional.pad(u.reshape(*u.shape[:-1], n, k), (0, kp - k)).flatten(-2)
        return torch.cat([pad(x, self.h, self.E, self.EP), pad(b, self.G, self.N, self.NP), pad(c, self.G, self.N, self.NP)], -1)

    def rows(self):
        z = torch.full((self.T, self.h * self.EP), float("nan"))       # the gate is not this kernel's business
        p = torch.cat([z, self.channels(self.xbc), self.dt], -1)
        out = torch.zeros(self.T, (p.shape[1] + 7) // 8 * 8 + 8)
        out[:, :p.shape[1]] = p
        return out.to(self.proj_dtype).to(DEV)

    def weights(self):
        dev = lambda t: t.float().contiguous().to(DEV)
        return (dev(self.channels(self.conv.T).T), dev(self.channels(self.conv_b[None])[0]), dev(self.bias), dev(self.A), dev(self.D))

    def want(self):
        x, b, c = oracle.silu(oracle.short_conv(self.xbc.double(), self.conv.double(), self.conv_b.double())).split(
            [self.h * self.E, self.G * self.N, self.G * self.N], -1)
        return oracle.ssd(x.view(self.T, self.h, self.E), b.view(self.T, self.G, self.N), c.view(self.T, self.G, self.N),
                          oracle.softplus(self.dt.double() + self.bias.double()), self.A.double(), self.D.double())

    def fresh(self, slots=4):
        """States whose old contents must not matter."""
        nan = lambda *s: torch.full(s, float("nan"), device=DEV)
        return nan(slots, self.h, self.NP, self.EP), nan(slots, self.taps, self.h * self.EP + 2 * self.G * self.NP)

    def run(self, cuts, dtype, runs, slot=2, segment=0, state=None, y=None):
        H, T = self.ops, self.T
        proj, w = self.rows(), self.weights()
        st, cv = state if state is not None else self.fresh()
        y = torch.full((T, self.h * self.EP), float("nan"), dtype=dtype, device=DEV) if y is None else y
        at, cuts = 0, list(cuts)
        while at < T:
            n = min(cuts.pop(0) if cuts else T - at, T - at)
            pr, o = proj[at:at + n], y[at:at + n]
            kw = dict(h=self.h, g=self.G, w=w, state=st, conv_state=cv, y=o)
            if n == 1:
                H.ssd_decode(pr, 1, row_slots=i32([slot]), positions=i32([at]), **kw)
            else:
                tiles = -(-n // 128)
                if segment and n > segment:
                    kw.update(segment=segment, ws=torch.full((H.ssd_ws_elems(self.h, self.EP, self.NP, tiles),), float("nan"), device=DEV))
                u = torch.zeros(n, self.h * self.EP + 2 * self.G * self.NP, dtype=dtype, device=DEV)
                H.ssd_prefill(pr, n, seq_slots=i32([slot]), tile_seq=i32([0] * tiles), tile_q0=i32([128 * t for t in range(tiles)]),
                              q_start=i32([0]), q_lens=i32([n]), ctx_lens=i32([at + n]), n_tiles=tiles, n_seqs=1, u=u, runs=runs, **kw)
            at += n
        return y.view(T, self.h, self.EP)[..., :self.E], st, cv


@pytest.mark.parametrize("form", ["runs", "runs-f32-rows", "segments", "scan-bf16", "scan-f32"])
@pytest.mark.parametrize("h,E,N,G,taps,T", [(2, 64, 128, 1, 4, 330), (6, 20, 24, 3, 3, 300), (1, 16, 16, 1, 1, 140), (4, 48, 200, 2, 5, 290),
                                            (3, 7, 5, 1, 2, 150), (2, 96, 64, 2, 4, 400), (1, 33, 40, 1, 9, 150)])
def test_state_space_layer_in_portions_equals_the_recurrence(H, form, h, E, N, G, taps, T):
    f32 = form == "scan-f32"
    s = Ssd(H, h, E, N, G, taps, T, h * E + N, torch.float32 if (f32 or form == "runs-f32-rows") else torch.bfloat16)
    want, S = s.want()
    dt = torch.float32 if f32 else torch.bfloat16
    for cuts in ([], [2, 3, 1, 1, 64, 1, 65], [128, 1, 1, 2], [1] * 12 + [7, 63], [260, 2]):
        got, st, cv = s.run(cuts, dt, not form.startswith("scan"), segment=128 if form == "segments" else 0)
        assert rel(got, want) < (1e-5 if f32 else 1.2e-2), cuts          # bf16: x, B and C are rounded once
        assert rel(st[2, :, :N, :E], S) < (1e-5 if f32 else 1.2e-2), cuts
        if N < s.NP:
            assert float(st[2, :, N:].abs().max()) == 0
        assert bool(torch.isnan(st[[0, 1, 3]]).all()) and bool(torch.isnan(cv[[0, 1, 3]]).all())    # nobody else's slot


def test_the_runs_keep_32_bits(H):
    """Against the recurrence on x, B and C as the convolution kernel stored them, runs and segments agree to 32-bit
    rounding, also over steep decays."""
    h, E, N, G, taps, T = 3, 32, 48, 1, 4, 520
    s = Ssd(H, h, E, N, G, taps, T, 8, torch.bfloat16)
    s.A = torch.tensor([-5.0, 0.0, 3.0])                                   # memories of hundreds of tokens, a few, none
    w = s.weights()
    proj = s.rows()
    for segment in (0, 256):
        st, cv = s.fresh()
        u = torch.zeros(T, h * E + 2 * N, dtype=torch.bfloat16, device=DEV)
        y = torch.zeros(T, h * E, dtype=torch.bfloat16, device=DEV)
        tiles = -(-T // 128)
        ws = torch.empty(H.ssd_ws_elems(h, E, N, tiles), device=DEV) if segment else None
        H.ssd_prefill(proj, T, h=h, g=G, w=w, state=st, conv_state=cv, seq_slots=i32([1]), tile_seq=i32([0] * tiles),
                      tile_q0=i32([128 * t for t in range(tiles)]), q_start=i32([0]), q_lens=i32([T]), ctx_lens=i32([T]), n_tiles=tiles,
                      n_seqs=1, u=u, y=y, runs=True, segment=segment, ws=ws)
        x, b, c = u.double().cpu().split([h * E, N, N], -1)
        want, S = oracle.ssd(x.view(T, h, E), b.view(T, 1, N), c.view(T, 1, N), oracle.softplus(s.dt.double() + s.bias.double()),
                             s.A.double(), s.D.double())
        assert rel(st[1], S) < 2e-6 and rel(y.view(T, h, E), want) < 4e-3


def test_a_token_far_back_decides_the_read_out(H):
    """One loud token near the start, long memories, and a query for it hundreds of tokens later."""
    h, E, N, G, taps, T = 2, 32, 64, 1, 4, 700
    s = Ssd(H, h, E, N, G, taps, T, 9, torch.bfloat16, scale_dt=0.0)
    s.xbc = s.xbc * 0.02
    s.A = torch.full((h,), -9.0)
    s.xbc[3] = b16(8 * torch.randn(s.xbc.shape[1], generator=gen(1)).abs())
    s.xbc[T - 1, h * E + N:] = s.xbc[3, h * E:h * E + N]
    want, _ = s.want()
    assert float(want[T - 1].abs().max()) > 5 * float(want[300:T - 1].abs().max())       # it does decide
    for cuts in ([], [600] + [1] * 100, [4, 90, 2, 300, 64, 2]):
        got, _, _ = s.run(cuts, torch.bfloat16, True)
        assert rel(got[T - 1], want[T - 1]) < 1.2e-2


def test_ragged_batch_of_chunks_and_decode_rows_keeps_states_apart(H):
    """Sequences of unequal lengths in one launch, some with a past, then decode rows beside a padding row; slots used again."""
    h, E, N, G, taps = 2, 48, 40, 2, 4
    lens, pasts, slots = [130, 2, 64, 65, 300, 1], [0, 70, 0, 3, 0, 5], [4, 0, 6, 2, 1, 5]
    seqs = [Ssd(H, h, E, N, G, taps, n + p + 1, 10 * i, torch.bfloat16) for i, (n, p) in enumerate(zip(lens, pasts))]
    for s in seqs[1:]:
        for k in ("conv", "conv_b", "bias", "A", "D"):
            setattr(s, k, getattr(seqs[0], k))
    state = seqs[0].fresh(7)
    for s, p, sl in zip(seqs, pasts, slots):
        if p:                                                             # what came before, on its own
            t, s.T = s.T, p
            full = s.xbc, s.dt
            s.xbc, s.dt = s.xbc[:p], s.dt[:p]
            s.run([], torch.bfloat16, True, slot=sl, state=state)
            s.T, (s.xbc, s.dt) = t, full
    rows = torch.cat([s.rows()[p:p + n] for s, n, p in zip(seqs, lens, pasts)])
    M, start = rows.shape[0], np.cumsum([0] + lens[:-1]).tolist()
    tiles = [(i, t * 128) for i, n in enumerate(lens) for t in range(-(-n // 128))]
    y = torch.zeros(M, h * seqs[0].EP, dtype=torch.bfloat16, device=DEV)
    for segment in (0, 128):
        st = tuple(t.clone() for t in state)
        ws = torch.empty(H.ssd_ws_elems(h, seqs[0].EP, seqs[0].NP, len(tiles)), device=DEV) if segment else None
        H.ssd_prefill(rows, M, h=h, g=G, w=seqs[0].weights(), state=st[0], conv_state=st[1], seq_slots=i32(slots),
                      tile_seq=i32([t[0] for t in tiles]), tile_q0=i32([t[1] for t in tiles]), q_start=i32(start), q_lens=i32(lens),
                      ctx_lens=i32([n + p for n, p in zip(lens, pasts)]), n_tiles=len(tiles), n_seqs=len(lens),
                      u=torch.zeros(M, seqs[0].channels(seqs[0].xbc).shape[1], dtype=torch.bfloat16, device=DEV), y=y, runs=True,
                      segment=segment, ws=ws)
        for s, n, p, a, sl in zip(seqs, lens, pasts, start, slots):
            want, _ = s.want()
            assert rel(y[a:a + n].view(n, h, -1)[..., :E], want[p:p + n]) < 1.2e-2, (segment, n)
        assert bool(torch.isnan(st[0][3]).all())
    # one more token each, in one decode step; row 2 is padding, row 4 starts afresh in a used slot
    order = [3, 0, None, 5, None]
    nxt = torch.stack([seqs[i].rows()[-1] if i is not None else seqs[1].rows()[0] for i in order])
    rs, ps = [slots[i] if i is not None else -1 for i in order], [seqs[i].T - 1 if i is not None else 9 for i in order]
    rs[4], ps[4] = slots[2], 0
    out = torch.full((5, h * seqs[0].EP), 7.0, dtype=torch.bfloat16, device=DEV)
    kept = st[0][slots[4]].clone()
    H.ssd_decode(nxt, 5, h=h, g=G, w=seqs[0].weights(), state=st[0], conv_state=st[1], row_slots=i32(rs), positions=i32(ps), y=out)
    for r, i in enumerate(order):
        if i is not None:
            want, _ = seqs[i].want()
            assert rel(out[r].view(h, -1)[:, :E], want[-1]) < 1.2e-2, r
    assert rel(out[4].view(h, -1)[:, :E], seqs[1].want()[0][0]) < 1.2e-2
    assert bool((out[2] == 7).all()) and torch.equal(st[0][slots[4]], kept)


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 3e-6), (torch.bfloat16, 8e-3)])
@pytest.mark.parametrize("M,h,E,groups", [(3, 4, 32, 2), (700, 8, 64, 1), (5, 6, 20, 4), (9, 3, 7, 3), (40, 64, 64, 8), (5000, 16, 64, 2)])
def test_gate_and_norm_in_groups(H, M, h, E, groups, dtype, tol):
    g = gen(M)
    EP = pad16(E)
    y, z, w = (torch.randn(M, h * E, generator=g) for _ in range(2)), None, 1 + 0.3 * torch.randn(h * E, generator=g)
    y, z = (t.to(dtype) for t in y)
    pad = lambda t: torch.nn.functional.pad(t.view(M, h, E), (0, EP - E)).flatten(1).to(DEV)
    zz = torch.zeros(M, h * EP + 24, dtype=dtype, device=DEV)
    zz[:, :h * EP] = pad(z)
    out = torch.zeros(M, (h * E + 63) // 64 * 64, dtype=dtype, device=DEV)
    H.gated_norm(pad(y), zz, M, h=h, e=E, ep=EP, groups=groups, w=w.to(DEV), eps=1e-3, out=out)
    assert rel(out[:, :h * E], oracle.gated_group_norm(y.double(), z.double(), w.double(), groups, 1e-3)) < tol


# ---------------------------------------------------------------- mixture of experts
def routed(H, M, E, top, N, dtype, mode, seed=0, sharp=3.0):
    from oxide_tech_llm_engine_b200 import ops

    g = gen(seed + M + E)
    h = torch.zeros(M, (N + 63) // 64 * 64)
    h[:, :N] = torch.randn(M, N, generator=g)
    rw = torch.zeros((E + 63) // 64 * 64, h.shape[1])
    rw[:E, :N] = torch.randn(E, N, generator=g) * sharp * N ** -0.5
    h, rw = h.to(dtype), rw.to(dtype)
    hd, rd = h.to(DEV), rw.to(DEV)
    n = M * top
    wt, ex, sl, cnt = torch.zeros(n, device=DEV), i32([0] * n), i32([0] * n), i32([0] * E)
    kw = dict(e=E, top=top, weight=wt, expert=ex, slot=sl)
    rows = max(E * 128, (n + 127 * E) // 128 * 128)
    xs = torch.zeros(rows, h.shape[1], dtype=dtype, device=DEV)
    if mode == "packed":
        lg = torch.zeros(M, rw.shape[0], device=DEV)
        ops.gemm(hd, rd, out=lg, epi=ops.EPI_STORE_F32)
        H.moe_route(hd, rd[:E], M, mode=2, logits=lg, counts=cnt, **kw)
        H.moe_scatter(hd, M, e=E, top=top, expert=ex, slot=sl, counts=cnt, xs=xs)
    elif mode == "slab":
        H.moe_route(hd, rd[:E], M, mode=1, counts=cnt, xs=xs, **kw)
    else:
        H.moe_route(hd, rd[:E], M, **kw)
    ids, v = oracle.choose(h.double() @ rw[:E].double().T, top)
    return h, hd, ids, v, wt, ex, sl, cnt, xs


@pytest.mark.parametrize("mode,dtype", [("pairs", torch.float32), ("pairs", torch.bfloat16), ("slab", torch.bfloat16), ("packed", torch.bfloat16)])
@pytest.mark.parametrize("M,E,top,N", [(1, 5, 2, 64), (3, 16, 1, 192), (100, 33, 3, 76), (128, 130, 9, 128), (128, 1, 1, 64), (77, 512, 32, 256), (500, 8, 2, 96),
                                       (1000, 64, 8, 512)])
def test_router_and_placement(H, M, E, top, N, mode, dtype):
    if mode == "slab" and M > 128:
        M = 128
    h, hd, ids, v, wt, ex, sl, cnt, xs = routed(H, M, E, top, N, dtype, mode)
    got = ex.view(M, top).cpu().long()
    # the same experts, in order of their scores, up to ties to rounding
    same = got == ids
    assert float((~same).float().mean()) < 0.01
    assert rel(wt.view(M, top).cpu()[same], v[same]) < 5e-5
    assert float((wt.view(M, top).sum(-1) - 1).abs().max()) < 1e-5
    assert all(len(set(r)) == top for r in got.tolist())
    s = sl.view(M, top).cpu().long()
    if mode == "pairs":
        assert s.flatten().tolist() == list(range(M * top))
        return
    c = torch.bincount(got.flatten(), minlength=E)
    assert torch.equal(c, cnt.cpu().long())
    first = torch.arange(E) * 128 if mode == "slab" else (torch.cumsum((c + 127) // 128, 0) - (c + 127) // 128) * 128
    assert len(set(s.flatten().tolist())) == M * top
    assert bool(((s >= first[got]) & (s < first[got] + c[got])).all())
    for k in range(top):
        assert torch.equal(xs[s[:, k].to(DEV)], hd)


@pytest.mark.parametrize("mode", ["slab", "packed"])
@pytest.mark.parametrize("E,N,K,bn", [(5, 64, 64, 64), (9, 192, 320, 128), (70, 256, 128, 256), (3, 320, 64, 128), (1, 64, 192, 64)])
def test_expert_products_of_unequal_groups(mode, E, N, K, bn):
    """Grouped GEMM over slabs and over packed rows: empty experts, single rows, several tiles, squared ReLU."""
    from oxide_tech_llm_engine_b200 import ops

    g = gen(E * N)
    sizes = [0, 1, 128, 5, 0, 127, 300, 129, 0]
    counts = [(sizes[i % 9] if mode == "packed" else min(128, sizes[i % 9])) for i in range(E)]
    if E == 1:
        counts = [37]
    first = np.cumsum([0] + [(c + 127) // 128 * 128 for c in counts]) if mode == "packed" else np.arange(E + 1) * 128
    w = (torch.randn(E, N, K, generator=g) * K ** -0.5).to(torch.bfloat16)
    x = torch.randn(max(128, int(first[-1])), K, generator=g).to(torch.bfloat16)
    m_tiles = max(1, sum((c + 127) // 128 for c in counts)) if mode == "packed" else E
    m_tiles = min(m_tiles, x.shape[0] // 128)
    for act in (0, 2):
        out = torch.full((x.shape[0], N), 3.0, dtype=torch.bfloat16, device=DEV)
        xd, od, cnt, tk = x.to(DEV), out, i32(counts), i32([0])
        if mode == "slab":
            xd, od = xd.view(E, 128, K), od.view(E, 128, N)
        ops.gemm(xd, w.to(DEV), out=od, group_counts=cnt, m_tiles=m_tiles, act=act, bn=bn, done_ticket=tk, reset_on_done=cnt)
        for e, c in enumerate(counts):
            a = int(first[e])
            want = x[a:a + c].double() @ w[e].double().T
            if act:
                want = oracle.relu_squared(want)
            if c:
                assert rel(out[a:a + c], want) < 6e-3, (e, c)
            end = int(first[e + 1])
            assert bool((out[a + c:end] == 3).all())                       # rows past the group stay untouched
        assert cnt.tolist() == [0] * E and tk.tolist() == [0]


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 3e-6), (torch.bfloat16, 6e-3)])
@pytest.mark.parametrize("pairs,top,E,N,K", [(2, 2, 5, 64, 64), (9, 3, 7, 70, 128), (8, 8, 64, 320, 2048), (1, 1, 1, 1, 8)])
def test_expert_products_of_single_rows(H, pairs, top, E, N, K, dtype, tol):
    g = gen(N)
    w = (torch.randn(E, N, K, generator=g) * K ** -0.5).to(dtype)
    x, xp = torch.randn(pairs // top, K, generator=g).to(dtype), torch.randn(pairs, K, generator=g).to(dtype)
    ex = torch.randint(0, E, (pairs,), generator=g, dtype=torch.int32)
    for per_pair, src, act in ((False, x, 2), (True, xp, 0)):
        y = torch.zeros(pairs, N + 3, dtype=dtype, device=DEV)
        H.moe_rows(src.to(DEV), w.to(DEV), ex.to(DEV), pairs, top=top, per_pair=per_pair, y=y, act=act)
        want = torch.stack([w[ex[i]].double() @ src[i if per_pair else i // top].double() for i in range(pairs)])
        assert rel(y[:, :N], oracle.relu_squared(want) if act else want) < tol and float(y[:, N:].abs().max()) == 0


# ---------------------------------------------------------------- whole models
def toks(n, vocab, seed=0):
    return np.random.default_rng(seed).integers(0, vocab, size=n).tolist()


class Expected:
    """Logits of the plain implementation, and which tokens make clear choices of experts."""

    def __init__(self, c, w, tokens):
        m: list = []
        self.logits = oracle.forward(c, w, tokens, margins=m).numpy()
        self.clear = (torch.stack(m).min(0).values > 0.03).numpy() if m else np.ones(len(tokens), dtype=bool)

    def close(self, got, dtype, at=slice(None)):
        """32-bit: every row to rounding. bf16: rows to a few per cent, but for close calls of a router, which rounding
        may turn."""
        want, clear = self.logits[at], self.clear[at]
        rows = np.array([hm.error(got[i:i + 1], want[i:i + 1]) for i in range(len(want))])
        if dtype == "float32":
            return rows.max() < 2e-4
        return not clear.any() or (rows[clear].max() < 0.06 and (len(rows) < 20 or np.median(rows) < 0.015))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(pm.CONFIGS))
def test_prompts_portions_and_batches_equal_the_plain_implementation(name, dtype):
    c = pm.CONFIGS[name]
    w = pm.weights(c, 2)
    eng = hm.engine(c, w, dtype=dtype, live=3, blocks=56)
    seqs = [toks(n, c["vocab"], n) for n in (1, 45, 150, 2, 97, 290, 33, 128)]
    want = [Expected(c, w, t) for t in seqs]
    for t, x in zip(seqs, want):
        assert x.close(hm.feed_all(eng, 0, t, []), dtype)
        assert x.close(hm.feed_all(eng, 0, t, [2, 3, 1, 1, 17, 2, 64]), dtype)
    for seed in (1, 2):
        for got, x in zip(hm.interleaved(eng, seqs, seed), want):
            assert x.close(got, dtype)
    assert eng.sched.num_free_blocks() == 56 and eng.sched.num_free_slots() == 3
    eng.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding_token_by_token(dtype):
    c = pm.CONFIGS["mixed"]
    w = pm.weights(c, 2)
    eng = hm.engine(c, w, dtype=dtype, live=2, blocks=48)
    t = toks(300, c["vocab"], 5)
    assert Expected(c, w, t).close(hm.feed_all(eng, 0, t, [1] * 300), dtype)
    assert eng.stats["graph_replays"] > 250
    eng.close()


def test_side_streams_change_nothing(monkeypatch):
    """Decode steps whose layer parts run on streams of their own give the logits of the single stream, up to the order
    in which split sums arrive."""
    c = pm.CONFIGS["mixed"]
    w = pm.weights(c, 3)
    seqs = [toks(40, c["vocab"], i) for i in range(4)]
    out = []
    for on in ("1", "0"):
        monkeypatch.setenv("OXB_STREAMS", on)
        eng = hm.engine(c, w, live=4, blocks=48)
        assert (eng.model.streams2 is not None) == (on == "1")
        rows = [eng.feed([(i, s[:8], [7]) for i, s in enumerate(seqs)])]
        for j in range(8, 40):
            rows.append(eng.feed([(i, s[j:j + 1], [0]) for i, s in enumerate(seqs)]))
        out.append(np.stack(rows))
        eng.close()
    for i, s in enumerate(seqs):
        x = Expected(c, w, s)
        same = np.array([hm.error(a[i:i + 1], b[i:i + 1]) for a, b in zip(*out)])
        assert same[x.clear[7:]].max() < 0.01
        assert x.close(out[0][:, i], "bfloat16", slice(7, None))


def test_layer_outputs_follow_every_layer():
    c = pm.CONFIGS["mixed"]
    w = pm.weights(c, 2)
    eng = hm.engine(c, w, dtype="float32")
    t = toks(37, c["vocab"], 8)
    seen = {}
    eng.model.layer_hook = lambda i, x: seen.__setitem__(i, x.cpu())
    eng.feed([(0, t, [])])
    _, want = oracle.forward(c, w, t, want_layers=True)
    assert sorted(seen) == list(range(len(want)))
    for i, x in enumerate(want):
        assert rel(seen[i], x) < 2e-5
    eng.close()


@pytest.mark.parametrize("burst", [0, 6])
@pytest.mark.parametrize("name", ["mixed", "ones"])
def test_greedy_generation_through_the_engine(name, burst):
    """32-bit, so that the tokens are the plain implementation's: chunked prompts, a pool and slots that are short, graph
    replays, decode bursts."""
    c = pm.CONFIGS[name]
    w = pm.weights(c, 4)
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
    c = pm.CONFIGS["mixed"]
    w = pm.weights(c, 4)
    eng = hm.engine(c, w, live=3, blocks=40, tokens=64, speculative="ngram", chunk_max=64)
    assert eng._drafter is None              # a state cannot be cut back
    prompts = [toks(n, c["vocab"], n) for n in (20, 33, 150)]
    outs = eng.generate(prompts, SamplingParams(greedy=True, max_tokens=20, ignore_eos=True))
    for p, o in zip(prompts, outs):
        lg = oracle.forward(c, w, p + o[:-1]).numpy()[len(p) - 1:]
        assert (lg.max(-1) - lg[np.arange(20), o]).max() < 0.4 * lg.std()
    s = eng.generate(prompts, SamplingParams(temperature=0.8, top_k=20, top_p=0.9, seed=1, max_tokens=8, ignore_eos=True))
    assert all(len(x) == 8 and 0 <= min(x) and max(x) < c["vocab"] for x in s)
    eng.close()


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_trace_replay_program(tmp_path, dtype):
    c = pm.CONFIGS["mixed"]
    w = pm.weights(c, 6)
    hm.write_model(tmp_path / "m", c, w)
    t = toks(170, c["vocab"], 3)
    want = Expected(c, w, t)
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
    assert want.close(read(0), dtype, [0, 149]) and not (tmp_path / "out" / "1.f32").exists()
    assert want.close(read(2), dtype, [39, 169]) and want.close(read(3), dtype, [19])
