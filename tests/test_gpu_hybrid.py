"""Kernels and serving of layer-list decoders on the GPU, against the plain implementation: every
mechanism alone, then whole models in 32-bit (sharp) and bf16."""
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import hybrid_models as hm
import hybrid_oracle as oracle
from oxide_tech_llm_engine_b200.sampling_params import SamplingParams

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


def gen(seed):
    return torch.Generator().manual_seed(seed)


def rel(a, b):
    a, b = a.double().cpu(), b.double().cpu()
    return float((a - b).abs().max() / b.abs().max().clamp_min(1e-30))


# ---------------------------------------------------------------- residual streams and norm
@pytest.mark.parametrize("dtype,tol", [(torch.float32, 3e-6), (torch.bfloat16, 6e-3)])
@pytest.mark.parametrize("S,N,rows", [(1, 64, 3), (2, 4096, 5), (3, 200, 700), (5, 76, 9), (9, 130, 4), (16, 33, 2)])
def test_stream_norm_embedding_update_and_readout(H, S, N, rows, dtype, tol):
    g = gen(S * 1000 + N)
    vocab, buckets = 50, 23
    emb, big = (torch.randn(n, N, generator=g).to(dtype) for n in (vocab, buckets + 1))
    tok = torch.randint(0, vocab, (rows,), generator=g, dtype=torch.int32)
    prev = torch.randint(0, vocab, (rows,), generator=g, dtype=torch.int32)
    prev[0] = -1
    w1, w2 = torch.randn(N, generator=g) * 0.2, torch.randn(N, generator=g) * 0.2
    cin, out, mix = torch.randn(S, generator=g), torch.randn(S, generator=g), torch.randn(S, S, generator=g)
    ld = (N + 63) // 64 * 64
    x = torch.full((rows, S, N), float("nan"), device=DEV)
    h = torch.zeros(rows, ld, dtype=dtype, device=DEV)
    clear = torch.ones(rows, 12, device=DEV)
    c = lambda t: t.to(DEV)
    H.stream_norm(x, rows, norm_w=c(w1), eps=1e-3, h=h, tokens=c(tok), prev=c(prev), embed=c(emb), bigram=c(big), mul_prev=70001,
                  mul_cur=50021, in_w=c(cin), clear=clear)
    b = [buckets if p < 0 else (p * 70001 + t * 50021) % buckets for p, t in zip(prev.tolist(), tok.tolist())]
    e = emb[tok.long()].double() + big[b].double()
    xs = torch.stack([e] * S)
    want = oracle.norm_around_zero(torch.einsum("s,std->td", cin.double(), xs), w1.double(), 1e-3)
    assert rel(h[:, :N], want) < tol and float(clear.abs().max()) == 0 and float(h[:, N:].abs().max() if ld > N else 0) == 0
    assert rel(x, xs.transpose(0, 1)) < 1e-6
    y = torch.zeros(rows, ld, device=DEV)
    y[:, :N] = c(torch.randn(rows, N, generator=g))
    yc = y[:, :N].double().cpu()
    H.stream_norm(x, rows, norm_w=c(w2), eps=1e-3, h=h, y=y, mix=c(mix), out_w=c(out), in_w=c(cin))
    xs = torch.einsum("sz,std->ztd", mix.double(), xs) + out.double()[:, None, None] * yc[None]
    assert rel(x, xs.transpose(0, 1)) < 3e-6 and float(y.abs().max()) == 0
    assert rel(h[:, :N], oracle.norm_around_zero(torch.einsum("s,std->td", cin.double(), xs), w2.double(), 1e-3)) < tol
    # the last one: plain sum of the streams, only the mapped rows
    y[:, :N] = 1.0
    rmap = torch.full((rows,), -1, dtype=torch.int32)
    rmap[rows - 1] = 0
    h2 = torch.zeros(1, ld, dtype=dtype, device=DEV)
    before = x.clone()
    H.stream_norm(x, rows, norm_w=c(w1), eps=1e-3, h=h2, y=y, mix=c(mix), out_w=c(out), store_x=False, row_map=c(rmap))
    xs = torch.einsum("sz,std->ztd", mix.double(), xs) + out.double()[:, None, None]
    assert rel(h2[0, :N], oracle.norm_around_zero(xs.sum(0)[-1], w1.double(), 1e-3)) < tol and torch.equal(x, before)


# ---------------------------------------------------------------- projections -> heads
@pytest.mark.parametrize("store,proj_dt", [("f32", torch.float32), ("bf16", torch.float32), ("bf16", torch.bfloat16)])
@pytest.mark.parametrize("heads,G,D,E,dims,inter", [(4, 2, 64, 64, 64, True), (3, 1, 40, 24, 12, True), (6, 6, 33, 50, 30, False),
                                                    (16, 4, 128, 96, 0, True)])
def test_heads_norm_over_the_projection_rotation_and_cache_write(H, heads, G, D, E, dims, inter, store, proj_dt):
    from oxide_tech_llm_engine_b200.models.layer_spec import RotarySpec

    g = gen(D)
    T, DP, EP = 5, 144, 128
    dt = torch.float32 if store == "f32" else torch.bfloat16
    W = heads * D + G * (D + E)
    proj = (torch.randn(T, W + 3, generator=g) * 2).to(proj_dt)
    qw, kw = 1 + 0.3 * torch.randn(heads * D, generator=g), 1 + 0.3 * torch.randn(G * D, generator=g)
    pos = torch.tensor([0, 1, 777, 30011, 262143], dtype=torch.int32)
    slots = torch.tensor([5, 16, 31, -1, 47])
    kc, vc = torch.full((3, G, 16, DP), 9.0, dtype=dt, device=DEV), torch.full((3, G, 16, EP), 9.0, dtype=dt, device=DEV)
    q = torch.zeros(T, heads * DP, dtype=dt, device=DEV)
    rot = H.Rotary(RotarySpec(dims, 1e6, inter), DEV)
    H.heads(proj.to(DEV), T, h=heads, g=G, d=D, e=E, rot=rot, positions=pos.to(DEV), q_out=q, q_hd=DP, q_norm=qw.to(DEV),
            k_norm=kw.to(DEV), eps=1e-3, k_cache=kc, v_cache=vc, slots=slots.to(DEV))
    p = proj.double()
    wq = (oracle.rms(p[:, :heads * D], 1e-3) * qw).view(T, heads, D)
    wk = (oracle.rms(p[:, heads * D:(heads + G) * D], 1e-3) * kw).view(T, G, D)
    if dims:
        wq, wk = oracle.rotate(wq, pos, 1e6, dims, inter), oracle.rotate(wk, pos, 1e6, dims, inter)
    wv = p[:, (heads + G) * D:W].view(T, G, E)
    tol = 3e-6 if store == "f32" else 4e-3
    got = q.view(T, heads, DP).cpu()
    assert rel(got[..., :D], wq) < tol and float(got[..., D:].abs().max()) == 0
    for t, s in enumerate(slots.tolist()):
        if s >= 0:
            assert rel(kc[s // 16, :, s % 16, :D], wk[t]) < tol and rel(vc[s // 16, :, s % 16, :E], wv[t]) < tol
    untouched = torch.ones(48, dtype=torch.bool)
    untouched[[5, 16, 31, 47]] = False
    assert bool((kc.permute(0, 2, 1, 3).reshape(48, -1).cpu()[untouched] == 9).all())


# ---------------------------------------------------------------- attention
def paged(k, v, DP, EP, dt, seed):
    """Caches with shuffled pages holding k [T, G, D], v [T, G, E]; unused pages hold large values."""
    T, G, D = k.shape
    nb = (T + 15) // 16
    perm = torch.randperm(nb + 3, generator=gen(seed))
    kc, vc = torch.full((nb + 3, G, 16, DP), 50.0), torch.full((nb + 3, G, 16, EP), 50.0)
    for t in range(T):
        b = perm[t // 16]
        kc[b, :, t % 16] = 0
        vc[b, :, t % 16] = 0
        kc[b, :, t % 16, :D] = k[t]
        vc[b, :, t % 16, :v.shape[2]] = v[t]
    return kc.to(dt).to(DEV), vc.to(dt).to(DEV), perm[:nb].to(torch.int32)


def run_attention(H, path, q, k, v, scale, size, keep, mode, splits=4, **extra):
    """Rows of the last `n` positions through the prompt kernel, or every row through the decode kernel. `extra`: further
    options of the kernels (chunk, sink)."""
    from oxide_tech_llm_engine_b200 import ops

    T, heads, D = q.shape
    G, E = k.shape[1], v.shape[2]
    tc = path == "tc"
    dt = torch.float32 if path == "f32" else torch.bfloat16
    P = 64 if max(D, E) <= 64 else 128
    DP, EP = (P, P) if tc else (D, E)
    kc, vc, bt = paged(k, v, DP, EP, dt, T)
    out = torch.full((T, heads * E), float("nan"), dtype=dt, device=DEV)
    qp = torch.zeros(T, heads, DP, dtype=dt, device=DEV)
    qp[..., :D] = q.to(DEV)
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=DEV)
    kw = dict(window=size, keep_first=keep, scale=scale, **extra)
    if mode == "decode":
        tables = bt[None].repeat(T, 1).contiguous().to(DEV)
        lens = i32(list(range(1, T + 1)))
        if tc:
            po, pm = torch.empty(T * heads * splits * P, device=DEV), torch.empty(T * heads * splits * 2, device=DEV)
            pps = max(4, -(-((T + 15) // 16) // splits))
            ops.paged_decode(qp, kc, vc, tables, lens, i32([(pps + 3) // 4 * 4]), po, pm, out, batch=T, max_splits=splits, out_d=E,
                             exact_p=True, **kw)
        else:
            H.row_attention(qp.view(T, -1), DP, kc, vc, tables, n=T, h=heads, d=D, e=E, out=out, seq_lens=lens, **kw)
        return out.view(T, heads, E)
    n = mode            # the last n positions as one prompt chunk
    tiles = -(-n // 128)
    args = dict(tile_seq=i32([0] * tiles), tile_q0=i32([128 * t for t in range(tiles)]), q_start=i32([0]), q_lens=i32([n]),
                ctx_lens=i32([T]))
    qc, oc = qp[T - n:].contiguous(), torch.full((n, heads * E), float("nan"), dtype=dt, device=DEV)
    table = bt[None].contiguous().to(DEV)
    if tc:
        ops.paged_prefill(qc, kc, vc, table, args["tile_seq"], args["tile_q0"], args["q_start"], args["q_lens"], args["ctx_lens"],
                          oc, n_tiles=tiles, out_d=E, exact_p=True, **kw)
    else:
        H.row_attention(qc.view(n, -1), DP, kc, vc, table, n=tiles, h=heads, d=D, e=E, out=oc, **args, **kw)
    out[T - n:] = oc
    return out.view(T, heads, E)


@pytest.mark.parametrize("path", ["tc", "bf16", "f32"])
@pytest.mark.parametrize("heads,G,D,E,T,size,keep", [(4, 2, 64, 64, 300, 44, 6), (3, 1, 48, 96, 420, 129, 17), (2, 2, 96, 32, 200, 16, 0),
                                                     (8, 1, 128, 128, 530, 257, 130), (2, 1, 80, 72, 150, 1, 3), (4, 4, 32, 40, 270, 1000, 5)])
def test_attention_sees_the_window_and_the_kept_first_positions_and_nothing_else(H, path, heads, G, D, E, T, size, keep):
    g = gen(T + D)
    b = lambda t: t.to(torch.bfloat16).float()
    q, k, v = b(torch.randn(T, heads, D, generator=g)), b(torch.randn(T, G, D, generator=g)), b(torch.randn(T, G, E, generator=g))
    scale = 1.3 * D ** -0.5
    tol = 2e-5 if path == "f32" else 5e-3     # the bf16 paths round their output
    want = oracle.attention(q.double(), k.double(), v.double(), scale, size, keep)
    for mode in ("decode", T, T // 2 + 1, 2):
        got = run_attention(H, path, q, k, v, scale, size, keep, mode)
        lo = 0 if mode == "decode" else T - mode
        assert rel(got[lo:], want[lo:]) < tol, mode


@pytest.mark.parametrize("path", ["tc", "f32"])
def test_one_standing_out_key_at_every_edge(H, path):
    """A key that would take nearly all the weight is placed just inside and just outside every edge."""
    heads, G, D, E, T = 2, 1, 64, 48, 290
    g = gen(3)
    b = lambda t: t.to(torch.bfloat16).float()
    q, k0 = b(torch.randn(T, heads, D, generator=g)), b(torch.randn(T, G, D, generator=g) * 0.1)
    v = b(torch.randn(T, G, E, generator=g))
    q[:, 1] = q[:, 0]
    size, keep = 50, 18
    for i in (49, 50, 68, 127, 128, 176, T - 1):
        for j in {i - size + 1, i - size, i - size - 1, keep - 1, keep, 0, 15, 16, i}:
            if not 0 <= j <= i:
                continue
            k = k0.clone()
            k[j, 0] = b(2.0 * q[i, 0])
            want = oracle.attention(q.double(), k.double(), v.double(), 0.2, size, keep)
            for mode in ("decode", T):
                got = run_attention(H, path, q, k, v, 0.2, size, keep, mode)
                assert rel(got[i], want[i]) < (2e-5 if path == "f32" else 5e-3), (i, j, mode)
            # the case is sharp: the key is seen or not, and that decides the row
            hit = float((want[i, 0] - v[j, 0]).abs().max()) < 0.05
            assert hit == oracle.visible(i, j, size, keep), (i, j)


# ---------------------------------------------------------------- retention
def run_retention(H, q, k, v, gate, decay, cuts, dtype, slots, proj_f32, chunked=True, rot=None, positions=None, k_scale=1.0, eps=1e-3,
                  state=None):
    T, h, D = q.shape
    E = v.shape[2]
    pdt = torch.float32 if (dtype == torch.float32 or proj_f32) else torch.bfloat16
    proj = torch.cat([q.reshape(T, -1), k.reshape(T, -1), v.reshape(T, -1), gate.reshape(T, -1)], 1).to(pdt).to(DEV)
    out = torch.full((T, h * E), float("nan"), dtype=dtype, device=DEV)
    state = torch.full((4, h, D, E), float("nan"), device=DEV) if state is None else state     # old contents must not matter
    pw = H.decay_powers(decay, DEV)
    rot = H.Rotary(rot, DEV)
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=DEV)
    at = 0
    while at < T:
        n = min(cuts.pop(0) if cuts else T - at, T - at)
        pr = proj[at:at + n].contiguous()
        o = out[at:at + n]
        kw = dict(h=h, d=D, e=E, decay_pow=pw, eps=eps, state=state, out=o)
        pos = i32(list(range(at, at + n)))
        if n == 1:
            H.retention_decode(pr, 1, rot=rot, k_scale=k_scale, row_slots=i32([slots]), positions=pos, **kw)
        else:
            tiles = -(-n // 128)
            qr, kr = torch.empty(h, n, D, device=DEV), torch.empty(h, n, D, device=DEV)
            H.heads(pr, n, h=h, g=h, d=D, e=E, rot=rot, positions=pos, q_out=qr, q_hd=D, k_out=kr, k_scale=k_scale)
            if chunked:
                kw["ws"] = torch.full((2 * tiles * h * D * E,), float("nan"), device=DEV)
            else:
                kw["o_buf"] = torch.empty(n * h * E, device=DEV)
            H.retention_prefill(pr, n, seq_slots=i32([slots]), tile_seq=i32([0] * tiles), tile_q0=i32([128 * t for t in range(tiles)]),
                                q_start=i32([0]), q_lens=i32([n]), ctx_lens=i32([at + n]), n_tiles=tiles, n_seqs=1, q_rot=qr, k_rot=kr,
                                **kw)
        at += n
    return out.view(T, h, E), state


@pytest.mark.parametrize("form", ["chunks", "chunks-f32-rows", "scan", "scan-f32"])
@pytest.mark.parametrize("h,D,E,T,decay", [(2, 64, 64, 330, [0.97, 0.9999]), (3, 40, 20, 200, [1.0, 0.5, 0.99]), (1, 128, 256, 140, [0.995]),
                                           (2, 33, 30, 150, [0.9, 0.999]), (1, 96, 7, 129, [0.98]), (4, 256, 128, 190, [0.9, 0.99, 0.999, 1.0])])
def test_retention_in_portions_equals_the_recurrence(H, form, h, D, E, T, decay):
    from oxide_tech_llm_engine_b200.models.layer_spec import RotarySpec

    g = gen(D * E)
    b = lambda t: t.to(torch.bfloat16).float()
    q, k, v, gate = (b(torch.randn(T, h, n, generator=g)) for n in (D, D, E, E))
    dims = D // 4 * 2
    spec = RotarySpec(dims, 3000.0, False) if dims else None
    pos = torch.arange(T)
    rq, rk = (oracle.rotate(x.double(), pos, 3000.0, dims, False) if dims else x.double() for x in (q, k))
    o, S = oracle.retention(rq, rk * D ** -0.5, v.double(), decay)
    want = oracle.rms(o, 1e-3) * oracle.silu(gate.double())
    dt = torch.float32 if form == "scan-f32" else torch.bfloat16
    for cuts in ([], [2, 3, 1, 1, 64, 1, 65], [128, 1, 1, 2], [1] * 12 + [7, 63]):
        got, state = run_retention(H, q, k, v, gate, decay, list(cuts), dt, 2, form == "chunks-f32-rows", form.startswith("chunks"),
                                   spec, k_scale=D ** -0.5)
        assert rel(got, want) < (2e-5 if form == "scan-f32" else 5e-3), cuts
        assert rel(state[2], S) < (1e-5 if form.startswith("chunks") else 3e-6), cuts
        assert bool(torch.isnan(state[[0, 1, 3]]).all())       # nobody else's slot is touched


def test_retention_recalls_one_key_from_far_back(H):
    """A single key / value pair at the start decides the read-out hundreds of tokens later."""
    h, D, E, T = 2, 64, 32, 700
    g = gen(9)
    q, k, v = torch.randn(T, h, D, generator=g) * 0.01, torch.randn(T, h, D, generator=g) * 0.01, torch.randn(T, h, E, generator=g)
    k[3] = 40.0 * torch.randn(h, D, generator=g)
    q[T - 1] = k[3]
    b = lambda t: t.to(torch.bfloat16).float()
    q, k, v, gate = b(q), b(k), b(v), torch.ones(T, h, E) * 2
    o, _ = oracle.retention(q.double(), k.double(), v.double(), [0.999, 1.0])
    want = oracle.rms(o, 1e-3) * oracle.silu(gate.double())
    for cuts in ([], [600] + [1] * 100, [4, 90, 2, 300, 64, 2]):
        got, _ = run_retention(H, q, k, v, gate, [0.999, 1.0], list(cuts), torch.bfloat16, 0, False)
        assert rel(got[T - 1], want[T - 1]) < 5e-3


def test_ragged_batch_of_chunks_and_decode_rows_keeps_states_apart(H):
    """Sequences of unequal lengths in one launch, some with a past, next to decode rows and a padding row."""
    h, D, E = 2, 48, 64
    lens, pasts = [130, 2, 64, 65, 257], [0, 70, 0, 5, 0]
    g = gen(4)
    b = lambda t: t.to(torch.bfloat16).float()
    seqs = [[b(torch.randn(n + p, h, x, generator=g)) for x in (D, D, E, E)] for n, p in zip(lens, pasts)]
    decay = [0.98, 0.9995]
    state = torch.full((7, h, D, E), float("nan"), device=DEV)
    slots = [4, 0, 6, 2, 1]
    for (q, k, v, gt), p, s in zip(seqs, pasts, slots):
        if p:
            run_retention(H, q[:p], k[:p], v[:p], gt[:p], decay, [], torch.bfloat16, s, False, state=state)
    rows = [torch.cat([x[p:].reshape(n, -1) for x in sq], 1) for sq, n, p in zip(seqs, lens, pasts)]
    proj = torch.cat(rows).to(torch.bfloat16).to(DEV)
    M = proj.shape[0]
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=DEV)
    start = np.cumsum([0] + lens[:-1]).tolist()
    tiles = [(s, t * 128) for s, n in enumerate(lens) for t in range(-(-n // 128))]
    qr, kr = torch.empty(h, M, D, device=DEV), torch.empty(h, M, D, device=DEV)
    H.heads(proj, M, h=h, g=h, d=D, e=E, rot=H.Rotary(None, DEV), positions=i32([0] * M), q_out=qr, q_hd=D, k_out=kr)
    out = torch.zeros(M, h * E, dtype=torch.bfloat16, device=DEV)
    H.retention_prefill(proj, M, h=h, d=D, e=E, decay_pow=H.decay_powers(decay, DEV), eps=1e-3, state=state, seq_slots=i32(slots),
                        tile_seq=i32([t[0] for t in tiles]), tile_q0=i32([t[1] for t in tiles]), q_start=i32(start), q_lens=i32(lens),
                        ctx_lens=i32([n + p for n, p in zip(lens, pasts)]), n_tiles=len(tiles), n_seqs=len(lens), q_rot=qr, k_rot=kr,
                        ws=torch.empty(2 * len(tiles) * h * D * E, device=DEV), out=out)
    for i, ((q, k, v, gt), n, p) in enumerate(zip(seqs, lens, pasts)):
        o, S = oracle.retention(q.double(), k.double(), v.double(), decay)
        want = oracle.rms(o, 1e-3) * oracle.silu(gt.double())
        assert rel(out[start[i]:start[i] + n].view(n, h, E), want[p:]) < 5e-3 and rel(state[slots[i]], S) < 1e-5
    assert bool(torch.isnan(state[[3, 5]]).all())
    # decode rows: three sequences go on, a fresh one starts in a used slot, one row is padding
    step = b(torch.randn(5, h, 2 * (D + E), generator=g))
    rows = torch.cat([step[:, :, a:z].reshape(5, -1) for a, z in ((0, D), (D, 2 * D), (2 * D, 2 * D + E), (2 * D + E, 2 * (D + E)))], 1)
    out = torch.full((5, h * E), 7.0, dtype=torch.bfloat16, device=DEV)
    before = state.clone()
    H.retention_decode(rows.to(torch.bfloat16).to(DEV), 5, h=h, d=D, e=E, decay_pow=H.decay_powers(decay, DEV), rot=H.Rotary(None, DEV),
                       k_scale=1.0, eps=1e-3, state=state, row_slots=i32([6, 4, -1, 0, 2]), positions=i32([64, 130, 9, 72, 0]), out=out)
    for r, s in ((0, 6), (1, 4), (3, 0), (4, 2)):
        S0 = None if r == 4 else before[s].double().cpu()
        o, S = oracle.retention(*(step[r:r + 1, :, a:z].double() for a, z in ((0, D), (D, 2 * D), (2 * D, 2 * D + E))), decay, S0)
        want = oracle.rms(o, 1e-3) * oracle.silu(step[r:r + 1, :, 2 * D + E:].double())
        assert rel(out[r].view(1, h, E), want) < 5e-3 and rel(state[s], S) < 3e-6
    assert bool((out[2] == 7).all()) and torch.equal(state[1], before[1])


# ---------------------------------------------------------------- 32-bit products
@pytest.mark.parametrize("M,N,K", [(1, 70, 33), (8, 129, 192), (9, 64, 64), (130, 65, 76), (200, 257, 515)])
def test_gemm_and_gated_unit_in_32_bit(H, M, N, K):
    g = gen(M)
    a, w = torch.randn(M, K, generator=g), torch.randn(N, K, generator=g)
    out = torch.zeros(M, N + 2, device=DEV)
    H.gemm_f32(a.to(DEV), w.to(DEV), out)
    assert rel(out[:, :N], a.double() @ w.double().T) < 2e-6 and float(out[:, N:].abs().max()) == 0
    gu, act = torch.randn(M, 2 * N, generator=g), torch.zeros(M, N, device=DEV)
    H.glu_f32(gu.to(DEV), act, M, N, 0)
    assert rel(act, oracle.silu(gu[:, :N].double()) * gu[:, N:].double()) < 1e-6


# ---------------------------------------------------------------- whole models
def toks(n, vocab, seed=0):
    return np.random.default_rng(seed).integers(0, vocab, size=n).tolist()


def close(got, want, dtype):
    """32-bit: every row to rounding. bf16: rows to a few per cent (rounding of activations; single rows
    more, where a head's read-out is nearly zero before its norm)."""
    rows = np.array([hm.error(got[i:i + 1], want[i:i + 1]) for i in range(len(want))])
    if dtype == "float32":
        return rows.max() < 2e-4
    return rows.max() < 0.3 and (len(rows) < 20 or np.median(rows) < 0.05)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(hm.CONFIGS))
def test_prompts_portions_and_batches_equal_the_plain_implementation(name, dtype):
    c = hm.CONFIGS[name]
    w = hm.weights(c, 2)
    eng = hm.engine(c, w, dtype=dtype, live=3, blocks=48)
    seqs = [toks(n, c["vocab"], n) for n in (1, 45, 150, 2, 97, 230, 33, 128)]
    want = [oracle.forward(c, w, t).numpy() for t in seqs]
    for t, x in zip(seqs, want):
        assert close(hm.feed_all(eng, 0, t, []), x, dtype)
        assert close(hm.feed_all(eng, 0, t, [2, 3, 1, 1, 17, 2, 64]), x, dtype)
    for seed in (1, 2):
        for got, x in zip(hm.interleaved(eng, seqs, seed), want):
            assert close(got, x, dtype)
    assert eng.sched.num_free_blocks() == 48
    eng.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding_token_by_token(dtype):
    c = hm.CONFIGS["mixed"]
    w = hm.weights(c, 2)
    eng = hm.engine(c, w, dtype=dtype, live=2, blocks=48)
    t = toks(300, c["vocab"], 5)
    want = oracle.forward(c, w, t).numpy()
    assert close(hm.feed_all(eng, 0, t, [1] * 300), want, dtype)
    assert eng.stats["graph_replays"] > 250
    eng.close()


def test_layer_outputs_follow_every_run_of_the_loop():
    c = hm.CONFIGS["mixed"]
    w = hm.weights(c, 2)
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
@pytest.mark.parametrize("name", ["mixed", "attention", "retention"])
def test_greedy_generation_through_the_engine(name, burst):
    """32-bit, so that the tokens are the plain implementation's: chunked prompts, a pool and slots that are
    short, graph replays, decode bursts (the previous token advances on the device)."""
    c = hm.CONFIGS[name]
    w = hm.weights(c, 4)
    eng = hm.engine(c, w, dtype="float32", live=3, blocks=14, tokens=40, chunk_min=4, chunk_max=32, sla_budget=False,
                    decode_burst=burst)
    prompts = [toks(n, c["vocab"], 70 + n) for n in (3, 60, 41, 17, 1)]
    if burst:
        prompts = prompts[2:]                # all run at once: bursts start when nothing waits
    outs = eng.generate(prompts, SamplingParams(greedy=True, max_tokens=30, ignore_eos=True))
    for p, o in zip(prompts, outs):
        lg = oracle.forward(c, w, p + o[:-1]).numpy()[len(p) - 1:]
        assert len(o) == 30
        gap = lg.max(-1) - lg[np.arange(30), o]
        assert gap.max() < 1e-3 * lg.std(), gap          # the argmax itself, or a tie to rounding
    assert eng.stats["graph_replays"] > 0 and (not burst or eng.stats.get("burst_steps", 0) > 0)
    assert eng.sched.num_free_blocks() == 14
    eng.close()


def test_sampling_and_drafts_in_bf16():
    c = hm.CONFIGS["attention"]
    w = hm.weights(c, 4)
    eng = hm.engine(c, w, live=3, blocks=40, tokens=64, speculative="ngram", chunk_max=64)
    assert eng._drafter is not None          # no recurrent layer: drafts can be taken back
    prompts = [toks(n, c["vocab"], n) for n in (20, 33)]
    rep = [p + p for p in prompts]           # repeats make the n-gram drafter propose
    outs = eng.generate(rep, SamplingParams(greedy=True, max_tokens=20, ignore_eos=True))
    for p, o in zip(rep, outs):
        lg = oracle.forward(c, w, p + o[:-1]).numpy()[len(p) - 1:]
        assert (lg.max(-1) - lg[np.arange(20), o]).max() < 0.3 * lg.std()
    s = eng.generate(prompts, SamplingParams(temperature=0.8, top_k=20, top_p=0.9, seed=1, max_tokens=8, ignore_eos=True))
    assert all(len(x) == 8 and 0 <= min(x) and max(x) < c["vocab"] for x in s)
    eng.close()


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_trace_replay_program(tmp_path, dtype):
    import json

    c = hm.CONFIGS["retention"]
    w = hm.weights(c, 6)
    hm.write_model(tmp_path / "m", c, w)
    t = toks(70, c["vocab"], 3)
    want = oracle.forward(c, w, t).numpy()
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": t[:50], "want": [0, 49]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": t[50:51], "want": []}, {"id": "b", "tokens": t[:2], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "b", "tokens": t[2:40], "want": [37]}, {"id": "a", "tokens": t[51:], "want": [18]}],
              "end": ["a", "b"]}]
    r = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path / "m"), "--dtype", dtype, "--out",
                        str(tmp_path / "out"), "--max-tokens", "192"], input="".join(json.dumps(s) + "\n" for s in steps), text=True,
                       capture_output=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == ["done 0", "done 1", "done 2"]
    read = lambda n: np.fromfile(tmp_path / "out" / f"{n}.f32", dtype="<f4").reshape(-1, c["vocab"])
    assert close(read(0), want[[0, 49]], dtype) and not (tmp_path / "out" / "1.f32").exists()
    assert close(read(2), want[[39, 69]], dtype)


def test_refusals():
    from oxide_tech_llm_engine_b200.errors import ConfigError
    from oxide_tech_llm_engine_b200.models.config import preset
    from oxide_tech_llm_engine_b200.models.llama import DeviceModel

    with pytest.raises(ConfigError):
        hm.engine(hm.CONFIGS["mixed"], hm.weights(hm.CONFIGS["mixed"]), h2o_pruning=True)
    with pytest.raises(ConfigError):
        DeviceModel(preset("tiny"), dtype="float32")
