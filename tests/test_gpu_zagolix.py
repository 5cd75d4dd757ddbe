"""Kernels and serving of Zagolix models on the GPU against the plain implementation: every mechanism alone, then whole
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
import zagolix_models as zm
import zagolix_oracle as oracle
from oxide_tech_llm_engine_b200.sampling_params import SamplingParams
from test_gpu_hybrid import gen, paged, rel
from test_gpu_povatar import b16, i32

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


def chunk(n, ctx):
    """Tile arguments of the last n of ctx positions of one sequence."""
    tiles = -(-n // 128)
    return tiles, dict(tile_seq=i32([0] * tiles), tile_q0=i32([128 * t for t in range(tiles)]), q_start=i32([0]), q_lens=i32([n]),
                       ctx_lens=i32([ctx]))


# ---------------------------------------------------------------- norms on either side
@pytest.mark.parametrize("dtype,tol", [(torch.float32, 3e-6), (torch.bfloat16, 6e-3)])
@pytest.mark.parametrize("N,rows,top", [(64, 3, 2), (200, 700, 3), (76, 5, 1), (2048, 330, 6), (4096, 300, 2), (4096, 4, 2), (9000, 2, 3)])
def test_the_norm_of_the_weighted_expert_rows(H, N, rows, top, dtype, tol):
    g = gen(N + rows)
    ld, eps = (N + 63) // 64 * 64, 1e-3
    c = lambda t: t.to(DEV)
    w, n1 = (1 + 0.3 * torch.randn(N, generator=g) for _ in range(2))
    x0 = torch.randn(rows, N, generator=g)
    x, h = c(x0).clone(), torch.zeros(rows, ld, dtype=dtype, device=DEV)
    er = torch.randn(rows * top + 5, ld, generator=g).to(dtype)
    slot = torch.randperm(rows * top + 5, generator=g)[:rows * top].to(torch.int32)
    wt = torch.rand(rows * top, generator=g)
    H.branch_norm(x, rows, norm_w=[c(n1)], h=[h], eps=eps, branches=[(None, c(w), 1.0, False)], experts=(c(er), c(slot), c(wt), top))
    e = torch.zeros(rows, N, dtype=torch.float64)
    for i in range(rows * top):
        e[i // top] += wt[i].double() * er[slot[i], :N].double()
    want = x0.double() + plain.rms(e, eps) * w
    assert rel(x, want) < 3e-6 and rel(h[:, :N], plain.rms(want, eps) * n1) < tol


# ---------------------------------------------------------------- heads of two maps, biases, temperature
@pytest.mark.parametrize("dtype,proj_dtype,tol", [(torch.float32, torch.float32, 3e-6), (torch.bfloat16, torch.bfloat16, 5e-3),
                                                  (torch.bfloat16, torch.float32, 5e-3)])
@pytest.mark.parametrize("heads,G,D,E,coef,every", [(4, 2, 32, 48, 0.7, 13.0), (3, 1, 20, 36, 0.0, 1.0), (6, 3, 7, 9, 0.2, 64.0), (2, 2, 64, 128, 1.5, 1.0)])
def test_two_maps_biases_and_temperature(H, heads, G, D, E, coef, every, dtype, proj_dtype, tol):
    g = gen(D)
    T = 5
    W = 2 * heads * D + 2 * G * D + G * E
    proj, bias = b16(torch.randn(T, W, generator=g)), torch.randn(W, generator=g)
    pos = torch.tensor([0, 11, 12, 63, 100000], dtype=torch.int32)
    P = 2 * D + 8
    ld = (W + 3) // 4 * 4
    pr = torch.zeros(T, ld, dtype=proj_dtype, device=DEV)
    pr[:, :W] = proj.to(DEV)
    kc, vc = torch.zeros(2, G, 16, P, dtype=dtype, device=DEV), torch.zeros(2, G, 16, E, dtype=dtype, device=DEV)
    q = torch.zeros(T, 2 * heads * P, dtype=dtype, device=DEV)
    slots = torch.tensor([3, 17, 18, -1, 31])
    H.heads(pr, T, h=2 * heads, g=2 * G, d=D, e=E, rot=H.Rotary(None, DEV), positions=pos.to(DEV), q_out=q, q_hd=P, k_cache=kc, v_cache=vc,
            slots=slots.to(DEV), maps=2, bias=bias.to(DEV), temp_coef=coef, temp_every=every)
    full = (proj + bias).double()
    qw = full[:, :2 * heads * D].view(T, heads, 2, D) * oracle.temperature(pos, coef, every)[:, None, None, None]
    got = q.view(T, heads, 2, P).cpu()
    for m in (0, 1):          # a query lies in its map's columns, the other map's are zero
        assert rel(got[:, :, m, m * D:(m + 1) * D], qw[:, :, m]) < tol
        assert float(got[:, :, m, (1 - m) * D:(2 - m) * D].abs().max()) == 0 and float(got[..., 2 * D:].abs().max()) == 0
    kw, vw = full[:, 2 * heads * D:2 * (heads + G) * D].view(T, G, 2 * D), full[:, 2 * (heads + G) * D:].view(T, G, E)
    for t, s in enumerate(slots.tolist()):
        if s >= 0:
            assert rel(kc[s // 16, :, s % 16, :2 * D], kw[t]) < tol and rel(vc[s // 16, :, s % 16], vw[t]) < tol
    assert float(kc[0, :, :3].abs().max()) == 0 and float(vc[0, :, 4:].abs().max()) == 0


# ---------------------------------------------------------------- differential attention
def run_differential(H, path, q, k, v, scale, lam, diff, eps, mode, splits=4):
    """q [T, H, 2, D], k [T, G, 2, D], v [T, G, E] through the decode kernel, or the last `mode` positions as one portion."""
    from oxide_tech_llm_engine_b200 import ops

    T, heads, _, D = q.shape
    G, E = k.shape[1], v.shape[2]
    dt = torch.float32 if path == "f32" else torch.bfloat16
    big = max(2 * D, E)
    DP, EP = (next(z for z in (64, 128, 256) if z >= big),) * 2 if path == "tc" else (2 * D, E)
    kc, vc, bt = paged(k.reshape(T, G, 2 * D), v, DP, EP, dt, T)
    qp = torch.zeros(T, heads, 2, DP, dtype=dt, device=DEV)
    for m in (0, 1):
        qp[:, :, m, m * D:(m + 1) * D] = q[:, :, m].to(DEV)
    qp = qp.view(T, 2 * heads, DP)
    lo = 0 if mode == "decode" else T - mode
    out = torch.full((T, heads * E), float("nan"), dtype=dt, device=DEV)
    both = torch.full((T, 2 * heads * E), float("nan"), device=DEV)
    if mode == "decode":
        tables, lens = bt[None].repeat(T, 1).contiguous().to(DEV), i32(list(range(1, T + 1)))
        if path == "tc":
            po, pm = torch.empty(T * 2 * heads * splits * DP, device=DEV), torch.empty(T * 2 * heads * splits * 2, device=DEV)
            pps = max(4, -(-((T + 15) // 16) // splits))
            ops.paged_decode(qp, kc, vc, tables, lens, i32([(pps + 3) // 4 * 4]), po, pm, out, batch=T, max_splits=splits, out_d=E, exact_p=True,
                             scale=scale, diff=(lam, 1.0 - diff, eps))
            return out.view(T, heads, E)
        H.row_attention(qp.reshape(T, -1), DP, kc, vc, tables, n=T, h=2 * heads, d=2 * D, e=E, window=0, keep_first=0, scale=scale, out=both,
                        seq_lens=lens)
    else:
        n_tiles, a = chunk(mode, T)
        qc, table = qp[lo:].contiguous(), bt[None].contiguous().to(DEV)
        args = (kc, vc, table, a["tile_seq"], a["tile_q0"], a["q_start"], a["q_lens"], a["ctx_lens"], both[lo:])
        if path == "tc" and DP > 128:
            H.prefill_pages(qc, *args, n_tiles=n_tiles, scale=scale, out_d=E)
        elif path == "tc":
            ops.paged_prefill(qc, *args, n_tiles=n_tiles, out_d=E, exact_p=True, scale=scale)
        else:
            H.row_attention(qc.view(mode, -1), DP, kc, vc, table, n=n_tiles, h=2 * heads, d=2 * D, e=E, window=0, keep_first=0, scale=scale,
                            out=both[lo:], **a)
    H.diff_norm(both[lo:], T - lo, h=heads, e=E, lam=lam, gain=1.0 - diff, eps=eps, out=out[lo:])
    return out.view(T, heads, E)


@pytest.mark.parametrize("path", ["tc", "bf16", "f32"])
@pytest.mark.parametrize("heads,G,D,E,T", [(4, 2, 32, 64, 300), (3, 1, 24, 96, 270), (8, 1, 64, 128, 150), (2, 1, 12, 40, 129), (2, 1, 72, 136, 200),
                                           (5, 1, 100, 256, 140), (1, 1, 4, 20, 33)])
def test_differential_attention(H, path, heads, G, D, E, T):
    g = gen(T + D)
    q, k = b16(1.5 * torch.randn(T, heads, 2, D, generator=g)), b16(torch.randn(T, G, 2, D, generator=g))
    v = b16(torch.randn(T, G, E, generator=g))
    lam, diff, eps, scale = 0.6, 0.3, 1e-2, 1.3 * D ** -0.5
    want = oracle.differential(q.double(), k.double(), v.double(), scale, lam, diff, eps)
    for mode in ("decode", T, T // 2 + 1, 2):
        got = run_differential(H, path, q, k, v, scale, lam, diff, eps, mode)
        lo = 0 if mode == "decode" else T - mode
        assert rel(got[lo:], want[lo:]) < (3e-5 if path == "f32" else 8e-3), mode


@pytest.mark.parametrize("path", ["tc", "f32"])
def test_one_standing_out_key_of_either_map(H, path):
    """A key of one map that takes nearly all of that map's weight: far away, first, newest and at page and tile borders."""
    heads, G, D, E, T = 2, 1, 32, 48, 290
    g = gen(3)
    q, k0, v = b16(torch.randn(T, heads, 2, D, generator=g)), b16(0.1 * torch.randn(T, G, 2, D, generator=g)), b16(torch.randn(T, G, E, generator=g))
    q[:, 1] = q[:, 0]
    for i in (0, 1, 15, 16, 127, 128, 255, 256, T - 1):
        for j in {0, 1, 15, 16, 127, 128, 129, i - 1, i} & set(range(i + 1)):
            for m in (0, 1):
                k = k0.clone()
                k[j, 0, m] = b16(2.0 * q[i, 0, m])
                want = oracle.differential(q.double(), k.double(), v.double(), 0.3, 0.5, 0.2, 1e-2)
                a = oracle.causal(q[:, :, m].double(), k[:, :, m].double(), v.double(), 0.3)
                assert float((a[i, 0] - v[j, 0]).abs().max()) < 0.2       # the case is sharp
                for mode in ("decode", T):
                    got = run_differential(H, path, q, k, v, 0.3, 0.5, 0.2, 1e-2, mode)
                    assert rel(got[i], want[i]) < (3e-5 if path == "f32" else 8e-3), (i, j, m, mode)


# ---------------------------------------------------------------- latent attention
@pytest.mark.parametrize("dtype,proj_dtype,tol", [(torch.float32, torch.float32, 3e-6), (torch.bfloat16, torch.bfloat16, 6e-3),
                                                  (torch.bfloat16, torch.float32, 6e-3)])
@pytest.mark.parametrize("Q,R,T_", [(52, 72, 12), (1536, 512, 64), (8, 4, 2), (30, 33, 0)])
def test_latents_and_rotated_key_parts_go_to_the_cache(H, Q, R, T_, dtype, proj_dtype, tol):
    from oxide_tech_llm_engine_b200.models.layer_spec import RotarySpec

    g = gen(Q)
    M, col, eps = 6, (Q + 7) // 8 * 8, 1e-3
    proj = b16(torch.randn(M, col + R + T_ + 3, generator=g))
    pos = torch.tensor([0, 1, 15, 16, 777, 200000], dtype=torch.int32)
    qn, kn = 1 + 0.3 * torch.randn(Q, generator=g), 1 + 0.3 * torch.randn(R, generator=g)
    CP = (R + T_ + 15) // 16 * 16
    cache = torch.full((3, 1, 16, CP), 9.0, dtype=dtype, device=DEV)
    cq = torch.zeros(M, (Q + 63) // 64 * 64, dtype=dtype, device=DEV)
    slots = torch.tensor([0, 5, 47, 16, -1, 30])
    rot = H.Rotary(RotarySpec(T_, 1000.0, True) if T_ else None, DEV)
    H.latent_rows(proj.to(proj_dtype).to(DEV), M, q_rank=Q, q_norm=qn.to(DEV), q_out=cq, positions=pos.to(DEV), eps=eps, kv_col=col, kv_rank=R,
                  kv_norm=kn.to(DEV), cache=cache, slots=slots.to(DEV), rot=rot)
    p = proj.double()
    assert rel(cq[:, :Q], plain.rms(p[:, :Q], eps) * qn) < tol and (Q % 64 == 0 or float(cq[:, Q:].abs().max()) == 0)
    z = plain.rms(p[:, col:col + R], eps) * kn
    kr = oracle.rotate_pairs(p[:, None, col + R:col + R + T_], pos, 1000.0)[:, 0]
    flat = cache.view(48, CP)
    for t, s in enumerate(slots.tolist()):
        if s >= 0:
            assert rel(flat[s, :R], z[t]) < tol and (T_ == 0 or rel(flat[s, R:R + T_], kr[t]) < tol)
            assert R + T_ == CP or bool((flat[s, R + T_:] == 9).all())
    rest = sorted(set(range(48)) - set(slots.tolist()))
    assert bool((flat[rest] == 9).all())
    # a layer that reads another one's cache
    H.latent_rows(proj.to(proj_dtype).to(DEV), M, q_rank=Q, q_norm=qn.to(DEV), q_out=cq, positions=pos.to(DEV), eps=eps)
    assert rel(cq[:, :Q], plain.rms(p[:, :Q], eps) * qn) < tol


def latent_cache(lens, R, T_, seed, scale=1.0):
    """Shuffled pages of latents for sequences of unequal lengths; unused rows hold large values. Returns cache, tables, rows."""
    g = gen(seed)
    CP, W = (R + T_ + 15) // 16 * 16, max((n + 15) // 16 for n in lens) + 1
    perm = torch.randperm(len(lens) * W + 3, generator=g).to(torch.int32)
    cache = torch.full((len(perm), 1, 16, CP), 50.0)
    cache[..., R + T_:] = 0
    bt, rows = perm[:len(lens) * W].view(len(lens), W).contiguous(), []
    for i, n in enumerate(lens):
        z = b16(scale * torch.randn(n, R + T_, generator=g))
        for t in range(n):
            cache[int(bt[i, t // 16]), 0, t % 16, :R + T_] = z[t]
        rows.append(z)
    return cache.to(torch.bfloat16), bt.to(DEV), rows, CP


def latent_want(q, z, R, scale):
    w = torch.softmax(q.double() @ z.double().T * scale, -1)
    return w @ z[:, :R].double()


def run_latent_decode(H, q, cache, bt, lens, R, scale, splits=16):
    B, heads, CP = q.shape
    hd = (R + 7) // 8 * 8
    po, pm = (torch.full((B * heads * splits * n,), float("nan"), device=DEV) for n in (R, 2))
    out = torch.full((B, heads * hd), float("nan"), dtype=torch.bfloat16, device=DEV)
    H.latent_decode(q.to(torch.bfloat16).to(DEV), cache, bt, i32(lens), po, pm, out, rows=B, kv_rank=R, max_splits=splits, scale=scale, o_hd=hd)
    return out.view(B, heads, hd)[..., :R].cpu()


@pytest.mark.parametrize("heads,R,T_", [(16, 512, 64), (3, 72, 12), (40, 256, 32), (33, 96, 48), (1, 4, 2), (17, 160, 0), (64, 512, 64), (6, 700, 30)])
def test_decoding_against_latents_in_batches_of_unequal_lengths(H, heads, R, T_):
    lens = [1, 300, 0, 16, 17, 64, 65, 129, 1027]
    cache, bt, rows, CP = latent_cache(lens, R, T_, heads + R)
    assert H.latent_decode_heads(heads, R, CP) >= min(heads, 16)
    q = torch.zeros(len(lens), heads, CP)
    q[..., :R + T_] = b16(torch.randn(len(lens), heads, R + T_, generator=gen(R)))
    scale = 1.5 * (R + T_) ** -0.5
    for splits in (16, 3, 1):
        got = run_latent_decode(H, q, cache.to(DEV), bt, lens, R, scale, splits)
        for i, n in enumerate(lens):
            if n == 0:
                assert float(got[i].abs().max()) == 0          # a padding row
            else:
                assert rel(got[i], latent_want(q[i, :, :R + T_], rows[i], R, scale)) < 6e-3, (splits, n)


@pytest.mark.parametrize("heads,R,T_", [(5, 96, 16), (20, 512, 64), (33, 256, 32)])
def test_standing_out_latents_and_growing_scores(H, heads, R, T_):
    """One position that takes nearly everything, at page, tile and split borders; then scores that rise tile after tile by far
    more than the reference's slack, and fall again."""
    n = 400
    cache, bt, rows, CP = latent_cache([n], R, T_, 5, 0.1)
    q = torch.zeros(1, heads, CP)
    q[0, :, :R + T_] = b16(torch.randn(heads, R + T_, generator=gen(1)))
    for j in (0, 1, 15, 16, 63, 64, 65, 127, 128, 129, 191, 192, 255, 256, 383, 384, 398, 399):
        c, z = cache.clone(), rows[0].clone()
        z[j] = b16(q[0, 2, :R + T_])
        c[int(bt[0, j // 16]), 0, j % 16, :R + T_] = z[j]
        want = latent_want(q[0, :, :R + T_], z, R, 0.3)
        assert float((want[2] - z[j, :R]).abs().max()) < 0.05       # the case is sharp
        for splits in (1, 4):
            assert rel(run_latent_decode(H, q, c.to(DEV), bt, [n], R, 0.3, splits)[0], want) < 6e-3, j
        # one position less: the newest is not seen
        if j == n - 1:
            got = run_latent_decode(H, q, c.to(DEV), bt, [n - 1], R, 0.3)[0]
            assert rel(got, latent_want(q[0, :, :R + T_], z[:n - 1], R, 0.3)) < 6e-3
    for sign in (1, -1):
        z = rows[0].clone()
        ramp = torch.linspace(-40, 40, n)[:, None] * sign
        z[:, R:] = b16(ramp * torch.ones(1, T_) / T_)
        qq = q.clone()
        qq[0, :, R:R + T_] = 1.0
        c = cache.clone()
        for t in range(n):
            c[int(bt[0, t // 16]), 0, t % 16, :R + T_] = z[t]
        want = latent_want(qq[0, :, :R + T_], z, R, 1.0)
        for splits in (1, 3):
            assert rel(run_latent_decode(H, qq, c.to(DEV), bt, [n], R, 1.0, splits)[0], want) < 8e-3, sign


@pytest.mark.parametrize("dk,dv,D,E,heads", [(64, 64, 40, 48, 3), (128, 128, 80, 72, 2), (192, 128, 192, 128, 2), 
                                             (256, 256, 200, 136, 1), (256, 256, 224, 256, 2)])
def test_prompts_over_plain_rows_of_keys_and_values(H, dk, dv, D, E, heads):
    """Ragged prompts with a past: portions of several sizes, rows of other sequences and unused rows in between."""
    g = gen(dk + D)
    ctx, q_len = [300, 2, 129, 65], [300, 2, 3, 17]
    pages = [(c + 15) // 16 * 16 for c in ctx]
    row0 = np.cumsum([0] + pages[:-1]).tolist()
    kv = torch.full((sum(pages), heads * (dk + dv)), 20.0)
    M = sum(q_len)
    q = torch.zeros(M, heads, dk)
    q[..., :D] = b16(torch.randn(M, heads, D, generator=g))
    out = torch.full((M, heads * E), float("nan"), dtype=torch.bfloat16, device=DEV)
    scale, start, want = 1.4 * D ** -0.5, np.cumsum([0] + q_len[:-1]).tolist(), []
    for c, n, r, s in zip(ctx, q_len, row0, start):
        k, v = b16(torch.randn(c, heads, D, generator=g)), b16(torch.randn(c, heads, E, generator=g))
        k[0] *= 2.0            # the first position stands out
        rows = kv[r:r + c]
        rows[:] = 0
        rows[:, :heads * dk].view(c, heads, dk)[..., :D] = k
        rows[:, heads * dk:].view(c, heads, dv)[..., :E] = v
        full = torch.zeros(c, heads, D)
        full[c - n:] = q[s:s + n, :, :D]
        want.append(oracle.causal(full.double(), k.double(), v.double(), scale)[c - n:])
    tiles = [(i, t * 128) for i, n in enumerate(q_len) for t in range(-(-n // 128))]
    H.prefill_rows(q.to(torch.bfloat16).to(DEV), kv.to(torch.bfloat16).to(DEV), i32([t[0] for t in tiles]), i32([t[1] for t in tiles]), i32(start),
                   i32(q_len), i32(ctx), i32(row0), out, dk=dk, dv=dv, g=heads, n_tiles=len(tiles), scale=scale, out_d=E)
    assert H.prefill_size(D, E) == (dk, dv)
    for s, n, w in zip(start, q_len, want):
        assert rel(out[s:s + n].view(n, heads, E), w) < 6e-3, n


def test_gathered_latents(H):
    lens = [40, 16, 1, 33]
    cache, bt, rows, CP = latent_cache(lens, 24, 8, 1)
    out = torch.full((48 + 16 + 16 + 48, CP), 7.0, dtype=torch.bfloat16, device=DEV)
    row0 = [0, 48, 64, 80]
    H.latent_gather(cache.to(DEV), bt, i32(lens), i32(row0), seq0=0, n_seqs=4, max_pages=3, out=out)
    for r, n, z in zip(row0, lens, rows):
        assert rel(out[r:r + n, :32], z) == 0
    assert bool((out[40:48] == 7).all()) and bool((out[65:80] == 7).all())
    part = torch.zeros(64, CP, dtype=torch.bfloat16, device=DEV)
    H.latent_gather(cache.to(DEV), bt, i32(lens), i32([0, 0, 0, 16]), seq0=2, n_seqs=2, max_pages=3, out=part)
    assert rel(part[:1, :32], rows[2]) == 0 and rel(part[16:49, :32], rows[3]) == 0


@pytest.mark.parametrize("heads,M,N,K", [(3, 5, 40, 24), (16, 64, 512, 128), (7, 200, 72, 8), (1, 3, 64, 64), (40, 129, 64, 256)])
def test_products_per_head(heads, M, N, K):
    """Equal groups in one grouped GEMM: strided views of rows in and out."""
    from oxide_tech_llm_engine_b200 import ops

    g = gen(heads + M)
    x, w = torch.randn(M, heads, K + 16, generator=g).to(torch.bfloat16), (torch.randn(heads, N, K, generator=g) * K ** -0.5).to(torch.bfloat16)
    out = torch.full((M, heads, (N + 15) // 8 * 8), 3.0, dtype=torch.bfloat16, device=DEV)
    ops.gemm(x.to(DEV)[:, :, 8:8 + K].transpose(0, 1), w.to(DEV), out=out[:, :, :N].transpose(0, 1), bn=64)
    want = torch.einsum("mhk,hnk->mhn", x[:, :, 8:8 + K].double(), w.double())
    assert rel(out[:, :, :N], want) < 5e-3 and bool((out[:, :, N:] == 3).all())


# ---------------------------------------------------------------- matrix memory
class Memory:
    """A matrix-memory layer's inputs, run in portions."""

    def __init__(self, H, h, D, E, T, seed, proj_dtype, cap=9.0, fb=3.0):
        g = gen(seed)
        self.ops, self.h, self.D, self.E, self.T, self.cap = H, h, D, E, T, cap
        W = 2 * h * (D + E)
        self.proj = torch.zeros(T, (W + 7) // 8 * 8)
        self.proj[:, :W] = b16(torch.randn(T, W, generator=g))
        self.z = 2 * torch.randn(T, 2 * h, generator=g)
        self.z_bias = torch.cat([0.5 + torch.randn(h, generator=g), fb + 2 * torch.randn(h, generator=g)])
        self.norm = 1 + 0.3 * torch.randn(h * E, generator=g)
        self.proj_dtype = proj_dtype

    def parts(self):
        h, D, E, T = self.h, self.D, self.E, self.T
        p = self.proj.double()
        q, k, v, gate = p[:, :2 * h * (D + E)].split([h * D, h * D, h * E, h * E], 1)
        i, f = oracle.log_gates(*(self.z + self.z_bias).double().split([h, h], 1), self.cap)
        return q.view(T, h, D) * D ** -0.5, k.view(T, h, D), v.view(T, h, E), gate, i, f

    def want(self, eps=1e-5):
        q, k, v, gate, i, f = self.parts()
        o, st = oracle.mlstm(q, k, v, i, f)
        return plain.rms(o, eps).reshape(self.T, -1) * self.norm * oracle.sigmoid(gate), st

    def fresh(self, slots=4):
        """States whose old contents must not matter."""
        return (torch.full((slots, self.h, self.D * self.E + self.D), float("nan"), device=DEV),
                torch.full((slots, self.h), float("nan"), device=DEV))

    def kw(self, state):
        return dict(h=self.h, d=self.D, e=self.E, z_bias=self.z_bias.to(DEV), cap=self.cap, eps=1e-5, norm_w=self.norm.to(DEV), state=state[0],
                    state_m=state[1])

    def run(self, cuts, dtype, chunks, slot=2, state=None):
        H, T = self.ops, self.T
        proj, z = self.proj.to(self.proj_dtype).to(DEV), self.z.to(DEV)
        state = state if state is not None else self.fresh()
        out = torch.full((T, (self.h * self.E + 3) // 4 * 4), float("nan"), dtype=dtype, device=DEV)
        at, cuts = 0, list(cuts)
        while at < T:
            n = min(cuts.pop(0) if cuts else T - at, T - at)
            kw = dict(z=z[at:at + n], out=out[at:at + n], **self.kw(state))
            if n == 1:
                H.memory_decode(proj[at:at + 1], 1, row_slots=i32([slot]), positions=i32([at]), **kw)
            else:
                tiles, a = chunk(n, at + n)
                size = H.memory_ws_elems(self.h, self.D, self.E, tiles) if chunks else n * self.h * self.E + self.h * (self.D + 1)
                H.memory_prefill(proj[at:at + n], n, seq_slots=i32([slot]), n_tiles=tiles, n_seqs=1, chunks=chunks,
                                 ws=torch.full((size,), float("nan"), device=DEV), **a, **kw)
            at += n
        return out[:, :self.h * self.E], state

    def state_error(self, state, slot, want):
        S, n, m = want
        st = state[0][slot].cpu()
        return max(rel(st[:, :self.D * self.E].view(self.h, self.D, self.E), S), rel(st[:, self.D * self.E:], n), rel(state[1][slot], m))


@pytest.mark.parametrize("form", ["chunks", "chunks-f32-rows", "scan-bf16", "scan-f32"])
@pytest.mark.parametrize("h,D,E,T", [(2, 64, 128, 330), (3, 40, 56, 300), (1, 4, 12, 140), (2, 32, 272, 200), (1, 256, 512, 150), (3, 7, 5, 150),
                                     (4, 24, 20, 260)])
def test_memory_in_portions_equals_the_recurrence(H, form, h, D, E, T):
    f32 = form == "scan-f32"
    s = Memory(H, h, D, E, T, h * E + D, torch.float32 if (f32 or form == "chunks-f32-rows") else torch.bfloat16)
    want, st_want = s.want()
    dt = torch.float32 if f32 else torch.bfloat16
    for cuts in ([], [2, 3, 1, 1, 64, 1, 65], [128, 1, 1, 2], [1] * 12 + [7, 63], [130, 2]):
        got, st = s.run(cuts, dt, not form.startswith("scan"))
        assert rel(got, want) < (2e-5 if f32 else 6e-3), cuts
        assert s.state_error(st, 2, st_want) < 2e-5, cuts                 # 32-bit in every form
        assert all(bool(torch.isnan(x[[0, 1, 3]]).all()) for x in st)     # nobody else's slot


def test_decode_rows_take_their_gates_from_the_rows(H):
    h, D, E, N, rows = 3, 24, 40, 192, 5
    s = Memory(H, h, D, E, rows, 4, torch.bfloat16)
    g = gen(9)
    hid, w = torch.randn(rows, N, generator=g).to(torch.bfloat16), (2 * N ** -0.5 * torch.randn(64, N, generator=g)).to(torch.bfloat16)
    s.z = (hid.double() @ w.double().T)[:, :2 * h].float()
    q, k, v, gate, i, f = s.parts()
    st = (torch.zeros(8, h, D * E + D, device=DEV), torch.full((8, h), 5.0, device=DEV))
    out = torch.full((rows, h * E), 7.0, dtype=torch.bfloat16, device=DEV)
    H.memory_decode(s.proj.to(torch.bfloat16).to(DEV), rows, hidden=hid.to(DEV), z_w=w.to(DEV), row_slots=i32([1, 0, -1, 7, 4]),
                    positions=i32([0, 0, 0, 0, 0]), out=out, **s.kw(st))
    for r in (0, 1, 3, 4):       # each row alone, from the zero state and a maximum of 0
        o, _ = oracle.mlstm(*(x[r:r + 1] for x in (q, k, v, i, f)))
        want = plain.rms(o, 1e-5).reshape(1, -1) * s.norm * oracle.sigmoid(gate[r:r + 1])
        assert rel(out[r:r + 1], want) < 6e-3
    assert bool((out[2] == 7).all()) and bool((st[1][[2, 3, 5, 6]] == 5).all())


@pytest.mark.parametrize("cap", [0.5, 15.0, 80.0])
def test_gates_of_every_size(H, cap):
    """Input gates from exp(-cap) to exp(cap), forget gates that keep nothing and everything; the maximum goes up and down."""
    h, D, E, T = 4, 16, 32, 300
    s = Memory(H, h, D, E, T, 5, torch.bfloat16, cap=cap)
    s.z = s.z * torch.tensor([1.0, 20.0, 200.0, 5.0] * 2)
    s.z_bias = torch.tensor([-30.0, 0.0, 0.0, 30.0, 0.0, 20.0, -3.0, 60.0])
    want, st_want = s.want()
    for cuts in ([], [100, 1, 1, 64, 2]):
        got, st = s.run(cuts, torch.bfloat16, True)
        assert rel(got, want) < 8e-3 and s.state_error(st, 2, st_want) < 1e-4
        got, st = s.run(cuts, torch.bfloat16, False)
        assert rel(got, want) < 8e-3 and s.state_error(st, 2, st_want) < 1e-4


def test_a_token_far_back_decides_the_read_out(H):
    """One token with an input gate that stands out, memories that keep it, and a query for it hundreds of tokens later."""
    h, D, E, T = 2, 64, 48, 700
    s = Memory(H, h, D, E, T, 9, torch.bfloat16, cap=15.0)
    s.z[:] = 0
    s.z_bias = torch.tensor([-4.0] * h + [14.0] * h)
    s.z[3, :h] = 12.0
    s.proj[T - 1, :h * D] = s.proj[3, h * D:2 * h * D]                    # the query is that token's key
    want, _ = s.want()
    q, k, v, gate, i, f = s.parts()
    lone = plain.rms(v[3], 1e-5).reshape(1, -1) * s.norm * oracle.sigmoid(gate[T - 1:])
    assert rel(want[T - 1:], lone) < 0.1                                  # it does decide
    for cuts in ([], [600] + [1] * 100, [4, 90, 2, 300, 64, 2]):
        got, _ = s.run(cuts, torch.bfloat16, True)
        assert rel(got[T - 1], want[T - 1]) < 6e-3, cuts


def test_ragged_batch_of_chunks_and_decode_rows_keeps_memories_apart(H):
    """Sequences of unequal lengths in one launch, some with a past, then decode rows beside a padding row; slots used again."""
    h, D, E = 2, 40, 48
    lens, pasts, slots = [130, 2, 64, 65, 300, 1], [0, 70, 0, 3, 0, 5], [4, 0, 6, 2, 1, 5]
    seqs = [Memory(H, h, D, E, n + p + 1, 10 * i, torch.bfloat16) for i, (n, p) in enumerate(zip(lens, pasts))]
    for s in seqs[1:]:
        s.z_bias, s.norm = seqs[0].z_bias, seqs[0].norm
    state = seqs[0].fresh(7)
    for s, p, sl in zip(seqs, pasts, slots):
        if p:                                                             # what came before, on its own
            full = s.T, s.proj, s.z
            s.T, s.proj, s.z = p, s.proj[:p], s.z[:p]
            s.run([], torch.bfloat16, True, slot=sl, state=state)
            s.T, s.proj, s.z = full
    rows = torch.cat([s.proj[p:p + n] for s, n, p in zip(seqs, lens, pasts)]).to(torch.bfloat16).to(DEV)
    z = torch.cat([s.z[p:p + n] for s, n, p in zip(seqs, lens, pasts)]).to(DEV)
    M, start = rows.shape[0], np.cumsum([0] + lens[:-1]).tolist()
    tiles = [(i, t * 128) for i, n in enumerate(lens) for t in range(-(-n // 128))]
    for chunks in (True, False):
        st = tuple(t.clone() for t in state)
        out = torch.zeros(M, h * E, dtype=torch.bfloat16, device=DEV)
        n_ws = H.memory_ws_elems(h, D, E, len(tiles)) if chunks else M * h * E + len(lens) * h * (D + 1)
        H.memory_prefill(rows, M, z=z, seq_slots=i32(slots), tile_seq=i32([t[0] for t in tiles]), tile_q0=i32([t[1] for t in tiles]),
                         q_start=i32(start), q_lens=i32(lens), ctx_lens=i32([n + p for n, p in zip(lens, pasts)]), n_tiles=len(tiles),
                         n_seqs=len(lens), ws=torch.empty(n_ws, device=DEV), chunks=chunks, out=out, **seqs[0].kw(st))
        for s, n, p, a in zip(seqs, lens, pasts, start):
            assert rel(out[a:a + n], s.want()[0][p:p + n]) < 6e-3, (chunks, n)
        assert bool(torch.isnan(st[0][3]).all())
        # one more token each, in one decode step; row 2 is padding, row 4 starts afresh in a used slot
        order = [3, 0, None, 5, None]
        pick = lambda t: torch.stack([t(seqs[i])[-1] if i is not None else t(seqs[1])[0] for i in order])
        rs, ps = [slots[i] if i is not None else -1 for i in order], [seqs[i].T - 1 if i is not None else 9 for i in order]
        rs[4], ps[4] = slots[2], 0
        o = torch.full((5, h * E), 7.0, dtype=torch.bfloat16, device=DEV)
        H.memory_decode(pick(lambda s: s.proj).to(torch.bfloat16).to(DEV), 5, z=pick(lambda s: s.z).to(DEV), row_slots=i32(rs), positions=i32(ps),
                        out=o, **seqs[0].kw(st))
        for r, i in enumerate(order):
            if i is not None:
                assert rel(o[r], seqs[i].want()[0][-1]) < 6e-3, r
        assert rel(o[4], seqs[1].want()[0][0]) < 6e-3 and bool((o[2] == 7).all())


# ---------------------------------------------------------------- experts
@pytest.mark.parametrize("mode,dtype", [("pairs", torch.float32), ("slab", torch.bfloat16), ("packed", torch.bfloat16)])
@pytest.mark.parametrize("M,E,top,groups,keep,N", [(7, 15, 2, 5, 2, 64), (100, 64, 6, 8, 4, 192), (128, 12, 1, 3, 1, 76), (64, 8, 3, 0, 0, 64),
                                                   (90, 512, 9, 32, 5, 256), (33, 4, 2, 4, 3, 64), (300, 66, 5, 6, 3, 96), (20, 1, 1, 1, 1, 64)])
def test_router_with_groups(H, M, E, top, groups, keep, N, mode, dtype):
    from oxide_tech_llm_engine_b200 import ops

    if mode == "slab":
        M = min(M, 128)
    g = gen(M + E)
    h, rw = torch.zeros(M, (N + 63) // 64 * 64), torch.zeros((E + 63) // 64 * 64, (N + 63) // 64 * 64)
    h[:, :N], rw[:E, :N] = torch.randn(M, N, generator=g), torch.randn(E, N, generator=g) * 2 * N ** -0.5
    h, rw = h.to(dtype), rw.to(dtype)
    hd, rd = h.to(DEV), rw.to(DEV)
    wt, ex, sl, cnt = torch.zeros(M * top, device=DEV), i32([0] * (M * top)), i32([0] * (M * top)), i32([0] * E)
    kw = dict(e=E, top=top, weight=wt, expert=ex, slot=sl, softmax=False, groups=groups, keep=keep)
    xs = torch.zeros(max(E * 128, (M * top + 127 * E) // 128 * 128), h.shape[1], dtype=dtype, device=DEV)
    if mode == "packed":
        lg = torch.zeros(M, rw.shape[0], device=DEV)
        ops.gemm(hd, rd, out=lg, epi=ops.EPI_STORE_F32)
        H.moe_route(hd, rd[:E], M, mode=2, logits=lg, counts=cnt, **kw)
        H.moe_scatter(hd, M, e=E, top=top, expert=ex, slot=sl, counts=cnt, xs=xs)
    else:
        H.moe_route(hd, rd[:E], M, mode=1 if mode == "slab" else 0, counts=cnt if mode == "slab" else None, xs=xs if mode == "slab" else None, **kw)
    z = h.double() @ rw[:E].double().T
    gr = {"count": groups, "keep": keep} if groups else None
    ids, v = oracle.choose(z, top, gr)
    clear = oracle.margin(z, top, gr) > 1e-4
    got, w = ex.view(M, top).cpu().long(), wt.view(M, top).cpu()
    assert float(clear.float().mean()) > 0.9
    assert torch.equal(got.sort(-1).values[clear], ids.sort(-1).values[clear])
    assert rel(w, torch.sigmoid(z).gather(1, got)) < 5e-5                 # the scores themselves, not divided by their sum
    if mode != "pairs":
        s = sl.view(M, top).cpu().long()
        assert torch.equal(torch.bincount(got.flatten(), minlength=E), cnt.cpu().long())
        assert all(torch.equal(xs[s[:, k].to(DEV)], hd) for k in range(top))


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 3e-6), (torch.bfloat16, 8e-3)])
@pytest.mark.parametrize("pairs,top,E,F,K", [(4, 2, 5, 64, 64), (9, 3, 7, 192, 128), (6, 6, 64, 1408, 2048)])
def test_gated_experts_of_single_rows(H, pairs, top, E, F, K, dtype, tol):
    from oxide_tech_llm_engine_b200.models.llama import interleave32

    g = gen(F)
    gate, up = ((torch.randn(E, F, K, generator=g) * K ** -0.5).to(dtype) for _ in range(2))
    w = torch.stack([interleave32(a, b) for a, b in zip(gate, up)]).contiguous()
    x = torch.randn(pairs // top, K, generator=g).to(dtype)
    ex = torch.randint(0, E, (pairs,), generator=g, dtype=torch.int32)
    y = torch.zeros(pairs, F + 8, dtype=dtype, device=DEV)
    H.moe_rows(x.to(DEV), w.to(DEV), ex.to(DEV), pairs, top=top, per_pair=False, y=y, act=3)
    want = torch.stack([oracle.silu(gate[ex[i]].double() @ x[i // top].double()) * (up[ex[i]].double() @ x[i // top].double()) for i in range(pairs)])
    assert rel(y[:, :F], want) < tol and float(y[:, F:].abs().max()) == 0


@pytest.mark.parametrize("mode", ["slab", "packed"])
@pytest.mark.parametrize("E,F,K,bn", [(5, 64, 64, 64), (9, 192, 320, 128), (70, 128, 128, 256)])
def test_gated_expert_products_of_unequal_groups(mode, E, F, K, bn):
    from oxide_tech_llm_engine_b200 import ops
    from oxide_tech_llm_engine_b200.models.llama import interleave32

    g = gen(E * F)
    sizes = [0, 1, 128, 5, 0, 127, 300, 129, 0]
    counts = [(sizes[i % 9] if mode == "packed" else min(128, sizes[i % 9])) for i in range(E)]
    first = np.cumsum([0] + [(c + 127) // 128 * 128 for c in counts]) if mode == "packed" else np.arange(E + 1) * 128
    gate, up = ((torch.randn(E, F, K, generator=g) * K ** -0.5).to(torch.bfloat16) for _ in range(2))
    w = torch.stack([interleave32(a, b) for a, b in zip(gate, up)]).contiguous()
    x = torch.randn(max(128, int(first[-1])), K, generator=g).to(torch.bfloat16)
    m_tiles = min(max(1, sum((c + 127) // 128 for c in counts)) if mode == "packed" else E, x.shape[0] // 128)
    out = torch.full((x.shape[0], F), 3.0, dtype=torch.bfloat16, device=DEV)
    xd, od = x.to(DEV), out
    if mode == "slab":
        xd, od = xd.view(E, 128, K), od.view(E, 128, F)
    ops.gemm(xd, w.to(DEV), out=od, epi=ops.EPI_SWIGLU_BF16, group_counts=i32(counts), m_tiles=m_tiles, bn=bn)
    for e, c in enumerate(counts):
        a, end = int(first[e]), int(first[e + 1])
        r = x[a:a + c].double()
        if c:
            assert rel(out[a:a + c], oracle.silu(r @ gate[e].double().T) * (r @ up[e].double().T)) < 8e-3, (e, c)
        assert bool((out[a + c:end] == 3).all())                           # rows past the group stay untouched


# ---------------------------------------------------------------- whole models
def toks(n, vocab, seed=0):
    return np.random.default_rng(seed).integers(0, vocab, size=n).tolist()


def row_errors(got, want):
    return np.array([hm.error(got[i:i + 1], want[i:i + 1]) for i in range(len(want))])


def rounding(c, w, t, draws=4):
    """How far 16-bit storage of what enters the products moves each row of logits: the plain implementation with relative
    noise of that size on the normed rows, queries, keys, values, read-outs and activations; the largest of a few draws."""
    names = ("rms", "causal", "mlstm", "silu", "gelu_tanh")
    kept, want, worst = {n: getattr(oracle, n) for n in names}, oracle.forward(c, w, t).numpy(), 0.0
    for seed in range(draws):
        g = gen(seed)
        noisy = lambda x: x * (1 + 2.0 ** -9 * (2 * torch.rand(x.shape, generator=g, dtype=x.dtype) - 1))
        try:
            oracle.rms = lambda x, eps: noisy(kept["rms"](noisy(x), eps))
            oracle.causal = lambda q, k, v, scale: noisy(kept["causal"](noisy(q), noisy(k), noisy(v), scale))
            oracle.mlstm = lambda q, k, v, i, f: (noisy(kept["mlstm"](noisy(q), noisy(k), noisy(v), i, f)[0]), None)
            oracle.silu, oracle.gelu_tanh = lambda z: noisy(kept["silu"](noisy(z))), lambda z: noisy(kept["gelu_tanh"](noisy(z)))
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
        limit = 2e-4 if self.dtype == "float32" else 0.01 + 4 * self.noise[at]
        return [(i, float(e[i])) for i in np.flatnonzero(e > limit)]


def clear_tokens(c, w, n, seed, gap):
    """A sequence in which no router's choice is close enough for 16-bit rounding to turn it: the tokens of a longer one
    that are clear, until all are."""
    t = toks(n, c["vocab"], seed)
    while True:
        m: list = []
        oracle.forward(c, w, t, margins=m)
        ok = (torch.stack(m).min(0).values > gap).tolist() if m else [True] * len(t)
        if all(ok):
            return t
        t = [a for a, b in zip(t, ok) if b]


@pytest.mark.parametrize("name", list(zm.CONFIGS))
def test_prompts_portions_and_batches_equal_the_plain_implementation(name):
    c = zm.CONFIGS[name]
    w = zm.weights(c, 2)
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


@pytest.mark.parametrize("name", list(zm.CONFIGS))
def test_bf16_prompts_portions_and_batches_with_experts(name):
    """Sequences whose experts are clear: everything that is cut from the front of one is clear as well."""
    c = zm.CONFIGS[name]
    w = zm.weights(c, 2)
    t = clear_tokens(c, w, 330, 1, 0.004 if name == "wide" else 0.015)      # many experts: closer scores
    x = Expected(c, w, t, "bfloat16")
    assert len(t) >= 8 and np.median(x.noise) < 0.03
    eng = hm.engine(c, w, live=3, blocks=80)
    for cuts in ([], [2, 3, 1, 1, 17, 2, 64], [1] * 30):
        assert not x.wrong(hm.feed_all(eng, 0, t, cuts)), cuts
    lens = [len(t), 1, len(t) // 2, 2, len(t) - 1, 5]
    for seed in (1, 2):
        for got, n in zip(hm.interleaved(eng, [t[:n] for n in lens], seed), lens):
            assert not x.wrong(got, slice(0, n))
    eng.close()


def without_experts(c):
    """The same layers with dense feed-forwards: no choice that rounding could turn."""
    c = json.loads(json.dumps(c))
    for L in c["layers"]:
        if L["mlp"]:
            L["mlp"] = {"kind": "dense", "ff": 56}
    return c


@pytest.mark.parametrize("name", list(zm.CONFIGS))
def test_bf16_rows_of_models_without_experts(name):
    """bf16 kernels sharply, over whole prompts, portions, batches and long decoding."""
    c = without_experts(zm.CONFIGS[name])
    w = zm.weights(c, 3)
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
    c = zm.CONFIGS["mixed"] if dtype == "float32" else without_experts(zm.CONFIGS["mixed"])
    w = zm.weights(c, 2)
    eng = hm.engine(c, w, dtype=dtype, live=2, blocks=48)
    t = toks(300, c["vocab"], 5)
    assert not Expected(c, w, t, dtype).wrong(hm.feed_all(eng, 0, t, [1] * 300))
    assert eng.stats["graph_replays"] > 250
    eng.close()


def test_prompts_whose_contexts_take_several_passes(monkeypatch):
    from oxide_tech_llm_engine_b200.models import hybrid

    monkeypatch.setattr(hybrid, "KV_PASS_ROWS", 96)
    c = without_experts(zm.CONFIGS["wide"])
    w = zm.weights(c, 5)
    eng = hm.engine(c, w, live=4, blocks=96)
    seqs = [toks(n, c["vocab"], n) for n in (150, 40, 33, 250)]
    first = eng.feed([(i, t[:n], [n - 1]) for i, (t, n) in enumerate(zip(seqs, (100, 20, 30, 130)))])
    rest = eng.feed([(i, t[n:], [len(t) - n - 1]) for i, (t, n) in enumerate(zip(seqs, (100, 20, 30, 130)))])
    for i, (t, n) in enumerate(zip(seqs, (100, 20, 30, 130))):
        x = Expected(c, w, t, "bfloat16")
        assert not x.wrong(first[i:i + 1], [n - 1]) and not x.wrong(rest[i:i + 1], [len(t) - 1])
    eng.close()


def test_layer_outputs_follow_every_layer():
    c = zm.CONFIGS["mixed"]
    w = zm.weights(c, 2)
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
@pytest.mark.parametrize("name", ["mixed", "ones", "wide"])
def test_greedy_generation_through_the_engine(name, burst):
    """32-bit, so that the tokens are the plain implementation's: chunked prompts, a pool and slots that are short, graph
    replays, decode bursts."""
    c = zm.CONFIGS[name]
    w = zm.weights(c, 4)
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
    c = without_experts(zm.CONFIGS["mixed"])
    w = zm.weights(c, 4)
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
    c = without_experts(zm.CONFIGS["mixed"]) if dtype == "bfloat16" else zm.CONFIGS["mixed"]
    w = zm.weights(c, 6)
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
