"""Python front-ends of the layer-list kernels (``csrc/kernels/{stream_ops,mixer_ops,attn_rows,retention,ssd,moe_ops,latent,latent_decode,memory,
attn_prefill_wide,talking,gru}.cu``).

Activations, weights and caches are bf16, or fp32 throughout; residual streams, states, norms, scores
and angles are fp32 in both cases. As in `ops`, nothing here falls back to PyTorch.
"""
from __future__ import annotations

from typing import Optional

import torch

from .. import ops
from .._build import hybrid_ext


class Rotary:
    """Device frequencies of a layer_spec.RotarySpec, each as the sum of two fp32 numbers, and the factor on sin and cos."""

    def __init__(self, spec, device):
        self.interleaved = bool(spec is not None and spec.interleaved)
        self.hi = self.lo = None
        self.gain = 1.0
        if spec is not None and spec.dims > 0:
            freqs, self.gain = spec.frequencies()
            f = torch.tensor(freqs, dtype=torch.float64)
            hi = f.to(torch.float32)
            self.hi = hi.to(device)
            self.lo = (f - hi.to(torch.float64)).to(torch.float32).to(device)


def retention_chunk() -> int:
    return int(hybrid_ext().RETENTION_CHUNK)


def max_streams() -> int:
    return int(hybrid_ext().MAX_STREAMS)


def retention_chunks_ok(d: int, e: int) -> bool:
    return bool(hybrid_ext().retention_chunks_ok(d, e))


def set_pdl(on: bool) -> None:
    hybrid_ext().set_pdl(bool(on))


def decay_powers(decay, device) -> torch.Tensor:
    """[heads, chunk + 1] fp32: decay^0 .. decay^chunk, each rounded once."""
    d = torch.tensor([float(x) for x in decay], dtype=torch.float64)
    n = torch.arange(retention_chunk() + 1, dtype=torch.float64)
    return torch.pow(d[:, None], n[None, :]).to(torch.float32).to(device).contiguous()


def stream_norm(x: torch.Tensor, rows: int, *, norm_w: torch.Tensor, eps: float, h: torch.Tensor, w_offset: float = 1.0,
                tokens=None, prev=None, embed=None, bigram=None, mul_prev: int = 0, mul_cur: int = 0,
                y: Optional[torch.Tensor] = None, zero_y: bool = True, mix=None, out_w=None, in_w=None,
                store_x: bool = True, row_map=None, clear=None) -> None:
    """Embedding or hyper-connection update of the residual streams x [M, S, N], read-out for the next
    sublayer and its RMS norm (StreamNormParams in csrc/kernels/hybrid.cuh). `clear`: fp32 rows zeroed on
    the way, the accumulator of the split-K GEMM that follows."""
    hybrid_ext().stream_norm(x, rows, tokens, prev, embed, bigram, mul_prev, mul_cur, y, zero_y, mix, out_w, in_w, store_x,
                             norm_w, eps, w_offset, h, row_map, clear, ops.status_word(x.device))
    ops._bump()


def heads(proj: torch.Tensor, m: int, *, h: int, g: int, d: int, e: int, rot: Rotary, positions, q_out, q_hd: int,
          q_norm=None, k_norm=None, eps: float = 1e-5, k_scale: float = 1.0, k_out=None, k_cache=None, v_cache=None,
          slots=None, q_pd: int = 0, maps: int = 1, bias=None, temp_coef: float = 0.0, temp_every: float = 1.0,
          k_rms=None) -> None:
    """Projection rows q | k | v -> normed and rotated heads; k and v into the paged cache with q [M, h * q_hd], or
    q and k to dense fp32 buffers [heads, M, d]; g = 0: queries only, q_pd columns apart (HeadsParams). `k_rms`: keys that are
    values, the cache takes them as they are and k_rms [blocks, 16] their norm's factor."""
    hybrid_ext().heads(proj, m, h, g, d, e, q_norm, k_norm, eps, rot.hi, rot.lo, rot.interleaved, rot.gain, positions,
                       k_scale, q_out, q_hd, k_out, k_cache, v_cache, slots, q_pd, maps, bias, temp_coef, temp_every, k_rms,
                       ops.status_word(proj.device))
    ops._bump()


def diff_norm(a, m: int, *, h: int, e: int, lam: float, gain: float, eps: float, out) -> None:
    """The two maps of every head (fp32, side by side) -> a1 - lam a2, divided by its root mean square, times gain."""
    hybrid_ext().diff_norm(a, m, h, e, lam, gain, eps, out)
    ops._bump()


def latent_rows(proj, m: int, *, q_rank: int, q_norm, q_out, positions, eps: float, kv_col: int = 0, kv_rank: int = 0, kv_norm=None,
                cache=None, slots=None, rot: Optional[Rotary] = None) -> None:
    """Normed query latent of every row; with kv_rank > 0 also the normed latent and the rotated key part into the
    paged cache [blocks, 1, 16, values] (LatentRowsParams)."""
    r = rot if rot is not None else Rotary(None, proj.device)
    hybrid_ext().latent_rows(proj, m, q_rank, q_norm, q_out, kv_col, kv_rank, kv_norm, cache, slots, r.hi, r.lo, r.interleaved,
                             r.gain, positions, eps, ops.status_word(proj.device))
    ops._bump()


def latent_gather(cache, block_tables, ctx_lens, row0, *, seq0: int, n_seqs: int, max_pages: int, out) -> None:
    """Cache rows of sequences seq0 .. in order of position, from row0[sequence] on."""
    hybrid_ext().latent_gather(cache, block_tables, ctx_lens, row0, seq0, n_seqs, max_pages, out, ops.status_word(cache.device))
    ops._bump()


def latent_decode_heads(heads: int, kv_rank: int, row: int) -> int:
    """Heads that one CTA of the decode kernel takes; 0: latents that it has no room for."""
    return int(hybrid_ext().latent_decode_heads(heads, kv_rank, row))


def latent_decode(q, cache, block_tables, seq_lens, part_o, part_ml, out, *, rows: int, kv_rank: int,
                  max_splits: int, scale: float, o_hd: int) -> None:
    """Decode rows of latent attention against the cached latents (split-KV and merge)."""
    hybrid_ext().latent_decode(q, cache, block_tables, seq_lens, rows, kv_rank, max_splits, scale, part_o, part_ml,
                               out, o_hd, ops.status_word(q.device))
    ops._bump(2)


PREFILL_SIZES = ((64, 64), (128, 128), (192, 128), (256, 256))   # (keys, values) of prefill_rows and prefill_pages


def prefill_size(dk: int, dv: int) -> Optional[tuple]:
    """Smallest built head sizes that hold keys of dk and values of dv."""
    return next((z for z in PREFILL_SIZES if z[0] >= dk and z[1] >= dv), None)


def prefill_rows(q, kv, tile_seq, tile_q0, q_start, q_lens, ctx_lens, row0, out, *, dk: int, dv: int, g: int, n_tiles: int,
                 scale: float, out_d: int) -> None:
    """Causal attention of prompt tiles over plain rows of keys (g heads of dk columns) and values (behind them)."""
    hybrid_ext().prefill_rows(q, kv, dk, dv, g * dk, g, row0, tile_seq, tile_q0, q_start, q_lens, ctx_lens, out, n_tiles, scale, out_d,
                              ops.status_word(q.device))
    ops._bump()


def prefill_pages(q, k_cache, v_cache, block_tables, tile_seq, tile_q0, q_start, q_lens, ctx_lens, out, *, n_tiles: int, scale: float,
                  out_d: int) -> None:
    """Causal attention of prompt tiles over the paged cache, heads of up to 256 values."""
    hybrid_ext().prefill_pages(q, k_cache, v_cache, block_tables, tile_seq, tile_q0, q_start, q_lens, ctx_lens, out, n_tiles, scale, out_d,
                               ops.status_word(q.device))
    ops._bump()


def memory_chunk() -> int:
    return int(hybrid_ext().MEMORY_CHUNK)


def memory_chunks_ok(d: int, e: int) -> bool:
    return bool(hybrid_ext().memory_chunks_ok(d, e))


def memory_ws_elems(h: int, d: int, e: int, n_tiles: int) -> int:
    return 2 * n_tiles * h * (d * e + d + 3)


def memory_decode(proj, rows: int, *, h: int, d: int, e: int, z_bias, cap: float, eps: float, norm_w, state, state_m, row_slots,
                  positions, out, z=None, hidden=None, z_w=None) -> None:
    """Matrix memory, one token per row: gates (from pre-activations `z`, or from the rows and the gate weights), state
    update, read-out, head norm and gate in one launch."""
    hybrid_ext().memory_decode(proj, rows, h, d, e, z, hidden, z_w, z_bias, cap, eps, norm_w, state, state_m, row_slots, positions,
                               out, ops.status_word(proj.device))
    ops._bump()


def memory_prefill(proj, m: int, *, h: int, d: int, e: int, z, z_bias, cap: float, eps: float, norm_w, state, state_m, seq_slots,
                   tile_seq, tile_q0, q_start, q_lens, ctx_lens, n_tiles: int, n_seqs: int, ws, chunks: bool, out) -> None:
    """Prompt chunks: the chunked tensor-core form, or token by token."""
    hybrid_ext().memory_prefill(proj, m, h, d, e, z, z_bias, cap, eps, norm_w, state, state_m, seq_slots, tile_seq, tile_q0, q_start,
                                q_lens, ctx_lens, n_tiles, n_seqs, ws, chunks, out, ops.status_word(proj.device))
    ops._bump(3 if chunks else 2)


def row_attention(q, q_hd: int, k_cache, v_cache, block_tables, *, n: int, h: int, d: int, e: int, window: int,
                  keep_first: int, scale: float, out, chunk: int = 0, sink: float = float("-inf"), seq_lens=None,
                  tile_seq=None, tile_q0=None, q_start=None, q_lens=None, ctx_lens=None, o_hd: int = 0, sinks=None,
                  out_gain: float = 1.0) -> None:
    """Softmax attention of any head size in fp32 FMAs: decode rows (seq_lens) or prompt tiles."""
    hybrid_ext().row_attention(q, q_hd, k_cache, v_cache, block_tables, seq_lens, tile_seq, tile_q0, q_start, q_lens,
                               ctx_lens, n, h, d, e, window, keep_first, chunk, scale, sink, sinks, out_gain, out, o_hd,
                               ops.status_word(q.device))
    ops._bump()


def retention_decode(proj, rows: int, *, h: int, d: int, e: int, decay_pow, rot: Rotary, k_scale: float, eps: float, state,
                     row_slots, positions, out) -> None:
    """One token per row: rotation, state update, read-out, head norm and gate in one launch."""
    hybrid_ext().retention_decode(proj, rows, h, d, e, decay_pow, rot.hi, rot.lo, rot.interleaved, rot.gain, k_scale, eps,
                                  state, row_slots, positions, out, ops.status_word(proj.device))
    ops._bump()


def retention_prefill(proj, m: int, *, h: int, d: int, e: int, decay_pow, eps: float, state, seq_slots, tile_seq, tile_q0,
                      q_start, q_lens, ctx_lens, n_tiles: int, n_seqs: int, q_rot, k_rot, out, ws=None, o_buf=None) -> None:
    """Prompt chunks: the chunked tensor-core form with a workspace `ws`, else token by token."""
    hybrid_ext().retention_prefill(proj, m, h, d, e, decay_pow, eps, state, seq_slots, tile_seq, tile_q0, q_start, q_lens,
                                   ctx_lens, n_tiles, n_seqs, q_rot, k_rot, ws, o_buf, out, ops.status_word(proj.device))
    ops._bump(3 if ws is not None else 2)


def ssd_chunks_ok(n: int) -> bool:
    return bool(hybrid_ext().ssd_chunks_ok(n))


def ssd_segment(h: int, ep: int, n_tiles: int, n_seqs: int) -> int:
    """Rows per segment for a step of so many tiles and sequences; 0: sequences are walked whole."""
    return int(hybrid_ext().ssd_segment(h, ep, n_tiles, n_seqs))


def ssd_ws_elems(h: int, ep: int, np_: int, n_tiles: int) -> int:
    return n_tiles * h * (np_ * ep + 1)


def max_experts() -> tuple[int, int]:
    """Largest number of experts, and of chosen ones."""
    ext = hybrid_ext()
    return int(ext.MAX_EXPERTS), int(ext.MAX_TOP)


def max_groups() -> int:
    return int(hybrid_ext().MAX_GROUPS)


def branch_norm(x: torch.Tensor, rows: int, *, norm_w, h, eps: float, w_offset: float = 0.0, tokens=None, embed=None,
                embed_scale: float = 1.0, branches=(), experts=None, store_x: bool = True, row_map=None, clear=None, base=None,
                split=None, split_off: int = 0, x0_tokens=None) -> None:
    """Embedding or the sum of a layer's branches into the residual stream x [M, N], and its RMS norm with one weight per
    output (BranchNormParams in csrc/kernels/hybrid.cuh). `branches`: (fp32 rows, norm weight or None, gain, clear);
    `experts`: (rows, slots, weights, chosen per row); a branch whose rows are None is their weighted sum. `base`: the branches
    are added to this vector instead of the stream. `split` (instead of h): operand rows of a product over [x; embedding]."""
    rows_e, slot, weight, top = experts if experts is not None else (None, None, None, 0)
    hybrid_ext().branch_norm(x, rows, tokens, embed, embed_scale, [b[0] for b in branches], [b[1] for b in branches],
                             [b[2] for b in branches], [bool(b[3]) for b in branches], rows_e, slot, weight, top, store_x,
                             list(norm_w), list(h), eps, w_offset, row_map, clear, base, split, split_off, x0_tokens,
                             ops.status_word(x.device))
    ops._bump()


def ssd_decode(proj, rows: int, *, h: int, g: int, w, state, conv_state, row_slots, positions, y) -> None:
    """State-space layer, one token per row: convolution, step size, state update and read-out in one launch. `w`:
    (conv, conv bias, dt_bias, A_log, D) in fp32."""
    hybrid_ext().ssd_decode(proj, rows, h, g, list(w), state, conv_state, row_slots, positions, y, ops.status_word(proj.device))
    ops._bump()


def ssd_prefill(proj, m: int, *, h: int, g: int, w, state, conv_state, seq_slots, tile_seq, tile_q0, q_start, q_lens, ctx_lens,
                n_tiles: int, n_seqs: int, u, y, runs: bool, segment: int = 0, ws=None) -> None:
    """Prompt chunks: convolution into `u`, then runs of 64 tokens on tensor cores (`runs`) or token by token. `segment` (see
    ssd_segment): rows of a sequence that are walked in one piece, with `ws` for the states between the pieces."""
    hybrid_ext().ssd_prefill(proj, m, h, g, list(w), state, conv_state, seq_slots, tile_seq, tile_q0, q_start, q_lens, ctx_lens,
                             n_tiles, n_seqs, u, y, runs, segment, ws, ops.status_word(proj.device))
    ops._bump(4 if segment else 2)


def gated_norm(y, z, m: int, *, h: int, e: int, ep: int, groups: int, w, eps: float, out) -> None:
    """out = (y * silu(z)) normalised in `groups` equal parts, times w; heads of e values lie ep apart in y and z."""
    hybrid_ext().gated_norm(y, z, m, h, e, ep, groups, w, eps, out)
    ops._bump()


def moe_route(h, router, m: int, *, e: int, top: int, weight, expert, slot, mode: int = 0, logits=None, counts=None, xs=None,
              softmax: bool = True, groups: int = 0, keep: int = 0) -> None:
    """Chosen experts, their weights and row slots (MoeRouteParams); logits from h and router unless given."""
    hybrid_ext().moe_route(h, router, logits, m, e, top, weight, expert, slot, mode, counts, xs, softmax, groups, keep,
                           ops.status_word(h.device))
    ops._bump()


def moe_scatter(h, m: int, *, e: int, top: int, expert, slot, counts, xs) -> None:
    """Ranks -> packed rows, and the rows' copies there."""
    hybrid_ext().moe_scatter(h, m, e, top, expert, slot, counts, xs, ops.status_word(h.device))
    ops._bump()


def moe_rows(x, w, expert, pairs: int, *, top: int, per_pair: bool, y, act: int = 0) -> None:
    """Expert products of single (row, choice) pairs."""
    hybrid_ext().moe_rows(x, w, expert, pairs, top, per_pair, act, y)
    ops._bump()


def talk_decode_ok(h: int, g: int, dp: int) -> bool:
    return bool(hybrid_ext().talk_decode_ok(h, g, dp))


def talk_prefill_ok(h: int, dp: int) -> bool:
    return bool(hybrid_ext().talk_prefill_ok(h, dp))


def talk_span(window: int, max_ctx: int) -> int:
    """Keys per row of a tile's scores."""
    return int(hybrid_ext().talk_span(window, max_ctx))


def talk_bias(talk: torch.Tensor, r1: torch.Tensor, r2: torch.Tensor, n: int) -> torch.Tensor:
    """[heads, n] fp32: the heads' distance biases r1 ln(1 + r2 distance), mixed like their scores."""
    t, a, b = (x.double() for x in (talk, r1, r2))
    far = torch.arange(n, dtype=torch.float64, device=talk.device)
    return (t @ (a[:, None] * torch.log1p(b[:, None] * far))).float().contiguous()


def talk_decode(q, cache, k_rms, block_tables, seq_lens, *, rows: int, h: int, d: int, window: int, scale: float, cap: float, talk, bias,
                gate, out, part_o=None, part_ml=None, max_splits: int = 0) -> None:
    """Decode rows of talking heads (TalkParams): split-KV and merge, or without `part_o` the kernel for any sizes."""
    hybrid_ext().talk_decode(q, cache, k_rms, block_tables, seq_lens, rows, h, d, window, scale, cap, talk, bias, gate,
                             part_o, part_ml, max_splits, out, ops.status_word(q.device))
    ops._bump(1 if part_o is None else 2)


def talk_prefill(q, cache, k_rms, block_tables, tile_seq, tile_q0, q_start, q_lens, ctx_lens, *, n_tiles: int, h: int, d: int, window: int,
                 scale: float, cap: float, talk, bias, gate, out, scores=None, span: int = 0) -> None:
    """Prompt tiles of talking heads: mixed scores into `scores` [n_tiles, h, 128, span] fp32, then softmax and sums; without
    `scores` the kernel for any sizes."""
    hybrid_ext().talk_prefill(q, cache, k_rms, block_tables, tile_seq, tile_q0, q_start, q_lens, ctx_lens, n_tiles, h, d, window, scale, cap,
                              talk, bias, gate, scores, span, out, ops.status_word(q.device))
    ops._bump(1 if scores is None else 2)


def gru_ws_elems(n: int, n_tiles: int) -> int:
    return n_tiles * (1 + int(hybrid_ext().GRU_PARTS)) * 2 * n


def gru_decode(proj, rows: int, *, bias, gain: float, state, row_slots, positions, out) -> None:
    """Gated recurrence (GruParams), one token per row."""
    hybrid_ext().gru_decode(proj, rows, bias, gain, state, row_slots, positions, out, ops.status_word(proj.device))
    ops._bump()


def gru_prefill(proj, m: int, *, bias, gain: float, state, seq_slots, tile_seq, tile_q0, q_start, q_lens, ctx_lens, n_tiles: int, ws,
                out) -> None:
    """Prompt tiles: what every part of a tile makes of a state, then the outputs."""
    hybrid_ext().gru_prefill(proj, m, bias, gain, state, seq_slots, tile_seq, tile_q0, q_start, q_lens, ctx_lens, n_tiles, ws, out,
                             ops.status_word(proj.device))
    ops._bump(2)


def gemm_f32(a, w, out) -> None:
    """out = a @ w^T in fp32 FMAs."""
    hybrid_ext().gemm_f32(a, w, out)
    ops._bump()


def glu_f32(gu, out, m: int, i: int, act: int) -> None:
    """act(gate) * up, or with act 2 the square of relu of rows without a gate."""
    hybrid_ext().glu_f32(gu, out, m, i, act)
    ops._bump()
