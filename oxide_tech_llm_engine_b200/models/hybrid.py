"""Device model of layer-list decoders: layers of different kinds (softmax attention over the paged KV
cache, retention or a state-space layer with a per-sequence state, two mixers side by side), dense or
mixture-of-experts feed-forwards behind or beside the mixer, hyper-connected residual streams, looped
layers, a hashed bigram embedding. One GPU; bf16 kernels, or fp32 throughout (`dtype="float32"`).

Launch sequence of a step (every row is a token, decode rows first, then prompt chunks):

    stream_norm   embedding (+ bigram row) -> all streams, read-out and norm of the first sublayer
    per sublayer:
      attention:  gemm(q|k|v) -> heads (norm, rotation, paged K/V write) -> paged_decode / paged_prefill
      retention:  gemm(q|k|v|gate) -> retention_decode (one launch) / heads + chunked retention
                  -> gemm(O, fp32 accumulator)
      MLP:        gemm(gate|up, SwiGLU epilogue) -> gemm(down, fp32 accumulator)
      stream_norm stream update with the accumulator, read-out and norm of the next sublayer
    final stream_norm over the logit rows -> gemm(head)

and with mixer and feed-forward side by side:

    branch_norm   embedding -> residual, norms of the first layer's mixer and feed-forward
    per layer:
      gemm(q|k|v | z|x|B|C|dt) -> heads, paged attention -> gemm(O, fp32)
                               -> convolution, state-space layer, gated_norm -> gemm(O, fp32)
      moe_route (-> moe_scatter) -> grouped gemm(up, squared ReLU) -> grouped gemm(down)
      branch_norm   norms of both mixer outputs, weighted expert rows, residual, norms of the next layer
    final branch_norm over the logit rows -> gemm(head)

and with a norm on either side of every sublayer:

    branch_norm   embedding -> residual, norm of the first sublayer
    per sublayer:
      differential attention: as attention, two maps per head; their difference and its norm in the merge (decoding)
                              or in diff_norm
      latent attention:       gemm(query latent | latent) -> latent_rows -> gemm(q)
        decoding:  heads (rotation), grouped gemm(q W_uk) -> latent_decode -> grouped gemm(W_uv)
        prompts:   heads (rotation), latent_gather -> gemm(keys | values of all heads) -> prefill_rows
      matrix memory:          gemm(q|k|v|gate) -> memory_decode / gemm(gates, fp32), chunked memory
                  -> gemm(O, fp32 accumulator)
      MLP:        as above;  experts: moe_route (-> moe_scatter) -> grouped gemm(gate|up, SwiGLU) -> grouped gemm(down)
      branch_norm  norm of the sublayer's result (of the weighted expert rows), residual, norm of the next sublayer
    final branch_norm over the logit rows -> gemm(head)

and with one plain residual stream, x <- x + m f(norm(x)):

    branch_norm   embedding -> residual, norm of the first sublayer
    per sublayer:
      pair:           gemm(q|k|v | z|x|g) -> heads, paged attention with sinks | gated recurrence -> gemm(O of both)
      talking heads:  gemm(q|k|gate) -> heads (norms; keys that are values) -> talk_decode / scores and values of a tile
      MLP:            gemm(up, squared ReLU) -> gemm(down)
      branch_norm     the result times m into the residual, norm of the next sublayer
    ahead of a pass of the loop:
      branch_norm     the stream and the embedding as operand rows -> gemm -> branch_norm (plus the pass's vector) as the stream
    final branch_norm over the logit rows -> gemm(head) -> softcap

In a captured decode step of side-by-side layers the three lines between two branch_norms run on streams of their own: the
experts beside the projection and the mixers, the state-space mixer beside the attention.

KV blocks come from the scheduler's paged pool like any model's (one cache per attention run, so a
looped layer has one per pass); recurrent states live in slots that the scheduler hands to running
sequences. All sizes and constants come from the LayerSpec list; matrices are zero-padded to the
tile grid at load.
"""
from __future__ import annotations

import math
import os
from contextlib import contextmanager, nullcontext
from typing import Optional

import numpy as np
import torch

from .. import ops
from ..errors import ConfigError
from ..ops import hybrid as hops
from .config import ModelConfig
from .gemm_shapes import GemmShapes
from .llama import StepInputs, interleave32
from .weights import WeightSource


def round_up(n: int, k: int) -> int:
    return (n + k - 1) // k * k


def tc_head(a) -> int:
    """Padded head size of the tensor-core attention kernels for a spec, 0 when they do not take it."""
    big = max(a.maps * a.dim, a.vdim)
    if a.heads * a.maps // a.kv_heads > 16 or big > 256:
        return 0
    if big > 128:      # plain causal attention only
        return 256 if not (a.window or a.chunk or a.sink is not None or a.sinks) else 0
    return 64 if big <= 64 else 128


def latent_layout(a) -> tuple:
    """(key columns, value columns, first unrotated column) of a latent-attention head; no value columns: the prompt
    kernel does not take heads of these sizes."""
    at = round_up(a.rot_dim, 8)
    z = hops.prefill_size(at + round_up(a.dim, 8), round_up(a.vdim, 8))
    return (*z, at) if z is not None else (at + round_up(a.dim, 8), 0, at)


def talk_head(a) -> int:
    """Padded head size of the talking-heads kernels, 0 when they do not take it."""
    return 0 if a.dim > 128 else (64 if a.dim <= 64 else 128)


TALK_SCORE_BYTES = 2 << 30   # mixed scores of prompt tiles that are held at a time

def talk_pass(n_tiles: int, scores: int) -> int:
    """Prompt tiles per pass: about equal passes whose scores (so many per tile) fit."""
    most = max(1, TALK_SCORE_BYTES // (4 * scores))
    return -(-n_tiles // -(-n_tiles // most))


KV_PASS_ROWS = 65536      # positions whose keys and values are expanded at a time


class _Sublayer:
    """What stream_norm needs around a sublayer, and the function that runs it."""

    def __init__(self, norm, hc, run, last_of: int):
        self.norm, self.hc, self.run = norm, hc, run
        self.last_of = last_of       # index of the layer run that this sublayer ends, or -1


class _NormedSublayer:
    """Norm weights of a sublayer's input and result (the latter times the layer scale, or none), the function that runs it,
    and the factor on its result. `base`: the result takes the place of the stream, plus this vector (the entry of a pass, whose
    input is not normed)."""

    def __init__(self, norm, out, run, last_of: int, gain: float = 1.0, base=None):
        self.norm, self.out, self.run, self.last_of, self.gain, self.base = norm, out, run, last_of, gain, base


class _ParallelLayer:
    """Norm weights of the layer's inputs (mixer, feed-forward), of its two mixer outputs, and the function that runs it."""

    def __init__(self, norms: list, out: tuple, run):
        self.norms, self.out, self.run = norms, out, run


class AttentionRun:
    """One run of an attention layer: weights shared by all passes, a KV cache of its own. Its projection rows
    may be the first columns of wider ones (a layer with two mixers). With two maps per head both keys of a value head
    lie in one cache row, and a query has zeros where the other map's key is."""

    def __init__(self, m: "HybridModel", spec, w: dict):
        self.m, self.spec, self.w = m, spec, w
        a = spec
        self.nq, self.dk = a.heads * a.maps, a.maps * a.dim     # query heads, values of a key row
        self.width = a.in_width
        self.acc_k = round_up(a.out_dim, 64)
        # head sizes of the tensor-core kernels: q, k and v padded with zeros
        self.tc = m.dtype == torch.bfloat16 and tc_head(a) > 0
        self.dp, self.ep = (tc_head(a),) * 2 if self.tc else (self.dk, a.vdim)
        self.k = torch.zeros(m.num_blocks, a.kv_heads, 16, self.dp, dtype=m.dtype, device=m.device)
        self.v = torch.zeros(m.num_blocks, a.kv_heads, 16, self.ep, dtype=m.dtype, device=m.device)
        m.k_cache.append(self.k)
        m.v_cache.append(self.v)

    def __call__(self, s: StepInputs, h: torch.Tensor) -> None:
        self.m.into_acc(self.attend(s, self.m.project(h, self.w["w_in"], self.width)), self.w["w_o"])

    def attend(self, s: StepInputs, proj: torch.Tensor, out: Optional[torch.Tensor] = None, gain: float = 1.0) -> torch.Tensor:
        """Projection rows -> heads' results times `gain`, in `out` or a buffer of their own."""
        m, a, w, M = self.m, self.spec, self.w, s.m
        q = m.buffer(("q", self.nq * self.dp, a.dim, a.maps), self.nq * self.dp)
        hops.heads(proj, M, h=self.nq, g=a.kv_heads * a.maps, d=a.dim, e=a.vdim, rot=w["rot"], positions=s.positions, q_out=q,
                   q_hd=self.dp, q_norm=w["q_norm"], k_norm=w["k_norm"], eps=m.cfg.rms_eps, k_cache=self.k,
                   v_cache=self.v, slots=s.slot_mapping, maps=a.maps, bias=w.get("bias"), temp_coef=a.temp_coef,
                   temp_every=a.temp_every)
        out = m.buffer(("o", a.out_dim), self.acc_k) if out is None else out
        # both maps' results in fp32, where the difference is not taken in the merge
        both = m.maps_buffer(self.nq * a.vdim) if a.diff is not None else out
        lam = (w["lam"], 1.0 - a.diff, m.cfg.rms_eps) if a.diff is not None else ()
        nd = s.n_decode
        kw = dict(window=a.window, keep_first=a.keep_first if a.window else 0, scale=a.scale, chunk=a.chunk,
                  sink=-math.inf if a.sink is None else a.sink, sinks=w.get("sinks"), out_gain=gain)
        done = 0       # rows whose difference has been taken
        if self.tc:
            if nd > 0:
                ops.paged_decode(q[:nd].view(nd, self.nq, self.dp), self.k, self.v, s.block_tables, s.seq_lens,
                                 s.pages_per_split, m.part_o, m.part_ml, out[:nd], batch=nd, max_splits=m.max_splits, out_d=a.vdim,
                                 exact_p=True, diff=lam, **kw)
                done = nd
            if s.n_prefill > 0:
                args = (q.view(-1, self.nq, self.dp), self.k, self.v, s.prefill_block_tables, s.tile_seq, s.tile_q0,
                        s.q_start, s.q_lens, s.ctx_lens, both)
                if self.dp > 128:
                    hops.prefill_pages(*args, n_tiles=s.n_tiles, scale=a.scale, out_d=a.vdim)
                else:
                    ops.paged_prefill(*args, n_tiles=s.n_tiles, out_d=a.vdim, exact_p=True, **kw)
        else:
            kw.update(h=self.nq, d=self.dk, e=a.vdim, out=both)
            if nd > 0:
                hops.row_attention(q, self.dp, self.k, self.v, s.block_tables, n=nd, seq_lens=s.seq_lens, **kw)
            if s.n_prefill > 0:
                hops.row_attention(q, self.dp, self.k, self.v, s.prefill_block_tables, n=s.n_tiles, tile_seq=s.tile_seq,
                                   tile_q0=s.tile_q0, q_start=s.q_start, q_lens=s.q_lens, ctx_lens=s.ctx_lens, **kw)
        if lam and done < M:
            hops.diff_norm(both[done:], M - done, h=a.heads, e=a.vdim, lam=lam[0], gain=lam[1], eps=lam[2], out=out[done:])
        return out[:M]


class TalkingRun:
    """One run of attention with talking heads: a cache of unnormed keys, which are the values, and their norms' factors."""

    def __init__(self, m: "HybridModel", spec, w: dict):
        self.m, self.spec, self.w = m, spec, w
        a = spec
        self.width, self.acc_k = a.in_width, round_up(a.out_dim, 64)
        dp = talk_head(a) if m.dtype == torch.bfloat16 else 0
        self.dp = dp or round_up(a.dim, 8)
        self.decode_tc = dp > 0 and hops.talk_decode_ok(a.heads, a.kv_heads, dp)
        self.prefill_tc = dp > 0 and hops.talk_prefill_ok(a.heads, dp)
        self.cache = torch.zeros(m.num_blocks, a.kv_heads, 16, self.dp, dtype=m.dtype, device=m.device)
        self.k_rms = torch.zeros(m.num_blocks, 16, dtype=torch.float32, device=m.device)
        m.k_cache.append(self.cache)
        m.v_cache.append(self.k_rms)

    def __call__(self, s: StepInputs, h: torch.Tensor) -> None:
        m, a, w, M, nd = self.m, self.spec, self.w, s.m, s.n_decode
        proj = m.project(h, w["w_in"], self.width)
        q = m.buffer(("q_talk", a.heads, a.dim), round_up(a.heads * self.dp, 8))
        hops.heads(proj, M, h=a.heads, g=a.kv_heads, d=a.dim, e=a.dim, rot=w["rot"], positions=s.positions, q_out=q, q_hd=self.dp,
                   q_norm=w["q_norm"], eps=m.cfg.rms_eps, k_cache=self.cache, slots=s.slot_mapping, k_rms=self.k_rms)
        out = m.buffer(("o", a.out_dim), self.acc_k)
        gate = proj[:, a.gate_col:]
        kw = dict(h=a.heads, d=a.dim, window=a.window, scale=a.scale, cap=a.softcap, talk=w["talk"], bias=w["bias"], gate=gate, out=out)
        if nd > 0:
            parts = dict(part_o=m.part_o, part_ml=m.part_ml, max_splits=m.max_splits) if self.decode_tc else {}
            hops.talk_decode(q, self.cache, self.k_rms, s.block_tables, s.seq_lens, rows=nd, **kw, **parts)
        if s.n_prefill > 0:
            seqs = (s.q_start, s.q_lens, s.ctx_lens)
            span = hops.talk_span(a.window, s.max_ctx)
            per = a.heads * 128 * span       # scores of a tile
            step = talk_pass(s.n_tiles, per) if self.prefill_tc else s.n_tiles
            for t0 in range(0, s.n_tiles, step):
                n = min(step, s.n_tiles - t0)
                ws = dict(scores=m.scratch("talk_scores", n * per), span=span) if self.prefill_tc else {}
                hops.talk_prefill(q, self.cache, self.k_rms, s.prefill_block_tables, s.tile_seq[t0:], s.tile_q0[t0:], *seqs, n_tiles=n,
                                  **kw, **ws)
        m.into_acc(out[:M], w["w_o"])


class GruRun:
    """One run of a gated recurrence: a state per slot."""

    def __init__(self, m: "HybridModel", spec, w: dict):
        self.m, self.spec, self.w = m, spec, w
        self.state = torch.zeros(m.state_slots, spec.width_p, dtype=torch.float32, device=m.device)
        m.states.append(self.state)

    def mix(self, s: StepInputs, proj: torch.Tensor, out: torch.Tensor, gain: float) -> None:
        """Projection rows z | x | g -> states times silu(g) times `gain`."""
        m, w, nd = self.m, self.w, s.n_decode
        kw = dict(bias=w["bias"], gain=gain, state=self.state, out=out)
        if nd > 0:
            hops.gru_decode(proj, nd, row_slots=s.decode_slots, positions=s.positions, **kw)
        if s.n_prefill > 0:
            hops.gru_prefill(proj, s.m, seq_slots=s.prefill_slots, tile_seq=s.tile_seq, tile_q0=s.tile_q0, q_start=s.q_start, q_lens=s.q_lens,
                             ctx_lens=s.ctx_lens, n_tiles=s.n_tiles, ws=m.scratch("gru_ws", hops.gru_ws_elems(self.spec.width_p, s.n_tiles)), **kw)


class PairRun:
    """Attention and a gated recurrence on the same rows, their results weighted and side by side in one row, so one output
    projection adds them up."""

    def __init__(self, m: "HybridModel", spec, w: dict):
        self.m, self.spec, self.w = m, spec, w
        self.left, self.right = AttentionRun(m, spec.left, w["left"]), GruRun(m, spec.right, w["right"])
        self.split, self.width = round_up(self.left.width, 64), m._in_width(spec)
        self.lk = round_up(spec.left.out_dim, 64)
        self.acc_k = self.lk + round_up(spec.right.out_dim, 64)

    def __call__(self, s: StepInputs, h: torch.Tensor) -> None:
        m, g = self.m, self.spec.gains
        proj = m.project(h, self.w["w_in"], self.width)
        out = m.buffer(("pair", self.lk, self.acc_k, self.spec.left.out_dim), self.acc_k)
        self.left.attend(s, proj, out, g[0])
        self.right.mix(s, proj[:, self.split:], out[:, self.lk:], g[1])
        m.into_acc(out[:s.m], self.w["w_o"])


class EntryRun:
    """x <- W [x; embedding] ahead of a pass of the loop. Its input rows come from branch_norm; bf16 rows hold x in two terms."""

    def __init__(self, m: "HybridModel", w: torch.Tensor):
        self.m, self.w = m, w
        self.acc_k = (3 if m.dtype == torch.bfloat16 else 2) * m.dp

    def rows(self) -> torch.Tensor:
        return self.m.buffer(("entry", self.acc_k), self.acc_k)

    def __call__(self, s: StepInputs, h: torch.Tensor) -> None:
        self.m.into_acc(self.rows()[:s.m], self.w)


class LatentRun:
    """One run of a latent-attention layer; the cache is its own or that of the layer it reads. Heads lie in padded
    layouts: queries and expanded keys [rotated | unrotated | zeros], so both parts start on 16 bytes."""

    def __init__(self, m: "HybridModel", spec, w: dict):
        self.m, self.spec, self.w = m, spec, w
        a = spec
        self.width, self.cp = a.in_width, a.cache_row
        self.dk, self.dv, self.at = latent_layout(a)
        self.d8, self.r8, self.ep = round_up(a.dim, 8), round_up(a.kv_rank, 8), round_up(a.vdim, 8)
        self.acc_k = round_up(a.heads * self.ep, 64)
        bf16 = m.dtype == torch.bfloat16
        self.expand = bf16 and self.dv > 0                                    # prompts over expanded keys and values
        self.tc = bf16 and hops.latent_decode_heads(a.heads, a.kv_rank, self.cp) > 0
        if a.kv_from is None:
            self.cache = torch.zeros(m.num_blocks, 1, 16, self.cp, dtype=m.dtype, device=m.device)
            m.k_cache.append(self.cache)
        else:
            self.cache = m.latents[a.kv_from].cache

    def __call__(self, s: StepInputs, h: torch.Tensor) -> None:
        m, a, w, M = self.m, self.spec, self.w, s.m
        proj = m.project(h, w["w_in"], self.width)
        cq = m.buffer(("cq", a.q_rank), round_up(a.q_rank, 64))
        kw = dict(kv_col=a.kv_col, kv_rank=a.kv_rank, kv_norm=w["kv_norm"], cache=self.cache, slots=s.slot_mapping,
                  rot=w["rot"]) if a.kv_from is None else {}
        hops.latent_rows(proj, M, q_rank=a.q_rank, q_norm=w["q_norm"], q_out=cq, positions=s.positions, eps=m.cfg.rms_eps, **kw)
        q = m.buffer(("q_up", a.heads, self.dk), round_up(a.heads * self.dk, 64))
        m.product(cq[:M], w["w_uq"], q)
        o = m.buffer(("o_lat", a.heads, self.ep), self.acc_k)
        na = s.n_decode if self.expand else M
        if na > 0:
            self._absorbed(s, q, o, na)
        if self.expand and s.n_prefill > 0:
            self._expanded(s, q, o)
        m.into_acc(o[:M], w["w_o"])

    def _absorbed(self, s: StepInputs, q: torch.Tensor, o: torch.Tensor, n: int) -> None:
        """Rows against the latents: queries times W_uk, sums of latents times W_uv."""
        m, a, w, H, nd = self.m, self.spec, self.w, self.spec.heads, s.n_decode
        qa = m.buffer(("q_lat", H, self.cp, a.kv_rank), H * self.cp)
        ctx = m.buffer(("ctx", H, self.r8, a.kv_rank), H * self.r8)
        if a.rot is not None:
            hops.heads(q, n, h=H, g=0, d=a.rot_dim, e=4, rot=w["rot"], positions=s.positions, q_out=qa[:, a.kv_rank:], q_hd=self.cp,
                       q_pd=self.dk)
        heads = lambda t, width, lo, hi: t[:n, :H * width].view(n, H, width)[:, :, lo:hi].transpose(0, 1)
        m.per_head(heads(q, self.dk, self.at, self.at + self.d8), w["w_uk"], heads(qa, self.cp, 0, a.kv_rank))
        kw = dict(h=H, d=a.kv_rank + a.rot_dim, e=a.kv_rank, window=0, keep_first=0, scale=a.scale, out=ctx, o_hd=self.r8)
        if nd > 0 and self.tc:
            hops.latent_decode(qa[:nd].view(nd, H, self.cp), self.cache, s.block_tables, s.seq_lens, m.part_o, m.part_ml, ctx, rows=nd,
                               kv_rank=a.kv_rank, max_splits=m.max_splits, scale=a.scale, o_hd=self.r8)
        elif nd > 0:
            hops.row_attention(qa, self.cp, self.cache, self.cache, s.block_tables, n=nd, seq_lens=s.seq_lens, **kw)
        if n > nd:       # prompts that are not expanded
            hops.row_attention(qa, self.cp, self.cache, self.cache, s.prefill_block_tables, n=s.n_tiles, tile_seq=s.tile_seq,
                               tile_q0=s.tile_q0, q_start=s.q_start, q_lens=s.q_lens, ctx_lens=s.ctx_lens, **kw)
        m.per_head(heads(ctx, self.r8, 0, self.r8), w["w_uv"], heads(o, self.ep, 0, self.ep))

    def _expanded(self, s: StepInputs, q: torch.Tensor, o: torch.Tensor) -> None:
        m, a, w, H, nd = self.m, self.spec, self.w, self.spec.heads, s.n_decode
        if a.rot is not None:      # in place: a row's heads are read and written by one CTA, value by value
            hops.heads(q[nd:], s.m - nd, h=H, g=0, d=a.rot_dim, e=4, rot=w["rot"], positions=s.positions[nd:], q_out=q[nd:],
                       q_hd=self.dk, q_pd=self.dk)
        for i, (s0, s1, t0, t1, rows, pages) in enumerate(s.kv_passes):
            lat = m.rows("latents", rows, self.cp)
            kv = m.rows("kv", rows, H * (self.dk + self.dv))
            if m.gathered != (i, id(self.cache)):
                hops.latent_gather(self.cache, s.prefill_block_tables, s.ctx_lens, s.kv_start, seq0=s0, n_seqs=s1 - s0, max_pages=pages,
                                   out=lat)
                m.gathered = (i, id(self.cache))
            m.product(lat, w["w_kv"], kv)
            hops.prefill_rows(q[:, :H * self.dk].view(-1, H, self.dk), kv, s.tile_seq[t0:], s.tile_q0[t0:], s.q_start, s.q_lens,
                              s.ctx_lens, s.kv_start, o, dk=self.dk, dv=self.dv, g=H, n_tiles=t1 - t0, scale=a.scale, out_d=self.ep)


class MemoryRun:
    """One run of a matrix-memory layer: a memory with its normaliser and a running maximum per slot."""

    def __init__(self, m: "HybridModel", spec, w: dict):
        self.m, self.spec, self.w = m, spec, w
        r = spec
        self.width, self.acc_k = r.in_width, round_up(r.out_dim, 64)
        f32 = dict(dtype=torch.float32, device=m.device)
        self.state = torch.zeros(m.state_slots, r.heads, r.dim * r.vdim + r.dim, **f32)
        self.state_m = torch.zeros(m.state_slots, r.heads, **f32)
        m.states += [self.state, self.state_m]
        self.chunks = m.dtype == torch.bfloat16 and hops.memory_chunks_ok(r.dim, r.vdim)
        self.zp = round_up(2 * r.heads, 64)

    def __call__(self, s: StepInputs, h: torch.Tensor) -> None:
        m, r, w, M, nd = self.m, self.spec, self.w, s.m, s.n_decode
        proj = m.project(h, w["w_in"], self.width)
        out = m.buffer(("o", r.out_dim), self.acc_k)
        kw = dict(h=r.heads, d=r.dim, e=r.vdim, z_bias=w["z_bias"], cap=r.gate_cap, eps=m.cfg.rms_eps, norm_w=w["norm"],
                  state=self.state, state_m=self.state_m)
        z = None
        if m.dtype == torch.float32 or s.n_prefill > 0:
            # pre-activations of the gates in fp32; bf16 decode rows take theirs from the rows themselves
            lo = 0 if m.dtype == torch.float32 else nd
            z = m.gates_buffer(self.zp)
            m.product_f32(h[lo:], w["w_z"], z[lo:M])
        if nd > 0:
            own = dict(z=z) if m.dtype == torch.float32 else dict(hidden=h, z_w=w["w_z"])
            hops.memory_decode(proj, nd, row_slots=s.decode_slots, positions=s.positions, out=out, **own, **kw)
        if s.n_prefill > 0:
            n = (hops.memory_ws_elems(r.heads, r.dim, r.vdim, s.n_tiles) if self.chunks
                 else M * r.out_dim + s.n_prefill * r.heads * (r.dim + 1))
            hops.memory_prefill(proj, M, z=z, seq_slots=s.prefill_slots, tile_seq=s.tile_seq, tile_q0=s.tile_q0, q_start=s.q_start,
                                q_lens=s.q_lens, ctx_lens=s.ctx_lens, n_tiles=s.n_tiles, n_seqs=s.n_prefill,
                                ws=m.scratch("chunk_states", n), chunks=self.chunks, out=out, **kw)
        m.into_acc(out[:M], w["w_o"])


class RetentionRun:
    """One run of a retention layer: weights shared by all passes, a state per slot of its own."""

    def __init__(self, m: "HybridModel", spec, w: dict):
        self.m, self.spec, self.w = m, spec, w
        r = spec
        self.width = 2 * r.heads * (r.dim + r.vdim)
        self.k_scale = r.dim ** -0.5
        self.state = torch.zeros(m.state_slots, r.heads, r.dim, r.vdim, dtype=torch.float32, device=m.device)
        m.states.append(self.state)
        self.chunked = m.dtype == torch.bfloat16 and hops.retention_chunks_ok(r.dim, r.vdim)

    def __call__(self, s: StepInputs, h: torch.Tensor) -> None:
        m, r, w, M = self.m, self.spec, self.w, s.m
        proj = m.project(h, w["w_in"], self.width)
        out = m.buffer(("o", r.out_dim), round_up(r.out_dim, 64))
        nd = s.n_decode
        kw = dict(h=r.heads, d=r.dim, e=r.vdim, decay_pow=w["decay_pow"], eps=m.cfg.rms_eps, state=self.state, out=out)
        if nd > 0:
            hops.retention_decode(proj, nd, rot=w["rot"], k_scale=self.k_scale, row_slots=s.decode_slots,
                                  positions=s.positions, **kw)
        if s.n_prefill > 0:
            hd = r.heads * r.dim
            q_rot, k_rot = (m.scratch(n, M * hd).view(r.heads, M, r.dim) for n in ("q_rot", "k_rot"))
            hops.heads(proj[nd:M], M - nd, h=r.heads, g=r.heads, d=r.dim, e=r.vdim, rot=w["rot"], positions=s.positions[nd:],
                       q_out=q_rot[:, nd:], q_hd=r.dim, k_out=k_rot[:, nd:], k_scale=self.k_scale)
            if self.chunked:
                kw["ws"] = m.scratch("chunk_states", 2 * s.n_tiles * r.state_elems)
            else:
                kw["o_buf"] = m.scratch("ret_o", M * r.out_dim)
            hops.retention_prefill(proj, M, seq_slots=s.prefill_slots, tile_seq=s.tile_seq, tile_q0=s.tile_q0,
                                   q_start=s.q_start, q_lens=s.q_lens, ctx_lens=s.ctx_lens, n_tiles=s.n_tiles,
                                   n_seqs=s.n_prefill, q_rot=q_rot, k_rot=k_rot, **kw)
        m.into_acc(out[:M], w["w_o"])


class SsdRun:
    """One run of a state-space layer: a recurrent and a convolution state per slot."""

    def __init__(self, m: "HybridModel", spec, w: dict):
        self.m, self.spec, self.w = m, spec, w
        r = spec
        f32 = dict(dtype=torch.float32, device=m.device)
        self.state = torch.zeros(m.state_slots, r.heads, r.state_p, r.vdim_p, **f32)
        self.conv_state = torch.zeros(m.state_slots, r.taps, r.channels_p, **f32)
        m.states += [self.state, self.conv_state]
        self.runs = m.dtype == torch.bfloat16 and hops.ssd_chunks_ok(r.state_p)

    def mix(self, s: StepInputs, proj: torch.Tensor, start=nullcontext()) -> torch.Tensor:
        """Projection rows z | x | B | C | dt -> gated and normed rows [M, heads * vdim]. `start`: context of the first launch."""
        m, r, w, M, nd = self.m, self.spec, self.w, s.m, s.n_decode
        y = m.buffer(("ssd_y", r.heads * r.vdim_p), r.heads * r.vdim_p)
        kw = dict(h=r.heads, g=r.groups, w=w["ssd"], state=self.state, conv_state=self.conv_state, y=y)
        if nd > 0:
            with start:
                hops.ssd_decode(proj, nd, row_slots=s.decode_slots, positions=s.positions, **kw)
        if s.n_prefill > 0:
            seg = hops.ssd_segment(r.heads, r.vdim_p, s.n_tiles, s.n_prefill) if self.runs else 0
            if seg:
                kw.update(segment=seg, ws=m.scratch("ssd_ws", hops.ssd_ws_elems(r.heads, r.vdim_p, r.state_p, s.n_tiles)))
            hops.ssd_prefill(proj, M, seq_slots=s.prefill_slots, tile_seq=s.tile_seq, tile_q0=s.tile_q0, q_start=s.q_start,
                             q_lens=s.q_lens, ctx_lens=s.ctx_lens, n_tiles=s.n_tiles, n_seqs=s.n_prefill,
                             u=m.buffer(("ssd_u", r.channels_p), r.channels_p), runs=self.runs, **kw)
        out = m.buffer(("ssd_o", r.inner), round_up(r.inner, 64))
        hops.gated_norm(y, proj, M, h=r.heads, e=r.vdim, ep=r.vdim_p, groups=r.norm_groups, w=w["norm"], eps=m.cfg.rms_eps, out=out)
        return out[:M]


class MoeRun:
    """Mixture of experts. Its result stays where the experts leave it: `experts` = (rows, slots, weights, top)
    for the kernel that adds the weighted rows to the residual."""

    def __init__(self, m: "HybridModel", spec, w: dict):
        self.m, self.spec, self.w = m, spec, w
        self.fp = round_up(spec.ff, 64)
        self.acc_k = 0             # no fp32 accumulator
        self.b = m.moe_buffers(spec.experts, spec.top, self.fp)

    def __call__(self, s: StepInputs, h: torch.Tensor, start=nullcontext()) -> tuple:
        m, e, w, b, M = self.m, self.spec, self.w, self.b, s.m
        E, top = e.experts, e.top
        route = dict(e=E, top=top, weight=b["weight"], expert=b["expert"], slot=b["slot"], softmax=e.scores == "softmax",
                     groups=e.groups, keep=e.keep)
        if m.dtype == torch.float32 or m.few_rows(M):
            with start:
                hops.moe_route(h, w["router"], M, **route)
            pairs = M * top
            rows, act = b["out"][:pairs], b["act"][:pairs]
            hops.moe_rows(h, w["up"], b["expert"], pairs, top=top, per_pair=False, y=act, act=3 if e.glu else 2)
            hops.moe_rows(act, w["down"], b["expert"], pairs, top=top, per_pair=True, y=rows)
            return rows, b["slot"], b["weight"], top
        if M <= 128:
            # one slab of 128 rows per expert: a single launch routes and places
            xs, act, rows = (b[k][:E * 128] for k in ("xs", "act", "out"))
            with start:
                hops.moe_route(h, w["router"], M, mode=1, counts=b["counts"], xs=xs, **route)
            m_tiles = min(E, M * top)
            gx, ga, gr = xs.view(E, 128, -1), act.view(E, 128, -1), rows.view(E, 128, -1)
        else:
            m_tiles = (M * top + 127 * min(E, M * top)) // 128
            n = m_tiles * 128
            gx, ga, gr = b["xs"][:n], b["act"][:n], b["out"][:n]
            rows = gr
            logits = b["logits"][:M]
            ops.gemm(h, w["router_p"], out=logits, epi=ops.EPI_STORE_F32, **m._gemm_shape(M, logits.shape[1], m.dp, store=True))
            hops.moe_route(h, w["router"], M, mode=2, logits=logits, counts=b["counts"], **route)
            hops.moe_scatter(h, M, e=E, top=top, expert=b["expert"], slot=b["slot"], counts=b["counts"], xs=gx)
        if e.glu:
            ops.gemm(gx, w["up"], out=ga, epi=ops.EPI_SWIGLU_BF16, group_counts=b["counts"], m_tiles=m_tiles,
                     bn=m.group_bn(m_tiles, 2 * self.fp, whole=True))
        else:
            ops.gemm(gx, w["up"], out=ga, group_counts=b["counts"], m_tiles=m_tiles, act=2, bn=m.group_bn(m_tiles, self.fp))
        ops.gemm(ga, w["down"], out=gr, group_counts=b["counts"], m_tiles=m_tiles, bn=m.group_bn(m_tiles, m.dp),
                 done_ticket=b["ticket"], reset_on_done=b["counts"])
        return rows, b["slot"], b["weight"], top


class ParallelRun:
    """Two mixers on the same rows, each into an accumulator of its own, beside a feed-forward."""

    def __init__(self, m: "HybridModel", spec, w: dict, mlp):
        self.m, self.w, self.mlp = m, w, mlp
        self.left = AttentionRun(m, spec.left, w["left"])
        self.right = SsdRun(m, spec.right, w["right"])
        self.split = round_up(self.left.width, 64)        # first column of the right mixer's projection
        self.width = m._in_width(spec)
        self.k = (round_up(spec.left.out_dim, 64), round_up(spec.right.out_dim, 64))

    def clears(self, M: int) -> tuple:
        """Which accumulators have to be zero when the layer starts."""
        return tuple(self.m.adds_up(M, k) for k in self.k)

    def __call__(self, s: StepInputs, h: torch.Tensor, h2: Optional[torch.Tensor]) -> Optional[tuple]:
        m, w = self.m, self.w
        if m.side_streams(s):
            return self._on_streams(s, h, h2)
        proj = m.project(h, w["w_in"], self.width)
        m.into_branch(0, self.left.attend(s, proj), w["left"]["w_o"])
        m.into_branch(1, self.right.mix(s, proj[:, self.split:]), w["right"]["w_o"])
        return self.mlp(s, h2) if self.mlp is not None else None

    def _on_streams(self, s: StepInputs, h: torch.Tensor, h2: Optional[torch.Tensor]) -> Optional[tuple]:
        """The same, forked and joined. A launch that waits for another stream takes a full dependency, not a
        programmatic one."""
        m, w = self.m, self.w
        main, experts = torch.cuda.current_stream(m.device), None
        s_right, s_moe = m.streams2
        if self.mlp is not None:
            s_moe.wait_stream(main)
            with torch.cuda.stream(s_moe):
                experts = self.mlp(s, h2, start=m.full_dependency())
        proj = m.project(h, w["w_in"], self.width)
        s_right.wait_stream(main)
        with torch.cuda.stream(s_right):
            m.into_branch(1, self.right.mix(s, proj[:, self.split:], start=m.full_dependency()), w["right"]["w_o"])
        m.into_branch(0, self.left.attend(s, proj), w["left"]["w_o"])
        main.wait_stream(s_right)
        if self.mlp is not None:
            main.wait_stream(s_moe)
        return experts


class MlpRun:
    def __init__(self, m: "HybridModel", spec, w: dict):
        self.m, self.spec, self.w = m, spec, w
        self.ip = self.acc_k = round_up(spec.ff, 64)
        self.act = {"gelu_tanh": 1, "relu2": 2}.get(spec.act, 0)

    def __call__(self, s: StepInputs, h: torch.Tensor) -> None:
        m, M = self.m, s.m
        act = m.buffer(("act", self.ip), self.ip)
        w = self.w["w_gu"]
        if not self.spec.glu:
            if m.dtype == torch.float32:
                u = m.scratch("gate_up", M * self.ip).view(M, self.ip)
                hops.gemm_f32(h, w, u)
                hops.glu_f32(u, act, M, self.ip, self.act)
            elif m.few_rows(M):
                ops.gemv(h, w, act[:M], act=self.act)
            else:
                ops.gemm(h, w, out=act[:M], act=self.act, **m._gemm_shape(M, self.ip, m.dp, store=True))
        elif m.dtype == torch.float32:
            gu = m.scratch("gate_up", M * 2 * self.ip).view(M, 2 * self.ip)
            hops.gemm_f32(h, w, gu)
            hops.glu_f32(gu, act, M, self.ip, self.act)
        elif m.few_rows(M):
            ops.gemv(h, w, act[:M], swiglu=True, act=self.act)
        else:
            ops.gemm(h, w, out=act[:M], epi=ops.EPI_SWIGLU_BF16, act=self.act,
                     **m._gemm_shape(M, 2 * self.ip, m.dp, swiglu=True))
        m.into_acc(act[:M], self.w["w_down"])


RUNS = {"attention": AttentionRun, "retention": RetentionRun, "latent_attention": LatentRun, "mlstm": MemoryRun,
        "talking_attention": TalkingRun, "parallel": PairRun}
MLP_RUNS = {"dense": MlpRun, "moe": MoeRun}


class HybridModel(GemmShapes):
    supports_kv_tiers = False      # caches of different shapes, states that are not in blocks
    supports_block_mass = False

    def __init__(self, cfg: ModelConfig, *, rank: int = 0, world: int = 1, group=None,
                 device: Optional[torch.device] = None, max_tokens: int = 2048, max_seqs: int = 256,
                 num_blocks: int = 1024, max_blocks_per_seq: int = 512, max_logits: Optional[int] = None,
                 max_splits: int = 16, weight_mode: str = "bf16", tile_weights: Optional[bool] = None,
                 layer_range: Optional[tuple] = None, dtype: str = "bfloat16", state_slots: int = 0):
        if world != 1 or layer_range is not None:
            raise ConfigError(f"{cfg.name}: layer-list models are served on one GPU (tp = pp = 1)")
        if weight_mode != "bf16":
            raise ConfigError(f"{cfg.name}: weight mode {weight_mode!r} is not built for layer-list models")
        if dtype not in ("bfloat16", "float32"):
            raise ConfigError(f"unknown dtype {dtype!r}")
        self.streams = max(1, cfg.streams)
        if self.streams > hops.max_streams():
            raise ConfigError(f"{self.streams} residual streams, at most {hops.max_streams()}")
        self.cfg, self.tp, self.rank = cfg, 1, 0
        self.dtype = torch.bfloat16 if dtype == "bfloat16" else torch.float32
        self.device = device or torch.device("cuda", torch.cuda.current_device())
        self.weight_mode = weight_mode
        pdl = os.environ.get("OXB_PDL", "1") != "0"
        self._pdl = pdl
        ops.set_pdl(pdl)
        hops.set_pdl(pdl)
        self._sms = torch.cuda.get_device_properties(self.device).multi_processor_count
        self._gemm_cfg: dict = {}
        self.gemv_max_rows = int(os.environ.get("OXB_GEMV_MAX", "2")) if os.environ.get("OXB_GEMV", "1") != "0" else 0
        self.tile_weights = (os.environ.get("OXB_TILE_WEIGHTS", "1") != "0") if tile_weights is None else tile_weights
        self.max_tokens, self.max_seqs = max_tokens, max_seqs
        self.max_logits = max_logits or max(max_seqs, 64)
        self.max_splits = max_splits
        self.num_blocks, self.max_blocks_per_seq = num_blocks, max_blocks_per_seq
        self.state_slots = state_slots if cfg.is_recurrent else 0
        if cfg.is_recurrent and state_slots < 1:
            raise ConfigError(f"{cfg.name} has recurrent layers: state_slots must be at least 1")
        d = cfg.d_model
        self.dp = round_up(d, 64)
        dev = self.device
        self.parallel = any(L.parallel for L in cfg.layers)
        if self.parallel and (cfg.streams or cfg.loop or cfg.bigram or not all(L.parallel for L in cfg.layers)):
            raise ConfigError(f"{cfg.name}: layers with mixer and feed-forward side by side come without hyper-connected streams, "
                              "loops and a bigram embedding, and without other layers")
        self.sandwich = any(L.post_norm for L in cfg.layers)
        if self.sandwich and (self.parallel or cfg.streams or cfg.loop or cfg.bigram or not all(L.post_norm for L in cfg.layers)):
            raise ConfigError(f"{cfg.name}: layers with a norm behind every sublayer come without hyper-connected streams, loops and "
                              "a bigram embedding, and without other layers")
        # one residual stream that branch_norm carries from sublayer to sublayer
        self.single = self.sandwich or cfg.residual_mult is not None
        if cfg.residual_mult is not None and (self.parallel or self.sandwich or cfg.streams or cfg.bigram):
            raise ConfigError(f"{cfg.name}: layers over one plain residual stream come without hyper-connected streams, a bigram embedding "
                              "and other layers")
        moe = [L.mlp for L in cfg.layers if L.mlp is not None and L.mlp.kind == "moe"]
        if any(e.experts > hops.max_experts()[0] or e.top > hops.max_experts()[1] for e in moe):
            raise ConfigError(f"{cfg.name}: at most {hops.max_experts()[0]} experts, {hops.max_experts()[1]} of them chosen")
        if any(e.groups > hops.max_groups() for e in moe):
            raise ConfigError(f"{cfg.name}: at most {hops.max_groups()} groups of experts")
        att = [p for L in cfg.layers for p in L.mixer.parts if p.kind == "attention"]
        lat = [p for L in cfg.layers for p in L.mixer.parts if p.kind == "latent_attention"]
        talk = [p for L in cfg.layers for p in L.mixer.parts if p.kind == "talking_attention"]
        # CTAs per sequence and split of the decode attention
        self.hkv = min([a.kv_heads for a in att] + [1 for _ in lat], default=1)   # (talking heads: one, their window is short)
        self.x = torch.zeros(max_tokens, self.streams, d, dtype=torch.float32, device=dev)
        self.h = torch.zeros(max_tokens, self.dp, dtype=self.dtype, device=dev)
        n_acc = 2 if self.parallel else 1
        self.branches = torch.zeros(n_acc, max_tokens, self.dp, dtype=torch.float32, device=dev)
        self.acc = self.branches[0]
        self.h2 = torch.zeros_like(self.h) if self.parallel else None
        on = self.parallel and os.environ.get("OXB_STREAMS", "1") != "0"
        self.streams2 = tuple(torch.cuda.Stream(dev) for _ in range(2)) if on else None
        self.vp = round_up(cfg.vocab_size, 64)
        self.v_l = cfg.vocab_size
        self.lm_h = torch.zeros(self.max_logits, self.dp, dtype=self.dtype, device=dev)
        self.logits_buf = torch.zeros(self.max_logits, self.vp, dtype=torch.float32, device=dev)
        self.logits = self.logits_buf[:, :cfg.vocab_size]
        heads = max([a.heads * a.maps for a in att] + [a.heads for a in lat + talk], default=1)
        part = max([a.heads * a.maps * max(128, tc_head(a)) for a in att] + [a.heads * a.kv_rank for a in lat] +
                   [a.heads * talk_head(a) for a in talk], default=128)
        self.part_o = torch.zeros(max_seqs * max_splits * part, dtype=torch.float32, device=dev)
        self.part_ml = torch.zeros(max_seqs * heads * max_splits * 2, dtype=torch.float32, device=dev)
        widths = [self._in_width(L.mixer) for L in cfg.layers]
        self.proj = torch.zeros(max_tokens * max(widths), dtype=self.dtype, device=dev)
        self.proj_acc = (torch.zeros(max_tokens * max(widths), dtype=torch.float32, device=dev)
                         if self.dtype == torch.bfloat16 else None)
        self._buffers: dict = {}
        self._scratch: dict = {}
        self._moe: dict = {}
        self._rows: dict = {}
        self.latents: dict = {}       # runs of latent attention by layer
        self.gathered = None          # (pass, cache) of this step whose latents lie in the gather buffer
        self.k_cache: list = []
        self.v_cache: list = []
        self.states: list = []
        self.embed = self.bigram = self.head = self.out_norm = None
        self.sublayers: list = []
        self._rots: dict = {}         # device frequencies by RotarySpec
        self.layer_hook = None        # called with (layer run, summed streams [rows, width]) after every layer run

    # ------------------------------------------------------------------ sizes
    @staticmethod
    def _in_width(mix) -> int:
        if mix.kind == "parallel":
            n = HybridModel._in_width(mix.left) + (mix.right.width_p if mix.right.kind == "ssd" else mix.right.in_width)
            return round_up(n, 256 if n >= 2048 else 64)      # wide projections in whole tiles of the widest kind
        return round_up(mix.in_width, 64)

    @staticmethod
    def kv_block_bytes(cfg: ModelConfig, tp: int = 1, dtype: str = "bfloat16") -> int:
        """Device bytes of one 16-token KV block over all attention runs (0: no attention layers)."""
        total, size = 0, 2 if dtype == "bfloat16" else 4
        for a in (p for i in cfg.layer_runs for p in cfg.layers[i].mixer.parts):
            if a.kind == "latent_attention":
                total += 16 * a.cache_row * size if a.kv_from is None else 0
            elif a.kind == "talking_attention":
                dp = (talk_head(a) if dtype == "bfloat16" else 0) or round_up(a.dim, 8)
                total += 16 * (a.kv_heads * dp * size + 4)
            elif a.kind == "attention" and dtype == "bfloat16" and tc_head(a):
                total += a.kv_heads * 16 * 2 * tc_head(a) * 2
            elif a.kind == "attention":
                total += 16 * a.cache_values * size
        return total

    @staticmethod
    def state_bytes_per_seq(cfg: ModelConfig) -> int:
        return sum(4 * getattr(p, "state_elems", 0) for i in cfg.layer_runs for p in cfg.layers[i].mixer.parts)

    @staticmethod
    def step_bytes(cfg: ModelConfig, max_tokens: int, max_seqs: int) -> int:
        """Device bytes of a step's work space: streams, fp32 projections, rotated q / k, chunk states of
        retention, rows of the experts."""
        parts = [p for L in cfg.layers for p in L.mixer.parts]
        wide = max(p.width_p if p.kind == "ssd" else p.in_width if p.kind in ("min_gru", "talking_attention") else p.heads * getattr(p, "maps", 1) * (p.dim + p.vdim) for p in parts)
        chunk = max((p.state_elems for p in parts if p.kind in ("retention", "mlstm")), default=0)
        # gathered latents, keys and values of all heads in the largest pass
        lat = max((p.cache_row + p.heads * sum(latent_layout(p)[:2]) for p in parts if p.kind == "latent_attention"), default=0)
        n = max((4 * p.heads * 128 * (p.window + 256) + TALK_SCORE_BYTES for p in parts if p.kind == "talking_attention"), default=0)
        n += 2 * lat * max(KV_PASS_ROWS, max_tokens) + max_tokens * 4 * (max(1, cfg.streams) * cfg.d_model + 6 * wide) + 8 * (max_tokens // 128 + max_seqs) * chunk
        return n + max((HybridModel._moe_rows(L.mlp.experts, L.mlp.top, max_tokens) * 4 * (2 * cfg.d_model + L.mlp.ff)
                        for L in cfg.layers if L.mlp is not None and L.mlp.kind == "moe"), default=0)

    @staticmethod
    def _moe_rows(experts: int, top: int, max_tokens: int) -> int:
        """Rows of the expert buffers: 128-row slabs of every expert, or packed rows in whole 128-row tiles."""
        return max(experts * 128, (max_tokens * top + 127 * experts + 127) // 128 * 128)

    def moe_buffers(self, experts: int, top: int, fp: int) -> dict:
        """Work space of a mixture of experts, shared by the layers of one shape."""
        b = self._moe.get((experts, top, fp))
        if b is None:
            dev, n, T = self.device, self._moe_rows(experts, top, self.max_tokens), self.max_tokens
            i32 = dict(dtype=torch.int32, device=dev)
            b = {"weight": torch.zeros(T * top, device=dev), "expert": torch.zeros(T * top, **i32), "slot": torch.zeros(T * top, **i32),
                 "counts": torch.zeros(experts, **i32), "ticket": torch.zeros(1, **i32),
                 "act": torch.zeros(n, fp, dtype=self.dtype, device=dev), "out": torch.zeros(n, self.dp, dtype=self.dtype, device=dev)}
            if self.dtype == torch.bfloat16:
                b["xs"] = torch.zeros(n, self.dp, dtype=self.dtype, device=dev)
                b["logits"] = torch.zeros(T, round_up(experts, 64), device=dev)
            self._moe[experts, top, fp] = b
        return b

    def group_bn(self, m_tiles: int, n: int, whole: bool = False) -> int:
        """Tile width of an expert GEMM: narrow while the tiles would not fill the SMs; `whole`: a divisor of n."""
        for bn in (256, 128):
            if whole and n % bn:
                continue
            if m_tiles * ((n + bn - 1) // bn) >= self._sms:
                return bn
        return 64

    def buffer(self, key: tuple, width: int) -> torch.Tensor:
        """[max_tokens, width] activation rows of one layout. Columns that no kernel of that layout writes
        (padding of heads or rows) stay zero, which is why layouts do not share memory."""
        b = self._buffers.get(key)
        if b is None:
            b = self._buffers[key] = torch.zeros(self.max_tokens, width, dtype=self.dtype, device=self.device)
        return b

    def maps_buffer(self, width: int) -> torch.Tensor:
        """fp32 rows of both maps of differential attention, shared by the layers of one width."""
        return self._f32_rows("maps", width)

    def gates_buffer(self, width: int) -> torch.Tensor:
        return self._f32_rows("gates", width)

    def _f32_rows(self, name: str, width: int) -> torch.Tensor:
        b = self._buffers.get((name, width))
        if b is None:
            b = self._buffers[name, width] = torch.zeros(self.max_tokens, width, dtype=torch.float32, device=self.device)
        return b

    def rows(self, name: str, n: int, width: int) -> torch.Tensor:
        """[n, width] rows of prompt steps in the model's dtype, grown on demand; never uninitialised memory."""
        b = self._rows.get(name)
        if b is None or b.numel() < n * width:
            self._rows[name] = b = torch.zeros(n * width, dtype=self.dtype, device=self.device)
        return b[:n * width].view(n, width)

    def scratch(self, name: str, n: int) -> torch.Tensor:
        """fp32 work space of prompt chunks (steps that are never captured in a graph), grown on demand."""
        b = self._scratch.get(name)
        if b is None or b.numel() < n:
            self._scratch[name] = b = torch.empty(n, dtype=torch.float32, device=self.device)
        return b[:n]

    # ------------------------------------------------------------------ weights
    def _pad(self, w: torch.Tensor) -> torch.Tensor:
        n, k = w.shape
        np_, kp = round_up(n, 64), round_up(k, 64)
        if (np_, kp) != (n, k):
            out = torch.zeros(np_, kp, dtype=w.dtype, device=w.device)
            out[:n, :k] = w
            w = out
        return ops.tile_weight(w) if self.tile_weights and self.dtype == torch.bfloat16 else w.contiguous()

    def _ssd_weights(self, r, p: str, mat, vec) -> dict:
        """Tensors of a state-space layer in the padded channel layout (z | x | B | C | dt; zero rows as padding)."""
        def blocks(t: torch.Tensor, n: int, k: int, kp: int) -> torch.Tensor:
            """n blocks of k rows -> n blocks of kp."""
            out = t.new_zeros(n, kp, *t.shape[1:])
            out[:, :k] = t.view(n, k, *t.shape[1:])
            return out.flatten(0, 1)

        inner, gn = r.inner, r.groups * r.state

        def channels(t: torch.Tensor) -> torch.Tensor:
            x, b, c = t.split([inner, gn, gn])
            return torch.cat([blocks(x, r.heads, r.vdim, r.vdim_p), blocks(b, r.groups, r.state, r.state_p),
                              blocks(c, r.groups, r.state, r.state_p)])

        w = mat(p + "in")
        z, xbc, dt = w.split([inner, inner + 2 * gn, r.heads])
        return {"in": torch.cat([blocks(z, r.heads, r.vdim, r.vdim_p), channels(xbc), dt]),
                "ssd": tuple(t.contiguous() for t in (channels(vec(p + "conv")), channels(vec(p + "conv.b")), vec(p + "dt_bias"),
                                                      vec(p + "A_log"), vec(p + "D"))),
                "norm": vec(p + "norm"), "w_o": self._pad(mat(p + "o"))}

    def _moe_weights(self, e, p: str, mat) -> dict:
        fp = round_up(e.ff, 64)
        kw = dict(dtype=self.dtype, device=self.device)
        up, down = torch.zeros(e.experts, (2 if e.glu else 1) * fp, self.dp, **kw), torch.zeros(e.experts, self.dp, fp, **kw)
        router = torch.zeros(round_up(e.experts, 64), self.dp, **kw)
        d = self.cfg.d_model
        for i in range(e.experts):
            if e.glu:
                g, u = (torch.cat([t, t.new_zeros(fp - e.ff, d)]) for t in (mat(f"{p}e{i}.gate"), mat(f"{p}e{i}.up")))
                up[i, :, :d] = interleave32(g, u)
            else:
                up[i, :e.ff, :d] = mat(f"{p}e{i}.up")
            down[i, :d, :e.ff] = mat(f"{p}e{i}.down")
        router[:e.experts, :d] = mat(p + "router")
        return {"up": up, "down": down, "router": router[:e.experts], "router_p": router}

    def _rotary(self, spec) -> hops.Rotary:
        if spec not in self._rots:
            self._rots[spec] = hops.Rotary(spec, self.device)
        return self._rots[spec]

    def _mixer_weights(self, mx, p: str, mat, vec) -> dict:
        if mx.kind == "latent_attention":
            return self._latent_weights(mx, p, mat, vec)
        if mx.kind == "talking_attention":
            return self._talking_weights(mx, p, mat, vec)
        if mx.kind == "parallel":
            return self._pair_weights(mx, p, mat, vec)
        names = ("q", "k", "v") if mx.kind == "attention" else ("q", "k", "v", "g")
        w = {"w_in": self._pad(torch.cat([mat(p + n) for n in names])), "w_o": self._pad(mat(p + "o")),
             "rot": self._rotary(getattr(mx, "rot", None)), "q_norm": None, "k_norm": None}
        if mx.kind == "attention":
            if mx.qk_norm == "projection":
                w["q_norm"], w["k_norm"] = vec(p + "q.norm"), vec(p + "k.norm")
            if mx.bias:
                w["bias"] = torch.cat([vec(f"{p}{n}.b") for n in names])
            if mx.diff is not None:
                a, b, c, d = (vec(p + n).double().cpu() for n in ("lq1", "lk1", "lq2", "lk2"))
                w["lam"] = float(torch.exp((a * b).sum()) - torch.exp((c * d).sum())) + mx.diff
        elif mx.kind == "retention":
            w["decay_pow"] = hops.decay_powers(mx.decay, self.device)
        elif mx.kind == "mlstm":
            z = torch.cat([mat(p + "i"), mat(p + "f")])
            wz = z.new_zeros(round_up(z.shape[0], 64), self.dp)
            wz[:z.shape[0], :z.shape[1]] = z
            w.update(w_z=wz, z_bias=torch.cat([vec(p + "i.b"), vec(p + "f.b")]), norm=vec(p + "norm"))
        return w

    def _talking_weights(self, a, p: str, mat, vec) -> dict:
        """The keys' norm weights are part of the queries' (fp32 products), the distance biases a table of the mixed heads."""
        q, k, g = mat(p + "q"), mat(p + "k"), mat(p + "g")
        w_in = q.new_zeros(a.in_width, q.shape[1])
        w_in[:q.shape[0]], w_in[q.shape[0]:q.shape[0] + k.shape[0]], w_in[a.gate_col:] = q, k, g
        wk = vec(p + "k.norm").view(a.kv_heads, 1, a.dim).expand(a.kv_heads, a.heads // a.kv_heads, a.dim).reshape(-1)
        talk = mat(p + "talk").float().contiguous()      # a matrix: of the model's dtype, like the others
        far = 16 * self.max_blocks_per_seq      # no distance is larger
        far = min(a.window, far) if a.window else far
        return {"w_in": self._pad(w_in), "w_o": self._pad(mat(p + "o")), "rot": self._rotary(None), "q_norm": (vec(p + "q.norm") * wk).contiguous(),
                "talk": talk, "bias": hops.talk_bias(talk, vec(p + "r1"), vec(p + "r2"), far)}

    def _pair_weights(self, mx, p: str, mat, vec) -> dict:
        """q | k | v of the attention, then z | x | g of the recurrence; the output matrices side by side."""
        a, r = mx.left, mx.right
        rows = [mat(f"{p}left.{n}") for n in ("q", "k", "v")]
        w_in = rows[0].new_zeros(self._in_width(mx), rows[0].shape[1])
        w_in[:a.in_width] = torch.cat(rows)
        at, bias = round_up(a.in_width, 64), torch.zeros(2, r.width_p, dtype=torch.float32, device=self.device)
        for i, n in enumerate(("z", "x", "g")):
            w_in[at + i * r.width_p:at + i * r.width_p + r.width] = mat(f"{p}right.{n}")
            if n != "g":
                bias[i, :r.width] = vec(f"{p}right.{n}.b")
        lo, ro = mat(p + "left.o"), mat(p + "right.o")
        lk = round_up(a.out_dim, 64)
        w_o = lo.new_zeros(lo.shape[0], lk + round_up(r.out_dim, 64))
        w_o[:, :a.out_dim], w_o[:, lk:lk + r.out_dim] = lo, ro
        return {"w_in": self._pad(w_in), "w_o": self._pad(w_o), "right": {"bias": bias.view(-1)},
                "left": {"rot": self._rotary(a.rot), "q_norm": None, "k_norm": None, "sinks": vec(p + "left.sink")}}

    def _latent_weights(self, a, p: str, mat, vec) -> dict:
        """Tensors of latent attention in the head layouts of LatentRun. The expansion of a step's latents to keys takes the
        rotated part through a unit matrix, so one product makes whole keys and values."""
        H, R, D, T, E = a.heads, a.kv_rank, a.dim, a.rot_dim, a.vdim
        dk, dv, at = latent_layout(a)
        d8, r8, ep = round_up(D, 8), round_up(R, 8), round_up(E, 8)
        uq, uk, uv = mat(p + "uq").view(H, D + T, a.q_rank), mat(p + "uk").view(H, D, R), mat(p + "uv").view(H, E, R)
        q = uq.new_zeros(H, dk, a.q_rank)
        q[:, :T], q[:, at:at + D] = uq[:, D:], uq[:, :D]
        k = uk.new_zeros(H, R, d8)
        k[:, :, :D] = uk.transpose(1, 2)
        v = uv.new_zeros(H, ep, r8)
        v[:, :E, :R] = uv
        o = mat(p + "o").view(-1, H, E)
        wo = o.new_zeros(o.shape[0], H, ep)
        wo[:, :, :E] = o
        dq = mat(p + "dq")
        rows = [dq, dq.new_zeros(a.kv_col - a.q_rank, dq.shape[1])] + ([mat(p + "dkv")] if a.kv_from is None else [])
        w = {"w_in": self._pad(torch.cat(rows)), "w_uq": self._pad(q.flatten(0, 1)), "w_uk": k, "w_uv": v,
             "w_o": self._pad(wo.flatten(1)), "rot": self._rotary(a.rot), "q_norm": vec(p + "dq.norm"),
             "kv_norm": vec(p + "dkv.norm") if a.kv_from is None else None}
        if dv and self.dtype == torch.bfloat16:
            kv = uk.new_zeros(H * (dk + dv), a.cache_row)
            keys, values = kv[:H * dk].view(H, dk, -1), kv[H * dk:].view(H, dv, -1)
            keys[:, at:at + D, :R], values[:, :E, :R] = uk, uv
            for t in range(T):
                keys[:, t, R + t] = 1.0
            w["w_kv"] = ops.tile_weight(kv) if self.tile_weights else kv
        return w

    def _mlp_weights(self, f, p: str, mat) -> dict:
        if f.kind == "moe":
            return self._moe_weights(f, p, mat)
        if not f.glu:
            return {"w_gu": self._pad(mat(p + "up")), "w_down": self._pad(mat(p + "down"))}
        ip = round_up(f.ff, 64)
        g, u = mat(p + "gate"), mat(p + "up")
        if ip != f.ff:   # whole units of the interleaved layout; act(0) * 0 adds nothing
            g, u = (torch.cat([t, t.new_zeros(ip - f.ff, t.shape[1])]) for t in (g, u))
        gu = interleave32(g, u) if self.dtype == torch.bfloat16 else torch.cat([g, u])
        return {"w_gu": self._pad(gu), "w_down": self._pad(mat(p + "down"))}

    def _build_sandwich(self, mat, vec) -> None:
        """Layers with a norm on either side of every sublayer; the layer scale is part of the second one's weight."""
        self.k_cache, self.v_cache, self.states, self.sublayers, self.latents = [], [], [], [], {}
        for i, L in enumerate(self.cfg.layers):
            p = f"l{i}."
            norms = [(vec(f"{p}norm{q}"), vec(f"{p}norm{q}b") * vec(f"{p}ls{q}")) for q in range(1, L.sublayers + 1)]
            mixer = RUNS[L.mixer.kind](self, L.mixer, self._mixer_weights(L.mixer, p + "mix.", mat, vec))
            if L.mixer.kind == "latent_attention":
                self.latents[i] = mixer
            self.sublayers.append(_NormedSublayer(*norms[0], mixer, i if L.mlp is None else -1))
            if L.mlp is not None:
                self.sublayers.append(_NormedSublayer(*norms[1], MLP_RUNS[L.mlp.kind](self, L.mlp, self._mlp_weights(L.mlp, p + "mlp.", mat)), i))
        torch.cuda.empty_cache()

    def _build_single(self, mat, vec) -> None:
        """Layers over one plain residual stream, with the entries of the loop's passes."""
        cfg, m = self.cfg, self.cfg.residual_mult
        self.k_cache, self.v_cache, self.states, self.sublayers = [], [], [], []
        entry, starts = None, cfg.pass_starts if cfg.loop_inject else {}
        if starts:
            w, d = mat("loop.in"), cfg.d_model
            x, x0 = w[:, :d], w[:, d:]
            parts = [x, x, x0] if self.dtype == torch.bfloat16 else [x, x0]
            wide = w.new_zeros(d, len(parts) * self.dp)
            for i, t in enumerate(parts):
                wide[:, i * self.dp:i * self.dp + d] = t
            entry, step = EntryRun(self, self._pad(wide)), vec("loop.step")
        ws = [(self._mixer_weights(L.mixer, f"l{i}.mix.", mat, vec), self._mlp_weights(L.mlp, f"l{i}.mlp.", mat) if L.mlp is not None else None,
               [vec(f"l{i}.norm{q}") for q in range(1, L.sublayers + 1)]) for i, L in enumerate(cfg.layers)]
        for ri, li in enumerate(cfg.layer_runs):
            L, (w, mw, norms) = cfg.layers[li], ws[li]
            if ri in starts:
                self.sublayers.append(_NormedSublayer(None, None, entry, -1, base=step[starts[ri]].contiguous()))
            self.sublayers.append(_NormedSublayer(norms[0], None, RUNS[L.mixer.kind](self, L.mixer, w), ri if mw is None else -1, gain=m))
            if mw is not None:
                self.sublayers.append(_NormedSublayer(norms[1], None, MLP_RUNS[L.mlp.kind](self, L.mlp, mw), ri, gain=m))
        torch.cuda.empty_cache()

    def _build_parallel(self, get) -> None:
        """Layers whose mixer and feed-forward run side by side."""
        mat = lambda name: get(name, False)
        vec = lambda name: get(name, True).contiguous()
        self.embed, self.head, self.out_norm = mat("embed").contiguous(), self._pad(mat("head")), vec("final.norm")
        self.k_cache, self.v_cache, self.states, self.sublayers = [], [], [], []
        for i, L in enumerate(self.cfg.layers):
            p, mx = f"l{i}.", L.mixer
            a = mx.left
            q = torch.cat([mat(f"{p}mix.left.{n}") for n in ("q", "k", "v")])
            ssd = self._ssd_weights(mx.right, p + "mix.right.", mat, vec)
            right = ssd.pop("in")
            w_in = q.new_zeros(self._in_width(mx), q.shape[1])
            w_in[:q.shape[0]] = q
            at = round_up(q.shape[0], 64)
            w_in[at:at + right.shape[0]] = right
            w = {"w_in": self._pad(w_in), "right": ssd,
                 "left": {"rot": self._rotary(a.rot), "q_norm": None, "k_norm": None, "w_o": self._pad(mat(p + "mix.left.o"))}}
            mlp = MoeRun(self, L.mlp, self._moe_weights(L.mlp, p + "mlp.", mat)) if L.mlp is not None else None
            norms = [vec(p + "norm1")] + ([vec(p + "norm2")] if mlp is not None else [])
            out = (vec(p + "mix.left.out"), vec(p + "mix.right.out"))
            self.sublayers.append(_ParallelLayer(norms, out, ParallelRun(self, mx, w, mlp)))
        torch.cuda.empty_cache()

    def _build(self, get) -> None:
        """`get(name, fp32)` returns a named tensor on the device, in fp32 or in the model's dtype."""
        if self.parallel:
            return self._build_parallel(get)
        cfg = self.cfg
        mat = lambda name: get(name, False)
        vec = lambda name: get(name, True).contiguous()
        self.embed = mat("embed").contiguous()
        self.bigram = mat("bigram").contiguous() if cfg.bigram is not None else None
        self.head = self._pad(mat("embed" if cfg.tie_embeddings else "head"))
        self.out_norm = vec("final.norm") * cfg.logit_scale - cfg.norm_weight_offset * (1.0 - cfg.logit_scale)
        if cfg.residual_mult is not None:
            return self._build_single(mat, vec)
        if self.sandwich:
            return self._build_sandwich(mat, vec)
        one = torch.ones(1, dtype=torch.float32, device=self.device)

        def hc(p: str, q: int) -> dict:
            if not cfg.streams:
                return {"in": one, "out": one, "mix": one}
            return {k: vec(f"{p}hc{q}.{k}") for k in ("in", "out", "mix")}

        layers = []
        for i, L in enumerate(cfg.layers):
            p = f"l{i}."
            w = self._mixer_weights(L.mixer, p + "mix.", mat, vec)
            subs = [(vec(p + "norm1"), hc(p, 1))]
            mw = None
            if L.mlp is not None:
                mw = self._mlp_weights(L.mlp, p + "mlp.", mat)
                subs.append((vec(p + "norm2"), hc(p, 2)))
            layers.append((L, w, mw, subs))
        self.k_cache, self.v_cache, self.states, self.sublayers = [], [], [], []
        for ri, li in enumerate(cfg.layer_runs):
            L, w, mw, subs = layers[li]
            self.sublayers.append(_Sublayer(*subs[0], RUNS[L.mixer.kind](self, L.mixer, w), ri if mw is None else -1))
            if mw is not None:
                self.sublayers.append(_Sublayer(*subs[1], MlpRun(self, L.mlp, mw), ri))
        torch.cuda.empty_cache()

    def load(self, src: WeightSource) -> None:
        def get(name: str, f32: bool) -> torch.Tensor:
            t = torch.from_numpy(np.ascontiguousarray(src.f32(name), dtype=np.float32)).to(self.device)
            return t if f32 else t.to(self.dtype)

        self._build(get)

    def init_random(self, seed: int = 0, std: float = 0.02) -> None:
        """Random weights generated on the device (benchmarks): N(0, std) matrices, unit norms, and
        hyper-connections that act as a plain residual."""
        from .layer_spec import initial_matrix, initial_vector, layer_list_tensors

        g = torch.Generator(device=self.device)
        g.manual_seed(seed)
        shapes = dict(layer_list_tensors(self.cfg))

        def get(name: str, f32: bool) -> torch.Tensor:
            shape = shapes[name]
            if ".hc" in name:
                s = self.streams
                t = torch.eye(s) if name.endswith(".mix") else torch.full(shape, 1.0 / s if name.endswith(".in") else 1.0)
                return t.to(self.device)
            if len(shape) == 1:
                return torch.from_numpy(initial_vector(self.cfg, name, shape)).to(self.device)
            t = torch.empty(*shape, dtype=torch.float32 if f32 else self.dtype, device=self.device)
            t = t.normal_(0.0, self.cfg.d_model ** -0.5 if name.endswith(".router") else std, generator=g)
            start = initial_matrix(name, shape)
            return t if start is None else t + torch.from_numpy(start).to(t)

        self._build(get)

    # ------------------------------------------------------------------ streams
    def side_streams(self, s: StepInputs) -> bool:
        """Whether the parts of a layer run on streams of their own: small decode steps that are being captured."""
        return (self.streams2 is not None and s.n_prefill == 0 and s.m <= 128 and self.dtype == torch.bfloat16
                and torch.cuda.is_current_stream_capturing())

    @contextmanager
    def full_dependency(self):
        """Launches inside take no programmatic dependency (the ones of this module's kernels)."""
        hops.set_pdl(False)
        try:
            yield
        finally:
            hops.set_pdl(self._pdl)

    # ------------------------------------------------------------------ projections
    def few_rows(self, M: int) -> bool:
        """A handful of rows takes the weight-streaming GEMV instead of 128-row MMA tiles."""
        return M <= self.gemv_max_rows

    def _proj_splits(self, M: int, sub: Optional[_Sublayer]) -> Optional[torch.Tensor]:
        """The fp32 accumulator rows that the next sublayer's input GEMM will add its K splits into (they
        are cleared by the stream_norm before it), or None when that GEMM stores its result."""
        width = getattr(sub.run, "width", 0) if sub is not None else 0
        if not width or self.dtype == torch.float32 or self.few_rows(M):
            return None
        n = round_up(width, 64)
        gc = self._gemm_shape(M, n, self.dp)
        return self.proj_acc[:M * n].view(M, n) if gc["splits"] > 1 and not gc["fixup"] else None

    def project(self, h: torch.Tensor, w: torch.Tensor, width: int) -> torch.Tensor:
        """h @ w^T of a mixer's stacked input projections; fp32 when the GEMM splits K, else the model's dtype."""
        M, n = h.shape[0], round_up(width, 64)
        out = self.proj[:M * n].view(M, n)
        if self.dtype == torch.float32:
            hops.gemm_f32(h, w, out)
        elif self.few_rows(M):
            ops.gemv(h, w, out)
        else:
            gc = self._gemm_shape(M, n, self.dp)
            if gc["splits"] > 1 and not gc["fixup"]:
                out = self.proj_acc[:M * n].view(M, n)
                ops.gemm(h, w, epi=ops.EPI_RED_F32, dst_ptrs=[out.data_ptr()], **gc)
            else:
                ops.gemm(h, w, out=out, **gc)
        return out

    def product(self, x: torch.Tensor, w: torch.Tensor, out: torch.Tensor) -> None:
        """out[:M] = x @ w^T in the model's dtype."""
        M, k = x.shape
        n = w.shape[0] * 128 if w.dim() == 4 else w.shape[0]
        out = out[:M, :n]
        if self.dtype == torch.float32:
            hops.gemm_f32(x, w, out)
        elif self.few_rows(M):
            ops.gemv(x, w, out)
        else:
            ops.gemm(x, w, out=out, **self._gemm_shape(M, n, k, store=True))

    def product_f32(self, x: torch.Tensor, w: torch.Tensor, out: torch.Tensor) -> None:
        """out = x @ w^T in fp32, w row-major."""
        M, k = x.shape
        if self.dtype == torch.float32:
            hops.gemm_f32(x, w, out)
        elif self.few_rows(M):
            ops.gemv(x, w, out)
        else:
            ops.gemm(x, w, out=out, epi=ops.EPI_STORE_F32, **self._gemm_shape(M, w.shape[0], k, store=True))

    def per_head(self, x: torch.Tensor, w: torch.Tensor, out: torch.Tensor) -> None:
        """out[h] = x[h] @ w[h]^T: x [heads, M, K] and out [heads, M, N] views of rows, w [heads, N, K]."""
        if self.dtype == torch.float32:
            for h in range(w.shape[0]):
                hops.gemm_f32(x[h], w[h], out[h])
        else:
            ops.gemm(x, w, out=out, bn=128 if w.shape[0] * w.shape[1] >= 128 * self._sms else 64)

    def adds_up(self, M: int, k: int) -> bool:
        """Whether an output projection of K = k splits K and adds its parts into the accumulator (which then has
        to be zero); otherwise it stores."""
        return (self.dtype == torch.bfloat16 and not self.few_rows(M)
                and self._gemm_shape(M, self.dp, k, routed=True)["splits"] > 1)

    def into_branch(self, b: int, x: torch.Tensor, w: torch.Tensor) -> None:
        """branches[b] = x @ w^T (fp32)."""
        M, k = x.shape
        if not self.adds_up(M, k) and self.dtype == torch.bfloat16 and not self.few_rows(M):
            ops.gemm(x, w, out=self.branches[b, :M], epi=ops.EPI_STORE_F32, **self._gemm_shape(M, self.dp, k, routed=True))
        else:
            self.into_acc(x, w, self.branches[b])

    def into_acc(self, x: torch.Tensor, w: torch.Tensor, acc: Optional[torch.Tensor] = None) -> None:
        """acc = x @ w^T (fp32). The accumulator is zero here: stream_norm clears what it has read, branch_norm where
        the next product adds its splits up."""
        M, k = x.shape
        if acc is None and self.single:
            return self.into_branch(0, x, w)
        acc = (self.acc if acc is None else acc)[:M]
        if self.dtype == torch.float32:
            hops.gemm_f32(x, w, acc)
        elif self.few_rows(M):
            ops.gemv(x, w, acc)
        else:
            ops.gemm(x, w, epi=ops.EPI_RED_F32, dst_ptrs=[acc.data_ptr()], rows_per_owner=M,
                     **self._gemm_shape(M, self.dp, k, routed=True))

    # ------------------------------------------------------------------ forward
    def forward(self, s: StepInputs, hidden_in: Optional[torch.Tensor] = None) -> torch.Tensor:
        """Runs one step; returns fp32 logits [n_logits, vocab] (a view of a static buffer; steps with more
        logit rows than the buffer holds get one of their own)."""
        if self.parallel:
            return self._forward_parallel(s)
        if self.single:
            return self._forward_single(s)
        cfg, M = self.cfg, s.m
        h = self.h[:M]
        subs = self.sublayers
        bg = cfg.bigram
        hops.stream_norm(self.x, M, tokens=s.token_ids, prev=s.prev_ids if bg is not None else None, embed=self.embed,
                         bigram=self.bigram, mul_prev=bg.mul_prev if bg else 0, mul_cur=bg.mul_cur if bg else 0,
                         in_w=subs[0].hc["in"], norm_w=subs[0].norm, eps=cfg.rms_eps, h=h,
                         clear=self._proj_splits(M, subs[0]))
        n_log = max(s.n_logits, 1)
        lm_h, logits = self._logit_rows(n_log)
        for i, sub in enumerate(subs):
            sub.run(s, h)
            kw = dict(y=self.acc, mix=sub.hc["mix"], out_w=sub.hc["out"], eps=cfg.rms_eps)
            if i + 1 < len(subs):
                nxt = subs[i + 1]
                hops.stream_norm(self.x, M, in_w=nxt.hc["in"], norm_w=nxt.norm, h=h, clear=self._proj_splits(M, nxt), **kw)
            else:
                hops.stream_norm(self.x, M, in_w=None, norm_w=self.out_norm, h=lm_h, row_map=s.logit_map,
                                 store_x=self.layer_hook is not None, **kw)
            if self.layer_hook is not None and sub.last_of >= 0:
                self.layer_hook(sub.last_of, self.x[:M].sum(1))
        return self._head(lm_h, logits, n_log)

    def _forward_parallel(self, s: StepInputs) -> torch.Tensor:
        cfg, M, layers = self.cfg, s.m, self.sublayers
        h, h2 = self.h[:M], self.h2[:M]
        x = self.x.view(self.max_tokens, -1)
        n_log = max(s.n_logits, 1)
        lm_h, logits = self._logit_rows(n_log)
        experts = None
        for i in range(len(layers) + 1):
            # what the layer before left, into the residual; then the norms of this one (or of the head)
            last = i == len(layers)
            clears = (False, False) if last else layers[i].run.clears(M)
            kw = dict(eps=cfg.rms_eps, w_offset=cfg.norm_weight_offset)
            if i == 0:
                kw.update(tokens=s.token_ids, embed=self.embed, embed_scale=cfg.emb_scale)
                out = (None, None)
            else:
                kw.update(experts=experts)
                out = layers[i - 1].out
            kw["branches"] = [(self.branches[b], out[b], 0.5, clears[b]) for b in range(2)]
            if last:
                kw.update(norm_w=[self.out_norm], h=[lm_h], row_map=s.logit_map, store_x=self.layer_hook is not None)
            else:
                norms = layers[i].norms
                kw.update(norm_w=norms, h=[h, h2][:len(norms)], clear=self._proj_splits(M, layers[i]))
            joins = i > 0 and self.side_streams(s)
            with self.full_dependency() if joins else nullcontext():
                hops.branch_norm(x, M, **kw)
            if self.layer_hook is not None and i > 0:
                self.layer_hook(i - 1, x[:M])
            if not last:
                experts = layers[i].run(s, h, h2)
        return self._head(lm_h, logits, n_log)

    def _forward_single(self, s: StepInputs) -> torch.Tensor:
        cfg, M, subs = self.cfg, s.m, self.sublayers
        h = self.h[:M]
        x = self.x.view(self.max_tokens, -1)
        n_log = max(s.n_logits, 1)
        lm_h, logits = self._logit_rows(n_log)
        experts = self.gathered = None
        for i in range(len(subs) + 1):
            # what the sublayer before left into the residual (through its norm, where it has one); then the norm of this one (or
            # of the head), or the operand rows of the entry of a pass
            last = i == len(subs)
            # the accumulator has to be zero when the next sublayer that adds its splits up in it starts
            user = next((t.run.acc_k for t in subs[i:] if t.run.acc_k), 0)
            clear = bool(user) and self.adds_up(M, user)
            kw = dict(eps=cfg.rms_eps, w_offset=cfg.norm_weight_offset)
            if i == 0:
                kw.update(tokens=s.token_ids, embed=self.embed, embed_scale=cfg.emb_scale, branches=[(self.acc, None, 1.0, clear)])
            elif subs[i - 1].run.acc_k:
                kw.update(branches=[(self.acc, subs[i - 1].out, subs[i - 1].gain, clear)], base=subs[i - 1].base)
            else:
                kw.update(branches=[(None, subs[i - 1].out, 1.0, False)], experts=experts)
            if not last and subs[i].base is not None:
                kw.update(norm_w=(), h=(), split=subs[i].run.rows(), split_off=self.dp, x0_tokens=s.token_ids, embed=self.embed,
                          embed_scale=cfg.emb_scale)
            elif last:
                kw.update(norm_w=[self.out_norm], h=[lm_h], row_map=s.logit_map, store_x=self.layer_hook is not None)
            else:
                kw.update(norm_w=[subs[i].norm], h=[h], clear=self._proj_splits(M, subs[i]))
            hops.branch_norm(x, M, **kw)
            if self.layer_hook is not None and i > 0 and subs[i - 1].last_of >= 0:
                self.layer_hook(subs[i - 1].last_of, x[:M])
            if not last:
                experts = subs[i].run(s, h)
        return self._head(lm_h, logits, n_log)

    def _logit_rows(self, n_log: int) -> tuple:
        """Static buffers of the normed logit rows and the logits; larger ones for a step that has more of them."""
        if n_log <= self.max_logits:
            return self.lm_h, self.logits_buf
        return (torch.zeros(n_log, self.dp, dtype=self.dtype, device=self.device),
                torch.empty(n_log, self.vp, dtype=torch.float32, device=self.device))

    def _head(self, lm_h: torch.Tensor, logits: torch.Tensor, n_log: int) -> torch.Tensor:
        lm_h, logits = lm_h[:n_log], logits[:n_log]
        if self.dtype == torch.float32:
            hops.gemm_f32(lm_h, self.head, logits)
        elif self.few_rows(n_log):
            ops.gemv(lm_h, self.head, logits)
        else:
            ops.gemm(lm_h, self.head, out=logits, epi=ops.EPI_STORE_F32, **self._gemm_shape(n_log, self.vp, self.dp, store=True))
        if self.cfg.logit_softcap:
            ops.softcap(logits, self.cfg.logit_softcap)
        return logits[:, :self.cfg.vocab_size]

    # ------------------------------------------------------------------ state
    def copy_blocks(self, src: torch.Tensor, dst: torch.Tensor) -> None:
        """Copies KV blocks src[i] -> dst[i] in every cache (copy on write)."""
        s, d = src.long(), dst.long()
        for c in (*self.k_cache, *self.v_cache):
            c.index_copy_(0, d, c.index_select(0, s))

    def enable_block_mass(self) -> None:
        raise ConfigError(f"{self.cfg.name}: heavy-hitter pruning is built for the Llama family")

    def reset_sync_state(self) -> None:
        """Clears what kernels accumulate into, after a step that a device error cut short."""
        torch.cuda.synchronize(self.device)
        self.branches.zero_()
        for b in self._moe.values():
            b["counts"].zero_()
            b["ticket"].zero_()
        if self.proj_acc is not None:
            self.proj_acc.zero_()
        ops.gemm_workspace(self.device)[1].zero_()
        torch.cuda.synchronize(self.device)

    def close(self) -> None:
        self._buffers.clear()
        self._moe.clear()
        self._scratch.clear()
        self._rows.clear()
