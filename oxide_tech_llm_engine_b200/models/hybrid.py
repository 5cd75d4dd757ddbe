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

In a captured decode step the three lines between two branch_norms run on streams of their own: the
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


class _Sublayer:
    """What stream_norm needs around a sublayer, and the function that runs it."""

    def __init__(self, norm, hc, run, last_of: int):
        self.norm, self.hc, self.run = norm, hc, run
        self.last_of = last_of       # index of the layer run that this sublayer ends, or -1


class _ParallelLayer:
    """Norm weights of the layer's inputs (mixer, feed-forward), of its two mixer outputs, and the function that runs it."""

    def __init__(self, norms: list, out: tuple, run):
        self.norms, self.out, self.run = norms, out, run


class AttentionRun:
    """One run of an attention layer: weights shared by all passes, a KV cache of its own. Its projection rows
    may be the first columns of wider ones (a layer with two mixers)."""

    def __init__(self, m: "HybridModel", spec, w: dict):
        self.m, self.spec, self.w = m, spec, w
        a = spec
        self.group = a.heads // a.kv_heads
        self.width = a.heads * a.dim + a.kv_heads * (a.dim + a.vdim)
        big = max(a.dim, a.vdim)
        # head sizes of the tensor-core kernels: q, k and v padded to 64 or 128 with zeros
        self.tc = m.dtype == torch.bfloat16 and big <= 128 and self.group <= 16
        self.dp, self.ep = (64 if big <= 64 else 128,) * 2 if self.tc else (a.dim, a.vdim)
        self.k = torch.zeros(m.num_blocks, a.kv_heads, 16, self.dp, dtype=m.dtype, device=m.device)
        self.v = torch.zeros(m.num_blocks, a.kv_heads, 16, self.ep, dtype=m.dtype, device=m.device)
        m.k_cache.append(self.k)
        m.v_cache.append(self.v)

    def __call__(self, s: StepInputs, h: torch.Tensor) -> None:
        self.m.into_acc(self.attend(s, self.m.project(h, self.w["w_in"], self.width)), self.w["w_o"])

    def attend(self, s: StepInputs, proj: torch.Tensor) -> torch.Tensor:
        m, a, w, M = self.m, self.spec, self.w, s.m
        q = m.buffer(("q", a.heads * self.dp, a.dim), a.heads * self.dp)
        hops.heads(proj, M, h=a.heads, g=a.kv_heads, d=a.dim, e=a.vdim, rot=w["rot"], positions=s.positions, q_out=q,
                   q_hd=self.dp, q_norm=w["q_norm"], k_norm=w["k_norm"], eps=m.cfg.rms_eps, k_cache=self.k,
                   v_cache=self.v, slots=s.slot_mapping)
        out = m.buffer(("o", a.out_dim), round_up(a.out_dim, 64))
        nd = s.n_decode
        kw = dict(window=a.window, keep_first=a.keep_first if a.window else 0, scale=a.scale, chunk=a.chunk,
                  sink=-math.inf if a.sink is None else a.sink)
        if self.tc:
            kw.update(out_d=a.vdim, exact_p=True)
            if nd > 0:
                ops.paged_decode(q[:nd].view(nd, a.heads, self.dp), self.k, self.v, s.block_tables, s.seq_lens,
                                 s.pages_per_split, m.part_o, m.part_ml, out[:nd], batch=nd, max_splits=m.max_splits, **kw)
            if s.n_prefill > 0:
                ops.paged_prefill(q.view(-1, a.heads, self.dp), self.k, self.v, s.prefill_block_tables, s.tile_seq, s.tile_q0,
                                  s.q_start, s.q_lens, s.ctx_lens, out, n_tiles=s.n_tiles, **kw)
        else:
            kw.update(h=a.heads, d=a.dim, e=a.vdim, out=out)
            if nd > 0:
                hops.row_attention(q, self.dp, self.k, self.v, s.block_tables, n=nd, seq_lens=s.seq_lens, **kw)
            if s.n_prefill > 0:
                hops.row_attention(q, self.dp, self.k, self.v, s.prefill_block_tables, n=s.n_tiles, tile_seq=s.tile_seq,
                                   tile_q0=s.tile_q0, q_start=s.q_start, q_lens=s.q_lens, ctx_lens=s.ctx_lens, **kw)
        return out[:M]


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
        self.b = m.moe_buffers(spec.experts, spec.top, self.fp)

    def __call__(self, s: StepInputs, h: torch.Tensor, start=nullcontext()) -> tuple:
        m, e, w, b, M = self.m, self.spec, self.w, self.b, s.m
        E, top = e.experts, e.top
        route = dict(e=E, top=top, weight=b["weight"], expert=b["expert"], slot=b["slot"])
        if m.dtype == torch.float32 or m.few_rows(M):
            with start:
                hops.moe_route(h, w["router"], M, **route)
            pairs = M * top
            rows, act = b["out"][:pairs], b["act"][:pairs]
            hops.moe_rows(h, w["up"], b["expert"], pairs, top=top, per_pair=False, y=act, act=2)
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
        self.ip = round_up(spec.ff, 64)
        self.act = 1 if spec.act == "gelu_tanh" else 0

    def __call__(self, s: StepInputs, h: torch.Tensor) -> None:
        m, M = self.m, s.m
        act = m.buffer(("act", self.ip), self.ip)
        w = self.w["w_gu"]
        if m.dtype == torch.float32:
            gu = m.scratch("gate_up", M * 2 * self.ip).view(M, 2 * self.ip)
            hops.gemm_f32(h, w, gu)
            hops.glu_f32(gu, act, M, self.ip, self.act)
        elif m.few_rows(M):
            ops.gemv(h, w, act[:M], swiglu=True, act=self.act)
        else:
            ops.gemm(h, w, out=act[:M], epi=ops.EPI_SWIGLU_BF16, act=self.act,
                     **m._gemm_shape(M, 2 * self.ip, m.dp, swiglu=True))
        m.into_acc(act[:M], self.w["w_down"])


RUNS = {"attention": AttentionRun, "retention": RetentionRun}


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
        moe = [L.mlp for L in cfg.layers if L.mlp is not None and L.mlp.kind == "moe"]
        if any(e.experts > hops.max_experts()[0] or e.top > hops.max_experts()[1] for e in moe):
            raise ConfigError(f"{cfg.name}: at most {hops.max_experts()[0]} experts, {hops.max_experts()[1]} of them chosen")
        att = [p for L in cfg.layers for p in L.mixer.parts if p.kind == "attention"]
        self.hkv = min((a.kv_heads for a in att), default=1)
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
        heads = max((a.heads for a in att), default=1)
        self.part_o = torch.zeros(max_seqs * heads * max_splits * 128, dtype=torch.float32, device=dev)
        self.part_ml = torch.zeros(max_seqs * heads * max_splits * 2, dtype=torch.float32, device=dev)
        widths = [self._in_width(L.mixer) for L in cfg.layers]
        self.proj = torch.zeros(max_tokens * max(widths), dtype=self.dtype, device=dev)
        self.proj_acc = (torch.zeros(max_tokens * max(widths), dtype=torch.float32, device=dev)
                         if self.dtype == torch.bfloat16 else None)
        self._buffers: dict = {}
        self._scratch: dict = {}
        self._moe: dict = {}
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
            n = HybridModel._in_width(mix.left) + mix.right.width_p
            return round_up(n, 256 if n >= 2048 else 64)      # wide projections in whole tiles of the widest kind
        w = (mix.heads * mix.dim + mix.kv_heads * (mix.dim + mix.vdim) if mix.kind == "attention"
             else 2 * mix.heads * (mix.dim + mix.vdim))
        return round_up(w, 64)

    @staticmethod
    def kv_block_bytes(cfg: ModelConfig, tp: int = 1, dtype: str = "bfloat16") -> int:
        """Device bytes of one 16-token KV block over all attention runs (0: no attention layers)."""
        total = 0
        for a in (p for i in cfg.layer_runs for p in cfg.layers[i].mixer.parts if p.kind == "attention"):
            big = max(a.dim, a.vdim)
            if dtype == "bfloat16" and big <= 128 and a.heads // a.kv_heads <= 16:
                total += a.kv_heads * 16 * 2 * (64 if big <= 64 else 128) * 2
            else:
                total += a.kv_heads * 16 * (a.dim + a.vdim) * (2 if dtype == "bfloat16" else 4)
        return total

    @staticmethod
    def state_bytes_per_seq(cfg: ModelConfig) -> int:
        return sum(4 * getattr(p, "state_elems", 0) for i in cfg.layer_runs for p in cfg.layers[i].mixer.parts)

    @staticmethod
    def step_bytes(cfg: ModelConfig, max_tokens: int, max_seqs: int) -> int:
        """Device bytes of a step's work space: streams, fp32 projections, rotated q / k, chunk states of
        retention, rows of the experts."""
        parts = [p for L in cfg.layers for p in L.mixer.parts]
        wide = max(p.width_p if p.kind == "ssd" else p.heads * (p.dim + p.vdim) for p in parts)
        chunk = max((p.state_elems for p in parts if p.kind == "retention"), default=0)
        n = max_tokens * 4 * (max(1, cfg.streams) * cfg.d_model + 6 * wide) + 8 * (max_tokens // 128 + max_seqs) * chunk
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

    def group_bn(self, m_tiles: int, n: int) -> int:
        """Tile width of an expert GEMM: narrow while the tiles would not fill the SMs."""
        for bn in (256, 128):
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
        up, down = torch.zeros(e.experts, fp, self.dp, **kw), torch.zeros(e.experts, self.dp, fp, **kw)
        router = torch.zeros(round_up(e.experts, 64), self.dp, **kw)
        d = self.cfg.d_model
        for i in range(e.experts):
            up[i, :e.ff, :d] = mat(f"{p}e{i}.up")
            down[i, :d, :e.ff] = mat(f"{p}e{i}.down")
        router[:e.experts, :d] = mat(p + "router")
        return {"up": up, "down": down, "router": router[:e.experts], "router_p": router}

    def _build_parallel(self, get) -> None:
        """Layers whose mixer and feed-forward run side by side."""
        mat = lambda name: get(name, False)
        vec = lambda name: get(name, True).contiguous()
        self.embed, self.head, self.out_norm = mat("embed").contiguous(), self._pad(mat("head")), vec("final.norm")
        self.k_cache, self.v_cache, self.states, self.sublayers = [], [], [], []
        for i, L in enumerate(self.cfg.layers):
            p, mx = f"l{i}.", L.mixer
            a = mx.left
            if a.rot not in self._rots:
                self._rots[a.rot] = hops.Rotary(a.rot, self.device)
            q = torch.cat([mat(f"{p}mix.left.{n}") for n in ("q", "k", "v")])
            ssd = self._ssd_weights(mx.right, p + "mix.right.", mat, vec)
            right = ssd.pop("in")
            w_in = q.new_zeros(self._in_width(mx), q.shape[1])
            w_in[:q.shape[0]] = q
            at = round_up(q.shape[0], 64)
            w_in[at:at + right.shape[0]] = right
            w = {"w_in": self._pad(w_in), "right": ssd,
                 "left": {"rot": self._rots[a.rot], "q_norm": None, "k_norm": None, "w_o": self._pad(mat(p + "mix.left.o"))}}
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
        self.head = self._pad(mat("head"))
        self.out_norm = vec("final.norm")
        one = torch.ones(1, dtype=torch.float32, device=self.device)
        rots = self._rots

        def hc(p: str, q: int) -> dict:
            if not cfg.streams:
                return {"in": one, "out": one, "mix": one}
            return {k: vec(f"{p}hc{q}.{k}") for k in ("in", "out", "mix")}

        layers = []
        for i, L in enumerate(cfg.layers):
            p, mx = f"l{i}.", L.mixer
            names = ("q", "k", "v") if mx.kind == "attention" else ("q", "k", "v", "g")
            if mx.rot not in rots:
                rots[mx.rot] = hops.Rotary(mx.rot, self.device)
            w = {"w_in": self._pad(torch.cat([mat(f"{p}mix.{n}") for n in names])), "w_o": self._pad(mat(p + "mix.o")),
                 "rot": rots[mx.rot], "q_norm": None, "k_norm": None}
            if mx.kind == "attention" and mx.qk_norm == "projection":
                w["q_norm"], w["k_norm"] = vec(p + "mix.q.norm"), vec(p + "mix.k.norm")
            if mx.kind == "retention":
                w["decay_pow"] = hops.decay_powers(mx.decay, self.device)
            subs = [(vec(p + "norm1"), hc(p, 1))]
            mw = None
            if L.mlp is not None:
                ip = round_up(L.mlp.ff, 64)
                g, u = mat(p + "mlp.gate"), mat(p + "mlp.up")
                if ip != L.mlp.ff:   # whole units of the interleaved layout; act(0) * 0 adds nothing
                    g, u = (torch.cat([t, t.new_zeros(ip - L.mlp.ff, t.shape[1])]) for t in (g, u))
                gu = interleave32(g, u) if self.dtype == torch.bfloat16 else torch.cat([g, u])
                mw = {"w_gu": self._pad(gu), "w_down": self._pad(mat(p + "mlp.down"))}
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
        from .layer_spec import initial_vector, layer_list_tensors

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
            return t.normal_(0.0, self.cfg.d_model ** -0.5 if name.endswith(".router") else std, generator=g)

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
        """acc = x @ w^T (fp32). The accumulator is zero here: stream_norm clears what it has read."""
        M, k = x.shape
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
