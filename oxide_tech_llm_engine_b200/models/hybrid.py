"""Device model of layer-list decoders: layers of different kinds (softmax attention over the paged KV
cache, retention with a per-sequence state), hyper-connected residual streams, looped layers, a
hashed bigram embedding. One GPU; bf16 kernels, or fp32 throughout (`dtype="float32"`).

Launch sequence of a step (every row is a token, decode rows first, then prompt chunks):

    stream_norm   embedding (+ bigram row) -> all streams, read-out and norm of the first sublayer
    per sublayer:
      attention:  gemm(q|k|v) -> heads (norm, rotation, paged K/V write) -> paged_decode / paged_prefill
      retention:  gemm(q|k|v|gate) -> retention_decode (one launch) / heads + chunked retention
                  -> gemm(O, fp32 accumulator)
      MLP:        gemm(gate|up, SwiGLU epilogue) -> gemm(down, fp32 accumulator)
      stream_norm stream update with the accumulator, read-out and norm of the next sublayer
    final stream_norm over the logit rows -> gemm(head)

KV blocks come from the scheduler's paged pool like any model's (one cache per attention run, so a
looped layer has one per pass); recurrent states live in slots that the scheduler hands to running
sequences. All sizes and constants come from the LayerSpec list; matrices are zero-padded to the
tile grid at load.
"""
from __future__ import annotations

import math
import os
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


class AttentionRun:
    """One run of an attention layer: weights shared by all passes, a KV cache of its own."""

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
        m, a, w, M = self.m, self.spec, self.w, s.m
        proj = m.project(h, w["w_in"], self.width)
        q = m.buffer(("q", a.heads * self.dp, a.dim), a.heads * self.dp)
        hops.heads(proj, M, h=a.heads, g=a.kv_heads, d=a.dim, e=a.vdim, rot=w["rot"], positions=s.positions, q_out=q,
                   q_hd=self.dp, q_norm=w["q_norm"], k_norm=w["k_norm"], eps=m.cfg.rms_eps, k_cache=self.k,
                   v_cache=self.v, slots=s.slot_mapping)
        out = m.buffer(("o", a.out_dim), round_up(a.out_dim, 64))
        nd = s.n_decode
        kw = dict(window=a.window, keep_first=a.keep_first if a.window else 0, scale=a.scale)
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
        att = [L.mixer for L in cfg.layers if L.mixer.kind == "attention"]
        self.hkv = min((a.kv_heads for a in att), default=1)
        self.x = torch.zeros(max_tokens, self.streams, d, dtype=torch.float32, device=dev)
        self.h = torch.zeros(max_tokens, self.dp, dtype=self.dtype, device=dev)
        self.acc = torch.zeros(max_tokens, self.dp, dtype=torch.float32, device=dev)
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
        self.k_cache: list = []
        self.v_cache: list = []
        self.states: list = []
        self.embed = self.bigram = self.head = self.out_norm = None
        self.sublayers: list = []
        self.layer_hook = None        # called with (layer run, summed streams [rows, width]) after every layer run

    # ------------------------------------------------------------------ sizes
    @staticmethod
    def _in_width(mix) -> int:
        w = (mix.heads * mix.dim + mix.kv_heads * (mix.dim + mix.vdim) if mix.kind == "attention"
             else 2 * mix.heads * (mix.dim + mix.vdim))
        return round_up(w, 64)

    @staticmethod
    def kv_block_bytes(cfg: ModelConfig, tp: int = 1, dtype: str = "bfloat16") -> int:
        """Device bytes of one 16-token KV block over all attention runs (0: no attention layers)."""
        total = 0
        for i in cfg.layer_runs:
            a = cfg.layers[i].mixer
            if a.kind != "attention":
                continue
            big = max(a.dim, a.vdim)
            if dtype == "bfloat16" and big <= 128 and a.heads // a.kv_heads <= 16:
                total += a.kv_heads * 16 * 2 * (64 if big <= 64 else 128) * 2
            else:
                total += a.kv_heads * 16 * (a.dim + a.vdim) * (2 if dtype == "bfloat16" else 4)
        return total

    @staticmethod
    def state_bytes_per_seq(cfg: ModelConfig) -> int:
        return sum(4 * cfg.layers[i].mixer.state_elems for i in cfg.layer_runs if cfg.layers[i].mixer.kind == "retention")

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

    def _build(self, get) -> None:
        """`get(name, fp32)` returns a named tensor on the device, in fp32 or in the model's dtype."""
        cfg = self.cfg
        mat = lambda name: get(name, False)
        vec = lambda name: get(name, True).contiguous()
        self.embed = mat("embed").contiguous()
        self.bigram = mat("bigram").contiguous() if cfg.bigram is not None else None
        self.head = self._pad(mat("head"))
        self.out_norm = vec("final.norm")
        one = torch.ones(1, dtype=torch.float32, device=self.device)
        rots: dict = {}

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
        from .layer_spec import layer_list_tensors

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
                return torch.full(shape, 1.0 if name.endswith((".q.norm", ".k.norm")) else 0.0, device=self.device)
            t = torch.empty(*shape, dtype=self.dtype, device=self.device)
            return t.normal_(0.0, std, generator=g)

        self._build(get)

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

    def into_acc(self, x: torch.Tensor, w: torch.Tensor) -> None:
        """acc = x @ w^T (fp32). The accumulator is zero here: stream_norm clears what it has read."""
        M, k = x.shape
        acc = self.acc[:M]
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
        cfg, M = self.cfg, s.m
        h = self.h[:M]
        subs = self.sublayers
        bg = cfg.bigram
        hops.stream_norm(self.x, M, tokens=s.token_ids, prev=s.prev_ids if bg is not None else None, embed=self.embed,
                         bigram=self.bigram, mul_prev=bg.mul_prev if bg else 0, mul_cur=bg.mul_cur if bg else 0,
                         in_w=subs[0].hc["in"], norm_w=subs[0].norm, eps=cfg.rms_eps, h=h,
                         clear=self._proj_splits(M, subs[0]))
        n_log = max(s.n_logits, 1)
        lm_h, logits = self.lm_h, self.logits_buf
        if n_log > self.max_logits:
            lm_h = torch.zeros(n_log, self.dp, dtype=self.dtype, device=self.device)
            logits = torch.empty(n_log, self.vp, dtype=torch.float32, device=self.device)
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
        lm_h, logits = lm_h[:n_log], logits[:n_log]
        if self.dtype == torch.float32:
            hops.gemm_f32(lm_h, self.head, logits)
        elif self.few_rows(n_log):
            ops.gemv(lm_h, self.head, logits)
        else:
            ops.gemm(lm_h, self.head, out=logits, epi=ops.EPI_STORE_F32, **self._gemm_shape(n_log, self.vp, self.dp, store=True))
        return logits[:, :cfg.vocab_size]

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
        self.acc.zero_()
        if self.proj_acc is not None:
            self.proj_acc.zero_()
        ops.gemm_workspace(self.device)[1].zero_()
        torch.cuda.synchronize(self.device)

    def close(self) -> None:
        self._buffers.clear()
        self._scratch.clear()
