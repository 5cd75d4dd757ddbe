"""Descriptions of decoders that are given as a list of layers rather than as one repeated block.

A `LayerSpec` names a token mixer (attention, retention, several side by side, ...) and a feed-forward
(dense, mixture of experts), each with its own sizes and constants, so layers of one model may differ in kind, in head layout and in window. The
specs are plain data: `models.hybrid` builds the device layers from them, `models.cpu_hybrid` the
CPU ones, `models.weights` the tensor list. A further design adds its mixer here as one more
dataclass with the constants as fields, and registers its configuration reader in
`models.registry`.
"""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Any, Optional, Union

from ..errors import ConfigError


@dataclass(frozen=True)
class YarnSpec:
    """YaRN scaling of rotation frequencies: pairs that turn fewer than `slow` times within `original`
    positions are slowed down by `factor`, pairs that turn more than `fast` times stay, a ramp over the
    pair index lies between; sin and cos carry the factor 0.1 ln(factor) + 1."""
    factor: float
    original: float
    fast: float
    slow: float

    def frequencies(self, dims: int, base: float, freqs: list) -> tuple[list, float]:
        def pair_that_turns(n: float) -> float:
            return dims * math.log(self.original / (2.0 * math.pi * n)) / (2.0 * math.log(base))

        lo = max(math.floor(pair_that_turns(self.fast)), 0)
        hi = min(math.ceil(pair_that_turns(self.slow)), dims - 1)
        out = []
        for i, f in enumerate(freqs):
            r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
            out.append(f / self.factor * r + f * (1.0 - r))
        return out, 0.1 * math.log(self.factor) + 1.0


@dataclass(frozen=True)
class RotarySpec:
    """Rotation of the first `dims` dimensions of every head: pairs (2i, 2i+1) when `interleaved`,
    else (i, i + dims/2), by the angle position * base^(-2i/dims), its frequency scaled by `scaling`."""
    dims: int
    base: float
    interleaved: bool = False
    scaling: Optional[YarnSpec] = None

    def frequencies(self) -> tuple[list, float]:
        """Frequency of every pair, and the factor on sin and cos."""
        f = [float(self.base) ** (-2.0 * i / self.dims) for i in range(self.dims // 2)]
        return (f, 1.0) if self.scaling is None else self.scaling.frequencies(self.dims, float(self.base), f)


@dataclass(frozen=True)
class AttentionSpec:
    """Softmax attention with grouped key/value heads. `window` 0: every earlier position is visible;
    else the last `window` positions and the first `keep_first` ones of the sequence (which keep their
    true positions). `chunk` (instead of a window): only positions of the same chunk, counted from position
    0. `sink`: score of one more term of the softmax denominator that has no value; `sinks`: a learned one per head. `qk_norm` "projection": RMS norm over all heads of q (of k) at once, before the
    rotation. `bias`: q, k and v have biases. `temp_coef`: q is multiplied by 1 + temp_coef ln(floor((p + 1) / temp_every) + 1)
    at position p. `diff`: differential attention, every head has two maps over the same values (q and k hold
    [map 1, map 2] head by head); with lambda = exp(lq1 . lk1) - exp(lq2 . lk2) + diff the result is a1 - lambda a2 divided
    by its root mean square, times 1 - diff."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot: Optional[RotarySpec] = None
    window: int = 0
    keep_first: int = 0
    qk_norm: str = "none"      # none | projection
    chunk: int = 0
    sink: Optional[float] = None
    bias: bool = False
    temp_coef: float = 0.0
    temp_every: float = 1.0
    diff: Optional[float] = None
    sinks: bool = False

    kind = "attention"

    @property
    def parts(self) -> tuple:
        return (self,)

    @property
    def maps(self) -> int:
        return 1 if self.diff is None else 2

    @property
    def out_dim(self) -> int:
        return self.heads * self.vdim

    @property
    def in_width(self) -> int:
        return self.maps * self.heads * self.dim + self.cache_values

    @property
    def cache_values(self) -> int:
        """Values that a token keeps in the cache."""
        return self.kv_heads * (self.maps * self.dim + self.vdim)

    def tensors(self, d: int) -> list[tuple[str, tuple[int, ...]]]:
        rows = {"q": self.heads * self.maps * self.dim, "k": self.kv_heads * self.maps * self.dim, "v": self.kv_heads * self.vdim}
        out = []
        for n, r in rows.items():
            out += [(n, (r, d))] + ([(n + ".b", (r,))] if self.bias else [])
        if self.diff is not None:
            out += [(n, (self.dim,)) for n in ("lq1", "lk1", "lq2", "lk2")]
        if self.sinks:
            out.append(("sink", (self.heads,)))
        out.append(("o", (d, self.out_dim)))
        if self.qk_norm == "projection":
            out += [("q.norm", (self.heads * self.dim,)), ("k.norm", (self.kv_heads * self.dim,))]
        return out


@dataclass(frozen=True)
class TalkingSpec:
    """Attention whose heads mix their scores (talking heads) over one projection that is key and value: k = W_k h is the value as
    it is and, by its RMS norm over all heads, the key; q is normed the same way. A head's score is softcap tanh(q . k scale / softcap)
    (`softcap` 0: as it is) minus r1_h ln(1 + r2_h distance); head h goes on with sum_g talk[h, g] score_g, and a softmax over the
    last `window` positions (0: all). The result is multiplied by sigmoid(W_g h). No rotation."""
    heads: int
    kv_heads: int
    dim: int
    scale: float
    softcap: float = 0.0
    window: int = 0

    kind = "talking_attention"

    @property
    def parts(self) -> tuple:
        return (self,)

    @property
    def vdim(self) -> int:
        return self.dim

    @property
    def out_dim(self) -> int:
        return self.heads * self.dim

    @property
    def gate_col(self) -> int:
        """Column of the gate in the projection, behind q and k."""
        return _pad16((self.heads + self.kv_heads) * self.dim)

    @property
    def in_width(self) -> int:
        return self.gate_col + self.out_dim

    @property
    def cache_values(self) -> int:
        """Values that a token keeps: its keys before the norm, which are its values (and one fp32 number, their norm)."""
        return self.kv_heads * self.dim

    def tensors(self, d: int) -> list[tuple[str, tuple[int, ...]]]:
        hd, gd, h = self.out_dim, self.cache_values, self.heads
        return [("q", (hd, d)), ("k", (gd, d)), ("q.norm", (hd,)), ("k.norm", (gd,)), ("r1", (h,)), ("r2", (h,)), ("talk", (h, h)),
                ("g", (hd, d)), ("o", (d, hd))]


@dataclass(frozen=True)
class LatentSpec:
    """Latent attention. Queries: W_uq of the normed W_dq h, per head `dim` values and, rotated, rot.dims more. A token
    keeps the normed first `kv_rank` values of W_dkv h (the latent) and the rotated rest, one key part for all heads;
    keys and values of a head are W_uk and W_uv of the latent. `kv_from`: the layer has no W_dkv and reads what that
    layer keeps."""
    heads: int
    dim: int
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    rot: Optional[RotarySpec] = None
    kv_from: Optional[int] = None

    kind = "latent_attention"

    @property
    def parts(self) -> tuple:
        return (self,)

    @property
    def rot_dim(self) -> int:
        return self.rot.dims if self.rot is not None else 0

    @property
    def out_dim(self) -> int:
        return self.heads * self.vdim

    @property
    def kv_col(self) -> int:
        """Column of the latent in the projection, behind the query latent."""
        return (self.q_rank + 7) // 8 * 8

    @property
    def in_width(self) -> int:
        return self.kv_col + (self.kv_rank + self.rot_dim if self.kv_from is None else 0)

    @property
    def cache_row(self) -> int:
        return _pad16(self.kv_rank + self.rot_dim)

    @property
    def cache_values(self) -> int:
        return self.kv_rank + self.rot_dim if self.kv_from is None else 0

    def tensors(self, d: int) -> list[tuple[str, tuple[int, ...]]]:
        h, r = self.heads, self.kv_rank
        out = [("dq", (self.q_rank, d)), ("dq.norm", (self.q_rank,)), ("uq", (h * (self.dim + self.rot_dim), self.q_rank))]
        if self.kv_from is None:
            out += [("dkv", (r + self.rot_dim, d)), ("dkv.norm", (r,))]
        return out + [("uk", (h * self.dim, r)), ("uv", (h * self.vdim, r)), ("o", (d, self.out_dim))]


@dataclass(frozen=True)
class MemorySpec:
    """Matrix memory with exponential gates under a running maximum (mLSTM of xLSTM): see memory.cu for the recurrence. Gate
    pre-activations are capped by cap tanh(z / cap); every head's output is divided by its root mean square, times `norm`,
    times sigmoid(W_g h)."""
    heads: int
    dim: int
    vdim: int
    gate_cap: float

    kind = "mlstm"

    @property
    def parts(self) -> tuple:
        return (self,)

    @property
    def out_dim(self) -> int:
        return self.heads * self.vdim

    @property
    def in_width(self) -> int:
        return 2 * self.heads * (self.dim + self.vdim)

    @property
    def state_elems(self) -> int:
        """fp32 values of one sequence's state: the memory, its normaliser and the running maximum."""
        return self.heads * (self.dim * self.vdim + self.dim + 1)

    def tensors(self, d: int) -> list[tuple[str, tuple[int, ...]]]:
        h, hd, hv = self.heads, self.heads * self.dim, self.heads * self.vdim
        return [("q", (hd, d)), ("k", (hd, d)), ("v", (hv, d)), ("g", (hv, d)), ("o", (d, hv)), ("norm", (hv,)), ("i", (h, d)),
                ("i.b", (h,)), ("f", (h, d)), ("f.b", (h,))]


@dataclass(frozen=True)
class RetentionSpec:
    """Linear attention with a fixed decay per head: S <- decay S + k v^T, o = S^T q, the keys scaled by
    dim^(-1/2); every head's output is normalised by its root mean square and gated by silu(W_g h)."""
    heads: int
    dim: int
    vdim: int
    decay: tuple
    rot: Optional[RotarySpec] = None

    kind = "retention"

    @property
    def parts(self) -> tuple:
        return (self,)

    @property
    def out_dim(self) -> int:
        return self.heads * self.vdim

    @property
    def in_width(self) -> int:
        return 2 * self.heads * (self.dim + self.vdim)

    @property
    def state_elems(self) -> int:
        """fp32 values of one sequence's state."""
        return self.heads * self.dim * self.vdim

    def tensors(self, d: int) -> list[tuple[str, tuple[int, ...]]]:
        hd, hv = self.heads * self.dim, self.heads * self.vdim
        return [("q", (hd, d)), ("k", (hd, d)), ("v", (hv, d)), ("g", (hv, d)), ("o", (d, hv))]


def _pad16(n: int) -> int:
    return (n + 15) // 16 * 16


@dataclass(frozen=True)
class SsdSpec:
    """State-space layer with one decay per head and step (Mamba-2). The input projection gives z | x | B | C |
    step sizes; x, B and C pass a causal convolution of `taps` taps and silu; with dt = softplus(dt + dt_bias),
    S <- exp(-exp(A_log) dt) S + dt B x^T, y = S^T C + D x (S: state x vdim per head, head h uses B and C of group
    h / (heads / groups)); y * silu(z) is normalised in `norm_groups` equal parts and projected."""
    heads: int
    vdim: int
    state: int
    groups: int
    taps: int
    norm_groups: int

    kind = "ssd"

    @property
    def parts(self) -> tuple:
        return (self,)

    @property
    def inner(self) -> int:
        return self.heads * self.vdim

    @property
    def out_dim(self) -> int:
        return self.inner

    # device layout: heads and states padded to whole 16-value pieces with zero channels
    @property
    def vdim_p(self) -> int:
        return _pad16(self.vdim)

    @property
    def state_p(self) -> int:
        return _pad16(self.state)

    @property
    def channels_p(self) -> int:
        """Channels of the convolution."""
        return self.heads * self.vdim_p + 2 * self.groups * self.state_p

    @property
    def width_p(self) -> int:
        """Columns of the projection."""
        return self.heads * self.vdim_p + self.channels_p + self.heads

    @property
    def state_elems(self) -> int:
        """fp32 values of one sequence's state: the recurrence's and the convolution's."""
        return self.heads * self.state_p * self.vdim_p + self.taps * self.channels_p

    def tensors(self, d: int) -> list[tuple[str, tuple[int, ...]]]:
        gn, h = self.groups * self.state, self.heads
        return [("in", (2 * self.inner + 2 * gn + h, d)), ("conv", (self.inner + 2 * gn, self.taps)),
                ("conv.b", (self.inner + 2 * gn,)), ("dt_bias", (h,)), ("A_log", (h,)), ("D", (h,)), ("norm", (self.inner,)),
                ("o", (d, self.inner))]


@dataclass(frozen=True)
class GruSpec:
    """Gated recurrence whose gates read only the current token (minGRU): z = sigmoid(W_z h + b_z), u = W_x h + b_x,
    S <- (1 - z) S + z c(u) element by element with c(u) = u + 1/2 from 0 on and sigmoid(u) below, output S silu(W_g h)."""
    width: int

    kind = "min_gru"

    @property
    def parts(self) -> tuple:
        return (self,)

    @property
    def out_dim(self) -> int:
        return self.width

    @property
    def width_p(self) -> int:
        """Columns of each of the three projections (zero channels as padding)."""
        return _pad16(self.width)

    @property
    def in_width(self) -> int:
        return 3 * self.width_p

    @property
    def state_elems(self) -> int:
        return self.width_p

    def tensors(self, d: int) -> list[tuple[str, tuple[int, ...]]]:
        n = self.width
        return [("z", (n, d)), ("z.b", (n,)), ("x", (n, d)), ("x.b", (n,)), ("g", (n, d)), ("o", (d, n))]


@dataclass(frozen=True)
class ParallelSpec:
    """Two mixers side by side on the same input. The result is half the sum of the two outputs, each by its own RMS norm
    over the model width, or with `gains` the outputs as they are, weighted by these two numbers."""
    left: AttentionSpec
    right: Union[SsdSpec, GruSpec]
    gains: Optional[tuple] = None

    kind = "parallel"

    @property
    def parts(self) -> tuple:
        return (*self.left.parts, *self.right.parts)

    def tensors(self, d: int) -> list[tuple[str, tuple[int, ...]]]:
        out = []
        for side in ("left", "right"):
            out += [(f"{side}.{n}", s) for n, s in getattr(self, side).tensors(d)]
        return out if self.gains is not None else out + [("left.out", (d,)), ("right.out", (d,))]


@dataclass(frozen=True)
class DenseMlpSpec:
    """W_down (act(W_gate h) * (W_up h)), or with `act` "relu2" W_down relu(W_up h)^2."""
    ff: int
    act: str = "silu"          # silu | gelu_tanh | relu2

    kind = "dense"

    @property
    def glu(self) -> bool:
        return self.act != "relu2"

    def tensors(self, d: int) -> list[tuple[str, tuple[int, ...]]]:
        if not self.glu:
            return [("up", (self.ff, d)), ("down", (d, self.ff))]
        return [("gate", (self.ff, d)), ("up", (self.ff, d)), ("down", (d, self.ff))]


@dataclass(frozen=True)
class MoeSpec:
    """Mixture of `experts` feed-forwards W_down act(W_up h), or with `act` "silu_glu" W_down (silu(W_gate h) * (W_up h)).
    A token uses the `top` ones with the largest scores. `scores` "softmax": over all experts, the weights are the chosen
    scores divided by their sum; "sigmoid": the weights are the chosen scores. `groups` > 0: the experts form that many
    equal groups of neighbours, and only those of the `keep` groups with the largest sum of two largest scores can be
    chosen."""
    ff: int
    experts: int
    top: int
    act: str = "relu2"         # relu2 (square of relu) | silu_glu
    scores: str = "softmax"    # softmax | sigmoid
    groups: int = 0
    keep: int = 0

    kind = "moe"

    @property
    def glu(self) -> bool:
        return self.act == "silu_glu"

    def tensors(self, d: int) -> list[tuple[str, tuple[int, ...]]]:
        out = []
        for e in range(self.experts):
            out += [(f"e{e}.gate", (self.ff, d))] if self.glu else []
            out += [(f"e{e}.up", (self.ff, d)), (f"e{e}.down", (d, self.ff))]
        return out + [("router", (self.experts, d))]


@dataclass(frozen=True)
class LayerSpec:
    """`parallel`: mixer and feed-forward read the same residual stream, each through its own norm, and both are
    added to it; else the feed-forward follows the mixer. `post_norm`: a sublayer's result passes a norm of its own
    and an element-wise scale before it is added."""
    mixer: Union[AttentionSpec, RetentionSpec, SsdSpec, ParallelSpec, LatentSpec, MemorySpec, TalkingSpec]
    mlp: Union[DenseMlpSpec, MoeSpec, None]
    parallel: bool = False
    post_norm: bool = False

    @property
    def sublayers(self) -> int:
        return 1 if self.mlp is None else 2


@dataclass(frozen=True)
class BigramSpec:
    """Second embedding table addressed by a hash of the previous and the current token:
    (previous * mul_prev + current * mul_cur) mod buckets; row `buckets` for a first token."""
    buckets: int
    mul_prev: int
    mul_cur: int


def layer_runs(n_layers: int, loop: Optional[tuple]) -> list[int]:
    """Layer index of every layer run in order. `loop` (start, stop, times): layers start .. stop-1 run
    `times` times in a row with the same weights; every pass keeps its own cache or state."""
    if loop is None:
        return list(range(n_layers))
    a, b, t = loop
    if not (0 <= a < b <= n_layers and t >= 1):
        raise ConfigError(f"loop {loop} does not fit {n_layers} layers")
    return list(range(a)) + list(range(a, b)) * t + list(range(b, n_layers))


def rotary_from_json(c: Optional[dict], interleaved: bool, dim: int) -> Optional[RotarySpec]:
    if not c:
        return None
    dims = int(c["dims"])
    if dims % 2 or dims > dim or dims < 0:
        raise ConfigError(f"rotary dims {dims} do not fit a head of {dim}")
    sc = c.get("scaling")
    yarn = YarnSpec(*(float(sc[k]) for k in ("factor", "original", "fast", "slow"))) if sc else None
    return RotarySpec(dims, float(c["base"]), interleaved, yarn) if dims else None


def mlp_from_json(c: Optional[dict]) -> Optional[DenseMlpSpec]:
    if c is None:
        return None
    if c.get("kind") != "dense":
        raise ConfigError(f"feed-forward kind {c.get('kind')!r} is not part of this engine")
    return DenseMlpSpec(int(c["ff"]))


def attention_from_json(c: dict) -> AttentionSpec:
    mask = c.get("mask") or {}
    a = AttentionSpec(heads=int(c["heads"]), kv_heads=int(c["kv_heads"]), dim=int(c["dim"]), vdim=int(c["vdim"]),
                      scale=float(c["scale"]), rot=rotary_from_json(c.get("rot"), True, int(c["dim"])),
                      window=int(mask.get("size", 0)), keep_first=int(mask.get("keep_first", 0)), qk_norm="projection")
    if a.heads % a.kv_heads:
        raise ConfigError(f"{a.heads} query heads do not divide over {a.kv_heads} key/value heads")
    return a


def retention_from_json(c: dict) -> RetentionSpec:
    r = RetentionSpec(heads=int(c["heads"]), dim=int(c["dim"]), vdim=int(c["vdim"]),
                      decay=tuple(float(x) for x in c["decay"]), rot=rotary_from_json(c.get("rot"), False, int(c["dim"])))
    if len(r.decay) != r.heads:
        raise ConfigError(f"{len(r.decay)} decays for {r.heads} retention heads")
    return r


MIXERS_FROM_JSON = {"attention": attention_from_json, "retention": retention_from_json}


def layer_from_json(c: dict) -> LayerSpec:
    if c["type"] not in MIXERS_FROM_JSON:
        raise ConfigError(f"layer type {c['type']!r} is not part of this engine")
    return LayerSpec(MIXERS_FROM_JSON[c["type"]](c["mixer"]), mlp_from_json(c.get("mlp")))


def kipolix_config(c: dict[str, Any], shapes: Optional[dict] = None):
    """ModelConfig of a Kipolix checkpoint from its config.json. The configuration has no tokenizer,
    so there is no end-of-text id (-1 never matches a token)."""
    from .config import ModelConfig

    layers = tuple(layer_from_json(x) for x in c["layers"])
    lp = c.get("loop")
    loop = (int(lp["start"]), int(lp["stop"]), int(lp["times"])) if lp else None
    layer_runs(len(layers), loop)
    bg = (c.get("embedding") or {}).get("bigram")
    bigram = BigramSpec(int(bg["buckets"]), int(bg["mul_prev"]), int(bg["mul_cur"])) if bg else None
    att = next((x.mixer for x in layers if x.mixer.kind == "attention"), None)
    mlp = next((x.mlp for x in layers if x.mlp is not None), None)
    any_m = att or layers[0].mixer
    return ModelConfig(name="kipolix", arch="kipolix", n_layers=len(layers), d_model=int(c["width"]),
                       n_heads=any_m.heads, n_kv_heads=getattr(any_m, "kv_heads", any_m.heads), head_dim=any_m.dim,
                       ffn_dim=mlp.ff if mlp else 0, vocab_size=int(c["vocab"]), max_ctx=1 << 20,
                       rms_eps=float(c["norm"]["eps"]), norm_weight_offset=1.0, bos_id=-1, eos_id=-1,
                       layers=layers, loop=loop, streams=int(c.get("streams", 0)), bigram=bigram)


def kipolix_json(cfg) -> dict[str, Any]:
    """config.json of a Kipolix ModelConfig (inverse of kipolix_config)."""
    layers = []
    for L in cfg.layers:
        m = L.mixer
        c: dict[str, Any] = {"heads": m.heads, "dim": m.dim, "vdim": m.vdim}
        if m.rot is not None:
            c["rot"] = {"dims": m.rot.dims, "base": m.rot.base}
        if m.kind == "attention":
            c.update(kv_heads=m.kv_heads, scale=m.scale, mask={"size": m.window, "keep_first": m.keep_first})
        else:
            c["decay"] = list(m.decay)
        layers.append({"type": m.kind, "mixer": c, "mlp": None if L.mlp is None else {"kind": "dense", "ff": L.mlp.ff}})
    out = {"architecture": "Kipolix", "vocab": cfg.vocab_size, "width": cfg.d_model, "norm": {"eps": cfg.rms_eps},
           "embedding": {}, "layers": layers}
    if cfg.streams:
        out["streams"] = cfg.streams
    if cfg.bigram is not None:
        b = cfg.bigram
        out["embedding"]["bigram"] = {"buckets": b.buckets, "mul_prev": b.mul_prev, "mul_cur": b.mul_cur}
    if cfg.loop is not None:
        out["loop"] = dict(zip(("start", "stop", "times"), cfg.loop))
    return out


def chunked_attention_from_json(c: dict) -> AttentionSpec:
    """Left mixer of a Povatar layer: rotation of the half layout, chunks, and a sink of score 0."""
    a = AttentionSpec(heads=int(c["heads"]), kv_heads=int(c["kv_heads"]), dim=int(c["dim"]), vdim=int(c["vdim"]),
                      scale=float(c["scale"]), rot=rotary_from_json(c.get("rot"), False, int(c["dim"])),
                      chunk=int((c.get("mask") or {}).get("size", 0)), sink=0.0)
    if a.heads % a.kv_heads:
        raise ConfigError(f"{a.heads} query heads do not divide over {a.kv_heads} key/value heads")
    return a


def ssd_from_json(c: dict) -> SsdSpec:
    s = SsdSpec(heads=int(c["heads"]), vdim=int(c["vdim"]), state=int(c["state"]), groups=int(c["groups"]), taps=int(c["conv"]),
                norm_groups=int(c["norm_groups"]))
    if s.heads % s.groups:
        raise ConfigError(f"{s.heads} heads do not divide over {s.groups} groups")
    if s.inner % s.norm_groups:
        raise ConfigError(f"{s.inner} values do not divide into {s.norm_groups} norm groups")
    return s


def moe_from_json(c: Optional[dict]) -> Optional[MoeSpec]:
    if c is None:
        return None
    if c.get("kind") != "moe":
        raise ConfigError(f"feed-forward kind {c.get('kind')!r} is not part of this design")
    m = MoeSpec(int(c["expert"]["ff"]), int(c["router"]["experts"]), int(c["router"]["top"]))
    if not 1 <= m.top <= m.experts:
        raise ConfigError(f"{m.top} of {m.experts} experts")
    return m


def povatar_layer(c: dict) -> LayerSpec:
    if c["type"] != "parallel":
        raise ConfigError(f"layer type {c['type']!r} is not part of this design")
    mx = c["mixer"]
    return LayerSpec(ParallelSpec(chunked_attention_from_json(mx["left"]), ssd_from_json(mx["right"])), moe_from_json(c.get("mlp")),
                     parallel=True)


def povatar_model(layers: tuple, *, width: int, vocab: int, eps: float, emb_scale: float, name: str = "povatar"):
    """ModelConfig of Povatar layers. No tokenizer comes with the design, so there is no end-of-text id."""
    from .config import ModelConfig

    left = layers[0].mixer.left
    return ModelConfig(name=name, arch="povatar", n_layers=len(layers), d_model=width, n_heads=left.heads,
                       n_kv_heads=left.kv_heads, head_dim=left.dim, ffn_dim=max((L.mlp.ff for L in layers if L.mlp), default=0),
                       vocab_size=vocab, max_ctx=1 << 20, rms_eps=eps, emb_scale=emb_scale, bos_id=-1, eos_id=-1, layers=layers)


def povatar_config(c: dict[str, Any]):
    """ModelConfig of a Povatar checkpoint from its config.json."""
    return povatar_model(tuple(povatar_layer(x) for x in c["layers"]), width=int(c["width"]), vocab=int(c["vocab"]),
                         eps=float(c["norm"]["eps"]), emb_scale=float((c.get("embedding") or {}).get("scale", 1.0)))


def povatar_json(cfg) -> dict[str, Any]:
    """config.json of a Povatar ModelConfig (inverse of povatar_config)."""
    layers = []
    for L in cfg.layers:
        a, r = L.mixer.left, L.mixer.right
        left: dict[str, Any] = {"heads": a.heads, "kv_heads": a.kv_heads, "dim": a.dim, "vdim": a.vdim, "scale": a.scale}
        if a.chunk:
            left["mask"] = {"size": a.chunk}
        if a.rot is not None:
            left["rot"] = {"base": a.rot.base, "dims": a.rot.dims}
            if a.rot.scaling is not None:
                y = a.rot.scaling
                left["rot"]["scaling"] = {"factor": y.factor, "original": y.original, "fast": y.fast, "slow": y.slow}
        right = {"heads": r.heads, "vdim": r.vdim, "state": r.state, "groups": r.groups, "conv": r.taps, "norm_groups": r.norm_groups}
        mlp = None if L.mlp is None else {"kind": "moe", "expert": {"ff": L.mlp.ff},
                                          "router": {"experts": L.mlp.experts, "top": L.mlp.top}}
        layers.append({"type": "parallel", "mixer": {"left": left, "right": right}, "mlp": mlp})
    return {"architecture": "Povatar", "vocab": cfg.vocab_size, "width": cfg.d_model, "norm": {"eps": cfg.rms_eps},
            "embedding": {"scale": cfg.emb_scale}, "layers": layers}


def gated_moe_from_json(c: dict) -> MoeSpec:
    """Gated experts behind sigmoid scores, in groups where the router has them."""
    r = c["router"]
    g = r.get("groups") or {}
    m = MoeSpec(int(c["expert"]["ff"]), int(r["experts"]), int(r["top"]), act="silu_glu", scores="sigmoid",
                groups=int(g.get("count", 0)), keep=int(g.get("keep", 0)))
    if m.groups and (m.experts % m.groups or not 1 <= m.keep <= m.groups):
        raise ConfigError(f"{m.keep} of {m.groups} groups of {m.experts} experts")
    if not 1 <= m.top <= (m.experts // m.groups * m.keep if m.groups else m.experts):
        raise ConfigError(f"{m.top} of {m.experts} experts")
    return m


def zagolix_mixer(c: dict, kind: str):
    n = lambda k: int(c[k])
    if kind == "attention":
        t = c.get("q_temp") or {}
        a = AttentionSpec(n("heads"), n("kv_heads"), n("dim"), n("vdim"), float(c["scale"]), bias=True, diff=float(c["diff"]),
                          temp_coef=float(t.get("coef", 0.0)), temp_every=float(t.get("every", 1.0)))
        if a.heads % a.kv_heads:
            raise ConfigError(f"{a.heads} query heads do not divide over {a.kv_heads} key/value heads")
        return a
    if kind == "latent_attention":
        rot = rotary_from_json(c.get("rot"), True, n("rot_dim"))
        if (rot.dims if rot else 0) != n("rot_dim"):
            raise ConfigError(f"{c.get('rot')} does not rotate all of {n('rot_dim')} dimensions")
        src = c.get("kv_from")
        return LatentSpec(n("heads"), n("dim"), n("vdim"), n("q_rank"), n("kv_rank"), float(c["scale"]), rot,
                          None if src is None else int(src))
    if kind == "mlstm":
        return MemorySpec(n("heads"), n("dim"), n("vdim"), float(c["gate_cap"]))
    raise ConfigError(f"layer type {kind!r} is not part of this design")


def zagolix_mlp(c: Optional[dict]):
    if c is None:
        return None
    if c.get("kind") == "dense":
        return DenseMlpSpec(int(c["ff"]), act="gelu_tanh")
    if c.get("kind") == "moe":
        return gated_moe_from_json(c)
    raise ConfigError(f"feed-forward kind {c.get('kind')!r} is not part of this design")


def zagolix_model(layers: tuple, *, width: int, vocab: int, eps: float, emb_scale: float, name: str = "zagolix"):
    """ModelConfig of Zagolix layers. No tokenizer comes with the design, so there is no end-of-text id."""
    from .config import ModelConfig

    for i, L in enumerate(layers):
        m, j = L.mixer, getattr(L.mixer, "kv_from", None)
        if j is None:
            continue
        o = layers[j].mixer if 0 <= j < i else None
        if not isinstance(o, LatentSpec) or o.kv_from is not None or (o.kv_rank, o.rot) != (m.kv_rank, m.rot):
            raise ConfigError(f"layer {i} cannot read what layer {j} keeps")
    any_m = layers[0].mixer
    return ModelConfig(name=name, arch="zagolix", n_layers=len(layers), d_model=width, n_heads=any_m.heads,
                       n_kv_heads=getattr(any_m, "kv_heads", any_m.heads), head_dim=any_m.dim,
                       ffn_dim=max((L.mlp.ff for L in layers if L.mlp), default=0), vocab_size=vocab, max_ctx=1 << 20, rms_eps=eps,
                       emb_scale=emb_scale, tie_embeddings=True, bos_id=-1, eos_id=-1, layers=layers)


def zagolix_config(c: dict[str, Any]):
    """ModelConfig of a Zagolix checkpoint from its config.json."""
    layers = tuple(LayerSpec(zagolix_mixer(x["mixer"], x["type"]), zagolix_mlp(x.get("mlp")), post_norm=True) for x in c["layers"])
    return zagolix_model(layers, width=int(c["width"]), vocab=int(c["vocab"]), eps=float(c["norm"]["eps"]),
                         emb_scale=float((c.get("embedding") or {}).get("scale", 1.0)))


def zagolix_json(cfg) -> dict[str, Any]:
    """config.json of a Zagolix ModelConfig (inverse of zagolix_config)."""
    layers = []
    for L in cfg.layers:
        m, f = L.mixer, L.mlp
        c: dict[str, Any] = {"heads": m.heads, "dim": m.dim, "vdim": m.vdim}
        if m.kind == "attention":
            c.update(kv_heads=m.kv_heads, scale=m.scale, diff=m.diff)
            if m.temp_coef:
                c["q_temp"] = {"coef": m.temp_coef, "every": m.temp_every}
        elif m.kind == "latent_attention":
            c.update(q_rank=m.q_rank, kv_rank=m.kv_rank, scale=m.scale, rot_dim=m.rot_dim)
            if m.rot is not None:
                c["rot"] = {"base": m.rot.base, "dims": m.rot.dims}
            if m.kv_from is not None:
                c["kv_from"] = m.kv_from
        else:
            c["gate_cap"] = m.gate_cap
        mlp = None
        if f is not None and f.kind == "dense":
            mlp = {"kind": "dense", "ff": f.ff}
        elif f is not None:
            mlp = {"kind": "moe", "expert": {"ff": f.ff}, "router": {"experts": f.experts, "top": f.top}}
            if f.groups:
                mlp["router"]["groups"] = {"count": f.groups, "keep": f.keep}
        layers.append({"type": m.kind, "mixer": c, "mlp": mlp})
    return {"architecture": "Zagolix", "vocab": cfg.vocab_size, "width": cfg.d_model, "norm": {"eps": cfg.rms_eps},
            "embedding": {"scale": cfg.emb_scale}, "layers": layers}


def vokepel_attention(c: dict) -> AttentionSpec:
    """Left mixer of a Vokepel pair: rotation of neighbouring pairs, a window, a learned sink per head."""
    a = AttentionSpec(heads=int(c["heads"]), kv_heads=int(c["kv_heads"]), dim=int(c["dim"]), vdim=int(c["vdim"]),
                      scale=float(c["scale"]), rot=rotary_from_json(c.get("rot"), True, int(c["dim"])),
                      window=int((c.get("mask") or {}).get("size", 0)), sinks=True)
    if a.heads % a.kv_heads:
        raise ConfigError(f"{a.heads} query heads do not divide over {a.kv_heads} key/value heads")
    return a


def vokepel_mixer(c: dict, kind: str):
    if kind == "attention":
        t = TalkingSpec(int(c["heads"]), int(c["kv_heads"]), int(c["dim"]), float(c["scale"]), float(c.get("softcap") or 0.0),
                        int((c.get("mask") or {}).get("size", 0)))
        if t.heads % t.kv_heads:
            raise ConfigError(f"{t.heads} query heads do not divide over {t.kv_heads} key/value heads")
        if int(c.get("vdim", t.dim)) != t.dim:
            raise ConfigError(f"values of {c['vdim']} cannot be keys of {t.dim}")
        return t
    if kind == "parallel":
        return ParallelSpec(vokepel_attention(c["left"]), GruSpec(int(c["right"]["width"])),
                            (float(c["left_scale"]), float(c["right_scale"])))
    raise ConfigError(f"layer type {kind!r} is not part of this design")


def vokepel_mlp(c: Optional[dict]) -> Optional[DenseMlpSpec]:
    if c is None:
        return None
    if c.get("kind") != "dense":
        raise ConfigError(f"feed-forward kind {c.get('kind')!r} is not part of this design")
    return DenseMlpSpec(int(c["ff"]), act="relu2")


def vokepel_model(layers: tuple, *, width: int, vocab: int, eps: float, residual_mult: float, loop: Optional[tuple] = None,
                  logit_scale: float = 1.0, logit_softcap: float = 0.0, name: str = "vokepel"):
    """ModelConfig of Vokepel layers. No tokenizer comes with the design, so there is no end-of-text id."""
    from .config import ModelConfig

    layer_runs(len(layers), loop)
    a = layers[0].mixer.parts[0]
    return ModelConfig(name=name, arch="vokepel", n_layers=len(layers), d_model=width, n_heads=a.heads, n_kv_heads=a.kv_heads,
                       head_dim=a.dim, ffn_dim=max((L.mlp.ff for L in layers if L.mlp), default=0), vocab_size=vocab,
                       max_ctx=1 << 20, rms_eps=eps, tie_embeddings=True, bos_id=-1, eos_id=-1, layers=layers, loop=loop,
                       residual_mult=residual_mult, loop_inject=loop is not None, logit_scale=logit_scale, logit_softcap=logit_softcap)


def vokepel_config(c: dict[str, Any]):
    """ModelConfig of a Vokepel checkpoint from its config.json."""
    layers = tuple(LayerSpec(vokepel_mixer(x["mixer"], x["type"]), vokepel_mlp(x.get("mlp"))) for x in c["layers"])
    lp = c.get("loop")
    return vokepel_model(layers, width=int(c["width"]), vocab=int(c["vocab"]), eps=float(c["norm"]["eps"]),
                         residual_mult=float(c.get("residual_mult", 1.0)),
                         loop=(int(lp["start"]), int(lp["stop"]), int(lp["times"])) if lp else None,
                         logit_scale=float(c.get("logit_scale", 1.0)), logit_softcap=float(c.get("logit_softcap") or 0.0))


def vokepel_json(cfg) -> dict[str, Any]:
    """config.json of a Vokepel ModelConfig (inverse of vokepel_config)."""
    layers = []
    for L in cfg.layers:
        m = L.mixer
        a = m.left if m.kind == "parallel" else m
        c: dict[str, Any] = {"heads": a.heads, "kv_heads": a.kv_heads, "dim": a.dim, "vdim": a.vdim, "scale": a.scale,
                             "mask": {"size": a.window}}
        if m.kind == "parallel":
            if a.rot is not None:
                c["rot"] = {"base": a.rot.base, "dims": a.rot.dims}
            c = {"left": c, "right": {"width": m.right.width}, "left_scale": m.gains[0], "right_scale": m.gains[1]}
        else:
            c["softcap"] = m.softcap
        layers.append({"type": "parallel" if m.kind == "parallel" else "attention", "mixer": c,
                       "mlp": None if L.mlp is None else {"kind": "dense", "ff": L.mlp.ff}})
    out = {"architecture": "Vokepel", "vocab": cfg.vocab_size, "width": cfg.d_model, "norm": {"eps": cfg.rms_eps}, "layers": layers,
           "residual_mult": cfg.residual_mult, "logit_scale": cfg.logit_scale, "logit_softcap": cfg.logit_softcap}
    if cfg.loop is not None:
        out["loop"] = dict(zip(("start", "stop", "times"), cfg.loop))
    return out


def initial_vector(cfg, name: str, shape: tuple):
    """Starting values of a vector (synthetic weights): unit norms (stored as the distance from one where the design
    does so), step sizes of 0.001 to 0.1, decay rates of 1 to 16, distance biases of a few slopes."""
    import numpy as np

    n = shape[0]
    ramp = np.arange(n, dtype=np.float64) / max(1, n - 1)
    if name.endswith(".dt_bias"):
        v = np.log(np.expm1(10.0 ** (-3.0 + 2.0 * ramp)))
    elif name.endswith(".A_log"):
        v = np.log(1.0 + 15.0 * ramp)
    elif name.endswith(".f.b"):
        v = 3.0 + 3.0 * ramp      # forget gates that keep 20 to 400 tokens
    elif name.endswith(".z.b"):
        v = -1.0 - 5.0 * ramp     # update gates that keep 3 to 400 tokens
    elif name.endswith(".r1"):
        v = 2.0 ** (1.0 - 4.0 * ramp)
    elif name.endswith(".r2"):
        v = np.full(n, 0.25)
    elif name.endswith((".b", ".sink", ".lq1", ".lk1", ".lq2", ".lk2")):
        v = np.zeros(n)
    elif name.endswith((".q.norm", ".k.norm", ".D")):
        v = np.ones(n)
    else:
        v = np.full(n, 1.0 - cfg.norm_weight_offset)
    return v.astype(np.float32)


def initial_matrix(name: str, shape: tuple):
    """What synthetic matrices are added to: heads that keep their scores, passes that start with the stream as it is; else None."""
    import numpy as np

    return np.eye(*shape, dtype=np.float32) if name.endswith(".talk") or name == "loop.in" else None


def layer_list_tensors(cfg) -> list[tuple[str, tuple[int, ...]]]:
    """(name, row-major shape) of every tensor of a layer-list model."""
    d, s = cfg.d_model, cfg.streams
    out = [("embed", (cfg.vocab_size, d))]
    if cfg.bigram is not None:
        out.append(("bigram", (cfg.bigram.buckets + 1, d)))
    if cfg.loop_inject:
        out += [("loop.in", (d, 2 * d)), ("loop.step", (cfg.loop[2], d))]
    for i, L in enumerate(cfg.layers):
        p = f"l{i}."
        for q in range(1, L.sublayers + 1):
            out.append((p + f"norm{q}", (d,)))
            if L.post_norm:
                out += [(p + f"norm{q}b", (d,)), (p + f"ls{q}", (d,))]
            if s:
                out += [(p + f"hc{q}.in", (s,)), (p + f"hc{q}.out", (s,)), (p + f"hc{q}.mix", (s, s))]
        out += [(p + "mix." + n, sh) for n, sh in L.mixer.tensors(d)]
        if L.mlp is not None:
            out += [(p + "mlp." + n, sh) for n, sh in L.mlp.tensors(d)]
    out.append(("final.norm", (d,)))
    return out if cfg.tie_embeddings else out + [("head", (cfg.vocab_size, d))]
