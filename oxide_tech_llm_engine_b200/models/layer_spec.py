"""Descriptions of decoders that are given as a list of layers rather than as one repeated block.

A `LayerSpec` names a token mixer (attention, retention, ...) and a feed-forward, each with its own
sizes and constants, so layers of one model may differ in kind, in head layout and in window. The
specs are plain data: `models.hybrid` builds the device layers from them, `models.cpu_hybrid` the
CPU ones, `models.weights` the tensor list. A further design adds its mixer here as one more
dataclass with the constants as fields, and registers its configuration reader in
`models.registry`.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Optional, Union

from ..errors import ConfigError


@dataclass(frozen=True)
class RotarySpec:
    """Rotation of the first `dims` dimensions of every head: pairs (2i, 2i+1) when `interleaved`,
    else (i, i + dims/2), by the angle position * base^(-2i/dims)."""
    dims: int
    base: float
    interleaved: bool = False


@dataclass(frozen=True)
class AttentionSpec:
    """Softmax attention with grouped key/value heads. `window` 0: every earlier position is visible;
    else the last `window` positions and the first `keep_first` ones of the sequence (which keep their
    true positions). `qk_norm` "projection": RMS norm over all heads of q (of k) at once, before the
    rotation."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot: Optional[RotarySpec] = None
    window: int = 0
    keep_first: int = 0
    qk_norm: str = "none"      # none | projection

    kind = "attention"

    @property
    def out_dim(self) -> int:
        return self.heads * self.vdim

    def tensors(self, d: int) -> list[tuple[str, tuple[int, ...]]]:
        out = [("q", (self.heads * self.dim, d)), ("k", (self.kv_heads * self.dim, d)),
               ("v", (self.kv_heads * self.vdim, d)), ("o", (d, self.out_dim))]
        if self.qk_norm == "projection":
            out += [("q.norm", (self.heads * self.dim,)), ("k.norm", (self.kv_heads * self.dim,))]
        return out


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
    def out_dim(self) -> int:
        return self.heads * self.vdim

    @property
    def state_elems(self) -> int:
        """fp32 values of one sequence's state."""
        return self.heads * self.dim * self.vdim

    def tensors(self, d: int) -> list[tuple[str, tuple[int, ...]]]:
        hd, hv = self.heads * self.dim, self.heads * self.vdim
        return [("q", (hd, d)), ("k", (hd, d)), ("v", (hv, d)), ("g", (hv, d)), ("o", (d, hv))]


@dataclass(frozen=True)
class DenseMlpSpec:
    """W_down (act(W_gate h) * (W_up h))."""
    ff: int
    act: str = "silu"          # silu | gelu_tanh

    def tensors(self, d: int) -> list[tuple[str, tuple[int, ...]]]:
        return [("gate", (self.ff, d)), ("up", (self.ff, d)), ("down", (d, self.ff))]


@dataclass(frozen=True)
class LayerSpec:
    mixer: Union[AttentionSpec, RetentionSpec]
    mlp: Optional[DenseMlpSpec]

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
    return RotarySpec(dims, float(c["base"]), interleaved) if dims else None


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


def layer_list_tensors(cfg) -> list[tuple[str, tuple[int, ...]]]:
    """(name, row-major shape) of every tensor of a layer-list model."""
    d, s = cfg.d_model, cfg.streams
    out = [("embed", (cfg.vocab_size, d))]
    if cfg.bigram is not None:
        out.append(("bigram", (cfg.bigram.buckets + 1, d)))
    for i, L in enumerate(cfg.layers):
        p = f"l{i}."
        for q in range(1, L.sublayers + 1):
            out.append((p + f"norm{q}", (d,)))
            if s:
                out += [(p + f"hc{q}.in", (s,)), (p + f"hc{q}.out", (s,)), (p + f"hc{q}.mix", (s, s))]
        out += [(p + "mix." + n, sh) for n, sh in L.mixer.tensors(d)]
        if L.mlp is not None:
            out += [(p + "mlp." + n, sh) for n, sh in L.mlp.tensors(d)]
    out += [("final.norm", (d,)), ("head", (cfg.vocab_size, d))]
    return out
