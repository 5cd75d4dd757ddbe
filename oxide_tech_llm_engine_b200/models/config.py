"""Model hyper-parameters, named presets and GGUF-metadata -> config mapping.

Reference parity: Llama3Config::from_gguf (oxide-models/src/llama3.rs:165-312) reads
`{arch}.embedding_length/block_count/attention.head_count(_kv)/context_length/rope.freq_base/
attention.layer_norm_rms_epsilon/rope.scaling.*/attention.sliding_window/final_logit_softcapping`,
derives head_dim from `blk.0.attn_q.weight`, the FFN width from `blk.0.ffn_gate.weight` and the
vocabulary from `token_embd.weight`; tiny_test_config (llama3.rs:66-91). MoE keys
(`{arch}.expert_count`, `{arch}.expert_used_count`) are an addition: the reference loads no experts.
"""
from __future__ import annotations

from dataclasses import asdict, dataclass, field, replace
from typing import Any


@dataclass
class ModelConfig:
    name: str = "llama"
    arch: str = "llama"
    n_layers: int = 2
    d_model: int = 128
    n_heads: int = 4
    n_kv_heads: int = 2
    head_dim: int = 32
    ffn_dim: int = 256
    vocab_size: int = 1024
    max_ctx: int = 8192
    rope_theta: float = 10000.0
    rope_scaling: str = "none"  # none | linear | llama3 | yarn
    rope_factor: float = 1.0
    rope_orig_ctx: int = 8192
    rope_low_freq_factor: float = 1.0
    rope_high_freq_factor: float = 4.0
    rms_eps: float = 1e-5
    norm_weight_offset: float = 0.0  # Gemma stores (w - 1)
    emb_scale: float = 1.0  # Gemma multiplies embeddings by sqrt(d_model)
    act: str = "silu"  # silu | gelu_tanh
    qk_norm: bool = False
    attn_bias: bool = False
    sliding_window: int = 0
    logit_softcap: float = 0.0
    tie_embeddings: bool = False
    # mixture of experts (0 experts = dense FFN)
    n_experts: int = 0
    n_experts_used: int = 0
    routed_scale: float = 1.0
    bos_id: int = 1
    eos_id: int = 2
    # layer-list designs (models.layer_spec): one LayerSpec per layer, the range of layers that runs
    # several times, the number of hyper-connected residual streams (0: one plain residual), and the
    # second embedding. Empty for the Llama family.
    layers: tuple = ()
    loop: Any = None           # (start, stop, times)
    streams: int = 0
    bigram: Any = None         # layer_spec.BigramSpec
    # one plain residual stream with a norm before every sublayer, whose result is added times this (None: the other kinds)
    residual_mult: Any = None
    loop_inject: bool = False  # every pass of the loop starts with x <- W_in [x; embedding] + a vector of the pass
    logit_scale: float = 1.0   # before the softcap

    @property
    def q_dim(self) -> int:
        return self.n_heads * self.head_dim

    @property
    def kv_dim(self) -> int:
        return self.n_kv_heads * self.head_dim

    @property
    def is_moe(self) -> bool:
        return self.n_experts > 0

    @property
    def layer_runs(self) -> list:
        """Layer index of every layer run, in order (a looped layer counts each time)."""
        from .layer_spec import layer_runs

        return layer_runs(self.n_layers, self.loop)

    @property
    def pass_starts(self) -> dict:
        """Number of the pass by the index of the layer run that it begins with."""
        if self.loop is None:
            return {}
        a, b, times = self.loop
        return {a + t * (b - a): t for t in range(times)}

    @property
    def is_recurrent(self) -> bool:
        """Some layer carries a per-sequence state besides the paged KV."""
        return any(hasattr(part, "state_elems") for L in self.layers for part in L.mixer.parts)

    def n_params(self) -> int:
        if self.layers:
            from math import prod

            from .layer_spec import layer_list_tensors

            return sum(prod(s) for _, s in layer_list_tensors(self))
        per_layer = self.d_model * (self.q_dim + 2 * self.kv_dim) + self.q_dim * self.d_model
        ffn = 3 * self.d_model * self.ffn_dim
        per_layer += ffn * max(1, self.n_experts) + (self.n_experts * self.d_model if self.is_moe else 0)
        per_layer += 2 * self.d_model
        emb = self.vocab_size * self.d_model * (1 if self.tie_embeddings else 2)
        return self.n_layers * per_layer + emb + self.d_model

    def active_params(self) -> int:
        if self.layers:
            idle = sum((3 if L.mlp.glu else 2) * (L.mlp.experts - L.mlp.top) * L.mlp.ff * self.d_model for L in self.layers
                       if L.mlp is not None and L.mlp.kind == "moe")
            return self.n_params() - idle
        if not self.is_moe:
            return self.n_params()
        per_layer = self.d_model * (self.q_dim + 2 * self.kv_dim) + self.q_dim * self.d_model
        per_layer += 3 * self.d_model * self.ffn_dim * self.n_experts_used
        return self.n_layers * per_layer + 2 * self.vocab_size * self.d_model

    def kv_bytes_per_token(self, dtype_bytes: int = 2) -> int:
        if self.layers:
            return sum(getattr(m, "cache_values", 0) for i in self.layer_runs for m in self.layers[i].mixer.parts) * dtype_bytes
        return 2 * self.n_layers * self.kv_dim * dtype_bytes

    def to_dict(self) -> dict[str, Any]:
        return asdict(self)


PRESETS: dict[str, ModelConfig] = {
    # the reference's tiny test model (llama3.rs:66-91): h=128, L=2, 4/2 heads, vocab 1024
    "tiny": ModelConfig(name="tiny", n_layers=2, d_model=128, n_heads=4, n_kv_heads=2, head_dim=64,
                        ffn_dim=256, vocab_size=1024, max_ctx=2048),
    "tiny-moe": ModelConfig(name="tiny-moe", arch="mixtral", n_layers=2, d_model=128, n_heads=4,
                            n_kv_heads=2, head_dim=64, ffn_dim=256, vocab_size=1024, max_ctx=2048,
                            n_experts=8, n_experts_used=2),
    # CPU plumbing config: 22 layers, 2048-d, 32q/4kv heads of 64, FFN 5632, vocab 32000
    "tinyllama-1.1b": ModelConfig(name="tinyllama-1.1b", n_layers=22, d_model=2048, n_heads=32,
                                  n_kv_heads=4, head_dim=64, ffn_dim=5632, vocab_size=32000,
                                  rope_theta=10000.0, rms_eps=1e-5, max_ctx=2048),
    "llama3-8b": ModelConfig(name="llama3-8b", n_layers=32, d_model=4096, n_heads=32, n_kv_heads=8,
                             head_dim=128, ffn_dim=14336, vocab_size=128256, rope_theta=500000.0,
                             rms_eps=1e-5, max_ctx=131072, bos_id=128000, eos_id=128001),
    "llama3-70b": ModelConfig(name="llama3-70b", n_layers=80, d_model=8192, n_heads=64, n_kv_heads=8,
                              head_dim=128, ffn_dim=28672, vocab_size=128256, rope_theta=500000.0,
                              rms_eps=1e-5, max_ctx=131072, bos_id=128000, eos_id=128001),
    "mixtral-8x7b": ModelConfig(name="mixtral-8x7b", arch="mixtral", n_layers=32, d_model=4096,
                                n_heads=32, n_kv_heads=8, head_dim=128, ffn_dim=14336, vocab_size=32000,
                                rope_theta=1000000.0, rms_eps=1e-5, max_ctx=32768, n_experts=8,
                                n_experts_used=2),
}


def _kipolix_preset(name: str, *, width: int, vocab: int, ff: int, pattern: str, heads: int, kv_heads: int, dim: int,
                    window: int, keep_first: int, r_heads: int, r_dim: int, r_vdim: int, streams: int = 2,
                    loop=None, buckets: int = 0) -> ModelConfig:
    """A Kipolix-shaped configuration: one letter per layer, 'a' attention or 'r' retention. Decays are
    1 - 2^(-5 - i), the usual multi-scale choice of retention heads."""
    from .layer_spec import AttentionSpec, BigramSpec, DenseMlpSpec, LayerSpec, RetentionSpec, RotarySpec

    att = AttentionSpec(heads, kv_heads, dim, dim, dim ** -0.5, RotarySpec(dim // 2, 10000.0, True), window,
                        keep_first, "projection")
    ret = RetentionSpec(r_heads, r_dim, r_vdim, tuple(1.0 - 2.0 ** (-5 - 8.0 * i / max(1, r_heads)) for i in range(r_heads)),
                        RotarySpec(r_dim, 500000.0, False))
    mlp = DenseMlpSpec(ff)
    layers = tuple(LayerSpec(att if ch == "a" else ret, mlp) for ch in pattern)
    return ModelConfig(name=name, arch="kipolix", n_layers=len(layers), d_model=width, n_heads=heads, n_kv_heads=kv_heads,
                       head_dim=dim, ffn_dim=ff, vocab_size=vocab, max_ctx=1 << 20, rms_eps=1e-5, norm_weight_offset=1.0,
                       bos_id=-1, eos_id=-1, layers=layers, loop=loop, streams=streams,
                       bigram=BigramSpec(buckets, 40503, 10007) if buckets else None)


def _povatar_preset(name: str, *, width: int, vocab: int, n_layers: int, heads: int, kv_heads: int, dim: int, chunk: int,
                    s_heads: int, s_vdim: int, state: int, groups: int, ff: int, experts: int, top: int) -> ModelConfig:
    """A Povatar-shaped configuration of equal layers: a quarter of every head rotates, four taps."""
    from .layer_spec import AttentionSpec, LayerSpec, MoeSpec, ParallelSpec, RotarySpec, SsdSpec, YarnSpec, povatar_model

    left = AttentionSpec(heads, kv_heads, dim, dim, dim ** -0.5, RotarySpec(dim // 4, 500000.0, False, YarnSpec(8.0, 8192, 32.0, 1.0)),
                         chunk=chunk, sink=0.0)
    layer = LayerSpec(ParallelSpec(left, SsdSpec(s_heads, s_vdim, state, groups, 4, groups)), MoeSpec(ff, experts, top), parallel=True)
    return povatar_model((layer,) * n_layers, width=width, vocab=vocab, eps=1e-5, emb_scale=width ** 0.5, name=name)


def _zagolix_preset(name: str, *, width: int, vocab: int, pattern: str, ff: int, heads: int, kv_heads: int, dim: int, l_heads: int,
                    l_dim: int, rot: int, l_vdim: int, q_rank: int, kv_rank: int, m_heads: int, m_dim: int, m_vdim: int, e_ff: int,
                    experts: int, top: int, groups: int, keep: int) -> ModelConfig:
    """A Zagolix-shaped configuration: one letter per layer, 'a' differential attention, 'l' latent attention, 's' latent
    attention that reads what the last 'l' keeps, 'm' matrix memory. The first layer's feed-forward is dense."""
    from .layer_spec import AttentionSpec, DenseMlpSpec, LatentSpec, LayerSpec, MemorySpec, MoeSpec, RotarySpec, zagolix_model

    moe = MoeSpec(e_ff, experts, top, act="silu_glu", scores="sigmoid", groups=groups, keep=keep)
    layers, owner = [], None
    for i, ch in enumerate(pattern):
        if ch == "a":
            mx = AttentionSpec(heads, kv_heads, dim, 2 * dim, dim ** -0.5, bias=True, diff=0.5, temp_coef=0.1, temp_every=8192.0)
        elif ch == "m":
            mx = MemorySpec(m_heads, m_dim, m_vdim, 15.0)
        else:
            owner = i if ch == "l" else owner
            mx = LatentSpec(l_heads, l_dim, l_vdim, q_rank, kv_rank, (l_dim + rot) ** -0.5, RotarySpec(rot, 10000.0, True),
                            owner if ch == "s" else None)
        layers.append(LayerSpec(mx, DenseMlpSpec(ff, act="gelu_tanh") if i == 0 else moe, post_norm=True))
    return zagolix_model(tuple(layers), width=width, vocab=vocab, eps=1e-5, emb_scale=width ** 0.5, name=name)


def _vokepel_preset(name: str, *, width: int, vocab: int, pattern: str, ff: int, heads: int, kv_heads: int, dim: int, window: int,
                    t_heads: int, t_kv: int, t_dim: int, t_window: int, gru: int, loop=None) -> ModelConfig:
    """A Vokepel-shaped configuration: one letter per layer, 'p' attention with sinks beside a gated recurrence, 't' talking
    heads."""
    from .layer_spec import (AttentionSpec, DenseMlpSpec, GruSpec, LayerSpec, ParallelSpec, RotarySpec, TalkingSpec,
                             vokepel_model)

    left = AttentionSpec(heads, kv_heads, dim, dim, dim ** -0.5, RotarySpec(dim, 500000.0, True), window, sinks=True)
    pair = ParallelSpec(left, GruSpec(gru), (0.5, 0.5))
    talk = TalkingSpec(t_heads, t_kv, t_dim, t_dim ** -0.5, 30.0, t_window)
    layers = tuple(LayerSpec(pair if ch == "p" else talk, DenseMlpSpec(ff, act="relu2")) for ch in pattern)
    return vokepel_model(layers, width=width, vocab=vocab, eps=1e-5, residual_mult=0.5, loop=loop, logit_scale=0.5,
                         logit_softcap=30.0, name=name)


LAYER_LIST_PRESETS = {
    "kipolix-tiny": dict(width=128, vocab=1024, ff=256, pattern="arar", heads=4, kv_heads=2, dim=64, window=56,
                         keep_first=3, r_heads=2, r_dim=64, r_vdim=64, streams=2, loop=(1, 3, 2), buckets=1000),
    # the shapes of llama3-8b's layers (width, FFN, heads), alternating attention and retention
    "kipolix-8b": dict(width=4096, vocab=128256, ff=14336, pattern="ar" * 16, heads=32, kv_heads=8, dim=128, window=4096,
                       keep_first=16, r_heads=32, r_dim=128, r_vdim=128, streams=2, buckets=65521),
}


POVATAR_PRESETS = {
    "povatar-tiny": dict(width=128, vocab=1024, n_layers=3, heads=4, kv_heads=2, dim=64, chunk=80, s_heads=4, s_vdim=48, state=40,
                         groups=2, ff=80, experts=12, top=3),
    # layers of a mid-size mixture: heads of 128 over 8192-token chunks, a state of 128 x 64 per head, 8 of 64 experts
    "povatar-16b": dict(width=2048, vocab=128256, n_layers=32, heads=16, kv_heads=4, dim=128, chunk=8192, s_heads=64, s_vdim=64,
                        state=128, groups=8, ff=1408, experts=64, top=8),
}


ZAGOLIX_PRESETS = {
    "zagolix-tiny": dict(width=128, vocab=1024, pattern="alsm", ff=256, heads=2, kv_heads=1, dim=32, l_heads=3, l_dim=32, rot=16,
                         l_vdim=48, q_rank=56, kv_rank=64, m_heads=2, m_dim=32, m_vdim=64, e_ff=80, experts=9, top=3, groups=3, keep=2),
    # layers of a mid-size mixture: latents of 512 + 64 values, two layers per latent, memories of 256 x 512, 8 of 64 experts
    "zagolix-16b": dict(width=2048, vocab=128256, pattern="alsm" * 8, ff=10944, heads=16, kv_heads=4, dim=64, l_heads=16, l_dim=128,
                        rot=64, l_vdim=128, q_rank=1536, kv_rank=512, m_heads=4, m_dim=256, m_vdim=512, e_ff=1408, experts=64,
                        top=6, groups=8, keep=4),
}


VOKEPEL_PRESETS = {
    "vokepel-tiny": dict(width=128, vocab=1024, pattern="ptp", ff=320, heads=4, kv_heads=2, dim=32, window=72, t_heads=3, t_kv=1,
                         t_dim=48, t_window=40, gru=144, loop=(1, 3, 2)),
    # the shapes of llama3-8b's layers (width, heads), eight of 24 layers run twice
    "vokepel-8b": dict(width=4096, vocab=128256, pattern="pt" * 12, ff=16384, heads=32, kv_heads=8, dim=128, window=4096, t_heads=32,
                       t_kv=8, t_dim=128, t_window=1024, gru=4096, loop=(8, 16, 2)),
}


def preset_names() -> list:
    return [*PRESETS, *LAYER_LIST_PRESETS, *POVATAR_PRESETS, *ZAGOLIX_PRESETS, *VOKEPEL_PRESETS]


def preset(name: str, **overrides) -> ModelConfig:
    if name in LAYER_LIST_PRESETS:
        return replace(_kipolix_preset(name, **LAYER_LIST_PRESETS[name]), **overrides)
    if name in POVATAR_PRESETS:
        return replace(_povatar_preset(name, **POVATAR_PRESETS[name]), **overrides)
    if name in ZAGOLIX_PRESETS:
        return replace(_zagolix_preset(name, **ZAGOLIX_PRESETS[name]), **overrides)
    if name in VOKEPEL_PRESETS:
        return replace(_vokepel_preset(name, **VOKEPEL_PRESETS[name]), **overrides)
    if name not in PRESETS:
        raise KeyError(f"unknown model preset {name!r}; known: {sorted(preset_names())}")
    return replace(PRESETS[name], **overrides)


def config_from_gguf(g) -> ModelConfig:
    """Build a ModelConfig from GGUF metadata and tensor shapes."""
    md = g.metadata
    arch = str(md.get("general.architecture", "llama"))

    def get(key, default=None):
        return md.get(f"{arch}.{key}", default)

    d_model = int(get("embedding_length"))
    n_layers = int(get("block_count"))
    n_heads = int(get("attention.head_count"))
    n_kv = int(get("attention.head_count_kv", n_heads))
    if "blk.0.attn_q.weight" in g.tensors:
        q_out = g.tensors["blk.0.attn_q.weight"].torch_shape[0]
        head_dim = q_out // n_heads
    elif "blk.0.attn_qkv.weight" in g.tensors:
        qkv_out = g.tensors["blk.0.attn_qkv.weight"].torch_shape[0]
        head_dim = qkv_out // (n_heads + 2 * n_kv)
    else:
        head_dim = int(get("attention.key_length", d_model // n_heads))
    n_experts = int(get("expert_count", 0) or 0)
    if n_experts > 0 and "blk.0.ffn_gate_exps.weight" in g.tensors:
        ffn = g.tensors["blk.0.ffn_gate_exps.weight"].torch_shape[-2]
    elif "blk.0.ffn_gate.weight" in g.tensors:
        ffn = g.tensors["blk.0.ffn_gate.weight"].torch_shape[0]
    else:
        ffn = int(get("feed_forward_length", 4 * d_model))
    vocab = g.tensors["token_embd.weight"].torch_shape[0] if "token_embd.weight" in g.tensors else int(
        get("vocab_size", 32000))
    scaling = str(get("rope.scaling.type", "none") or "none")
    factor = float(get("rope.scaling.factor", 1.0) or 1.0)
    if scaling == "none" and factor > 1.0:
        scaling = "llama3" if arch == "llama" else "linear"
    is_gemma = arch.startswith("gemma")
    cfg = ModelConfig(
        name=str(md.get("general.name", arch)), arch=arch, n_layers=n_layers, d_model=d_model,
        n_heads=n_heads, n_kv_heads=n_kv, head_dim=head_dim, ffn_dim=int(ffn), vocab_size=int(vocab),
        max_ctx=int(get("context_length", 8192)), rope_theta=float(get("rope.freq_base", 10000.0)),
        rope_scaling=scaling, rope_factor=factor,
        rope_orig_ctx=int(get("rope.scaling.original_context_length", 8192) or 8192),
        rms_eps=float(get("attention.layer_norm_rms_epsilon", 1e-5)),
        norm_weight_offset=1.0 if is_gemma else 0.0,
        emb_scale=float(d_model) ** 0.5 if is_gemma else 1.0,
        act="gelu_tanh" if is_gemma else "silu",
        qk_norm="blk.0.attn_q_norm.weight" in g.tensors,
        attn_bias="blk.0.attn_q.bias" in g.tensors,
        sliding_window=int(get("attention.sliding_window", 0) or 0),
        logit_softcap=float(get("final_logit_softcapping", 0.0) or 0.0),
        tie_embeddings="output.weight" not in g.tensors,
        n_experts=n_experts, n_experts_used=int(get("expert_used_count", 0) or 0),
        bos_id=int(md.get("tokenizer.ggml.bos_token_id", 1)),
        eos_id=int(md.get("tokenizer.ggml.eos_token_id", 2)),
    )
    return cfg


def gguf_metadata(cfg: ModelConfig) -> dict[str, Any]:
    """Metadata block of a GGUF checkpoint for this config (inverse of config_from_gguf)."""
    if cfg.layers:
        raise ValueError(f"{cfg.name}: layer-list models have no GGUF form (SafeTensors with config.json)")
    a = cfg.arch
    md: dict[str, Any] = {
        "general.architecture": a,
        "general.name": cfg.name,
        f"{a}.embedding_length": cfg.d_model,
        f"{a}.block_count": cfg.n_layers,
        f"{a}.attention.head_count": cfg.n_heads,
        f"{a}.attention.head_count_kv": cfg.n_kv_heads,
        f"{a}.context_length": cfg.max_ctx,
        f"{a}.feed_forward_length": cfg.ffn_dim,
        f"{a}.rope.freq_base": float(cfg.rope_theta),
        f"{a}.attention.layer_norm_rms_epsilon": float(cfg.rms_eps),
        f"{a}.attention.key_length": cfg.head_dim,
        "tokenizer.ggml.bos_token_id": cfg.bos_id,
        "tokenizer.ggml.eos_token_id": cfg.eos_id,
    }
    if cfg.rope_scaling != "none":
        md[f"{a}.rope.scaling.type"] = cfg.rope_scaling
        md[f"{a}.rope.scaling.factor"] = float(cfg.rope_factor)
        md[f"{a}.rope.scaling.original_context_length"] = cfg.rope_orig_ctx
    if cfg.sliding_window:
        md[f"{a}.attention.sliding_window"] = cfg.sliding_window
    if cfg.logit_softcap:
        md[f"{a}.final_logit_softcapping"] = float(cfg.logit_softcap)
    if cfg.is_moe:
        md[f"{a}.expert_count"] = cfg.n_experts
        md[f"{a}.expert_used_count"] = cfg.n_experts_used
    return md
