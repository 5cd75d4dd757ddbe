"""Model registry: which configuration reader and which device / CPU model class serve an architecture.

An entry covers everything that differs between designs; the engine, its scheduler, cache manager,
sampler, server and command line see only `ModelConfig` and the interface that the classes share
(`load`, `init_random`, `forward`, `copy_blocks`, `kv_block_bytes`, `state_bytes_per_seq`,
`reset_sync_state`, `close`).
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Callable, Optional

from ..errors import ConfigError


@dataclass(frozen=True)
class Architecture:
    name: str
    device_model: Callable[[], type]           # lazily imported classes
    cpu_model: Callable[[], type]
    from_json: Optional[Callable[[dict], Any]] = None   # reader of a native config.json ("architecture" key)
    hf_names: bool = True                       # checkpoint tensors carry Hugging Face names


def _llama():
    from .llama import DeviceModel

    return DeviceModel


def _llama_cpu():
    from .cpu_model import CpuPagedModel

    return CpuPagedModel


def _hybrid():
    from .hybrid import HybridModel

    return HybridModel


def _hybrid_cpu():
    from .cpu_hybrid import CpuHybridModel

    return CpuHybridModel


def _kipolix_json(c: dict):
    from .layer_spec import kipolix_config

    return kipolix_config(c)


def _povatar_json(c: dict):
    from .layer_spec import povatar_config

    return povatar_config(c)


def _zagolix_json(c: dict):
    from .layer_spec import zagolix_config

    return zagolix_config(c)


def _vokepel_json(c: dict):
    from .layer_spec import vokepel_config

    return vokepel_config(c)


ARCHITECTURES: dict[str, Architecture] = {}


def register(a: Architecture) -> None:
    ARCHITECTURES[a.name] = a


register(Architecture("llama", _llama, _llama_cpu))
register(Architecture("mixtral", _llama, _llama_cpu))
register(Architecture("kipolix", _hybrid, _hybrid_cpu, from_json=_kipolix_json, hf_names=False))
register(Architecture("povatar", _hybrid, _hybrid_cpu, from_json=_povatar_json, hf_names=False))
register(Architecture("zagolix", _hybrid, _hybrid_cpu, from_json=_zagolix_json, hf_names=False))
register(Architecture("vokepel", _hybrid, _hybrid_cpu, from_json=_vokepel_json, hf_names=False))


def architecture(cfg) -> Architecture:
    """Entry of a model configuration (any other GGUF architecture name is a Llama-family one)."""
    return ARCHITECTURES.get(cfg.arch, ARCHITECTURES["llama"])


def config_from_json(c: dict):
    """ModelConfig of a config.json that names its design in "architecture"; None when it does not
    (a Hugging Face configuration)."""
    name = c.get("architecture")
    if name is None:
        return None
    a = ARCHITECTURES.get(str(name).lower())
    if a is None or a.from_json is None:
        known = sorted(k for k, v in ARCHITECTURES.items() if v.from_json is not None)
        raise ConfigError(f"architecture {name!r} is not part of this engine; known: {known}")
    return a.from_json(c)
