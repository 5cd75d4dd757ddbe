"""Small Zagolix models for the tests: configurations of unlike sizes and weights under which a wrong key, state, gate,
map or expert shows in the logits."""
import numpy as np

from hybrid_models import bf16_exact


def att(heads, kv, dim, vdim, diff=0.4, temp=(0.7, 13), gain=1.5):
    c = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": gain * dim ** -0.5, "diff": diff}
    if temp:
        c["q_temp"] = {"coef": temp[0], "every": temp[1]}
    return {"type": "attention", "mixer": c, "mlp": None}


def lat(heads, dim, vdim, q_rank, kv_rank, rot, base=1000.0, src=None, gain=1.5):
    c = {"heads": heads, "dim": dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "rot_dim": rot,
         "rot": {"base": base, "dims": rot}, "scale": gain * (dim + rot) ** -0.5}
    if src is not None:
        c["kv_from"] = src
    return {"type": "latent_attention", "mixer": c, "mlp": None}


def mem(heads, dim, vdim, cap=9.0):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}, "mlp": None}


def dense(layer, ff):
    return {**layer, "mlp": {"kind": "dense", "ff": ff}}


def moe(layer, experts, top, ff, groups=None):
    """`groups`: (count, keep)."""
    r = {"experts": experts, "top": top}
    if groups:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    return {**layer, "mlp": {"kind": "moe", "expert": {"ff": ff}, "router": r}}


def model(width, vocab, layers, eps=1e-5, scale=3.0):
    return {"architecture": "Zagolix", "width": width, "vocab": vocab, "norm": {"eps": eps}, "embedding": {"scale": scale},
            "layers": layers}


CONFIGS = {
    # all kinds in an order of their own; shared latents used twice, a layer without MLP, sizes that are no multiples of 16
    "mixed": model(160, 300, [moe(mem(3, 40, 56), 15, 2, 40, (5, 2)), dense(lat(5, 24, 40, 52, 72, 12), 100), moe(att(4, 2, 32, 48), 8, 3, 72),
                              lat(3, 56, 24, 28, 72, 12, src=1), moe(att(6, 3, 40, 96, diff=0.75, temp=(0.3, 32)), 12, 1, 36, (3, 1)),
                              dense(lat(7, 16, 64, 40, 72, 12, src=1), 60)], eps=1e-3),
    # everything one (or the smallest), a width that is no multiple of 8
    "ones": model(76, 130, [dense(att(1, 1, 4, 20, diff=0.1, temp=None), 20), moe(lat(1, 4, 4, 8, 4, 2), 1, 1, 20),
                            moe(mem(1, 4, 12, cap=2.0), 2, 2, 36, (1, 1)), moe(lat(2, 12, 20, 20, 4, 2, src=1), 4, 2, 28, (4, 3))], scale=1.0),
    # recurrent only: no pages
    "memory": model(96, 90, [dense(mem(2, 32, 144), 64), moe(mem(4, 24, 20, cap=20.0), 6, 2, 32, (2, 2)), mem(1, 80, 64)]),
    # no state; the key and value sizes of the tensor-core kernels for wide heads
    "wide": model(128, 200, [moe(att(2, 1, 72, 136, temp=(0.2, 64)), 66, 5, 24, (6, 3)), dense(lat(3, 112, 128, 64, 96, 48), 64),
                             lat(17, 8, 16, 24, 96, 48, src=1), dense(lat(2, 136, 200, 88, 160, 32, base=500.0), 64),
                             dense(att(10, 1, 16, 64), 32)]),
    # head and latent sizes beyond the tensor-core kernels
    "huge": model(64, 100, [dense(att(2, 1, 136, 40), 32), moe(lat(2, 264, 24, 40, 528, 16), 3, 1, 32),
                            dense(lat(1, 24, 280, 16, 528, 16, src=1), 32), dense(mem(1, 520, 36), 32)]),
}


def weights(cfg, seed=0):
    """Random weights that bf16 holds exactly: peaked softmax, memories from a few to hundreds of tokens, input gates of
    several sizes, routers with clear choices."""
    from oxide_tech_llm_engine_b200.models.layer_spec import layer_list_tensors, zagolix_config

    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in layer_list_tensors(zagolix_config(cfg)):
        x = rng.standard_normal(shape).astype(np.float32)
        leaf = name.rsplit(".", 1)[-1]
        if name.endswith(".f.b"):
            x = 3.0 + 2.0 * x
        elif name.endswith(".i.b"):
            x = 0.5 + 1.0 * x
        elif leaf == "b":
            x = 0.3 * x
        elif leaf in ("lq1", "lk1", "lq2", "lk2"):
            x = 0.8 * x / np.sqrt(shape[0])
        elif leaf.startswith("ls"):
            x = 0.8 + 0.2 * x
        elif len(shape) == 1:
            x = 1.0 + 0.2 * x
        elif name == "embed":
            x = x / cfg["embedding"]["scale"]
        elif leaf == "router":
            x = x * (2.5 / np.sqrt(shape[1]))
        elif leaf in ("i", "f"):
            x = x * (2.0 / np.sqrt(shape[1]))
        else:
            x = x / np.sqrt(shape[1])
        out[name] = bf16_exact(x)
    return out
