"""Small Povatar models for the tests: configurations of unlike sizes and weights under which a wrong key, chunk
edge, sink, state, convolution input or expert shows in the logits."""
import numpy as np

from hybrid_models import bf16_exact


def left(heads, kv, dim, vdim, chunk, rot=None, gain=1.5):
    """`rot`: (dims, base) or (dims, base, factor, original, fast, slow)."""
    c = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": gain * dim ** -0.5}
    if chunk:
        c["mask"] = {"size": chunk}
    if rot:
        c["rot"] = {"dims": rot[0], "base": rot[1]}
        if len(rot) > 2:
            c["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), rot[2:]))
    return c


def right(heads, vdim, state, groups, taps, norm_groups):
    return {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": taps, "norm_groups": norm_groups}


def layer(a, b, moe=None):
    """`moe`: (experts, top, ff)."""
    mlp = {"kind": "moe", "router": {"experts": moe[0], "top": moe[1]}, "expert": {"ff": moe[2]}} if moe else None
    return {"type": "parallel", "mixer": {"left": a, "right": b}, "mlp": mlp}


def model(width, vocab, layers, eps=1e-5, scale=3.0):
    return {"architecture": "Povatar", "width": width, "vocab": vocab, "norm": {"eps": eps}, "embedding": {"scale": scale},
            "layers": layers}


CONFIGS = {
    # unlike layers: grouped heads, dim != vdim, norm parts across heads, sizes that are no multiples of 16, no MLP once
    "mixed": model(160, 300, [
        layer(left(6, 3, 48, 32, 37, (24, 10000.0, 8.0, 64, 20.0, 1.0)), right(6, 20, 24, 3, 3, 4), (7, 3, 40)),
        layer(left(5, 1, 80, 96, 16), right(2, 48, 80, 1, 5, 1)),
        layer(left(4, 4, 64, 64, 130, (64, 500.0)), right(8, 64, 128, 2, 4, 8), (33, 1, 100))], eps=1e-3),
    # everything one, and a width that is no multiple of 8
    "ones": model(76, 130, [layer(left(1, 1, 20, 36, 1, (8, 100.0)), right(1, 16, 16, 1, 1, 1), (1, 1, 20)),
                            layer(left(2, 1, 64, 64, 0, (32, 10000.0, 2.0, 32, 4.0, 0.5)), right(3, 7, 5, 1, 2, 3), (2, 2, 36))],
                  scale=1.0),
    # head and state sizes beyond the tensor-core kernels, many experts, many chosen
    "wide": model(128, 200, [layer(left(2, 1, 144, 72, 41, (40, 10000.0, 4.0, 100, 16.0, 1.0)), right(4, 24, 272, 4, 9, 2), (130, 9, 24)),
                             layer(left(3, 3, 16, 144, 70, (16, 50.0)), right(2, 80, 96, 1, 4, 5), (70, 2, 64))]),
}


def weights(cfg, seed=0):
    """Random weights that bf16 holds exactly: peaked softmax, memories from a few to hundreds of tokens, step sizes
    around 0.2, routers with clear choices."""
    from oxide_tech_llm_engine_b200.models.layer_spec import layer_list_tensors, povatar_config

    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in layer_list_tensors(povatar_config(cfg)):
        x = rng.standard_normal(shape).astype(np.float32)
        leaf = name.rsplit(".", 1)[-1]
        if name.endswith(".dt_bias"):
            x = -1.5 + 0.5 * x
        elif leaf == "A_log":
            x = -2.5 + 1.5 * x
        elif leaf == "D":
            x = 0.7 + 0.3 * x
        elif name.endswith(".conv"):
            x = 0.6 * x
        elif name.endswith(".conv.b"):
            x = 0.2 * x
        elif len(shape) == 1:
            x = 1.0 + 0.2 * x
        elif name == "embed":
            x = x / cfg["embedding"]["scale"]
        elif leaf == "router":
            x = x * (2.5 / np.sqrt(shape[1]))
        else:
            x = x * ((0.7 if leaf in ("o", "down") else 1.0) / np.sqrt(shape[1]))
        out[name] = bf16_exact(x)
    return out
