"""Small Vokepel models for the tests: configurations of unlike sizes and weights under which a wrong key, window, sink, head,
state or pass shows in the logits."""
import numpy as np

from hybrid_models import bf16_exact


def talk(heads, kv, dim, window, cap=12.0, gain=2.0):
    return {"type": "attention", "mlp": None,
            "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": dim, "scale": gain * dim ** -0.5, "softcap": cap, "mask": {"size": window}}}


def pair(heads, kv, dim, vdim, rot, window, gru, gains=(0.7, 1.2), base=3000.0, gain=1.5):
    left = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": gain * dim ** -0.5, "mask": {"size": window}}
    if rot:
        left["rot"] = {"base": base, "dims": rot}
    return {"type": "parallel", "mlp": None,
            "mixer": {"left": left, "right": {"width": gru}, "left_scale": gains[0], "right_scale": gains[1]}}


def mlp(layer, ff):
    return {**layer, "mlp": {"kind": "dense", "ff": ff}}


def model(width, vocab, layers, loop=None, mult=0.6, logit=(0.4, 9.0), eps=1e-5):
    c = {"architecture": "Vokepel", "width": width, "vocab": vocab, "norm": {"eps": eps}, "layers": layers, "residual_mult": mult,
         "logit_scale": logit[0], "logit_softcap": logit[1]}
    if loop:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    return c


CONFIGS = {
    # both kinds, a loop over the middle, dim != vdim, heads that are no multiple of 8, a layer without MLP
    "mixed": model(160, 300, [mlp(pair(6, 3, 48, 32, 20, 23, 72), 200), mlp(talk(5, 1, 40, 37), 96), pair(4, 1, 80, 96, 80, 70, 200, gains=(1.1, 0.4)),
                              mlp(talk(6, 3, 72, 90, cap=8.0), 130)], loop=(1, 3, 2), eps=1e-3),
    # everything one or the smallest, a width that is no multiple of 8, passes of a single layer, no rotation
    "ones": model(76, 130, [mlp(talk(1, 1, 4, 1), 20), mlp(pair(1, 1, 4, 12, 2, 1, 5), 36), pair(2, 2, 12, 20, 0, 9, 28), mlp(talk(2, 2, 20, 17), 28)],
                  loop=(3, 4, 1), mult=1.0, logit=(1.0, 30.0)),
    # no state: many heads, wide ones, no loop
    "talk": model(128, 200, [mlp(talk(20, 5, 40, 50), 64), mlp(talk(16, 2, 96, 33), 64), talk(9, 9, 64, 130, cap=6.0)], mult=0.8),
    # no talking heads; the whole model three times
    "pair": model(96, 90, [mlp(pair(4, 2, 32, 48, 32, 40, 100), 64), pair(3, 1, 24, 20, 12, 200, 64, gains=(0.3, 1.0))], loop=(0, 2, 3), mult=0.4),
    # head sizes and counts beyond the tensor-core kernels
    "huge": model(64, 100, [mlp(talk(2, 1, 136, 30), 32), mlp(talk(34, 2, 16, 45), 32), mlp(pair(2, 1, 144, 40, 30, 41, 48), 32),
                            mlp(talk(66, 33, 8, 20), 32)], loop=(0, 1, 2)),
}


def weights(cfg, seed=0):
    """Random weights that bf16 holds exactly: peaked softmax, heads that hear one another, sinks of some weight, states of a few to
    hundreds of tokens."""
    from oxide_tech_llm_engine_b200.models.layer_spec import layer_list_tensors, vokepel_config

    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in layer_list_tensors(vokepel_config(cfg)):
        x = rng.standard_normal(shape).astype(np.float32)
        leaf = name.rsplit(".", 1)[-1]
        if name.endswith(".z.b"):
            x = -2.5 + 1.5 * x
        elif name.endswith(".x.b"):
            x = 0.3 * x
        elif leaf == "sink":
            x = 1.5 + x
        elif leaf == "r1":
            x = 1.0 + 0.6 * x
        elif leaf == "r2":
            x = 0.4 + 0.6 * np.abs(x)
        elif leaf == "talk":
            x = 0.8 * np.eye(*shape) + 0.5 * x / np.sqrt(shape[0])
        elif leaf == "step":
            x = 0.4 * x
        elif len(shape) == 1:
            x = 1.0 + 0.2 * x
        elif name == "loop.in":
            d = shape[0]
            x = np.concatenate([0.7 * np.eye(d), 0.4 * np.eye(d)], 1) + 0.3 * x / np.sqrt(d)
        elif name != "embed":
            x = x / np.sqrt(shape[1])
        out[name] = bf16_exact(x)
    return out
