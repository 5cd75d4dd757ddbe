"""Small layer-list models for the tests: configurations of unlike sizes and weights under which a wrong
key, window edge, state or stream shows in the logits."""
import json
import os

import numpy as np

from oxide_tech_llm_engine_b200.formats.safetensors import write_safetensors


def att(heads, kv, dim, vdim, rot, window, keep, base=10000.0, gain=1.0):
    return {"type": "attention", "mlp": None,
            "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "rot": {"base": base, "dims": rot},
                      "scale": gain * dim ** -0.5, "mask": {"size": window, "keep_first": keep}}}


def ret(heads, dim, vdim, rot, decay, base=5000.0):
    return {"type": "retention", "mlp": None,
            "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "rot": {"base": base, "dims": rot}, "decay": decay}}


def mlp(layer, ff):
    return {**layer, "mlp": {"kind": "dense", "ff": ff}}


def model(width, vocab, layers, streams=2, loop=None, buckets=61, mul=(7, 11), eps=1e-5):
    c = {"architecture": "Kipolix", "width": width, "vocab": vocab, "norm": {"eps": eps}, "streams": streams, "layers": layers,
         "embedding": {"bigram": {"buckets": buckets, "mul_prev": mul[0], "mul_cur": mul[1]}} if buckets else {}}
    if loop:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    return c


CONFIGS = {
    # both kinds, unlike head layouts, dim != vdim, a loop over a prefix, three streams, a layer without MLP
    "mixed": model(160, 300, [mlp(ret(3, 40, 24, 16, [0.9, 0.98, 0.9995]), 200),
                              mlp(att(6, 3, 48, 32, 20, 23, 5, gain=1.5), 96),
                              att(5, 1, 80, 96, 80, 70, 17, gain=1.5),
                              mlp(ret(1, 64, 160, 64, [0.999]), 130)], streams=3, loop=(0, 2, 2), eps=1e-3),
    # attention only: no state slots; widths that are no multiple of 8, one stream, no kept first positions
    "attention": model(76, 130, [mlp(att(2, 2, 20, 36, 8, 16, 0, gain=1.5), 36), mlp(att(4, 1, 64, 64, 64, 33, 1, gain=1.5), 70)],
                       streams=1, buckets=0),
    # recurrent only: no KV pages in use; four streams, the whole model looped, decay 1 and a fast one
    "retention": model(96, 90, [mlp(ret(2, 32, 48, 32, [1.0, 0.25]), 64), ret(4, 24, 20, 12, [0.99, 0.97, 0.9, 0.5])],
                       streams=4, loop=(0, 2, 2), mul=(13, 5)),
    # head sizes beyond the tensor-core attention, more streams than four, no bigram, window of one
    "wide": model(128, 200, [mlp(att(2, 1, 144, 72, 40, 41, 3, gain=1.5), 64), mlp(att(3, 3, 16, 144, 16, 1, 2), 64),
                             mlp(ret(1, 136, 264, 8, [0.995]), 96)], streams=5, buckets=0),
}


def weights(cfg, seed=0):
    """Random weights that bf16 holds exactly; q / k projections are large enough for peaked softmax."""
    from oxide_tech_llm_engine_b200.models.layer_spec import kipolix_config, layer_list_tensors

    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in layer_list_tensors(kipolix_config(cfg)):
        x = rng.standard_normal(shape).astype(np.float32)
        if ".hc" in name:
            s = shape[0]
            if name.endswith(".mix"):
                x = 0.9 * np.eye(s) + 0.15 * x
            elif name.endswith(".in"):
                x = 1.0 / s + 0.3 * x
            else:
                x = 0.6 + 0.2 * x
        elif name.endswith((".q.norm", ".k.norm")):
            x = 1.0 + 0.2 * x
        elif len(shape) == 1:
            x = 0.2 * x
        elif name in ("embed", "bigram"):
            x = x * 0.7
        else:
            x = x * ((0.7 if name.endswith((".o", ".down")) else 1.0) / np.sqrt(shape[1]))
        out[name] = bf16_exact(x)
    return out


def bf16_exact(x):
    """The values rounded to what bf16 holds."""
    u = np.ascontiguousarray(x, dtype=np.float32).view(np.uint32)
    return ((u + 0x8000) & 0xFFFF0000).astype(np.uint32).view(np.float32).reshape(np.shape(x)).copy()


class DictSource:
    """A checkpoint in memory, with the interface of models.weights.WeightSource."""

    def __init__(self, cfg, w):
        from oxide_tech_llm_engine_b200.models.registry import config_from_json

        self.cfg, self.w = config_from_json(cfg), w

    def names(self):
        return self.w.keys()

    def has(self, n):
        return n in self.w

    def type_name(self, n):
        return "BF16"

    def shape(self, n):
        return self.w[n].shape

    def f32(self, n):
        return self.w[n]


def write_model(path, cfg, w):
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    write_safetensors(os.path.join(path, "model.safetensors"), w, dtype="BF16")


def engine(cfg, w, *, backend="cuda", dtype="bfloat16", live=4, blocks=64, tokens=None, **kw):
    from oxide_tech_llm_engine_b200.config import EngineConfig
    from oxide_tech_llm_engine_b200.engine.engine import LLMEngine

    base = dict(backend=backend, dtype=dtype, max_num_seqs=live, num_kv_blocks=blocks, ctx_size=blocks * 16,
                max_num_batched_tokens=tokens or blocks * 16, graph_buckets=(1, 2, 4, 8), enable_radix=False)
    base.update(kw)
    return LLMEngine(EngineConfig(**base), weights=DictSource(cfg, w))


def error(got, want):
    """Largest row error: rms of the difference (mean taken off) over the rms of the reference logits."""
    got, want = np.asarray(got, dtype=np.float64), np.asarray(want, dtype=np.float64)
    d = got - want
    d = d - d.mean(-1, keepdims=True)
    scale = np.sqrt(((want - want.mean(-1, keepdims=True)) ** 2).mean())
    return float((np.sqrt((d ** 2).mean(-1)) / scale).max())


def feed_all(eng, rid, tokens, cuts):
    """Feeds one request in portions of the given sizes (the last one takes the rest); all logits."""
    out, at = [], 0
    cuts = list(cuts)
    while at < len(tokens):
        n = min(cuts.pop(0) if cuts else len(tokens) - at, len(tokens) - at)
        out.append(eng.feed([(rid, tokens[at:at + n], list(range(n)))]))
        at += n
    eng.cancel(rid)
    return np.concatenate(out)


def interleaved(eng, seqs, seed):
    """Runs several requests at once in random portions (single tokens beside chunks, some left out of a
    step, as many live as the engine has slots); returns the logits of every token of each."""
    rng = np.random.default_rng(seed)
    live, waiting = [], list(range(len(seqs)))
    at, out = [0] * len(seqs), [[] for _ in seqs]
    while live or waiting:
        while waiting and len(live) < eng.cfg.max_num_seqs:
            live.append(waiting.pop(0))
        pick = [r for r in live if rng.random() < 0.8] or live[:1]
        entries = []
        for r in pick:
            n = int(rng.choice([1, 1, 1, 2, 3, 16, 17, 40, 64, 65]))
            n = min(n, len(seqs[r]) - at[r])
            entries.append((r, seqs[r][at[r]:at[r] + n], list(range(n))))
        rows = eng.feed(entries)
        k = 0
        for r, toks, _ in entries:
            out[r].append(rows[k:k + len(toks)])
            k += len(toks)
            at[r] += len(toks)
            if at[r] == len(seqs[r]):
                eng.cancel(r)
                live.remove(r)
    return [np.concatenate(o) for o in out]
