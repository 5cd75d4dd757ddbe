"""Plain, slow implementation of the Vokepel design: one function per mechanism, float64 on the CPU, written from
the equations. It shares no code with the product path and is what the tests compare the engine with. A sequence
is always computed whole, and token by token where the mechanism is recurrent: no cache, page, chunk or batch of
the engine's could hide a fault here.

`cfg` is the model's own configuration dictionary, `w` maps tensor names to float tensors.
"""
from __future__ import annotations

import math

import torch

from hybrid_oracle import F64, layer_runs, rms, rotate, silu


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


# ---------------------------------------------------------------- scores
def raw_scores(q, k, scale):
    """q [T, H, D], k [T, G, D] -> [H, T, T], query first."""
    return torch.einsum("ihd,jhd->hij", q, k.repeat_interleave(q.shape[1] // k.shape[1], 1)) * scale


def cap(s, limit):
    return limit * torch.tanh(s / limit)


def distance_bias(T, r1, r2):
    """What a head takes off the score of a key: [H, T, T], 0 where the key comes after the query."""
    d = (torch.arange(T)[:, None] - torch.arange(T)[None, :]).clamp(min=0).to(r1.dtype)
    return r1[:, None, None] * torch.log(1.0 + r2[:, None, None] * d)


def talk(s, t):
    """Scores of every head as a sum over those of all heads."""
    return torch.einsum("hg,gij->hij", t, s)


def masked_softmax(s, size, sink=None):
    """Softmax over the last `size` positions up to the query's own; `sink` [H]: one more term of the denominator."""
    T = s.shape[1]
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    s = s.masked_fill(~((j <= i) & (i - j < size))[None], -math.inf)
    if sink is None:
        return torch.softmax(s, -1)
    return torch.softmax(torch.cat([s, sink[:, None, None].expand(-1, T, 1)], -1), -1)[..., :T]


def values_of(p, v):
    """p [H, T, T], v [T, G, E] -> [T, H, E]."""
    return torch.einsum("hij,jhe->ihe", p, v.repeat_interleave(p.shape[0] // v.shape[1], 1))


# ---------------------------------------------------------------- mixers
def mix_attention(c, w, p, h, pos, eps):
    """Talking heads over one projection that is both key (normed) and value (as it is), with an output gate."""
    T, (H, G, D) = h.shape[0], (c["heads"], c["kv_heads"], c["dim"])
    q, k = h @ w[p + "q"].T, h @ w[p + "k"].T
    v = k.view(T, G, D)
    q, k = (rms(q, eps) * w[p + "q.norm"]).view(T, H, D), (rms(k, eps) * w[p + "k.norm"]).view(T, G, D)
    s = cap(raw_scores(q, k, c["scale"]), c["softcap"]) - distance_bias(T, w[p + "r1"], w[p + "r2"])
    a = values_of(masked_softmax(talk(s, w[p + "talk"]), c["mask"]["size"]), v).reshape(T, H * D)
    return (a * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def mix_sink(c, w, p, h, pos, eps):
    """Rotated grouped attention with a learned sink per head."""
    T, (H, G, D, E) = h.shape[0], (c["heads"], c["kv_heads"], c["dim"], c["vdim"])
    q, k, v = (h @ w[p + "q"].T).view(T, H, D), (h @ w[p + "k"].T).view(T, G, D), (h @ w[p + "v"].T).view(T, G, E)
    if c.get("rot"):
        q, k = (rotate(x, pos, c["rot"]["base"], c["rot"]["dims"], True) for x in (q, k))
    a = values_of(masked_softmax(raw_scores(q, k, c["scale"]), c["mask"]["size"], w[p + "sink"]), v)
    return a.reshape(T, H * E) @ w[p + "o"].T


def candidate(u):
    return torch.where(u >= 0, u + 0.5, sigmoid(u))


def gru(z, c, state=None):
    """S <- (1 - z) S + z c, element by element; z, c [T, N]. Returns all states."""
    S = torch.zeros_like(c[0]) if state is None else state
    out = []
    for t in range(len(c)):
        S = (1.0 - z[t]) * S + z[t] * c[t]
        out.append(S)
    return torch.stack(out)


def mix_gru(c, w, p, h, pos, eps):
    z, u = sigmoid(h @ w[p + "z"].T + w[p + "z.b"]), h @ w[p + "x"].T + w[p + "x.b"]
    return (gru(z, candidate(u)) * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


def mix_parallel(c, w, p, h, pos, eps):
    return (c["left_scale"] * mix_sink(c["left"], w, p + "left.", h, pos, eps)
            + c["right_scale"] * mix_gru(c["right"], w, p + "right.", h, pos, eps))


MIXERS = {"attention": mix_attention, "parallel": mix_parallel}


def feed_forward(w, p, h):
    return torch.relu(h @ w[p + "up"].T).square() @ w[p + "down"].T


# ---------------------------------------------------------------- model
def enter_pass(x, x0, w, t):
    """What happens to the stream before pass t of the loop."""
    return torch.cat([x, x0], -1) @ w["loop.in"].T + w["loop.step"][t]


def pass_starts(cfg):
    """Pass number by index of the layer run that it begins with."""
    lp = cfg.get("loop")
    return {lp["start"] + t * (lp["stop"] - lp["start"]): t for t in range(lp["times"])} if lp else {}


def forward(cfg, w, tokens, want_layers=False):
    """Logits [T, vocab] of one whole sequence (and the residual stream after every layer run)."""
    w = {k: torch.as_tensor(v).to(F64) for k, v in w.items()}
    eps, m = cfg["norm"]["eps"], cfg["residual_mult"]
    pos = torch.arange(len(tokens))
    x = x0 = w["embed"][torch.as_tensor([int(t) for t in tokens])]
    seen, starts = [], pass_starts(cfg)
    for run, li in enumerate(layer_runs(cfg)):
        L, p = cfg["layers"][li], f"l{li}."
        if run in starts:
            x = enter_pass(x, x0, w, starts[run])
        x = x + m * MIXERS[L["type"]](L["mixer"], w, p + "mix.", rms(x, eps) * w[p + "norm1"], pos, eps)
        if L["mlp"] is not None:
            x = x + m * feed_forward(w, p + "mlp.", rms(x, eps) * w[p + "norm2"])
        seen.append(x)
    logits = cap((rms(x, eps) * w["final.norm"]) @ w["embed"].T * cfg["logit_scale"], cfg["logit_softcap"])
    return (logits, torch.stack(seen)) if want_layers else logits
