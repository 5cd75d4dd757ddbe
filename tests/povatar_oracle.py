"""Plain, slow implementation of the Povatar design: one function per mechanism, float64 on the CPU,
written from the equations. It shares no code with the product path and is what the tests compare the
engine with. A sequence is always computed whole, and token by token where the mechanism is recurrent:
no cache, page, chunk or batch of the engine's could hide a fault here.

`cfg` is the model's own configuration dictionary, `w` maps tensor names to float tensors.
"""
from __future__ import annotations

import math

import torch

from hybrid_oracle import F64, rms, silu


# ---------------------------------------------------------------- rotation
def yarn_frequencies(base, dims, scaling=None):
    """Frequencies of the dims/2 rotation pairs and the factor on cos and sin. With `scaling`, slowly turning
    pairs are slowed down by `factor`, fast ones stay, and a ramp over the pair index lies between."""
    f = [float(base) ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not scaling:
        return torch.tensor(f, dtype=F64), 1.0

    def turns(t):
        return dims * math.log(scaling["original"] / (2.0 * math.pi * t)) / (2.0 * math.log(base))

    lo = max(math.floor(turns(scaling["fast"])), 0)
    hi = min(math.ceil(turns(scaling["slow"])), dims - 1)
    out = []
    for i, x in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(x / scaling["factor"] * ramp + x * (1.0 - ramp))
    return torch.tensor(out, dtype=F64), 0.1 * math.log(scaling["factor"]) + 1.0


def rotate_half(x, pos, freqs, gain):
    """x [T, heads, D]: dimension i turns with dimension i + len(freqs); both cos and sin carry `gain`."""
    out = x.clone()
    n = len(freqs)
    for i in range(n):
        a = pos.to(x.dtype) * freqs[i]
        c, s = (gain * torch.cos(a))[:, None], (gain * torch.sin(a))[:, None]
        u, v = x[:, :, i], x[:, :, i + n]
        out[:, :, i] = u * c - v * s
        out[:, :, i + n] = v * c + u * s
    return out


# ---------------------------------------------------------------- attention
def same_chunk(i, j, size):
    """Whether position i attends to position j: both in one chunk counted from the sequence's start."""
    return j <= i and (not size or i // size == j // size)


def chunk_attention(q, k, v, scale, size, sink=True):
    """q [T, H, D], k [T, G, D], v [T, G, E] -> [T, H, E]; the softmax has 1 added to its denominator."""
    T, H, _ = q.shape
    G = k.shape[1]
    kk, vv = k.repeat_interleave(H // G, 1), v.repeat_interleave(H // G, 1)
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for i in range(T):
        see = torch.tensor([same_chunk(i, j, size) for j in range(i + 1)])
        s = torch.einsum("hd,jhd->hj", q[i], kk[:i + 1][see]) * scale
        m = torch.clamp(s.max(-1, keepdim=True).values, min=0.0)      # the sink's score is 0
        e = torch.exp(s - m)
        p = e / (e.sum(-1, keepdim=True) + (torch.exp(-m) if sink else 0.0))
        out[i] = torch.einsum("hj,jhe->he", p, vv[:i + 1][see])
    return out


def left_mixer(c, w, p, h, pos):
    T, (H, G, D, E) = h.shape[0], (c["heads"], c["kv_heads"], c["dim"], c["vdim"])
    q, k = (h @ w[p + "q"].T).view(T, H, D), (h @ w[p + "k"].T).view(T, G, D)
    v = (h @ w[p + "v"].T).view(T, G, E)
    rot = c.get("rot")
    if rot:
        f, gain = yarn_frequencies(rot["base"], rot["dims"], rot.get("scaling"))
        q, k = rotate_half(q, pos, f, gain), rotate_half(k, pos, f, gain)
    o = chunk_attention(q, k, v, c["scale"], (c.get("mask") or {}).get("size", 0))
    return o.reshape(T, H * E) @ w[p + "o"].T


# ---------------------------------------------------------------- state-space duality
def short_conv(u, w, b):
    """Causal convolution per channel: u [T, ch], w [ch, taps] (last column: the current token), b [ch]."""
    T, taps = u.shape[0], w.shape[1]
    out = torch.zeros_like(u)
    for t in range(T):
        acc = b.clone()
        for j in range(taps):
            s = t - (taps - 1) + j
            if s >= 0:
                acc = acc + w[:, j] * u[s]
        out[t] = acc
    return out


def softplus(z):
    return torch.clamp(z, min=0.0) + torch.log1p(torch.exp(-z.abs()))


def ssd(x, B, C, dt, A_log, D, state=None):
    """x [T, H, E], B and C [T, G, N], dt [T, H] (after softplus): S <- exp(-exp(A_log) dt) S + dt B x^T,
    y = S^T C + D x, token by token; returns y and the last state [H, N, E]."""
    T, H, E = x.shape
    G, N = B.shape[1:]
    S = torch.zeros(H, N, E, dtype=x.dtype) if state is None else state.clone()
    y = torch.zeros_like(x)
    Bh, Ch = B.repeat_interleave(H // G, 1), C.repeat_interleave(H // G, 1)     # head h uses group h // (H / G)
    for t in range(T):
        a = torch.exp(-torch.exp(A_log) * dt[t])
        S = a[:, None, None] * S + (dt[t][:, None] * Bh[t])[:, :, None] * x[t][:, None, :]
        y[t] = torch.einsum("hne,hn->he", S, Ch[t]) + D[:, None] * x[t]
    return y, S


def gated_group_norm(y, z, w, groups, eps):
    """(y silu(z)) normalised in `groups` equal parts, each by its own root mean square, times w."""
    u = y * silu(z)
    return rms(u.view(u.shape[0], groups, -1), eps).reshape(u.shape) * w


def right_mixer(c, w, p, h, eps):
    T, (H, G, N, E) = h.shape[0], (c["heads"], c["groups"], c["state"], c["vdim"])
    inner = H * E
    proj = h @ w[p + "in"].T
    z, xbc, dt = proj[:, :inner], proj[:, inner:2 * inner + 2 * G * N], proj[:, 2 * inner + 2 * G * N:]
    u = silu(short_conv(xbc, w[p + "conv"], w[p + "conv.b"]))
    x, B, C = u[:, :inner].view(T, H, E), u[:, inner:inner + G * N].view(T, G, N), u[:, inner + G * N:].view(T, G, N)
    y, _ = ssd(x, B, C, softplus(dt + w[p + "dt_bias"]), w[p + "A_log"], w[p + "D"])
    return gated_group_norm(y.reshape(T, inner), z, w[p + "norm"], c["norm_groups"], eps) @ w[p + "o"].T


# ---------------------------------------------------------------- mixture of experts
def choose(logits, top):
    """Softmax over all experts, the `top` largest scores, divided by their sum: [T, top] ids and weights."""
    s = torch.softmax(logits, -1)
    ids = torch.argsort(s, dim=-1, descending=True, stable=True)[:, :top]
    v = s.gather(1, ids)
    return ids, v / (v.sum(-1, keepdim=True) + 1e-20)


def relu_squared(z):
    return torch.clamp(z, min=0.0) ** 2


def margin(logits, top):
    """How clear the choice of a token is: gap between the last chosen and the next logit, in their standard deviation."""
    s = torch.sort(logits, -1, descending=True).values
    return (s[:, top - 1] - s[:, top]) / logits.std() if s.shape[1] > top else torch.full((len(s),), math.inf, dtype=s.dtype)


def experts(c, w, p, h, margins=None):
    lg, top = h @ w[p + "router"].T, c["router"]["top"]
    if margins is not None:
        margins.append(margin(lg, top))
    ids, wt = choose(lg, top)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, a in zip(ids[t].tolist(), wt[t]):
            out[t] += a * (w[f"{p}e{e}.down"] @ relu_squared(w[f"{p}e{e}.up"] @ h[t]))
    return out


# ---------------------------------------------------------------- model
def forward(cfg, w, tokens, want_layers=False, margins=None):
    """Logits [T, vocab] of one whole sequence (and the residual stream after every layer). `margins`: a list that takes
    the tokens' margins of every router."""
    w = {k: torch.as_tensor(v).to(F64) for k, v in w.items()}
    eps = cfg["norm"]["eps"]
    pos = torch.arange(len(tokens))
    x = w["embed"][torch.as_tensor([int(t) for t in tokens])] * cfg["embedding"]["scale"]
    seen = []
    for i, L in enumerate(cfg["layers"]):
        p = f"l{i}."
        h = rms(x, eps) * w[p + "norm1"]
        a = left_mixer(L["mixer"]["left"], w, p + "mix.left.", h, pos)
        b = right_mixer(L["mixer"]["right"], w, p + "mix.right.", h, eps)
        y = 0.5 * (rms(a, eps) * w[p + "mix.left.out"] + rms(b, eps) * w[p + "mix.right.out"])
        if L["mlp"] is not None:
            y = y + experts(L["mlp"], w, p + "mlp.", rms(x, eps) * w[p + "norm2"], margins)
        x = x + y
        seen.append(x)
    logits = rms(x, eps) * w["final.norm"] @ w["head"].T
    return (logits, torch.stack(seen)) if want_layers else logits
