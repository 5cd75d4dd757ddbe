"""Plain, slow implementation of the Zagolix design: one function per mechanism, float64 on the CPU, written from
the equations. It shares no code with the product path and is what the tests compare the engine with. A sequence
is always computed whole, and token by token where the mechanism is recurrent: no cache, page, chunk or batch of
the engine's could hide a fault here.

`cfg` is the model's own configuration dictionary, `w` maps tensor names to float tensors.
"""
from __future__ import annotations

import math

import torch

from hybrid_oracle import F64, rms, silu


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


# ---------------------------------------------------------------- matrix memory
def log_gates(zi, zf, cap):
    """Capped pre-activations -> log input gate and log forget gate."""
    i, f = cap * torch.tanh(zi / cap), cap * torch.tanh(zf / cap)
    return i, -torch.log1p(torch.exp(-f))


def mlstm(q, k, v, i, f):
    """q, k [T, H, D], v [T, H, E], log gates [T, H]: decaying sums of k v^T and of k under a running maximum m, which
    starts at 0. Returns the read-outs and the last (S, n, m)."""
    T, H, D = q.shape
    S, n, m = torch.zeros(H, D, v.shape[2], dtype=q.dtype), torch.zeros(H, D, dtype=q.dtype), torch.zeros(H, dtype=q.dtype)
    out = torch.zeros_like(v)
    for t in range(T):
        new = torch.maximum(f[t] + m, i[t])
        a, b = torch.exp(f[t] + m - new), torch.exp(i[t] - new)
        m = new
        S = a[:, None, None] * S + b[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = a[:, None] * n + b[:, None] * k[t]
        den = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        out[t] = torch.einsum("hde,hd->he", S, q[t]) / den[:, None]
    return out, (S, n, m)


def mix_mlstm(c, w, p, h, pos, eps, latents, layer):
    T, (H, D, E) = h.shape[0], (c["heads"], c["dim"], c["vdim"])
    q = (h @ w[p + "q"].T).view(T, H, D) * D ** -0.5
    k, v = (h @ w[p + "k"].T).view(T, H, D), (h @ w[p + "v"].T).view(T, H, E)
    i, f = log_gates(h @ w[p + "i"].T + w[p + "i.b"], h @ w[p + "f"].T + w[p + "f.b"], c["gate_cap"])
    o, _ = mlstm(q, k, v, i, f)
    o = rms(o, eps).reshape(T, H * E) * w[p + "norm"]
    return (o * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


# ---------------------------------------------------------------- softmax attention
def causal(q, k, v, scale):
    """q [T, H, D], k [T, G, D], v [T, G, E] -> [T, H, E]."""
    T, H, _ = q.shape
    kk, vv = k.repeat_interleave(H // k.shape[1], 1), v.repeat_interleave(H // v.shape[1], 1)
    s = torch.einsum("ihd,jhd->hij", q, kk) * scale
    s = s.masked_fill(torch.ones(T, T).triu(1).bool()[None], -math.inf)
    return torch.einsum("hij,jhe->ihe", torch.softmax(s, -1), vv)


def temperature(pos, coef, every):
    """Factor of a query at each position."""
    return torch.tensor([1.0 + coef * math.log(math.floor((int(x) + 1) / every) + 1) for x in pos], dtype=F64)


def map_weight(lq1, lk1, lq2, lk2, diff):
    return torch.exp((lq1 * lk1).sum()) - torch.exp((lq2 * lk2).sum()) + diff


def differential(q, k, v, scale, lam, diff, eps):
    """q [T, H, 2, D], k [T, G, 2, D], v [T, G, E]: two maps over the same values, the second subtracted."""
    a = [causal(q[:, :, j], k[:, :, j], v, scale) for j in (0, 1)]
    return rms(a[0] - lam * a[1], eps) * (1.0 - diff)


def mix_attention(c, w, p, h, pos, eps, latents, layer):
    T, (H, G, D, E) = h.shape[0], (c["heads"], c["kv_heads"], c["dim"], c["vdim"])
    q, k, v = (h @ w[p + n].T + w[p + n + ".b"] for n in "qkv")
    q, k, v = q.view(T, H, 2, D), k.view(T, G, 2, D), v.view(T, G, E)
    t = c.get("q_temp")
    if t:
        q = q * temperature(pos, t["coef"], t["every"])[:, None, None, None]
    lam = map_weight(*(w[p + n] for n in ("lq1", "lk1", "lq2", "lk2")), c["diff"])
    return differential(q, k, v, c["scale"], lam, c["diff"], eps).reshape(T, H * E) @ w[p + "o"].T


# ---------------------------------------------------------------- latent attention
def rotate_pairs(x, pos, base):
    """x [T, heads, R]: dimensions 2i and 2i + 1 turn by position * base^(-2i / R)."""
    out = x.clone()
    R = x.shape[2]
    for i in range(R // 2):
        a = pos.to(x.dtype) * float(base) ** (-2.0 * i / R)
        c, s = torch.cos(a)[:, None], torch.sin(a)[:, None]
        u, v = x[:, :, 2 * i], x[:, :, 2 * i + 1]
        out[:, :, 2 * i] = u * c - v * s
        out[:, :, 2 * i + 1] = v * c + u * s
    return out


def latent(c, w, p, h, pos, eps):
    """What a layer keeps of a token: the normed latent and the rotated key part that all heads share."""
    r = c["kv_rank"]
    x = h @ w[p + "dkv"].T
    return rms(x[:, :r], eps) * w[p + "dkv.norm"], rotate_pairs(x[:, None, r:], pos, c["rot"]["base"])


def mix_latent(c, w, p, h, pos, eps, latents, layer):
    T, (H, D, R, E) = h.shape[0], (c["heads"], c["dim"], c["rot_dim"], c["vdim"])
    q = ((rms(h @ w[p + "dq"].T, eps) * w[p + "dq.norm"]) @ w[p + "uq"].T).view(T, H, D + R)
    q = torch.cat([q[:, :, :D], rotate_pairs(q[:, :, D:], pos, c["rot"]["base"])], -1)
    if "kv_from" not in c:
        latents[layer] = latent(c, w, p, h, pos, eps)
    z, kr = latents[c.get("kv_from", layer)]
    k = torch.cat([(z @ w[p + "uk"].T).view(T, H, D), kr.expand(T, H, R)], -1)
    return causal(q, k, (z @ w[p + "uv"].T).view(T, H, E), c["scale"]).reshape(T, H * E) @ w[p + "o"].T


MIXERS = {"mlstm": mix_mlstm, "attention": mix_attention, "latent_attention": mix_latent}


# ---------------------------------------------------------------- feed-forward
def dense(w, p, h):
    return (gelu_tanh(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def choose(logits, top, groups=None):
    """Sigmoid scores; the best `keep` of `count` equal groups of neighbours (by the sum of a group's two largest
    scores), then the `top` largest scores among them: [T, top] ids and their scores."""
    s = sigmoid(logits)
    if groups:
        g = s.view(len(s), groups["count"], -1)
        rank = torch.argsort(torch.sort(g, -1, descending=True).values[..., :2].sum(-1), dim=-1, descending=True, stable=True)
        keep = torch.zeros(g.shape[:2], dtype=torch.bool).scatter_(1, rank[:, :groups["keep"]], True)
        open_ = keep.repeat_interleave(g.shape[2], 1)
    else:
        open_ = torch.ones_like(s, dtype=torch.bool)
    ids = torch.argsort(torch.where(open_, s, torch.full_like(s, -1.0)), dim=-1, descending=True, stable=True)[:, :top]
    return ids, s.gather(1, ids)


def margin(logits, top, groups=None):
    """How clear the choice of each token is: the smaller gap of the groups' and the experts' choice, in scores."""
    s = sigmoid(logits)
    gap = torch.full((len(s),), math.inf, dtype=s.dtype)
    if groups and groups["keep"] < groups["count"]:
        t = torch.sort(torch.sort(s.view(len(s), groups["count"], -1), -1, descending=True).values[..., :2].sum(-1), -1, descending=True).values
        gap = t[:, groups["keep"] - 1] - t[:, groups["keep"]]
    ids, v = choose(logits, top, groups)
    n_open = s.shape[1] if not groups else s.shape[1] // groups["count"] * groups["keep"]
    if n_open > top:
        more = choose(logits, top + 1, groups)[1]
        gap = torch.minimum(gap, more[:, top - 1] - more[:, top])
    return gap


def experts(c, w, p, h, margins=None):
    lg, r = h @ w[p + "router"].T, c["router"]
    if margins is not None:
        margins.append(margin(lg, r["top"], r.get("groups")))
    ids, wt = choose(lg, r["top"], r.get("groups"))
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, a in zip(ids[t].tolist(), wt[t]):
            q = f"{p}e{e}."
            out[t] += a * (w[q + "down"] @ (silu(w[q + "gate"] @ h[t]) * (w[q + "up"] @ h[t])))
    return out


# ---------------------------------------------------------------- model
def forward(cfg, w, tokens, want_layers=False, margins=None):
    """Logits [T, vocab] of one whole sequence (and the residual stream after every layer). `margins`: a list that takes
    the tokens' margins of every router."""
    w = {k: torch.as_tensor(v).to(F64) for k, v in w.items()}
    eps = cfg["norm"]["eps"]
    pos = torch.arange(len(tokens))
    x = w["embed"][torch.as_tensor([int(t) for t in tokens])] * cfg["embedding"]["scale"]
    seen, latents = [], {}
    for i, L in enumerate(cfg["layers"]):
        p = f"l{i}."
        y = MIXERS[L["type"]](L["mixer"], w, p + "mix.", rms(x, eps) * w[p + "norm1"], pos, eps, latents, i)
        x = x + rms(y, eps) * w[p + "norm1b"] * w[p + "ls1"]
        if L["mlp"] is not None:
            h = rms(x, eps) * w[p + "norm2"]
            y = dense(w, p + "mlp.", h) if L["mlp"]["kind"] == "dense" else experts(L["mlp"], w, p + "mlp.", h, margins)
            x = x + rms(y, eps) * w[p + "norm2b"] * w[p + "ls2"]
        seen.append(x)
    logits = rms(x, eps) * w["final.norm"] @ w["embed"].T
    return (logits, torch.stack(seen)) if want_layers else logits
