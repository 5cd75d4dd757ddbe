"""Plain, slow implementation of the layer-list decoders (the Kipolix design): one function per
mechanism, float64 on the CPU, written from the equations. It shares no code with the product path
and is what the tests compare the engine with.

`cfg` is the model's own configuration dictionary, `w` maps tensor names to float tensors. A
sequence is always computed whole and token by token where the mechanism is recurrent: there is no
cache, page, chunk or batch here that could hide a fault of the engine's.
"""
from __future__ import annotations

import math

import torch

F64 = torch.float64


def rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last dimension."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm_around_zero(x, w, eps):
    """RMS norm whose stored weight is the distance from one."""
    return rms(x, eps) * (1.0 + w)


def silu(z):
    return z / (1.0 + torch.exp(-z))


def rotate(x, pos, base, dims, interleaved):
    """Rotary positions on the first `dims` dimensions of x [T, heads, D]; pairs are (2i, 2i+1) when
    `interleaved`, else (i, i + dims/2)."""
    out = x.clone()
    half = dims // 2
    for i in range(half):
        a = pos.to(x.dtype) * float(base) ** (-2.0 * i / dims)
        c, s = torch.cos(a)[:, None], torch.sin(a)[:, None]
        iu, iv = (2 * i, 2 * i + 1) if interleaved else (i, i + half)
        u, v = x[:, :, iu], x[:, :, iv]
        out[:, :, iu] = u * c - v * s
        out[:, :, iv] = v * c + u * s
    return out


def visible(i, j, size, keep_first):
    """Whether position i attends to position j: its window of `size` positions, and the first ones."""
    return j <= i and (i - j < size or j < keep_first)


def attention(q, k, v, scale, size, keep_first):
    """q [T, H, D], k [T, G, D], v [T, G, E] -> [T, H, E]; ordinary softmax over the visible keys."""
    T, H, _ = q.shape
    G = k.shape[1]
    kk, vv = k.repeat_interleave(H // G, 1), v.repeat_interleave(H // G, 1)
    s = torch.einsum("ihd,jhd->hij", q, kk) * scale
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    see = (j <= i) & ((i - j < size) | (j < keep_first))
    s = s.masked_fill(~see[None], -math.inf)
    return torch.einsum("hij,jhe->ihe", torch.softmax(s, -1), vv)


def retention(q, k, v, decay, state=None):
    """S <- decay_h S + k v^T;  o = S^T q, token by token. q, k [T, H, D], v [T, H, E]."""
    T, H, D = q.shape
    S = torch.zeros(H, D, v.shape[-1], dtype=q.dtype) if state is None else state.clone()
    g = torch.as_tensor(decay, dtype=q.dtype)[:, None, None]
    out = []
    for t in range(T):
        S = g * S + k[t][:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hde,hd->he", S, q[t]))
    return torch.stack(out), S


def mixer_attention(m, w, p, h, pos, eps):
    T = h.shape[0]
    H, G, D, E = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms(h @ w[p + "q"].T, eps) * w[p + "q.norm"]
    k = rms(h @ w[p + "k"].T, eps) * w[p + "k.norm"]
    v = (h @ w[p + "v"].T).view(T, G, E)
    q, k = q.view(T, H, D), k.view(T, G, D)
    q = rotate(q, pos, m["rot"]["base"], m["rot"]["dims"], True)
    k = rotate(k, pos, m["rot"]["base"], m["rot"]["dims"], True)
    o = attention(q, k, v, m["scale"], m["mask"]["size"], m["mask"]["keep_first"])
    return o.reshape(T, H * E) @ w[p + "o"].T


def mixer_retention(m, w, p, h, pos, eps):
    T = h.shape[0]
    H, D, E = m["heads"], m["dim"], m["vdim"]
    q, k = (h @ w[p + "q"].T).view(T, H, D), (h @ w[p + "k"].T).view(T, H, D)
    v = (h @ w[p + "v"].T).view(T, H, E)
    q = rotate(q, pos, m["rot"]["base"], m["rot"]["dims"], False)
    k = rotate(k, pos, m["rot"]["base"], m["rot"]["dims"], False) * D ** -0.5
    o, _ = retention(q, k, v, m["decay"])
    o = rms(o, eps).reshape(T, H * E)
    return (o * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


def feed_forward(w, p, h):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def embedding(cfg, w, tokens):
    x = w["embed"][torch.as_tensor(tokens)]
    bg = cfg["embedding"].get("bigram")
    if bg:
        for t, tok in enumerate(tokens):
            row = bg["buckets"] if t == 0 else (tokens[t - 1] * bg["mul_prev"] + tok * bg["mul_cur"]) % bg["buckets"]
            x[t] = x[t] + w["bigram"][row]
    return x


def layer_runs(cfg):
    """Layer indices in the order they run."""
    n, lp = len(cfg["layers"]), cfg.get("loop")
    if not lp:
        return list(range(n))
    a, b = lp["start"], lp["stop"]
    return list(range(a)) + list(range(a, b)) * lp["times"] + list(range(b, n))


MIXERS = {"attention": mixer_attention, "retention": mixer_retention}


def sublayer(xs, w, p, q, norm_w, eps, fn):
    """One hyper-connected sublayer over the streams xs [s, T, d]."""
    cin, out, mix = w[f"{p}hc{q}.in"], w[f"{p}hc{q}.out"], w[f"{p}hc{q}.mix"]
    u = torch.einsum("s,std->td", cin, xs)
    y = fn(norm_around_zero(u, norm_w, eps))
    return torch.einsum("sz,std->ztd", mix, xs) + out[:, None, None] * y[None]


def forward(cfg, w, tokens, want_layers=False, mixers=MIXERS):
    """Logits [T, vocab] of one whole sequence (and the summed streams after every layer run)."""
    w = {k: torch.as_tensor(v).to(F64) for k, v in w.items()}
    tokens = [int(t) for t in tokens]
    eps = cfg["norm"]["eps"]
    pos = torch.arange(len(tokens))
    x = embedding(cfg, w, tokens)
    xs = torch.stack([x] * cfg["streams"])
    seen = []
    for li in layer_runs(cfg):
        L, p = cfg["layers"][li], f"l{li}."
        xs = sublayer(xs, w, p, 1, w[p + "norm1"], eps,
                      lambda h: mixers[L["type"]](L["mixer"], w, p + "mix.", h, pos, eps))
        if L["mlp"] is not None:
            xs = sublayer(xs, w, p, 2, w[p + "norm2"], eps, lambda h: feed_forward(w, p + "mlp.", h))
        seen.append(xs.sum(0))
    logits = norm_around_zero(xs.sum(0), w["final.norm"], eps) @ w["head"].T
    return (logits, torch.stack(seen)) if want_layers else logits
