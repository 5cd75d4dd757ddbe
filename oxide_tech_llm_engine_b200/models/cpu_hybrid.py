"""CPU backend of layer-list decoders: the same step plans, paged KV blocks and state slots as the device
model, in fp32 torch ops, so the scheduler, slot manager, server and command line run without a GPU.
"""
from __future__ import annotations

from typing import Optional

import numpy as np
import torch

from .config import ModelConfig
from .weights import WeightSource, tensor_names


class CpuHybridModel:
    supports_kv_tiers = False
    supports_block_mass = False

    def __init__(self, cfg: ModelConfig, src: WeightSource, num_blocks: int, state_slots: int = 0):
        self.cfg, self.num_blocks = cfg, num_blocks
        self.w = {n: torch.from_numpy(np.ascontiguousarray(src.f32(n), dtype=np.float32)) for n, _ in tensor_names(cfg)}
        self.embed = self.w["embed"]
        self.head = self.w["embed" if cfg.tie_embeddings else "head"]
        self.runs = []
        self.pk, self.pv, self.states = [], [], []
        for li in cfg.layer_runs:
            at = []      # index of the cache or state of every mixer of the layer
            for mx in cfg.layers[li].mixer.parts:
                if mx.kind == "attention":
                    at.append(len(self.pk))
                    self.pk.append(torch.zeros(num_blocks, mx.kv_heads, 16, mx.maps * mx.dim))
                    self.pv.append(torch.zeros(num_blocks, mx.kv_heads, 16, mx.vdim))
                elif mx.kind == "latent_attention":   # the latents, and the rotated key parts of all heads
                    if mx.kv_from is not None:
                        at.append(self.runs[mx.kv_from][1][0])
                        continue
                    at.append(len(self.pk))
                    self.pk.append(torch.zeros(num_blocks, 1, 16, mx.rot_dim))
                    self.pv.append(torch.zeros(num_blocks, 1, 16, mx.kv_rank))
                elif mx.kind == "talking_attention":   # keys before their norm, which are the values, and the norm's factor
                    at.append(len(self.pk))
                    self.pk.append(torch.zeros(num_blocks, mx.kv_heads, 16, mx.dim))
                    self.pv.append(torch.zeros(num_blocks, 1, 16, 1))
                elif mx.kind == "min_gru":
                    at.append(len(self.states))
                    self.states.append(torch.zeros(state_slots, mx.width))
                elif mx.kind == "mlstm":   # memory, normaliser, running maximum
                    at.append(len(self.states))
                    self.states.append((torch.zeros(state_slots, mx.heads, mx.dim, mx.vdim), torch.zeros(state_slots, mx.heads, mx.dim),
                                        torch.zeros(state_slots, mx.heads)))
                elif mx.kind == "ssd":   # state, and the last inputs of the convolution, the newest last
                    at.append(len(self.states))
                    self.states.append((torch.zeros(state_slots, mx.heads, mx.state, mx.vdim),
                                        torch.zeros(state_slots, mx.taps - 1, mx.inner + 2 * mx.groups * mx.state)))
                else:
                    at.append(len(self.states))
                    self.states.append(torch.zeros(state_slots, mx.heads, mx.dim, mx.vdim))
            self.runs.append((li, at))
        self.logits: Optional[torch.Tensor] = None

    def copy_blocks(self, src, dst) -> None:
        s, d = torch.as_tensor(np.asarray(src, dtype=np.int64)), torch.as_tensor(np.asarray(dst, dtype=np.int64))
        for c in (*self.pk, *self.pv):
            c[d] = c[s]

    # ------------------------------------------------------------------ pieces
    def _unit(self, x: torch.Tensor) -> torch.Tensor:
        return x * torch.rsqrt(x.pow(2).mean(-1, keepdim=True) + self.cfg.rms_eps)

    @staticmethod
    def _rotate(x: torch.Tensor, pos: torch.Tensor, rot) -> torch.Tensor:
        if rot is None:
            return x
        half = rot.dims // 2
        f, gain = rot.frequencies()
        ang = pos.double()[:, None] * torch.tensor(f, dtype=torch.float64)[None]
        cs, sn = (gain * torch.cos(ang)).float()[:, None], (gain * torch.sin(ang)).float()[:, None]
        head, rest = x[..., :rot.dims], x[..., rot.dims:]
        if rot.interleaved:
            u, v = head[..., 0::2], head[..., 1::2]
            out = torch.stack([u * cs - v * sn, v * cs + u * sn], -1).flatten(-2)
        else:
            u, v = head[..., :half], head[..., half:]
            out = torch.cat([u * cs - v * sn, v * cs + u * sn], -1)
        return torch.cat([out, rest], -1)

    def _attention(self, a, p: str, ci: int, h, pos, seqs, blk, off):
        T, w, n2 = h.shape[0], self.w, a.maps
        q, k, v = (h @ w[p + n].T + (w[f"{p}{n}.b"] if a.bias else 0.0) for n in ("q", "k", "v"))
        if a.qk_norm == "projection":
            q, k = self._unit(q) * w[p + "q.norm"], self._unit(k) * w[p + "k.norm"]
        q = self._rotate(q.view(T, a.heads * n2, a.dim), pos, a.rot)
        if a.temp_coef:
            q = q * (1.0 + a.temp_coef * torch.log(torch.floor((pos + 1) / a.temp_every) + 1.0))[:, None, None]
        self.pk[ci][blk, :, off] = self._rotate(k.view(T, a.kv_heads * n2, a.dim), pos, a.rot).reshape(T, a.kv_heads, n2 * a.dim)
        self.pv[ci][blk, :, off] = v.view(T, a.kv_heads, a.vdim)
        out = torch.zeros(T, a.heads * n2, a.vdim)
        for r0, n, ctx, table, _ in seqs:
            keys = self._pages(self.pk[ci], table, ctx).reshape(ctx, a.kv_heads, n2, a.dim)
            values = self._pages(self.pv[ci], table, ctx)
            g = a.heads // a.kv_heads
            keys = keys.repeat_interleave(g, 1).reshape(ctx, a.heads * n2, a.dim)
            i = torch.arange(ctx - n, ctx)[:, None]
            j = torch.arange(ctx)[None]
            see = j <= i
            if a.window:
                see = see & ((i - j < a.window) | (j < a.keep_first))
            if a.chunk:
                see = see & (i // a.chunk == j // a.chunk)
            s = torch.einsum("ihd,jhd->hij", q[r0:r0 + n], keys) * a.scale
            s = s.masked_fill(~see[None], float("-inf"))
            if a.sink is not None:
                s = torch.cat([s, torch.full_like(s[..., :1], a.sink)], -1)
            if a.sinks:
                s = torch.cat([s, w[p + "sink"][:, None, None].expand(-1, n, 1)], -1)
            out[r0:r0 + n] = torch.einsum("hij,jhe->ihe", torch.softmax(s, -1)[..., :ctx], values.repeat_interleave(g * n2, 1))
        if a.diff is not None:
            lam = torch.exp((w[p + "lq1"] * w[p + "lk1"]).sum()) - torch.exp((w[p + "lq2"] * w[p + "lk2"]).sum()) + a.diff
            two = out.view(T, a.heads, 2, a.vdim)
            out = self._unit(two[:, :, 0] - lam * two[:, :, 1]) * (1.0 - a.diff)
        return out.reshape(T, -1) @ w[p + "o"].T

    @staticmethod
    def _pages(c: torch.Tensor, table, ctx: int) -> torch.Tensor:
        """Cached rows of a sequence in order: [ctx, heads, values]."""
        pages = torch.as_tensor(table[:(ctx + 15) // 16].astype(np.int64))
        return c[pages].permute(0, 2, 1, 3).reshape(-1, c.shape[1], c.shape[3])[:ctx]

    def _latent(self, a, p: str, ci: int, h, pos, seqs, blk, off):
        T, w, H = h.shape[0], self.w, a.heads
        q = ((self._unit(h @ w[p + "dq"].T) * w[p + "dq.norm"]) @ w[p + "uq"].T).view(T, H, a.dim + a.rot_dim)
        qn, qr = q[..., :a.dim], self._rotate(q[..., a.dim:], pos, a.rot)
        if a.kv_from is None:
            kv = h @ w[p + "dkv"].T
            self.pv[ci][blk, :, off] = (self._unit(kv[:, :a.kv_rank]) * w[p + "dkv.norm"])[:, None]
            self.pk[ci][blk, :, off] = self._rotate(kv[:, None, a.kv_rank:], pos, a.rot)
        out = torch.zeros(T, H, a.vdim)
        uk, uv = w[p + "uk"].view(H, a.dim, -1), w[p + "uv"].view(H, a.vdim, -1)
        for r0, n, ctx, table, _ in seqs:
            c, kr = self._pages(self.pv[ci], table, ctx)[:, 0], self._pages(self.pk[ci], table, ctx)[:, 0]
            s = torch.einsum("ihd,hdr,jr->hij", qn[r0:r0 + n], uk, c) + torch.einsum("ihd,jd->hij", qr[r0:r0 + n], kr)
            see = torch.arange(ctx)[None] <= torch.arange(ctx - n, ctx)[:, None]
            pr = torch.softmax((s * a.scale).masked_fill(~see[None], float("-inf")), -1)
            out[r0:r0 + n] = torch.einsum("hij,jr,her->ihe", pr, c, uv)
        return out.reshape(T, -1) @ w[p + "o"].T

    def _memory(self, r, p: str, ci: int, h, seqs):
        T, w, F = h.shape[0], self.w, torch.nn.functional
        q = (h @ w[p + "q"].T).view(T, r.heads, r.dim) * r.dim ** -0.5
        k, v = (h @ w[p + "k"].T).view(T, r.heads, r.dim), (h @ w[p + "v"].T).view(T, r.heads, r.vdim)
        cap = lambda n: r.gate_cap * torch.tanh((h @ w[p + n].T + w[f"{p}{n}.b"]) / r.gate_cap)
        gi, gf = cap("i"), F.logsigmoid(cap("f"))
        out = torch.zeros(T, r.heads, r.vdim)
        for r0, n, ctx, _, slot in seqs:
            S, N, m = (torch.zeros_like(x[slot]) if ctx == n else x[slot] for x in self.states[ci])
            for t in range(r0, r0 + n):
                m2 = torch.maximum(gf[t] + m, gi[t])
                keep, add, m = torch.exp(gf[t] + m - m2), torch.exp(gi[t] - m2), m2
                S = keep[:, None, None] * S + (add[:, None] * k[t])[:, :, None] * v[t][:, None, :]
                N = keep[:, None] * N + add[:, None] * k[t]
                den = torch.maximum((N * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
                out[t] = torch.einsum("hde,hd->he", S, q[t]) / den[:, None]
            for x, y in zip(self.states[ci], (S, N, m)):
                x[slot] = y
        return (self._unit(out).reshape(T, -1) * w[p + "norm"] * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T

    def _retention(self, r, p: str, ci: int, h, pos, seqs):
        T, w = h.shape[0], self.w
        q = self._rotate((h @ w[p + "q"].T).view(T, r.heads, r.dim), pos, r.rot)
        k = self._rotate((h @ w[p + "k"].T).view(T, r.heads, r.dim), pos, r.rot) * r.dim ** -0.5
        v = (h @ w[p + "v"].T).view(T, r.heads, r.vdim)
        gamma = torch.tensor(r.decay, dtype=torch.float32)[:, None, None]
        out = torch.zeros(T, r.heads, r.vdim)
        for r0, n, ctx, _, slot in seqs:
            S = torch.zeros_like(self.states[ci][slot]) if ctx == n else self.states[ci][slot]
            for t in range(r0, r0 + n):
                S = gamma * S + k[t][:, :, None] * v[t][:, None, :]
                out[t] = torch.einsum("hde,hd->he", S, q[t])
            self.states[ci][slot] = S
        gate = torch.nn.functional.silu(h @ w[p + "g"].T)
        return (self._unit(out).reshape(T, -1) * gate) @ w[p + "o"].T

    def _talking(self, a, p: str, ci: int, h, pos, seqs, blk, off):
        T, w, g = h.shape[0], self.w, a.heads // a.kv_heads
        q, k = h @ w[p + "q"].T, h @ w[p + "k"].T
        # the keys' norm weights act on the queries, the norm itself is a number per cached token
        wk = w[p + "k.norm"].view(a.kv_heads, a.dim).repeat_interleave(g, 0)
        q = (self._unit(q) * w[p + "q.norm"]).view(T, a.heads, a.dim) * wk
        self.pk[ci][blk, :, off] = k.view(T, a.kv_heads, a.dim)
        self.pv[ci][blk, 0, off] = torch.rsqrt(k.pow(2).mean(-1, keepdim=True) + self.cfg.rms_eps)
        out = torch.zeros(T, a.heads, a.dim)
        for r0, n, ctx, table, _ in seqs:
            rows = self._pages(self.pk[ci], table, ctx).repeat_interleave(g, 1)
            s = torch.einsum("ihd,jhd->hij", q[r0:r0 + n], rows) * (self._pages(self.pv[ci], table, ctx)[:, 0, 0] * a.scale)
            if a.softcap:
                s = a.softcap * torch.tanh(s / a.softcap)
            i, j = torch.arange(ctx - n, ctx)[:, None], torch.arange(ctx)[None]
            far = (i - j).clamp(min=0)
            s = s - w[p + "r1"][:, None, None] * torch.log1p(w[p + "r2"][:, None, None] * far)
            s = torch.einsum("hg,gij->hij", w[p + "talk"], s)
            see = (j <= i) & ((i - j < a.window) if a.window else True)
            out[r0:r0 + n] = torch.einsum("hij,jhe->ihe", torch.softmax(s.masked_fill(~see[None], float("-inf")), -1), rows)
        return (out.reshape(T, -1) * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T

    def _gru(self, r, p: str, ci: int, h, seqs):
        w = self.w
        z, u = torch.sigmoid(h @ w[p + "z"].T + w[p + "z.b"]), h @ w[p + "x"].T + w[p + "x.b"]
        c = torch.where(u >= 0, u + 0.5, torch.sigmoid(u))
        out = torch.zeros_like(c)
        for r0, n, ctx, _, slot in seqs:
            S = torch.zeros_like(self.states[ci][slot]) if ctx == n else self.states[ci][slot]
            for t in range(r0, r0 + n):
                S = S + z[t] * (c[t] - S)
                out[t] = S
            self.states[ci][slot] = S
        return (out * torch.nn.functional.silu(h @ w[p + "g"].T)) @ w[p + "o"].T

    def _ssd(self, r, p: str, ci: int, h, seqs):
        T, w, F = h.shape[0], self.w, torch.nn.functional
        gn = r.groups * r.state
        z, xbc, dt = (h @ w[p + "in"].T).split([r.inner, r.inner + 2 * gn, r.heads], -1)
        dt = F.softplus(dt + w[p + "dt_bias"], threshold=40.0)
        decay = torch.exp(-torch.exp(w[p + "A_log"]) * dt)
        state, past = self.states[ci]
        y = torch.zeros(T, r.heads, r.vdim)
        per = r.heads // r.groups
        for r0, n, ctx, _, slot in seqs:
            fresh = ctx == n
            rows = torch.cat([torch.zeros_like(past[slot]) if fresh else past[slot], xbc[r0:r0 + n]])
            u = F.silu(F.conv1d(rows.T[None], w[p + "conv"][:, None], w[p + "conv.b"], groups=rows.shape[1])[0].T)
            past[slot] = rows[n:]
            x, b, c = u.split([r.inner, gn, gn], -1)
            x = x.view(n, r.heads, r.vdim)
            b, c = (t.view(n, r.groups, r.state).repeat_interleave(per, 1) for t in (b, c))
            S = torch.zeros_like(state[slot]) if fresh else state[slot]
            for t in range(n):
                g = r0 + t
                S = decay[g][:, None, None] * S + (dt[g][:, None] * b[t])[:, :, None] * x[t][:, None, :]
                y[g] = torch.einsum("hne,hn->he", S, c[t]) + w[p + "D"][:, None] * x[t]
            state[slot] = S
        u = (y.reshape(T, -1) * F.silu(z)).view(T, r.norm_groups, -1)
        return (self._unit(u).reshape(T, -1) * w[p + "norm"]) @ w[p + "o"].T

    def _moe(self, e, p: str, h):
        w, F = self.w, torch.nn.functional
        z = h @ w[p + "router"].T
        s = torch.softmax(z, -1) if e.scores == "softmax" else torch.sigmoid(z)
        open_ = s
        if e.groups:
            best = torch.topk(s.view(len(s), e.groups, -1), min(2, e.experts // e.groups), -1).values.sum(-1)
            kept = torch.zeros_like(best).scatter_(1, torch.topk(best, e.keep, -1).indices, 1.0)
            open_ = torch.where(kept.repeat_interleave(e.experts // e.groups, 1) > 0, s, torch.full_like(s, -1.0))
        v, ids = torch.topk(open_, e.top, -1)
        if e.scores == "softmax":
            v = v / (v.sum(-1, keepdim=True) + 1e-20)
        out = torch.zeros_like(h)
        for i in range(e.experts):
            t, k = torch.nonzero(ids == i, as_tuple=True)
            if t.numel():
                q, x = f"{p}e{i}.", h[t]
                u = x @ w[q + "up"].T
                u = F.silu(x @ w[q + "gate"].T) * u if e.glu else torch.relu(u).square()
                out.index_add_(0, t, v[t, k][:, None] * (u @ w[q + "down"].T))
        return out

    def _dense(self, f, p: str, h):
        w, F = self.w, torch.nn.functional
        if not f.glu:
            return torch.relu(h @ w[p + "up"].T).square() @ w[p + "down"].T
        act = (lambda z: F.gelu(z, approximate="tanh")) if f.act == "gelu_tanh" else F.silu
        return (act(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T

    def _mix(self, mx, p: str, at: list, h, pos, seqs, blk, off):
        if mx.kind == "parallel":      # (the weighted sum; the other form belongs to _parallel_layers)
            return (mx.gains[0] * self._mix(mx.left, p + "left.", at[:1], h, pos, seqs, blk, off)
                    + mx.gains[1] * self._mix(mx.right, p + "right.", at[1:], h, pos, seqs, blk, off))
        ci = at[0]
        if mx.kind == "talking_attention":
            return self._talking(mx, p, ci, h, pos, seqs, blk, off)
        if mx.kind == "min_gru":
            return self._gru(mx, p, ci, h, seqs)
        if mx.kind == "attention":
            return self._attention(mx, p, ci, h, pos, seqs, blk, off)
        if mx.kind == "latent_attention":
            return self._latent(mx, p, ci, h, pos, seqs, blk, off)
        if mx.kind == "mlstm":
            return self._memory(mx, p, ci, h, seqs)
        return self._retention(mx, p, ci, h, pos, seqs)

    def _feed(self, f, p: str, h):
        return self._moe(f, p, h) if f.kind == "moe" else self._dense(f, p, h)

    def _sandwich_layers(self, x, pos, seqs, blk, off):
        """Layers with a norm on either side of every sublayer; returns the stream."""
        w, one = self.w, self.cfg.norm_weight_offset
        for li, at in self.runs:
            L, p = self.cfg.layers[li], f"l{li}."
            y = self._mix(L.mixer, p + "mix.", at, self._unit(x) * (w[p + "norm1"] + one), pos, seqs, blk, off)
            x = x + self._unit(y) * w[p + "norm1b"] * w[p + "ls1"]
            if L.mlp is not None:
                y = self._feed(L.mlp, p + "mlp.", self._unit(x) * (w[p + "norm2"] + one))
                x = x + self._unit(y) * w[p + "norm2b"] * w[p + "ls2"]
        return x

    def _single_layers(self, x, pos, seqs, blk, off):
        """One plain residual stream, a norm before every sublayer; returns the stream."""
        cfg, w, one, x0 = self.cfg, self.w, self.cfg.norm_weight_offset, x
        starts = cfg.pass_starts
        for ri, (li, at) in enumerate(self.runs):
            L, p = cfg.layers[li], f"l{li}."
            if cfg.loop_inject and ri in starts:
                x = torch.cat([x, x0], -1) @ w["loop.in"].T + w["loop.step"][starts[ri]]
            h = self._unit(x) * (w[p + "norm1"] + one)
            x = x + cfg.residual_mult * self._mix(L.mixer, p + "mix.", at, h, pos, seqs, blk, off)
            if L.mlp is not None:
                x = x + cfg.residual_mult * self._feed(L.mlp, p + "mlp.", self._unit(x) * (w[p + "norm2"] + one))
        return x

    def _parallel_layers(self, x, pos, seqs, blk, off):
        """Layers whose mixer and feed-forward read one residual stream side by side; returns the stream."""
        w, one = self.w, self.cfg.norm_weight_offset
        for li, (left, right) in self.runs:
            L, p = self.cfg.layers[li], f"l{li}."
            u = self._unit(x)
            h = u * (w[p + "norm1"] + one)
            a = self._attention(L.mixer.left, p + "mix.left.", left, h, pos, seqs, blk, off)
            b = self._ssd(L.mixer.right, p + "mix.right.", right, h, seqs)
            y = 0.5 * (self._unit(a) * w[p + "mix.left.out"] + self._unit(b) * w[p + "mix.right.out"])
            if L.mlp is not None:
                y = y + self._moe(L.mlp, p + "mlp.", u * (w[p + "norm2"] + one))
            x = x + y
        return x

    # ------------------------------------------------------------------ step
    @torch.no_grad()
    def forward_plan(self, plan) -> torch.Tensor:
        cfg, w = self.cfg, self.w
        tok = torch.as_tensor(plan.token_ids.astype(np.int64))
        pos = torch.as_tensor(plan.positions.astype(np.int64))
        nd, W = plan.n_decode, plan.max_blocks
        dbt, pbt = plan.decode_block_tables.reshape(nd, W), plan.prefill_block_tables.reshape(plan.n_prefill, W)
        # (first row, rows, context after the step, block table, state slot) of every sequence
        seqs = [(i, 1, int(plan.decode_seq_lens[i]), dbt[i], int(plan.decode_slots[i])) for i in range(nd)]
        seqs += [(int(plan.q_start[i]), int(plan.q_lens[i]), int(plan.ctx_lens[i]), pbt[i], int(plan.prefill_slots[i]))
                 for i in range(plan.n_prefill)]
        blk, off = torch.as_tensor(plan.slot_mapping // 16), torch.as_tensor(plan.slot_mapping % 16)
        x = w["embed"][tok]
        if cfg.bigram is not None:
            b = cfg.bigram
            prev = torch.as_tensor(plan.prev_ids.astype(np.int64))
            row = torch.where(prev < 0, torch.full_like(prev, b.buckets), (prev * b.mul_prev + tok * b.mul_cur) % b.buckets)
            x = x + w["bigram"][row]
        if cfg.residual_mult is not None:
            return self._head(self._single_layers(x * cfg.emb_scale, pos, seqs, blk, off), plan)
        if any(L.parallel for L in cfg.layers):
            return self._head(self._parallel_layers(x * cfg.emb_scale, pos, seqs, blk, off), plan)
        if any(L.post_norm for L in cfg.layers):
            return self._head(self._sandwich_layers(x * cfg.emb_scale, pos, seqs, blk, off), plan)
        xs = x[None].repeat(max(1, cfg.streams), 1, 1)
        one = torch.ones(1)

        def sub(p: str, q: int, fn):
            nonlocal xs
            ci, co, mix = ([w[f"{p}hc{q}.{k}"] for k in ("in", "out", "mix")] if cfg.streams else (one, one, one[None]))
            h = self._unit(torch.einsum("s,std->td", ci, xs)) * (w[f"{p}norm{q}"] + cfg.norm_weight_offset)
            xs = torch.einsum("sz,std->ztd", mix, xs) + co[:, None, None] * fn(h)[None]

        for li, at in self.runs:
            L, p = cfg.layers[li], f"l{li}."
            sub(p, 1, lambda h: self._mix(L.mixer, p + "mix.", at, h, pos, seqs, blk, off))
            if L.mlp is not None:
                sub(p, 2, lambda h: self._feed(L.mlp, p + "mlp.", h))
        return self._head(xs.sum(0), plan)

    def _head(self, x: torch.Tensor, plan) -> torch.Tensor:
        rows = torch.as_tensor(plan.logit_rows.astype(np.int64))
        hl = self._unit(x[rows]) * (self.w["final.norm"] + self.cfg.norm_weight_offset)
        self.logits = hl @ self.head.T * self.cfg.logit_scale
        if self.cfg.logit_softcap:
            self.logits = self.cfg.logit_softcap * torch.tanh(self.logits / self.cfg.logit_softcap)
        return self.logits
