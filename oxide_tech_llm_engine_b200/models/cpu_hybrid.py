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
        self.runs = []
        self.pk, self.pv, self.states = [], [], []
        for li in cfg.layer_runs:
            at = []      # index of the cache or state of every mixer of the layer
            for mx in cfg.layers[li].mixer.parts:
                if mx.kind == "attention":
                    at.append(len(self.pk))
                    self.pk.append(torch.zeros(num_blocks, mx.kv_heads, 16, mx.dim))
                    self.pv.append(torch.zeros(num_blocks, mx.kv_heads, 16, mx.vdim))
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
        T, w = h.shape[0], self.w
        q, k = h @ w[p + "q"].T, h @ w[p + "k"].T
        if a.qk_norm == "projection":
            q, k = self._unit(q) * w[p + "q.norm"], self._unit(k) * w[p + "k.norm"]
        q = self._rotate(q.view(T, a.heads, a.dim), pos, a.rot)
        self.pk[ci][blk, :, off] = self._rotate(k.view(T, a.kv_heads, a.dim), pos, a.rot)
        self.pv[ci][blk, :, off] = (h @ w[p + "v"].T).view(T, a.kv_heads, a.vdim)
        out = torch.zeros(T, a.heads, a.vdim)
        g = a.heads // a.kv_heads
        for r0, n, ctx, table, _ in seqs:
            pages = torch.as_tensor(table[:(ctx + 15) // 16].astype(np.int64))
            take = lambda c: c[pages].permute(0, 2, 1, 3).reshape(-1, c.shape[1], c.shape[3])[:ctx].repeat_interleave(g, 1)
            i = torch.arange(ctx - n, ctx)[:, None]
            j = torch.arange(ctx)[None]
            see = j <= i
            if a.window:
                see = see & ((i - j < a.window) | (j < a.keep_first))
            if a.chunk:
                see = see & (i // a.chunk == j // a.chunk)
            s = torch.einsum("ihd,jhd->hij", q[r0:r0 + n], take(self.pk[ci])) * a.scale
            s = s.masked_fill(~see[None], float("-inf"))
            if a.sink is not None:
                s = torch.cat([s, torch.full_like(s[..., :1], a.sink)], -1)
            out[r0:r0 + n] = torch.einsum("hij,jhe->ihe", torch.softmax(s, -1)[..., :ctx], take(self.pv[ci]))
        return out.reshape(T, -1) @ w[p + "o"].T

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
        w = self.w
        s = torch.softmax(h @ w[p + "router"].T, -1)
        v, ids = torch.topk(s, e.top, -1)
        v = v / (v.sum(-1, keepdim=True) + 1e-20)
        out = torch.zeros_like(h)
        for i in range(e.experts):
            t, k = torch.nonzero(ids == i, as_tuple=True)
            if t.numel():
                y = torch.relu(h[t] @ w[f"{p}e{i}.up"].T).square() @ w[f"{p}e{i}.down"].T
                out.index_add_(0, t, v[t, k][:, None] * y)
        return out

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
        if any(L.parallel for L in cfg.layers):
            return self._head(self._parallel_layers(x * cfg.emb_scale, pos, seqs, blk, off), plan)
        xs = x[None].repeat(max(1, cfg.streams), 1, 1)
        one = torch.ones(1)

        def sub(p: str, q: int, fn):
            nonlocal xs
            ci, co, mix = ([w[f"{p}hc{q}.{k}"] for k in ("in", "out", "mix")] if cfg.streams else (one, one, one[None]))
            h = self._unit(torch.einsum("s,std->td", ci, xs)) * (w[f"{p}norm{q}"] + cfg.norm_weight_offset)
            xs = torch.einsum("sz,std->ztd", mix, xs) + co[:, None, None] * fn(h)[None]

        for li, (ci,) in self.runs:
            L, p = cfg.layers[li], f"l{li}."
            if L.mixer.kind == "attention":
                sub(p, 1, lambda h: self._attention(L.mixer, p + "mix.", ci, h, pos, seqs, blk, off))
            else:
                sub(p, 1, lambda h: self._retention(L.mixer, p + "mix.", ci, h, pos, seqs))
            if L.mlp is not None:
                act = (lambda z: torch.nn.functional.gelu(z, approximate="tanh")) if L.mlp.act == "gelu_tanh" else torch.nn.functional.silu
                sub(p, 2, lambda h: (act(h @ w[p + "mlp.gate"].T) * (h @ w[p + "mlp.up"].T)) @ w[p + "mlp.down"].T)
        return self._head(xs.sum(0), plan)

    def _head(self, x: torch.Tensor, plan) -> torch.Tensor:
        rows = torch.as_tensor(plan.logit_rows.astype(np.int64))
        hl = self._unit(x[rows]) * (self.w["final.norm"] + self.cfg.norm_weight_offset)
        self.logits = hl @ self.w["head"].T
        return self.logits
