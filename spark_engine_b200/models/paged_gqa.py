"""Grouped-query attention over a paged cache.  The projected heads pass short causal convolutions, or a norm per head, a rotation
and a temperature of the queries; scores may be soft-capped, biased by distance (a learned table or a slope per head), limited to
chunks or a window; a sink may enter the denominator, a gate per head may scale the output.

The cache holds the finished keys and values (heads padded to 16) in pages shared by all slots, or is another layer's
(`source`).  With convolutions a slot's state is the last `taps - 1` projected rows (`tail`).  Verify rows (`commit=False`) write
their cache rows in place past the committed length and leave the tail alone; `commit_rows` advances it by the accepted prefix."""
from __future__ import annotations

import math

import torch

from .. import ops
from ..config import ModelConfig, PagedGqaConfig
from ..oracle import layers as L
from .layout import pad
from .parallel_mixers import PendingRows
from .plan import Plan


class PagedGqaMixer(PendingRows):
    paged = True

    def __init__(self, cfg: ModelConfig, c: PagedGqaConfig, w: dict, n_slots: int, n_pages: int, page: int, pages, device, dtype,
                 source: "PagedGqaMixer" = None, out_scale: float = 1.0):
        self.cfg, self.c, self.w, self.dtype, self.source, self.out_scale = cfg, c, w, dtype, source, out_scale
        self.H, self.Dp, self.Vp = c.n_heads, pad(c.head_dim, 16), pad(c.v_dim, 16)
        self.nq, self.nk, self.nv = c.n_heads * self.Dp, c.n_kv_heads * self.Dp, c.n_kv_heads * self.Vp
        self.columns = self.nq + (0 if source is not None else self.nk + self.nv)     # projected heads; the gate's columns follow
        self.page, self.pages = page, pages
        if source is not None:
            self.k, self.v = source.k, source.v
        else:
            self.k = torch.zeros(n_pages, page, self.nk, device=device, dtype=dtype)
            self.v = torch.zeros(n_pages, page, self.nv, device=device, dtype=dtype)
        self.tail = torch.zeros(n_slots, c.conv_k - 1, self.columns, device=device, dtype=dtype) if c.conv_k else None
        self.inv_freq = (c.rope_theta ** (-torch.arange(c.rope_dims // 2, dtype=torch.float64) * 2 / max(c.rope_dims, 1)) / c.rope_factor).to(device)
        self.slopes = None
        if c.slopes:
            self.slopes = torch.tensor([2.0 ** (-8 * (h + 1) / c.n_heads) for h in range(c.n_heads)], dtype=torch.float32, device=device)

    def reset(self, slot: int):
        if self.tail is not None:
            self.tail[slot].zero_()

    def forward(self, h, plan: Plan, seqs, commit: bool):
        proj = ops.linear(h, self.w["qkv"])
        o = self.attend(proj, plan, commit)
        self.pending = None if commit or self.tail is None else ((proj,), plan)
        return ops.linear(o, self.w["o"], out_f32=True)

    def attend(self, proj, plan: Plan, commit: bool, out=None):
        """Heads' outputs [R, heads * padded value width] of the projected rows (into `out` if given)."""
        o = ops.paged_gqa(self, proj, plan, commit, out)
        return o if o is not None else self._rows(proj, plan, commit, out)

    def commit_rows(self, args, plan, n_rows):
        proj, = args
        if ops.conv_tail(self, proj, plan, n_rows):
            return
        for s, n in zip(plan.segs, n_rows.tolist()):
            self._advance(s.slot, proj[s.r0: s.r0 + n])

    def _advance(self, slot, rows):
        t = self.tail[slot]
        if t.shape[0]:
            self.tail[slot] = torch.cat((t, rows.to(t.dtype)))[-t.shape[0]:]

    # -- plain form over the page table (CPU) -------------------------------------------------
    def _heads(self, y, n: int, norm, pos):
        """Normed and rotated heads [T, n, Dp]."""
        c = self.c
        y = y.float().reshape(-1, n, self.Dp)[..., : c.head_dim]
        if c.qk_norm:
            y = L.rms(y, self.w[norm], self.cfg.norm_eps)
        if c.rope_dims:
            a = (pos.double().unsqueeze(1) * self.inv_freq).float().unsqueeze(1)
            u, v = y[..., 0: c.rope_dims: 2], y[..., 1: c.rope_dims: 2]
            turned = torch.stack((u * a.cos() - v * a.sin(), v * a.cos() + u * a.sin()), -1).flatten(-2)
            y = torch.cat((turned, y[..., c.rope_dims:]), -1)
        return torch.nn.functional.pad(y, (0, self.Dp - c.head_dim))

    def _finished(self, proj, s, pos, commit):
        """Queries [T, H, Dp] and the segment's cache rows (None on another layer's cache)."""
        c, y = self.c, proj[s.r0: s.r0 + s.n].float()
        if c.conv_k:
            y = L.causal_conv(y, self.w["conv_t"].t(), tail=self.tail[s.slot].float())
            if commit:
                self._advance(s.slot, proj[s.r0: s.r0 + s.n])
            return y[:, : self.nq].view(s.n, self.H, self.Dp), y[:, self.nq: self.nq + self.nk], y[:, self.nq + self.nk:]
        q = self._heads(y[:, : self.nq], self.H, "q_norm", pos)
        if c.temp_coef:
            q = q * torch.tensor([1 + c.temp_coef * math.log(math.floor((p + 1) / c.temp_every) + 1) for p in pos.tolist()]).view(-1, 1, 1)
        if self.source is not None:
            return q, None, None
        k = self._heads(y[:, self.nq: self.nq + self.nk], c.n_kv_heads, "k_norm", pos)
        return q, k.reshape(s.n, self.nk), y[:, self.nq + self.nk: self.nq + self.nk + self.nv]

    def _rows(self, proj, plan, commit, out=None):
        c, w = self.c, self.w
        H, G, D, V = c.n_heads, c.n_kv_heads, self.Dp, self.Vp
        kf, vf = self.k.view(-1, self.nk), self.v.view(-1, self.nv)
        if out is None:
            out = proj.new_empty(proj.shape[0], H * V)
        for s in plan.segs:
            sl, n = slice(s.r0, s.r0 + s.n), s.pos0 + s.n
            pos, t = plan.pos[sl], torch.arange(n)
            q, k, v = self._finished(proj, s, pos, commit)
            idx = self.pages[s.slot, t // self.page].long() * self.page + t % self.page
            assert int(idx.min()) >= 0, "a position without a page"
            if k is not None:
                kf[idx[s.pos0:]] = k.to(kf.dtype)
                vf[idx[s.pos0:]] = v.to(vf.dtype)
            sc = torch.einsum("tgrd,sgd->grts", q.view(s.n, G, H // G, D), kf[idx].float().view(n, G, D)).reshape(H, s.n, n) * c.scale
            if c.softcap:
                sc = c.softcap * torch.tanh(sc / c.softcap)
            dist = pos.view(-1, 1) - t.view(1, -1)
            if "dist_bias" in w:
                sc = sc + w["dist_bias"][:, dist.clamp(0, w["dist_bias"].shape[1] - 1)]
            if self.slopes is not None:
                sc = sc - self.slopes.view(H, 1, 1) * dist
            seen = dist >= 0
            if c.chunk:
                seen &= pos.view(-1, 1) // c.chunk == t.view(1, -1) // c.chunk
            if c.window:
                seen &= dist < c.window
            sc = sc.masked_fill(~seen, float("-inf"))
            m = sc.amax(-1, keepdim=True)
            snk = w["sink"].view(H, 1, 1) if "sink" in w else None
            m = torch.maximum(m, snk) if snk is not None else m
            e = torch.exp(sc - m)
            p = e / (e.sum(-1, keepdim=True) + (torch.exp(snk - m) if snk is not None else 0))
            o = torch.einsum("grts,sgd->tgrd", p.view(G, H // G, s.n, n), vf[idx].float().view(n, G, V)).reshape(s.n, H, V)
            if c.gated:
                o = o * torch.sigmoid(proj[sl, self.columns: self.columns + H].float()).unsqueeze(-1)
            out[sl] = (o * self.out_scale).reshape(s.n, H * V).to(out.dtype)
        return out

    def compact(self, seqs, seg, rows):
        assert rows == list(range(len(rows))), "paged attention rows verify chains"

    def state_tensors(self):
        d = {} if self.source is not None else {"k": self.k, "v": self.v}
        return d if self.tail is None else dict(d, tail=self.tail)
