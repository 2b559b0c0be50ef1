"""Grouped-query attention over a paged cache: short causal convolutions on the projected queries, keys and values, soft-capped
scores with a learned bias per distance and head, chunked visibility, a sink that only enters the denominator.

The cache holds the convolved keys and values (heads padded to 16) in pages shared by all slots; a slot's state is the last
`taps - 1` projected rows (`tail`).  Verify rows (`commit=False`) write their cache rows in place past the committed length
and leave the tail alone; `commit_rows` advances it by the accepted prefix."""
from __future__ import annotations

import torch

from .. import ops
from ..config import ModelConfig
from ..oracle import layers as L
from .layout import pad
from .parallel_mixers import PendingRows
from .plan import Plan


class PagedGqaMixer(PendingRows):
    paged = True

    def __init__(self, cfg: ModelConfig, spec, w: dict, n_slots: int, n_pages: int, page: int, pages, device, dtype):
        c = spec.mixer
        self.cfg, self.c, self.w, self.dtype = cfg, c, w, dtype
        self.Dp, self.Vp = pad(c.head_dim, 16), pad(c.v_dim, 16)
        self.nq, self.nk, self.nv = c.n_heads * self.Dp, c.n_kv_heads * self.Dp, c.n_kv_heads * self.Vp
        self.page, self.pages = page, pages
        self.k = torch.zeros(n_pages, page, self.nk, device=device, dtype=dtype)
        self.v = torch.zeros(n_pages, page, self.nv, device=device, dtype=dtype)
        self.tail = torch.zeros(n_slots, c.conv_k - 1, self.nq + self.nk + self.nv, device=device, dtype=dtype)

    def reset(self, slot: int):
        self.tail[slot].zero_()

    def forward(self, h, plan: Plan, seqs, commit: bool):
        proj = ops.linear(h, self.w["qkv"])
        o = ops.paged_gqa(self, proj, plan, commit)
        if o is None:
            o = self._rows(proj, plan, commit)
        self.pending = None if commit else ((proj,), plan)
        return ops.linear(o, self.w["o"], out_f32=True)

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

    def _rows(self, proj, plan, commit):
        """Plain form over the page table (CPU)."""
        c, w = self.c, self.w
        H, G, D, V = c.n_heads, c.n_kv_heads, self.Dp, self.Vp
        kf, vf = self.k.view(-1, self.nk), self.v.view(-1, self.nv)
        out = proj.new_empty(proj.shape[0], H * V)
        for s in plan.segs:
            sl, n = slice(s.r0, s.r0 + s.n), s.pos0 + s.n
            y = L.causal_conv(proj[sl].float(), w["conv_t"].t(), tail=self.tail[s.slot].float())
            if commit:
                self._advance(s.slot, proj[sl])
            t = torch.arange(n)
            idx = self.pages[s.slot, t // self.page].long() * self.page + t % self.page
            assert int(idx.min()) >= 0, "a position without a page"
            kf[idx[s.pos0:]] = y[:, self.nq: self.nq + self.nk].to(kf.dtype)
            vf[idx[s.pos0:]] = y[:, self.nq + self.nk:].to(vf.dtype)
            q = y[:, : self.nq].view(s.n, G, H // G, D)
            sc = torch.einsum("tgrd,sgd->grts", q, kf[idx].float().view(n, G, D)).reshape(H, s.n, n) * c.scale
            if c.softcap:
                sc = c.softcap * torch.tanh(sc / c.softcap)
            dist = plan.pos[sl].view(-1, 1) - t.view(1, -1)
            sc = sc + w["dist_bias"][:, dist.clamp(0, w["dist_bias"].shape[1] - 1)]
            seen = dist >= 0
            if c.chunk:
                seen &= plan.pos[sl].view(-1, 1) // c.chunk == t.view(1, -1) // c.chunk
            sc = sc.masked_fill(~seen, float("-inf"))
            snk = w["sink"].view(H, 1, 1)
            m = torch.maximum(sc.amax(-1, keepdim=True), snk)
            e = torch.exp(sc - m)
            p = e / (torch.exp(snk - m) + e.sum(-1, keepdim=True))
            o = torch.einsum("grts,sgd->tgrd", p.view(G, H // G, s.n, n), vf[idx].float().view(n, G, V))
            out[sl] = o.reshape(s.n, H * V).to(out.dtype)
        return out

    def compact(self, seqs, seg, rows):
        assert rows == list(range(len(rows))), "paged attention rows verify chains"

    def state_tensors(self):
        return {"k": self.k, "v": self.v, "tail": self.tail}
