"""Mixers of parallel blocks: lightning (constant-decay linear attention), wkv (token-shifted recurrence with per-channel
decay), latent attention over a paged cache.

A parallel block has one norm; its mixer and its feed-forward read the same rows and their outputs are added to the residual
together.  The projections of a row are therefore one product (mixer and gate / up matrices stacked), and so are the
outputs: the gated mixer output and the activated feed-forward row lie side by side in `cat`, the two output matrices
side by side along K.  `forward` returns the block's fp32 update of the residual.

Verify rows (`commit=False`) leave recurrent states untouched and keep their inputs pending; `commit` replays the accepted
prefix.  Cache rows are written in place past the committed length."""
from __future__ import annotations

from typing import List

import torch

from .. import ops
from ..config import ModelConfig
from ..oracle import layers as L
from .layout import pad
from .plan import Plan


class PendingRows:
    """Slot states that verify rows leave alone: `pending` = (inputs, plan) until the accepted prefix is replayed by
    `commit_rows(inputs, plan, device row counts)`."""
    pending = None

    def commit(self, accepted: List[List[int]]):
        if self.pending is None:
            return
        args, plan = self.pending
        dev = args[0].device
        for rows in accepted:
            assert rows == list(range(len(rows))), "these layers verify chains"
        self.commit_rows(args, plan, torch.tensor([len(r) for r in accepted], dtype=torch.int32, device=dev))
        self.pending = None


class _ParallelMixer(PendingRows):
    wants_f32_rows = False               # needs the fp32 norm output besides the activation rows

    def __init__(self, cfg: ModelConfig, spec, w: dict, dtype):
        self.cfg, self.c, self.w, self.dtype, self.eps = cfg, spec.mixer, w, dtype, cfg.norm_eps
        self.F = spec.ffn
        self.Fp = pad(spec.ffn, 8)

    def _concat(self, o, n, group, gate, kind, ff, out=None):
        """cat rows [mixer | feed-forward] for the output product."""
        off = pad(n, 8)
        return ops.gate_concat(o, n, group, self.w.get("norm"), self.eps, gate, kind, ff if self.F else None, self.F, off,
                               off + self.Fp, self.dtype, out)


class LightningMixer(_ParallelMixer):
    def __init__(self, cfg, spec, w, n_slots, device, dtype):
        super().__init__(cfg, spec, w, dtype)
        c = self.c
        self.nk, self.nv = c.n_heads * c.head_dim, c.n_heads * c.v_dim
        k8, v8 = pad(self.nk, 8), pad(self.nv, 8)
        self.o_k, self.o_v, self.o_g, self.o_ff = k8, 2 * k8, 2 * k8 + v8, 2 * k8 + 2 * v8
        self.S = torch.zeros(n_slots, c.n_heads, c.head_dim, c.v_dim, device=device, dtype=torch.float32)

    def reset(self, slot: int):
        self.S[slot].zero_()

    def _state(self, proj, plan, commit, n_rows=None):
        c = self.c
        return ops.linear_state(proj[:, : self.nk], proj[:, self.o_k: self.o_k + self.nk], proj[:, self.o_v: self.o_v + self.nv],
                                c.n_heads, c.head_dim, c.v_dim, self.S, plan, commit, act=True, log2a=self.w["log2_decay"],
                                n_rows=n_rows)

    def forward(self, h, plan: Plan, seqs, commit: bool, h32=None):
        proj = ops.linear(h, self.w["in"])
        o = self._state(proj, plan, commit)
        self.pending = None if commit else ((proj,), plan)
        cat = self._concat(o, self.nv, self.nv, proj[:, self.o_g: self.o_g + self.nv], "sigmoid", proj[:, self.o_ff:])
        return ops.linear(cat, self.w["out"], out_f32=True)

    def commit_rows(self, args, plan, n_rows):
        self._state(args[0], plan, True, n_rows)

    def state_tensors(self):
        return {"S": self.S}


class WkvMixer(_ParallelMixer):
    wants_f32_rows = True

    def __init__(self, cfg, spec, w, n_slots, device, dtype):
        super().__init__(cfg, spec, w, dtype)
        c = self.c
        self.n = c.n_heads * c.head_dim
        self.S = torch.zeros(n_slots, c.n_heads, c.head_dim, c.head_dim, device=device, dtype=torch.float32)
        # prompts multiply a two-term bf16 sum of the rank activations: [w2 | w2]
        self.w2x2 = torch.cat((w["w2"], w["w2"]), 1).contiguous() if dtype == torch.bfloat16 else None
        self.carried = torch.zeros(n_slots, cfg.hidden, device=device, dtype=torch.float32)     # the previous token's row

    def reset(self, slot: int):
        self.S[slot].zero_()
        self.carried[slot].zero_()

    def _state(self, rkvg, logw, h32, plan, commit, n_rows=None):
        c = self.c
        return ops.linear_state(rkvg[0], rkvg[1], rkvg[2], c.n_heads, c.head_dim, c.head_dim, self.S, plan, commit, logw=logw,
                                u=self.w["u"], h32=h32, carried=self.carried, n_rows=n_rows)

    def forward(self, h, plan: Plan, seqs, commit: bool, h32=None):
        w = self.w
        mix = ops.token_shift(h32, self.carried, w["mu"], plan, self.dtype)              # r k v g w
        rkvg = ops.linear_stack(mix[:4], w["rkvg"])
        logw = ops.channel_decay(ops.linear(mix[4], w["w1"], out_f32=True), w["w2"], w["w0"], self.n, self.w2x2)
        o = self._state(rkvg, logw, h32, plan, commit)
        self.pending = None if commit else ((rkvg, logw, h32), plan)
        ff = ops.linear(h, w["ff"]) if self.F else None
        cat = self._concat(o, self.n, self.c.head_dim, rkvg[3], "silu", ff)
        return ops.linear(cat, w["out"], out_f32=True)

    def commit_rows(self, args, plan, n_rows):
        self._state(*args, plan, True, n_rows)

    def state_tensors(self):
        return {"S": self.S, "carried": self.carried}


class LatentMixer(_ParallelMixer):
    """The cache holds one row per token, [normed latent | rotated key part] with both parts padded to 16, in pages shared by
    all slots (`pages`: the model's page table).  Decode rows attend in the absorbed form, prompts on up-projected keys
    and values.  Queries come from their own latent (`q_rank`) or from the row; without `rope_dim` nothing is rotated; in a
    sequential block (no feed-forward here) the output product is the mixer's alone."""
    paged = True

    def __init__(self, cfg, spec, w, n_pages, page, pages, device, dtype):
        super().__init__(cfg, spec, w, dtype)
        c = self.c
        self.Dp, self.Rp, self.Vp, self.Lp = pad(c.head_dim, 16), pad(c.rope_dim, 16), pad(c.v_dim, 16), pad(c.kv_rank, 16)
        self.nv = c.n_heads * c.v_dim
        self.nq = c.n_heads * (self.Dp + self.Rp)                # query columns, behind uq or in the projected row itself
        o = {"dq": 0, "lat": pad(c.q_rank, 8) if c.q_rank else self.nq}
        o["rot"] = o["lat"] + self.Lp
        o["g"] = o["rot"] + self.Rp
        o["ff"] = o["g"] + pad(self.nv if c.gate == "element" else c.n_heads, 8)
        self.off, self.page, self.pages = o, page, pages
        self.lat = torch.zeros(n_pages, page, self.Lp + self.Rp, device=device, dtype=dtype)
        # shapes of the tensor-core kernels (heads as MMA rows, rows staged in shared memory); else one CTA per row and head
        hm = 16 if c.n_heads <= 16 else (32 if c.n_heads <= 32 else 64)
        kw = self.Lp + self.Rp
        self.decode_tc_ok = c.n_heads <= 64 and (hm + 64) * (kw + 8) * 2 + hm * (65 * 4 + 72 * 4) <= 200 * 1024
        vp = next((x for x in (32, 64, 128, 256) if self.Vp <= x), 0)
        self.prefill_ok = vp > 0 and (256 * (self.Dp + self.Rp + 8) + 128 * (vp + 8)) * 2 <= 220 * 1024

    def reset(self, slot: int):
        pass

    def forward(self, h, plan: Plan, seqs, commit: bool, h32=None):
        proj = ops.linear(h, self.w["in"])
        nvp = pad(self.nv, 8)
        cat = torch.empty(h.shape[0], nvp + self.Fp, dtype=self.dtype, device=h.device)
        if nvp > self.nv:
            cat[:, self.nv: nvp] = 0
        if ops.latent_mixer(self, proj, plan, cat) is None:
            self._rows(proj, plan, cat)
        if self.F:
            self._concat(None, self.nv, 0, None, None, proj[:, self.off["ff"]:], out=cat)
        return ops.linear(cat, self.w["out"], out_f32=True)

    def _rows(self, proj, plan, cat):
        """Plain form over the page table (CPU)."""
        c, w, off = self.c, self.w, self.off
        R, H, D, Ro, V = proj.shape[0], c.n_heads, c.head_dim, c.rope_dim, c.v_dim
        rope = L.rope_interleaved if c.rope_interleaved else L.rope_neox
        if c.q_rank:
            cq = L.rms(proj[:, : c.q_rank].float(), w["dq_norm"], self.eps)
            cq = torch.cat((cq, cq.new_zeros(R, w["uq"].shape[1] - c.q_rank)), 1)
            q = (cq @ w["uq"].float().t()).view(R, H, self.Dp + self.Rp)
        else:
            q = proj[:, : self.nq].float().reshape(R, H, self.Dp + self.Rp)
        qr = rope(q[..., self.Dp: self.Dp + Ro], plan.pos, Ro, c.rope_theta)
        lat = L.rms(proj[:, off["lat"]: off["lat"] + c.kv_rank].float(), w["kv_norm"], self.eps)
        kr = rope(proj[:, off["rot"]: off["rot"] + Ro].float().view(R, 1, Ro), plan.pos, Ro, c.rope_theta)[:, 0]
        up = w["kv_up"].float().view(H, self.Dp + self.Vp, self.Lp)[:, :, : c.kv_rank]
        flat = self.lat.view(-1, self.Lp + self.Rp)
        for s in plan.segs:
            sl, n = slice(s.r0, s.r0 + s.n), s.pos0 + s.n
            t = torch.arange(n)
            idx = self.pages[s.slot, t // self.page].long() * self.page + t % self.page
            assert int(idx.min()) >= 0, "a position without a page"
            flat[idx[s.pos0:], : c.kv_rank] = lat[sl].to(flat.dtype)
            flat[idx[s.pos0:], self.Lp: self.Lp + Ro] = kr[sl].to(flat.dtype)
            ctx = flat[idx].float()
            kv = torch.einsum("sl,hdl->shd", ctx[:, : c.kv_rank], up)
            sc = torch.einsum("thd,shd->hts", q[sl, :, :D], kv[..., :D]) + torch.einsum("thd,sd->hts", qr[sl], ctx[:, self.Lp: self.Lp + Ro])
            sc = (sc * c.scale).masked_fill(t.view(1, 1, n) > plan.pos[sl].view(1, -1, 1), float("-inf"))
            if c.sink:                           # one more score, without a value
                sc = torch.cat((sc, w["sink"].view(H, 1, 1).expand(H, s.n, 1)), -1)
            o = torch.einsum("hts,shd->thd", torch.softmax(sc, -1)[..., :n], kv[..., self.Dp: self.Dp + V])
            gate = proj[sl, off["g"]: off["g"] + (self.nv if c.gate == "element" else H)].float()
            o = o * torch.sigmoid(gate).view(s.n, H, -1)
            cat[sl, : self.nv] = o.reshape(s.n, self.nv).to(cat.dtype)

    def commit(self, accepted):
        pass

    def compact(self, seqs, seg, rows):
        assert rows == list(range(len(rows))), "paged latent rows verify chains"

    def state_tensors(self):
        return {"lat": self.lat}
