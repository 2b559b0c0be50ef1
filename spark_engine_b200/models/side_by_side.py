"""Two mixers on the same rows: grouped-query attention over the paged cache (left) and linear attention with a decay per token
and key channel (right), outputs scaled and added.

All projections of a row are one product, and so are the outputs: the attention's heads and the gated, normed rows of the
recurrence lie side by side in one row, the two output matrices side by side along K.  Verify rows (`commit=False`) leave the
recurrent state alone; `commit_rows` replays the accepted prefix."""
from __future__ import annotations

import torch

from .. import ops
from ..config import ModelConfig
from .layout import pad
from .paged_gqa import PagedGqaMixer
from .parallel_mixers import PendingRows
from .plan import Plan


class GlaState:
    """Recurrent side: S <- diag(decay) S + k v^T, o = S^T q / sqrt(dim), per head."""

    def __init__(self, cfg: ModelConfig, c, w: dict, n_slots: int, at: int, device, dtype):
        """`at`: first column of [q | k | v | gate | decay rank] (parts padded to 8) in the projected rows."""
        self.c, self.w, self.dtype, self.eps = c, w, dtype, cfg.norm_eps
        self.nk, self.nv, self.nv8 = c.n_heads * c.head_dim, c.n_heads * c.v_dim, pad(c.n_heads * c.v_dim, 8)
        k8 = pad(self.nk, 8)
        self.at = at, at + k8, at + 2 * k8, at + 2 * k8 + self.nv8, at + 2 * k8 + 2 * self.nv8
        self.S = torch.zeros(n_slots, c.n_heads, c.head_dim, c.v_dim, device=device, dtype=torch.float32)

    def run(self, proj, plan: Plan, commit: bool, n_rows=None):
        c, (q, k, v, _, r) = self.c, self.at
        decays = (proj[:, r: r + c.decay_rank], self.w["a2"], self.w["a2_b"], c.tau)
        return ops.linear_state(proj[:, q: q + self.nk], proj[:, k: k + self.nk], proj[:, v: v + self.nv], c.n_heads, c.head_dim, c.v_dim,
                                self.S, plan, commit, n_rows=n_rows, qscale=c.head_dim ** -0.5, low_rank=decays)

    def put(self, o, proj, out):
        """norm per head * silu(gate) -> out (a column range of the output product's rows)."""
        g = self.at[3]
        ops.gate_concat(o, self.nv, self.c.v_dim, self.w["norm"], self.eps, proj[:, g: g + self.nv], "silu", None, 0, self.nv8,
                        out.stride(0), self.dtype, out)


class SideBySideMixer(PendingRows):
    paged = True

    def __init__(self, cfg: ModelConfig, spec, w: dict, n_slots: int, n_pages: int, page: int, pages, device, dtype):
        c = spec.mixer
        self.w, self.dtype = w, dtype
        self.left = PagedGqaMixer(cfg, c.left, w, n_slots, n_pages, page, pages, device, dtype, out_scale=c.left_scale)
        self.nl = self.left.H * self.left.Vp
        self.right = GlaState(cfg, c.right, w, n_slots, self.left.columns, device, dtype)

    def reset(self, slot: int):
        self.right.S[slot].zero_()

    def forward(self, h, plan: Plan, seqs, commit: bool):
        proj = ops.linear(h, self.w["in"])
        cat = torch.empty(h.shape[0], self.nl + self.right.nv8, dtype=self.dtype, device=h.device)
        self.left.attend(proj, plan, commit, cat[:, : self.nl])
        self.right.put(self.right.run(proj, plan, commit), proj, cat[:, self.nl:])
        self.pending = None if commit else ((proj,), plan)
        return ops.linear(cat, self.w["out"], out_f32=True)

    def commit_rows(self, args, plan, n_rows):
        self.right.run(*args, plan, True, n_rows)

    def compact(self, seqs, seg, rows):
        self.left.compact(seqs, seg, rows)

    def state_tensors(self):
        return {**self.left.state_tensors(), "S": self.right.S}
