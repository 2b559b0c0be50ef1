"""Input convolution of a sublayer: its normed rows h become h + conv(h), a causal convolution over time with a few taps per channel.

The convolution is part of the launch that updates the residual and norms the rows (`ops.add_norm_rows`).  A slot's state is its last
`taps - 1` normed rows (fp32).  Verify rows (`commit=False`) leave it alone and keep their normed rows pending; `commit_rows` advances
it by the accepted prefix."""
from __future__ import annotations

import torch

from .. import ops
from .parallel_mixers import PendingRows


class InputConv(PendingRows):
    def __init__(self, w: torch.Tensor, n_slots: int, device):
        """`w` [taps, width]: the last tap multiplies the row itself."""
        self.w, self.taps = w, w.shape[0]
        self.tail = torch.zeros(n_slots, self.taps - 1, w.shape[1], dtype=torch.float32, device=device)

    def reset(self, slot: int):
        self.tail[slot].zero_()

    def keep(self, rows, plan, commit: bool):
        """`rows`: the normed rows of a pass that did not commit."""
        self.pending = None if commit else ((rows,), plan)

    def commit_rows(self, args, plan, n_rows):
        ops.advance_tail(self.tail, args[0], plan, n_rows)

    def state_tensors(self):
        return {"tail": self.tail}
