"""Helpers of architectures that read their own checkpoint format (models/registry.py): zero padding to the kernels'
alignment, and tensors taken from a flat dict by name with their shapes checked."""
from __future__ import annotations

from typing import Dict, Optional

import torch


def pad(n: int, m: int) -> int:
    return (n + m - 1) // m * m


def stack_rows(parts, to: int = 8) -> torch.Tensor:
    """Row blocks stacked, each padded to a multiple of `to` rows."""
    out = []
    for t in parts:
        n = pad(t.shape[0], to) - t.shape[0]
        out += [t, t.new_zeros(n, t.shape[1])] if n else [t]
    return torch.cat(out)


def pad_cols(t: torch.Tensor, n: int) -> torch.Tensor:
    return t if t.shape[-1] == n else torch.cat((t, t.new_zeros(*t.shape[:-1], n - t.shape[-1])), -1)


def pad_head_rows(t: torch.Tensor, heads: int, to: int) -> torch.Tensor:
    """[heads * d, n] -> [heads * to, n]: every head's rows padded with zero rows."""
    d, n = t.shape[0] // heads, t.shape[1]
    if d == to:
        return t
    out = t.new_zeros(heads, to, n)
    out[:, :d] = t.view(heads, d, n)
    return out.view(heads * to, n)


def pad_head_cols(t: torch.Tensor, heads: int, to: int) -> torch.Tensor:
    """[m, heads * d] -> [m, heads * to]: every head's columns padded with zero columns."""
    m, d = t.shape[0], t.shape[1] // heads
    return pad_cols(t.view(m, heads, d), to).reshape(m, heads * to)


def latent_up(uk: torch.Tensor, uv: torch.Tensor, c, dtype) -> Dict[str, torch.Tensor]:
    """Key and value matrices over the latents, [heads * dim | heads * v, latent], as the runner uses them: uk_t [heads, latent, dim]
    and uv [heads, v, latent] for absorbed rows, kv_up (per head [key | value], padded to 16) for prompts."""
    H, D, V, Lp = c.n_heads, c.head_dim, c.v_dim, pad(c.kv_rank, 16)
    Dp, Vp = pad(D, 16), pad(V, 16)
    uk, uv = pad_cols(uk, Lp).view(H, D, Lp), pad_cols(uv, Lp).view(H, V, Lp)
    up = uk.new_zeros(H, Dp + Vp, Lp)
    up[:, :D], up[:, Dp: Dp + V] = uk, uv
    wd = lambda t: t.to(dtype).contiguous()
    return {"uk_t": wd(pad_cols(uk.transpose(1, 2), Dp)), "uv": wd(uv), "kv_up": wd(up.view(H * (Dp + Vp), Lp))}


def taker(tensors: Dict[str, torch.Tensor], device):
    """get(name, shape=None): the tensor on `device`; its shape must be the given one (None entries: any)."""
    def get(name: str, shape: Optional[tuple] = None) -> torch.Tensor:
        if name not in tensors:
            raise ValueError(f"tensor {name} is missing from the checkpoint")
        t = tensors[name]
        if shape is not None and (len(shape) != t.dim() or any(a is not None and a != b for a, b in zip(shape, t.shape))):
            raise ValueError(f"tensor {name} has shape {tuple(t.shape)}, the configuration says {shape}")
        return t.to(device)
    return get
