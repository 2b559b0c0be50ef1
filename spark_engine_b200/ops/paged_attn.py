"""CUDA implementation of grouped-query attention over a paged cache (`csrc/kernels/paged_attn.cu`): short convolutions, or norms
and rotations, into the cache, prompt tiles, split-KV decode rows, and the FP32-unit rows of the 32-bit mode."""
from __future__ import annotations

import ctypes as C

import torch

from . import cuda as cu
from .cuda import P, check, lib, scratch, status_word, stream
from .parallel_block import _iota, _is32, _max_ctx, _short_long

PAGE = 64
SMEM = 220 * 1024            # dynamic shared memory the kernels ask for at most


class ConvPrep(C.Structure):
    _fields_ = [(n, C.c_void_p) for n in ("proj", "w", "tail", "q", "k", "v", "segs", "n_rows", "pages", "status")] \
        + [(n, C.c_int) for n in ("ldp", "C", "taps", "nq", "nk", "nv", "page_ld", "tile", "commit", "store")]


class PagedAttn(C.Structure):
    _fields_ = [(n, C.c_void_p) for n in ("q", "k", "v", "out", "pos", "rows", "row_slot", "pages", "bias", "sink", "part_o", "part_ml", "segs",
                                          "slopes", "gate")] \
        + [(n, C.c_int) for n in ("page_ld", "H", "G", "D", "V", "ldq", "bias_n", "chunk", "seg_ld", "nsplit", "window", "ldg", "ldo")] \
        + [("scale", C.c_float), ("cap", C.c_float), ("out_scale", C.c_float)]


class HeadPrep(C.Structure):
    _fields_ = [(n, C.c_void_p) for n in ("proj", "q_norm", "k_norm", "q", "k", "v", "inv_freq", "pos", "row_slot", "pages", "status")] \
        + [("temp_every", C.c_double)] + [(n, C.c_int) for n in ("ldp", "R", "H", "G", "D", "Dp", "Vp", "rot", "page_ld")] \
        + [("eps", C.c_float), ("temp_coef", C.c_float)]


def decode_fits(D: int, V: int) -> bool:
    return ((16 + PAGE) * (D + 8) + PAGE * (V + 8) + 2 * 16 * 72) * 2 + 16 * 68 * 4 <= SMEM


def prefill_fits(D: int, V: int) -> bool:
    vp = next((x for x in (32, 64, 128, 256) if V <= x), 0)
    return vp > 0 and ((128 + 2 * PAGE) * (D + 8) + 2 * PAGE * (vp + 8)) * 2 + 2 * (128 + PAGE) * 4 <= SMEM


def _conv(mx, proj, plan, d, q, commit, n_rows=None):
    a = ConvPrep(P(proj), P(mx.w["conv_t"]), P(mx.tail), P(q), P(mx.k), P(mx.v), P(d["seg"]), P(n_rows), P(mx.pages),
                 P(status_word(proj.device)), proj.stride(0), proj.shape[1], mx.c.conv_k, mx.nq, mx.nk, mx.nv, mx.pages.shape[1], 0,
                 int(commit), int(q is not None))
    if cu.dbg.CHECK:
        cu._check_slots("conv_prep", plan, mx.tail.shape[0])
    check(lib().spark_conv_prep(C.byref(a), len(plan.segs), max(s.n for s in plan.segs), _is32(proj.dtype), stream()), "spark_conv_prep")


def commit_tail(mx, proj, plan, n_rows):
    _conv(mx, proj, plan, cu._plan_dev(plan, proj.device), None, True, n_rows)


def _heads(mx, proj, d, q):
    """Norm, rotation and temperature of the heads: queries to `q`, keys and values to their pages (a layer that reads another
    layer's cache has queries only)."""
    c, w = mx.c, mx.w
    a = HeadPrep(P(proj), P(w.get("q_norm")), P(w.get("k_norm")), P(q), P(mx.k), P(mx.v), P(mx.inv_freq), P(d["pos32"]), P(d["row_slot"]),
                 P(mx.pages), P(status_word(proj.device)), c.temp_every, proj.stride(0), proj.shape[0], c.n_heads,
                 0 if mx.source is not None else c.n_kv_heads, c.head_dim, mx.Dp, mx.Vp, c.rope_dims, mx.pages.shape[1], mx.cfg.norm_eps,
                 c.temp_coef)
    check(lib().spark_head_prep(C.byref(a), _is32(proj.dtype), stream()), "spark_head_prep")


def mixer(mx, proj, plan, commit, out=None):
    """Attention of every row of `proj` (projected heads, then the gate's columns): [R, heads * padded value width]."""
    c, w, dev, dt = mx.c, mx.w, proj.device, proj.dtype
    d = cu._plan_dev(plan, dev)
    R = proj.shape[0]
    q = torch.empty(R, mx.nq, dtype=dt, device=dev)
    if c.conv_k:
        _conv(mx, proj, plan, d, q, commit)
    else:
        _heads(mx, proj, d, q)
    if out is None:
        out = torch.empty(R, c.n_heads * mx.Vp, dtype=dt, device=dev)
    bias = w.get("dist_bias")
    gate = proj[:, mx.columns:] if c.gated else None
    a = PagedAttn(q=P(q), k=P(mx.k), v=P(mx.v), out=P(out), pos=P(d["pos32"]), row_slot=P(d["row_slot"]), pages=P(mx.pages), bias=P(bias),
                  sink=P(w.get("sink")), slopes=P(mx.slopes), gate=P(gate), page_ld=mx.pages.shape[1], H=c.n_heads, G=c.n_kv_heads, D=mx.Dp,
                  V=mx.Vp, ldq=mx.nq, bias_n=bias.shape[1] if bias is not None else 0, chunk=c.chunk, window=c.window, seg_ld=5,
                  ldg=proj.stride(0), ldo=out.stride(0), scale=c.scale, cap=c.softcap, out_scale=mx.out_scale)
    rows, ns, tab, longs = None, R, None, []
    if not _is32(dt) and prefill_fits(mx.Dp, mx.Vp):
        rows, ns, tab, longs, _ = _short_long(plan, dev)
    if ns:
        a.rows = P(rows)
        if _is32(dt) or not decode_fits(mx.Dp, mx.Vp):
            check(lib().spark_paged_rows(C.byref(a), ns, _is32(dt), stream()), "spark_paged_rows")
        else:
            a.nsplit = (_max_ctx(plan, d) + PAGE - 1) // PAGE
            span = c.chunk or c.window                     # pages that an aligned chunk or a window can touch
            if span:
                a.nsplit = min(a.nsplit, (span + 2 * PAGE - 2) // PAGE)
            step = min(ns, max(16, 4096 // a.nsplit))      # bounds the partial results of long contexts
            if rows is None and ns > step:
                a.rows = P(_iota(R, dev))
            part_o = scratch("paged_part_o", step * c.n_heads * a.nsplit * mx.Vp, torch.float32, dev)
            part_ml = scratch("paged_part_ml", step * c.n_heads * a.nsplit * 2, torch.float32, dev)
            a.part_o, a.part_ml = P(part_o), P(part_ml)
            base = a.rows
            for r in range(0, ns, step):
                if base:
                    a.rows = base + 4 * r
                check(lib().spark_paged_decode(C.byref(a), min(step, ns - r), stream()), "spark_paged_decode")
    if longs:
        a.segs = P(tab)
        check(lib().spark_paged_prefill(C.byref(a), len(longs), max(s.n for s in longs), stream()), "spark_paged_prefill")
    return out

