"""CUDA implementations of the ops of models whose layers carry their own sizes (`csrc/kernels/block_rows.cu`, `row_tiles.cu`,
`linear_state.cu`, `latent.cu`, `mla.cu`): row ops around the block, the decayed linear recurrences, latent attention over a paged
cache.  bf16 and fp32
activations; what the mechanisms keep in fp32 (residual, norms, states, decays, scores, softmax weights) is fp32 in both."""
from __future__ import annotations

import ctypes as C

import torch

from . import cuda as cu
from .cuda import P, check, lib, scratch, status_word, stream

CHUNK_MIN_ROWS = 32          # segments of at least this many rows take the chunked / flash kernels
LC = 64                      # rows per chunk of the chunked recurrences


def _is32(dtype) -> int:
    return int(dtype == torch.float32)


# ----------------------------------------------------------------------------- rows
def embed_scaled(table, ids32, scale: float, pos=None, out=None):
    R, H = ids32.shape[0], table.shape[1]
    cu.dbg.check_index("embed token ids", ids32, 0, table.shape[0])
    if out is None:
        out = torch.empty(R, H, dtype=torch.float32, device=table.device)
    p32, freq = (pos[0].to(torch.int32), pos[1]) if pos is not None else (None, None)
    check(lib().spark_embed_scaled(P(table), P(ids32), P(out), R, H, table.shape[0], float(scale), P(p32), P(freq), _is32(table.dtype),
                                   P(status_word(table.device)), stream()), "spark_embed_scaled")
    return out


class RowUpdate(C.Structure):
    """Arguments of the row update (csrc/kernels/block_rows.cu)."""
    _fields_ = [(n, C.c_void_p) for n in ("res", "delta", "y", "inv", "wts", "ids", "shared", "sg", "self_w", "self_x", "scale", "post_w",
                                          "w", "b", "out", "out32")] \
        + [(n, C.c_int) for n in ("H", "slots", "norm", "one_plus")] + [("eps", C.c_float), ("post_eps", C.c_float)]


class RowTiles(C.Structure):
    """Arguments of the row update over tiles of a sequence (csrc/kernels/row_tiles.cu)."""
    _fields_ = [("u", RowUpdate)] + [(n, C.c_void_p) for n in ("res_out", "stack", "avg", "conv_w", "tail", "rows", "segs")] \
        + [(n, C.c_int) for n in ("k", "groups", "taps", "tile", "commit", "R")]


def add_norm_rows(delta, res, norm, dtype, want_f32=False, conv=None, ctx=None):
    """res (fp32) += delta (None, a tensor, a deferred MoE output, or an ops.Update of one), in place unless `ctx` says otherwise;
    returns (h in `dtype`, res, fp32 copy of h or None).  Grouped norms, depth averages and input convolutions (`conv`) run in the
    tiled form, which leaves the old residual as it is."""
    R, H = res.shape
    assert res.dtype == torch.float32 and res.is_contiguous()
    depth = getattr(delta, "depth", None)
    tiled = conv is not None or depth is not None or (ctx is not None and ctx.fresh) or (norm is not None and norm.groups > 1)
    if tiled and getattr(delta, "post", None) is not None:      # (the tiled form does not norm updates)
        assert depth is None
        res, delta = add_norm_rows(delta, res.clone(), None, dtype)[1], None
    u = RowUpdate(res=P(res), H=H)
    keep = []
    x = delta
    if hasattr(delta, "post"):
        x = delta.x
        u.scale = P(delta.scale)
        if delta.post is not None:
            u.post_w, u.post_eps = P(delta.post.w), delta.post.eps
    if isinstance(x, cu.PendingMoe):
        assert x.shared is None or x.shared.dtype == torch.float32
        u.y, u.inv, u.wts, u.ids, u.slots = P(x.y), P(x.inv), P(x.wts), P(x.ids), x.slots
        u.shared, u.sg, u.self_w, u.self_x = P(x.shared), P(x.sg), P(x.self_w), P(x.self_x)
    elif x is not None:
        x = x.float().contiguous()
        u.delta = P(x)
    keep.append(x)
    h = torch.empty(R, H, dtype=dtype, device=res.device)
    h32 = h if dtype == torch.float32 else (torch.empty(R, H, dtype=torch.float32, device=res.device) if want_f32 else None)
    u.out, u.out32 = P(h), P(h32) if h32 is not h else None
    if norm is not None:
        u.norm, u.w, u.b, u.eps, u.one_plus = (1 if norm.b is None else 2), P(norm.w), P(norm.b), norm.eps, int(norm.one_plus)
    if tiled:
        if x is not None or depth is not None:
            new = torch.empty_like(res)
            _row_tiles(u, R, new, norm, depth, conv, ctx, _is32(dtype))
            res = new
        else:
            _row_tiles(u, R, None, norm, None, conv, ctx, _is32(dtype))
        return h, res, h32
    check(lib().spark_row_update(C.byref(u), R, _is32(dtype), stream()), "spark_row_update")
    return h, res, h32


SM_THREADS = 1024            # resident threads per SM (registers); a launch of many rows is one wave of tiles


def tile_threads(R: int) -> int:
    """Threads of a CTA at most (a row's bits do not depend on it): few rows are one step of the whole CTA."""
    return 1024 if R <= 148 else 512


def tile_rows(R: int, H: int, taps: int) -> int:
    """Rows per CTA of the tiled row update: tiles cover the rows before them anew, so they are as long as one wave allows."""
    threads = min(tile_threads(R), -(-H // 128) * 32)
    return max(1, taps - 1, -(-R // (148 * (SM_THREADS // threads))))


def _row_tiles(u, R, new, norm, depth, conv, ctx, f32):
    a = RowTiles(u=u, res_out=P(new), groups=norm.groups if norm is not None else 1, R=R, tile=tile_rows(R, u.H, 0), commit=1)
    nseg, longest = 1, R
    if depth is not None:
        assert depth.stack.is_contiguous() and depth.stack.shape[1] == R and depth.stack.dtype == torch.float32
        a.stack, a.avg, a.k = P(depth.stack), P(depth.a), depth.k
    if conv is not None:
        plan = ctx.plan
        d = cu._plan_dev(plan, conv.tail.device)
        if cu.dbg.CHECK:
            cu._check_slots("row_tiles", plan, conv.tail.shape[0])
        nseg, longest = len(plan.segs), max(s.n for s in plan.segs)
        a.conv_w, a.tail, a.segs, a.taps, a.commit = P(conv.w), P(conv.tail), P(d["seg"]), conv.taps, int(ctx.commit)
        a.tile = tile_rows(R, u.H, conv.taps)
        rows = None
        if not ctx.commit:
            rows = torch.empty(R, u.H, dtype=torch.float32, device=conv.tail.device)
            a.rows = P(rows)
        conv.keep(rows, plan, ctx.commit)
    check(lib().spark_row_tiles(C.byref(a), nseg, longest, tile_threads(R), f32, stream()), "spark_row_tiles")


def advance_tail(tail, rows, plan, n_rows):
    d = cu._plan_dev(plan, tail.device)
    check(lib().spark_tail_advance(P(tail), P(rows), P(d["seg"]), len(plan.segs), P(n_rows), tail.shape[1], tail.shape[2], stream()),
          "spark_tail_advance")


def token_shift(h32, carried, mu, plan, dtype):
    d = cu._plan_dev(plan, h32.device)
    R, H = h32.shape
    n = mu.shape[0]
    out = torch.empty(n, R, H, dtype=dtype, device=h32.device)
    check(lib().spark_token_shift(P(h32), P(carried), P(d["row_slot"]), P(d["row_j"]), P(mu), n, P(out), R, H, _is32(dtype), stream()),
          "spark_token_shift")
    return out


def channel_decay(z, w2, w0, n: int, w2x2=None):
    """z [R, rank] fp32 -> log decay -exp(w2 tanh(z) + w0) [R, n] fp32.  `w2x2`: [w2 | w2] in bf16."""
    R, r = z.shape
    if w2x2 is not None and R >= 64:
        # prompts: tanh as a two-term bf16 sum against [w2 | w2], one tensor-core product
        t = torch.empty(R, 2 * r, dtype=torch.bfloat16, device=z.device)
        check(lib().spark_tanh_split(P(z), z.stride(0), P(t), R, r, stream()), "spark_tanh_split")
        out = cu.dense_linear(t, w2x2, out_f32=True)
        check(lib().spark_neg_exp_bias(P(out), P(w0), R, n, stream()), "spark_neg_exp_bias")
        return out
    out = torch.empty(R, n, dtype=torch.float32, device=z.device)
    check(lib().spark_channel_decay(P(z), z.stride(0), P(w2), w2.stride(0), r, P(w0), P(out), R, n, _is32(w2.dtype), stream()),
          "spark_channel_decay")
    return out


def log_sigmoid_decay(z, w2, b, n: int, tau: float):
    """z [R, rank] in the activation type (columns up to w2's padded rank are readable) -> ln(sigmoid(w2 z + b)) / tau fp32."""
    R, r = z.shape[0], w2.shape[1]
    out = torch.empty(R, n, dtype=torch.float32, device=z.device)
    check(lib().spark_log_sigmoid_decay(P(z), z.stride(0), P(w2), w2.stride(0), r, P(b), float(tau), P(out), R, n, _is32(w2.dtype), stream()),
          "spark_log_sigmoid_decay")
    return out


def swiglu_rows(gu, wts=None, perm=None, glu=0.0):
    """silu(gate) * up of [gate | up] rows (`glu`: see `cuda._glu`); `wts` (fp32): gate and up of row r count wts[perm[r]] times."""
    R, n = gu.shape[0], gu.shape[1] // 2
    out = torch.empty(R, n, dtype=gu.dtype, device=gu.device)
    check(lib().spark_swiglu_rows(P(gu), gu.stride(0), n, P(wts), P(perm), P(out), n, R, cu._glu(glu), _is32(gu.dtype), stream()),
          "spark_swiglu_rows")
    return out


def linear_swiglu(x, w, glu=0.0):
    """silu(x G^T) * (x U^T) for w = [G | U] (halves of a multiple of 128 rows); `glu`: see `cuda._glu`."""
    R, F = x.shape[0], w.shape[0] // 2
    if w.dtype != torch.bfloat16 or R <= 16 or w.shape[1] % 8 or F % 128 or (isinstance(glu, tuple) and glu[1:] != (1.0, 0.0)):
        return swiglu_rows(cu.dense_linear(x, w), glu=glu)
    x = cu._as_bf16(x).contiguous()
    out = torch.empty(R, F, dtype=torch.bfloat16, device=x.device)
    check(lib().spark_gemm_bf16_swiglu(P(x), P(w), P(out), R, F, w.shape[1], x.stride(0), w.stride(0), F,
                                       float(glu[0] if isinstance(glu, tuple) else glu), P(status_word(x.device)),
                                       stream()), "spark_gemm_bf16_swiglu")
    return out


GATES = {None: 0, "sigmoid": 1, "silu": 2}


def gate_concat(o, n, group, w, eps, gate, kind, ff, F, off, width, dtype, out=None, gate_div=1):
    """[ group-norm(o) * w * gate | gelu(ff gate) * ff up ] -> [R, width]; `ff` = [gate | up] columns (up at width - off)."""
    src = o if o is not None else ff
    R = src.shape[0]
    if out is None:
        out = torch.empty(R, width, dtype=dtype, device=src.device)
    check(lib().spark_gate_concat(P(o), 0 if o is None else o.stride(0), n, group, P(w), float(eps), P(gate),
                                  0 if gate is None else gate.stride(0), GATES[kind], gate_div, P(ff), 0 if ff is None else ff.stride(0),
                                  width - off, F, P(out), width, off, R, _is32(dtype), stream()), "spark_gate_concat")
    return out


def linear_stack(xs, w):
    """xs [n, R, K], w [n, N, K] -> [n, R, N]: n independent products of equal shape."""
    n, R, K = xs.shape
    N = w.shape[1]
    dev = xs.device
    if w.dtype == torch.float32 or K % 8:
        y = torch.empty(n, R, N, dtype=xs.dtype, device=dev)
        return cu.gemm_simt(xs, K, R * K, w, K, N * K, y, N, R * N, n, R, N, K)
    if R <= 16 and cu.gemv_rows(K) >= R:
        y = torch.empty(n, R, N, dtype=torch.bfloat16, device=dev)
        return cu.gemv_bf16_items(xs, K, R * K, w, N * K, K, y, N, R * N, n, R, N, K, _iota(n, dev))
    return torch.stack([cu.dense_linear(xs[i], w[i]) for i in range(n)]) if n == 1 else _stack_gemm(xs, w)


def _stack_gemm(xs, w):
    n, R, _ = xs.shape
    y = torch.empty(n, R, w.shape[1], dtype=torch.bfloat16, device=xs.device)
    for i in range(n):
        cu.dense_linear(xs[i], w[i], out=y[i])
    return y


_iotas = {}


def _iota(n, dev):
    key = (n, str(dev))
    if key not in _iotas:
        _iotas[key] = torch.arange(n, dtype=torch.int32, device=dev)
    return _iotas[key]


# ----------------------------------------------------------------------------- recurrences
def _split(plan, dev):
    """Segment tables of a committed plan: (short segments, long segments), each (device table, segments)."""
    d = cu._plan_dev(plan, dev)
    if "seg_split" not in d:
        longs = [s for s in plan.segs if s.n >= CHUNK_MIN_ROWS]
        if not longs:
            d["seg_split"] = ((d["seg"], plan.segs), (None, []))
        else:
            shorts = [s for s in plan.segs if s.n < CHUNK_MIN_ROWS]
            tab = lambda ss: torch.tensor([[s.slot, s.r0, s.n, s.pos0] for s in ss], dtype=torch.int32).to(dev) if ss else None
            d["seg_split"] = ((tab(shorts), shorts), (d["seg"] if not shorts else tab(longs), longs))
    return d["seg_split"]


class LowRankDecay(C.Structure):
    """Decays formed by the sequential recurrence (csrc/kernels/linear_state.cu)."""
    _fields_ = [(n, C.c_void_p) for n in ("z", "w2", "b")] + [(n, C.c_int) for n in ("ldz", "ldw", "rank")] + [("inv_tau", C.c_float)]


def linear_state(q, k, v, H, D, V, S, plan, commit, act=False, log2a=None, logw=None, u=None, h32=None, carried=None,
                 n_rows=None, qscale=1.0, low_rank=None):
    """Decayed linear attention of every segment from its slot's state S [slots, H, D, V]; returns o fp32 [R, H * V], times
    `qscale`.  `log2a` [H]: constant decay per head; else `logw` [R, H * D] (log decay) and `u` (bonus; None: outputs read the
    state behind the current token), with the token-shift row carried along (h32 rows -> carried [slots, width]); or `low_rank` =
    (z, w2, b, tau) of `log_sigmoid_decay`, part of the recurrence's launch for decode rows.  `n_rows`: device counts of
    accepted rows (commit)."""
    dev = q.device
    d = cu._plan_dev(plan, dev)
    R = q.shape[0]
    o = torch.empty(R, H * V, dtype=torch.float32, device=dev)
    if cu.dbg.CHECK:
        cu._check_slots("linear_state", plan, S.shape[0])
    width = h32.shape[1] if h32 is not None else 0
    lr = None
    if low_rank is not None:
        z, w2, b, tau = low_rank
        if R <= cu.DECODE_ROWS_MAX and z.stride(0) % 8 == 0 and z.data_ptr() % 16 == 0:
            lr = LowRankDecay(P(z), P(w2), P(b), z.stride(0), w2.stride(0), w2.shape[1], 1.0 / tau)
        else:
            logw = log_sigmoid_decay(z, w2, b, H * D, tau)

    def args(seg):
        return (P(q), q.stride(0), P(k), k.stride(0), P(v), v.stride(0), D, V, P(log2a), P(logw), P(u), P(S), P(seg), P(n_rows), P(o),
                P(h32), P(carried), width, H, D, V, int(commit), int(act), float(qscale))
    if lr is not None:
        check(lib().spark_linear_seq_lowrank(*args(d["seg"]), len(plan.segs), C.byref(lr), _is32(q.dtype), stream()), "spark_linear_seq_lowrank")
        return o
    short, longs = (d["seg"], plan.segs), (None, [])
    if n_rows is None and commit and q.dtype == torch.bfloat16 and D <= 128:
        short, longs = _split(plan, dev)
    if short[1]:
        check(lib().spark_linear_seq(*args(short[0]), len(short[1]), _is32(q.dtype), stream()), "spark_linear_seq")
    if longs[1]:
        if "lin_chunks" not in d:
            chunks, first = [], []
            for i, sg in enumerate(longs[1]):
                first.append(len(chunks))
                chunks += [(i, c) for c in range((sg.n + LC - 1) // LC)]
            d["lin_chunks"] = (torch.tensor(chunks, dtype=torch.int32).to(dev), torch.tensor(first, dtype=torch.int32).to(dev))
        chunks, first = d["lin_chunks"]
        nch = chunks.shape[0]
        ws_u = scratch("lin_ws_u", nch * H * D * V, torch.float32, dev)
        ws_d = scratch("lin_ws_d", nch * H * D, torch.float32, dev)
        check(lib().spark_linear_chunked(*args(longs[0]), len(longs[1]), P(chunks), nch, P(first), P(ws_u), P(ws_d), stream()),
              "spark_linear_chunked")
    return o


# ----------------------------------------------------------------------------- latent attention
def _short_long(plan, dev):
    """Rows of segments below CHUNK_MIN_ROWS as an int32 row list (None = every row) and the table of the other segments
    with their offsets in the gathered context: (rows or None, count, table [n, 5], segments, gathered rows)."""
    d = cu._plan_dev(plan, dev)
    if "latent_split" not in d:
        longs = [s for s in plan.segs if s.n >= CHUNK_MIN_ROWS]
        if not longs:
            d["latent_split"] = (None, plan.rows, None, [], 0)
        else:
            rows = [r for s in plan.segs if s.n < CHUNK_MIN_ROWS for r in range(s.r0, s.r0 + s.n)]
            tab, off = [], 0
            for s in longs:
                tab.append([s.slot, s.r0, s.n, s.pos0, off])
                off += s.pos0 + s.n
            d["latent_split"] = (torch.tensor(rows, dtype=torch.int32).to(dev) if rows else None, len(rows),
                                 torch.tensor(tab, dtype=torch.int32).to(dev), longs, off)
    return d["latent_split"]


def _max_ctx(plan, d):
    if "max_ctx" not in d:
        d["max_ctx"] = max(s.pos0 + s.n for s in plan.segs)
    return d["max_ctx"]


def _heads_product(x, ldx, xh, w, y, ldy, yh, R, gate=None, rows=None):
    """y[r, h] = x[r, h] w[h]^T over heads: x at r * ldx + h * xh, w [H, N, K], y at r * ldy + h * yh.  `gate` [plan rows, H * N]:
    outputs times its sigmoid (row r's gate is row rows[r], or r)."""
    H, N, K = w.shape

    def act(r):
        if gate is None:
            return None
        return cu.out_act("gate", gate[r:] if rows is None else gate, rows[r:] if rows is not None else None, batch_cols=N)
    if w.dtype == torch.float32 or R > 64 or K % 8 or xh % 8 or ldx % 8 or x.data_ptr() % 16:
        return cu.gemm_simt(x, ldx, xh, w, K, N * K, y, ldy, yh, H, R, N, K, act(0))
    step = min(16, cu.gemv_rows(K))
    for r in range(0, R, step):                         # every head's matrix is streamed once per 16 rows
        cu.gemv_bf16_items(x[r:], ldx, xh, w, N * K, K, y[r:], ldy, yh, H, min(step, R - r), N, K, _iota(H, x.device), act(r))
    return y


def latent_mixer(mx, proj, plan, cat):
    """Latent attention of every row of `proj` (columns: mx.off), per-head outputs into cat[:, :H * V] (gated)."""
    c, w, dev, dt = mx.c, mx.w, proj.device, proj.dtype
    d = cu._plan_dev(plan, dev)
    R, H, D, V = proj.shape[0], c.n_heads, c.head_dim, c.v_dim
    Dp, Rp, Vp, Lp, KW = mx.Dp, mx.Rp, mx.Vp, mx.Lp, mx.Lp + mx.Rp
    pages, pld = mx.pages, mx.pages.shape[1]
    is32 = _is32(dt)
    if not hasattr(mx, "_inv"):
        mx._inv = (c.rope_theta ** (-torch.arange(c.rope_dim // 2, dtype=torch.float64) * 2 / c.rope_dim)).to(dev)
    cq = torch.empty(R, w["uq"].shape[1], dtype=dt, device=dev) if c.q_rank else None
    check(lib().spark_latent_prep(P(proj), proj.stride(0), mx.off["dq"], mx.off["lat"], mx.off["rot"], R, c.q_rank, cq.shape[1] if c.q_rank else 0,
                                  c.kv_rank, Lp, c.rope_dim, Rp, int(c.rope_interleaved), float(mx.eps), P(w.get("dq_norm")), P(w["kv_norm"]),
                                  P(mx._inv), P(d["pos32"]), P(d["row_slot"]), P(pages), pld, P(cq), P(mx.lat), is32, P(status_word(dev)),
                                  stream()), "spark_latent_prep")
    q = cu.dense_linear(cq, w["uq"]) if c.q_rank else proj[:, : mx.nq]       # [R, H * (Dp + Rp)]
    gate = proj[:, mx.off["g"]:]
    each = gate if c.gate == "element" else None
    sink = w["sink"] if c.sink else None
    rows, ns, tab, longs, ctx = (None, R, None, [], 0) if is32 else _short_long(plan, dev)
    if longs and not mx.prefill_ok:
        rows, ns, longs = None, R, []
    if ns:
        qs = q if rows is None else cu.gather_rows(q, rows)
        o = _latent_absorbed(mx, qs, rows, ns, gate if each is None else None, sink, d, plan, is32)
        dst = cat if rows is None else torch.empty(ns, H * V, dtype=dt, device=dev)
        _heads_product(o, H * Lp, Lp, w["uv"], dst, dst.stride(0), V, ns, each, rows)
        if rows is not None:
            cat[:, : H * V].index_copy_(0, rows.long(), dst)
    if longs:
        lat = scratch("latent_ctx", ctx * KW, torch.bfloat16, dev)[: ctx * KW].view(ctx, KW)
        check(lib().spark_latent_gather(P(mx.lat), KW * 2, P(tab), len(longs), max(s.pos0 + s.n for s in longs), P(pages), pld, P(lat),
                                        stream()), "spark_latent_gather")
        kv = cu.dense_linear(lat[:, :Lp], w["kv_up"])
        qr = q[:, Dp:]
        check(lib().spark_latent_qrope(P(qr), q.stride(0), Dp + Rp, P(qr), q.stride(0), Dp + Rp, R, H, c.rope_dim, Rp,
                                       int(c.rope_interleaved), P(mx._inv), P(d["pos32"]), None, 0, 0, stream()), "spark_latent_qrope")
        check(lib().spark_latent_prefill(P(q), q.stride(0), P(kv), kv.stride(0), P(lat), KW, P(tab), len(longs), max(s.n for s in longs),
                                         H, Dp, Rp, V, Vp, Lp, float(c.scale), P(gate), proj.stride(0), int(each is not None), P(sink), P(cat),
                                         cat.stride(0), stream()), "spark_latent_prefill")
    return cat


def _latent_absorbed(mx, q, rows, n, gate, sink, d, plan, is32):
    """Absorbed attention rows [n, H, Lp] (gated per head if `gate`): q [n, H * (Dp + Rp)] before rotation."""
    ldg = gate.stride(0) if gate is not None else 0
    c, w, dev = mx.c, mx.w, q.device
    H, Dp, Rp, Lp = c.n_heads, mx.Dp, mx.Rp, mx.Lp
    KW = Lp + Rp
    pages, pld = mx.pages, mx.pages.shape[1]
    qf = torch.empty(n, H * KW, dtype=q.dtype, device=dev)
    _heads_product(q, q.stride(0), Dp + Rp, w["uk_t"], qf, H * KW, KW, n)
    qr, qt = q[:, Dp:], qf[:, Lp:]
    check(lib().spark_latent_qrope(P(qr), q.stride(0), Dp + Rp, P(qt), H * KW, KW, n, H, c.rope_dim, Rp, int(c.rope_interleaved),
                                   P(mx._inv), P(d["pos32"]), P(rows), 1, is32, stream()), "spark_latent_qrope")
    o = torch.empty(n, H * Lp, dtype=q.dtype, device=dev)
    if is32 or not mx.decode_tc_ok:
        check(lib().spark_latent_rows(P(qf), P(mx.lat), P(d["pos32"]), P(rows), P(d["row_slot"]), P(pages), pld, n, H, Lp, Rp, float(c.scale),
                                      P(gate), ldg, P(sink), P(o), is32, stream()), "spark_latent_rows")
        return o
    nsplit = (_max_ctx(plan, d) + 63) // 64
    step = n if n <= 16 else 16                            # bounds the partial results of long contexts
    part_o = scratch("latent_part_o", step * H * nsplit * Lp, torch.float32, dev)
    part_ml = scratch("latent_part_ml", step * H * nsplit * 2, torch.float32, dev)
    if rows is None and n > step:
        rows = _iota(n, dev)
    for r in range(0, n, step):
        m = min(step, n - r)
        check(lib().spark_mla_attn_paged(P(qf[r:]), P(mx.lat), P(d["pos32"]), P(rows[r:]) if rows is not None else None, P(d["row_slot"]),
                                         P(pages), pld, P(part_o), P(part_ml), nsplit, m, H, Lp, Rp, float(c.scale), P(gate), ldg,
                                         P(sink), P(o[r:]), stream()), "spark_mla_attn_paged")
    return o
