"""Operator layer: one Python entry point per op; the sm_100a kernels run on a B200, plain PyTorch
runs on CPU (fp32 plumbing and oracle tests).

On a CUDA device the kernel library MUST be present: an op whose kernel is missing raises instead of
silently running an eager fallback (set SPARK_ALLOW_TORCH_FALLBACK=1 to run the PyTorch/ATen
baseline path on purpose, e.g. for A/B timing against the library path).
"""
from __future__ import annotations

import math
import os
from typing import Optional

import torch
import torch.nn.functional as F

from ..oracle import layers as L
from ..quant.formats import QuantWeight

_FALLBACK = os.environ.get("SPARK_ALLOW_TORCH_FALLBACK", "0") == "1"
_cuda_ops = None


def cuda_ops():
    """The kernel bindings (loaded on first use on a CUDA device)."""
    global _cuda_ops
    if _cuda_ops is None:
        from . import cuda as _c
        _cuda_ops = _c
    return _cuda_ops


def block_ops():
    """The parallel-block bindings."""
    from . import parallel_block
    return parallel_block


def use_kernels(t: torch.Tensor) -> bool:
    return t.is_cuda and not _FALLBACK


def set_fallback(on: bool):
    """Route CUDA tensors through PyTorch/ATen ops (the library baseline) instead of the kernels."""
    global _FALLBACK
    _FALLBACK = on


# ----------------------------------------------------------------------------- basic ops
def embed(table: torch.Tensor, ids: torch.Tensor, dtype, scale: float = 1.0, pos=None, out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Token embedding rows (times `scale`), into `out` if given.  `pos` = (positions, angle per position of every channel pair): the
    sines (even channels) and cosines (odd ones) of the row's position are added.  On the device the residual stream is fp32
    (activations bf16)."""
    if use_kernels(table):
        if scale != 1.0 or table.dtype == torch.float32 or pos is not None or out is not None:
            return block_ops().embed_scaled(table, ids.to(torch.int32), scale, pos, out)
        return cuda_ops().embed(table, ids.to(torch.int32))
    x = table[ids].to(dtype)
    if scale != 1.0:
        x = x * scale
    if pos is not None:
        a = (pos[0].double().unsqueeze(1) * pos[1]).to(x.dtype)
        x = x + torch.stack((a.sin(), a.cos()), -1).flatten(1)[:, : x.shape[1]]
    return x if out is None else out.copy_(x)


def to_tensor(x):
    """Plain tensor of a block output that may still be deferred (uncombined MoE of a decode round, row-parallel
    product)."""
    if x is None or isinstance(x, torch.Tensor):
        return x
    if isinstance(x, Partial):
        return linear(x.x, x.w)
    return x.tensor()


def residual_add(res, delta) -> torch.Tensor:
    if isinstance(delta, Update):
        return add_norm_rows(delta, res, None, res.dtype)[1]
    res, delta = to_tensor(res), to_tensor(delta)
    if use_kernels(res) and res.dtype == torch.float32 and res.dim() == 2:
        return cuda_ops().residual_add(res, delta)
    return res + delta.to(res.dtype)


def argmax(logits: torch.Tensor) -> torch.Tensor:
    """Greedy token per row (ties -> lowest id), int32."""
    if use_kernels(logits):
        return cuda_ops().argmax(logits)
    return torch.argmax(logits, -1).to(torch.int32)


def gumbel_perturb(logits: torch.Tensor, temps, seeds, positions, offset: int, vocab: int) -> torch.Tensor:
    """fp32 logits [R, V_local] of vocabulary ids [offset, offset + V_local): rows with temperature > 0 become
    logits / T + g(seed, position, global id); greedy rows are returned unchanged.  The arg-max of the result (over
    all ranks' slices) is the sampled token.  temps/seeds/positions are Python sequences of length R."""
    if not any(t > 0 for t in temps):
        return logits
    x = logits.float() if logits.dtype != torch.float32 else logits.clone()
    if use_kernels(x):
        dev = x.device
        t = torch.tensor(list(temps), dtype=torch.float32).to(dev, non_blocking=True)
        sd = torch.tensor([int(v) for v in seeds], dtype=torch.int64).to(dev, non_blocking=True)
        ps = torch.tensor([int(v) for v in positions], dtype=torch.int64).to(dev, non_blocking=True)
        return cuda_ops().gumbel_perturb(x.contiguous(), t, sd, ps, offset)
    from ..spec.sampling import gumbel_noise_ref
    V = x.shape[1]
    for r, T in enumerate(temps):
        if T > 0:
            x[r] = x[r] / T + gumbel_noise_ref(int(seeds[r]), int(positions[r]), vocab, x.device)[offset: offset + V]
    return x


def lm_head(h, w) -> torch.Tensor:
    """Logits in fp32."""
    if use_kernels(h) and not isinstance(w, QuantWeight):
        return cuda_ops().dense_linear(h, w, out_f32=True)
    return linear(h, w).float()


def linear(x: torch.Tensor, w, out_f32: bool = False) -> torch.Tensor:
    """y = x @ W^T for a dense `[N,K]` tensor or a quantised weight object (`out_f32`: dense weights only)."""
    if out_f32:
        return cuda_ops().dense_linear(x, w, out_f32=True) if use_kernels(x) else (x @ w.to(x.dtype).t()).float()
    if isinstance(w, QuantWeight):
        if use_kernels(x):
            return cuda_ops().quant_linear(x, w)
        return (x.float() @ w.dequant().to(x.device).t()).to(x.dtype)
    if use_kernels(x):
        return cuda_ops().dense_linear(x, w)
    return x @ w.to(x.dtype).t()


def linear_relu2(x: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """max(x W^T, 0)^2 (the activation is the product's epilogue)."""
    if use_kernels(x):
        c = cuda_ops()
        return c.dense_linear(x, w, act=c.out_act("relu2"))
    return relu2(x @ w.to(x.dtype).t())


def linear_swiglu(x: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """silu(x G^T) * (x U^T) for w = [G | U] stacked."""
    if use_kernels(x):
        return block_ops().linear_swiglu(x, w)
    gu = x @ w.to(x.dtype).t()
    n = gu.shape[1] // 2
    return L.swiglu(gu[:, :n].float(), gu[:, n:].float()).to(x.dtype)


def linear_token_gate(x: torch.Tensor, w: torch.Tensor, table: torch.Tensor, ids: torch.Tensor, off: int, n: int) -> torch.Tensor:
    """gelu_tanh(x W^T) * table[ids, off : off + n] (columns from n on are zero; ids outside the table give zero rows)."""
    if use_kernels(x):
        c = cuda_ops()
        return c.dense_linear(x, w, act=c.out_act("token_gate", table, ids.to(torch.int32), off, n))
    y = gelu_tanh(x @ w.to(x.dtype).t())
    y[:, n:] = 0
    inside = (ids >= 0) & (ids < table.shape[0])
    e = table[torch.where(inside, ids, torch.zeros_like(ids))][:, off: off + n].float() * inside.unsqueeze(1)
    y[:, :n] *= e
    return y.to(x.dtype)


def linear_pair(x, w_a, w_b):
    """Two independent projections of the same rows.  On the device, decode-size batches run the second one on a
    side stream next to the first (parallel branches of the captured graph)."""
    if use_kernels(x) and x.shape[0] <= 16 and cuda_ops().SIDE_STREAMS:
        c = cuda_ops()
        main = torch.cuda.current_stream()
        side = c._side_stream(x.device)
        side.wait_stream(main)
        with torch.cuda.stream(side):
            b = linear(x, w_b)
        a = linear(x, w_a)
        main.wait_stream(side)
        return a, b
    return linear(x, w_a), linear(x, w_b)


def rmsnorm(x, w, eps):
    x = to_tensor(x)
    if use_kernels(x):
        return cuda_ops().rmsnorm(x, w, eps)
    return L.rms(x.float(), w.float(), eps).to(x.dtype)


class Partial:
    """A row-parallel product x @ W_shard^T that has not been computed yet: under tensor parallelism the
    GEMV, the all-reduce, the residual add and the next RMSNorm run as one kernel."""

    def __init__(self, x, w):
        self.x, self.w = x, w


def row_parallel(x, w, tp=None):
    """Output projection of a mixer.  Without tensor parallelism: the product.  With it: this rank's partial
    product, deferred when the fused GEMV + all-reduce kernel can take it (EXL3 weights, <= 16 rows)."""
    if tp is not None and tp.can_fuse_gemv(x, w):
        return Partial(x, w)
    return linear(x, w)


def add_rmsnorm(delta, res, w, eps, tp=None):
    """res' = res + delta (delta may be None); returns (rmsnorm(res') * w, res').  With `tp`, delta is this
    rank's partial sum and is all-reduced first (one fused kernel on the device)."""
    if tp is not None and delta is not None:
        return tp.add_rmsnorm(delta, res, w, eps)
    if use_kernels(res):
        return cuda_ops().add_rmsnorm(delta, res, w, eps)
    delta = to_tensor(delta)
    if delta is not None:
        res = res + delta
    return L.rms(res.float(), w.float(), eps).to(res.dtype), res


def swiglu(gu: torch.Tensor, limit: float = 0.0) -> torch.Tensor:
    """gu = [gate | up] halves along the last axis."""
    if use_kernels(gu):
        return cuda_ops().swiglu(gu, limit)
    F_ = gu.shape[-1] // 2
    return L.swiglu(gu[..., :F_].float(), gu[..., F_:].float(), limit).to(gu.dtype)


# ----------------------------------------------------------------------------- MoE
def route(h, w, c):
    """Router: returns (weights [R,k] fp32, expert ids [R,k] int64, shared gate [R,1] or None)."""
    logits = linear(h, w["gate"]).float()
    sg = None
    if c.shared_gate:
        sg = torch.sigmoid(logits[:, c.n_routes:])
        logits = logits[:, : c.n_routes]
    if c.router == "topk_softmax":
        z = logits + w["bias"].float().to(logits.device) if "bias" in w else logits
        idx = torch.sort(z, dim=-1, descending=True, stable=True).indices[:, : c.top_k]
        return torch.softmax(torch.gather(z, 1, idx), -1) * c.route_scale, idx, sg
    if c.router in ("softmax", "softmax_bias"):
        p = torch.softmax(logits, -1)
        sel = p if c.router == "softmax" else p + w["bias"].float().to(p.device)
    elif c.router == "sigmoid":
        idx = torch.sort(logits, dim=-1, descending=True, stable=True).indices[:, : c.top_k]
        return torch.sigmoid(torch.gather(logits, 1, idx)) * c.route_scale, idx, sg
    elif c.router == "sigmoid_bias":
        p = torch.sigmoid(logits)
        sel = p + w["bias"].float().to(p.device)
    else:
        p = torch.sqrt(F.softplus(logits))
        sel = p + w["bias"].float().to(p.device)
    idx = torch.sort(sel, dim=-1, descending=True, stable=True).indices[:, : c.top_k]
    wts = torch.gather(p, 1, idx)
    wts = wts / wts.sum(-1, keepdim=True).clamp_min(1e-20) * c.route_scale
    return wts, idx, sg


def moe(h, w, c, defer: bool = False):
    """Routed experts (slot-order weighted sum) + shared expert.  `defer` (decode rounds on the device): the
    uncombined expert outputs are returned and the combine runs fused with the next residual update."""
    if use_kernels(h):
        return cuda_ops().moe(h, w, c, defer)
    R = h.shape[0]
    wts, idx, sg = route(h, w, c)
    out = torch.zeros(R, h.shape[1], dtype=torch.float32, device=h.device)
    hf = h.float()
    single = c.act == "relu2"                    # one up matrix instead of [gate | up]
    wgu, wd = w["w_up" if single else "w_gu"], w["w_down"]
    lo, hi = w.get("ep", (0, c.n_experts))       # expert-parallel rank: only its own experts, partial output
    for slot in range(c.top_k):
        for e in idx[:, slot].unique().tolist():
            if not lo <= e < hi:
                continue
            rows = (idx[:, slot] == e).nonzero(as_tuple=True)[0]
            a = wts[rows, slot].unsqueeze(1)
            gu = (hf[rows] * a if c.weight_input else hf[rows]) @ _expert(wgu, e - lo).t()
            n = gu.shape[1] // 2
            y = (relu2(gu) if single else L.swiglu(gu[:, :n], gu[:, n:], *c.glu)) @ _expert(wd, e - lo).t()
            out[rows] += y if c.weight_input else a * y
    if c.n_identity:
        out += (wts * (idx >= c.n_experts)).sum(-1, keepdim=True) * hf
    if "s_up" in w:
        sh = linear(relu2(linear(h, w["s_up"])), w["s_down"]).float()
        out = out + (sg * sh if sg is not None else sh)
    elif "s_gu" in w:
        gu = linear(h, w["s_gu"]).float()
        Fs = gu.shape[1] // 2
        sh = linear(L.swiglu(gu[:, :Fs], gu[:, Fs:], *c.glu).to(h.dtype), w["s_down"]).float()
        out = out + (sg * sh if sg is not None else sh)
    return out.to(h.dtype)


def _expert(w, e):
    if isinstance(w, QuantWeight):
        return w.dequant_expert(e)
    return w[e].float()


# ----------------------------------------------------------------------------- mixers (fast paths)
def gdn_mixer(mixer, proj, ab, plan, commit) -> Optional[torch.Tensor]:
    if use_kernels(proj):
        return cuda_ops().gdn_mixer(mixer, proj, ab, plan, commit)
    return None


def gdn_commit(mixer, proj, ab, plan, accepted) -> bool:
    if use_kernels(proj):
        return cuda_ops().gdn_commit(mixer, proj, ab, plan, accepted)
    return False


def kda_mixer(mixer, pre, lr, plan, commit) -> Optional[torch.Tensor]:
    if use_kernels(pre):
        return cuda_ops().kda_mixer(mixer, pre, lr, plan, commit)
    return None


def kda_commit(mixer, pre, lr, plan, accepted) -> bool:
    if use_kernels(pre):
        return cuda_ops().kda_commit(mixer, pre, lr, plan, accepted)
    return False


def mla_mixer(mixer, h, plan, seqs) -> Optional[torch.Tensor]:
    if use_kernels(h):
        return cuda_ops().mla_mixer(mixer, h, plan, seqs)
    return None


def attn_mixer(mixer, qkv, plan, seqs) -> Optional[torch.Tensor]:
    if use_kernels(qkv):
        return cuda_ops().attn_mixer(mixer, qkv, plan, seqs)
    return None


# ----------------------------------------------------------------------------- hyper-connections
def _reduced(x, tp):
    """Block output as a plain tensor; under tensor parallelism this rank's partial sum is all-reduced first."""
    if x is None:
        return None
    if tp is not None:
        return tp.reduce(x)
    return to_tensor(x)


def hc_gated_site(X, pend, w, eps, tp=None):
    """Gated hyper-connection site.  `pend` = (block output, post) of the previous site, applied to the streams first:
    X[:, s] += post[:, s] * x.  Returns (X, mixed row h, hidden copy in fp32 or None, post for this site's block)."""
    if pend is not None:
        pend = (_reduced(pend[0], tp), pend[1])
    if use_kernels(X) and X.shape[1] == 4 and w["down"].shape[0] == 32 and X.dtype == torch.float32:
        return cuda_ops().hc_gated_site(X, pend, w, eps)
    if pend is not None:
        X = X + pend[1].unsqueeze(-1).to(X.dtype) * pend[0].to(X.dtype).unsqueeze(1)
    post, mixed = L.hc_gated_mix(X.float(), {k: v.float() for k, v in w.items() if torch.is_tensor(v)}, eps)
    return X, mixed.to(X.dtype), None, post


def mhc_site(X, pend, w, iters, eps, tp=None):
    """mHC site.  `pend` = (block output, post, comb) of the previous site, applied first.  Returns (X, h, post, comb)."""
    if pend is not None:
        pend = (_reduced(pend[0], tp),) + tuple(pend[1:])
    if use_kernels(X) and X.shape[1] == 4 and X.dtype == torch.float32:
        return cuda_ops().mhc_site(X, pend, w, iters, eps)
    if pend is not None:
        X = L.mhc_post(X.float(), pend[0].float(), pend[1], pend[2]).to(X.dtype)
    h, post, comb = L.mhc_pre(X.float(), {k: v.float() for k, v in w.items() if torch.is_tensor(v)}, iters, eps)
    return X, h.to(X.dtype), post, comb


def mhc_final(X, pend, norm_w, eps, tp=None):
    """Last update, then the mean over streams and its RMSNorm.  Returns (hidden fp32-or-input dtype [T,D], normed row)."""
    if pend is not None:
        pend = (_reduced(pend[0], tp),) + tuple(pend[1:])
    if use_kernels(X) and X.shape[1] == 4 and X.dtype == torch.float32:
        _, h, mean = cuda_ops().mhc_site(X, pend, None, 0, eps, mode=2, norm=norm_w)
        return mean, h
    if pend is not None:
        X = L.mhc_post(X.float(), pend[0].float(), pend[1], pend[2]).to(X.dtype)
    m = X.mean(1)
    return m, rmsnorm(m, norm_w, eps)


def ngram_embed(model, X, plan, w):
    """Hashed n-gram rows need the token history of each sequence: the model keeps it per slot."""
    from ..models.ngram import ngram_rows_for_plan
    cfg = model.cfg
    emb = ngram_rows_for_plan(model, plan)                   # [R, heads*dim] fp32 on X.device
    if use_kernels(X):                                       # the two projections on the GEMV / tcgen05 GEMM kernels
        eb = emb.to(torch.bfloat16)
        key_raw = linear(eb, w["key"]).float()
        val = linear(eb, w["value"]).float()
    else:
        key_raw = emb @ w["key"].float().t()
        val = emb @ w["value"].float().t()
    if use_kernels(X) and X.dtype == torch.float32 and X.dim() == 2:
        return cuda_ops().ngram_gate(X.contiguous(), key_raw, val, w["norm_k"], w["norm_q"], cfg.norm_eps)
    key = L.rms(key_raw, w["norm_k"].float(), cfg.norm_eps)
    d = (key * L.rms(X.float(), w["norm_q"].float(), cfg.norm_eps)).sum(-1, keepdim=True) / math.sqrt(X.shape[-1])
    gate = torch.sigmoid(torch.sign(d) * torch.sqrt(d.abs().clamp_min(cfg.norm_eps)))
    return (X.float() + gate * val).to(X.dtype)


# ----------------------------------------------------------------------------- residual updates of models with layer specs
class RowNorm:
    """RMS norm (weight w or 1 + w) over each of `groups` equal parts of the row, or with a bias vector a layer norm."""

    def __init__(self, w, eps: float, b=None, one_plus: bool = False, groups: int = 1):
        assert b is None or groups == 1
        self.w, self.eps, self.b, self.one_plus, self.groups = w, eps, b, one_plus, groups

    def plain(self, x):
        if self.groups > 1:
            y = L.rms(x.view(*x.shape[:-1], self.groups, -1), None, self.eps).view(x.shape)
            return y * (1 + self.w if self.one_plus else self.w)
        return L.rms(x, self.w.float(), self.eps, self.one_plus) if self.b is None else L.layer_norm(x, self.w, self.b, self.eps)


class DepthAverage:
    """Result number `k` of the layers: it is put into `stack` [results + 1, R, H] (0: the embedding), and the sum of a[j] * stack[j]
    over j <= k goes on in its place."""

    def __init__(self, stack, k: int, a):
        self.stack, self.k, self.a = stack, k, a

    def plain(self, x):
        self.stack[self.k] = x
        return torch.einsum("j,jrh->rh", self.a, self.stack[: self.k + 1])


class RowContext:
    """What a row update needs to know of its pass: the plan (an input convolution looks at the sequence's earlier rows), whether
    states advance, and whether the residual must be left as it is (`fresh`: the new one is another tensor)."""

    def __init__(self, plan, commit: bool = True, fresh: bool = False):
        self.plan, self.commit, self.fresh = plan, commit, fresh


class Update:
    """A block output on its way into the residual stream: `x` (a tensor, or a deferred MoE output), times the per-channel
    `scale`, or RMS-normed by `post` (a RowNorm) first; `depth`: a DepthAverage of the sum."""
    depth: Optional[DepthAverage] = None

    def __init__(self, x, scale=None, post: Optional[RowNorm] = None):
        self.x, self.scale, self.post = x, scale, post

    def plain(self):
        x = to_tensor(self.x).float()
        if self.post is not None:
            x = self.post.plain(x)
        return x * self.scale if self.scale is not None else x


def add_norm_rows(delta, res, norm: Optional[RowNorm], dtype, want_f32: bool = False, conv=None, ctx: Optional[RowContext] = None):
    """res' = res + delta (None, a tensor or an Update); returns (h = norm(res') in `dtype` (norm None: res' itself), res',
    fp32 h if asked).  `conv` (an InputConv): h + conv(h) over the sequences of `ctx.plan` instead of h."""
    if use_kernels(res):
        return block_ops().add_norm_rows(delta, res, norm, dtype, want_f32, conv, ctx)
    if delta is not None:
        res = res + (delta.plain() if isinstance(delta, Update) else delta)
        if isinstance(delta, Update) and delta.depth is not None:
            res = delta.depth.plain(res)
    h = res.float() if norm is None else norm.plain(res.float())
    if conv is not None:
        rows, h = h, h.clone()
        for s in ctx.plan.segs:
            y = rows[s.r0: s.r0 + s.n]
            h[s.r0: s.r0 + s.n] += L.causal_conv(y, conv.w.t(), tail=conv.tail[s.slot])
        if ctx.commit:
            advance_tail(conv.tail, rows, ctx.plan, None)
        conv.keep(rows, ctx.plan, ctx.commit)
    return h.to(dtype), res, h


def advance_tail(tail, rows, plan, n_rows):
    """The last rows of every segment's sequence behind n_rows[i] more rows (None: all of segment i's): `tail` [slots, kept, H]."""
    if use_kernels(tail):
        return block_ops().advance_tail(tail, rows, plan, n_rows)
    kept = tail.shape[1]
    for i, s in enumerate(plan.segs):
        n = s.n if n_rows is None else int(n_rows[i])
        tail[s.slot] = torch.cat((tail[s.slot], rows[s.r0: s.r0 + n]))[n: n + kept]


def relu2(x):
    return torch.relu(x).square()


def paged_gqa(mixer, proj, plan, commit, out=None):
    if use_kernels(proj):
        from . import paged_attn
        return paged_attn.mixer(mixer, proj, plan, commit, out)
    return None


def conv_tail(mixer, proj, plan, n_rows) -> bool:
    """Advance the convolution tails of the plan's slots by n_rows[i] rows of segment i."""
    if use_kernels(proj):
        from . import paged_attn
        paged_attn.commit_tail(mixer, proj, plan, n_rows)
        return True
    return False


# ----------------------------------------------------------------------------- parallel block
def gelu_tanh(x):
    return F.gelu(x.float(), approximate="tanh")


def gate_concat(o, n, group, w, eps, gate, kind, ff, width_ff, off, width, dtype, out=None):
    """Input row of a parallel block's output product: [ group-RMSNorm(o) * w * gate(g), padded to `off` | gelu(ff gate) *
    (ff up) ].  group 0 = no norm, kind = sigmoid | silu | None (no gate); o None = the mixer part is in `out` already."""
    src = o if o is not None else out
    if use_kernels(src):
        return block_ops().gate_concat(o, n, group, w, eps, gate, kind, ff, width_ff, off, width, dtype, out)
    R = src.shape[0]
    if out is None:
        out = torch.zeros(R, width, dtype=dtype)
    if o is not None:
        x = o.float()
        if group:
            x = x.view(R, n // group, group)
            x = (x * torch.rsqrt(x.pow(2).mean(-1, keepdim=True) + eps)).reshape(R, n)
        if w is not None:
            x = x * w
        if kind is not None:
            x = x * (torch.sigmoid(gate.float()) if kind == "sigmoid" else F.silu(gate.float()))
        out[:, :n] = x.to(dtype)
        out[:, n:off] = 0
    if ff is not None:
        up = width - off
        out[:, off: off + width_ff] = (gelu_tanh(ff[:, :width_ff]) * ff[:, up: up + width_ff].float()).to(dtype)
    return out


def token_shift(h32, carried, mu, plan, dtype):
    """[n, R, H]: for each mu row the mix h + (h' - h) mu of a row and its predecessor (the carried row of the slot for the
    first row of a segment)."""
    if use_kernels(h32):
        return block_ops().token_shift(h32, carried, mu, plan, dtype)
    prev = torch.empty_like(h32)
    for s in plan.segs:
        prev[s.r0] = carried[s.slot]
        prev[s.r0 + 1: s.r0 + s.n] = h32[s.r0: s.r0 + s.n - 1]
    return (h32 + (prev - h32) * mu.unsqueeze(1)).to(dtype)


def linear_stack(xs, w):
    """n independent products [n, R, K] x [n, N, K] -> [n, R, N]."""
    if use_kernels(xs):
        return block_ops().linear_stack(xs, w)
    return torch.einsum("nrk,nok->nro", xs, w.to(xs.dtype))


def channel_decay(z, w2, w0, n: int, w2x2=None):
    """log decay -exp(w2 tanh(z) + w0) [R, n] in fp32."""
    if use_kernels(z):
        return block_ops().channel_decay(z, w2, w0, n, w2x2)
    return -torch.exp(torch.tanh(z.float()) @ w2.float().t() + w0)


def log_sigmoid_decay(z, w2, b, n: int, tau: float):
    """ln(sigmoid(z w2^T + b)) / tau [R, n] in fp32: the log of sigmoid(..)^(1/tau)."""
    if use_kernels(z):
        return block_ops().log_sigmoid_decay(z, w2, b, n, tau)
    return F.logsigmoid(z.float() @ w2.float().t()[: z.shape[1]] + b) / tau


def linear_state(q, k, v, H, D, V, S, plan, commit, act=False, log2a=None, logw=None, u=None, h32=None, carried=None,
                 n_rows=None, qscale=1.0, low_rank=None):
    """Decayed linear attention (constant decay per head; or decay per channel and token, with a bonus `u` for the current
    token, or without one on the state after the current token): o fp32 [R, H * V], times `qscale`; the slots' states advance
    when `commit` (by n_rows[i] rows of segment i if given).  `low_rank` = (z, w2, b, tau): the channel decays are
    log_sigmoid_decay(z, w2, b, H * D, tau)."""
    if use_kernels(q):
        return block_ops().linear_state(q, k, v, H, D, V, S, plan, commit, act, log2a, logw, u, h32, carried, n_rows, qscale, low_rank)
    if low_rank is not None:
        logw = log_sigmoid_decay(*low_rank[:3], H * D, low_rank[3])
    R = q.shape[0]
    q, k, v = q.float().view(R, H, D), k.float().view(R, H, D), v.float().view(R, H, V)
    if act:
        q, k, v = F.silu(q), F.silu(k), F.silu(v)
    o = q.new_zeros(R, H, V)
    a = torch.exp2(log2a).view(H, 1, 1) if log2a is not None else None
    for i, s in enumerate(plan.segs):
        St = S[s.slot]
        n = s.n if n_rows is None else min(s.n, int(n_rows[i]))
        for r in range(s.r0, s.r0 + n):
            kv = k[r].unsqueeze(-1) * v[r].unsqueeze(-2)
            if a is not None or u is None:
                St = (a if a is not None else torch.exp(logw[r]).view(H, D, 1)) * St + kv
                o[r] = torch.einsum("hd,hdv->hv", q[r], St)
            else:
                o[r] = torch.einsum("hd,hdv->hv", q[r], St + u.view(H, D, 1) * kv)
                St = torch.exp(logw[r]).view(H, D, 1) * St + kv
        if commit and n:
            S[s.slot] = St
            if carried is not None:
                carried[s.slot] = h32[s.r0 + n - 1]
    return o.view(R, H * V) * qscale


def latent_mixer(mixer, proj, plan, cat):
    if use_kernels(proj):
        return block_ops().latent_mixer(mixer, proj, plan, cat)
    return None
