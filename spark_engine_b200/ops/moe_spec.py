"""Routed feed-forwards of models whose layers carry their own sizes (dense bf16 weights, or fp32 in the 32-bit mode): experts with
one up matrix and a squared relu, or gated experts (SwiGLU, or with a limit, a slope of the sigmoid and a shift of the up half) whose
input or output is multiplied by the routing weight; identity experts, a shared expert with or without a gate.  Routing, sorting and the products are the engine's MoE kernels: decode rows take the fused router
and one GEMV item per (row, expert) pair, prompts the grouped tcgen05 GEMM over the sorted pairs, the 32-bit mode (and widths
that are no multiple of 8) the grouped FP32-unit product.  Activation and input weight are part of the products (the experts
have no biases, so weighting the input is weighting gate and up); the combine (slot order, identity weight times the input row,
shared expert) runs inside the residual update (`PendingMoe`)."""
from __future__ import annotations

import torch

from . import cuda as cu
from .cuda import P, check, lib, scratch, stream
from .parallel_block import add_norm_rows, linear_swiglu, swiglu_rows


def _route(h, w, c, self_w):
    """(weights, expert ids with -1 for identity, source rows, shared gate)."""
    R, H = h.shape
    dev, gate = h.device, w["gate"]
    if R > cu.DECODE_ROWS_MAX or R * c.top_k > cu.DECODE_PAIRS_MAX or h.dtype != torch.bfloat16 or H % 8 or R * H * 2 > 200 * 1024:
        return cu.moe_route(h, w, c, self_w=self_w)
    ld = (gate.shape[0] + 7) // 8 * 8
    logits = scratch("router_logits", cu.DECODE_ROWS_MAX * ld, torch.float32, dev)
    counter = scratch("router_counter", 4, torch.int32, dev, zero=True)
    wts = torch.empty(R, c.top_k, dtype=torch.float32, device=dev)
    ids = torch.empty(R, c.top_k, dtype=torch.int32, device=dev)
    prow = torch.empty(R, c.top_k, dtype=torch.int32, device=dev)
    sg = torch.empty(R, dtype=torch.float32, device=dev) if c.shared_gate else None
    check(lib().spark_moe_router_topk(P(h), h.stride(0), P(gate), gate.stride(0), P(logits), ld, R, H, c.n_routes, c.top_k,
                                      cu.ROUTER_KIND[c.router], P(w.get("bias")), float(c.route_scale), int(c.shared_gate), c.top_k, 0, 0,
                                      c.n_experts, 0, 1, P(wts), P(ids), P(prow), P(sg), P(counter), c.n_identity, P(self_w), stream()),
          "spark_moe_router_topk")
    return wts, ids, prow, sg


def _shared(h, w, c):
    if c.act == "relu2":
        return cu.dense_linear(cu.dense_linear(h, w["s_up"], act=cu.out_act("relu2")), w["s_down"], out_f32=True)
    return cu.dense_linear(linear_swiglu(h, w["s_gu"], c.glu), w["s_down"], out_f32=True)


def _grouped_simt(h, w, c, wts, perm, tiles, ntile, max_tiles):
    """Sorted pairs on the FP32 units; the up product gathers its rows itself.  `wts`: input weights of the pairs."""
    relu2 = c.act == "relu2"
    wu, wd = w["w_up" if relu2 else "w_gu"], w["w_down"]
    E, Nu, H = wu.shape
    Fp = wd.shape[2]
    Pn, f32 = perm.numel(), int(h.dtype == torch.float32)
    act = torch.empty(Pn, Nu, dtype=h.dtype, device=h.device)
    y = torch.empty(Pn, H, dtype=torch.float32, device=h.device)
    oact = cu.out_act("relu2") if relu2 else None
    check(lib().spark_gemm_simt_grouped(P(h), H, P(wu), H, Nu * H, P(act), Nu, Nu, H, P(tiles), P(ntile), max_tiles, P(perm), c.top_k,
                                        f32, f32, cu._act(oact), stream()), "spark_gemm_simt_grouped")
    if not relu2:
        act = swiglu_rows(act, wts, perm, c.glu)
    check(lib().spark_gemm_simt_grouped(P(act), Fp, P(wd), Fp, H * Fp, P(y), H, H, Fp, P(tiles), P(ntile), max_tiles, None, 1, f32, 1, None,
                                        stream()), "spark_gemm_simt_grouped")
    return y


def moe(h, w, c, defer: bool = False):
    """Block output of every row: a `PendingMoe` (`defer`) or its fp32 tensor."""
    relu2 = c.act == "relu2"
    wu, wd = w["w_up" if relu2 else "w_gu"], w["w_down"]
    h = h.to(wu.dtype).contiguous()
    R, H = h.shape
    E, Nu, _ = wu.shape
    Fp = wd.shape[2]
    dev = h.device
    simt = h.dtype != torch.bfloat16 or H % 8 != 0
    pairs = not simt and R <= cu.DECODE_ROWS_MAX and R * c.top_k <= cu.DECODE_PAIRS_MAX
    self_w = torch.empty(R, dtype=torch.float32, device=dev) if c.n_identity else None
    side = shared = None
    if c.n_shared:
        # decode rows: the shared expert does not depend on the router, so it runs on a side stream next to it (a captured graph
        # keeps the fork)
        main = torch.cuda.current_stream()
        side = cu._side_stream(dev) if cu.SIDE_STREAMS and pairs else None
        if side is not None:
            side.wait_stream(main)
        with torch.cuda.stream(side if side is not None else main):
            shared = _shared(h, w, c)
    wts, ids, prow, sg = _route(h, w, c, self_w)
    inv, xw = None, wts if c.weight_input else None
    if pairs:
        n, pe = R * c.top_k, ids.view(-1)
        a = cu.gemv_bf16(h, wu, items=n, rows_per_item=1, pair_expert=pe, pair_row=prow.view(-1), expert_stride=Nu * H, n=Nu, k=H,
                         oact=cu.out_act("relu2") if relu2 else None)
        y = cu.gemv_bf16(a, wd, items=n, rows_per_item=1, pair_expert=pe, act=0 if relu2 else 1, limit=c.glu, out_f32=True, expert_stride=H * Fp, n=H,
                         k=Fp, x_weight=xw)
    else:
        perm, inv, _, tiles, ntile, max_tiles = cu.moe_sort(ids.view(-1), E)
        if simt:
            y = _grouped_simt(h, w, c, xw, perm, tiles, ntile, max_tiles)
        else:
            a = cu.gather_rows(h, torch.div(perm, c.top_k, rounding_mode="floor").to(torch.int32))
            a = cu.grouped_gemm(a, wu.view(E * Nu, H), tiles, ntile, max_tiles, E, Nu, Fp, 2 if relu2 else 1, c.glu, wts=xw, perm=perm)
            y = cu.grouped_gemm(a, wd.view(E * H, Fp), tiles, ntile, max_tiles, E, H, H, 0)
    if side is not None:
        torch.cuda.current_stream().wait_stream(side)
    pm = cu.PendingMoe(y, None if c.weight_input else wts, ids, c.top_k, R, H, shared, sg, inv, self_w, h if self_w is not None else None)
    if defer:
        return pm
    return add_norm_rows(pm, torch.zeros(R, H, dtype=torch.float32, device=dev), None, h.dtype)[1]
