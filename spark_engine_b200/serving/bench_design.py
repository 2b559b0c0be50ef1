"""`bench.py --design NAME`: prefill and decode throughput of a design with random weights at a few layer sizes of real models,
beside the closest existing family at equal size, and the kernels of its mechanisms beside their like kernels as fractions of
the measured copy bandwidth / GEMM throughput.

  vabunex   beside KDA linear attention + latent attention in sequential pre-norm blocks with dense feed-forwards
  debisun   beside grouped-query attention (rotary, no chunks) with softmax-routed SwiGLU experts, as many parameters
  zapolorn  beside grouped-query attention (rotary, whole context) with dense and softmax-routed SwiGLU feed-forwards of its sizes
  zakusun   beside latent attention (low-rank queries, a rotated part) with softmax-routed SwiGLU experts of its sizes

Device-timed with CUDA events.  Model figures stream more weights and activations than L2 holds; kernel figures write a
buffer larger than L2 between iterations (median of the iterations)."""
from __future__ import annotations

import json
import os
import statistics

import torch

from ..config import AttnConfig, EngineConfig, KdaConfig, MlaConfig, ModelConfig, MoeConfig, debisun_style, glm_style, vabunex_style, \
    zakusun_style, zapolorn_style
from ..models.build import build_random_model, decode_step_bytes
from ..models.plan import make_plan
from ..ops import cuda as cu
from .engine import LLMEngine

DEV = "cuda"
SIZES = {"1024": (1024, 2816), "2048": (2048, 5632), "4096": (4096, 11264)}
VOCAB = 32768


def vabunex_config(hidden: int, ffn: int):
    return vabunex_style(12, hidden, ffn, VOCAB)


def closest_config(hidden: int, ffn: int, layers: int):
    """Same number of layer runs, heads, head sizes, latent sizes and feed-forward width."""
    c = glm_style(layers, "dense")
    c.name, c.hidden, c.vocab, c.mtp_layers = "kda + latent attention, dense", hidden, VOCAB, 0
    c.layer_types = ["mla" if i % 4 == 0 else "kda" for i in range(layers)]
    h = hidden // 128
    c.kda = KdaConfig(n_heads=h, head_dim=128, conv_k=4, gate_rank=64)
    c.mla = MlaConfig(n_heads=h, q_lora=768, kv_lora=512, head_dim=128, rope_dim=64, idx_heads=4, idx_dim=64, pool=4, topk_pools=1 << 20)
    c.moe.dense_layers, c.moe.dense_ffn, c.moe.swiglu_limit = layers, ffn, 0.0
    return c


def _timed(fn, n: int = 5, flush=None) -> float:
    """Median milliseconds of n runs after 3 warm-ups."""
    for _ in range(3):
        fn()
    ts = []
    for _ in range(n):
        if flush is not None:
            flush.zero_()
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        torch.cuda.synchronize()
        a.record()
        fn()
        b.record()
        torch.cuda.synchronize()
        ts.append(a.elapsed_time(b))
    return statistics.median(ts)


def model_figures(cfg, steps: int, warmup: int, prompts=(2048, 8192)) -> dict:
    W = build_random_model(cfg, DEV, seed=0)
    eng = LLMEngine(cfg, W, EngineConfig(prefill_chunk=8192), device=DEV, max_seqs=16, kv_tokens_per_seq=max(prompts) + 512)
    g = torch.Generator().manual_seed(0)
    ids = torch.randint(0, cfg.vocab, (max(prompts),), generator=g).tolist()
    out = {"prefill_tok_s": {}, "decode_tok_s": {}, "decode_ms_per_step": {}}
    for n in prompts:
        out["prefill_tok_s"][str(n)] = round(n / _timed(lambda: eng.prefill(0, ids[:n]), max(3, warmup)) * 1e3)
    for s in range(16):
        eng.prefill(s, ids[:1024])
    for n in (1, 4, 16):
        slots = list(range(n))
        cur = eng.decode_steps(slots, [1] * n, max(3, warmup))[-1]
        eng.decode_steps(slots, cur, 4)
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        torch.cuda.synchronize()
        a.record()
        eng.decode_steps(slots, cur, steps)
        b.record()
        torch.cuda.synchronize()
        ms = a.elapsed_time(b) / steps
        out["decode_ms_per_step"][str(n)] = round(ms, 4)
        out["decode_tok_s"][str(n)] = round(n * 1e3 / ms)
        if n == 4:
            out["decode_step_weight_bytes"] = decode_step_bytes(W, cfg, n)
    eng.check_device_status()
    return out


class Figures:
    """Kernel times as fractions of their roofline (bytes over the copy bandwidth or flops over the GEMM throughput)."""

    def __init__(self, peaks: dict):
        self.hbm, self.tf = peaks.get("hbm_gbs", 6650.0) * 1e6, peaks.get("bf16_tflops", 1590.0) * 1e9    # bytes, flops per millisecond
        self.flush = torch.empty(512 << 20, dtype=torch.uint8, device=DEV)
        self.g = torch.Generator(device=DEV).manual_seed(0)
        self.out, self.frac = {}, {}

    def rnd(self, *s):
        return torch.randn(*s, device=DEV, generator=self.g)

    def put(self, name, like, fn, nbytes=0, flops=0):
        if name.endswith("decode"):              # short kernels: replayed from a graph, no host time between launches
            fn()
            torch.cuda.synchronize()
            graph = torch.cuda.CUDAGraph()
            with torch.cuda.graph(graph):
                fn()
            fn = graph.replay
        ms = _timed(fn, 7, self.flush)
        roof = max(nbytes / self.hbm, flops / self.tf)
        self.frac[name] = roof / ms
        self.out[name] = {"us": round(ms * 1e3, 1), "of_roofline": round(roof / ms, 4),
                          "bound": "bytes" if nbytes / self.hbm >= flops / self.tf else "flops", "like": like}

    def done(self) -> dict:
        for k, v in self.out.items():
            if v["like"]:
                v["distance_ratio"] = round(self.frac[v["like"]] / self.frac[k], 2)      # > 1: farther than the like kernel
        return self.out


def vabunex_kernels(peaks: dict, T: int = 8192, H: int = 16, ctx: int = 8192, R: int = 4) -> dict:
    """Kernels at hidden size 2048 (16 heads of 128, wkv 32 of 64)."""
    from .. import ops
    from ..models.model import KdaMixer
    fig = Figures(peaks)
    rnd, put = fig.rnd, fig.put
    n = H * 128
    pl, pd = make_plan([(0, [1] * T, 0)], device=DEV), make_plan([(s, [1], ctx - 1) for s in range(R)], device=DEV)
    for tag, plan, rows in (("prefill", pl, T), ("decode", pd, R)):
        st = 2 * R * H * 128 * 128 * 4 if tag == "decode" else 2 * H * 128 * 128 * 4
        x = rnd(rows, 4 * n).bfloat16()
        S = torch.zeros(R, H, 128, 128, device=DEV)
        l2 = torch.full((H,), -0.01, device=DEV)
        put(f"lightning recurrence, {tag}", f"kda recurrence, {tag}",
            lambda: ops.linear_state(x[:, :n], x[:, n: 2 * n], x[:, 2 * n: 3 * n], H, 128, 128, S, plan, True, act=True, log2a=l2),
            rows * n * (3 * 2 + 4) + st)
        S2 = torch.zeros(R, 2 * H, 64, 64, device=DEV)
        lw, u = -torch.rand(rows, n, device=DEV, generator=fig.g), rnd(2 * H, 64)
        put(f"wkv recurrence, {tag}", f"kda recurrence, {tag}",
            lambda: ops.linear_state(x[:, :n], x[:, n: 2 * n], x[:, 2 * n: 3 * n], 2 * H, 64, 64, S2, plan, True, logw=lw, u=u),
            rows * n * (3 * 2 + 4 + 4) + st // 2)
        cfg = closest_config(2048, 5632, 1)
        w = {"conv": rnd(3 * n, 4), "f_b": rnd(n, 64) * 0.1, "g_b": rnd(n, 64) * 0.1, "A_log": rnd(H), "dt_bias": rnd(n),
             "o_norm": rnd(128)}
        km = KdaMixer(cfg, w, R, DEV, torch.bfloat16)
        lr = rnd(rows, 2 * 64 + 16).bfloat16()
        put(f"kda recurrence, {tag}", "", lambda: cu.kda_mixer(km, x, lr, plan, True),
            rows * n * (3 * 2 + 2 * 4 + 2) + st)
        F = 5632
        ff, o = rnd(rows, n + 2 * F).bfloat16(), rnd(rows, n)
        nw = torch.ones(n, device=DEV)
        put(f"gate + feed-forward rows, {tag}", f"swiglu rows, {tag}",
            lambda: ops.gate_concat(o, n, n, nw, 1e-5, ff[:, :n], "sigmoid", ff[:, n:], F, n, n + F, torch.bfloat16),
            rows * (n * 4 + n * 2 + 2 * F * 2 + (n + F) * 2))
        gu = rnd(rows, 2 * F).bfloat16()
        put(f"swiglu rows, {tag}", "", lambda: ops.swiglu(gu), rows * 3 * F * 2)
        res, d32, d16, nw2 = rnd(rows, 2048), rnd(rows, 2048), rnd(rows, 2048).bfloat16(), torch.ones(2048, device=DEV)
        rn = ops.RowNorm(nw2, 1e-5, one_plus=True)
        put(f"residual + norm rows, {tag}", f"residual + norm rows (bf16 update), {tag}",
            lambda: ops.add_norm_rows(d32, res, rn, torch.bfloat16), rows * 2048 * (4 * 3 + 2))
        put(f"residual + norm rows (bf16 update), {tag}", "", lambda: ops.add_rmsnorm(d16, res, nw2, 1e-5), rows * 2048 * (4 * 2 + 2 + 2))
    # latent attention, kernels only
    D, Rr, Vd, L = 128, 64, 128, 512
    q, kv, lat = rnd(T, H * (D + Rr)).bfloat16(), rnd(T, H * (D + Vd)).bfloat16(), rnd(T, L + Rr).bfloat16()
    tab, dst = torch.tensor([[0, 0, T, 0, 0]], dtype=torch.int32, device=DEV), torch.empty(T, H * Vd, dtype=torch.bfloat16, device=DEV)
    from ..ops import parallel_block as pb
    P, lib, stream = pb.P, pb.lib, pb.stream
    flops = T * T / 2 * H * (D + Rr + Vd) * 2
    put("latent attention, prefill", "latent attention of the closest model, prefill",
        lambda: lib().spark_latent_prefill(P(q), q.stride(0), P(kv), kv.stride(0), P(lat), L + Rr, P(tab), 1, T, H, D, Rr, Vd, Vd, L, 0.07,
                                           None, 0, 0, None, P(dst), H * Vd, stream()), flops=flops)
    for tag, rows, c in (("prefill", 2048, 2048), ("decode", R, ctx)):
        qf, ol = rnd(rows, H, L + Rr).bfloat16(), torch.empty(rows, H, L, dtype=torch.bfloat16, device=DEV)
        cache = rnd(R * c, L + Rr).bfloat16()
        pos = (torch.arange(rows, device=DEV) if tag == "prefill" else torch.full((rows,), c - 1, device=DEV)).int()
        slot = torch.zeros(rows, dtype=torch.int32, device=DEV) if tag == "prefill" else torch.arange(rows, dtype=torch.int32, device=DEV)
        ns = c // 64
        po, pm = torch.empty(rows * H * ns * L, device=DEV), torch.empty(rows * H * ns * 2, device=DEV)
        nb = R * c * (L + Rr) * 2 if tag == "decode" else 0
        fl = c * c / 2 * H * (D + Rr + Vd) * 2 if tag == "prefill" else rows * c * H * (2 * L + Rr) * 2
        kvb = slot.long() * c
        if tag == "decode":
            pages = torch.arange(R * ns, dtype=torch.int32, device=DEV).view(R, ns)
            put("latent attention, decode", "latent attention of the closest model, decode",
                lambda: lib().spark_mla_attn_paged(P(qf), P(cache), P(pos), None, P(slot), P(pages), ns, P(po), P(pm), ns, rows, H, L, Rr,
                                                   0.07, None, 0, None, P(ol), stream()), nb, fl)
        put(f"latent attention of the closest model, {tag}", "",
            lambda: lib().spark_mla_attn(P(qf), P(cache), P(pos), P(kvb), None, None, 0, P(po), P(pm), ns, None, rows, H, L, Rr, 0.07, P(ol),
                                         stream(), None, None, None, 0), nb, fl)
    return fig.done()


# ----------------------------------------------------------------------------- debisun
DEB_SIZES = {"1024": (1024, 4096), "2048": (2048, 8192), "4096": (4096, 16384)}
DEB_EXPERTS, DEB_TOP = 32, 4


def debisun_config(hidden: int, ffn: int):
    return debisun_style(12, hidden, ffn, VOCAB, experts=DEB_EXPERTS, top=DEB_TOP)


def debisun_closest(hidden: int, ffn: int, layers: int):
    """The same heads and experts; SwiGLU widths are two thirds, so that the three matrices hold as many parameters as two."""
    w = lambda n: (2 * n // 3 + 127) // 128 * 128
    h = hidden // 128
    return ModelConfig(name="gqa + swiglu experts, dense weights", family="hybrid", n_layers=layers, layer_types=["attn"] * layers, hidden=hidden,
                       vocab=VOCAB, attn=AttnConfig(n_q_heads=h, n_kv_heads=max(1, h // 4), head_dim=128, rope_dim=64),
                       moe=MoeConfig(n_experts=DEB_EXPERTS, top_k=DEB_TOP, ffn=w(ffn // 4), n_shared=1, shared_ffn=w(ffn // 4), router="softmax",
                                     shared_gate=True, dense_layers=1, dense_ffn=w(ffn)), weight_format="dense")


def debisun_kernels(peaks: dict, T: int = 8192, ctx: int = 8192, R: int = 4) -> dict:
    """Kernels at hidden size 2048 (16 query and 4 key / value heads of 128, 32 experts of 2048, top 4)."""
    import dataclasses
    import types
    from .. import ops
    from ..models.layout import pad
    from ..models.model import AttnMixer
    from ..models.paged_gqa import PagedGqaMixer
    from ..ops import moe_spec
    fig = Figures(peaks)
    rnd, put = fig.rnd, fig.put
    N, H, G, D = 2048, 16, 4, 128
    cfg = debisun_config(N, 8192)
    near = debisun_closest(N, 8192, 1)
    spec = dataclasses.replace(cfg.layer_specs[0], mixer=dataclasses.replace(cfg.layer_specs[0].mixer, chunk=ctx))     # one chunk: all keys
    C = (H + 2 * G) * D
    w = {"conv_t": rnd(4, C) * 0.5, "dist_bias": rnd(H, 1025), "sink": torch.zeros(H, device=DEV)}
    pages = torch.arange(R * ctx // 64, dtype=torch.int32, device=DEV).view(R, -1).contiguous()
    mx = PagedGqaMixer(cfg, spec.mixer, w, R, R * ctx // 64, 64, pages, DEV, torch.bfloat16)
    at = AttnMixer(near, {}, R * ctx, DEV, torch.bfloat16)
    for t in (mx.k, mx.v, at.k, at.v):
        t.copy_(rnd(*t.shape))
    seqs = [types.SimpleNamespace(kv_base=i * ctx, kv_cap=ctx) for i in range(R)]
    from ..ops import paged_attn as pa
    lib, P, stream = cu.lib, cu.P, cu.stream
    for tag, rows in (("prefill", T), ("decode", R)):
        plan = lambda: make_plan([(0, [1] * T, 0)] if tag == "prefill" else [(s, [1], ctx - 1) for s in range(R)], device=DEV)
        p1, p2 = plan(), plan()
        proj = rnd(rows, C).bfloat16()
        fl = T * T / 2 * H * 2 * D * 2 if tag == "prefill" else R * ctx * H * 2 * D * 2
        nb = 0 if tag == "prefill" else R * ctx * G * 2 * D * 2
        # whole mixers (convolution or rotation into the cache, then attention): the attention is nearly all of the time
        put(f"paged attention with its convolution, {tag}", f"dense attention with its rotation, {tag}",
            lambda: pa.mixer(mx, proj, p1, True), nb + rows * C * 4, fl)
        put(f"dense attention with its rotation, {tag}", "", lambda: cu.attn_mixer(at, proj, p2, seqs), nb + rows * C * 4, fl)
        d, q = cu._plan_dev(p1, DEV), torch.empty(rows, H * D, dtype=torch.bfloat16, device=DEV)
        put(f"convolution into the cache, {tag}", f"rotation into the cache, {tag}", lambda: pa._conv(mx, proj, p1, d, q, True), rows * C * 4)
        d2 = cu._plan_dev(p2, DEV)
        put(f"rotation into the cache, {tag}", "",
            lambda: lib().spark_attn_prep(P(proj), C, rows, H, G, D, 64, 0, 0, 0, 0, 4, 0, 1e-6, None, None, None, None, P(at.inv), P(d2["pos32"]),
                                          P(d2["row_kv"]), P(d2["row_j"]), P(q), P(at.k), P(at.v), None, None, None, None, None, stream(), None),
            rows * C * 4)
        # residual updates
        res, d32, d16, one = rnd(rows, N), rnd(rows, N), rnd(rows, N).bfloat16(), torch.ones(N, device=DEV)
        ln, rn = ops.RowNorm(one, 1e-5, one), ops.RowNorm(one, 1e-5)
        put(f"scaled update + layer norm, {tag}", f"update + RMS norm, {tag}",
            lambda: ops.add_norm_rows(ops.Update(d32, one), res, ln, torch.bfloat16), rows * N * 14)
        put(f"normed update + layer norm, {tag}", f"update + RMS norm, {tag}",
            lambda: ops.add_norm_rows(ops.Update(d32, post=rn), res, ln, torch.bfloat16), rows * N * 14)
        put(f"update + RMS norm, {tag}", "", lambda: ops.add_rmsnorm(d16, res, one, 1e-5), rows * N * 12)
        # token side: gate product with the token rows in its epilogue, and the projection back
        sd = cfg.side_dim
        table, ids, gw = rnd(VOCAB, sd).bfloat16(), torch.randint(0, VOCAB, (rows,), device=DEV).int(), rnd(pad(sd, 8), N).bfloat16()
        nb = rows * (N + 2 * sd) * 2 + sd * N * 2
        put(f"token gate product, {tag}", f"plain product of its shape, {tag}", lambda: ops.linear_token_gate(d16, gw, table, ids, 0, sd), nb,
            rows * N * sd * 2)
        put(f"plain product of its shape, {tag}", "", lambda: cu.dense_linear(d16, gw), nb, rows * N * sd * 2)
        up = rnd(8192, N).bfloat16()
        put(f"up product with squared relu, {tag}", f"plain up product, {tag}", lambda: ops.linear_relu2(d16, up), rows * (N + 8192) * 2 + 8192 * N * 2,
            rows * N * 8192 * 2)
        put(f"plain up product, {tag}", "", lambda: cu.dense_linear(d16, up), rows * (N + 8192) * 2 + 8192 * N * 2, rows * N * 8192 * 2)
        # routed feed-forwards: every kernel from the router to the combined rows
        c, c2 = cfg.layer_specs[1].moe, near.moe
        F, F2 = c.ffn, c2.ffn
        w1 = {"gate": rnd(c.n_routes + 1, N).bfloat16() * 0.05, "bias": 0.01 * rnd(c.n_routes), "w_up": (rnd(c.n_experts, F, N) * 0.02).bfloat16(),
              "w_down": (rnd(c.n_experts, N, F) * 0.02).bfloat16(), "s_up": (rnd(F, N) * 0.02).bfloat16(), "s_down": (rnd(N, F) * 0.02).bfloat16()}
        w2 = {"gate": rnd(c2.n_experts + 1, N).bfloat16() * 0.05, "w_gu": (rnd(c2.n_experts, 2 * F2, N) * 0.02).bfloat16(),
              "w_down": (rnd(c2.n_experts, N, F2) * 0.02).bfloat16(), "s_gu": (rnd(2 * F2, N) * 0.02).bfloat16(),
              "s_down": (rnd(N, F2) * 0.02).bfloat16()}

        def touched(c, ids):                     # bytes of the distinct experts a round reads, and the pairs that have an expert
            live = ids[(ids >= 0) & (ids < c.n_experts)]
            return live.unique().numel(), live.numel()
        e1, pairs1 = touched(c, moe_spec._route(d16, w1, c, torch.empty(rows, device=DEV))[1])
        e2, pairs2 = touched(c2, cu.moe_route(d16, w2, c2)[1])
        put(f"routed squared-relu experts + update, {tag}", f"routed SwiGLU experts + update, {tag}",
            lambda: ops.add_norm_rows(ops.Update(ops.moe(d16, w1, c, True), one), res, None, torch.bfloat16),
            (e1 + 1) * 2 * F * N * 2 + rows * N * 14, (pairs1 + rows) * 2 * F * N * 2)
        put(f"routed SwiGLU experts + update, {tag}", "",
            lambda: ops.add_rmsnorm(ops.moe(d16, w2, c2, True), res, one, 1e-5), (e2 + 1) * 3 * F2 * N * 2 + rows * N * 14,
            (pairs2 + rows) * 3 * F2 * N * 2)
        del w1, w2
    return fig.done()


# ----------------------------------------------------------------------------- zapolorn
ZAP_SIZES = {"1024": (1024, 3072), "2048": (2048, 6144), "4096": (4096, 12288)}
ZAP_WINDOW = 1024


def zapolorn_config(hidden: int, ffn: int):
    return zapolorn_style(12, hidden, ffn, VOCAB, experts=DEB_EXPERTS, top=DEB_TOP, window=ZAP_WINDOW)


def zapolorn_closest(hidden: int, ffn: int, layers: int):
    """The same heads, dense and routed feed-forwards (the dense ones first); attention over the whole context in every layer, no
    linear attention beside it."""
    h = hidden // 128
    return ModelConfig(name="gqa + swiglu, dense weights", family="hybrid", n_layers=layers, layer_types=["attn"] * layers, hidden=hidden, vocab=VOCAB,
                       attn=AttnConfig(n_q_heads=h, n_kv_heads=max(1, h // 4), head_dim=128, rope_dim=128),
                       moe=MoeConfig(n_experts=DEB_EXPERTS, top_k=DEB_TOP, ffn=ffn // 4, n_shared=1, shared_ffn=ffn // 4, router="softmax",
                                     dense_layers=layers // 2, dense_ffn=ffn), weight_format="dense")


def zapolorn_kernels(peaks: dict, T: int = 8192, ctx: int = 8192, R: int = 4) -> dict:
    """Kernels at hidden size 2048 (16 query and 4 key / value heads of 128, 32 experts of 1536, top 4; linear attention with 16 heads
    of 64 x 128).  Like kernels: the closest model's; for windows the chunked attention of Debisun with as many keys per row on
    average, for the recurrence and its decays those of Vabunex's wkv (and KDA)."""
    import dataclasses
    import types
    from .. import ops
    from ..models.model import AttnMixer
    from ..models.paged_gqa import PagedGqaMixer
    from ..ops import moe_spec
    from ..ops import paged_attn as pa
    fig = Figures(peaks)
    rnd, put = fig.rnd, fig.put
    N, H, G, D, F = 2048, 16, 4, 128, 6144
    cfg, near = zapolorn_config(N, F), zapolorn_closest(N, F, 2)
    C = (H + 2 * G) * D
    pages = torch.arange(R * ctx // 64, dtype=torch.int32, device=DEV).view(R, -1).contiguous()
    one_h = torch.ones(D, device=DEV)
    w = {"q_norm": one_h, "k_norm": one_h, "sink": torch.zeros(H, device=DEV)}
    mk = lambda c, w: PagedGqaMixer(cfg, c, w, R, R * ctx // 64, 64, pages, DEV, torch.bfloat16)
    whole, win = cfg.layer_specs[0].mixer.left, cfg.layer_specs[1].mixer
    chunked = dataclasses.replace(debisun_config(N, 8192).layer_specs[0].mixer, chunk=2 * ZAP_WINDOW)
    mw, mv = mk(whole, {k: w[k] for k in ("q_norm", "k_norm")}), mk(win, w)
    mc = mk(chunked, {"conv_t": rnd(4, C) * 0.5, "dist_bias": rnd(H, 1025), "sink": w["sink"]})
    at = AttnMixer(near, {}, R * ctx, DEV, torch.bfloat16)
    for t in (mw.k, mw.v, mv.k, mv.v, mc.k, mc.v, at.k, at.v):
        t.copy_(rnd(*t.shape))
    seqs = [types.SimpleNamespace(kv_base=i * ctx, kv_cap=ctx) for i in range(R)]
    lib, P, stream = cu.lib, cu.P, cu.stream
    for tag, rows in (("prefill", T), ("decode", R)):
        plan = lambda: make_plan([(0, [1] * T, 0)] if tag == "prefill" else [(s, [1], ctx - 1) for s in range(R)], device=DEV)
        p1, p2 = plan(), plan()
        proj = rnd(rows, C + 16).bfloat16()                            # [q | k | v | gate]
        fl = T * T / 2 * H * 2 * D * 2 if tag == "prefill" else R * ctx * H * 2 * D * 2
        nb = 0 if tag == "prefill" else R * ctx * G * 2 * D * 2
        io = rows * C * 4
        put(f"sloped attention with norms, {tag}", f"dense attention with its rotation, {tag}", lambda: pa.mixer(mw, proj, p1, True), nb + io, fl)
        put(f"dense attention with its rotation, {tag}", "", lambda: cu.attn_mixer(at, proj[:, :C].contiguous() if tag == "decode" else proj, p2, seqs),
            nb + io, fl)
        s = ZAP_WINDOW / (ctx if tag == "decode" else T / 2)
        put(f"window attention with norms and rotation, {tag}", f"chunked attention with its convolution (Debisun), {tag}",
            lambda: pa.mixer(mv, proj, p1, True), nb * s + io, fl * s)
        put(f"chunked attention with its convolution (Debisun), {tag}", "", lambda: pa.mixer(mc, proj[:, :C], p1, True),
            nb * s * (2 if tag == "decode" else 1) + io, fl * s * (2 if tag == "decode" else 1))
        d, q = cu._plan_dev(p1, DEV), torch.empty(rows, H * D, dtype=torch.bfloat16, device=DEV)
        put(f"norms and rotation into the cache, {tag}", f"rotation into the cache, {tag}", lambda: pa._heads(mv, proj, d, q), io)
        d2 = cu._plan_dev(p2, DEV)
        put(f"rotation into the cache, {tag}", "",
            lambda: lib().spark_attn_prep(P(proj), proj.stride(0), rows, H, G, D, 128, 0, 0, 0, 0, 4, 0, 1e-6, None, None, None, None, P(at.inv),
                                          P(d2["pos32"]), P(d2["row_kv"]), P(d2["row_j"]), P(q), P(at.k), P(at.v), None, None, None, None, None,
                                          stream(), None), io)
        # linear attention: 16 heads of 64 x 128 beside 32 wkv heads of 64 x 64
        st = lambda n: (2 * R if tag == "decode" else 2) * n * 4
        x, lw = rnd(rows, 2 * H * 64 + 2 * H * 128).bfloat16(), -0.1 * torch.rand(rows, H * 64, device=DEV, generator=fig.g)
        a2, b2 = (rnd(1024, 16) * 0.25).bfloat16(), torch.zeros(1024, device=DEV)
        dec = dict(logw=lw) if tag == "prefill" else dict(low_rank=(x[:, :16], a2, b2, 16.0))
        S = torch.zeros(R, H, 64, 128, device=DEV)
        put(f"gated linear attention recurrence, {tag}", f"wkv recurrence (Vabunex), {tag}",
            lambda: ops.linear_state(x[:, :1024], x[:, 1024:2048], x[:, 2048:4096], H, 64, 128, S, p1, True, qscale=0.125, **dec),
            rows * (2 * 1024 * 2 + 2048 * (2 + 4) + 1024 * 4) + st(H * 64 * 128))
        S2, lw2, u = torch.zeros(R, 32, 64, 64, device=DEV), -torch.rand(rows, N, device=DEV, generator=fig.g), rnd(32, 64)
        put(f"wkv recurrence (Vabunex), {tag}", "",
            lambda: ops.linear_state(x[:, :2048], x[:, 1024:3072], x[:, 2048:4096], 32, 64, 64, S2, p1, True, logw=lw2, u=u),
            rows * N * (3 * 2 + 4 + 4) + st(32 * 64 * 64))
        if tag == "prefill":                             # (decode rows: part of the recurrence's launch)
            put(f"decays of the linear attention, {tag}", f"decays of wkv (Vabunex), {tag}",
                lambda: ops.log_sigmoid_decay(x[:, :16], a2, b2, 1024, 16.0), rows * (16 * 2 + 1024 * 4) + 1024 * 32)
            z, w2 = rnd(rows, 64), (rnd(N, 64) * 0.1).bfloat16()
            w22, w0 = torch.cat((w2, w2), 1).contiguous(), torch.zeros(N, device=DEV)
            put(f"decays of wkv (Vabunex), {tag}", "", lambda: ops.channel_decay(z, w2, w0, N, w22), rows * (64 * 4 + N * 4) + N * 128)
        o, cat, nw = rnd(rows, N), torch.empty(rows, 2 * N, dtype=torch.bfloat16, device=DEV), torch.ones(N, device=DEV)
        gate = x[:, 2048:4096]
        put(f"norm and gate of the linear attention, {tag}", f"SwiGLU rows, {tag}",
            lambda: ops.gate_concat(o, N, 128, nw, 1e-6, gate, "silu", None, 0, N, 2 * N, torch.bfloat16, cat[:, N:]), rows * N * 8)
        gu = rnd(rows, 2 * N).bfloat16()
        put(f"SwiGLU rows, {tag}", "", lambda: ops.swiglu(gu), rows * N * 6)
        # residual updates
        res, d32, d16, one = rnd(rows, N), rnd(rows, N), rnd(rows, N).bfloat16(), torch.ones(N, device=DEV)
        rn = ops.RowNorm(one, 1e-6)
        put(f"normed update + cast, {tag}", f"update + RMS norm, {tag}",
            lambda: ops.add_norm_rows(ops.Update(d32, post=rn), res, None, torch.bfloat16), rows * N * 14)
        put(f"update + RMS norm, {tag}", "", lambda: ops.add_rmsnorm(d16, res, one, 1e-6), rows * N * 12)
        # dense feed-forward
        wgu, wd = (rnd(2 * F, N) * 0.02).bfloat16(), (rnd(N, F) * 0.02).bfloat16()
        nb, fl = 3 * F * N * 2 + rows * N * 6, rows * 3 * F * N * 2
        put(f"dense feed-forward, {tag}", f"dense feed-forward of the closest model, {tag}",
            lambda: ops.linear(ops.linear_swiglu(d16, wgu), wd, out_f32=True), nb, fl)
        put(f"dense feed-forward of the closest model, {tag}", "", lambda: ops.linear(ops.swiglu(ops.linear(d16, wgu)), wd), nb, fl)
        del wgu, wd
        # routed feed-forwards: every kernel from the router to the combined rows
        c, c2 = cfg.layer_specs[1].moe, near.moe
        Fe = c.ffn
        w1 = {"gate": rnd(c.n_experts, N).bfloat16() * 0.05, "w_gu": (rnd(c.n_experts, 2 * Fe, N) * 0.02).bfloat16(),
              "w_down": (rnd(c.n_experts, N, Fe) * 0.02).bfloat16(), "s_gu": (rnd(2 * Fe, N) * 0.02).bfloat16(), "s_down": (rnd(N, Fe) * 0.02).bfloat16()}
        e = moe_spec._route(d16, w1, c, None)[1].unique().numel()
        nb, fl = (e + 1) * 3 * Fe * N * 2 + rows * N * 14, rows * (c.top_k + 1) * 3 * Fe * N * 2
        put(f"routed experts + update, {tag}", f"routed experts of the closest model + update, {tag}",
            lambda: ops.add_norm_rows(ops.Update(ops.moe(d16, w1, c, True), post=rn), res, None, torch.bfloat16), nb, fl)
        put(f"routed experts of the closest model + update, {tag}", "", lambda: ops.add_rmsnorm(ops.moe(d16, w1, c2, tag == "decode"), res, one, 1e-6),
            nb, fl)
        del w1
    return fig.done()


# ----------------------------------------------------------------------------- zakusun
ZAK_SIZES = {"1024": (1024, 768), "2048": (2048, 1536), "4096": (4096, 3072)}


def zakusun_config(hidden: int, ffn: int):
    return zakusun_style(12, hidden, ffn, VOCAB, experts=DEB_EXPERTS, top=DEB_TOP)


def zakusun_closest(hidden: int, ffn: int, layers: int):
    """Latent attention in every layer (the same heads, values and latents; low-rank queries, a rotated part of 64), the same experts."""
    c = closest_config(hidden, ffn, layers)
    c.name, c.layer_types = "latent attention + swiglu experts, dense weights", ["mla"] * layers
    c.moe = MoeConfig(n_experts=DEB_EXPERTS, top_k=DEB_TOP, ffn=ffn, n_shared=0, router="softmax")
    return c


def zakusun_kernels(peaks: dict, T: int = 8192, ctx: int = 8192, R: int = 4) -> dict:
    """Kernels at hidden size 2048 (16 heads of 128, latents of 512, 32 experts of 1536, top 4, two norm groups, four taps).  Like
    kernels: Vabunex's latent attention (low-rank queries, a rotated part, a gate per head), the closest model's experts and row
    updates."""
    import dataclasses
    from .. import ops
    from ..models.input_conv import InputConv
    from ..models.model import Model
    from ..ops import moe_spec
    from ..ops import parallel_block as pb
    fig = Figures(peaks)
    rnd, put = fig.rnd, fig.put
    N, H, F, L = 2048, 16, 1536, 512
    P, lib, stream = pb.P, pb.lib, pb.stream
    cfg, near = zakusun_config(N, F), zakusun_closest(N, F, 1)
    cut = lambda c, kind: dataclasses.replace(c, n_layers=1, layer_types=[kind], layer_specs=[x for x in c.layer_specs if x.kind == kind][:1], loop=None)
    vab = cut(vabunex_config(N, 5632), "latent")
    vab.layer_specs = [dataclasses.replace(vab.layer_specs[0], ffn=0)]
    mixers = {}
    for name, c in (("latent attention with sink and element gate", cut(cfg, "latent")), ("latent attention (Vabunex)", vab)):
        m = Model(c, build_random_model(c, DEV, seed=0), device=DEV, dtype=torch.bfloat16, n_slots=R, kv_tokens=R * ctx)
        mixers[name] = m.layers[0][1]
        mixers[name].lat.copy_(rnd(*mixers[name].lat.shape))
    ours, like = mixers
    for tag, rows in (("prefill", T), ("decode", R)):
        plan = lambda: make_plan([(0, [1] * T, 0)] if tag == "prefill" else [(s, [1], ctx - 1) for s in range(R)], device=DEV)
        for name, mx in mixers.items():
            w, proj, p1 = mx.w, rnd(rows, mx.off["ff"]).bfloat16(), plan()
            cat = torch.empty(rows, H * 128, dtype=torch.bfloat16, device=DEV)
            up = 2 * 128 * H * L * 2                                            # flops (prompts) / bytes (decode rows) of both up matrices
            qc = sum(w[k].numel() for k in ("uq",) if k in w) * 2
            dq = 128 + mx.Rp
            fl = T * T / 2 * H * (dq + 128) * 2 + T * (up + qc) if tag == "prefill" else R * ctx * H * (2 * L + mx.Rp) * 2 + R * up
            nb = 0 if tag == "prefill" else R * ctx * (L + mx.Rp) * 2 + up + qc
            put(f"{name}, whole mixer, {tag}", f"{like}, whole mixer, {tag}" if name == ours else "",
                lambda mx=mx, proj=proj, p1=p1, cat=cat: pb.latent_mixer(mx, proj, p1, cat), nb + rows * (proj.shape[1] + H * 128) * 2, fl)
            if tag == "prefill":                                                # the attention kernel alone
                q, kv, lat = rnd(T, H * dq).bfloat16(), rnd(T, H * 256).bfloat16(), rnd(T, L + mx.Rp).bfloat16()
                tab = torch.tensor([[0, 0, T, 0, 0]], dtype=torch.int32, device=DEV)
                gate = proj[:, mx.off["g"]:]
                put(f"{name}, {tag}", f"{like}, {tag}" if name == ours else "",
                    lambda mx=mx, q=q, kv=kv, lat=lat, cat=cat, gate=gate: lib().spark_latent_prefill(
                        P(q), q.stride(0), P(kv), kv.stride(0), P(lat), lat.shape[1], P(tab), 1, T, H, 128, mx.Rp, 128, 128, L, 0.07, P(gate),
                        gate.stride(0), int(mx.c.gate == "element"), P(mx.w.get("sink")), P(cat), H * 128, stream()),
                    flops=T * T / 2 * H * (dq + 128) * 2)
        # residual updates: a plain one, and one behind the sixth layer
        res, d32, d16, one = rnd(rows, N), rnd(rows, N), rnd(rows, N).bfloat16(), torch.ones(N, device=DEV)
        cv = InputConv(rnd(4, N), R, DEV)
        ctx1, rn = ops.RowContext(plan(), True, True), ops.RowNorm(one, 1e-5, groups=2)
        put(f"update + grouped norm + convolution, {tag}", f"update + RMS norm, {tag}",
            lambda: ops.add_norm_rows(d32, res, rn, torch.bfloat16, conv=cv, ctx=ctx1), rows * N * 14)
        up = ops.Update(d32)
        up.depth = ops.DepthAverage(rnd(7, rows, N), 6, rnd(7))
        put(f"update + depth average of seven + grouped norm + convolution, {tag}", f"update + RMS norm, {tag}",
            lambda: ops.add_norm_rows(up, res, rn, torch.bfloat16, conv=cv, ctx=ctx1), rows * N * 42)
        put(f"update + RMS norm, {tag}", "", lambda: ops.add_rmsnorm(d16, res, one, 1e-5), rows * N * 12)
        table, ids = rnd(VOCAB, N).bfloat16(), torch.randint(0, VOCAB, (rows,), device=DEV).int()
        pos, freq = ctx1.plan.dev["pos32"], 1e4 ** (-torch.arange(N // 2, dtype=torch.float64, device=DEV) * 2 / N)
        put(f"embedding with positions, {tag}", f"embedding, {tag}", lambda: ops.embed(table, ids, torch.bfloat16, 1.0, (pos, freq)), rows * N * 6)
        put(f"embedding, {tag}", "", lambda: ops.embed(table, ids, torch.bfloat16), rows * N * 6)
        # routed feed-forwards: every kernel from the router to the combined rows
        c, c2 = cfg.layer_specs[0].moe, near.moe
        w1 = {"gate": rnd(c.n_experts, N).bfloat16() * 0.05, "bias": torch.zeros(c.n_experts, device=DEV),
              "w_gu": (rnd(c.n_experts, 2 * F, N) * 0.02).bfloat16(), "w_down": (rnd(c.n_experts, N, F) * 0.02).bfloat16()}
        e = moe_spec._route(d16, w1, c, None)[1].unique().numel()
        nb, fl = e * 3 * F * N * 2 + rows * N * 14, rows * c.top_k * 3 * F * N * 2
        ctx2 = ops.RowContext(ctx1.plan, True, True)
        put(f"routed experts + update, {tag}", f"routed experts of the closest model + update, {tag}",
            lambda: ops.add_norm_rows(ops.Update(ops.moe(d16, w1, c, True)), res, rn, torch.bfloat16, conv=cv, ctx=ctx2), nb, fl)
        put(f"routed experts of the closest model + update, {tag}", "", lambda: ops.add_rmsnorm(ops.moe(d16, w1, c2, tag == "decode"), res, one, 1e-6),
            nb, fl)
        del w1
    return fig.done()


DESIGNS = {
    "vabunex": (vabunex_config, closest_config, vabunex_kernels, SIZES,
                "KDA + latent attention (GLM-style layer types), sequential pre-norm blocks, dense feed-forward, bf16"),
    "debisun": (debisun_config, debisun_closest, debisun_kernels, DEB_SIZES,
                "grouped-query attention (rotary, whole context), softmax-routed SwiGLU experts of as many parameters, bf16"),
    "zapolorn": (zapolorn_config, zapolorn_closest, zapolorn_kernels, ZAP_SIZES,
                 "grouped-query attention (rotary, whole context), dense and softmax-routed SwiGLU feed-forwards of its sizes, bf16"),
    "zakusun": (zakusun_config, zakusun_closest, zakusun_kernels, ZAK_SIZES,
                "latent attention (low-rank queries, a rotated part, absorbed prompts), softmax-routed SwiGLU experts of its sizes, bf16"),
}


def run(args, clocks) -> int:
    here = os.path.dirname(os.path.dirname(os.path.dirname(os.path.abspath(__file__))))
    try:
        with open(os.path.join(here, "MEASURED_PEAKS.json")) as f:
            peaks = json.load(f)
    except OSError:
        peaks = {}
    config, closest, kernels, all_sizes, closest_text = DESIGNS[args.design]
    clocks.start()
    sizes = {}
    for name, (hidden, ffn) in all_sizes.items():
        cv = config(hidden, ffn)
        runs = len(cv.layer_runs())
        sizes[name] = {"layer_runs": runs, "ffn": ffn, args.design: model_figures(cv, args.steps, args.warmup)}
        cu._scratch.clear()
        torch.cuda.empty_cache()
        sizes[name]["closest"] = model_figures(closest(hidden, ffn, runs), args.steps, args.warmup)
        cu._scratch.clear()
        torch.cuda.empty_cache()
    out = {"metric": f"{args.design} prefill / decode throughput beside the closest existing family at equal size", "design": args.design,
           "closest": closest_text, "dtype": "bf16", "data": "synthetic", "sizes": sizes, "kernels": kernels(peaks),
           "clocks": clocks.stop(), "peaks": {k: peaks.get(k) for k in ("hbm_gbs", "bf16_tflops")}}
    print(json.dumps(out))
    return 0
