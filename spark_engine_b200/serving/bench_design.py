"""`bench.py --design vabunex`: prefill and decode throughput of a Vabunex model with random weights at a few layer sizes of
real models, beside the closest existing family at equal size (KDA linear attention + latent attention, sequential
pre-norm blocks with dense feed-forwards, bf16), and the kernels of the new mechanisms beside their like kernels as
fractions of the measured copy bandwidth / GEMM throughput.

Device-timed with CUDA events.  Model figures stream more weights and activations than L2 holds; kernel figures write a
buffer larger than L2 between iterations (median of the iterations)."""
from __future__ import annotations

import json
import os
import statistics

import torch

from ..config import EngineConfig, KdaConfig, MlaConfig, glm_style, vabunex_style
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


def kernel_figures(peaks: dict, T: int = 8192, H: int = 16, ctx: int = 8192, R: int = 4) -> dict:
    """Kernels at hidden size 2048 (16 heads of 128, wkv 32 of 64): {name: (ms, fraction of roofline, bound, like kernel)}."""
    from .. import ops
    from ..models.model import KdaMixer
    hbm, tf = peaks.get("hbm_gbs", 6650.0) * 1e6, peaks.get("bf16_tflops", 1590.0) * 1e9      # bytes, flops per millisecond
    flush = torch.empty(512 << 20, dtype=torch.uint8, device=DEV)
    g = torch.Generator(device=DEV).manual_seed(0)
    rnd = lambda *s: torch.randn(*s, device=DEV, generator=g)
    out = {}

    def put(name, like, fn, nbytes=0, flops=0):
        if name.endswith("decode"):              # short kernels: replayed from a graph, no host time between launches
            fn()
            torch.cuda.synchronize()
            graph = torch.cuda.CUDAGraph()
            with torch.cuda.graph(graph):
                fn()
            fn = graph.replay
        ms = _timed(fn, 7, flush)
        roof = max(nbytes / hbm, flops / tf)
        out[name] = {"us": round(ms * 1e3, 1), "of_roofline": round(roof / ms, 3), "bound": "bytes" if nbytes / hbm >= flops / tf else "flops",
                     "like": like}

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
        lw, u = -torch.rand(rows, n, device=DEV, generator=g), rnd(2 * H, 64)
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
                                           None, 0, P(dst), H * Vd, stream()), flops=flops)
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
                                                   0.07, None, 0, P(ol), stream()), nb, fl)
        put(f"latent attention of the closest model, {tag}", "",
            lambda: lib().spark_mla_attn(P(qf), P(cache), P(pos), P(kvb), None, None, 0, P(po), P(pm), ns, None, rows, H, L, Rr, 0.07, P(ol),
                                         stream(), None, None, None, 0), nb, fl)
    for v in out.values():
        if v["like"]:
            v["distance_ratio"] = round(out[v["like"]]["of_roofline"] / v["of_roofline"], 2)    # > 1: farther than the like kernel
    return out


def run(args, clocks) -> int:
    here = os.path.dirname(os.path.dirname(os.path.dirname(os.path.abspath(__file__))))
    try:
        with open(os.path.join(here, "MEASURED_PEAKS.json")) as f:
            peaks = json.load(f)
    except OSError:
        peaks = {}
    clocks.start()
    sizes = {}
    for name, (hidden, ffn) in SIZES.items():
        cv = vabunex_config(hidden, ffn)
        runs = len(cv.layer_runs())
        sizes[name] = {"layer_runs": runs, "ffn": ffn, "vabunex": model_figures(cv, args.steps, args.warmup)}
        torch.cuda.empty_cache()
        sizes[name]["closest"] = model_figures(closest_config(hidden, ffn, runs), args.steps, args.warmup)
        cu._scratch.clear()
        torch.cuda.empty_cache()
    out = {"metric": "vabunex prefill / decode throughput beside the closest existing family at equal size", "design": "vabunex",
           "closest": "KDA + latent attention (GLM-style layer types), sequential pre-norm blocks, dense feed-forward, bf16",
           "dtype": "bf16", "data": "synthetic", "sizes": sizes, "kernels": kernel_figures(peaks),
           "clocks": clocks.stop(),
           "peaks": {k: peaks.get(k) for k in ("hbm_gbs", "bf16_tflops")}}
    print(json.dumps(out))
    return 0
