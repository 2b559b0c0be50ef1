"""Zapolorn on a B200: the kernels of each mechanism and whole models, in bf16 and in 32-bit, against the plain implementation;
portions, mixed batches, page and window edges, captured decode rounds, the server.

A routed model in bf16 may take another expert than the plain one where two scores are closer than rounding, and later rows see
that token: such models are compared by the median of their rows in bf16, with a wide limit on the ninth decile (and by the worst
row in 32-bit); the expert kernels have a test of their own on rows without close calls."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch
import zapolorn_oracle as oracle
import zapolorn_util as U
from test_zapolorn import FAR, SLOPED, _serve, _setup, far_case, slope_case

from spark_engine_b200 import ops
from spark_engine_b200.config import EngineConfig, MoeConfig, PagedGqaConfig
from spark_engine_b200.models.paged_gqa import PagedGqaMixer
from spark_engine_b200.models.plan import make_plan
from spark_engine_b200.serving.engine import LLMEngine
from spark_engine_b200.serving.session import BatchSession
from spark_engine_b200.serving.worker import EngineServer

pytestmark = pytest.mark.gpu
DEV = "cuda"
TOL = {torch.float32: 3e-5, torch.bfloat16: 3e-2}
DTYPES = [torch.float32, torch.bfloat16]

# head sizes around the compiled widths, query heads beyond one MMA tile, shapes the tensor-core kernels do not take
SHAPES = dict(U.MECHANISMS)
SHAPES.update({
    "heads of 128": dict(layers=[U.window(U.dense(264), heads=8, kv_heads=2, dim=128, vdim=128, rot=64, scale=0.09),
                                 U.pair(None, heads=8, kv_heads=2, dim=128, vdim=128, scale=0.09, rheads=2, rdim=128, rvdim=128)], width=264),
    "wide values": dict(layers=[U.window(heads=2, kv_heads=1, dim=64, vdim=200, scale=0.12), U.pair(heads=2, kv_heads=1, rdim=64, rvdim=200)]),
    "wide keys": dict(layers=[U.window(heads=2, kv_heads=1, dim=256, vdim=256, rot=200, scale=0.06), U.pair(rheads=1, rdim=256, rvdim=32)], width=136),
    "very wide": dict(layers=[U.window(heads=1, kv_heads=1, dim=320, vdim=272, rot=320, scale=0.06)]),
    "40 query heads per key head": dict(layers=[U.window(heads=40, kv_heads=1, dim=16, vdim=8, scale=0.25), U.pair(heads=40, kv_heads=1, dim=16, vdim=8)]),
    "many experts": dict(layers=[U.window(U.moe(experts=70, top=6, ff=264, shared=136), dim=32, vdim=32)], width=136),
    "more pairs than a decode round's": dict(layers=[U.window(U.moe(experts=30, top=20, ff=24))]),
})


def agree(got, want, dtype, cfg):
    if dtype == torch.float32:
        assert U.error(got, want) < TOL[dtype]
        return
    d = (got.float().cpu() - want).double()
    e = (d - d.mean(-1, keepdim=True)).pow(2).mean(-1).sqrt() / want.double().std()
    limit = TOL[dtype] * len(cfg["layers"]) ** 0.5
    if any(x.get("mlp") and x["mlp"]["kind"] == "moe" for x in cfg["layers"]):
        assert e.quantile(0.5) < limit and e.quantile(0.9) < 4 * limit
    else:                                        # (a row whose mixer output nearly cancels is normed all the same)
        assert e.quantile(0.95) < limit and e.max() < 4 * limit


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(SHAPES))
def test_prompt_then_decoding(name, dtype):
    cfg, T = _setup(SHAPES[name])
    toks = U.prompt(160, cfg["vocab"])
    want = U.oracle_logits(cfg, T, toks)
    m = U.framework(cfg, T, DEV, dtype)
    agree(m.forward(make_plan([(0, toks, 0)], device=DEV)), want, dtype, cfg)
    out, i = [], 0
    for n in (2, 31, 2, 33, 64, *[1] * 28):
        out.append(m.forward(make_plan([(3, toks[i: i + n], i)], device=DEV)))
        i += n
    agree(torch.cat(out), want, dtype, cfg)


@pytest.mark.parametrize("dtype", DTYPES)
def test_mixed_batches_equal_each_request_alone(dtype):
    cfg, T = _setup(U.MIXED)
    mc = U.Z.read_config(cfg)
    ses = BatchSession(mc, U.Z.from_tensors(mc, T, DEV, dtype), EngineConfig(dtype="float32" if dtype == torch.float32 else "bfloat16"), DEV,
                       max_seqs=4, kv_tokens=320 + 192 + 64 + 128)
    lens = {"a": 300, "b": 180, "c": 3, "d": 100, "e": 121}
    toks = {k: U.prompt(n, cfg["vocab"], ord(k)) for k, n in lens.items()}
    want = {k: U.oracle_logits(cfg, T, t) for k, t in toks.items()}
    at, got_all = dict.fromkeys(lens, 0), {k: [] for k in lens}
    for st in (("a70", "b1", "c2"), ("a1", "b100", "d33"), ("a2", "b31", "c1", "d2"), ("/c", "a128", "b2", "d64"), ("/b", "a1", "d1"),
               ("/d", "a64", "e1"), ("a33", "e120"), ("a1",)):
        for x in st:
            if x[0] == "/":
                ses.end(x[1:])
        ent = [(x[0], toks[x[0]][at[x[0]]: at[x[0]] + int(x[1:])], list(range(int(x[1:])))) for x in st if x[0] != "/"]
        got, r = ses.step(ent), 0
        for k, t, _ in ent:
            got_all[k].append(got[r: r + len(t)])
            r += len(t)
            at[k] += len(t)
    assert at["a"] == 300
    for k, g in got_all.items():
        g = torch.cat(g)
        if len(g) > 10 or dtype == torch.float32:
            agree(g, want[k][: len(g)], dtype, cfg)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("size,at", FAR)
@pytest.mark.parametrize("borrowed", [False, True])
def test_a_key_is_seen_inside_the_window_only(size, at, dtype, borrowed):
    cfg, T, toks, without = far_case(size, at, borrowed)
    want = U.oracle_logits(cfg, T, toks)
    seen = 209 - at < size
    moved = U.error(U.oracle_logits(cfg, T, without)[-1:], want[-1:])
    if borrowed and not seen:                    # (the second layer reaches past the first one's window)
        moved = 1.0
    assert moved > 0.05 or not seen
    limit = TOL[dtype] if dtype == torch.float32 else min(0.4 * moved, 0.05) if seen else 0.05
    m = U.framework(cfg, T, DEV, dtype)
    assert U.error(m.forward(make_plan([(0, toks, 0)], device=DEV))[-1:], want[-1:]) < limit
    m.forward(make_plan([(1, toks[:-3], 0)], device=DEV))
    for i in range(207, 210):
        got = m.forward(make_plan([(1, toks[i: i + 1], i)], device=DEV))
    assert U.error(got, want[-1:]) < limit
    # hidden from the row, the planted token must not change a bit of what the row attends to
    if not seen and not borrowed:
        m.forward(make_plan([(2, without[:-3], 0)], device=DEV))
        for i in range(207, 210):
            same = m.forward(make_plan([(2, without[i: i + 1], i)], device=DEV))
        assert torch.equal(same, got)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("at", SLOPED)
def test_far_keys_under_a_slope(at, dtype):
    cfg, T, toks, without = slope_case(at)
    want = U.oracle_logits(cfg, T, toks)
    moved = U.error(U.oracle_logits(cfg, T, without)[-1:], want[-1:])
    limit = TOL[dtype] if dtype == torch.float32 else min(0.4 * moved, 0.05)
    m = U.framework(cfg, T, DEV, dtype)
    assert U.error(m.forward(make_plan([(0, toks, 0)], device=DEV))[-1:], want[-1:]) < limit
    m.forward(make_plan([(1, toks[:-3], 0)], device=DEV))
    for i in range(207, 210):
        got = m.forward(make_plan([(1, toks[i: i + 1], i)], device=DEV))
    assert U.error(got, want[-1:]) < limit


def attention_case(dtype, n, H, G, D, V, seed=0, **kw):
    """One attention mixer on its own, with the plain result of the projected rows; scores of a spread that makes every key and
    every constant show."""
    g = torch.Generator().manual_seed(seed)
    c = PagedGqaConfig(n_heads=H, n_kv_heads=G, head_dim=D, v_dim=V, conv_k=0, **kw)
    w = {}
    if c.qk_norm:
        w.update(q_norm=1 + 0.3 * torch.randn(D, generator=g), k_norm=1 + 0.3 * torch.randn(D, generator=g))
    w["sink"] = torch.randn(H, generator=g) * 2
    pages = torch.randperm(40, generator=g).to(torch.int32).view(2, 20)
    cfg = type("C", (), {"norm_eps": 1e-5})
    mx = PagedGqaMixer(cfg, c, {k: t.to(DEV) for k, t in w.items()}, 2, 40, 64, pages.to(DEV), DEV, dtype, out_scale=0.75)
    Dp, Vp = mx.Dp, mx.Vp
    rows = torch.randn(n, mx.columns + H, generator=g).to(dtype)
    heads = rows[:, : (H + G) * Dp].view(n, H + G, Dp)
    heads[..., D:] = 0
    vals = rows[:, (H + G) * Dp: mx.columns].view(n, G, Vp)
    vals[..., V:] = 0
    x = rows.double()
    q, k = x[:, : H * Dp].view(n, H, Dp)[..., :D], x[:, H * Dp: (H + G) * Dp].view(n, G, Dp)[..., :D]
    if c.qk_norm:
        q, k = oracle.rms_norm(q, w["q_norm"].double(), 1e-5), oracle.rms_norm(k, w["k_norm"].double(), 1e-5)
    if c.rope_dims:
        rot = {"dims": c.rope_dims, "base": c.rope_theta, "scaling": {"factor": c.rope_factor}}
        q, k = oracle.rotate_pairs(q, rot), oracle.rotate_pairs(k, rot)
    if c.temp_coef:
        q = q * torch.tensor([oracle.temperature(i, {"coef": c.temp_coef, "every": c.temp_every}) for i in range(n)]).view(n, 1, 1)
    slopes = torch.tensor([oracle.slope(h, H) for h in range(H)]).double() if c.slopes else None
    o = oracle.attend(q, k, x[:, (H + G) * Dp: mx.columns].view(n, G, Vp)[..., :V], c.scale, c.window or None, w["sink"].double(), slopes)
    if c.gated:
        o = o * torch.sigmoid(x[:, mx.columns:]).unsqueeze(-1)
    pad8 = (-rows.shape[1]) % 8
    return mx, torch.nn.functional.pad(rows, (0, pad8)).to(DEV), 0.75 * o


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kw", [
    dict(scale=0.2, window=77, qk_norm=True, rope_dims=24, rope_theta=50.0, rope_factor=1.5, gated=True),
    dict(scale=0.3, slopes=True, qk_norm=True, temp_coef=0.9, temp_every=13.0),
    dict(scale=0.15, slopes=True, window=130, rope_dims=8, gated=True, temp_coef=-0.1, temp_every=2.5)])
@pytest.mark.parametrize("H,G,D,V", [(6, 3, 24, 40), (8, 1, 128, 128), (5, 5, 40, 8), (20, 1, 32, 24)])
def test_attention_mechanisms(H, G, D, V, kw, dtype):
    mx, rows, want = attention_case(dtype, 290, H, G, D, V, **kw)
    tol = 2e-5 if dtype == torch.float32 else 3e-2
    n = rows.shape[0]
    check = lambda o, a, b: (o.view(-1, H, mx.Vp)[..., :V].double().cpu() - want[a:b]).norm() < tol * want[a:b].norm()
    assert check(mx.attend(rows, make_plan([(0, [1] * n, 0)], device=DEV), True), 0, n)
    i = 0
    for m in (3, 61, 1, 64, 31, 70, 1, 1, 58):
        wide = torch.full((m, H * mx.Vp + 24), 7.0, dtype=dtype, device=DEV)      # into a range of a wider row
        assert mx.attend(rows[i: i + m], make_plan([(1, [1] * m, i)], device=DEV), True, wide[:, 8: 8 + H * mx.Vp]) is not None
        assert check(wide[:, 8: 8 + H * mx.Vp].reshape(m, -1), i, i + m), (i, m)
        assert (wide[:, :8] == 7).all() and (wide[:, 8 + H * mx.Vp:] == 7).all()
        i += m
    assert i == n


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,D,V", [(1, 16, 16), (3, 20, 28), (2, 64, 200), (2, 128, 128), (1, 200, 40)])
@pytest.mark.parametrize("strength", [0.02, 1.0, 40.0])
def test_decayed_state(H, D, V, strength, dtype):
    """The recurrence with decays from next to none to total, in one prompt, in portions and token by token, with accepted rows."""
    g = torch.Generator().manual_seed(D)
    n = 200
    x = torch.randn(n, H * (2 * D + V), generator=g).to(dtype)
    lw = -strength * torch.rand(n, H * D, generator=g)
    q, k, v = x.double()[:, : H * D].view(n, H, D), x.double()[:, H * D: 2 * H * D].view(n, H, D), x.double()[:, 2 * H * D:].view(n, H, V)
    want = 0.3 * oracle.decayed_sums(q, k, v, torch.exp(lw.double()).view(n, H, D)).reshape(n, H * V)
    S = torch.zeros(3, H, D, V, device=DEV)
    xd, lwd = x.to(DEV), lw.to(DEV)
    run = lambda a, b, slot, commit=True, rows=None: ops.linear_state(
        xd[a:b, : H * D], xd[a:b, H * D: 2 * H * D], xd[a:b, 2 * H * D:], H, D, V, S, make_plan([(slot, [1] * (b - a), a)], device=DEV), commit,
        logw=lwd[a:b].contiguous(), qscale=0.3, n_rows=rows)
    close = lambda o, a, b: ((o.double().cpu() - want[a:b]).norm() / want[a:b].norm()) < 2e-5
    assert close(run(0, n, 0), 0, n)
    i = 0
    for m in (2, 64, 1, 33, 65, 5, 1, 29):
        assert close(run(i, i + m, 1), i, i + m), (i, m)
        i += m
    assert i == n and torch.allclose(S[0], S[1], atol=1e-3 * float(S[0].abs().max()))
    before = S[1].clone()
    run(i - 5, i, 1, commit=False)
    assert torch.equal(S[1], before)
    run(0, 100, 2)
    run(100, 106, 2, rows=torch.tensor([3], dtype=torch.int32, device=DEV))
    assert close(run(103, 140, 2), 103, 140)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("R", [1, 5, 300])
def test_channel_decays(R, dtype):
    g = torch.Generator().manual_seed(R)
    for rank, n, tau in ((24, 96, 12.0), (10, 60, 1.0), (64, 33, 0.5)):
        r8 = (rank + 7) // 8 * 8
        z, w2, b = torch.zeros(R, r8 + 8), torch.zeros(n, r8), 2 * torch.randn(n, generator=g)
        z[:, :rank], w2[:, :rank] = 4 * torch.randn(R, rank, generator=g), torch.randn(n, rank, generator=g)
        z, w2 = z.to(dtype), w2.to(dtype)
        want = torch.nn.functional.logsigmoid(z.double()[:, :r8] @ w2.double().T + b.double()) / tau
        got = ops.log_sigmoid_decay(z.to(DEV)[:, :rank], w2.to(DEV), b.to(DEV), n, tau).double().cpu()
        assert torch.allclose(got, want.clamp(min=-105), atol=3e-5, rtol=3e-6)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,D,V,rank", [(2, 20, 28, 10), (3, 64, 40, 64)])
def test_decays_inside_the_recurrence(H, D, V, rank, dtype):
    """Decode rows form their decays in the recurrence's own launch: as with decays computed first, whatever the batch is."""
    g = torch.Generator().manual_seed(rank)
    r8, n = (rank + 7) // 8 * 8, 12
    x = torch.randn(n, H * (2 * D + V), generator=g).to(dtype).to(DEV)
    z, w2, b = torch.zeros(n, r8 + 8), torch.zeros(H * D, r8), torch.randn(H * D, generator=g).to(DEV)
    z[:, :rank], w2[:, :rank] = torch.randn(n, rank, generator=g), torch.randn(H * D, rank, generator=g)
    z, w2 = z.to(dtype).to(DEV), w2.to(dtype).to(DEV)
    S = torch.randn(4, H, D, V, generator=g).to(DEV)
    S2 = S.clone()
    plan = lambda: make_plan([(3, [1] * 7, 50), (0, [1], 9), (1, [1] * 4, 0)], device=DEV)
    run = lambda S, **kw: ops.linear_state(x[:, : H * D], x[:, H * D: 2 * H * D], x[:, 2 * H * D:], H, D, V, S, plan(), True, qscale=0.5, **kw)
    a = run(S, low_rank=(z[:, :rank], w2, b, 3.0))
    c = run(S2, logw=ops.log_sigmoid_decay(z[:, :rank], w2, b, H * D, 3.0))
    assert torch.allclose(a, c, atol=1e-4, rtol=1e-4) and torch.allclose(S, S2, atol=1e-4, rtol=1e-4) and not torch.equal(S[3], S[2])


@pytest.mark.parametrize("R,K,F", [(1, 64, 128), (16, 1024, 512), (17, 264, 128), (300, 96, 384), (3, 75, 128), (40, 75, 256)])
def test_swiglu_products(R, K, F):
    g = torch.Generator().manual_seed(F)
    for dt in DTYPES:
        x, w = torch.randn(R, K, generator=g).to(dt), (torch.randn(2 * F, K, generator=g) * K ** -0.5).to(dt)
        y = x.double() @ w.double().T
        got = ops.linear_swiglu(x.to(DEV), w.to(DEV)).double().cpu()
        tol = dict(atol=1e-4, rtol=1e-4) if dt == torch.float32 else dict(atol=3e-2, rtol=2e-2)
        assert torch.allclose(got, oracle.silu(y[:, :F]) * y[:, F:], **tol)


@pytest.mark.parametrize("E,top,F", [(6, 2, 40), (1, 1, 8), (13, 1, 104), (60, 8, 136), (500, 30, 16)])
@pytest.mark.parametrize("H", [64, 264, 75])
def test_experts(E, top, F, H):
    """Fused decode router, pair GEMVs, grouped products and the FP32-unit form against the plain form on rows without close calls."""
    from spark_engine_b200.models.zapolorn import WIDE
    from spark_engine_b200.models.layout import pad, pad_cols, stack_rows
    g = torch.Generator().manual_seed(E)
    c = MoeConfig(n_experts=E, top_k=top, ffn=F, n_shared=1, shared_ffn=F, router="sigmoid", weight_input=True)
    rnd = lambda *s: torch.randn(*s, generator=g)
    flat = {"router": rnd(E, H) * 3 * H ** -0.5}
    for k in [f"e{j}." for j in range(E)] + ["shared."]:
        flat[k + "gate"], flat[k + "up"], flat[k + "down"] = rnd(F, H) * 2 * H ** -0.5, rnd(F, H) * H ** -0.5, rnd(H, F) * F ** -0.5
    flat = {k: t.bfloat16().float() for k, t in flat.items()}
    gu = lambda k: stack_rows([flat[k + "gate"], flat[k + "up"]], WIDE)
    down = lambda k: pad_cols(flat[k + "down"], pad(F, WIDE))
    w = {"gate": flat["router"], "w_gu": torch.stack([gu(f"e{j}.") for j in range(E)]), "w_down": torch.stack([down(f"e{j}.") for j in range(E)]),
         "s_gu": gu("shared."), "s_down": down("shared.")}
    mlp = {"router": {"experts": E, "top": top}, "shared": {"ff": F}}
    for R in (1, 16, 17, 230):
        h = rnd(R, H).bfloat16().float()
        want = oracle.experts(h, flat, "", mlp)
        s = (h @ flat["router"].T).sort(-1, descending=True).values
        clear = torch.ones(R, dtype=torch.bool) if top == E else s[:, top - 1] - s[:, top] > 1e-4
        assert clear.float().mean() > 0.8
        for dt in DTYPES:
            wd = {k: t.to(dt).cuda() for k, t in w.items()}
            got = ops.moe(h.to(dt).cuda(), wd, c).float().cpu()
            err = ((got - want).norm(dim=-1) / want.norm(dim=-1))[clear]
            assert err.max() < (2e-5 if dt == torch.float32 else 2e-2), (R, dt)


def test_rows_do_not_depend_on_the_batch():
    """The same decode rows alone, and beside other sequences whose pages and slots differ: bitwise equal."""
    cfg, T = _setup(U.MIXED)
    m = U.framework(cfg, T, DEV, torch.bfloat16)
    toks = U.prompt(100, cfg["vocab"])
    for s, n in ((0, 90), (1, 40), (2, 90), (3, 90)):
        m.forward(make_plan([(s, toks[:n], 0)], device=DEV))
    alone = m.forward(make_plan([(0, toks[90:91], 90)], device=DEV))
    both = m.forward(make_plan([(1, toks[40:41], 40), (3, toks[90:91], 90)], device=DEV))
    assert torch.equal(alone[0], both[1])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_captured_rounds_generate_the_oracles_text(dtype):
    """Greedy generation in captured rounds, 200 tokens across page and window borders: every token is the oracle's choice for the
    text before it (bf16: nearly always among the choices within rounding)."""
    cfg, T = _setup(U.MIXED)
    mc = U.Z.read_config(cfg)
    eng = LLMEngine(mc, U.Z.from_tensors(mc, T, DEV, getattr(torch, dtype)), EngineConfig(dtype=dtype), device=DEV, max_seqs=3, kv_tokens_per_seq=512)
    assert eng.use_graphs
    prompts = [U.prompt(n, cfg["vocab"], n) for n in (1, 100, 62)]
    outs = eng.generate(prompts, max_new=200)
    fed = [eng.model.seqs[s].length for s in range(3)]
    more = eng.decode_steps([0, 1, 2], [o[-1] for o in outs], 40)
    assert [eng.model.seqs[s].length for s in range(3)] == [n + 40 for n in fed]
    eng.check_device_status()
    for i, (p, o) in enumerate(zip(prompts, outs)):
        o = o + [r[i] for r in more]
        want = U.oracle_logits(cfg, T, p + o)[len(p) - 1: -1]
        gap = (want.amax(-1) - want.gather(1, torch.tensor(o).view(-1, 1))[:, 0]) / want.std()
        if dtype == "float32":
            assert gap.max() <= 1e-4, i
        else:
            assert gap.quantile(0.9) <= 0.25, i


@pytest.mark.parametrize("drafts", [False, True])
def test_server_in_32_bit_generates_the_oracles_text(drafts):
    cfg, T = _setup(U.MIXED)
    mc = U.Z.read_config(cfg)
    es = EngineServer(mc, U.Z.from_tensors(mc, T, DEV, torch.float32),
                      EngineConfig(max_seqs=2, kv_tokens=1024, prefill_chunk=48, spec="lookup" if drafts else "none", spec_depth=3,
                                   dtype="float32"), device=DEV)
    prompts = {i: U.prompt(n, cfg["vocab"], n) for i, n in enumerate((41, 7, 90, 3))}
    texts = {i: U.oracle_greedy(cfg, T, p, 12) for i, p in prompts.items()}
    if drafts:
        def draft(seq, depth):
            i, n = es.by_slot[seq.slot].id, len(seq.generated)
            d = (texts[i][n: n + 2] + [0])[:depth] if i in texts else []
            return d, [0.9] * len(d)
        es.spec.drafter = draft
    done = _serve(es, [{"id": i, "prompt_ids": p, "max_new": 12} for i, p in prompts.items()])
    for i, p in prompts.items():
        assert done[i]["token_ids"] == texts[i], i
    p = prompts[0] + done[0]["token_ids"] + [1, 2]
    assert _serve(es, [{"id": 9, "prompt_ids": p, "max_new": 6}])[9]["token_ids"] == U.oracle_greedy(cfg, T, p, 6)
    if drafts:
        assert 0 < es.totals["accepted_drafts"] < es.totals["drafted_tokens"]


def test_trace_runner(tmp_path):
    cfg, T = _setup(U.MIXED)
    U.write_checkpoint(tmp_path / "ck", cfg, T)
    toks = U.prompt(70, cfg["vocab"])
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": toks[:40], "want": [0, 39]}], "end": []},
             {"step": 1, "entries": [{"id": "y", "tokens": toks[:3], "want": []}], "end": ["y"]},
             {"step": 2, "entries": [{"id": "x", "tokens": toks[40:], "want": [29]}, {"id": "z", "tokens": toks[:1], "want": [0]}],
              "end": ["x", "z"]}]
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    r = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", str(tmp_path / "ck"), "--dtype", "float32",
                        "--out", str(tmp_path), "--max-tokens", "192"], input="\n".join(json.dumps(s) for s in steps) + "\n",
                       capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == ["done 0", "done 1", "done 2"]
    want = U.oracle_logits(cfg, T, toks)
    get = lambda i: torch.from_numpy(np.fromfile(tmp_path / f"{i}.f32", "<f4").reshape(-1, cfg["vocab"]))
    assert U.error(get(0), want[[0, 39]]) < 3e-5 and U.error(get(2), want[[69, 0]]) < 3e-5
    assert not (tmp_path / "1.f32").exists()
