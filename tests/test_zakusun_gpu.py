"""Zakusun on a B200: the kernels of each mechanism and whole models, in bf16 and in 32-bit, against the plain implementation;
portions, mixed batches, page edges, captured decode rounds, the server.

A routed model in bf16 may take another expert than the plain one where two logits are closer than rounding, and later rows see
that token: such models are compared by the median of their rows in bf16, with a wide limit on the ninth decile (and by the worst
row in 32-bit); the expert kernels have a test of their own on rows without close calls."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch
import zakusun_oracle as oracle
import zakusun_util as U
from test_zakusun import FAR, MIX_STEPS, _serve, _setup, far_case

from spark_engine_b200 import ops
from spark_engine_b200.config import EngineConfig, LatentConfig, LayerSpec, MoeConfig
from spark_engine_b200.models.input_conv import InputConv
from spark_engine_b200.models.layout import latent_up, pad, pad_cols, stack_rows
from spark_engine_b200.models.parallel_mixers import LatentMixer
from spark_engine_b200.models.plan import make_plan
from spark_engine_b200.ops import cuda as cu
from spark_engine_b200.serving.engine import LLMEngine
from spark_engine_b200.serving.session import BatchSession
from spark_engine_b200.serving.worker import EngineServer

pytestmark = pytest.mark.gpu
DEV = "cuda"
TOL = {torch.float32: 3e-5, torch.bfloat16: 3e-2}
DTYPES = [torch.float32, torch.bfloat16]

# head sizes around the compiled widths, heads beyond the MMA tiles, shapes the tensor-core kernels do not take
SHAPES = dict(U.MECHANISMS)
SHAPES.update({
    "heads of 128": dict(layers=[U.latent(U.moe(ff=136), heads=8, dim=128, vdim=128, kv_rank=256, scale=0.09)], width=264, groups=2),
    "20 heads": dict(layers=[U.latent(heads=20, dim=32, vdim=24, kv_rank=64)], width=128, groups=1),
    "70 heads": dict(layers=[U.latent(heads=70, dim=16, vdim=8, kv_rank=32)], width=128, groups=4),
    "wide values": dict(layers=[U.latent(heads=2, dim=64, vdim=200, kv_rank=72, scale=0.12)]),
    "wide latents": dict(layers=[U.latent(heads=2, dim=48, vdim=33, kv_rank=520, scale=0.12)]),
    "very wide": dict(layers=[U.latent(heads=1, dim=320, vdim=272, kv_rank=40, scale=0.06)]),
    "groups of 128": dict(layers=[U.latent(U.moe()), U.latent(U.moe())], width=384, groups=3),
    "many experts": dict(layers=[U.latent(U.moe(experts=70, top=6, ff=264), dim=32, vdim=32)], width=136, groups=2),
    "more pairs than a decode round's": dict(layers=[U.latent(U.moe(experts=30, top=20, ff=24))]),
})


def agree(got, want, dtype, cfg):
    if dtype == torch.float32:
        assert U.error(got, want) < TOL[dtype]
        return
    d = (got.float().cpu() - want).double()
    e = (d - d.mean(-1, keepdim=True)).pow(2).mean(-1).sqrt() / want.double().std()
    limit = TOL[dtype] * len(cfg["layers"]) ** 0.5
    if any(x.get("mlp") for x in cfg["layers"]):
        assert e.quantile(0.5) < limit and e.quantile(0.9) < 4 * limit
    else:
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
@pytest.mark.parametrize("at", FAR)
def test_far_keys(at, dtype):
    cfg, T, toks, without = far_case(at)
    want = U.oracle_logits(cfg, T, toks)
    moved = U.error(U.oracle_logits(cfg, T, without)[-1:], want[-1:])
    limit = TOL[dtype] if dtype == torch.float32 else min(0.4 * moved, 0.05)
    m = U.framework(cfg, T, DEV, dtype)
    assert U.error(m.forward(make_plan([(0, toks, 0)], device=DEV))[-1:], want[-1:]) < limit
    m.forward(make_plan([(1, toks[:-3], 0)], device=DEV))
    for i in range(207, 210):
        got = m.forward(make_plan([(1, toks[i: i + 1], i)], device=DEV))
    assert U.error(got, want[-1:]) < limit


def row_case(H, taps, groups, k, R, seed=0):
    """Rows of one update: residual, update, earlier results with their weights, norm, taps."""
    g = torch.Generator().manual_seed(seed)
    rnd = lambda *s: torch.randn(*s, generator=g)
    return dict(res=rnd(R, H), up=rnd(R, H), scale=1 + 0.2 * rnd(H), stack=rnd(k + 1, R, H), a=rnd(k + 1), w=1 + 0.3 * rnd(H), conv=0.5 * rnd(H, taps))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,groups", [(320, 2), (256, 2), (2048, 2), (72, 3), (75, 5), (50, 2), (1024, 1), (4608, 3), (640, 5), (24, 24)])
@pytest.mark.parametrize("taps", [1, 2, 4, 7])
def test_row_updates(H, groups, taps, dtype):
    """Update, depth average, grouped norm and convolution of several sequences in one launch; a sequence in portions down to one
    row (tiles of more rows than one, and fewer rows than taps, included); passes whose state advances later."""
    k, lens = 3, (1500, 1, 70, 2) if H < 1000 else (700, 1, 30, 2)
    R = sum(lens)
    c = row_case(H, taps, groups, k, R)
    norm = lambda w: ops.RowNorm(w, 1e-3, groups=groups)
    x = c["res"].double() + c["up"].double() * c["scale"]
    mixed = oracle.depth_average(c["a"].double(), [*c["stack"][:k].double(), x])
    h = oracle.grouped_rms_norm(mixed, c["w"].double(), 1e-3, groups)
    starts = [sum(lens[:i]) for i in range(len(lens))]
    want = torch.cat([oracle.input_convolution(h[s: s + n], c["conv"].double()) for s, n in zip(starts, lens)])
    d = {n: t.to(DEV) for n, t in c.items()}
    cv = InputConv(d["conv"].t().contiguous(), len(lens), DEV)
    tol = dict(atol=2e-5, rtol=2e-5) if dtype == torch.float32 else dict(atol=2e-2, rtol=1e-2)

    def run(items, commit=True):                     # items: (sequence, rows, first row)
        idx = torch.cat([torch.arange(starts[s] + p, starts[s] + p + n) for s, n, p in items]).to(DEV)
        stack = d["stack"][:, idx].contiguous()
        up = ops.Update(d["up"][idx], d["scale"])
        up.depth = ops.DepthAverage(stack, k, d["a"])
        res = d["res"][idx]
        keep = res.clone()
        ctx = ops.RowContext(make_plan([(s, [1] * n, p) for s, n, p in items], device=DEV), commit)
        out, new, _ = ops.add_norm_rows(up, res, norm(d["w"]), dtype, conv=cv, ctx=ctx)
        i = idx.cpu()
        assert torch.equal(res, keep) and torch.allclose(new.cpu().double(), mixed[i], atol=1e-5)
        assert torch.allclose(stack[k].cpu().double(), x[i], atol=1e-5) and torch.equal(stack[:k], d["stack"][:k, idx])
        assert out.dtype == dtype and torch.allclose(out.cpu().double(), want[i], **tol)
        return out

    whole = run([(s, n, 0) for s, n in enumerate(lens)])
    for s in range(len(lens)):
        cv.reset(s)
    parts, p = [], 0
    for n in (1, 1, 2, 5, 1, 300, 64, 3, lens[0] - 377):
        parts.append(run([(0, n, p)] + ([(2, lens[2], 0)] if n == 64 else [])))
        p += n
    assert p == lens[0] and torch.equal(torch.cat([x[:n] for x, n in zip(parts, (1, 1, 2, 5, 1, 300, 64, 3, lens[0] - 377))]), whole[: lens[0]])
    cv.reset(0), cv.reset(2)
    run([(2, 9, 0), (0, 4, 0)])
    state = cv.tail.clone()
    run([(0, 6, 4), (2, 5, 9)], commit=False)
    assert torch.equal(cv.tail, state)
    cv.commit_rows(cv.pending[0], cv.pending[1], torch.tensor([2, 5], dtype=torch.int32, device=DEV))
    cv.pending = None
    run([(0, 60, 6), (2, lens[2] - 14, 14)])
    assert torch.equal(cv.tail[1], state[1])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H", [96, 256, 75])
def test_routed_update_of_rows(H, dtype):
    """Expert outputs in pair order or sorted, identity and shared experts, combined inside the tiled update."""
    g = torch.Generator().manual_seed(H)
    rnd = lambda *s: torch.randn(*s, generator=g)
    R, S = 40, 6
    y, wts, res, shared, sg, self_w = rnd(R * S, H), rnd(R, S), rnd(R, H), rnd(R, H), rnd(R), rnd(R)
    self_x = rnd(R, H).to(dtype)
    ids = torch.randint(0, 9, (R, S), generator=g).int()
    ids[3, 1] = ids[7, 5] = -1
    inv = torch.randperm(R * S, generator=g).int()
    w = rnd(H)
    live = (wts * (ids >= 0)).double().unsqueeze(-1)
    for order in (None, inv):
        rows = (y if order is None else y[order.long()]).view(R, S, H).double()
        x = res.double() + (rows * live).sum(1) + self_w.double().unsqueeze(1) * self_x.double() + sg.double().unsqueeze(1) * shared.double()
        dv = lambda t: t.to(DEV)
        pm = cu.PendingMoe(dv(y), dv(wts), dv(ids), S, R, H, dv(shared), dv(sg), dv(order) if order is not None else None, dv(self_w), dv(self_x))
        out, new, _ = ops.add_norm_rows(ops.Update(pm), dv(res), ops.RowNorm(dv(w), 1e-3, groups=3 if H % 3 == 0 else 2), dtype)
        assert torch.allclose(new.cpu().double(), x, atol=1e-4)
        want = oracle.grouped_rms_norm(x, w.double(), 1e-3, 3 if H % 3 == 0 else 2)
        assert torch.allclose(out.cpu().double(), want, atol=1e-4 if dtype == torch.float32 else 4e-2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H", [64, 75, 1])
def test_sinusoidal_embedding(H, dtype):
    table = torch.randn(50, H, generator=torch.Generator().manual_seed(H)).to(dtype)
    pos = torch.tensor([0, 1, 2, 63, 64, 1000, 99999, 7])
    ids = torch.tensor([3, 49, 0, 7, 7, 8, 9, 3])
    freq = 1e4 ** (-torch.arange((H + 1) // 2, dtype=torch.float64) * 2 / H)
    out = torch.empty(2, 8, H, device=DEV)
    got = ops.embed(table.to(DEV), ids.to(DEV), dtype, 1.0, (pos.to(DEV), freq.to(DEV)), out[1])
    want = table[ids].double() + torch.stack([oracle.position_vector(int(p), H) for p in pos])
    assert got.data_ptr() == out[1].data_ptr() and (got.cpu() - want)[:6].abs().max() < 1e-4 and (got.cpu() - want).abs().max() < 8e-3


def attention_case(dtype, n, H, D, V, Lr, sink, gate, seed=0):
    """One attention mixer on its own, with the plain result of the projected rows; scores of a spread that makes every key show."""
    g = torch.Generator().manual_seed(seed)
    rnd = lambda *s: torch.randn(*s, generator=g)
    c = LatentConfig(n_heads=H, head_dim=D, v_dim=V, q_rank=0, kv_rank=Lr, rope_dim=0, scale=1.5 * (D * Lr) ** -0.5, sink=sink, gate=gate)
    uk, uv, kn, sk = rnd(H * D, Lr).to(dtype), (rnd(H * V, Lr) * Lr ** -0.5).to(dtype), 1 + 0.3 * rnd(Lr), 2 * rnd(H) + 2
    w = {"kv_norm": kn, "sink": sk, "out": torch.zeros(8, pad(H * V, 8), dtype=dtype), **latent_up(uk, uv, c, dtype)}
    pages = torch.randperm(40, generator=g).to(torch.int32).view(2, 20)
    cfg = type("C", (), {"norm_eps": 1e-5})
    mx = LatentMixer(cfg, LayerSpec("latent", c, 0), {k: t.to(DEV) for k, t in w.items()}, 40, 64, pages.to(DEV), DEV, dtype)
    rows = rnd(n, mx.off["ff"]).to(dtype)
    rows[:, : mx.nq].view(n, H, mx.Dp)[..., D:] = 0
    rows[:, mx.off["lat"] + Lr: mx.off["lat"] + mx.Lp] = 0
    x = rows.double()
    lat = oracle.rms_norm(x[:, mx.off["lat"]: mx.off["lat"] + Lr], kn.double(), 1e-5)
    q = x[:, : mx.nq].view(n, H, mx.Dp)[..., :D]
    o = oracle.attend(q, (lat @ uk.double().T).view(n, H, D), (lat @ uv.double().T).view(n, H, V), c.scale,
                      sk.double() if sink else torch.full((H,), float("-inf"), dtype=torch.float64))
    gt = x[:, mx.off["g"]: mx.off["g"] + (H * V if gate == "element" else H)]
    return mx, rows.to(DEV), (o * torch.sigmoid(gt).view(n, H, -1)).reshape(n, H * V)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sink,gate", [(True, "element"), (False, "element"), (True, "head")])
@pytest.mark.parametrize("H,D,V,Lr", [(3, 20, 36, 44), (16, 128, 128, 512), (5, 33, 50, 70), (24, 16, 7, 32), (70, 16, 8, 16), (2, 64, 200, 64)])
def test_attention_mechanisms(H, D, V, Lr, sink, gate, dtype):
    n = 290
    mx, rows, want = attention_case(dtype, n, H, D, V, Lr, sink, gate)
    tol = 3e-5 if dtype == torch.float32 else 3e-2
    nv = pad(H * V, 8)

    def run(items):                              # items: (slot, first row, rows)
        plan = make_plan([(s, [1] * m, a) for s, a, m in items], device=DEV)
        cat = torch.full((plan.rows, nv), 7.0, dtype=dtype, device=DEV)
        idx = torch.cat([torch.arange(a, a + m) for _, a, m in items])
        assert ops.latent_mixer(mx, rows[idx.to(DEV)].contiguous(), plan, cat) is not None
        got, ref = cat[:, : H * V].double().cpu(), want[idx]
        assert (cat[:, H * V:] == 7).all() and (got - ref).norm() < tol * ref.norm(), items
    run([(0, 0, n)])
    i = 0
    for m in (3, 61, 1, 64, 31, 70, 1, 1, 58):
        run([(1, i, m)] if m < 60 else [(0, n - 5, 5), (1, i, m), (0, n - 1, 1)])
        i += m
    assert i == n


@pytest.mark.parametrize("E,top,F", [(6, 2, 40), (1, 1, 8), (13, 1, 104), (60, 8, 136), (500, 30, 16)])
@pytest.mark.parametrize("H", [64, 264, 75])
@pytest.mark.parametrize("limit", [0.6, 1e9])
def test_experts(E, top, F, H, limit):
    """Fused decode router, pair GEMVs, grouped products and the FP32-unit form against the plain form on rows without close calls;
    logits far apart (all but the chosen ones vanish from a softmax over all)."""
    g = torch.Generator().manual_seed(E)
    c = MoeConfig(n_experts=E, top_k=top, ffn=F, n_shared=0, router="topk_softmax", swiglu_limit=limit, glu_alpha=1.702, glu_shift=1.0)
    rnd = lambda *s: torch.randn(*s, generator=g)
    for spread in (3.0, 60.0):
        flat = {"router": rnd(E, H) * spread * H ** -0.5, "router.b": spread / 3 * rnd(E)}
        for k in [f"e{j}." for j in range(E)]:
            flat[k + "gate"], flat[k + "up"], flat[k + "down"] = rnd(F, H) * 2 * H ** -0.5, rnd(F, H) * H ** -0.5, rnd(H, F) * F ** -0.5
        flat = {k: t.bfloat16().float() for k, t in flat.items()}
        w = {"gate": flat["router"], "w_gu": torch.stack([stack_rows([flat[f"e{j}.gate"], flat[f"e{j}.up"]], 128) for j in range(E)]),
             "w_down": torch.stack([pad_cols(flat[f"e{j}.down"], pad(F, 128)) for j in range(E)])}
        mlp = {"router": {"experts": E, "top": top}, "expert": {"limit": limit}}
        for R in (1, 16, 17, 230):
            h = rnd(R, H).bfloat16().float()
            want = oracle.experts(h, flat, "", mlp)
            s = (h @ flat["router"].T + flat["router.b"]).sort(-1, descending=True).values
            clear = torch.ones(R, dtype=torch.bool) if top == E else s[:, top - 1] - s[:, top] > 1e-3
            assert clear.float().mean() > 0.8
            for dt in DTYPES:
                wd = {k: t.to(dt).cuda() for k, t in w.items()}
                wd["bias"] = flat["router.b"].cuda()
                got = ops.moe(h.to(dt).cuda(), wd, c).float().cpu()
                err = ((got - want).norm(dim=-1) / want.norm(dim=-1))[clear]
                assert err.max() < (4e-5 if dt == torch.float32 else 2e-2), (R, dt, spread)


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
    """Greedy generation in captured rounds, 200 tokens across page borders: every token is the oracle's choice for the text before
    it (bf16: nearly always among the choices within rounding)."""
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
    """Every step of a mixed batch, by the runner's own process in 32-bit."""
    cfg, T = _setup(U.MIXED)
    U.write_checkpoint(tmp_path / "ck", cfg, T)
    lens = {"a": 130, "b": 66, "c": 5, "d": 64, "e": 127, "f": 2}
    toks = {k: U.prompt(n, cfg["vocab"], ord(k)) for k, n in lens.items()}
    at, steps, places = dict.fromkeys(lens, 0), [], []
    for i, st in enumerate(MIX_STEPS):
        ent = []
        for x in st:
            if x[0] != "/":
                n = int(x[1:])
                ent.append({"id": x[0], "tokens": toks[x[0]][at[x[0]]: at[x[0]] + n], "want": [0, n - 1] if n > 1 else [0]})
                at[x[0]] += n
        places.append([(e["id"], at[e["id"]] - len(e["tokens"]) + w) for e in ent for w in e["want"]])
        steps.append({"step": i, "entries": ent, "end": [x[1:] for x in st if x[0] == "/"]})
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    r = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", str(tmp_path / "ck"), "--dtype", "float32",
                        "--out", str(tmp_path), "--max-tokens", "448"], input="\n".join(json.dumps(s) for s in steps) + "\n",
                       capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(len(steps))]
    want = {k: U.oracle_logits(cfg, T, t) for k, t in toks.items()}
    for i, pl in enumerate(places):
        got = torch.from_numpy(np.fromfile(tmp_path / f"{i}.f32", "<f4").reshape(-1, cfg["vocab"]))
        assert U.error(got, torch.stack([want[k][p] for k, p in pl])) < 3e-5, i
