"""Debisun on a B200: the kernels of each mechanism and whole models, in bf16 and in 32-bit, against the plain implementation;
portions, mixed batches, page and chunk edges, captured decode rounds, the server.

A routed model in bf16 may take another expert than the plain one where two choice scores are closer than rounding, and a token
side of width one is +1 or -1 times its weight by the sign of a number that may be close to 0: such models are compared by the ninth
decile of their rows in bf16 (and by the worst row in 32-bit); the expert kernels have a test of their own on rows without close
calls."""
import json
import os
import subprocess
import sys

import debisun_oracle as oracle
import debisun_util as U
import numpy as np
import pytest
import torch
from test_debisun import FAR, _serve, _setup

from spark_engine_b200 import ops
from spark_engine_b200.config import EngineConfig, MoeConfig
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
    "heads of 128": dict(layers=[U.layer(U.dense(264), heads=8, kv_heads=2, dim=128, vdim=128, scale=0.09)], width=264),
    "wide values": dict(layers=[U.layer(heads=2, kv_heads=1, dim=64, vdim=200, scale=0.12)]),
    "wide keys": dict(layers=[U.layer(heads=2, kv_heads=1, dim=256, vdim=256, scale=0.06)], width=136),
    "very wide": dict(layers=[U.layer(heads=1, kv_heads=1, dim=320, vdim=272, scale=0.06)]),
    "40 query heads per key head": dict(layers=[U.layer(heads=40, kv_heads=1, dim=16, vdim=8, scale=0.25)]),
    "many experts": dict(layers=[U.layer(U.moe(experts=40, identity=24, top=6, ff=264, shared=136), dim=32, vdim=32)], width=136),
    "more pairs than a decode round's": dict(layers=[U.layer(U.moe(experts=30, identity=2, top=20, ff=24))]),
})


def agree(got, want, dtype, cfg):
    close_calls = cfg["token_side"]["dim"] == 1 or any(x.get("mlp") and x["mlp"]["kind"] == "moe" for x in cfg["layers"])
    if dtype == torch.float32 or not close_calls:
        assert U.error(got, want) < TOL[dtype] * (len(cfg["layers"]) ** 0.5 if dtype == torch.bfloat16 else 1)
        return
    d = (got.float().cpu() - want).double()
    e = (d - d.mean(-1, keepdim=True)).pow(2).mean(-1).sqrt() / want.double().std()
    assert e.quantile(0.9) < TOL[dtype] * len(cfg["layers"]) ** 0.5


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
    mc = U.D.read_config(cfg)
    ses = BatchSession(mc, U.D.from_tensors(mc, T, DEV, dtype), EngineConfig(dtype="float32" if dtype == torch.float32 else "bfloat16"), DEV,
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
@pytest.mark.parametrize("chunk,at", FAR)
def test_a_key_is_seen_inside_its_chunk_only(chunk, at, dtype):
    cfg, T = _setup(dict(layers=[U.layer(chunk=chunk)]), 7)
    qt, kt, fill = U.planted_pair(cfg, T)
    toks = [fill[i % len(fill)] for i in range(209)] + [qt]
    plain = U.oracle_logits(cfg, T, toks)
    other = list(toks)
    other[at] = kt
    want = U.oracle_logits(cfg, T, other)
    seen = 209 // chunk == at // chunk
    moved = U.error(plain[-1:], want[-1:])
    assert (moved > 0.05) == seen
    limit = TOL[dtype] if dtype == torch.float32 else min(0.4 * moved, 0.03) if seen else 0.03
    m = U.framework(cfg, T, DEV, dtype)
    assert U.error(m.forward(make_plan([(0, other, 0)], device=DEV))[-1:], want[-1:]) < limit
    m.forward(make_plan([(1, other[:-3], 0)], device=DEV))
    for i in range(207, 210):
        got = m.forward(make_plan([(1, other[i: i + 1], i)], device=DEV))
    assert U.error(got, want[-1:]) < limit
    # hidden from the row, the planted token must not change a bit of what the row attends to
    if not seen:
        m.forward(make_plan([(2, toks[:-3], 0)], device=DEV))
        for i in range(207, 210):
            same = m.forward(make_plan([(2, toks[i: i + 1], i)], device=DEV))
        assert torch.equal(same, got)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H", [8, 75, 264, 2048, 4096, 4100, 8192, 8200])
def test_row_updates(H, dtype):
    """Residual plus scaled rows, RMS-normed rows, or routed outputs; layer norm, RMS norm or the rows themselves."""
    from spark_engine_b200.ops import cuda as cu
    g = torch.Generator().manual_seed(H)
    rnd = lambda *s: torch.randn(*s, generator=g)
    for R in (3, 160):
        res, delta, sc, w, b, pw = rnd(R, H) + 0.5, rnd(R, H), rnd(H), 1 + 0.2 * rnd(H), rnd(H), rnd(H)
        slots = 3
        y, wts, ids = rnd(R * slots, H), torch.rand(R, slots, generator=g), torch.randint(-1, 4, (R, slots), generator=g)
        inv = torch.randperm(R * slots, generator=g)
        shared, sg, own, x = rnd(R, H), torch.rand(R, generator=g), torch.rand(R, generator=g), rnd(R, H).to(dtype)
        c = lambda t: t.cuda() if t is not None else None
        i32 = lambda t: t.to(torch.int32).cuda()
        mix = (y[inv].view(R, slots, H) * (wts * (ids >= 0)).unsqueeze(-1)).sum(1) + own.unsqueeze(1) * x.float() + sg.unsqueeze(1) * shared
        moe = cu.PendingMoe(c(y), c(wts), i32(ids), slots, R, H, c(shared), c(sg), i32(inv), c(own), c(x))
        rms = lambda t: t / torch.sqrt(t.pow(2).mean(-1, keepdim=True) + 1e-5)
        for upd, ref in ((None, 0), (ops.Update(c(delta), c(sc)), delta * sc), (ops.Update(moe, c(sc)), mix * sc),
                         (ops.Update(c(delta), post=ops.RowNorm(c(pw), 1e-5)), rms(delta) * pw)):
            new = res + ref
            for norm, h in ((None, new), (ops.RowNorm(c(w), 1e-5), rms(new) * w), (ops.RowNorm(c(w), 1e-5, one_plus=True), rms(new) * (1 + w)),
                            (ops.RowNorm(c(w), 1e-5, c(b)), torch.nn.functional.layer_norm(new, (H,), w, b, 1e-5))):
                got, X, h32 = ops.add_norm_rows(upd, res.clone().cuda(), norm, dtype, True)
                assert torch.allclose(X.cpu(), new, atol=2e-5) and torch.allclose(h32.cpu(), h, atol=1e-4)
                assert torch.allclose(got.float().cpu(), h, atol=1e-4, rtol=1e-5 if dtype == torch.float32 else 8e-3)


@pytest.mark.parametrize("R,N,K", [(1, 40, 64), (16, 512, 1024), (5, 2080, 256), (3, 2048, 7680), (16, 24000, 64), (40, 72, 128), (300, 520, 96),
                                   (700, 4096, 64), (9, 30, 37), (70, 30, 37)])
def test_activations_of_products(R, N, K):
    """Squared relu and token rows gated by the product, on every product kernel."""
    g = torch.Generator().manual_seed(N)
    for dt in DTYPES:
        x, w = torch.randn(R, K, generator=g).to(dt), (torch.randn(N, K, generator=g) * K ** -0.5).to(dt)
        table, n, off = torch.randn(50, 2 * N + 8, generator=g).to(dt), N - 3, N + 2
        ids = torch.randint(0, 50, (R,), generator=g)
        if R > 2:
            ids[1] = 50                                      # outside the table: a zero row
        ref = x.double() @ w.double().T
        tol = dict(atol=1e-4 if dt == torch.float32 else 2e-2, rtol=1e-4 if dt == torch.float32 else 1e-2)
        assert torch.allclose(ops.linear_relu2(x.cuda(), w.cuda()).cpu().double(), oracle.relu_squared(ref), **tol)
        e = table.double()[ids.clamp(max=49)][:, off: off + n] * (ids < 50).unsqueeze(1)
        want = torch.zeros(R, N, dtype=torch.float64)
        want[:, :n] = oracle.gelu_tanh(ref)[:, :n] * e
        got = ops.linear_token_gate(x.cuda(), w.cuda(), table.cuda(), ids.cuda(), off, n).cpu().double()
        assert torch.allclose(got, want, **tol)


@pytest.mark.parametrize("E,I,top,F", [(6, 3, 2, 40), (1, 0, 1, 8), (60, 20, 8, 136), (500, 100, 30, 16)])
@pytest.mark.parametrize("H", [64, 264, 75])
def test_experts(E, I, top, F, H):
    """Fused decode router, pair GEMVs, grouped products and the FP32-unit form against the plain form on rows without close calls."""
    from spark_engine_b200.models.layout import pad, pad_cols, stack_rows
    g = torch.Generator().manual_seed(E)
    c = MoeConfig(n_experts=E, n_identity=I, top_k=top, ffn=F, n_shared=1, shared_ffn=F, router="softmax_bias", route_scale=1.7, shared_gate=True,
                  act="relu2")
    rnd = lambda *s: torch.randn(*s, generator=g)
    flat = {"router": rnd(E + I, H) * 3 * H ** -0.5, "correction": 0.3 * rnd(E + I), "shared.sg": rnd(1, H) * H ** -0.5}
    for k in [f"e{j}." for j in range(E)] + ["shared."]:
        flat[k + "up"], flat[k + "down"] = rnd(F, H) * H ** -0.5, rnd(H, F) * F ** -0.5
    flat = {k: t if k == "correction" else t.bfloat16().float() for k, t in flat.items()}
    Fp = pad(F, 8)
    w = {"gate": torch.cat((flat["router"], flat["shared.sg"])), "bias": flat["correction"],
         "w_up": torch.stack([stack_rows([flat[f"e{j}.up"]]) for j in range(E)]), "w_down": torch.stack([pad_cols(flat[f"e{j}.down"], Fp) for j in range(E)]),
         "s_up": stack_rows([flat["shared.up"]]), "s_down": pad_cols(flat["shared.down"], Fp)}
    mlp = {"router": {"experts": E, "identity": I, "top": top, "scale": 1.7}, "shared": {"ff": F}}
    for R in (1, 16, 17, 230):
        h = rnd(R, H).bfloat16().float()
        want = oracle.experts(h, flat, "", mlp)
        s = (torch.softmax(h @ flat["router"].T, -1) + flat["correction"]).sort(-1, descending=True).values
        clear = torch.ones(R, dtype=torch.bool) if top == E + I else s[:, top - 1] - s[:, top] > 1e-5
        assert clear.float().mean() > 0.8
        for dt in DTYPES:
            wd = {k: t.cuda() if k == "bias" else t.to(dt).cuda() for k, t in w.items()}
            got = ops.moe(h.to(dt).cuda(), wd, c).float().cpu()
            err = ((got - want).norm(dim=-1) / want.norm(dim=-1))[clear]
            assert err.max() < (2e-5 if dt == torch.float32 else 1e-2), (R, dt)


def test_rows_do_not_depend_on_the_batch():
    """The same decode rows alone, and beside other sequences whose pages and slots differ: bitwise equal."""
    cfg, T = _setup(U.MIXED)
    m = U.framework(cfg, T, DEV, torch.bfloat16)
    toks = U.prompt(100, cfg["vocab"])
    for s, n in ((0, 90), (1, 40), (3, 90)):
        m.forward(make_plan([(s, toks[:n], 0)], device=DEV))
    alone = m.forward(make_plan([(0, toks[90:91], 90)], device=DEV))
    both = m.forward(make_plan([(1, toks[40:41], 40), (3, toks[90:91], 90)], device=DEV))
    assert torch.equal(alone[0], both[1])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_captured_rounds_generate_the_oracles_text(dtype):
    """Greedy generation in captured rounds, 200 tokens across page and chunk borders: every token is the oracle's choice for the
    text before it (bf16: nearly always among the choices within rounding)."""
    cfg, T = _setup(U.MIXED)
    mc = U.D.read_config(cfg)
    eng = LLMEngine(mc, U.D.from_tensors(mc, T, DEV, getattr(torch, dtype)), EngineConfig(dtype=dtype), device=DEV, max_seqs=3, kv_tokens_per_seq=512)
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
    mc = U.D.read_config(cfg)
    es = EngineServer(mc, U.D.from_tensors(mc, T, DEV, torch.float32),
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
