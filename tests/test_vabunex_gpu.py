"""Vabunex on a B200: the kernels of each mechanism and whole models, in bf16 and in 32-bit, against the plain
implementation; portions, mixed batches, page and chunk edges, captured decode rounds, the server."""
import itertools

import pytest
import torch
import vabunex_oracle as oracle
import vabunex_util as U
from test_vabunex import FAR, MECHANISMS, MIXED, _serve, _setup, planted_pair

from spark_engine_b200.config import EngineConfig
from spark_engine_b200.models.plan import make_plan
from spark_engine_b200.serving.engine import LLMEngine
from spark_engine_b200.serving.session import BatchSession
from spark_engine_b200.serving.worker import EngineServer

pytestmark = pytest.mark.gpu
TOL = {torch.float32: 2e-5, torch.bfloat16: 3e-2}


def tol(dtype, cfg):
    """Limit for the worst row: bf16 rounding of independent layer runs adds up like a random walk."""
    return TOL[dtype] * (len(oracle.layer_runs(cfg)) ** 0.5 if dtype == torch.bfloat16 else 1.0)


DTYPES = [torch.float32, torch.bfloat16]
DEV = "cuda"

# shapes of the tensor-core kernels: head sizes around the compiled widths, several value tiles, heads beyond one MMA tile
SHAPES = dict(MECHANISMS)
SHAPES.update({
    "lightning 64": dict(layers=[U.lightning(heads=2, dim=64, vdim=136, ff=264)], width=264),
    "lightning 128": dict(layers=[U.lightning(heads=2, dim=128, vdim=48)], width=136),
    "lightning 160": dict(layers=[U.lightning(heads=1, dim=160, vdim=32)], width=136),
    "wkv 64": dict(layers=[U.wkv(heads=3, dim=64, ff=136)], width=200),
    "wkv 128": dict(layers=[U.wkv(heads=1, dim=128)], width=136),
    "latent 128": dict(layers=[U.latent(heads=20, dim=128, vdim=128, rot_dim=64, q_rank=136, kv_rank=200, scale=0.09)], width=136),
    "latent wide value": dict(layers=[U.latent(heads=2, dim=48, vdim=200, rot_dim=24, kv_rank=72)]),
    "latent 66 heads": dict(layers=[U.latent(heads=66, dim=16, vdim=8, rot_dim=4)]),
})


def _ids(n, cfg, seed=0):
    return U.prompt(n, cfg["vocab"], seed)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(SHAPES))
def test_prompt_then_decoding(name, dtype):
    cfg, T = _setup(SHAPES[name])
    toks = _ids(150, cfg)
    want = U.oracle_logits(cfg, T, toks)
    m = U.framework(cfg, T, DEV, dtype)
    assert U.error(m.forward(make_plan([(0, toks, 0)], device=DEV)), want) < tol(dtype, cfg)
    out, i = [], 0
    for n in (2, 31, 2, 33, 64, *[1] * 18):
        out.append(m.forward(make_plan([(3, toks[i: i + n], i)], device=DEV)))
        i += n
    assert U.error(torch.cat(out), want) < tol(dtype, cfg)


@pytest.mark.parametrize("dtype", DTYPES)
def test_mixed_batches_equal_each_request_alone(dtype):
    cfg, T = _setup(MIXED)
    mc = U.V.read_config(cfg)
    W = U.V.from_tensors(mc, T, DEV, dtype)
    ses = BatchSession(mc, W, EngineConfig(dtype="float32" if dtype == torch.float32 else "bfloat16"), DEV, max_seqs=4,
                       kv_tokens=320 + 192 + 64 + 128)
    lens = {"a": 300, "b": 180, "c": 3, "d": 100, "e": 121}
    toks = {k: _ids(n, cfg, ord(k)) for k, n in lens.items()}
    want = {k: U.oracle_logits(cfg, T, t) for k, t in toks.items()}
    at = dict.fromkeys(lens, 0)
    for st in (("a70", "b1", "c2"), ("a1", "b100", "d33"), ("a2", "b31", "c1", "d2"), ("/c", "a128", "b2", "d64"), ("/b", "a1", "d1"),
               ("/d", "a64", "e1"), ("a33", "e120"), ("a1",)):
        for x in st:
            if x[0] == "/":
                ses.end(x[1:])
        ent = [(x[0], toks[x[0]][at[x[0]]: at[x[0]] + int(x[1:])], list(range(int(x[1:])))) for x in st if x[0] != "/"]
        got, r = ses.step(ent), 0
        for k, t, _ in ent:
            assert U.error(got[r: r + len(t)], want[k][at[k]: at[k] + len(t)]) < tol(dtype, cfg), (k, at[k], len(t))
            r += len(t)
            at[k] += len(t)
    assert at["a"] == 300


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("at", FAR)
def test_a_far_key_is_found(at, dtype):
    cfg, T = _setup(dict(layers=[U.latent()]), 7)
    qt, kt, fill = planted_pair(cfg, T)
    toks = [fill[i % len(fill)] for i in range(192)] + [qt, fill[0], qt]
    plain = U.oracle_logits(cfg, T, toks)
    toks[at] = kt
    want = U.oracle_logits(cfg, T, toks)
    tol = TOL[dtype] if dtype == torch.float32 else 0.4 * U.error(plain[-1:], want[-1:])
    m = U.framework(cfg, T, DEV, dtype)
    assert U.error(m.forward(make_plan([(0, toks, 0)], device=DEV))[-1:], want[-1:]) < tol
    m.forward(make_plan([(1, toks[:-3], 0)], device=DEV))
    for i in range(192, 195):
        got = m.forward(make_plan([(1, toks[i: i + 1], i)], device=DEV))
    assert U.error(got, want[-1:]) < tol


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("D,Vd", [(24, 40), (64, 64), (128, 72)])
@pytest.mark.parametrize("mode", ["scalar", "channel"])
def test_recurrences_carry_one_large_key_across_chunk_edges(mode, D, Vd, dtype):
    """Every place around the 16- and 64-row edges gets one large key in turn (heads = places); decays of 1, of 0 and strong
    ones; short and long segments of two sequences in one launch, from a state that is not zero."""
    from spark_engine_b200 import ops
    places = [0, 1, 15, 16, 17, 47, 48, 62, 63, 64, 65, 80, 127, 128]
    H, n0, n1 = len(places), 150, 9
    g = torch.Generator().manual_seed(5)
    rnd = lambda *s: torch.randn(*s, generator=g).to(dtype).float()
    q, k, v = (rnd(n0 + n1, H, x) * 0.3 for x in (D, D, Vd))
    for h, p in enumerate(places):
        k[p, h] *= 64
    q, k, v = (x.to(dtype).double() for x in (q, k, v))
    S0 = torch.randn(4, H, D, Vd, generator=g)
    if mode == "scalar":
        a = torch.tensor([1.0, 0.0, 0.5, 0.999, 0.01] * H)[:H].double()
        kw = {"log2a": torch.log2(a).clamp_min(-1000).float().cuda()}
        step = lambda S, t: (a.view(H, 1, 1) * S + k[t].unsqueeze(-1) * v[t].unsqueeze(-2),) * 2
    else:
        logw = -torch.exp(torch.randn(n0 + n1, H, D, generator=g) * 1.5 - 1).double()
        logw[:, 1] = logw[:, 1] * 30                         # decays that leave nothing within a few rows
        logw[:, 2] = -1e-6
        logw = logw.clamp_min(-105).float().double()
        u = torch.randn(H, D, generator=g)
        kw = {"logw": logw.float().view(-1, H * D).cuda(), "u": u.cuda()}

        def step(S, t):
            kv = k[t].unsqueeze(-1) * v[t].unsqueeze(-2)
            return torch.exp(logw[t]).unsqueeze(-1) * S + kv, S + u.double().unsqueeze(-1) * kv
    want, ends = [], {}
    for slot, r0, n in ((2, 0, n0), (1, n0, n1)):
        S = S0[slot].double()
        for t in range(r0, r0 + n):
            S, O = step(S, t)
            want.append(torch.einsum("hd,hdv->hv", q[t], O))
        ends[slot] = S
    want = torch.stack(want)
    plan = make_plan([(2, [0] * n0, 0), (1, [0] * n1, 0)], device=DEV)
    f = lambda x: x.to(dtype).view(n0 + n1, -1).cuda()
    for commit in (False, True):
        S = S0.clone().cuda()
        got = ops.linear_state(f(q), f(k), f(v), H, D, Vd, S, plan, commit, **kw).cpu().view(n0 + n1, H, Vd).double()
        scale = want.abs().amax((0, 2), keepdim=True)
        assert ((got - want) / scale).abs().max() < 3e-5, (commit, ((got - want) / scale).abs().amax((0, 2)))
        for slot in (1, 2):
            ref = ends[slot] if commit else S0[slot].double()
            assert torch.allclose(S[slot].cpu().double(), ref, rtol=1e-4, atol=1e-4 * float(ref.abs().max()))
    # commit of the first rows only
    S = S0.clone().cuda()
    cnt = torch.tensor([3, 0], dtype=torch.int32, device=DEV)
    ops.linear_state(f(q), f(k), f(v), H, D, Vd, S, plan, True, n_rows=cnt, **kw)
    ref = S0[2].double()
    for t in range(3):
        ref = step(ref, t)[0]
    assert torch.allclose(S[2].cpu().double(), ref, rtol=1e-4, atol=1e-4 * float(ref.abs().max())) and torch.equal(S[1].cpu(), S0[1])


def test_simt_product_shapes():
    from spark_engine_b200.ops import cuda as cu
    g = torch.Generator().manual_seed(0)
    for (M, N, K), dt in itertools.product([(1, 5, 3), (70, 130, 37), (16, 64, 100)], DTYPES):
        a, b = torch.randn(M, K, generator=g).to(dt), torch.randn(N, K, generator=g).to(dt)
        got = cu.dense_linear(a.cuda(), b.cuda(), out_f32=True).cpu().double()
        ref = a.double() @ b.double().T
        assert torch.allclose(got, ref, atol=2e-5 * K ** 0.5)


@pytest.mark.parametrize("N,K", [(2048, 6400), (2056, 10272), (4100, 7680)])
def test_long_contractions_of_decode_rows(N, K):
    """Output products of wide feed-forwards: rows staged in segments; one row's bits do not depend on the others."""
    from spark_engine_b200.ops import cuda as cu
    g = torch.Generator().manual_seed(1)
    x, w = torch.randn(16, K, generator=g).bfloat16().cuda(), (torch.randn(N, K, generator=g) * K ** -0.5).bfloat16().cuda()
    ref = x.double() @ w.double().T
    full = cu.dense_linear(x, w, out_f32=True)
    assert (full.double() - ref).abs().max() < 1e-4
    for r in (1, 3, 8, 9):
        assert torch.equal(cu.dense_linear(x[:r], w, out_f32=True), full[:r])


def test_rows_do_not_depend_on_the_batch():
    """The same decode rows alone, and beside other sequences whose pages and slots differ: bitwise equal."""
    cfg, T = _setup(MIXED)
    m = U.framework(cfg, T, DEV, torch.bfloat16)
    toks = _ids(100, cfg)
    for s, n in ((0, 90), (1, 40), (3, 90)):
        m.forward(make_plan([(s, toks[:n], 0)], device=DEV))
    alone = m.forward(make_plan([(0, toks[90:91], 90)], device=DEV))
    both = m.forward(make_plan([(1, toks[40:41], 40), (3, toks[90:91], 90)], device=DEV))
    assert torch.equal(alone[0], both[1])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_captured_rounds_generate_the_oracles_text(dtype):
    """Greedy generation in captured rounds, 200 tokens across page borders: every token is the oracle's choice for the text
    before it (bf16: among the choices within rounding)."""
    cfg, T = _setup(MIXED)
    mc = U.V.read_config(cfg)
    W = U.V.from_tensors(mc, T, DEV, getattr(torch, dtype))
    eng = LLMEngine(mc, W, EngineConfig(dtype=dtype), device=DEV, max_seqs=3, kv_tokens_per_seq=512)
    assert eng.use_graphs
    prompts = [_ids(n, cfg, n) for n in (1, 100, 62)]
    outs = eng.generate(prompts, max_new=200)
    fed = [eng.model.seqs[s].length for s in range(3)]
    more = eng.decode_steps([0, 1, 2], [o[-1] for o in outs], 40)
    assert [eng.model.seqs[s].length for s in range(3)] == [n + 40 for n in fed]
    eng.check_device_status()
    for i, (p, o) in enumerate(zip(prompts, outs)):
        o = o + [r[i] for r in more]
        want = U.oracle_logits(cfg, T, p + o)[len(p) - 1: -1]
        chosen = want.gather(1, torch.tensor(o).view(-1, 1))[:, 0]
        slack = 1e-4 if dtype == "float32" else 0.25
        assert (want.amax(-1) - chosen).max() <= slack * want.std(), i


@pytest.mark.parametrize("drafts", [False, True])
def test_server_in_32_bit_generates_the_oracles_text(drafts):
    cfg, T = _setup(MIXED)
    mc = U.V.read_config(cfg)
    es = EngineServer(mc, U.V.from_tensors(mc, T, DEV, torch.float32),
                      EngineConfig(max_seqs=2, kv_tokens=1024, prefill_chunk=48, spec="lookup" if drafts else "none", spec_depth=3,
                                   dtype="float32"), device=DEV)
    prompts = {i: _ids(n, cfg, n) for i, n in enumerate((41, 7, 90, 3))}
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
    """The command: a trace on standard input, one file of logits per step, `done` lines, exit code 0."""
    import json
    import os
    import subprocess
    import sys

    import numpy as np
    cfg, T = _setup(MIXED)
    U.write_checkpoint(tmp_path / "ck", cfg, T)
    toks = _ids(70, cfg)
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
    assert U.error(get(0), want[[0, 39]]) < 2e-5 and U.error(get(2), want[[69, 0]]) < 2e-5
    assert not (tmp_path / "1.f32").exists()
    assert oracle.layer_runs(cfg) == [0, 1, 2, 3, 1, 2, 3, 4]
