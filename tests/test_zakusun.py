"""Zakusun on the CPU: every mechanism against the plain implementation, the checkpoint reader, the paged latents and the
convolutions' state, portions and batches, prefix snapshots, speculation, and greedy generation through the engine and the
server's scheduler."""
import dataclasses
import json
import math

import pytest
import torch
import zakusun_oracle as oracle
import zakusun_util as U
from test_vabunex import _serve

from spark_engine_b200 import ops
from spark_engine_b200.cache.kv import KvManager
from spark_engine_b200.config import EngineConfig, ModelConfig, MoeConfig, get_model_config
from spark_engine_b200.models.checkpoint import load_checkpoint, load_config, save_checkpoint
from spark_engine_b200.models.input_conv import InputConv
from spark_engine_b200.models.model import Model
from spark_engine_b200.models.plan import make_plan
from spark_engine_b200.serving.engine import LLMEngine
from spark_engine_b200.serving.session import BatchSession
from spark_engine_b200.serving.worker import EngineServer


def _setup(name, seed=1):
    cfg = U.config(**(U.MECHANISMS[name] if isinstance(name, str) else name))
    return cfg, U.tensors(cfg, seed)


@pytest.mark.parametrize("name", list(U.MECHANISMS))
def test_whole_prompt_and_token_by_token(name):
    cfg, T = _setup(name)
    toks = U.prompt(80, cfg["vocab"])
    want = U.oracle_logits(cfg, T, toks)
    m = U.framework(cfg, T)
    assert U.error(m.forward(make_plan([(0, toks, 0)])), want) < 2e-5
    one = torch.cat([m.forward(make_plan([(2, [t], i)])) for i, t in enumerate(toks)])
    assert U.error(one, want) < 2e-5
    assert U.error(one[:3], want[:3]) < 2e-5


def test_residual_stream_after_every_layer():
    cfg, T = _setup(U.MIXED)
    toks, taps = U.prompt(9, cfg["vocab"]), []
    U.oracle_logits(cfg, T, toks, taps)
    m = U.framework(cfg, T)
    m.tap_layers = set(range(len(taps)))
    m.forward(make_plan([(1, toks, 0)]))
    for i, x in enumerate(taps):
        assert torch.allclose(m.taps[i].double(), x, atol=2e-4), i


def test_plain_mechanisms():
    """The plain functions themselves, on cases that can be done by hand."""
    x = torch.tensor([[3.0, 4.0, 0.0, 2.0]], dtype=torch.float64)
    y = oracle.grouped_rms_norm(x, torch.tensor([1.0, 2.0, 1.0, 1.0]), 0.0, 2)
    assert torch.allclose(y, torch.tensor([[3 / math.sqrt(12.5), 8 / math.sqrt(12.5), 0.0, math.sqrt(2.0)]], dtype=torch.float64))
    assert torch.allclose(oracle.rms_norm(x, torch.ones(4), 0.0)[0, 3], torch.tensor(2 / math.sqrt(29 / 4), dtype=torch.float64))
    v = oracle.position_vector(3, 5)
    f = 10000 ** (-2 / 5)
    assert v.tolist() == pytest.approx([math.sin(3), math.cos(3), math.sin(3 * f), math.cos(3 * f), math.sin(3 * f * f)])
    h = torch.tensor([[1.0], [2.0], [4.0]])
    assert oracle.input_convolution(h, torch.tensor([[0.5, 0.25]])).flatten().tolist() == [1.25, 2.5 + 0.5, 5.0 + 1.0]
    s, sink = torch.tensor([[1.0, 2.0]]), torch.tensor([3.0])
    assert torch.allclose(oracle.softmax_with(sink, s), torch.exp(s) / (torch.exp(s).sum() + math.exp(3.0)))
    W = {"gate": torch.tensor([[1.0], [-3.0]]), "up": torch.tensor([[-5.0], [0.5]]), "down": torch.eye(2)}
    sg = lambda z: 1 / (1 + math.exp(-1.702 * z))
    assert oracle.expert(torch.tensor([2.0]), W, "", 1.5).tolist() == pytest.approx([1.5 * sg(1.5) * -0.5, -6 * sg(-6.0) * 2.0])
    W = {"router": torch.tensor([[1.0], [2.0], [3.0]]), "router.b": torch.tensor([2.5, 0.0, 0.0])}
    w, ids = oracle.routed(torch.tensor([[1.0]]), W, "", 2)
    assert ids.tolist() == [[0, 2]] and torch.allclose(w, torch.softmax(torch.tensor([[3.5, 3.0]]), -1))
    assert oracle.depth_average(torch.tensor([2.0, -1.0]), [torch.tensor([1.0]), torch.tensor([5.0])]).tolist() == [-3.0]


@pytest.mark.parametrize("tensor", ["l0.mix.sink", "l0.canon1", "l0.canon2", "l1.dwa", "l0.mlp.router.b", "l0.mix.g", "l0.mix.dkv.norm"])
def test_every_small_tensor_shows(tensor):
    cfg, T = _setup(U.MIXED)
    toks = U.prompt(40, cfg["vocab"])
    want = U.oracle_logits(cfg, T, toks)
    assert U.error(U.framework(cfg, T).forward(make_plan([(0, toks, 0)])), want) < 2e-5
    x = T[tensor].float()
    T[tensor] = (torch.cat((x[..., 1:], x[..., :1]), -1) if x.dim() > 1 else x.flip(0) + 1.0).to(torch.bfloat16)
    other = U.oracle_logits(cfg, T, toks)
    assert U.error(other, want) > 0.02
    assert U.error(U.framework(cfg, T).forward(make_plan([(0, toks, 0)])), other) < 2e-5


@pytest.mark.parametrize("groups", [1, 2, 3, 8])
def test_grouped_norm(groups):
    g = torch.Generator().manual_seed(groups)
    x, w = torch.randn(7, 24, generator=g) * torch.arange(1, 25), torch.randn(24, generator=g)
    h, res, _ = ops.add_norm_rows(None, x, ops.RowNorm(w, 1e-3, groups=groups), torch.float32)
    assert torch.allclose(h, oracle.grouped_rms_norm(x, w, 1e-3, groups), atol=1e-5) and torch.equal(res, x)


@pytest.mark.parametrize("taps", [1, 2, 3, 6])
def test_input_convolution_over_cuts(taps):
    """Every cut of a sequence, beside another sequence; a pass that does not commit leaves the state alone until its accepted rows
    are replayed."""
    g = torch.Generator().manual_seed(taps)
    N, H = 14, 8
    rows, w = torch.randn(2, N, H, generator=g), torch.randn(H, taps, generator=g)
    want = [oracle.input_convolution(rows[s], w) for s in (0, 1)]
    cv = InputConv(w.t().contiguous(), 3, "cpu")
    run = lambda items, commit=True: ops.add_norm_rows(
        None, torch.cat([rows[s][p: p + len(t)] for s, t, p in items]), None, torch.float32, conv=cv,
        ctx=ops.RowContext(make_plan([(s + 1, t, p) for s, t, p in items]), commit))[0]
    for cut in range(1, N):
        cv.reset(1)
        got = torch.cat((run([(0, [1] * cut, 0)]), run([(0, [1] * (N - cut), cut)])))
        assert torch.allclose(got, want[0], atol=1e-5), cut
    cv.reset(1), cv.reset(2)
    got = run([(1, [1] * 5, 0), (0, [1] * 2, 0)])
    assert torch.allclose(got, torch.cat((want[1][:5], want[0][:2])), atol=1e-5)
    state = cv.tail.clone()
    run([(0, [1] * 6, 2), (1, [1] * 3, 5)], commit=False)
    assert torch.equal(cv.tail, state)
    cv.commit([[0, 1, 2], []])
    got = run([(1, [1] * 2, 5), (0, [1] * 9, 5)])
    assert torch.allclose(got, torch.cat((want[1][5:7], want[0][5:])), atol=1e-5)


def test_routing_and_activation():
    g = torch.Generator().manual_seed(0)
    R, n = 40, 24
    c = MoeConfig(n_experts=6, top_k=3, ffn=16, n_shared=0, router="topk_softmax", swiglu_limit=0.7, glu_alpha=1.702, glu_shift=1.0)
    assert not c.plain and MoeConfig().plain
    h = torch.randn(R, n, generator=g)
    w = {"gate": torch.randn(6, n, generator=g) * 30, "bias": 20 * torch.randn(6, generator=g), "w_gu": torch.randn(6, 32, n, generator=g) * 0.4,
         "w_down": torch.randn(6, n, 16, generator=g) * 0.2}
    flat = {"router": w["gate"], "router.b": w["bias"]}
    for e in range(6):
        flat[f"e{e}.gate"], flat[f"e{e}.up"], flat[f"e{e}.down"] = w["w_gu"][e, :16], w["w_gu"][e, 16:], w["w_down"][e]
    wts, ids, _ = ops.route(h, w, c)
    rw, ri = oracle.routed(h, flat, "", 3)
    assert torch.equal(ids, ri) and torch.allclose(wts, rw, atol=1e-6) and torch.allclose(wts.sum(-1), torch.ones(R))
    want = oracle.experts(h, flat, "", {"router": {"experts": 6, "top": 3}, "expert": {"limit": 0.7}})
    assert torch.allclose(ops.moe(h, w, c), want, atol=1e-5)
    for k, v in (("glu_alpha", 1.0), ("glu_shift", 0.0), ("swiglu_limit", 0.0)):
        assert not torch.allclose(ops.moe(h, w, dataclasses.replace(c, **{k: v})), want, atol=1e-2), k


@pytest.mark.parametrize("sizes", [[2] * 60, [3, 61, 2, 54], [64, 56], [69, 2, 49], [119, 1], [1, 1, 1, 117]])
def test_portions(sizes):
    cfg, T = _setup(U.MIXED)
    toks = U.prompt(sum(sizes), cfg["vocab"], 4)
    m, out, i = U.framework(cfg, T), [], 0
    for n in sizes:
        out.append(m.forward(make_plan([(1, toks[i: i + n], i)])))
        i += n
    assert U.error(torch.cat(out), U.oracle_logits(cfg, T, toks)) < 2e-5


MIX_STEPS = [("a20", "b1", "c2"), ("a1", "b40", "d33"), ("a50", "c3", "d1"), ("b25", "d30", "/c", "/b"), ("a2", "e64", "f2"),
             ("/f", "/d", "a57", "e1"), ("e62",)]


def test_mixed_batch_with_reused_pages_and_slots():
    """Four live requests of unequal length in one pool that is exactly as large as they need: portions beside single tokens,
    requests that pause, pages and slots (with the convolutions' states) that are given back and taken by others."""
    cfg, T = _setup(U.MIXED)
    lens = {"a": 130, "b": 66, "c": 5, "d": 64, "e": 127, "f": 2}
    toks = {k: U.prompt(n, cfg["vocab"], ord(k)) for k, n in lens.items()}
    want = {k: U.oracle_logits(cfg, T, t) for k, t in toks.items()}
    mc = U.Z.read_config(cfg)
    ses = BatchSession(mc, U.Z.from_tensors(mc, T), EngineConfig(), "cpu", max_seqs=4, kv_tokens=192 + 128 + 64 + 64)
    at, pages = dict.fromkeys(lens, 0), {}
    for st in MIX_STEPS:
        ent = [(x[0], toks[x[0]][at[x[0]]: at[x[0]] + int(x[1:])], list(range(int(x[1:])))) for x in st if x[0] != "/"]
        got, r = ses.step(ent), 0
        for k, t, _ in ent:
            assert U.error(got[r: r + len(t)], want[k][at[k]: at[k] + len(t)]) < 2e-5, (k, at[k])
            r += len(t)
            at[k] += len(t)
            pages.setdefault(k, set()).update(ses.kv.pool.get(ses.kv.lease[ses.slots[k]]).pages)
        for x in st:
            if x[0] == "/":
                ses.end(x[1:])
    assert at["a"] == 130 and at["e"] == 127 and pages["e"] & (pages["b"] | pages["c"])


FAR = [0, 1, 2, 3, 62, 63, 64, 65, 127, 128, 191, 192, 205, 206, 207, 208]


def far_case(at):
    """Tokens whose last one asks for the planted token at `at`; (cfg, tensors, tokens, the same without the planted token)."""
    cfg, T = _setup(dict(layers=[U.latent(heads=2, dim=24, vdim=40)], groups=2), 7)
    for k, f in (("embed", 4), ("l0.mix.uv", 4), ("l0.canon1", 0.25)):
        T[k] = (T[k].float() * f).to(torch.bfloat16)
    return (cfg, T, *U.planted(cfg, T, 210, at))


@pytest.mark.parametrize("at", FAR)
def test_far_keys(at):
    cfg, T, toks, without = far_case(at)
    want = U.oracle_logits(cfg, T, toks)
    assert U.error(U.oracle_logits(cfg, T, without)[-1:], want[-1:]) > 0.05
    m = U.framework(cfg, T)
    assert U.error(m.forward(make_plan([(0, toks, 0)])), want) < 2e-5
    m.forward(make_plan([(1, toks[:-3], 0)]))
    for i in range(207, 210):
        assert U.error(m.forward(make_plan([(1, toks[i: i + 1], i)])), want[i: i + 1]) < 2e-5


def test_checkpoint_reader(tmp_path):
    cfg, T = _setup(U.MIXED)
    U.write_checkpoint(tmp_path / "ck", cfg, T)
    mc = load_config(str(tmp_path / "ck"))
    assert mc.family == "zakusun" and mc.norm_groups == 3 and mc.input_conv == 4 and mc.layer_specs[1].moe is None
    mc, W = load_checkpoint(str(tmp_path / "ck"))
    assert ModelConfig.from_dict(json.loads(mc.to_json())) == mc
    toks = U.prompt(20, cfg["vocab"])
    want = Model(mc, W, n_slots=1, kv_tokens=64).forward(make_plan([(0, toks, 0)]))
    assert U.error(want, U.oracle_logits(cfg, T, toks)) < 2e-5
    save_checkpoint(W, mc, str(tmp_path / "own"))                # the framework's own checkpoint format carries the same weights
    mc2, W2 = load_checkpoint(str(tmp_path / "own"))
    assert mc2 == mc and torch.equal(Model(mc2, W2, n_slots=1, kv_tokens=64).forward(make_plan([(0, toks, 0)])), want)
    with pytest.raises(ValueError, match="l0.mlp.e3.up"):
        U.Z.from_tensors(mc, {k: t for k, t in T.items() if k != "l0.mlp.e3.up"})
    for k in ("l1.dwa", "l0.canon2", "l2.mix.sink"):
        with pytest.raises(ValueError, match="shape"):
            U.Z.from_tensors(mc, dict(T, **{k: T[k][1:]}))
    for bad in (dict(type="other"), dict(mlp={"kind": "other"}), dict(mlp=U.moe(experts=2, top=3))):
        with pytest.raises(ValueError):
            U.Z.read_config(dict(cfg, layers=[dict(cfg["layers"][0], **bad)]))
    with pytest.raises(ValueError):
        U.Z.read_config(U.config([U.latent()], groups=5))


def test_greedy_generation_long_and_batched():
    cfg, T = _setup(U.MIXED)
    mc = U.Z.read_config(cfg)
    eng = LLMEngine(mc, U.Z.from_tensors(mc, T), device="cpu", max_seqs=3, kv_tokens_per_seq=256)
    prompts = [U.prompt(n, cfg["vocab"], n) for n in (1, 60, 33)]
    for p, o in zip(prompts, eng.generate(prompts, max_new=110)):
        want = U.oracle_logits(cfg, T, p + o)[len(p) - 1: -1]
        assert o == want.argmax(-1).tolist()


@pytest.mark.parametrize("drafts", [False, True])
def test_scheduler_generates_the_oracles_text(drafts):
    """Requests through admission, shared prompt chunks, batched rounds (with drafts that are verified and committed), a
    continued conversation, more requests than slots."""
    cfg, T = _setup(U.MIXED)
    mc = U.Z.read_config(cfg)
    es = EngineServer(mc, U.Z.from_tensors(mc, T), EngineConfig(max_seqs=2, kv_tokens=1024, prefill_chunk=24, spec="lookup" if drafts else "none",
                                                               spec_depth=3))
    prompts = {i: U.prompt(n, cfg["vocab"], n) for i, n in enumerate((41, 7, 90, 3))}
    texts = {i: U.oracle_greedy(cfg, T, p, 12) for i, p in prompts.items()}
    if drafts:                                   # two right tokens, then a wrong one: accepted and rejected rows in every round
        def draft(seq, depth):
            i = es.by_slot[seq.slot].id
            n = len(seq.generated)
            d = (texts[i][n: n + 2] + [0])[:depth] if i in texts else []
            return d, [0.9] * len(d)
        es.spec.drafter = draft
    done = _serve(es, [{"id": i, "prompt_ids": p, "max_new": 12} for i, p in prompts.items()])
    for i, p in prompts.items():
        assert done[i]["token_ids"] == texts[i], i
    p = prompts[3] + done[3]["token_ids"] + [1, 2]
    again = _serve(es, [{"id": 9, "prompt_ids": p, "max_new": 6}, {"id": 10, "prompt_ids": p, "max_new": 6, "temperature": 0.8, "seed": 3}])
    assert again[9]["token_ids"] == U.oracle_greedy(cfg, T, p, 6) and again[9]["prefix_hit_tokens"] > 0
    assert len(again[10]["token_ids"]) == 6
    if drafts:
        assert 0 < es.totals["accepted_drafts"] < es.totals["drafted_tokens"]


def test_snapshot_moves_a_sequence_to_another_slot():
    cfg, T = _setup(U.MIXED)
    toks = U.prompt(80, cfg["vocab"], 2)
    m = U.framework(cfg, T, slots=3, tokens=128)
    kv = KvManager(m)
    assert kv.assign(0, 100) and kv.assign(2, 100)
    m.forward(make_plan([(0, toks[:70], 0)]))
    m.restore(2, m.snapshot(0))
    assert U.error(m.forward(make_plan([(2, toks[70:], 70)])), U.oracle_logits(cfg, T, toks)[70:]) < 2e-5


def test_preset():
    mc = get_model_config("zakusun-style", n_layers=3, hidden=256, ffn=64, vocab=100, experts=4, top=2)
    assert mc.layer_specs[2].moe.n_routes == 4 and mc.layer_specs[0].mixer.sink
    W = U.Z.random_weights(mc, dtype=torch.float32)
    assert torch.isfinite(Model(mc, W, n_slots=1, kv_tokens=64).forward(make_plan([(0, [1, 2, 3], 0)]))).all()
