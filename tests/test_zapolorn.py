"""Zapolorn on the CPU: every mechanism against the plain implementation, the checkpoint reader, the paged cache and the recurrent
state, portions and batches, prefix snapshots, speculation, and greedy generation through the engine and the server's
scheduler."""
import dataclasses
import json
import math

import pytest
import torch
import zapolorn_oracle as oracle
import zapolorn_util as U
from test_vabunex import _serve

from spark_engine_b200 import ops
from spark_engine_b200.cache.kv import KvManager
from spark_engine_b200.config import EngineConfig, ModelConfig, MoeConfig, get_model_config
from spark_engine_b200.models.checkpoint import load_checkpoint, load_config, save_checkpoint
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
    x = torch.tensor([[[3.0, 4.0, 0.0, 0.0]]] * 3, dtype=torch.float64)
    y = oracle.rotate_pairs(x, {"base": 100.0, "dims": 2, "scaling": {"factor": 2.0}})
    assert torch.allclose(y[2, 0], torch.tensor([3 * math.cos(1) - 4 * math.sin(1), 4 * math.cos(1) + 3 * math.sin(1), 0, 0], dtype=torch.float64))
    assert [oracle.temperature(p, {"coef": 1.0, "every": 4}) for p in (0, 2)] == [1.0, 1.0]
    assert oracle.temperature(3, {"coef": 1.0, "every": 4}) == oracle.temperature(6, {"coef": 1.0, "every": 4}) == 1 + math.log(2)
    assert [oracle.slope(h, 4) for h in range(4)] == [2.0 ** -2, 2.0 ** -4, 2.0 ** -6, 2.0 ** -8]
    assert [j for j in range(9) if oracle.visible(6, j, 3)] == [4, 5, 6]
    s, sink = torch.tensor([[1.0, 2.0]]), torch.tensor([3.0])
    assert torch.allclose(oracle.softmax_with(sink, s), torch.exp(s) / (torch.exp(s).sum() + math.exp(3.0)))
    q, k, v = (torch.tensor([[[a]], [[b]]]) for a, b in ((1.0, 2.0), (3.0, 4.0), (5.0, 6.0)))
    assert torch.allclose(oracle.decayed_sums(q, k, v, torch.full((2, 1, 1), 0.5)), torch.tensor([[[15.0]], [[2 * (7.5 + 24)]]]))


def test_the_sink_shows():
    """A sink far above the scores takes nearly all of the weight; leaving it out would show."""
    cfg, T = _setup("window attention")
    T["l0.mix.sink"] += 5
    m, toks = U.framework(cfg, T), U.prompt(30, cfg["vocab"])
    want = U.oracle_logits(cfg, T, toks)
    assert U.error(m.forward(make_plan([(0, toks, 0)])), want) < 2e-5
    # the output's norm hides the size of what is left, so compare a head whose sink is gone beside heads that keep theirs
    m.W["layers"][0]["mix"]["sink"][0] = float("-inf")
    assert U.error(m.forward(make_plan([(1, toks, 0)])), want) > 0.05


def test_routing():
    """Scores are the weights as they are, and they scale the experts' inputs."""
    g = torch.Generator().manual_seed(0)
    R, n = 40, 24
    c = MoeConfig(n_experts=6, top_k=3, ffn=16, n_shared=0, router="sigmoid", weight_input=True)
    h = torch.randn(R, n, generator=g)
    w = {"gate": torch.randn(6, n, generator=g) * 0.3, "w_gu": torch.randn(6, 32, n, generator=g) * 0.2, "w_down": torch.randn(6, n, 16, generator=g) * 0.2}
    flat = {"router": w["gate"]}
    for e in range(6):
        flat[f"e{e}.gate"], flat[f"e{e}.up"], flat[f"e{e}.down"] = w["w_gu"][e, :16], w["w_gu"][e, 16:], w["w_down"][e]
    wts, ids, _ = ops.route(h, w, c)
    rw, ri = oracle.routed(h, flat, "", 3)
    assert torch.equal(ids, ri) and torch.allclose(wts, rw, atol=1e-6) and (wts.sum(-1) - 1).abs().max() > 0.1
    want = oracle.experts(h, flat, "", {"router": {"top": 3}})
    assert torch.allclose(ops.moe(h, w, c), want, atol=1e-5)
    assert not torch.allclose(ops.moe(h, w, dataclasses.replace(c, weight_input=False)), want, atol=1e-2)


@pytest.mark.parametrize("sizes", [[2] * 60, [3, 61, 2, 54], [64, 56], [69, 2, 49], [119, 1]])
def test_portions(sizes):
    cfg, T = _setup(U.MIXED)
    toks = U.prompt(sum(sizes), cfg["vocab"], 4)
    m, out, i = U.framework(cfg, T), [], 0
    for n in sizes:
        out.append(m.forward(make_plan([(1, toks[i: i + n], i)])))
        i += n
    assert U.error(torch.cat(out), U.oracle_logits(cfg, T, toks)) < 2e-5


def test_mixed_batch_with_reused_pages_and_slots():
    """Four live requests of unequal length in one pool that is exactly as large as they need: portions beside single tokens,
    requests that pause, pages and slots (with their recurrent states) that are given back and taken by others."""
    cfg, T = _setup(U.MIXED)
    lens = {"a": 130, "b": 66, "c": 5, "d": 64, "e": 127, "f": 2}
    toks = {k: U.prompt(n, cfg["vocab"], ord(k)) for k, n in lens.items()}
    want = {k: U.oracle_logits(cfg, T, t) for k, t in toks.items()}
    mc = U.Z.read_config(cfg)
    ses = BatchSession(mc, U.Z.from_tensors(mc, T), EngineConfig(), "cpu", max_seqs=4, kv_tokens=192 + 128 + 64 + 64)
    at, pages = dict.fromkeys(lens, 0), {}
    for st in [("a20", "b1", "c2"), ("a1", "b40", "d33"), ("a50", "c3", "d1"), ("b25", "d30", "/c", "/b"), ("a2", "e64", "f2"),
               ("/f", "/d", "a57", "e1"), ("e62",)]:
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


# (window, place of the planted key) for a query at position 209: windows that begin inside a page, at a page, at the first token
FAR = [(70, 139), (70, 140), (70, 141), (70, 191), (70, 192), (17, 192), (18, 192), (18, 191), (82, 127), (82, 128), (1, 209), (1, 208), (209, 0),
       (210, 0), (1000, 0), (1000, 63), (1000, 64)]


def far_case(size, at, kv_from=False):
    """Tokens whose last one asks for the planted token at `at`; (cfg, tensors, tokens, the same without the planted token)."""
    layers = [U.window(size=size, rot=2, base=1e12, factor=1e6)]             # (angles of next to nothing)
    if kv_from:
        layers.append(U.window(size=size, kv_from=0, rot=2, base=1e12, factor=1e6))
    cfg, T = _setup(dict(layers=layers), 7)
    qt, kt, fill = U.planted_pair(cfg, T)
    toks = [fill[i % len(fill)] for i in range(209)] + [qt]
    other = list(toks)
    other[at] = kt
    return cfg, T, other, toks


@pytest.mark.parametrize("size,at", FAR)
def test_a_key_is_seen_inside_the_window_only(size, at):
    cfg, T, toks, without = far_case(size, at)
    want = U.oracle_logits(cfg, T, toks)
    moved = U.error(U.oracle_logits(cfg, T, without)[-1:], want[-1:])
    assert moved > 0.05 if 209 - at < size else moved < 1e-6        # leaving the key out / letting it in would show
    m = U.framework(cfg, T)
    assert U.error(m.forward(make_plan([(0, toks, 0)])), want) < 2e-5
    m.forward(make_plan([(1, toks[:-3], 0)]))
    for i in range(207, 210):
        assert U.error(m.forward(make_plan([(1, toks[i: i + 1], i)])), want[i: i + 1]) < 2e-5


def slope_case(at):
    """As far_case for whole-context attention: the planted key stands out for the head with the gentlest slope."""
    cfg, T = _setup(dict(layers=[U.pair(heads=4, kv_heads=2, coef=0.2, every=64, right=0.3)]), 7)
    qt, kt, fill = U.planted_pair(cfg, T)
    toks = [fill[i % len(fill)] for i in range(209)] + [qt]
    other = list(toks)
    other[at] = kt
    return cfg, T, other, toks


SLOPED = [0, 1, 63, 64, 127, 128, 192, 207, 208]


@pytest.mark.parametrize("at", SLOPED)
def test_far_keys_under_a_slope(at):
    cfg, T, toks, without = slope_case(at)
    want = U.oracle_logits(cfg, T, toks)
    assert U.error(U.oracle_logits(cfg, T, without)[-1:], want[-1:]) > 0.05
    m = U.framework(cfg, T)
    assert U.error(m.forward(make_plan([(0, toks, 0)])), want) < 2e-5
    m.forward(make_plan([(1, toks[:-3], 0)]))
    for i in range(207, 210):
        assert U.error(m.forward(make_plan([(1, toks[i: i + 1], i)])), want[i: i + 1]) < 2e-5


def test_a_borrowed_cache_is_the_other_layers():
    """A layer without keys of its own reads the ones the other layer cached, and has no cache of its own."""
    cfg, T = _setup("keys of another layer")
    m = U.framework(cfg, T)
    mix = [x for _, x, _ in m.layers]
    assert mix[1].k is mix[0].k and mix[3].v is mix[0].v and mix[2].k is not mix[0].k
    assert not mix[1].state_tensors() and set(mix[0].state_tensors()) == {"k", "v"}
    assert "k" not in {k.split(".")[-1] for k in T if k.startswith("l1.")}
    toks = U.prompt(30, cfg["vocab"])
    want = U.oracle_logits(cfg, T, toks)
    T["l0.mix.k"] = -T["l0.mix.k"]
    assert U.error(U.framework(cfg, T).forward(make_plan([(0, toks, 0)])), want) > 0.05


def test_checkpoint_reader(tmp_path):
    cfg, T = _setup(U.MIXED)
    U.write_checkpoint(tmp_path / "ck", cfg, T)
    mc = load_config(str(tmp_path / "ck"))
    assert mc.family == "zapolorn" and mc.block == "post" and mc.layer_specs[1].moe.weight_input and mc.layer_specs[3].moe is None
    mc, W = load_checkpoint(str(tmp_path / "ck"))
    assert ModelConfig.from_dict(json.loads(mc.to_json())) == mc
    toks = U.prompt(20, cfg["vocab"])
    want = Model(mc, W, n_slots=1, kv_tokens=64).forward(make_plan([(0, toks, 0)]))
    assert U.error(want, U.oracle_logits(cfg, T, toks)) < 2e-5
    save_checkpoint(W, mc, str(tmp_path / "own"))                # the framework's own checkpoint format carries the same weights
    mc2, W2 = load_checkpoint(str(tmp_path / "own"))
    assert mc2 == mc and torch.equal(Model(mc2, W2, n_slots=1, kv_tokens=64).forward(make_plan([(0, toks, 0)])), want)
    with pytest.raises(ValueError, match="l1.mlp.e3.up"):
        U.Z.from_tensors(mc, {k: t for k, t in T.items() if k != "l1.mlp.e3.up"})
    with pytest.raises(ValueError, match="shape"):
        U.Z.from_tensors(mc, dict(T, **{"l0.mix.k.norm": T["l0.mix.k.norm"][1:]}))
    for bad in (dict(type="other"), dict(mlp={"kind": "other"})):
        with pytest.raises(ValueError):
            U.Z.read_config(dict(cfg, layers=[dict(cfg["layers"][0], **bad)]))
    for bad in ([U.window(heads=5, kv_heads=2)], [U.window(rot=5)], [U.window(kv_from=0)], [U.pair(), U.window(kv_from=0)],
                [U.window(), U.window(kv_from=0, dim=24)], [U.window(), U.window(kv_from=0), U.window(kv_from=1)]):
        with pytest.raises(ValueError):
            U.Z.read_config(U.config(bad))


def test_optional_parts_of_the_configuration():
    """Without a scaling nothing is slowed, without a rotation nothing turns, without a window everything is seen."""
    cfg, T = _setup("window attention")
    m = cfg["layers"][0]["mixer"]
    for drop in ("scaling", "rot", "mask"):
        (m["rot"] if drop == "scaling" else m).pop(drop)
        toks = U.prompt(90, cfg["vocab"])
        assert U.error(U.framework(cfg, T).forward(make_plan([(0, toks, 0)])), U.oracle_logits(cfg, T, toks)) < 2e-5


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
    mc = get_model_config("zapolorn-style", n_layers=4, hidden=256, ffn=64, vocab=100, experts=4, top=2)
    assert mc.layer_specs[0].ffn == 64 and mc.layer_specs[1].moe.n_routes == 4 and mc.layer_specs[2].mixer.kv_from == 1
    W = U.Z.random_weights(mc, dtype=torch.float32)
    assert torch.isfinite(Model(mc, W, n_slots=1, kv_tokens=64).forward(make_plan([(0, [1, 2, 3], 0)]))).all()
