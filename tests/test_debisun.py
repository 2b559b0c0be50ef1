"""Debisun on the CPU: every mechanism against the plain implementation, the checkpoint reader, the paged cache and the
convolution state, portions and batches, prefix snapshots, speculation, and greedy generation through the engine and the
server's scheduler."""
import json

import debisun_oracle as oracle
import debisun_util as U
import pytest
import torch
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
    m.tap_layers = set(range(4))
    m.forward(make_plan([(1, toks, 0)]))
    for i, x in enumerate(taps):
        assert torch.allclose(m.taps[i].double(), x, atol=2e-4), i


def test_distance_buckets():
    for rows, far in ((2, 3), (10, 90), (16, 128), (32, 1000), (8, 5)):
        got = U.D.distance_buckets(3 * far, rows, far)
        assert got.tolist() == [oracle.distance_bucket(n, rows, far) for n in range(3 * far)]
        assert int(got[far]) == rows - 1 and got[: rows // 2].tolist() == list(range(rows // 2)) and (got.diff() >= 0).all()


def test_the_sink_shows():
    """Scores far below the sink's: the weights sum to little, and leaving the sink out would show."""
    s = torch.tensor([[-4.0, -5.0, float("-inf")]], dtype=torch.float64)
    w = oracle.weights_with_silent_sink(s)
    assert torch.allclose(w, torch.exp(s) / (1 + torch.exp(s).sum()))
    cfg, T = _setup("attention")
    T["l0.mix.rel"] -= 4
    m, toks = U.framework(cfg, T), U.prompt(30, cfg["vocab"])
    want = U.oracle_logits(cfg, T, toks)
    assert U.error(m.forward(make_plan([(0, toks, 0)])), want) < 2e-5
    m.W["layers"][0]["mix"]["sink"].fill_(float("-inf"))
    assert U.error(m.forward(make_plan([(1, toks, 0)])), want) > 0.05


def test_routing():
    """The correction moves the choice and not the weights; identity experts return their input."""
    g = torch.Generator().manual_seed(0)
    R, n = 40, 24
    c = MoeConfig(n_experts=4, n_identity=3, top_k=3, ffn=16, n_shared=0, router="softmax_bias", route_scale=2.5, act="relu2")
    h, bias = torch.randn(R, n, generator=g), torch.tensor([0.0, -5.0, 0.3, 0.0, 0.2, 0.0, -0.1])
    w = {"gate": torch.randn(7, n, generator=g) * 0.3, "bias": bias, "w_up": torch.randn(4, 16, n, generator=g) * 0.2,
         "w_down": torch.randn(4, n, 16, generator=g) * 0.2}
    flat = {"router": w["gate"], "correction": bias}
    for e in range(4):
        flat[f"e{e}.up"], flat[f"e{e}.down"] = w["w_up"][e], w["w_down"][e]
    r = {"experts": 4, "identity": 3, "top": 3, "scale": 2.5}
    wts, ids, _ = ops.route(h, w, c)
    rw, ri = oracle.routed(h, flat, "", r)
    assert torch.equal(ids, ri) and torch.allclose(wts, rw, atol=1e-5) and not (ids == 1).any() and (ids >= 4).any()
    assert torch.allclose(wts.sum(-1), torch.full((R,), 2.5), atol=1e-4)
    assert torch.allclose(ops.moe(h, w, c), oracle.experts(h, flat, "", {"router": r}), atol=1e-4)


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
    requests that pause, pages and slots (with their convolution tails) that are given back and taken by others."""
    cfg, T = _setup(U.MIXED)
    lens = {"a": 130, "b": 66, "c": 5, "d": 64, "e": 127, "f": 2}
    toks = {k: U.prompt(n, cfg["vocab"], ord(k)) for k, n in lens.items()}
    want = {k: U.oracle_logits(cfg, T, t) for k, t in toks.items()}
    mc = U.D.read_config(cfg)
    ses = BatchSession(mc, U.D.from_tensors(mc, T), EngineConfig(), "cpu", max_seqs=4, kv_tokens=192 + 128 + 64 + 64)
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


# the planted key of a query at position 209: its chunk of 70 starts at 140; of 192 at 192; of 1000 at 0 (page borders, first tokens)
FAR = [(70, 139), (70, 140), (70, 141), (70, 191), (70, 192), (192, 191), (192, 192), (1000, 0), (1000, 1), (1000, 63), (1000, 64), (1000, 127),
       (1000, 128)]


@pytest.mark.parametrize("chunk,at", FAR)
def test_a_key_is_seen_inside_its_chunk_only(chunk, at):
    cfg, T = _setup(dict(layers=[U.layer(chunk=chunk)]), 7)
    qt, kt, fill = U.planted_pair(cfg, T)
    toks = [fill[i % len(fill)] for i in range(209)] + [qt]
    plain = U.oracle_logits(cfg, T, toks)
    toks[at] = kt
    want = U.oracle_logits(cfg, T, toks)
    moved = U.error(plain[-1:], want[-1:])
    assert moved > 0.05 if 209 // chunk == at // chunk else moved < 1e-6        # leaving the key out / letting it in would show
    m = U.framework(cfg, T)
    assert U.error(m.forward(make_plan([(0, toks, 0)])), want) < 2e-5
    m.forward(make_plan([(1, toks[:-3], 0)]))
    for i in range(207, 210):
        assert U.error(m.forward(make_plan([(1, toks[i: i + 1], i)])), want[i: i + 1]) < 2e-5


def test_checkpoint_reader(tmp_path):
    cfg, T = _setup(U.MIXED)
    U.write_checkpoint(tmp_path / "ck", cfg, T)
    mc = load_config(str(tmp_path / "ck"))
    assert mc.family == "debisun" and mc.block == "sequential" and mc.layer_specs[1].moe.n_identity == 2 and mc.layer_specs[2].moe is None
    mc, W = load_checkpoint(str(tmp_path / "ck"))
    assert ModelConfig.from_dict(json.loads(mc.to_json())) == mc
    toks = U.prompt(20, cfg["vocab"])
    want = Model(mc, W, n_slots=1, kv_tokens=64).forward(make_plan([(0, toks, 0)]))
    assert U.error(want, U.oracle_logits(cfg, T, toks)) < 2e-5
    save_checkpoint(W, mc, str(tmp_path / "own"))                # the framework's own checkpoint format carries the same weights
    mc2, W2 = load_checkpoint(str(tmp_path / "own"))
    assert mc2 == mc and torch.equal(Model(mc2, W2, n_slots=1, kv_tokens=64).forward(make_plan([(0, toks, 0)])), want)
    with pytest.raises(ValueError, match="l1.mlp.e3.up"):
        U.D.from_tensors(mc, {k: t for k, t in T.items() if k != "l1.mlp.e3.up"})
    with pytest.raises(ValueError, match="shape"):
        U.D.from_tensors(mc, dict(T, **{"l0.mix.k.conv": T["l0.mix.k.conv"][:, 1:]}))
    for bad in (dict(type="other"), dict(mlp={"kind": "other"})):
        with pytest.raises(ValueError):
            U.D.read_config(dict(cfg, layers=[dict(cfg["layers"][0], **bad)]))
    with pytest.raises(ValueError):
        U.D.read_config(U.config([U.layer(heads=5, kv_heads=2)]))


def test_greedy_generation_long_and_batched():
    cfg, T = _setup(U.MIXED)
    mc = U.D.read_config(cfg)
    eng = LLMEngine(mc, U.D.from_tensors(mc, T), device="cpu", max_seqs=3, kv_tokens_per_seq=256)
    prompts = [U.prompt(n, cfg["vocab"], n) for n in (1, 60, 33)]
    for p, o in zip(prompts, eng.generate(prompts, max_new=110)):
        want = U.oracle_logits(cfg, T, p + o)[len(p) - 1: -1]
        assert o == want.argmax(-1).tolist()


@pytest.mark.parametrize("drafts", [False, True])
def test_scheduler_generates_the_oracles_text(drafts):
    """Requests through admission, shared prompt chunks, batched rounds (with drafts that are verified and committed), a
    continued conversation, more requests than slots."""
    cfg, T = _setup(U.MIXED)
    mc = U.D.read_config(cfg)
    es = EngineServer(mc, U.D.from_tensors(mc, T), EngineConfig(max_seqs=2, kv_tokens=1024, prefill_chunk=24, spec="lookup" if drafts else "none",
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
    mc = get_model_config("debisun-style", n_layers=3, hidden=256, ffn=64, vocab=100, experts=4, top=2)
    assert mc.layer_specs[0].ffn == 64 and mc.layer_specs[2].moe.n_routes == 5
    W = U.D.random_weights(mc, dtype=torch.float32)
    assert torch.isfinite(Model(mc, W, n_slots=1, kv_tokens=64).forward(make_plan([(0, [1, 2, 3], 0)]))).all()
