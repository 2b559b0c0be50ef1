"""Vabunex on the CPU: every mechanism against the plain implementation, the checkpoint reader, the paged cache, portions
and batches, prefix snapshots, speculation, and greedy generation through the engine and the server's scheduler."""
import dataclasses
import json

import pytest
import torch
import vabunex_oracle as oracle
import vabunex_util as U

from spark_engine_b200.cache.kv import KvManager
from spark_engine_b200.config import EngineConfig, ModelConfig
from spark_engine_b200.models.checkpoint import load_checkpoint, load_config, save_checkpoint
from spark_engine_b200.models.plan import make_plan
from spark_engine_b200.runtime import rt
from spark_engine_b200.serving.engine import LLMEngine
from spark_engine_b200.serving.session import BatchSession
from spark_engine_b200.serving.worker import EngineServer

MIXED = dict(layers=[U.wkv(), U.lightning(ff=0), U.latent(), U.wkv(heads=2, dim=16, ff=0), U.latent(heads=2, rot_dim=8, ff=0)],
             loop=(1, 4, 2))
MECHANISMS = {
    "lightning": dict(layers=[U.lightning()]),
    "lightning no decay / full decay": dict(layers=[U.lightning(heads=2, decay=[1.0, 0.0])]),
    "wkv": dict(layers=[U.wkv()]),
    "latent": dict(layers=[U.latent()]),
    "latent equal sizes": dict(layers=[U.latent(heads=1, dim=16, vdim=16, rot_dim=16, q_rank=16, kv_rank=16, scale=1.0)]),
    "no feed-forward": dict(layers=[U.lightning(ff=0), U.wkv(ff=0), U.latent(ff=0)]),
    "odd width": dict(layers=[U.lightning(ff=37), U.wkv(ff=37), U.latent(ff=37, q_rank=21, kv_rank=19)], width=75),
    "loop": MIXED,
    "loop of everything": dict(layers=[U.wkv(), U.latent()], loop=(0, 2, 3)),
    "loop once": dict(layers=[U.wkv(), U.latent()], loop=(0, 1, 1)),
}


def _setup(name, seed=1):
    cfg = U.config(**(MECHANISMS[name] if isinstance(name, str) else name))
    return cfg, U.tensors(cfg, seed)


@pytest.mark.parametrize("name", list(MECHANISMS))
def test_whole_prompt_and_token_by_token(name):
    cfg, T = _setup(name)
    toks = U.prompt(70, cfg["vocab"])
    want = U.oracle_logits(cfg, T, toks)
    m = U.framework(cfg, T)
    assert U.error(m.forward(make_plan([(0, toks, 0)])), want) < 1e-5
    one = torch.cat([m.forward(make_plan([(2, [t], i)])) for i, t in enumerate(toks)])
    assert U.error(one, want) < 1e-5
    assert U.error(one[:3], want[:3]) < 1e-5


def test_residual_stream_after_every_run():
    cfg, T = _setup(MIXED)
    toks, taps = U.prompt(9, cfg["vocab"]), []
    U.oracle_logits(cfg, T, toks, taps)
    m = U.framework(cfg, T)
    assert len(m.layers) == len(taps) == 8
    m.tap_layers = set(range(8))
    m.forward(make_plan([(1, toks, 0)]))
    for i, x in enumerate(taps):
        assert torch.allclose(m.taps[i].double(), x, atol=1e-4), i


@pytest.mark.parametrize("sizes", [[2] * 60, [3, 61, 2, 54], [64, 56], [63, 2, 55], [119, 1]])
def test_portions(sizes):
    cfg, T = _setup(MIXED)
    toks = U.prompt(sum(sizes), cfg["vocab"], 4)
    m, out, i = U.framework(cfg, T), [], 0
    for n in sizes:
        out.append(m.forward(make_plan([(1, toks[i: i + n], i)])))
        i += n
    assert U.error(torch.cat(out), U.oracle_logits(cfg, T, toks)) < 1e-5


def test_mixed_batch_with_reused_pages_and_slots():
    """Four live requests of unequal length in one pool that is exactly as large as they need: portions beside single
    tokens, requests that pause, pages and slots that are given back and taken by others."""
    cfg, T = _setup(MIXED)
    lens = {"a": 130, "b": 66, "c": 5, "d": 64, "e": 127, "f": 2}
    toks = {k: U.prompt(n, cfg["vocab"], ord(k)) for k, n in lens.items()}
    want = {k: U.oracle_logits(cfg, T, t) for k, t in toks.items()}
    mc = U.V.read_config(cfg)
    ses = BatchSession(mc, U.V.from_tensors(mc, T), EngineConfig(), "cpu", max_seqs=4, kv_tokens=192 + 128 + 64 + 64)
    steps = [("a20", "b1", "c2"), ("a1", "b40", "d33"), ("a50", "c3", "d1"), ("b25", "d30", "/c", "/b"), ("a2", "e64", "f2"),
             ("/f", "/d", "a57", "e1"), ("e62",)]
    at, pages = dict.fromkeys(lens, 0), {}
    for st in steps:
        ent = []
        for x in st:
            if x[0] != "/":
                n = int(x[1:])
                ent.append((x[0], toks[x[0]][at[x[0]]: at[x[0]] + n], list(range(n))))
        got, r = ses.step(ent), 0
        for k, t, _ in ent:
            assert U.error(got[r: r + len(t)], want[k][at[k]: at[k] + len(t)]) < 1e-5, (k, at[k])
            r += len(t)
            at[k] += len(t)
            pages.setdefault(k, set()).update(ses.kv.pool.get(ses.kv.lease[ses.slots[k]]).pages)
        for x in st:
            if x[0] == "/":
                ses.end(x[1:])
    assert at["a"] == 130 and at["e"] == 127 and pages["e"] & (pages["b"] | pages["c"])
    with pytest.raises(RuntimeError):
        ses.step([("g", toks["a"] * 2, [])])
    with pytest.raises(ValueError):
        ses.step([("h", [cfg["vocab"]], [])])


def planted_pair(cfg, T, boost=None):
    """(query token, key token, filler tokens): in a one-layer latent model the key token's score stands out for the query
    token (rotated parts silenced), the fillers score far below."""
    c = cfg["layers"][0]["mixer"]
    H, D, R, L = c["heads"], c["dim"], c["rot_dim"], c["kv_rank"]
    T["l0.mix.uq"].view(H, D + R, -1)[:, D:] = 0
    W = U.oracle_weights(T)
    x = W["embed"] * cfg["embedding"]["scale"]
    h = oracle.norm_zero_centred(x, W["l0.norm1"], cfg["norm"]["eps"])
    q = (oracle.unit_rms(h @ W["l0.mix.dq"].T, 1e-5) * W["l0.mix.dq.norm"]) @ W["l0.mix.uq"].T
    k = (oracle.unit_rms((h @ W["l0.mix.dkv"].T)[:, :L], 1e-5) * W["l0.mix.dkv.norm"]) @ W["l0.mix.uk"].T
    sc = torch.einsum("ahd,bhd->hab", q.view(-1, H, D + R)[..., :D], k.view(-1, H, D))[0]
    qt, kt = divmod(int(sc.argmax()), sc.shape[1])
    c["scale"] = float(25.0 / sc[qt, kt])
    return qt, kt, [int(t) for t in torch.argsort(sc[qt])[: cfg["vocab"] // 2] if int(t) not in (qt, kt)]


FAR = [0, 1, 62, 63, 64, 65, 127, 128, 190, 191]


@pytest.mark.parametrize("at", FAR)
def test_a_far_key_is_found(at):
    cfg, T = _setup(dict(layers=[U.latent()]), 7)
    qt, kt, fill = planted_pair(cfg, T)
    toks = [fill[i % len(fill)] for i in range(192)] + [qt, fill[0], qt]
    plain = U.oracle_logits(cfg, T, toks)
    toks[at] = kt
    want = U.oracle_logits(cfg, T, toks)
    assert U.error(plain[-1:], want[-1:]) > 0.05            # leaving the key out would show
    m = U.framework(cfg, T)
    assert U.error(m.forward(make_plan([(0, toks, 0)])), want) < 1e-5
    m.forward(make_plan([(1, toks[:-3], 0)]))
    for i in range(192, 195):
        assert U.error(m.forward(make_plan([(1, toks[i: i + 1], i)])), want[i: i + 1]) < 1e-5


def test_rotation_depends_on_distance_and_pairs():
    x = torch.randn(5, 2, 14, dtype=torch.float64)
    from spark_engine_b200.oracle import layers as L
    pos = torch.tensor([0, 1, 63, 64, 1000])
    got = L.rope_interleaved(x, pos, 10, 300.0)
    assert torch.allclose(got, oracle.rotate_interleaved(x, pos, 10, 300.0), atol=1e-4)
    assert torch.equal(got[..., 10:], x[..., 10:]) and torch.equal(got[0], x[0])


def test_a_single_update_survives_and_a_strong_decay_erases():
    """One large key at the start of a sequence: kept by decay 1, gone at decay 0, carried over portion borders."""
    from spark_engine_b200 import ops
    H, D, Vd, T = 2, 8, 12, 130
    g = torch.Generator().manual_seed(0)
    q, k, v = (torch.randn(T, H, n, generator=g) * 0.1 for n in (D, D, Vd))
    k[0] *= 100
    for decay in ([1.0, 0.0], [0.999, 0.5]):
        want = oracle.decay_scan(q.double(), k.double(), v.double(), torch.tensor(decay, dtype=torch.float64))
        S = torch.zeros(3, H, D, Vd)
        l2 = torch.tensor([-1000.0 if x == 0 else float(torch.log2(torch.tensor(x))) for x in decay])
        got = []
        for a, b in ((0, 64), (64, 65), (65, 130)):
            plan = make_plan([(1, [0] * (b - a), a)])
            f = lambda t: t[a:b].reshape(b - a, -1)
            got.append(ops.linear_state(f(q), f(k), f(v), H, D, Vd, S, plan, True, log2a=l2))
        assert torch.allclose(torch.cat(got).view(T, H, Vd).double(), want, atol=1e-4)


def test_checkpoint_reader(tmp_path):
    cfg, T = _setup(MIXED)
    U.write_checkpoint(tmp_path / "ck", cfg, T)
    mc = load_config(str(tmp_path / "ck"))
    assert mc.family == "vabunex" and mc.layer_runs() == [0, 1, 2, 3, 1, 2, 3, 4]
    mc, W = load_checkpoint(str(tmp_path / "ck"))
    assert ModelConfig.from_dict(json.loads(mc.to_json())) == mc
    toks = U.prompt(20, cfg["vocab"])
    from spark_engine_b200.models.model import Model
    want = Model(mc, W, n_slots=1, kv_tokens=64).forward(make_plan([(0, toks, 0)]))
    assert U.error(want, U.oracle_logits(cfg, T, toks)) < 1e-5
    # the framework's own checkpoint format carries the same weights
    save_checkpoint(W, mc, str(tmp_path / "own"))
    mc2, W2 = load_checkpoint(str(tmp_path / "own"))
    assert torch.equal(Model(mc2, W2, n_slots=1, kv_tokens=64).forward(make_plan([(0, toks, 0)])), want)
    missing = {k: t for k, t in T.items() if k != "l2.mix.uv"}
    with pytest.raises(ValueError, match="l2.mix.uv"):
        U.V.from_tensors(mc, missing)
    with pytest.raises(ValueError, match="shape"):
        U.V.from_tensors(mc, dict(T, **{"l0.mix.u": T["l0.mix.u"][:1]}))
    with pytest.raises(ValueError, match="architecture"):
        (tmp_path / "bad").mkdir()
        (tmp_path / "bad" / "config.json").write_text(json.dumps(dict(cfg, architecture="other")))
        load_config(str(tmp_path / "bad"))
    with pytest.raises(ValueError):
        U.V.read_config(dict(cfg, loop={"start": 2, "stop": 9, "times": 2}))


def test_page_pool():
    p = rt().PagePool(64 * 6, 64)
    a, b = p.acquire(65), p.acquire(1)
    assert p.free_tokens() == 64 * 3 and len(p.get(a).pages) == 2
    assert p.grow(a, 64 * 5) and p.free_tokens() == 0 and not p.grow(b, 65) and p.acquire(1) == -1
    pages = set(p.get(a).pages)
    p.release(a)
    c = p.acquire(64 * 5)
    assert set(p.get(c).pages) == pages and p.get(c).cap == 320
    p.pin(b, True)
    assert p.lru_victim() == c


def test_greedy_generation_long_and_batched():
    cfg, T = _setup(MIXED)
    mc = U.V.read_config(cfg)
    eng = LLMEngine(mc, U.V.from_tensors(mc, T), device="cpu", max_seqs=3, kv_tokens_per_seq=256)
    prompts = [U.prompt(n, cfg["vocab"], n) for n in (1, 60, 33)]
    outs = eng.generate(prompts, max_new=70)
    for p, o in zip(prompts, outs):
        want = U.oracle_logits(cfg, T, p + o)[len(p) - 1: -1]
        assert o == want.argmax(-1).tolist()


def _serve(es, msgs):
    for m in msgs:
        es.submit(m)
    guard = 0
    while es.sched.has_work() and guard < 5000:
        es.step()
        guard += 1
    out, es.out = es.out, []
    return {m["id"]: m for m in out if m.get("done") or "error" in m}


@pytest.mark.parametrize("drafts", [False, True])
def test_scheduler_generates_the_oracles_text(drafts):
    """Requests through admission, shared prompt chunks, batched rounds (with drafts that are verified and committed), a
    continued conversation, more requests than slots."""
    cfg, T = _setup(MIXED)
    mc = U.V.read_config(cfg)
    es = EngineServer(mc, U.V.from_tensors(mc, T), EngineConfig(max_seqs=2, kv_tokens=1024, prefill_chunk=24, spec="lookup" if drafts else "none",
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
    cfg, T = _setup(MIXED)
    toks = U.prompt(80, cfg["vocab"], 2)
    m = U.framework(cfg, T, slots=3, tokens=128)
    kv = KvManager(m)
    assert kv.assign(0, 100) and kv.assign(2, 100)
    m.forward(make_plan([(0, toks[:70], 0)]))
    snap = m.snapshot(0)
    m.restore(2, snap)
    got = m.forward(make_plan([(2, toks[70:], 70)]))
    assert U.error(got, U.oracle_logits(cfg, T, toks)[70:]) < 1e-5


def test_switches():
    from spark_engine_b200.config import get_model_config
    mc = get_model_config("vabunex-style", n_layers=5)
    assert mc.layer_runs() == [0, 1, 2, 3, 4, 4] and mc.layer_specs[1].kind == "wkv"
    assert dataclasses.replace(mc).layer_specs
    with pytest.raises(ValueError):
        LLMEngine(mc, {}, EngineConfig(dtype="float8"), device="cuda")
