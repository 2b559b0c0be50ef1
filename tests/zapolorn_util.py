"""Small Zapolorn models for the tests: configurations in the checkpoint's own format and random tensors, with the plain
implementation (zapolorn_oracle) and the framework built from the same ones."""
import torch
import zapolorn_oracle as oracle
from vabunex_util import error, prompt, write_checkpoint  # noqa: F401  (model-independent helpers)

from spark_engine_b200.models import zapolorn as Z
from spark_engine_b200.models.model import Model


def dense(ff=52):
    return {"kind": "dense", "ff": ff}


def moe(experts=5, top=2, ff=28, shared=44):
    m = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared:
        m["shared"] = {"ff": shared}
    return m


def window(mlp=None, heads=6, kv_heads=3, dim=20, vdim=36, size=70, rot=12, base=700.0, factor=2.5, scale=0.41, kv_from=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "mask": {"size": size},
         "rot": {"base": base, "dims": rot, "scaling": {"factor": factor}}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m, "mlp": mlp}


def pair(mlp=None, heads=4, kv_heads=2, dim=24, vdim=40, scale=0.37, coef=0.3, every=19, rheads=3, rdim=20, rvdim=28, tau=5.0, left=0.8, right=1.1):
    return {"type": "parallel", "mlp": mlp,
            "mixer": {"left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "q_temp": {"coef": coef, "every": every}},
                      "right": {"heads": rheads, "dim": rdim, "vdim": rvdim, "tau": tau}, "left_scale": left, "right_scale": right}}


def config(layers, width=72, vocab=130, eps=1e-5, scale=3.5, logit_scale=0.7):
    return {"architecture": "Zapolorn", "embedding": {"scale": scale}, "layers": layers, "logit_scale": logit_scale, "norm": {"eps": eps},
            "vocab": vocab, "width": width}


def tensors(cfg, seed=0, rank=10):
    """Random tensors by checkpoint name, in bf16 as a checkpoint stores them; `rank`: of the decays."""
    g = torch.Generator().manual_seed(seed)
    mc = Z.read_config(cfg)
    rnd = lambda *s: torch.randn(*s, generator=g)
    T = {"embed": rnd(mc.vocab, mc.hidden) * mc.hidden ** -0.5, "final.norm": 1 + 0.2 * rnd(mc.hidden)}
    for i, spec in enumerate(mc.layer_specs):
        if spec.kind == "side_by_side":
            spec.mixer.right.decay_rank = rank
        for k, s in Z.layer_tensors(mc, spec).items():
            x = rnd(*s)
            if k.endswith("a2.b"):
                x = 1.5 * x + 1.5
            elif k.endswith("sink"):
                x = 1.5 * x
            elif len(s) == 1:
                x = 1 + 0.3 * x
            else:
                x = x * s[1] ** -0.5 * (3.0 if k.endswith("router") else 1.3)
            T[f"l{i}.{k}"] = x
    return {k: t.to(torch.bfloat16) for k, t in T.items()}


def oracle_weights(T, dtype=torch.float64):
    return {k: t.to(dtype) for k, t in T.items()}


def oracle_logits(cfg, T, tokens, taps=None):
    return oracle.forward(cfg, oracle_weights(T), tokens, taps).float()


def oracle_greedy(cfg, T, prompt, n):
    W, toks = oracle_weights(T), list(prompt)
    for _ in range(n):
        toks.append(int(oracle.forward(cfg, W, toks)[-1].argmax()))
    return toks[len(prompt):]


def framework(cfg, T, device="cpu", dtype=torch.float32, slots=4, tokens=1024):
    mc = Z.read_config(cfg)
    return Model(mc, Z.from_tensors(mc, T, device, dtype), device=device, dtype=dtype, n_slots=slots, kv_tokens=tokens * slots,
                 slot_tokens=tokens)


SMALL = dict(heads=4, kv_heads=1, dim=24, vdim=16, size=33, rot=8)
MIXED = dict(layers=[window(dense()), pair(moe()), window(moe(top=1, shared=0), kv_from=0, size=100), window(None, **SMALL),
                     pair(None, heads=3, kv_heads=3, dim=16, vdim=8, rheads=2, rdim=12, rvdim=44, tau=14.0), window(moe(), kv_from=3, **SMALL)])
MECHANISMS = {
    "window attention": dict(layers=[window()]),
    "window attention, equal sizes and ones": dict(layers=[window(heads=1, kv_heads=1, dim=16, vdim=16, size=1, rot=16, factor=1.0, scale=1.0)]),
    "window attention, no sharing of heads": dict(layers=[window(heads=4, kv_heads=4, rot=20)]),
    "window beyond the prompt": dict(layers=[window(size=1000, base=3e5)]),
    "window of a page": dict(layers=[window(size=64, rot=2)]),
    "keys of another layer": dict(layers=[window(dense(), size=9), window(kv_from=0, size=50, scale=0.2), window(size=4), window(kv_from=0, size=9)]),
    "side by side": dict(layers=[pair()]),
    "side by side, equal sizes and ones": dict(layers=[pair(heads=1, kv_heads=1, dim=16, vdim=16, scale=0.2, coef=1.0, every=1, rheads=1, rdim=16,
                                                            rvdim=16, tau=1.0, left=1.0, right=1.0)]),
    "side by side, heads of no power of two": dict(layers=[pair(heads=6, kv_heads=3, rheads=5, rdim=8, rvdim=12, every=7)]),
    "side by side, nothing on the left": dict(layers=[pair(left=0.0)]),
    "side by side, nothing on the right": dict(layers=[pair(right=0.0)]),
    "dense": dict(layers=[window(dense())]),
    "experts": dict(layers=[window(moe())]),
    "experts, all chosen": dict(layers=[pair(moe(experts=3, top=3))]),
    "experts, one of one": dict(layers=[window(moe(experts=1, top=1, shared=0))]),
    "odd sizes": dict(layers=[window(dense(37), dim=21, vdim=19, rot=6), pair(moe(ff=13, shared=9), dim=21, vdim=19, rdim=11, rvdim=13)], width=75),
    "different layers": MIXED,
}


def planted_pair(cfg, T):
    """(query token, key token, filler tokens): in a one-layer model whose scores depend on the tokens only, the key token's score
    stands out for the query token in the last head, the fillers score far below."""
    lc = cfg["layers"][0]
    left = lc["type"] == "parallel"
    c, p = (lc["mixer"]["left"], "l0.mix.left.") if left else (lc["mixer"], "l0.mix.")
    H, G, d = c["heads"], c["kv_heads"], c["dim"]
    T[p + "v"] *= 3
    W = oracle_weights(T)
    x, eps = W["embed"] * cfg["embedding"]["scale"], cfg["norm"]["eps"]
    q = oracle.rms_norm((x @ W[p + "q"].T).view(-1, H, d)[:, -1], W[p + "q.norm"], eps)
    k = oracle.rms_norm((x @ W[p + "k"].T).view(-1, G, d)[:, -1], W[p + "k.norm"], eps)
    sc = q @ k.T
    qt, kt = divmod(int(sc.argmax()), sc.shape[1])
    c["scale"] = float(12.0 / sc[qt, kt])
    return qt, kt, [int(t) for t in torch.argsort(sc[qt])[: cfg["vocab"] // 2] if int(t) not in (qt, kt)]
