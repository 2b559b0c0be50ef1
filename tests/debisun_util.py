"""Small Debisun models for the tests: configurations in the checkpoint's own format and random tensors, with the plain
implementation (debisun_oracle) and the framework built from the same ones."""
import debisun_oracle as oracle
import torch
from vabunex_util import error, prompt, write_checkpoint  # noqa: F401  (model-independent helpers)

from spark_engine_b200.models import debisun as D
from spark_engine_b200.models.model import Model


def attention(heads=6, kv_heads=3, dim=20, vdim=36, conv=4, scale=0.31, softcap=6.0, bias_max=90, chunk=70):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv, "scale": scale,
                                           "softcap": softcap, "bias_max": bias_max, "mask": {"size": chunk}}}


def dense(ff=52):
    return {"kind": "dense", "ff": ff}


def moe(experts=5, identity=2, top=3, ff=28, shared=44, scale=1.3):
    m = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "identity": identity, "top": top, "scale": scale}}
    if shared:
        m["shared"] = {"ff": shared}
    return m


def layer(mlp=None, **kw):
    return dict(attention(**kw), mlp=mlp)


def config(layers, width=72, vocab=130, side=12, eps=1e-5):
    return {"architecture": "Debisun", "layers": layers, "norm": {"eps": eps}, "token_side": {"dim": side}, "vocab": vocab, "width": width}


def tensors(cfg, seed=0, rel=10):
    """Random tensors by checkpoint name, in bf16 as a checkpoint stores them; `rel`: rows of the bias tables."""
    g = torch.Generator().manual_seed(seed)
    mc = D.read_config(cfg)
    rnd = lambda *s: torch.randn(*s, generator=g)
    n, v = mc.hidden, mc.vocab
    T = {"embed": rnd(v, n), "side.embed": rnd(v, mc.n_layers * mc.side_dim), "final.norm": 1 + 0.2 * rnd(n), "final.norm.b": 0.2 * rnd(n),
         "head": rnd(v, n) * n ** -0.5}
    for i, spec in enumerate(mc.layer_specs):
        spec.mixer.bias_buckets = rel
        for k, s in D.layer_tensors(mc, spec).items():
            x = rnd(*s)
            if k.endswith(".b"):
                x = 0.2 * x
            elif k.endswith("correction"):
                x = 0.3 * x
            elif len(s) == 1:
                x = 1 + 0.3 * x
            elif k.endswith("conv"):
                x = x * s[1] ** -0.5
            elif not k.endswith("rel"):
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
    mc = D.read_config(cfg)
    return Model(mc, D.from_tensors(mc, T, device, dtype), device=device, dtype=dtype, n_slots=slots, kv_tokens=tokens * slots,
                 slot_tokens=tokens)


MIXED = dict(layers=[layer(dense()), layer(moe(), heads=4, kv_heads=1, dim=24, vdim=16, conv=3, chunk=64, bias_max=40),
                     layer(None, heads=2, kv_heads=2, dim=16, vdim=8, conv=2, chunk=100), layer(moe(top=1, shared=0, identity=1), chunk=33)])
MECHANISMS = {
    "attention": dict(layers=[layer()]),
    "attention, equal sizes": dict(layers=[layer(heads=1, kv_heads=1, dim=16, vdim=16, conv=1, scale=1.0, bias_max=16, chunk=16)]),
    "attention, no sharing of keys": dict(layers=[layer(heads=4, kv_heads=4, conv=2)]),
    "attention, long convolution": dict(layers=[layer(conv=7)]),
    "attention, chunk of one": dict(layers=[layer(chunk=1)]),
    "attention, chunk beyond the prompt": dict(layers=[layer(chunk=1000, bias_max=1500)]),
    "attention, bias reaches its last row": dict(layers=[layer(chunk=90, bias_max=11)]),
    "dense": dict(layers=[layer(dense())]),
    "experts": dict(layers=[layer(moe())]),
    "experts, all chosen": dict(layers=[layer(moe(experts=2, identity=1, top=3, scale=1.0))]),
    "experts, one and no identity": dict(layers=[layer(moe(experts=1, identity=0, top=1, shared=0))]),
    "experts, mostly identity": dict(layers=[layer(moe(experts=1, identity=6, top=4))]),
    "odd sizes": dict(layers=[layer(dense(37), dim=21, vdim=19), layer(moe(ff=13, shared=9), dim=21, vdim=19)], width=75, side=5),
    "narrow side": dict(layers=[layer(dense()), layer(dense())], side=1),
    "different layers": MIXED,
}


def planted_pair(cfg, T):
    """(query token, key token, filler tokens): in a one-layer attention model the key token's score stands out for the query
    token in head 0 (convolutions pass the current token only, a flat bias), the fillers score far below."""
    c = cfg["layers"][0]["mixer"]
    H, G, d = c["heads"], c["kv_heads"], c["dim"]
    for s in "qkv":
        T[f"l0.mix.{s}.conv"].zero_()
        T[f"l0.mix.{s}.conv"][:, -1] = 1
    T["l0.mix.rel"].zero_()
    T["l0.mix.v"] *= 3
    W = oracle_weights(T)
    h = oracle.layer_norm(W["embed"], W["l0.norm1"], W["l0.norm1.b"], cfg["norm"]["eps"])
    q, k = (h @ W["l0.mix.q"].T).view(-1, H, d)[:, 0], (h @ W["l0.mix.k"].T).view(-1, G, d)[:, 0]
    sc = q @ k.T
    qt, kt = divmod(int(sc.argmax()), sc.shape[1])
    c["softcap"], c["scale"] = 40.0, float(18.0 / sc[qt, kt])
    return qt, kt, [int(t) for t in torch.argsort(sc[qt])[: cfg["vocab"] // 2] if int(t) not in (qt, kt)]
