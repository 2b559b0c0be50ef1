"""Small Zakusun models for the tests: configurations in the checkpoint's own format and random tensors, with the plain
implementation (zakusun_oracle) and the framework built from the same ones."""
import torch
import zakusun_oracle as oracle
from vabunex_util import error, prompt, write_checkpoint  # noqa: F401  (model-independent helpers)

from spark_engine_b200.models import zakusun as Z
from spark_engine_b200.models.model import Model


def moe(experts=5, top=2, ff=28, limit=0.8):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}


def latent(mlp=None, heads=3, dim=20, vdim=36, kv_rank=44, scale=0.41):
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale}, "mlp": mlp}


def config(layers, width=72, vocab=130, eps=1e-5, groups=3, taps=4, logit_scale=0.7):
    return {"architecture": "Zakusun", "canon": {"taps": taps}, "layers": layers, "logit_scale": logit_scale, "norm": {"eps": eps, "groups": groups},
            "vocab": vocab, "width": width}


def tensors(cfg, seed=0):
    """Random tensors by checkpoint name, in bf16 as a checkpoint stores them."""
    g = torch.Generator().manual_seed(seed)
    mc = Z.read_config(cfg)
    rnd = lambda *s: torch.randn(*s, generator=g)
    T = {"embed": 1.5 * rnd(mc.vocab, mc.hidden), "final.norm": 1 + 0.2 * rnd(mc.hidden)}
    for i in range(mc.n_layers):
        for k, s in Z.layer_tensors(mc, i).items():
            x = rnd(*s)
            if k.endswith(("sink", "router.b")):
                x = 1.5 * x
            elif k == "dwa":
                x = 0.5 * x + torch.tensor([0.0] * (i + 1) + [1.0])
            elif k.startswith("canon"):
                x = 0.4 * x
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


MIXED = dict(layers=[latent(moe()), latent(None, heads=5, dim=16, vdim=8, kv_rank=16, scale=0.3), latent(moe(experts=7, top=1, ff=40, limit=0.3)),
                     latent(moe(experts=3, top=3, ff=12, limit=5.0), heads=1, dim=33, vdim=50, kv_rank=70)])
MECHANISMS = {
    "attention": dict(layers=[latent()]),
    "attention, equal sizes and ones": dict(layers=[latent(heads=1, dim=16, vdim=16, kv_rank=16, scale=1.0)], groups=1, taps=1, logit_scale=1.0, width=16),
    "attention, no common sizes": dict(layers=[latent(heads=7, dim=19, vdim=13, kv_rank=29)], width=75, groups=5, taps=3),
    "two attention layers": dict(layers=[latent(), latent(heads=2)], groups=2, taps=2),
    "experts": dict(layers=[latent(moe())]),
    "experts, all chosen": dict(layers=[latent(moe(experts=3, top=3))], taps=2),
    "experts, one of one": dict(layers=[latent(moe(experts=1, top=1))], groups=1),
    "experts, nothing is clamped": dict(layers=[latent(moe(limit=1e9))]),
    "experts, everything is clamped": dict(layers=[latent(moe(limit=1e-3))]),
    "many groups": dict(layers=[latent(moe())], groups=18),
    "groups of an odd width": dict(layers=[latent(moe(ff=13))], width=50, groups=2),
    "no convolution but the token's own tap": dict(layers=[latent(moe()), latent(moe())], taps=1),
    "many taps": dict(layers=[latent(moe())], taps=9),
    "odd width": dict(layers=[latent(moe(ff=13), dim=21, vdim=19)], width=75, groups=5),
    "different layers": MIXED,
}


def planted(cfg, T, n, at):
    """Tokens (n of them, the last one asks) among which the one at `at` has a score that stands out for the last one in the last
    head, and the same tokens with a common one in its place; the scale of the scores is set for it."""
    c, W = cfg["layers"][0]["mixer"], oracle_weights(T)
    H, d, eps = c["heads"], c["dim"], cfg["norm"]["eps"]

    def scores(toks):
        h = oracle.input_convolution(oracle.grouped_rms_norm(oracle.embedding(toks, W), W["l0.norm1"], eps, cfg["norm"]["groups"]), W["l0.canon1"])
        q, k = (h[-1] @ W["l0.mix.q"].T).view(H, d)[-1], oracle.latents(h, W, "l0.mix.", eps) @ W["l0.mix.uk"].T
        return k.view(-1, H, d)[:, -1] @ q
    base = prompt(n, cfg["vocab"], 5)
    s = scores(base)
    low = [t for t, x in zip(base, s.tolist()) if x < 0][:8]
    base = [low[i % len(low)] for i in range(n - 1)] + [base[-1]]
    best = None
    for t in range(cfg["vocab"]):
        toks = list(base)
        toks[at] = t
        s = scores(toks)
        gap = float(s[at] - torch.cat((s[:at], s[at + 1:])).max())
        if best is None or gap > best[0]:
            best = (gap, toks)
    assert best[0] > 0
    c["scale"] = 9.0 / best[0]
    return best[1], base
