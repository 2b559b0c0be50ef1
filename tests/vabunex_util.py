"""Small Vabunex models for the tests: configurations in the checkpoint's own format and random tensors, with the plain
implementation (vabunex_oracle) and the framework built from the same ones."""
import json
import os

import torch
import vabunex_oracle as oracle

from spark_engine_b200.models import vabunex as V
from spark_engine_b200.models.model import Model


def lightning(heads=3, dim=24, vdim=40, decay=None, ff=56):
    decay = decay or [0.35 + 0.64 * i / max(heads - 1, 1) for i in range(heads)]
    return {"type": "lightning", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def wkv(heads=3, dim=24, ff=56):
    return {"type": "wkv", "mixer": {"heads": heads, "dim": dim}, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def latent(heads=3, dim=24, vdim=40, rot_dim=12, q_rank=44, kv_rank=36, base=700.0, scale=0.21, ff=56):
    return {"type": "latent_attention",
            "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "rot_dim": rot_dim, "q_rank": q_rank, "kv_rank": kv_rank,
                      "rot": {"base": base, "dims": rot_dim}, "scale": scale},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def config(layers, width=88, vocab=130, loop=None, eps=1e-5, scale=3.5):
    d = {"architecture": "Vabunex", "embedding": {"scale": scale}, "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width}
    if loop:
        d["loop"] = dict(zip(("start", "stop", "times"), loop))
    return d


def tensors(cfg, seed=0, rank=10):
    """Random tensors by checkpoint name, in bf16 as a checkpoint stores them."""
    g = torch.Generator().manual_seed(seed)
    mc = V.read_config(cfg)
    T = {"embed": torch.randn(mc.vocab, mc.hidden, generator=g) * mc.hidden ** -0.5, "final.norm": 0.2 * torch.randn(mc.hidden, generator=g),
         "head": torch.randn(mc.vocab, mc.hidden, generator=g) * mc.hidden ** -0.5}
    for i, spec in enumerate(mc.layer_specs):
        if spec.kind == "wkv":
            spec.mixer.decay_rank = rank
        for k, s in V.layer_tensors(spec, mc.hidden).items():
            n = k.split(".")[-1]
            x = torch.randn(*s, generator=g)
            if k.startswith("mix.mu."):
                x = torch.rand(*s, generator=g)
            elif n == "norm":
                x = 1 + 0.2 * x
            elif n == "norm1":
                x = 0.2 * x
            elif n == "w0":
                x = 1.2 * x - 1.5
            elif n == "u":
                x = 0.7 * x
            else:
                x = x * s[1] ** -0.5 * 1.3
            T[f"l{i}.{k}"] = x
    return {k: t.to(torch.bfloat16) for k, t in T.items()}


def write_checkpoint(directory, cfg, T):
    from spark_engine_b200.utils.safetensors_io import write_safetensors
    os.makedirs(directory, exist_ok=True)
    with open(os.path.join(directory, "config.json"), "w") as f:
        json.dump(cfg, f)
    write_safetensors(os.path.join(directory, "model.safetensors"), T, {})


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
    mc = V.read_config(cfg)
    return Model(mc, V.from_tensors(mc, T, device, dtype), device=device, dtype=dtype, n_slots=slots, kv_tokens=tokens * slots,
                 slot_tokens=tokens)


def error(got, want):
    """Root mean square error over the vocabulary relative to the spread of the expected logits, worst row."""
    d = (got.float().cpu() - want).double()
    d = d - d.mean(-1, keepdim=True)
    return float(d.pow(2).mean(-1).sqrt().max() / want.double().std())


def prompt(n, vocab, seed=0):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()
