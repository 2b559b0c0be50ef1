"""Vabunex: parallel blocks (one zero-centred norm feeds a mixer and a dense feed-forward, both outputs are added to the
residual) over three mixers -- constant-decay linear attention, a token-shifted recurrence with per-channel decay, latent
attention -- with an optional run of layers that is applied several times.

This module reads the checkpoint (config.json, tensor names) and lays the weights out for the runner:

  lightning  in = [q | k | v | g | gate | up] rows (every part padded to 8 rows), norm, log2 decays
  wkv        rkvg [4, heads * dim, hidden], w1 (padded to 8 rows), w2, w0, u, mu [5, hidden] (r k v g w), norm, ff = [gate | up]
  latent     in = [dq | latent | rotated key | g | gate | up] rows, dq_norm, kv_norm, uq (per head [dim | rot] padded to 16),
             uk_t [heads, latent, dim] and uv [heads, v, latent] for absorbed decode rows, kv_up (per head [key | value]
             padded to 16) for prompts
  all        out = [o | down] side by side along K: the mixer's output and the down projection are one product

Padding rows and columns are zero, so every slice the kernels address is 16-byte aligned whatever the model's sizes."""
from __future__ import annotations

import math
import os
from typing import Dict

import torch

from ..config import LatentConfig, LayerSpec, LightningConfig, LoopConfig, ModelConfig, WkvConfig
from .layout import latent_up, pad, pad_cols as _cols, stack_rows as _rows, taker


# ----------------------------------------------------------------------------- configuration
def _mixer(kind: str, m: dict):
    if kind == "lightning":
        return "lightning", LightningConfig(m["heads"], m["dim"], m["vdim"], [float(x) for x in m["decay"]])
    if kind == "wkv":
        return "wkv", WkvConfig(m["heads"], m["dim"], 0)                     # the decay rank is a tensor's shape
    if kind == "latent_attention":
        rot = m["rot"]
        if rot["dims"] != m["rot_dim"]:
            raise ValueError("latent_attention rotates exactly its rot_dim part")
        return "latent", LatentConfig(m["heads"], m["dim"], m["vdim"], m["q_rank"], m["kv_rank"], m["rot_dim"],
                                      float(rot["base"]), True, float(m["scale"]))
    raise ValueError(f"unknown mixer type {kind!r}")


def read_config(d: dict) -> ModelConfig:
    specs = []
    for x in d["layers"]:
        kind, mc = _mixer(x["type"], x["mixer"])
        mlp = x.get("mlp")
        if mlp is not None and mlp["kind"] != "dense":
            raise ValueError(f"unknown feed-forward kind {mlp['kind']!r}")
        specs.append(LayerSpec(kind, mc, int(mlp["ff"]) if mlp is not None else 0))
    lp = d.get("loop")
    loop = LoopConfig(int(lp["start"]), int(lp["stop"]), int(lp["times"])) if lp else None
    if loop is not None and not 0 <= loop.start <= loop.stop <= len(specs):
        raise ValueError("loop outside the layers")
    emb = d.get("embedding") or {}
    return ModelConfig(name="vabunex", family="vabunex", n_layers=len(specs), layer_types=[s.kind for s in specs],
                       hidden=int(d["width"]), vocab=int(d["vocab"]), norm_eps=float(d["norm"]["eps"]), layer_specs=specs,
                       loop=loop, norm_one_plus=True, embed_scale=float(emb.get("scale", 1.0)), weight_format="dense")


# ----------------------------------------------------------------------------- layout
def prepare_layer(raw: Dict[str, torch.Tensor], spec: LayerSpec, hidden: int, dtype) -> dict:
    """`raw`: this layer's tensors by their names behind the layer prefix, on the target device."""
    m = {k[4:]: t for k, t in raw.items() if k.startswith("mix.")}
    c, F = spec.mixer, spec.ffn
    f32 = lambda t: t.float().contiguous()
    wd = lambda t: t.to(dtype).contiguous()
    ff = [raw["mlp.gate"], raw["mlp.up"]] if F else []
    no = c.n_heads * (c.v_dim if spec.kind != "wkv" else c.head_dim)          # columns of the mixer's output matrix
    out = [_cols(m["o"], pad(no, 8))] + ([_cols(raw["mlp.down"], pad(F, 8))] if F else [])
    w = {"out": wd(torch.cat(out, 1))}
    if spec.kind == "lightning":
        w["in"] = wd(_rows([m["q"], m["k"], m["v"], m["g"]] + ff))
        w["norm"] = f32(m["norm"])
        w["log2_decay"] = torch.tensor([max(math.log2(x), -1000.0) if x > 0 else -1000.0 for x in c.decay], dtype=torch.float32,
                                       device=m["o"].device)
    elif spec.kind == "wkv":
        c.decay_rank = m["w1"].shape[0]
        r8 = pad(c.decay_rank, 8)
        w["rkvg"] = wd(torch.stack([m[s] for s in "rkvg"]))
        w["w1"] = wd(_rows([m["w1"]]))
        w["w2"] = wd(_cols(m["w2"], r8))
        w["w0"], w["u"], w["norm"] = f32(m["w0"]), f32(m["u"]), f32(m["norm"])
        w["mu"] = f32(torch.stack([m["mu." + s] for s in "rkvgw"]))
        if F:
            w["ff"] = wd(_rows(ff))
    else:
        H, D, R, L = c.n_heads, c.head_dim, c.rope_dim, c.kv_rank
        Dp, Rp = pad(D, 16), pad(R, 16)
        dkv = m["dkv"]
        w["in"] = wd(torch.cat((_rows([m["dq"]]), _rows([dkv[:L]], 16), _rows([dkv[L:]], 16), _rows([m["g"]] + ff))))
        w["dq_norm"], w["kv_norm"] = f32(m["dq.norm"]), f32(m["dkv.norm"])
        uq = _cols(m["uq"], pad(c.q_rank, 8)).view(H, D + R, -1)
        q = uq.new_zeros(H, Dp + Rp, uq.shape[-1])
        q[:, :D], q[:, Dp: Dp + R] = uq[:, :D], uq[:, D:]
        w["uq"] = wd(q.view(H * (Dp + Rp), -1))
        w.update(latent_up(m["uk"], m["uv"], c, dtype))
    return {"type": spec.kind, "in_norm": f32(raw["norm1"]), "mix": w, "mlp": {"ffn": F}}


def layer_tensors(spec: LayerSpec, hidden: int) -> Dict[str, tuple]:
    """Names and shapes of one layer's tensors behind the layer prefix."""
    c, H, F = spec.mixer, hidden, spec.ffn
    t = {"norm1": (H,)}
    if spec.kind == "lightning":
        nk, nv = c.n_heads * c.head_dim, c.n_heads * c.v_dim
        t.update({"mix.q": (nk, H), "mix.k": (nk, H), "mix.v": (nv, H), "mix.g": (nv, H), "mix.o": (H, nv), "mix.norm": (nv,)})
    elif spec.kind == "wkv":
        n = c.n_heads * c.head_dim
        t.update({f"mix.{s}": (n, H) for s in "rkvg"})
        t.update({f"mix.mu.{s}": (H,) for s in "rkvgw"})
        t.update({"mix.w0": (n,), "mix.u": (c.n_heads, c.head_dim), "mix.norm": (n,), "mix.o": (H, n)})
        if c.decay_rank:
            t.update({"mix.w1": (c.decay_rank, H), "mix.w2": (n, c.decay_rank)})
    else:
        h, L = c.n_heads, c.kv_rank
        t.update({"mix.dq": (c.q_rank, H), "mix.dq.norm": (c.q_rank,), "mix.uq": (h * (c.head_dim + c.rope_dim), c.q_rank),
                  "mix.dkv": (L + c.rope_dim, H), "mix.dkv.norm": (L,), "mix.uk": (h * c.head_dim, L), "mix.uv": (h * c.v_dim, L),
                  "mix.g": (h, H), "mix.o": (H, h * c.v_dim)})
    if F:
        t.update({"mlp.gate": (F, H), "mlp.up": (F, H), "mlp.down": (H, F)})
    return t


def _assemble(cfg: ModelConfig, get, layer, device, dtype) -> dict:
    return {"embed": get("embed").to(dtype).contiguous(), "final_norm": get("final.norm").float().contiguous(),
            "lm_head": get("head").to(dtype).contiguous(),
            "layers": [prepare_layer(layer(i), s, cfg.hidden, dtype) for i, s in enumerate(cfg.layer_specs)]}


def from_tensors(cfg: ModelConfig, tensors: Dict[str, torch.Tensor], device="cpu", dtype=torch.float32) -> dict:
    """Runner weights from a flat dict of checkpoint tensors (validated against the configuration)."""
    get = taker(tensors, device)

    def layer(i):
        spec, p = cfg.layer_specs[i], f"l{i}."
        raw = {k: get(p + k, s) for k, s in layer_tensors(spec, cfg.hidden).items()}
        if spec.kind == "wkv":
            raw.update({k: get(p + k) for k in ("mix.w1", "mix.w2")})
        return raw
    return _assemble(cfg, get, layer, device, dtype)


def load_weights(directory: str, cfg: ModelConfig, device="cpu", dtype=torch.bfloat16) -> dict:
    from .checkpoint import mapped_tensors
    return from_tensors(cfg, mapped_tensors(os.path.join(directory, "model.safetensors")), device, dtype)


def random_weights(cfg: ModelConfig, device="cpu", seed: int = 0, dtype=torch.bfloat16) -> dict:
    """Random weights of the configured sizes, generated on `device` layer by layer."""
    g = torch.Generator(device=device)
    g.manual_seed(seed)
    rnd = lambda *s: torch.randn(*s, device=device, generator=g)

    def layer(i):
        raw = {}
        for k, s in layer_tensors(cfg.layer_specs[i], cfg.hidden).items():
            name = k.split(".")[-1]
            if k.startswith("mix.mu."):
                raw[k] = torch.rand(*s, device=device, generator=g)
            elif name == "norm":
                raw[k] = 1 + 0.1 * rnd(*s)
            elif name in ("norm1", "u"):
                raw[k] = 0.1 * rnd(*s)
            elif name == "w0":
                raw[k] = rnd(*s) - 2.0
            else:
                raw[k] = (rnd(*s) * s[1] ** -0.5).to(torch.bfloat16)
        return raw

    top = {"embed": lambda: rnd(cfg.vocab, cfg.hidden) * cfg.hidden ** -0.5, "final.norm": lambda: 0.1 * rnd(cfg.hidden),
           "head": lambda: rnd(cfg.vocab, cfg.hidden) * cfg.hidden ** -0.5}
    return _assemble(cfg, lambda n: top[n](), layer, device, dtype)
