"""Zakusun: pre-norm blocks (RMS norms over groups of channels, a short convolution over time added to what every sublayer reads)
of latent attention without positions (direct queries, a learned sink per head, an element-wise output gate) and routed experts
with a clamped gated activation; sinusoidal positions on the embedding, and behind every layer a learned sum of the embedding and
all layers' results.

This module reads the checkpoint (config.json, tensor names) and lays the weights out for the runner:

  latent   in = [q (per head padded to 16) | latent (padded to 16) | gate] rows, kv_norm, sink; uk_t [heads, latent, dim] and
           uv [heads, v, latent] for absorbed decode rows, kv_up (per head [key | value] padded to 16) for prompts; out (columns
           padded to 8)
  mlp      gate = router rows, bias (added to the router's logits), w_gu / w_down expert stacks (widths padded to 128)
  layer    in_norm, post_norm; conv1, conv2 [taps, width]; depth [layers so far + 2]

Padding is zero.  The logit scale is part of the final norm's weight; the head is the embedding table."""
from __future__ import annotations

import os
from typing import Dict

import torch

from ..config import LatentConfig, LayerSpec, ModelConfig, MoeConfig
from .layout import latent_up, pad, pad_cols, pad_head_rows, stack_rows, taker

WIDE = 128
GLU_ALPHA, GLU_SHIFT = 1.702, 1.0


# ----------------------------------------------------------------------------- configuration
def _mixer(kind: str, m: dict) -> LatentConfig:
    if kind != "latent_attention":
        raise ValueError(f"unknown mixer type {kind!r}")
    return LatentConfig(n_heads=int(m["heads"]), head_dim=int(m["dim"]), v_dim=int(m["vdim"]), q_rank=0, kv_rank=int(m["kv_rank"]), rope_dim=0,
                        scale=float(m["scale"]), sink=True, gate="element")


def _mlp(m):
    if m is None:
        return None
    if m["kind"] != "moe":
        raise ValueError(f"unknown feed-forward kind {m['kind']!r}")
    r, e = m["router"], m["expert"]
    if not 0 < int(r["top"]) <= int(r["experts"]):
        raise ValueError(f"cannot choose {r['top']} of {r['experts']} experts")
    limit = max(float(e["limit"]), 1e-30)                    # (0 stands for "no limit" in MoeConfig)
    return MoeConfig(n_experts=int(r["experts"]), top_k=int(r["top"]), ffn=int(e["ff"]), n_shared=0, router="topk_softmax", swiglu_limit=limit,
                     glu_alpha=GLU_ALPHA, glu_shift=GLU_SHIFT)


def read_config(d: dict) -> ModelConfig:
    specs = [LayerSpec("latent", _mixer(x["type"], x["mixer"]), 0, _mlp(x.get("mlp"))) for x in d["layers"]]
    width, groups = int(d["width"]), int(d["norm"].get("groups", 1))
    if groups < 1 or width % groups:
        raise ValueError(f"cannot norm {width} channels in {groups} equal groups")
    return ModelConfig(name="zakusun", family="zakusun", n_layers=len(specs), layer_types=[s.kind for s in specs], hidden=width,
                       vocab=int(d["vocab"]), norm_eps=float(d["norm"]["eps"]), layer_specs=specs, block="sequential", norm_groups=groups,
                       input_conv=int(d["canon"]["taps"]), depth_average=True, positions="sinusoidal",
                       logit_scale=float(d.get("logit_scale", 1.0)), tied_head=True, weight_format="dense")


# ----------------------------------------------------------------------------- layout
def _f32(t):
    return t.float().contiguous()


def prepare_layer(raw: Dict[str, torch.Tensor], spec: LayerSpec, dtype) -> dict:
    """`raw`: this layer's tensors by their names behind the layer prefix, on the target device."""
    wd = lambda t: t.to(dtype).contiguous()
    m = {k[4:]: t for k, t in raw.items() if k.startswith("mix.")}
    f = {k[4:]: t for k, t in raw.items() if k.startswith("mlp.")}
    c, e = spec.mixer, spec.moe
    mix = {"in": wd(torch.cat((pad_head_rows(m["q"], c.n_heads, pad(c.head_dim, 16)), stack_rows([m["dkv"]], 16), stack_rows([m["g"]])))),
           "kv_norm": _f32(m["dkv.norm"]), "sink": _f32(m["sink"]), "out": wd(pad_cols(m["o"], pad(c.n_heads * c.v_dim, 8))),
           **latent_up(m["uk"], m["uv"], c, dtype)}
    w = {"type": spec.kind, "in_norm": _f32(raw["norm1"]), "conv1": _f32(raw["canon1"].t()), "depth": _f32(raw["dwa"]), "mix": mix, "mlp": {}}
    if e is not None:
        gu = lambda k: stack_rows([f[k + "gate"], f[k + "up"]], WIDE)
        down = lambda k: pad_cols(f[k + "down"], pad(e.ffn, WIDE))
        names = [f"e{j}." for j in range(e.n_experts)]
        w.update(post_norm=_f32(raw["norm2"]), conv2=_f32(raw["canon2"].t()))
        w["mlp"] = {"gate": wd(f["router"]), "bias": _f32(f["router.b"]), "w_gu": wd(torch.stack([gu(k) for k in names])),
                    "w_down": wd(torch.stack([down(k) for k in names]))}
    return w


def layer_tensors(cfg: ModelConfig, i: int) -> Dict[str, tuple]:
    """Names and shapes of layer i's tensors behind the layer prefix."""
    spec, N = cfg.layer_specs[i], cfg.hidden
    c, e = spec.mixer, spec.moe
    nv = c.n_heads * c.v_dim
    t = {"norm1": (N,), "canon1": (N, cfg.input_conv), "dwa": (i + 2,), "mix.q": (c.n_heads * c.head_dim, N), "mix.dkv": (c.kv_rank, N),
         "mix.dkv.norm": (c.kv_rank,), "mix.uk": (c.n_heads * c.head_dim, c.kv_rank), "mix.uv": (nv, c.kv_rank), "mix.sink": (c.n_heads,),
         "mix.g": (nv, N), "mix.o": (N, nv)}
    if e is not None:
        t.update({"norm2": (N,), "canon2": (N, cfg.input_conv), "mlp.router": (e.n_experts, N), "mlp.router.b": (e.n_experts,)})
        for j in range(e.n_experts):
            t.update({f"mlp.e{j}.gate": (e.ffn, N), f"mlp.e{j}.up": (e.ffn, N), f"mlp.e{j}.down": (N, e.ffn)})
    return t


def _assemble(cfg: ModelConfig, get, layer, dtype) -> dict:
    embed = get("embed", (cfg.vocab, cfg.hidden)).to(dtype).contiguous()
    return {"embed": embed, "lm_head": embed, "final_norm": _f32(get("final.norm", (cfg.hidden,)).float() * cfg.logit_scale),
            "layers": [prepare_layer(layer(i), s, dtype) for i, s in enumerate(cfg.layer_specs)]}


def from_tensors(cfg: ModelConfig, tensors: Dict[str, torch.Tensor], device="cpu", dtype=torch.float32) -> dict:
    """Runner weights from a flat dict of checkpoint tensors (validated against the configuration)."""
    get = taker(tensors, device)
    return _assemble(cfg, get, lambda i: {k: get(f"l{i}.{k}", s) for k, s in layer_tensors(cfg, i).items()}, dtype)


def load_weights(directory: str, cfg: ModelConfig, device="cpu", dtype=torch.bfloat16) -> dict:
    from .checkpoint import mapped_tensors
    return from_tensors(cfg, mapped_tensors(os.path.join(directory, "model.safetensors")), device, dtype)


def random_weights(cfg: ModelConfig, device="cpu", seed: int = 0, dtype=torch.bfloat16) -> dict:
    """Random weights of the configured sizes, generated on `device` layer by layer."""
    g = torch.Generator(device=device)
    g.manual_seed(seed)
    rnd = lambda *s: torch.randn(*s, device=device, generator=g)

    def tensor(name, shape):
        if name.endswith(("sink", "router.b")):
            return rnd(*shape)
        if name == "dwa":
            return torch.cat((0.3 * rnd(shape[0] - 1) / shape[0], torch.ones(1, device=device)))
        if len(shape) == 1:
            return 1 + 0.1 * rnd(*shape)
        return (rnd(*shape) * shape[1] ** -0.5).to(torch.bfloat16)
    return _assemble(cfg, tensor, lambda i: {k: tensor(k, s) for k, s in layer_tensors(cfg, i).items()}, dtype)
