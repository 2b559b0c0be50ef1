"""Debisun: pre-norm blocks (layer norms, per-channel scales on both branches) of chunked grouped-query attention and a
dense or routed squared-relu feed-forward, followed by a per-layer input from the token's own embedding row.

This module reads the checkpoint (config.json, tensor names) and lays the weights out for the runner:

  mix   qkv = [q | k | v] rows and conv_t [taps, rows] in the same order, every head padded to a multiple of 16 rows;
        dist_bias [heads, distances] (the bucketed table spread over distances, the last entry serves everything farther),
        sink [heads] (score of the key without a value: 0), o with the value heads' columns padded alike
  mlp   dense_up, dense_down, or gate = [router | shared gate] rows, bias (added to the choice scores), w_up / w_down expert
        stacks, s_up / s_down (shared expert); widths padded to 8
  side  gate, proj (padded to 8), norm; the token rows of all layers stay one table (W["side_embed"])

Padding is zero, so every slice the kernels address is 16-byte aligned whatever the model's sizes are."""
from __future__ import annotations

import math
import os
from typing import Dict

import torch

from ..config import LayerSpec, ModelConfig, MoeConfig, PagedGqaConfig
from .layout import pad, pad_cols, pad_head_cols, pad_head_rows, stack_rows, taker


# ----------------------------------------------------------------------------- configuration
def _mixer(kind: str, m: dict) -> PagedGqaConfig:
    if kind != "attention":
        raise ValueError(f"unknown mixer type {kind!r}")
    mask = m.get("mask")
    c = PagedGqaConfig(n_heads=m["heads"], n_kv_heads=m["kv_heads"], head_dim=m["dim"], v_dim=m["vdim"], conv_k=m["conv"],
                       scale=float(m["scale"]), softcap=float(m.get("softcap") or 0.0), bias_buckets=0, bias_max=m["bias_max"],
                       chunk=int(mask["size"]) if mask else 0)
    if c.n_heads % c.n_kv_heads:
        raise ValueError("attention heads must be a multiple of the key/value heads")
    return c


def _mlp(m):
    """(dense width, MoeConfig or None) of a layer's feed-forward."""
    if m is None:
        return 0, None
    if m["kind"] == "dense":
        return int(m["ff"]), None
    if m["kind"] != "moe":
        raise ValueError(f"unknown feed-forward kind {m['kind']!r}")
    r, shared = m["router"], m.get("shared")
    return 0, MoeConfig(n_experts=int(r["experts"]), n_identity=int(r.get("identity", 0)), top_k=int(r["top"]), ffn=int(m["expert"]["ff"]),
                        n_shared=1 if shared else 0, shared_ffn=int(shared["ff"]) if shared else 0, router="softmax_bias",
                        route_scale=float(r["scale"]), shared_gate=bool(shared), act="relu2")


def read_config(d: dict) -> ModelConfig:
    specs = []
    for x in d["layers"]:
        ffn, moe = _mlp(x.get("mlp"))
        specs.append(LayerSpec("gqa", _mixer(x["type"], x["mixer"]), ffn, moe))
    side = d.get("token_side")
    return ModelConfig(name="debisun", family="debisun", n_layers=len(specs), layer_types=[s.kind for s in specs], hidden=int(d["width"]),
                       vocab=int(d["vocab"]), norm_eps=float(d["norm"]["eps"]), layer_specs=specs, block="sequential", norm_kind="layer",
                       side_dim=int(side["dim"]) if side else 0, weight_format="dense")


# ----------------------------------------------------------------------------- layout
def distance_buckets(n: int, rows: int, far: int) -> torch.Tensor:
    """Row of the bias table for the distances 0 .. n-1: the distance itself below rows/2, then logarithmic up to `far`."""
    half = rows // 2
    return torch.tensor([i if i < half else min(rows - 1, half + math.floor(math.log(i / half) / math.log(far / half) * (rows - half)))
                         for i in range(n)])


def prepare_layer(raw: Dict[str, torch.Tensor], spec: LayerSpec, dtype) -> dict:
    """`raw`: this layer's tensors by their names behind the layer prefix, on the target device."""
    m = {k[4:]: t for k, t in raw.items() if k.startswith("mix.")}
    f = {k[4:]: t for k, t in raw.items() if k.startswith("mlp.")}
    c, e = spec.mixer, spec.moe
    f32 = lambda t: t.float().contiguous()
    wd = lambda t: t.to(dtype).contiguous()
    H, G, Dp, Vp = c.n_heads, c.n_kv_heads, pad(c.head_dim, 16), pad(c.v_dim, 16)
    heads = (("q", H, Dp), ("k", G, Dp), ("v", G, Vp))
    c.bias_buckets = m["rel"].shape[0]
    n = max(int(math.ceil(c.bias_max)) + 1, c.bias_buckets)
    near = distance_buckets(min(n, c.chunk) if c.chunk else n, c.bias_buckets, c.bias_max)
    mix = {"qkv": wd(torch.cat([pad_head_rows(m[s], n, d) for s, n, d in heads])),
           "conv_t": f32(torch.cat([pad_head_rows(m[s + ".conv"], n, d) for s, n, d in heads]).t()),
           "dist_bias": f32(m["rel"].float()[near.to(m["rel"].device)].t()),
           "sink": torch.zeros(H, dtype=torch.float32, device=m["o"].device), "o": wd(pad_head_cols(m["o"], H, Vp))}
    w = {"type": spec.kind, "in_norm": f32(raw["norm1"]), "in_norm_b": f32(raw["norm1.b"]), "ls1": f32(raw["ls1"]), "mix": mix, "mlp": {}}
    if spec.ffn or e is not None:
        w.update(post_norm=f32(raw["norm2"]), post_norm_b=f32(raw["norm2.b"]), ls2=f32(raw["ls2"]))
    if spec.ffn:
        w["mlp"] = {"dense_up": wd(stack_rows([f["up"]])), "dense_down": wd(pad_cols(f["down"], pad(spec.ffn, 8)))}
    elif e is not None:
        up = lambda k: stack_rows([f[k + ".up"]])
        down = lambda k: pad_cols(f[k + ".down"], pad(f[k + ".down"].shape[1], 8))
        names = [f"e{j}" for j in range(e.n_experts)]
        w["mlp"] = {"gate": wd(torch.cat([f["router"]] + ([f["shared.sg"]] if e.n_shared else []))), "bias": f32(f["correction"]),
                    "w_up": wd(torch.stack([up(k) for k in names])), "w_down": wd(torch.stack([down(k) for k in names]))}
        if e.n_shared:
            w["mlp"].update(s_up=wd(up("shared")), s_down=wd(down("shared")))
    if "side.gate" in raw:
        n8 = pad(raw["side.gate"].shape[0], 8)
        w["side"] = {"gate": wd(stack_rows([raw["side.gate"]])), "proj": wd(pad_cols(raw["side.proj"], n8)), "norm": f32(raw["side.norm"])}
    return w


def layer_tensors(cfg: ModelConfig, spec: LayerSpec) -> Dict[str, tuple]:
    """Names and shapes of one layer's tensors behind the layer prefix (None: the tensor decides)."""
    c, e, N = spec.mixer, spec.moe, cfg.hidden
    nq, nk, nv = c.n_heads * c.head_dim, c.n_kv_heads * c.head_dim, c.n_kv_heads * c.v_dim
    t = {"norm1": (N,), "norm1.b": (N,), "ls1": (N,), "mix.q": (nq, N), "mix.k": (nk, N), "mix.v": (nv, N), "mix.q.conv": (nq, c.conv_k),
         "mix.k.conv": (nk, c.conv_k), "mix.v.conv": (nv, c.conv_k), "mix.rel": (c.bias_buckets or None, c.n_heads),
         "mix.o": (N, c.n_heads * c.v_dim)}
    if spec.ffn or e is not None:
        t.update({"norm2": (N,), "norm2.b": (N,), "ls2": (N,)})
    if spec.ffn:
        t.update({"mlp.up": (spec.ffn, N), "mlp.down": (N, spec.ffn)})
    elif e is not None:
        t.update({"mlp.router": (e.n_routes, N), "mlp.correction": (e.n_routes,)})
        for k, n in [(f"e{j}", e.ffn) for j in range(e.n_experts)] + ([("shared", e.shared_ffn)] if e.n_shared else []):
            t.update({f"mlp.{k}.up": (n, N), f"mlp.{k}.down": (N, n)})
        if e.n_shared:
            t["mlp.shared.sg"] = (1, N)
    if cfg.side_dim:
        t.update({"side.gate": (cfg.side_dim, N), "side.proj": (N, cfg.side_dim), "side.norm": (N,)})
    return t


def _assemble(cfg: ModelConfig, get, layer, dtype, stored: bool) -> dict:
    W = {"embed": get("embed", (cfg.vocab, cfg.hidden)).to(dtype).contiguous(), "final_norm": get("final.norm", (cfg.hidden,)).float().contiguous(),
         "final_norm_b": get("final.norm.b", (cfg.hidden,)).float().contiguous(),
         "lm_head": get("head", (cfg.vocab, cfg.hidden)).to(dtype).contiguous()}
    if cfg.side_dim:
        t = get("side.embed", (cfg.vocab, None)) if stored else get("side.embed", (cfg.vocab, cfg.n_layers * cfg.side_dim))
        if t.shape[1] < cfg.n_layers * cfg.side_dim:
            raise ValueError(f"tensor side.embed has shape {tuple(t.shape)}, the configuration needs {cfg.n_layers * cfg.side_dim} columns")
        W["side_embed"] = t.to(dtype).contiguous()
    W["layers"] = [prepare_layer(layer(i, s), s, dtype) for i, s in enumerate(cfg.layer_specs)]
    return W


def from_tensors(cfg: ModelConfig, tensors: Dict[str, torch.Tensor], device="cpu", dtype=torch.float32) -> dict:
    """Runner weights from a flat dict of checkpoint tensors (validated against the configuration)."""
    get = taker(tensors, device)
    return _assemble(cfg, get, lambda i, spec: {k: get(f"l{i}.{k}", s) for k, s in layer_tensors(cfg, spec).items()},
                     dtype, True)


def load_weights(directory: str, cfg: ModelConfig, device="cpu", dtype=torch.bfloat16) -> dict:
    from .checkpoint import mapped_tensors
    return from_tensors(cfg, mapped_tensors(os.path.join(directory, "model.safetensors")), device, dtype)


def random_weights(cfg: ModelConfig, device="cpu", seed: int = 0, dtype=torch.bfloat16) -> dict:
    """Random weights of the configured sizes, generated on `device` layer by layer."""
    g = torch.Generator(device=device)
    g.manual_seed(seed)
    rnd = lambda *s: torch.randn(*s, device=device, generator=g)

    def tensor(name, shape):
        if name.endswith((".b", "correction")):
            return 0.1 * rnd(*shape)
        if len(shape) == 1:
            return (0.5 if ".ls" in "." + name else 1.0) * (1 + 0.1 * rnd(*shape))
        if name.endswith(("rel", "conv")):
            return rnd(*shape) * (0.5 if name.endswith("rel") else shape[1] ** -0.5)
        return (rnd(*shape) * shape[1] ** -0.5).to(torch.bfloat16)

    def layer(i, spec):
        spec.mixer.bias_buckets = spec.mixer.bias_buckets or 32
        return {k: tensor(k, s) for k, s in layer_tensors(cfg, spec).items()}
    return _assemble(cfg, tensor, layer, dtype, False)
