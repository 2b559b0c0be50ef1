"""Zapolorn: sublayers that read the residual itself and whose outputs are RMS-normed, over two mixers -- grouped-query window
attention (normed and rotated heads, a learned sink, a gate per head, optionally on another layer's keys and values), and
whole-context attention (tempered queries, a distance slope per head) side by side with gated linear attention -- and dense or
routed SwiGLU feed-forwards whose experts see their input times the routing weight.

This module reads the checkpoint (config.json, tensor names) and lays the weights out for the runner:

  attention     qkv = [q | k | v | gate] rows (with `kv_from`: [q | gate]), every head padded to a multiple of 16 rows; q_norm,
                k_norm; sink [heads]; o with the value heads' columns padded alike
  side by side  in = [left q | k | v | right q | k | v | gate | decay rank] rows; q_norm, k_norm; a2, a2_b (decays); norm
                [right heads * v] with the right side's scale in it; out = [left o | right o] side by side along K: the two
                outputs are one product (the left side's scale is applied to the attention's output)
  mlp           dense_gu = [gate | up], dense_down; or gate = router rows, w_gu / w_down expert stacks, s_gu / s_down (shared)

Feed-forward widths are padded to 128, other rows to 8, with zeros.  The logit scale is part of the final norm's weight; the
head is the embedding table."""
from __future__ import annotations

import os
from typing import Dict

import torch

from ..config import GlaConfig, LayerSpec, ModelConfig, MoeConfig, PagedGqaConfig, SideBySideConfig
from .layout import pad, pad_cols, pad_head_cols, pad_head_rows, stack_rows, taker

WIDE = 128


# ----------------------------------------------------------------------------- configuration
def _gqa(m: dict, **kw) -> PagedGqaConfig:
    c = PagedGqaConfig(n_heads=int(m["heads"]), n_kv_heads=int(m["kv_heads"]), head_dim=int(m["dim"]), v_dim=int(m["vdim"]), conv_k=0,
                       scale=float(m["scale"]), qk_norm=True, **kw)
    if c.n_heads % c.n_kv_heads:
        raise ValueError("attention heads must be a multiple of the key/value heads")
    return c


def _attention(m: dict) -> PagedGqaConfig:
    rot, mask, src = m.get("rot"), m.get("mask"), m.get("kv_from")
    dims = int(rot["dims"]) if rot else 0
    if dims % 2 or dims > m["dim"]:
        raise ValueError(f"cannot rotate {dims} of {m['dim']} dimensions in pairs")
    return _gqa(m, window=int(mask["size"]) if mask else 0, rope_dims=dims, rope_theta=float(rot["base"]) if rot else 1e4,
                rope_factor=float((rot.get("scaling") or {}).get("factor", 1.0)) if rot else 1.0, gated=True,
                kv_from=int(src) if src is not None else None)


def _mixer(kind: str, m: dict):
    if kind == "attention":
        return "gqa", _attention(m)
    if kind == "parallel":
        le, ri, t = m["left"], m["right"], m["left"].get("q_temp") or {}
        return "side_by_side", SideBySideConfig(
            _gqa(le, slopes=True, temp_coef=float(t.get("coef", 0.0)), temp_every=float(t.get("every", 1.0))),
            GlaConfig(int(ri["heads"]), int(ri["dim"]), int(ri["vdim"]), float(ri["tau"]), 0),         # the rank is a tensor's shape
            float(m["left_scale"]), float(m["right_scale"]))
    raise ValueError(f"unknown mixer type {kind!r}")


def _mlp(m):
    """(dense width, MoeConfig or None) of a layer's feed-forward."""
    if m is None:
        return 0, None
    if m["kind"] == "dense":
        return int(m["ff"]), None
    if m["kind"] != "moe":
        raise ValueError(f"unknown feed-forward kind {m['kind']!r}")
    r, shared = m["router"], m.get("shared")
    return 0, MoeConfig(n_experts=int(r["experts"]), top_k=int(r["top"]), ffn=int(m["expert"]["ff"]), n_shared=1 if shared else 0,
                        shared_ffn=int(shared["ff"]) if shared else 0, router="sigmoid", weight_input=True)


def read_config(d: dict) -> ModelConfig:
    specs = []
    for i, x in enumerate(d["layers"]):
        kind, mixer = _mixer(x["type"], x["mixer"])
        src = getattr(mixer, "kv_from", None)
        if src is not None:
            o = specs[src].mixer if 0 <= src < i and specs[src].kind == "gqa" else None
            if o is None or o.kv_from is not None or (o.n_kv_heads, o.head_dim, o.v_dim) != (mixer.n_kv_heads, mixer.head_dim, mixer.v_dim):
                raise ValueError(f"layer {i} cannot use the keys and values of layer {src}")
        specs.append(LayerSpec(kind, mixer, *_mlp(x.get("mlp"))))
    return ModelConfig(name="zapolorn", family="zapolorn", n_layers=len(specs), layer_types=[s.kind for s in specs], hidden=int(d["width"]),
                       vocab=int(d["vocab"]), norm_eps=float(d["norm"]["eps"]), layer_specs=specs, block="post",
                       embed_scale=float((d.get("embedding") or {}).get("scale", 1.0)), logit_scale=float(d.get("logit_scale", 1.0)),
                       tied_head=True, weight_format="dense")


# ----------------------------------------------------------------------------- layout
def _f32(t):
    return t.float().contiguous()


def _gqa_rows(m: Dict[str, torch.Tensor], c: PagedGqaConfig):
    """Projection rows of the heads: [q | k | v], or q alone."""
    Dp, Vp = pad(c.head_dim, 16), pad(c.v_dim, 16)
    own = () if c.kv_from is not None else (("k", c.n_kv_heads, Dp), ("v", c.n_kv_heads, Vp))
    return [pad_head_rows(m[s], n, d) for s, n, d in (("q", c.n_heads, Dp), *own)]


def _prepare_mixer(m: Dict[str, torch.Tensor], spec: LayerSpec, dtype) -> dict:
    wd = lambda t: t.to(dtype).contiguous()
    c = spec.mixer
    if spec.kind == "gqa":
        w = {"qkv": wd(torch.cat(_gqa_rows(m, c) + [stack_rows([m["g"]])])), "q_norm": _f32(m["q.norm"]), "sink": _f32(m["sink"]),
             "o": wd(pad_head_cols(m["o"], c.n_heads, pad(c.v_dim, 16)))}
        return w if c.kv_from is not None else dict(w, k_norm=_f32(m["k.norm"]))
    le, ri = ({k[len(s):]: t for k, t in m.items() if k.startswith(s)} for s in ("left.", "right."))
    g = c.right
    g.decay_rank = ri["a1"].shape[0]
    n8 = pad(g.n_heads * g.v_dim, 8)
    return {"in": wd(torch.cat(_gqa_rows(le, c.left) + [stack_rows([ri[s]]) for s in ("q", "k", "v", "g", "a1")])),
            "q_norm": _f32(le["q.norm"]), "k_norm": _f32(le["k.norm"]), "a2": wd(pad_cols(ri["a2"], pad(g.decay_rank, 8))),
            "a2_b": _f32(ri["a2.b"]), "norm": _f32(ri["norm"].float().repeat(g.n_heads) * c.right_scale),
            "out": wd(torch.cat((pad_head_cols(le["o"], c.left.n_heads, pad(c.left.v_dim, 16)), pad_cols(ri["o"], n8)), 1))}


def prepare_layer(raw: Dict[str, torch.Tensor], spec: LayerSpec, dtype) -> dict:
    """`raw`: this layer's tensors by their names behind the layer prefix, on the target device."""
    wd = lambda t: t.to(dtype).contiguous()
    f = {k[4:]: t for k, t in raw.items() if k.startswith("mlp.")}
    e = spec.moe
    w = {"type": spec.kind, "mix_norm": _f32(raw["norm1"]), "mlp": {},
         "mix": _prepare_mixer({k[4:]: t for k, t in raw.items() if k.startswith("mix.")}, spec, dtype)}
    gu = lambda k: stack_rows([f[k + "gate"], f[k + "up"]], WIDE)
    down = lambda k: pad_cols(f[k + "down"], pad(f[k + "down"].shape[1], WIDE))
    if spec.ffn or e is not None:
        w["post_norm"] = _f32(raw["norm2"])
    if spec.ffn:
        w["mlp"] = {"dense_gu": wd(gu("")), "dense_down": wd(down(""))}
    elif e is not None:
        names = [f"e{j}." for j in range(e.n_experts)]
        w["mlp"] = {"gate": wd(f["router"]), "w_gu": wd(torch.stack([gu(k) for k in names])), "w_down": wd(torch.stack([down(k) for k in names]))}
        if e.n_shared:
            w["mlp"].update(s_gu=wd(gu("shared.")), s_down=wd(down("shared.")))
    return w


def _gqa_tensors(c: PagedGqaConfig, N: int, p: str) -> Dict[str, tuple]:
    nq, nk, nv = c.n_heads * c.head_dim, c.n_kv_heads * c.head_dim, c.n_kv_heads * c.v_dim
    t = {p + "q": (nq, N), p + "q.norm": (c.head_dim,), p + "o": (N, c.n_heads * c.v_dim)}
    if c.kv_from is None:
        t.update({p + "k": (nk, N), p + "v": (nv, N), p + "k.norm": (c.head_dim,)})
    if c.gated:
        t.update({p + "sink": (c.n_heads,), p + "g": (c.n_heads, N)})
    return t


def layer_tensors(cfg: ModelConfig, spec: LayerSpec) -> Dict[str, tuple]:
    """Names and shapes of one layer's tensors behind the layer prefix (None: the tensor decides)."""
    c, e, N = spec.mixer, spec.moe, cfg.hidden
    t = {"norm1": (N,)}
    if spec.kind == "gqa":
        t.update(_gqa_tensors(c, N, "mix."))
    else:
        g, p = c.right, "mix.right."
        nk, nv, r = g.n_heads * g.head_dim, g.n_heads * g.v_dim, g.decay_rank or None
        t.update(_gqa_tensors(c.left, N, "mix.left."))
        t.update({p + "q": (nk, N), p + "k": (nk, N), p + "v": (nv, N), p + "g": (nv, N), p + "o": (N, nv), p + "norm": (g.v_dim,),
                  p + "a1": (r, N), p + "a2": (nk, r), p + "a2.b": (nk,)})
    if spec.ffn or e is not None:
        t["norm2"] = (N,)
    ffs = [("", spec.ffn)] if spec.ffn else []
    if e is not None:
        t["mlp.router"] = (e.n_experts, N)
        ffs = [(f"e{j}.", e.ffn) for j in range(e.n_experts)] + ([("shared.", e.shared_ffn)] if e.n_shared else [])
    for k, n in ffs:
        t.update({f"mlp.{k}gate": (n, N), f"mlp.{k}up": (n, N), f"mlp.{k}down": (N, n)})
    return t


def _assemble(cfg: ModelConfig, get, layer, dtype) -> dict:
    embed = get("embed", (cfg.vocab, cfg.hidden)).to(dtype).contiguous()
    return {"embed": embed, "lm_head": embed, "final_norm": _f32(get("final.norm", (cfg.hidden,)).float() * cfg.logit_scale),
            "layers": [prepare_layer(layer(i, s), s, dtype) for i, s in enumerate(cfg.layer_specs)]}


def from_tensors(cfg: ModelConfig, tensors: Dict[str, torch.Tensor], device="cpu", dtype=torch.float32) -> dict:
    """Runner weights from a flat dict of checkpoint tensors (validated against the configuration)."""
    get = taker(tensors, device)
    return _assemble(cfg, get, lambda i, spec: {k: get(f"l{i}.{k}", s) for k, s in layer_tensors(cfg, spec).items()}, dtype)


def load_weights(directory: str, cfg: ModelConfig, device="cpu", dtype=torch.bfloat16) -> dict:
    from .checkpoint import mapped_tensors
    return from_tensors(cfg, mapped_tensors(os.path.join(directory, "model.safetensors")), device, dtype)


def random_weights(cfg: ModelConfig, device="cpu", seed: int = 0, dtype=torch.bfloat16) -> dict:
    """Random weights of the configured sizes, generated on `device` layer by layer."""
    g = torch.Generator(device=device)
    g.manual_seed(seed)
    rnd = lambda *s: torch.randn(*s, device=device, generator=g)

    def tensor(name, shape):
        if name.endswith("a2.b"):
            return rnd(*shape) + 2.0
        if name.endswith("sink"):
            return rnd(*shape)
        if len(shape) == 1:
            return 1 + 0.1 * rnd(*shape)
        return (rnd(*shape) * shape[1] ** -0.5).to(torch.bfloat16)

    def layer(i, spec):
        if spec.kind == "side_by_side":
            spec.mixer.right.decay_rank = spec.mixer.right.decay_rank or 16
        return {k: tensor(k, s) for k, s in layer_tensors(cfg, spec).items()}
    return _assemble(cfg, tensor, layer, dtype)
