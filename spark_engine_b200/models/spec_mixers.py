"""Mixers of models whose layers carry their own sizes (`ModelConfig.layer_specs`), by the kind of a layer's spec."""
from __future__ import annotations

from .paged_gqa import PagedGqaMixer
from .parallel_mixers import LatentMixer, LightningMixer, WkvMixer
from .side_by_side import SideBySideMixer


def build_spec_mixer(cfg, spec, w: dict, n_slots: int, n_pages: int, page: int, pages, device, dtype, before=()):
    """`before`: the mixers of the layer runs so far (a layer may use the cache of an earlier one)."""
    if spec.kind == "lightning":
        return LightningMixer(cfg, spec, w, n_slots, device, dtype)
    if spec.kind == "wkv":
        return WkvMixer(cfg, spec, w, n_slots, device, dtype)
    if spec.kind == "latent":
        return LatentMixer(cfg, spec, w, n_pages, page, pages, device, dtype)
    if spec.kind == "gqa":
        src = spec.mixer.kv_from
        return PagedGqaMixer(cfg, spec.mixer, w, n_slots, n_pages, page, pages, device, dtype, None if src is None else before[src])
    if spec.kind == "side_by_side":
        return SideBySideMixer(cfg, spec, w, n_slots, n_pages, page, pages, device, dtype)
    raise ValueError(spec.kind)
