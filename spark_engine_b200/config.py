"""Typed configuration: model hyper-parameters and engine switches.

One `ModelConfig` describes every architecture the engine serves; the layer *types*
select the code path (gated-DeltaNet, KDA, softmax/sparse GQA, MLA+indexer, compressed
sparse attention), the dimensions come from the config.  The reference reads model
hyper-parameters from `config.json` (engine-rs/src/config.rs, engine-rs/src/ds41/cfg.rs:7-76)
and spreads ~900 environment switches over the code (docs/configuration.md:3-9); here a
single `EngineConfig` carries the small set of switches that matter, with `SPARK_*`
environment fallbacks and `--flag` overrides.
"""
from __future__ import annotations

import dataclasses
import json
import os
from dataclasses import dataclass, field
from typing import List, Optional


@dataclass
class AttnConfig:
    n_q_heads: int = 4
    n_kv_heads: int = 2
    head_dim: int = 64
    rope_dim: int = 64            # NeoX rotary on the first rope_dim dims (partial when < head_dim)
    rope_theta: float = 1e4
    yarn_factor: float = 1.0      # >1: YaRN scaling beyond yarn_orig_len
    yarn_orig_len: int = 262144
    qk_norm: bool = False         # Gemma-style (1+w) RMS norm on q and k
    gated: bool = False           # per-head sigmoid output gate (q projection is 2x wide)
    sparse_topk_blocks: int = 0   # 0 = dense; else top-k blocks of `block` tokens (+ tail)
    block: int = 4
    idx_heads: int = 4
    idx_dim: int = 128


@dataclass
class GdnConfig:
    n_k_heads: int = 4
    n_v_heads: int = 4
    head_dim: int = 64
    conv_k: int = 4


@dataclass
class KdaConfig:
    n_heads: int = 4
    head_dim: int = 64
    conv_k: int = 4
    gate_rank: int = 32           # low-rank f_a/f_b and g_a/g_b projections


@dataclass
class MlaConfig:
    n_heads: int = 4
    q_lora: int = 96
    kv_lora: int = 64
    head_dim: int = 32            # dk = dv (no-rope part)
    rope_dim: int = 0             # 0: GLM-style MLA without RoPE; >0: DeepSeek-style rope part
    rope_theta: float = 1e4
    # indexer (DSA)
    idx_heads: int = 4
    idx_dim: int = 32
    pool: int = 4
    topk_pools: int = 512
    sink: bool = False            # attention sink logit in the denominator (DS-style)
    window: int = 0               # sliding window (DS-style compressed sparse attention)
    compress: int = 0             # compression ratio of the global KV (0 = none)


@dataclass
class MoeConfig:
    n_experts: int = 16
    top_k: int = 4
    ffn: int = 128
    n_shared: int = 1
    shared_ffn: int = 0           # 0 -> ffn * n_shared
    router: str = "softmax"       # softmax | sigmoid_bias | sqrt_softplus | softmax_bias (bias: added to the choice scores only)
                                  # | sigmoid (the chosen scores are the weights as they are, times route_scale)
                                  # | topk_softmax (bias added to the logits, softmax over the chosen logits alone)
    route_scale: float = 1.0
    shared_gate: bool = False     # sigmoid(x . w_sg) on the shared expert
    swiglu_limit: float = 0.0     # clamp-SwiGLU limit (0 = off): gate at most the limit, up within +- the limit
    glu_alpha: float = 1.0        # the gate is gate * sigmoid(glu_alpha * gate)
    glu_shift: float = 0.0        # added to the (clamped) up half
    dense_layers: int = 0         # first N layers use a dense MLP of width dense_ffn
    dense_ffn: int = 0
    act: str = "swiglu"           # swiglu (gate and up matrices) | relu2 (squared relu of a single up matrix)
    n_identity: int = 0           # router outputs behind the experts' whose "expert" returns its input
    weight_input: bool = False    # an expert sees its input times the weight (its output is added as it is)

    @property
    def n_routes(self) -> int:
        return self.n_experts + self.n_identity

    @property
    def glu(self) -> tuple:
        """(limit, alpha, shift) of the gated activation."""
        return self.swiglu_limit, self.glu_alpha, self.glu_shift

    @property
    def plain(self) -> bool:
        """A router and experts that the quantised and expert-parallel paths know."""
        return self.act == "swiglu" and not self.weight_input and self.router != "topk_softmax" and self.glu[1:] == (1.0, 0.0)


@dataclass
class LightningConfig:
    """Linear attention with one constant decay per head (no softmax, no delta rule)."""
    n_heads: int = 2
    head_dim: int = 32
    v_dim: int = 32
    decay: List[float] = field(default_factory=lambda: [0.9, 0.99])


@dataclass
class WkvConfig:
    """Token-shifted recurrence with a learned decay per token and key channel and a bonus for the current token."""
    n_heads: int = 2
    head_dim: int = 32
    decay_rank: int = 16


@dataclass
class LatentConfig:
    """Dense causal attention over cached latents: low-rank or direct queries, one shared rotated key part (or none), optionally a
    learned sink per head in the denominator, an output gate per head or per element."""
    n_heads: int = 2
    head_dim: int = 32            # unrotated query / key dimensions per head
    v_dim: int = 32
    q_rank: int = 64              # 0: queries are projected from the row itself
    kv_rank: int = 48
    rope_dim: int = 16            # 0: no rotated part
    rope_theta: float = 1e4
    rope_interleaved: bool = True
    scale: float = 0.125
    sink: bool = False            # a score per head without key and value
    gate: str = "head"            # sigmoid gate per head | element (of the concatenated heads)


@dataclass
class PagedGqaConfig:
    """Grouped-query softmax attention over a paged cache.  Before the cache: short convolutions on q, k and v, or a norm per
    query / key head, a rotation and a temperature of the queries.  Scores: soft cap, a learned bias per distance bucket and
    head or a slope per head, chunked or windowed visibility, a sink in the denominator; a gate per head behind them."""
    n_heads: int = 4
    n_kv_heads: int = 2
    head_dim: int = 32
    v_dim: int = 32
    conv_k: int = 4               # taps of the causal convolutions (1: the current token only; 0: none)
    scale: float = 0.125
    softcap: float = 0.0          # 0: none
    bias_buckets: int = 32        # rows of the bias table (without one: unused)
    bias_max: int = 1024          # distance from which on the last row is used
    chunk: int = 0                # tokens see their own aligned chunk of the sequence (0: everything before them)
    window: int = 0               # tokens see themselves and the window - 1 before them (0: everything before them)
    qk_norm: bool = False         # RMS norm of every query and key head (weight per dimension, shared by the heads)
    rope_dims: int = 0            # leading dimensions of a head that rotate, adjacent pairs (0: none)
    rope_theta: float = 1e4
    rope_factor: float = 1.0      # every frequency is divided by it
    temp_coef: float = 0.0        # queries at position p times 1 + temp_coef * ln(floor((p + 1) / temp_every) + 1)
    temp_every: float = 1.0
    slopes: bool = False          # scores minus 2^(-8 (h + 1) / heads) times the distance
    gated: bool = False           # one sigmoid gate per head
    kv_from: Optional[int] = None  # keys and values are the ones in that layer's cache


@dataclass
class GlaConfig:
    """Linear attention with a decay per token and key channel, sigmoid(low-rank projection + bias)^(1 / tau); an RMS norm per
    head and a silu gate behind it."""
    n_heads: int = 2
    head_dim: int = 32
    v_dim: int = 32
    tau: float = 8.0
    decay_rank: int = 16


@dataclass
class SideBySideConfig:
    """Grouped-query attention and linear attention on the same rows, outputs scaled and added."""
    left: PagedGqaConfig = field(default_factory=lambda: PagedGqaConfig(conv_k=0))
    right: GlaConfig = field(default_factory=GlaConfig)
    left_scale: float = 1.0
    right_scale: float = 1.0

    def __post_init__(self):
        if isinstance(self.left, dict):
            self.left = PagedGqaConfig(**self.left)
        if isinstance(self.right, dict):
            self.right = GlaConfig(**self.right)


MIXER_CONFIGS = {"lightning": LightningConfig, "wkv": WkvConfig, "latent": LatentConfig, "gqa": PagedGqaConfig,
                 "side_by_side": SideBySideConfig}


@dataclass
class LayerSpec:
    """One layer of a model whose layers carry their own sizes."""
    kind: str = "lightning"       # key of MIXER_CONFIGS
    mixer: object = None
    ffn: int = 0                  # width of the dense feed-forward (0 = none)
    moe: Optional[MoeConfig] = None   # experts instead of the dense feed-forward


@dataclass
class LoopConfig:
    """Layers start .. stop-1 run `times` times in a row with the same weights, every pass with its own cache / state."""
    start: int = 0
    stop: int = 0
    times: int = 1


@dataclass
class ModelConfig:
    name: str = "tiny-hybrid"
    family: str = "hybrid"        # hybrid (Qwen-style) | glm | ds4 | vabunex | debisun | zapolorn | zakusun
    n_layers: int = 4
    layer_types: List[str] = field(default_factory=lambda: ["gdn", "gdn", "gdn", "attn"])
    hidden: int = 256
    vocab: int = 4096
    norm_eps: float = 1e-6
    attn: AttnConfig = field(default_factory=AttnConfig)
    gdn: GdnConfig = field(default_factory=GdnConfig)
    kda: KdaConfig = field(default_factory=KdaConfig)
    mla: MlaConfig = field(default_factory=MlaConfig)
    moe: MoeConfig = field(default_factory=MoeConfig)
    hc_streams: int = 1           # 1 = plain residual; 4 = hyper-connections (gated HC / mHC)
    hc_kind: str = "none"         # none | gated | mhc
    hc_rank: int = 32
    sinkhorn_iters: int = 20
    mtp_layers: int = 0           # MTP draft layers (chain drafter)
    mtp_depth: int = 3
    ngram_layers: List[int] = field(default_factory=list)   # layers with hashed n-gram embeddings
    ngram_rows: int = 0
    ngram_dim: int = 0
    ngram_heads: int = 16
    weight_format: str = "dense"  # dense | exl3 | mx (MXFP4 experts + FP8 dense)
    exl3_bits: int = 4
    kv_dtype: str = "bf16"        # bf16 | fp8
    kv_quant_on_cpu: bool = False  # the CPU runner keeps fp32 caches; set to model the packed FP8 latent rows there too

    layer_specs: List[LayerSpec] = field(default_factory=list)   # per-layer sizes; else the shared configs above
    loop: Optional[LoopConfig] = None
    block: str = "parallel"       # models with layer_specs: parallel (one norm, mixer + feed-forward) | sequential (pre-norm each)
                                  # | post (sublayers read the residual itself, their outputs are normed)
    norm_kind: str = "rms"        # models with layer_specs: rms | layer (weight and bias)
    norm_one_plus: bool = False   # norm weights are stored around zero
    norm_groups: int = 1          # equal parts of the row that are RMS-normed each on its own
    input_conv: int = 0           # taps of the causal convolution added to every sublayer's normed input (0: none; sequential blocks)
    depth_average: bool = False   # behind every layer the residual becomes a learned sum of the embedding and all layers' results
    positions: str = ""           # sinusoidal: added to the embedding ("": nothing is)
    embed_scale: float = 1.0
    logit_scale: float = 1.0
    tied_head: bool = False       # the logits' matrix is the embedding table (without its scale)
    side_dim: int = 0             # width of the per-layer token input (0 = none)

    def layer_runs(self) -> List[int]:
        """Weight layer of every layer run, in order."""
        lp = self.loop
        if lp is None:
            return list(range(self.n_layers))
        return [*range(lp.start), *(list(range(lp.start, lp.stop)) * lp.times), *range(lp.stop, self.n_layers)]

    def to_json(self) -> str:
        return json.dumps(dataclasses.asdict(self), indent=1)

    @staticmethod
    def from_dict(d: dict) -> "ModelConfig":
        d = dict(d)
        for key, cls in (("attn", AttnConfig), ("gdn", GdnConfig), ("kda", KdaConfig),
                         ("mla", MlaConfig), ("moe", MoeConfig)):
            if key in d and isinstance(d[key], dict):
                d[key] = cls(**d[key])
        if isinstance(d.get("loop"), dict):
            d["loop"] = LoopConfig(**d["loop"])
        moe = lambda m: MoeConfig(**m) if isinstance(m, dict) else m
        d["layer_specs"] = [x if isinstance(x, LayerSpec) else
                            LayerSpec(x["kind"], MIXER_CONFIGS[x["kind"]](**x["mixer"]), x["ffn"], moe(x.get("moe")))
                            for x in d.get("layer_specs", [])]
        return ModelConfig(**d)

    @staticmethod
    def from_json(path: str) -> "ModelConfig":
        with open(path) as f:
            d = json.load(f)
        if "architecture" in d:                 # a checkpoint's own configuration: the registry reads it
            from .models.registry import architecture
            return architecture(d).read_config(d)
        return ModelConfig.from_dict(d)


def _pattern(n_layers: int, period: int, a: str, b: str) -> List[str]:
    """`period-1` layers of kind `a`, then one of kind `b`, repeated."""
    return [b if (i + 1) % period == 0 else a for i in range(n_layers)]


def tiny_hybrid() -> ModelConfig:
    """Plumbing model: 3 gated-DeltaNet layers then 1 softmax GQA layer, 16-expert MoE."""
    return ModelConfig()


def qwen3next_style(n_layers: int = 48, weight_format: str = "exl3", kv_dtype: str = "bf16") -> ModelConfig:
    """Qwen3-Next-style hybrid: every 4th layer gated sparse GQA, the rest gated-DeltaNet;
    512 experts top-10 + shared; one MTP draft layer with chain depth 3."""
    return ModelConfig(
        name="qwen3next-style", family="hybrid", n_layers=n_layers,
        layer_types=_pattern(n_layers, 4, "gdn", "attn"), hidden=2048, vocab=151936,
        attn=AttnConfig(n_q_heads=16, n_kv_heads=2, head_dim=256, rope_dim=64, rope_theta=1e7,
                        yarn_factor=4.0, qk_norm=True, gated=True, sparse_topk_blocks=512, block=4,
                        idx_heads=4, idx_dim=128),
        gdn=GdnConfig(n_k_heads=16, n_v_heads=32, head_dim=128, conv_k=4),
        moe=MoeConfig(n_experts=512, top_k=10, ffn=512, n_shared=1, router="softmax", shared_gate=True),
        mtp_layers=1, mtp_depth=3, weight_format=weight_format, exl3_bits=4, kv_dtype=kv_dtype)


def glm_style(n_layers: int = 45, weight_format: str = "exl3") -> ModelConfig:
    """GLM-style: 3 KDA linear-attention layers per MLA layer with a DSA top-2048 indexer;
    288 experts top-8 (sigmoid+bias router, x2.5, clamp-SwiGLU 10) + shared expert."""
    types = ["mla" if i % 4 == 3 else "kda" for i in range(n_layers)]
    return ModelConfig(
        name="glm-style", family="glm", n_layers=n_layers, layer_types=types, hidden=4096, vocab=154880,
        norm_eps=1e-5,
        kda=KdaConfig(n_heads=64, head_dim=128, conv_k=4, gate_rank=128),
        mla=MlaConfig(n_heads=64, q_lora=1536, kv_lora=512, head_dim=256, rope_dim=64, idx_heads=32,
                      idx_dim=128, pool=4, topk_pools=512),
        moe=MoeConfig(n_experts=288, top_k=8, ffn=1536, n_shared=1, router="sigmoid_bias", route_scale=2.5,
                      swiglu_limit=10.0, dense_layers=3, dense_ffn=12288),
        hc_streams=1, hc_kind="none", mtp_layers=2, mtp_depth=5, weight_format=weight_format)


def ds4_style(n_layers: int = 40, weight_format: str = "mx") -> ModelConfig:
    """DeepSeek-V4-style: compressed sparse MLA with hierarchical top-k indexer, 384 experts
    top-6 (MXFP4) + shared (FP8), hashed n-gram tables streamed from host, FP8 KV."""
    return ModelConfig(
        name="ds4-style", family="ds4", n_layers=n_layers, layer_types=["mla"] * n_layers, hidden=4096,
        vocab=129280,
        mla=MlaConfig(n_heads=64, q_lora=1536, kv_lora=512, head_dim=128, rope_dim=64, idx_heads=16, idx_dim=128,
                      pool=4, topk_pools=512, sink=True, window=128, compress=4),
        moe=MoeConfig(n_experts=384, top_k=6, ffn=2048, n_shared=1, router="sqrt_softplus", route_scale=1.5,
                      swiglu_limit=10.0),
        mtp_layers=1, mtp_depth=3, ngram_layers=[1, 14], ngram_rows=1 << 22, ngram_dim=1024,
        weight_format=weight_format, kv_dtype="fp8")


def vabunex_style(n_layers: int = 12, hidden: int = 2048, ffn: int = 5632, vocab: int = 65536) -> ModelConfig:
    """Vabunex at the layer sizes of a small real model: two lightning, one wkv and one latent-attention layer per period of
    four, the second period run twice."""
    kinds = [("lightning", "wkv", "lightning", "latent")[i % 4] for i in range(n_layers)]
    heads = hidden // 128
    mixers = {"latent": LatentConfig(n_heads=heads, head_dim=128, v_dim=128, q_rank=768, kv_rank=512, rope_dim=64,
                                     rope_theta=1e6, scale=192 ** -0.5),
              "lightning": LightningConfig(n_heads=heads, head_dim=128, v_dim=128,
                                           decay=[1.0 - 2.0 ** (-1 - 8 * h / heads) for h in range(heads)]),
              "wkv": WkvConfig(n_heads=hidden // 64, head_dim=64, decay_rank=64)}
    return ModelConfig(name="vabunex-style", family="vabunex", n_layers=n_layers, layer_types=kinds, hidden=hidden, vocab=vocab,
                       norm_eps=1e-5, layer_specs=[LayerSpec(k, dataclasses.replace(mixers[k]), ffn) for k in kinds],
                       loop=LoopConfig(min(4, n_layers), min(8, n_layers), 2), norm_one_plus=True, embed_scale=float(hidden) ** 0.5,
                       weight_format="dense")


def debisun_style(n_layers: int = 12, hidden: int = 2048, ffn: int = 8192, vocab: int = 65536, experts: int = 64, top: int = 4,
                  chunk: int = 2048) -> ModelConfig:
    """Debisun at the layer sizes of a small real model: a dense first layer, then experts (a quarter as wide, plus identity
    experts and a shared one), heads of 128 with four queries per key / value head."""
    heads = hidden // 128
    mixer = PagedGqaConfig(n_heads=heads, n_kv_heads=max(1, heads // 4), head_dim=128, v_dim=128, conv_k=4, scale=128 ** -0.5,
                           softcap=50.0, bias_buckets=32, bias_max=1024, chunk=chunk)
    moe = MoeConfig(n_experts=experts, n_identity=experts // 4, top_k=top, ffn=ffn // 4, n_shared=1, shared_ffn=ffn // 4,
                    router="softmax_bias", route_scale=1.5, shared_gate=True, act="relu2")
    specs = [LayerSpec("gqa", dataclasses.replace(mixer), 0 if i else ffn, dataclasses.replace(moe) if i else None)
             for i in range(n_layers)]
    return ModelConfig(name="debisun-style", family="debisun", n_layers=n_layers, layer_types=["gqa"] * n_layers, hidden=hidden,
                       vocab=vocab, norm_eps=1e-5, layer_specs=specs, block="sequential", norm_kind="layer", side_dim=hidden // 16,
                       weight_format="dense")


def zapolorn_style(n_layers: int = 12, hidden: int = 2048, ffn: int = 5632, vocab: int = 65536, experts: int = 64, top: int = 4,
                   window: int = 1024) -> ModelConfig:
    """Zapolorn at the layer sizes of a small real model, in periods of four: whole-context attention beside linear attention,
    window attention, window attention on the keys and values before it, window attention; dense and routed feed-forwards in
    turn; heads of 128 with four queries per key / value head."""
    heads = hidden // 128
    gqa = dict(n_heads=heads, n_kv_heads=max(1, heads // 4), head_dim=128, v_dim=128, conv_k=0, scale=128 ** -0.5, qk_norm=True)
    moe = MoeConfig(n_experts=experts, top_k=top, ffn=ffn // 4, n_shared=1, shared_ffn=ffn // 4, router="sigmoid", weight_input=True)
    specs = []
    for i in range(n_layers):
        if i % 4 == 0:
            left = PagedGqaConfig(**gqa, temp_coef=0.1, temp_every=8192, slopes=True)
            kind, mixer = "side_by_side", SideBySideConfig(left, GlaConfig(n_heads=heads, head_dim=64, v_dim=128, tau=8.0), 0.7, 0.7)
        else:
            kind, mixer = "gqa", PagedGqaConfig(**gqa, window=window, rope_dims=128, rope_theta=1e6, rope_factor=8.0, gated=True,
                                                kv_from=i - 1 if i % 4 == 2 else None)
        specs.append(LayerSpec(kind, mixer, 0 if i % 2 else ffn, dataclasses.replace(moe) if i % 2 else None))
    return ModelConfig(name="zapolorn-style", family="zapolorn", n_layers=n_layers, layer_types=[x.kind for x in specs], hidden=hidden,
                       vocab=vocab, norm_eps=1e-5, layer_specs=specs, block="post", embed_scale=float(hidden) ** 0.5, tied_head=True,
                       weight_format="dense")


def zakusun_style(n_layers: int = 12, hidden: int = 2048, ffn: int = 1536, vocab: int = 65536, experts: int = 64, top: int = 4,
                  taps: int = 4) -> ModelConfig:
    """Zakusun at the layer sizes of a small real model: latent attention (heads of 128, latents of 512), experts of width `ffn`,
    two norm groups."""
    heads = hidden // 128
    mixer = LatentConfig(n_heads=heads, head_dim=128, v_dim=128, q_rank=0, kv_rank=512, rope_dim=0, scale=128 ** -0.5, sink=True, gate="element")
    moe = MoeConfig(n_experts=experts, top_k=top, ffn=ffn, n_shared=0, router="topk_softmax", swiglu_limit=7.0, glu_alpha=1.702, glu_shift=1.0)
    specs = [LayerSpec("latent", dataclasses.replace(mixer), 0, dataclasses.replace(moe)) for _ in range(n_layers)]
    return ModelConfig(name="zakusun-style", family="zakusun", n_layers=n_layers, layer_types=["latent"] * n_layers, hidden=hidden, vocab=vocab,
                       norm_eps=1e-5, layer_specs=specs, block="sequential", norm_groups=2, input_conv=taps, depth_average=True,
                       positions="sinusoidal", tied_head=True, weight_format="dense")


def scaled_down(cfg: ModelConfig, hidden: int = 256, n_layers: int = 4, vocab: int = 1024) -> ModelConfig:
    """Same layer types, small dimensions: the CPU test shape of a large config."""
    c = dataclasses.replace(cfg)
    per = 4
    c.n_layers = n_layers
    c.layer_types = [cfg.layer_types[i % max(per, 1)] if i < len(cfg.layer_types) else cfg.layer_types[-1]
                     for i in range(n_layers)]
    c.hidden, c.vocab = hidden, vocab
    c.attn = dataclasses.replace(cfg.attn, n_q_heads=4, n_kv_heads=2, head_dim=64,
                                 rope_dim=min(cfg.attn.rope_dim, 32), idx_heads=2, idx_dim=32,
                                 sparse_topk_blocks=min(cfg.attn.sparse_topk_blocks, 8))
    c.gdn = dataclasses.replace(cfg.gdn, n_k_heads=2, n_v_heads=4, head_dim=32)
    c.kda = dataclasses.replace(cfg.kda, n_heads=4, head_dim=32, gate_rank=16)
    c.mla = dataclasses.replace(cfg.mla, n_heads=4, q_lora=64, kv_lora=32, head_dim=32,
                                rope_dim=16 if cfg.mla.rope_dim else 0, idx_heads=2, idx_dim=16,
                                topk_pools=min(cfg.mla.topk_pools, 8),
                                window=min(cfg.mla.window, 16))
    c.moe = dataclasses.replace(cfg.moe, n_experts=16, top_k=min(cfg.moe.top_k, 4), ffn=128,
                                dense_layers=min(cfg.moe.dense_layers, 1), dense_ffn=256 if cfg.moe.dense_layers else 0)
    c.ngram_layers = [i for i in cfg.ngram_layers if i < n_layers]
    c.ngram_rows = 4096 if cfg.ngram_rows else 0
    c.ngram_dim = 64 if cfg.ngram_dim else 0
    c.weight_format = "dense"
    c.name = cfg.name + "-small"
    return c


def _env(name: str, default, cast=str):
    v = os.environ.get("SPARK_" + name.upper())
    if v is None:
        return default
    if cast is bool:
        return v not in ("0", "false", "False", "")
    return cast(v)


@dataclass
class EngineConfig:
    """Engine switches (CLI `--flag`, JSON file, `SPARK_<NAME>` environment fallback)."""
    model: str = "tiny-hybrid"
    numerics: str = "deterministic"      # deterministic | fast (multimem hardware reductions)
    dtype: str = "bfloat16"              # activations and dense weights on the device: bfloat16 | float32 (models with layer_specs)
    tp: int = 1
    ep: int = 1
    max_seqs: int = 8
    max_rows: int = 64                   # rows per decode/verify forward
    prefill_chunk: int = 8192            # larger chunks amortise the one-off expert reconstruction (16K prompt: 14.7k tok/s at 4096, 17.1k at 8192)
    kv_tokens: int = 1 << 20             # KV budget in tokens
    kv_granule: int = 16384
    kv_backing: str = "dense"            # dense (one allocation of the whole budget) | vmm (address space reserved, backed on demand)
    cuda_graphs: bool = True
    spec: str = "mtp"                    # none | mtp | lookup | feature (tap-conditioned drafter) | stage (staged drafter)
    spec_depth: int = 3
    spec_policy: str = "theta"           # tau | theta | rate | cost
    spec_tree_widths: str = ""           # e.g. "3,2,1": verify a tree (widths per depth) built from the feature drafter's candidates
    comm: str = "fused"                  # fused (peer-memory kernels) | nccl (baseline)
    comm_wait_ms: float = 1000.0         # bound of every device-side wait
    step_deadline_s: float = 0.0         # > 0: a watchdog aborts the process when one engine step runs longer
    pcache_dir: Optional[str] = None
    pcache_bytes: int = 64 << 30
    host_mem_floor_gb: float = 2.0       # > 0: below this much available host memory the server sheds load
    meminfo_path: str = ""               # where the memory guard reads MemAvailable ("" = /proc/meminfo)
    socket: str = "/tmp/spark-b200.sock"
    host: str = "127.0.0.1"
    port: int = 8000
    profile: bool = False
    prewarm: bool = False         # run synthetic requests for 1..max_seqs streams before serving (captures the graphs)
    serve_log: bool = False       # one stderr line per admission / prefill forward / round ([serve-admit], [serve-round] ...)
    draft_trace: str = ""         # file ("-" = stderr) that gets one JSON line per speculative round
    nvtx: bool = False
    log_rounds: bool = False
    seed: int = 0

    @staticmethod
    def from_env(**over) -> "EngineConfig":
        c = EngineConfig()
        for f in dataclasses.fields(c):
            cur = getattr(c, f.name)
            cast = type(cur) if cur is not None else str
            setattr(c, f.name, _env(f.name, cur, cast))
        for k, v in over.items():
            if v is not None:
                setattr(c, k, v)
        return c

    def signature(self) -> str:
        """Flag signature: captured graphs are keyed on it so a changed switch forces a
        re-capture (reference: spec_probe.rs:316-327)."""
        keys = ("numerics", "dtype", "tp", "ep", "comm", "spec", "spec_depth", "cuda_graphs")
        return "|".join(f"{k}={getattr(self, k)}" for k in keys)


PRESETS = {
    "tiny-hybrid": tiny_hybrid,
    "qwen3next-style": qwen3next_style,
    "glm-style": glm_style,
    "ds4-style": ds4_style,
    "vabunex-style": vabunex_style,
    "debisun-style": debisun_style,
    "zapolorn-style": zapolorn_style,
    "zakusun-style": zakusun_style,
}


def get_model_config(name: str, **kw) -> ModelConfig:
    if name.endswith(".json"):
        return ModelConfig.from_json(name)
    return PRESETS[name](**kw)
