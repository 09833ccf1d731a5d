"""Model configurations: the hybrid (gated-GQA attention + Gated-DeltaNet) decoder, and the stream designs
(:class:`StreamDesign`: an fp32 residual stream, served in bf16 or fp32 on one GPU per process; no counterpart in the
reference): Zinutar (:class:`ZinutarConfig`, a looped decoder of parallel blocks), Fetotar (:class:`FetotarConfig`,
sandwich-normed layers of latent attention, Mamba-2 and mLSTM with a per-layer token input), Deluvik
(:class:`DeluvikConfig`, softmax attention with sinks, shared keys and short convolutions, a gated linear recurrence beside
windowed attention, mixtures of experts, norms on every branch's output) and Tobadra (:class:`TobadraConfig`, windowed attention
over turned values, lightning attention and a per-channel delta rule, grouped experts, gated branches).

One frozen dataclass describes every shape the kernels, the KV pools, the
tensor-parallel shard tables and the cost model derive from.  Layer kinds are
spelled out per layer (``"attn"`` / ``"gdn"``) rather than as an index set so a
checkpoint's ``layer_types`` list maps onto it one to one.

Parity: reference ``src/tilerl/config.py:11`` (``ModelConfig``), ``:114``
(``qwen38_27b``), ``:153`` (``tiny``).
"""
from __future__ import annotations

import json
import math
import os
from dataclasses import dataclass, replace
from importlib import import_module
from typing import Dict, Optional, Tuple

from .mixers import (MIXERS, BandScalingSpec, ChannelDeltaSpec, ClampedGluSpec, DenseSpec, GluSpec, LatentAttnSpec, LayerSpec, LightningSpec,
                     LruSpec, Mamba2Spec, MlstmSpec, MoeSpec, ParallelSpec, RotarySpec, RouterSpec, SoftmaxAttnSpec, YarnSpec, take)

ATTN = "attn"
GDN = "gdn"


@dataclass(frozen=True)
class ModelConfig:
    name: str
    hidden: int
    ffn: int
    vocab: int
    layer_types: Tuple[str, ...]
    # gated GQA attention
    n_q_heads: int
    n_kv_heads: int
    head_dim: int
    rotary_dim: int
    rope_theta: float
    attn_gated: bool = True
    # Gated DeltaNet
    gdn_k_heads: int = 0
    gdn_v_heads: int = 0
    gdn_head_dim: int = 0
    gdn_conv: int = 4
    # misc
    rms_eps: float = 1e-6
    max_ctx: int = 262144
    tie_embeddings: bool = False
    quant: str = "nvfp4"  # "nvfp4" | "fp8" | "bf16": format of the served linears
    lm_head_quant: str = "bf16"

    def __post_init__(self) -> None:
        object.__setattr__(self, "layer_types", tuple(self.layer_types))
        for t in self.layer_types:
            if t not in (ATTN, GDN):
                raise ValueError(f"unknown layer type {t!r}")
        if self.n_q_heads % self.n_kv_heads:
            raise ValueError("n_q_heads must be a multiple of n_kv_heads (GQA)")
        if self.rotary_dim % 2 or self.rotary_dim > self.head_dim:
            raise ValueError("rotary_dim must be even and <= head_dim")
        if self.n_gdn_layers:
            if self.gdn_k_heads <= 0 or self.gdn_v_heads <= 0 or self.gdn_head_dim <= 0:
                raise ValueError("GDN layers need gdn_k_heads/gdn_v_heads/gdn_head_dim")
            if self.gdn_v_heads % self.gdn_k_heads:
                raise ValueError("gdn_v_heads must be a multiple of gdn_k_heads")

    # ---- derived ---------------------------------------------------------
    @property
    def n_layers(self) -> int:
        return len(self.layer_types)

    @property
    def attn_layers(self) -> Tuple[int, ...]:
        return tuple(i for i, t in enumerate(self.layer_types) if t == ATTN)

    @property
    def gdn_layers(self) -> Tuple[int, ...]:
        return tuple(i for i, t in enumerate(self.layer_types) if t == GDN)

    @property
    def n_attn_layers(self) -> int:
        return len(self.attn_layers)

    @property
    def n_gdn_layers(self) -> int:
        return len(self.gdn_layers)

    @property
    def gqa_group(self) -> int:
        return self.n_q_heads // self.n_kv_heads

    @property
    def q_rows(self) -> int:
        """Rows of the q projection: per head [query(D); gate(D)] when gated."""
        return self.n_q_heads * self.head_dim * (2 if self.attn_gated else 1)

    @property
    def kv_rows(self) -> int:
        return self.n_kv_heads * self.head_dim

    @property
    def qkv_rows(self) -> int:
        return self.q_rows + 2 * self.kv_rows

    @property
    def attn_out_dim(self) -> int:
        return self.n_q_heads * self.head_dim

    @property
    def gdn_qk_dim(self) -> int:
        return self.gdn_k_heads * self.gdn_head_dim

    @property
    def gdn_v_dim(self) -> int:
        return self.gdn_v_heads * self.gdn_head_dim

    @property
    def gdn_conv_dim(self) -> int:
        """Channels that go through the depthwise conv: q, k, v."""
        return 2 * self.gdn_qk_dim + self.gdn_v_dim

    @property
    def gdn_in_rows(self) -> int:
        """Rows of the fused GDN input projection: [q; k; v; z; a; b]."""
        return self.gdn_conv_dim + self.gdn_v_dim + 2 * self.gdn_v_heads

    def attn_index(self, layer: int) -> int:
        return self.attn_layers.index(layer)

    def gdn_index(self, layer: int) -> int:
        return self.gdn_layers.index(layer)

    def n_params(self) -> int:
        h = self.hidden
        n = self.vocab * h * (1 if self.tie_embeddings else 2) + h
        for t in self.layer_types:
            n += 2 * h + 3 * h * self.ffn
            if t == ATTN:
                n += self.qkv_rows * h + h * self.attn_out_dim + 2 * self.head_dim
            else:
                n += self.gdn_in_rows * h + h * self.gdn_v_dim
                n += self.gdn_conv_dim * self.gdn_conv + 2 * self.gdn_v_heads + self.gdn_head_dim
        return n


def qwen38_27b() -> ModelConfig:
    """The 27B hybrid: 64 layers, every 4th (3, 7, ..., 63) gated GQA attention
    (24 q / 4 kv heads x 256, partial RoPE 64, theta 1e7), the rest Gated DeltaNet
    (16 key / 48 value heads x 128, conv width 4); SwiGLU FFN 17408; vocab 248320.
    Reference ``src/tilerl/config.py:114-140``."""
    types = tuple(ATTN if i % 4 == 3 else GDN for i in range(64))
    return ModelConfig(
        name="qwen38-27b", hidden=5120, ffn=17408, vocab=248320, layer_types=types,
        n_q_heads=24, n_kv_heads=4, head_dim=256, rotary_dim=64, rope_theta=1e7,
        gdn_k_heads=16, gdn_v_heads=48, gdn_head_dim=128, gdn_conv=4,
        rms_eps=1e-6, max_ctx=262144, tie_embeddings=False, quant="nvfp4",
    )


def qwen36_27b() -> ModelConfig:
    """Same shapes as :func:`qwen38_27b` (reference ``config.py:143``)."""
    return replace(qwen38_27b(), name="qwen36-27b")


def tiny_hybrid() -> ModelConfig:
    """Two-layer CPU gate model: layer 0 GDN (4 heads x 64, conv 4), layer 1
    gated GQA (4 q / 2 kv heads x 64, theta 1e6), d_model 256, FFN 768,
    vocab 1024, eps 1e-6."""
    return ModelConfig(
        name="tiny-hybrid", hidden=256, ffn=768, vocab=1024, layer_types=(GDN, ATTN),
        n_q_heads=4, n_kv_heads=2, head_dim=64, rotary_dim=64, rope_theta=1e6,
        gdn_k_heads=4, gdn_v_heads=4, gdn_head_dim=64, gdn_conv=4,
        rms_eps=1e-6, max_ctx=4096, tie_embeddings=False, quant="nvfp4",
    )


def tiny(max_ctx: int = 512) -> ModelConfig:
    """Smallest smoke model (attention layer first, then GDN), tied embeddings,
    byte vocabulary of 320.  Reference ``config.py:153``."""
    return ModelConfig(
        name="tiny" if max_ctx == 512 else "tiny-agent",
        hidden=64, ffn=128, vocab=320, layer_types=(ATTN, GDN),
        n_q_heads=4, n_kv_heads=2, head_dim=16, rotary_dim=16, rope_theta=1e7,
        gdn_k_heads=2, gdn_v_heads=2, gdn_head_dim=16, gdn_conv=4,
        rms_eps=1e-6, max_ctx=max_ctx, tie_embeddings=True, quant="bf16",
    )


def small_gpu() -> ModelConfig:
    """A 4-layer model with the 27B's head geometry (D=256, GDN 128) but narrow
    width; used by GPU kernel/engine tests and profiler captures so every kernel
    template instantiated for the 27B is exercised on a few hundred MB."""
    types = (GDN, GDN, GDN, ATTN)
    return ModelConfig(
        name="small-gpu", hidden=1024, ffn=3072, vocab=32768, layer_types=types,
        n_q_heads=8, n_kv_heads=2, head_dim=256, rotary_dim=64, rope_theta=1e7,
        gdn_k_heads=4, gdn_v_heads=8, gdn_head_dim=128, gdn_conv=4,
        rms_eps=1e-6, max_ctx=65536, tie_embeddings=False, quant="nvfp4",
    )


def small_gpu_tp() -> ModelConfig:
    """:func:`small_gpu` with head counts and widths that divide 2, 4 and 8 ways (8 q / 2 kv
    heads -- kv heads replicated from 4 ranks on, as the 27B's 4 kv heads are at 8 --, 8 key /
    16 value GDN heads, FFN 4096): the model of the tensor-parallel GPU gates."""
    types = (GDN, GDN, GDN, ATTN)
    return ModelConfig(
        name="small-gpu-tp", hidden=1024, ffn=4096, vocab=32768, layer_types=types,
        n_q_heads=8, n_kv_heads=2, head_dim=256, rotary_dim=64, rope_theta=1e7,
        gdn_k_heads=8, gdn_v_heads=16, gdn_head_dim=128, gdn_conv=4,
        rms_eps=1e-6, max_ctx=65536, tie_embeddings=False, quant="nvfp4",
    )


# ---- stream designs ----------------------------------------------------------------------------------
class StreamDesign:
    """What designs with an fp32 residual stream have in common: their ``config.json`` spells every size out, weights
    are served in bf16 (or fp32), one process serves one GPU, and they are not trained here."""
    architecture = ""
    tie_embeddings = False
    quant = "bf16"
    lm_head_quant = "bf16"
    # no Gated-DeltaNet layers: recurrent state, where a design has any, lives in a RecurrentPool
    n_gdn_layers = 0
    gdn_k_heads = gdn_v_heads = gdn_head_dim = gdn_conv_dim = 0

    @classmethod
    def from_dir(cls, j: Dict, path: str, name: str):
        """The configuration of a checkpoint directory whose ``config.json`` is ``j``."""
        return cls.from_json(j, name=name)

    @property
    def layout(self):
        """The module with the shapes and memory layout of the design's parameters."""
        return import_module(f"..{self.architecture.lower()}_layout", __name__)


# ---- Zinutar: looped parallel-block decoder with sigmoid-weighted attention ------------------------
@dataclass(frozen=True)
class AttnSpec:
    """One attention mixer without softmax: ``heads`` query heads over ``kv_heads`` key / value heads
    (contiguous groups), query / key width ``dim``, value width ``vdim``, score factor ``scale``."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float

    def __post_init__(self) -> None:
        if min(self.heads, self.kv_heads, self.dim, self.vdim) <= 0 or self.heads % self.kv_heads:
            raise ValueError(f"attention needs positive sizes and heads a multiple of kv_heads: {self}")

    @property
    def group(self) -> int:
        return self.heads // self.kv_heads


@dataclass(frozen=True)
class MlpSpec:
    """Feed-forward of width ``ff`` without a gate; ``kind`` names its form."""
    ff: int
    kind: str = "dense"

    def __post_init__(self) -> None:
        if self.kind != "dense":
            raise ValueError(f"unknown feed-forward kind {self.kind!r}")
        if self.ff <= 0:
            raise ValueError("feed-forward width must be positive")


@dataclass(frozen=True)
class BlockSpec:
    """One layer: an attention mixer and an optional feed-forward, both reading the same normed input."""
    mixer: AttnSpec
    mlp: Optional[MlpSpec] = None


@dataclass(frozen=True)
class LoopSpec:
    """Layers ``start .. stop-1`` run ``times`` times in a row with shared weights."""
    start: int
    stop: int
    times: int


@dataclass(frozen=True)
class LayerRun:
    """One execution of a layer: ``layer`` names its weights, ``kv`` its own cache, ``inject`` whether the
    embedding output is added to the stream right before it."""
    layer: int
    kv: int
    inject: bool = False


def _fields(d: Dict, known, where: str) -> None:
    extra = sorted(set(d) - set(known))
    if extra:
        raise ValueError(f"{where}: unknown keys {extra}")


@dataclass(frozen=True)
class ZinutarConfig(StreamDesign):
    """Sizes and constants of a Zinutar model.  Every layer has its own mixer and feed-forward sizes;
    :attr:`runs` spells the executions out in order, one KV cache each."""
    name: str
    hidden: int
    vocab: int
    layers: Tuple[BlockSpec, ...]
    loop: Optional[LoopSpec] = None
    rms_eps: float = 1e-5
    max_ctx: int = 1 << 20

    architecture = "Zinutar"

    def __post_init__(self) -> None:
        object.__setattr__(self, "layers", tuple(self.layers))
        if self.hidden <= 0 or self.vocab <= 0 or not self.layers:
            raise ValueError("a model needs a positive width and vocabulary and at least one layer")
        lo = self.loop
        if lo is not None and not (0 <= lo.start < lo.stop <= len(self.layers) and lo.times >= 1):
            raise ValueError(f"loop {lo} does not fit {len(self.layers)} layers")

    @property
    def runs(self) -> Tuple[LayerRun, ...]:
        lo, n = self.loop or LoopSpec(0, 1, 1), len(self.layers)
        order = [(i, False) for i in range(lo.start)]
        for t in range(lo.times):
            order += [(i, t > 0 and i == lo.start) for i in range(lo.start, lo.stop)]
        order += [(i, False) for i in range(lo.stop, n)]
        return tuple(LayerRun(i, kv, inj) for kv, (i, inj) in enumerate(order))

    @property
    def n_layers(self) -> int:
        return len(self.layers)

    @property
    def n_attn_layers(self) -> int:
        """KV caches a sequence holds: one per execution of an attention layer."""
        return len(self.runs)

    @property
    def n_q_heads(self) -> int:
        return max(b.mixer.heads for b in self.layers)

    @property
    def n_kv_heads(self) -> int:
        return max(b.mixer.kv_heads for b in self.layers)

    def n_params(self) -> int:
        h = self.hidden
        n = 2 * self.vocab * h + 2 * h
        for b in self.layers:
            a = b.mixer
            n += h + h * (a.heads + a.kv_heads) * a.dim + h * (a.kv_heads + a.heads) * a.vdim + a.heads
            if b.mlp is not None:
                n += 2 * h * b.mlp.ff + 4
        return n

    # ---- config.json -----------------------------------------------------------------------
    @classmethod
    def from_json(cls, j: Dict, name: str = "zinutar", max_ctx: Optional[int] = None) -> "ZinutarConfig":
        blocks = []
        for i, l in enumerate(j["layers"]):
            if l["type"] != "attention":
                raise ValueError(f"layer {i}: unknown mixer type {l['type']!r}")
            m, f = l["mixer"], l.get("mlp")
            _fields(m, ("heads", "kv_heads", "dim", "vdim", "scale"), f"layer {i} mixer")
            if f is not None:
                _fields(f, ("ff", "kind"), f"layer {i} mlp")
            blocks.append(BlockSpec(AttnSpec(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]),
                                             float(m["scale"])),
                                    None if f is None else MlpSpec(int(f["ff"]), f["kind"])))
        lo = j.get("loop")
        return cls(name=name, hidden=int(j["width"]), vocab=int(j["vocab"]), layers=tuple(blocks),
                   loop=None if lo is None else LoopSpec(int(lo["start"]), int(lo["stop"]), int(lo["times"])),
                   rms_eps=float(j["norm"]["eps"]), **({} if max_ctx is None else {"max_ctx": max_ctx}))

    def to_json(self) -> Dict:
        out: Dict = {"architecture": self.architecture, "width": self.hidden, "vocab": self.vocab,
                     "norm": {"eps": self.rms_eps}, "layers": []}
        for b in self.layers:
            a = b.mixer
            out["layers"].append({"type": "attention",
                                  "mixer": {"heads": a.heads, "kv_heads": a.kv_heads, "dim": a.dim, "vdim": a.vdim,
                                            "scale": a.scale},
                                  "mlp": None if b.mlp is None else {"kind": b.mlp.kind, "ff": b.mlp.ff}})
        if self.loop is not None:
            out["loop"] = {"start": self.loop.start, "stop": self.loop.stop, "times": self.loop.times}
        return out


def zinutar_uniform(name: str, *, hidden: int, vocab: int, n_layers: int, heads: int, kv_heads: int, dim: int, ff: int,
                    vdim: Optional[int] = None, loop: Optional[LoopSpec] = None, **kw) -> ZinutarConfig:
    """A Zinutar model whose layers all have one size, scores scaled by ``1 / sqrt(dim)``."""
    blk = BlockSpec(AttnSpec(heads, kv_heads, dim, vdim or dim, dim ** -0.5), MlpSpec(ff))
    return ZinutarConfig(name=name, hidden=hidden, vocab=vocab, layers=(blk,) * n_layers, loop=loop, **kw)


def zinutar_tiny() -> ZinutarConfig:
    """Smoke model: three layers of different sizes (one without a feed-forward), the first two looped
    twice, byte vocabulary of 320."""
    return ZinutarConfig(
        name="zinutar-tiny", hidden=72, vocab=320, rms_eps=1e-5, max_ctx=4096, loop=LoopSpec(0, 2, 2),
        layers=(BlockSpec(AttnSpec(6, 2, 24, 16, 0.3), MlpSpec(100)), BlockSpec(AttnSpec(4, 4, 16, 40, 0.2), None),
                BlockSpec(AttnSpec(5, 1, 32, 32, 0.25), MlpSpec(136))))


def zinutar_small() -> ZinutarConfig:
    """Four layers of a 1B-class width; profiler captures and GPU engine tests."""
    return zinutar_uniform("zinutar-small", hidden=2048, vocab=32768, n_layers=4, heads=16, kv_heads=4, dim=128, ff=8192,
                           loop=LoopSpec(1, 3, 2))


def zinutar_8b() -> ZinutarConfig:
    """Layers of an 8B-class dense decoder (width 4096, 16 query / 4 kv heads x 256, ff 14336), 32 of them."""
    return zinutar_uniform("zinutar-8b", hidden=4096, vocab=128256, n_layers=32, heads=16, kv_heads=4, dim=256, ff=14336)


# ---- Fetotar: sandwich-normed layers of three mixers, with a per-layer token input ---------------------
@dataclass(frozen=True)
class FetotarConfig(StreamDesign):
    """Sizes and constants of a Fetotar model.  Every layer has its own mixer and feed-forward; attention layers number
    the KV caches, recurrent layers the states, both in layer order."""
    name: str
    hidden: int
    vocab: int
    layers: Tuple[LayerSpec, ...]
    side_dim: int                   # width of a layer's share of the per-token side embedding
    embed_scale: float = 1.0
    norm_eps: float = 1e-6
    max_ctx: int = 1 << 20

    architecture = "Fetotar"

    def __post_init__(self) -> None:
        object.__setattr__(self, "layers", tuple(self.layers))
        if self.hidden <= 0 or self.vocab <= 0 or self.side_dim <= 0 or not self.layers:
            raise ValueError("a model needs positive sizes and at least one layer")

    @property
    def n_layers(self) -> int:
        return len(self.layers)

    @property
    def attn_mixers(self) -> Tuple[LatentAttnSpec, ...]:
        return tuple(l.mixer for l in self.layers if not l.mixer.recurrent)

    @property
    def recurrent_mixers(self) -> Tuple[object, ...]:
        return tuple(l.mixer for l in self.layers if l.mixer.recurrent)

    @property
    def n_attn_layers(self) -> int:
        return len(self.attn_mixers)

    @property
    def n_q_heads(self) -> int:
        return max([m.heads for m in self.attn_mixers] + [1])

    n_kv_heads = 1                  # one latent per token, whatever the heads

    def cache_index(self, layer: int) -> int:
        """Number of the layer's cache (attention) or state (recurrent)."""
        kind = self.layers[layer].mixer.recurrent
        return sum(l.mixer.recurrent == kind for l in self.layers[:layer])

    def n_params(self) -> int:
        from .fetotar_layout import tensor_shapes
        n = 0
        for shape in tensor_shapes(self).values():
            k = 1
            for x in shape:
                k *= x
            n += k
        return n

    # ---- config.json -----------------------------------------------------------------------
    @classmethod
    def from_json(cls, j: Dict, name: str = "fetotar", max_ctx: Optional[int] = None) -> "FetotarConfig":
        take(j, ("architecture", "width", "vocab", "norm", "embedding", "token_side", "layers"), "configuration")
        layers = []
        for i, l in enumerate(j["layers"]):
            l = take({"mlp": None, **l}, ("type", "mixer", "mlp"), f"layer {i}")
            if l["type"] not in MIXERS:
                raise ValueError(f"layer {i}: unknown mixer type {l['type']!r}")
            layers.append(LayerSpec(MIXERS[l["type"]].from_json(l["mixer"], f"layer {i} mixer"),
                                    None if l["mlp"] is None else ClampedGluSpec.from_json(l["mlp"], f"layer {i} mlp")))
        take(j["norm"], ("eps",), "norm"), take(j["embedding"], ("scale",), "embedding"), take(j["token_side"], ("dim",), "token_side")
        return cls(name=name, hidden=int(j["width"]), vocab=int(j["vocab"]), layers=tuple(layers),
                   side_dim=int(j["token_side"]["dim"]), embed_scale=float(j["embedding"]["scale"]),
                   norm_eps=float(j["norm"]["eps"]), **({} if max_ctx is None else {"max_ctx": max_ctx}))

    def to_json(self) -> Dict:
        return {"architecture": self.architecture, "width": self.hidden, "vocab": self.vocab, "norm": {"eps": self.norm_eps},
                "embedding": {"scale": self.embed_scale}, "token_side": {"dim": self.side_dim},
                "layers": [{"type": l.mixer.type, "mixer": l.mixer.to_json(), "mlp": None if l.mlp is None else l.mlp.to_json()}
                           for l in self.layers]}


def fetotar_tiny() -> FetotarConfig:
    """Smoke model: every mixer once, with and without a feed-forward, byte vocabulary of 320."""
    rot = RotarySpec(16, 10000.0, YarnSpec(4.0, 64.0, 8.0, 1.0))
    return FetotarConfig(
        name="fetotar-tiny", hidden=72, vocab=320, side_dim=20, embed_scale=1.5, norm_eps=1e-5, max_ctx=4096,
        layers=(LayerSpec(Mamba2Spec(4, 16, 24, 2, 4, 2), ClampedGluSpec(100, 2.0)),
                LayerSpec(LatentAttnSpec(5, 24, 16, 32, 40, 48, 0.16, 24, rot), None),
                LayerSpec(MlstmSpec(3, 24, 16, 10.0), ClampedGluSpec(64, 3.0))))


def fetotar_uniform(name: str, *, hidden: int, vocab: int, ff: int, heads: int, repeats: int, window: int, dim: int = 128,
                    rot_dim: int = 64, kv_rank: int = 512, q_rank: int = 1536, side_dim: int = 256, state: int = 128,
                    **kw) -> FetotarConfig:
    """A model of ``repeats`` x (mLSTM, latent attention, Mamba-2) layers of one width, each with a feed-forward; recurrent
    heads are ``dim`` wide on both sides."""
    attn = LatentAttnSpec(heads, dim, rot_dim, dim, q_rank, kv_rank, (dim + rot_dim) ** -0.5, window,
                          RotarySpec(rot_dim, 10000.0, YarnSpec(16.0, 4096.0, 32.0, 1.0)))
    glu = ClampedGluSpec(ff, 7.0)
    return FetotarConfig(name=name, hidden=hidden, vocab=vocab, side_dim=side_dim, **kw, layers=repeats * (
        LayerSpec(MlstmSpec(heads, dim, dim, 15.0), glu), LayerSpec(attn, glu),
        LayerSpec(Mamba2Spec(heads, dim, state, max(1, heads // 8), 4, 1), glu)))


def fetotar_small() -> FetotarConfig:
    """Three layers of a 1B-class width; profiler captures and GPU engine tests."""
    return fetotar_uniform("fetotar-small", hidden=2048, vocab=32768, ff=6144, heads=16, repeats=1, window=1024, q_rank=768)


# ---- Deluvik: attention beside a gated linear recurrence, shared keys, mixtures of experts ----------------------
# which optional parts the design's attention mixers have
_DELUVIK_ATTN = {"attention": dict(norm="all", half=True, capped=True, sink=True, tied=True),
                 "attention_2": dict(norm="all", half=True, conv=True, sink=True)}
_DELUVIK_LEFT = dict(norm="head", half=False, windowed=True)


def _deluvik_mixer(kind: str, m: Dict, where: str):
    if kind in _DELUVIK_ATTN:
        return SoftmaxAttnSpec.from_json(m, where, **_DELUVIK_ATTN[kind])
    if kind != "parallel":
        raise ValueError(f"{where}: unknown mixer type {kind!r}")
    take(m, ("left", "right", "left_scale", "right_scale"), where)
    return ParallelSpec(SoftmaxAttnSpec.from_json(m["left"], where + " left", **_DELUVIK_LEFT), LruSpec.from_json(m["right"], where + " right"),
                        float(m["left_scale"]), float(m["right_scale"]))


def _deluvik_mixer_json(m) -> Tuple[str, Dict]:
    if isinstance(m, ParallelSpec):
        return "parallel", {"left": m.left.to_json(), "right": m.right.to_json(), "left_scale": m.left_scale, "right_scale": m.right_scale}
    return ("attention" if m.tied else "attention_2"), m.to_json()


@dataclass(frozen=True)
class DeluvikConfig(StreamDesign):
    """Sizes and constants of a Deluvik model.  Every layer has its own mixer and feed-forward; a layer that reads another
    layer's keys and values (``kv_from``) has no KV cache of its own."""
    name: str
    hidden: int
    vocab: int
    layers: Tuple[LayerSpec, ...]
    logit_cap: float
    norm_eps: float = 1e-5
    max_ctx: int = 1 << 20

    architecture = "Deluvik"

    def __post_init__(self) -> None:
        object.__setattr__(self, "layers", tuple(self.layers))
        if self.hidden <= 0 or self.vocab <= 0 or not self.layers or self.logit_cap <= 0:
            raise ValueError("a model needs positive sizes, a positive cap on its logits and at least one layer")
        for i, l in enumerate(self.layers):
            a = self.attn(i)
            if a.kv_from is None:
                continue
            src = self.layers[a.kv_from].mixer if 0 <= a.kv_from < i else None
            if not isinstance(src, SoftmaxAttnSpec) or src.kv_from is not None or src.tied != a.tied or not a.same_keys(src):
                raise ValueError(f"layer {i} cannot read the keys of layer {a.kv_from}")

    def attn(self, layer: int) -> SoftmaxAttnSpec:
        """The attention of a layer (every layer has one)."""
        m = self.layers[layer].mixer
        return m.left if isinstance(m, ParallelSpec) else m

    @property
    def n_layers(self) -> int:
        return len(self.layers)

    @property
    def cache_owners(self) -> Tuple[int, ...]:
        """Layers with a KV cache, in the order of the caches."""
        return tuple(i for i in range(self.n_layers) if self.attn(i).kv_from is None)

    def cache_index(self, layer: int) -> int:
        """Number of the KV cache that the layer reads."""
        src = self.attn(layer).kv_from
        return self.cache_owners.index(layer if src is None else src)

    @property
    def n_attn_layers(self) -> int:
        return len(self.cache_owners)

    @property
    def n_q_heads(self) -> int:
        return max(self.attn(i).heads for i in range(self.n_layers))

    @property
    def n_kv_heads(self) -> int:
        return max(self.attn(i).kv_heads for i in range(self.n_layers))

    def n_params(self) -> int:
        from .deluvik_layout import tensor_shapes
        return sum(math.prod(s) for s in tensor_shapes(self).values())

    # ---- config.json -----------------------------------------------------------------------
    @classmethod
    def from_json(cls, j: Dict, name: str = "deluvik", max_ctx: Optional[int] = None) -> "DeluvikConfig":
        take(j, ("architecture", "width", "vocab", "norm", "logit_softcap", "layers"), "configuration")
        take(j["norm"], ("eps",), "norm")
        layers = []
        for i, l in enumerate(j["layers"]):
            l = take({"mlp": None, **l}, ("type", "mixer", "mlp"), f"layer {i}")
            f = l["mlp"]
            if f is not None:
                if f.get("kind") not in ("dense", "moe"):
                    raise ValueError(f"layer {i}: unknown feed-forward kind {f.get('kind')!r}")
                f = GluSpec.from_json(f, f"layer {i} mlp", "gelu") if f["kind"] == "dense" else MoeSpec.from_json(f, f"layer {i} mlp")
            layers.append(LayerSpec(_deluvik_mixer(l["type"], l["mixer"], f"layer {i} mixer"), f))
        return cls(name=name, hidden=int(j["width"]), vocab=int(j["vocab"]), layers=tuple(layers), logit_cap=float(j["logit_softcap"]),
                   norm_eps=float(j["norm"]["eps"]), **({} if max_ctx is None else {"max_ctx": max_ctx}))

    def to_json(self) -> Dict:
        layers = []
        for l in self.layers:
            kind, mixer = _deluvik_mixer_json(l.mixer)
            layers.append({"type": kind, "mixer": mixer, "mlp": None if l.mlp is None else l.mlp.to_json()})
        return {"architecture": self.architecture, "width": self.hidden, "vocab": self.vocab, "norm": {"eps": self.norm_eps},
                "logit_softcap": self.logit_cap, "layers": layers}


def deluvik_attention(heads, kv_heads, dim, scale, cap, rot) -> SoftmaxAttnSpec:
    """Mixer whose values are its keys: capped scores and a sink."""
    return SoftmaxAttnSpec(heads, kv_heads, dim, dim, scale, replace(rot, half=True), "all", None, cap, True, 0, True)


def deluvik_conv_attention(heads, kv_heads, dim, vdim, scale, conv, rot, kv_from=None) -> SoftmaxAttnSpec:
    """Mixer whose projections pass a short convolution, with a sink."""
    return SoftmaxAttnSpec(heads, kv_heads, dim, vdim, scale, replace(rot, half=True), "all", None, None, True, conv, False, kv_from)


def deluvik_parallel(left_scale, right_scale, right: LruSpec, heads, kv_heads, dim, vdim, scale, window, rot) -> ParallelSpec:
    """Windowed attention beside a gated linear recurrence."""
    return ParallelSpec(SoftmaxAttnSpec(heads, kv_heads, dim, vdim, scale, rot, "head", window), right, left_scale, right_scale)


def deluvik_tiny() -> DeluvikConfig:
    """Smoke model: every mixer, shared keys, both feed-forwards and none, byte vocabulary of 320."""
    rot, scaled = RotarySpec(16, 10000.0), RotarySpec(24, 5000.0, BandScalingSpec(4.0, 1.0, 4.0, 64.0))
    moe = MoeSpec(40, 6, 2, 56)
    return DeluvikConfig(
        name="deluvik-tiny", hidden=72, vocab=320, logit_cap=25.0, norm_eps=1e-5, max_ctx=4096,
        layers=(LayerSpec(deluvik_parallel(0.8, 1.1, LruSpec(60, 3, 4), 4, 2, 24, 32, 0.2, 24, rot), moe),
                LayerSpec(deluvik_attention(5, 1, 24, 0.2, 30.0, scaled), GluSpec(100, "gelu")),
                LayerSpec(deluvik_conv_attention(4, 2, 32, 16, 0.18, 3, rot), None),
                LayerSpec(deluvik_conv_attention(4, 2, 32, 16, 0.18, 3, rot, kv_from=2), moe)))


def deluvik_uniform(name: str, *, hidden: int, vocab: int, ff: int, expert_ff: int, experts: int, top: int, heads: int, kv_heads: int,
                    repeats: int, window: int, dim: int = 128, lru_blocks: int = 16, **kw) -> DeluvikConfig:
    """A model of ``repeats`` x (parallel, attention with a convolution, the same over the keys of the one before, attention over
    tied keys) layers of one width; the last of the four has a dense feed-forward, the others experts and a shared one."""
    rot, moe, layers = RotarySpec(dim, 500000.0), MoeSpec(expert_ff, experts, top, expert_ff), []
    for _ in range(repeats):
        n = len(layers)
        layers += [LayerSpec(deluvik_parallel(1.0, 1.0, LruSpec(hidden, lru_blocks, 4), heads, kv_heads, dim, dim, dim ** -0.5, window, rot), moe),
                   LayerSpec(deluvik_conv_attention(heads, kv_heads, dim, dim, dim ** -0.5, 4, rot), moe),
                   LayerSpec(deluvik_conv_attention(heads, kv_heads, dim, dim, dim ** -0.5, 4, rot, kv_from=n + 1), moe),
                   LayerSpec(deluvik_attention(heads, kv_heads, dim, dim ** -0.5, 50.0, replace(rot, scaling=BandScalingSpec(8.0, 1.0, 4.0, 8192.0))),
                             GluSpec(ff, "gelu"))]
    return DeluvikConfig(name=name, hidden=hidden, vocab=vocab, layers=tuple(layers), logit_cap=30.0, **kw)


def deluvik_small() -> DeluvikConfig:
    """Four layers of a 1B-class width; profiler captures and GPU engine tests."""
    return deluvik_uniform("deluvik-small", hidden=2048, vocab=32768, ff=6144, expert_ff=768, experts=32, top=4, heads=16, kv_heads=4,
                           repeats=1, window=1024)


# ---- Tobadra: turned values, lightning attention, per-channel delta rule, grouped experts, gated branches ------------
def tensor_shapes_in(path: str) -> Dict[str, Tuple[int, ...]]:
    """Shapes of the tensors in a directory's safetensors files, from their headers."""
    out: Dict[str, Tuple[int, ...]] = {}
    for f in sorted(os.listdir(path)):
        if f.endswith(".safetensors"):
            with open(os.path.join(path, f), "rb") as fh:
                head = json.loads(fh.read(int.from_bytes(fh.read(8), "little")))
            out.update({k: tuple(v["shape"]) for k, v in head.items() if k != "__metadata__"})
    return out


def _parameter_layer(weights_of, layer: int) -> int:
    """The layer whose parameters ``layer`` uses, by way of others that use them, too."""
    at = layer
    for _ in weights_of:
        if weights_of[at] is None:
            return at
        at = int(weights_of[at])
        if not 0 <= at < len(weights_of):
            break
    raise ValueError(f"layer {layer} uses the parameters of no layer")


@dataclass(frozen=True)
class TobadraConfig(StreamDesign):
    """Sizes and constants of a Tobadra model.  Every layer has its own mixer and feed-forward; attention layers number the KV
    caches.  A layer with ``weights_of`` uses another layer's parameters and keeps a cache or state of its own."""
    name: str
    hidden: int
    vocab: int
    layers: Tuple[LayerSpec, ...]
    canon: int                       # taps of the convolution on every mixer's input
    logit_scale: float = 1.0
    norm_eps: float = 1e-6
    max_ctx: int = 1 << 20

    architecture = "Tobadra"
    tie_embeddings = True
    MIXERS = (SoftmaxAttnSpec, LightningSpec, ChannelDeltaSpec)

    def __post_init__(self) -> None:
        object.__setattr__(self, "layers", tuple(self.layers))
        if self.hidden <= 0 or self.vocab <= 0 or not self.layers or self.canon < 1:
            raise ValueError("a model needs positive sizes, a tap and at least one layer")
        for i, l in enumerate(self.layers):
            if not isinstance(l.mixer, self.MIXERS):
                raise ValueError(f"layer {i}: not a mixer of this design: {l.mixer}")
            src = self.layers[_parameter_layer([x.weights_of for x in self.layers], i)]
            if (src.mixer, src.mlp) != (l.mixer, l.mlp):
                raise ValueError(f"layer {i} cannot use the parameters of layer {l.weights_of}")

    def source(self, layer: int) -> int:
        """The layer whose parameters this one uses."""
        return _parameter_layer([x.weights_of for x in self.layers], layer)

    @property
    def owners(self) -> Tuple[int, ...]:
        """Layers with parameters of their own."""
        return tuple(i for i, l in enumerate(self.layers) if l.weights_of is None)

    @property
    def n_layers(self) -> int:
        return len(self.layers)

    def attn(self, layer: int) -> SoftmaxAttnSpec:
        return self.layers[layer].mixer

    @property
    def cache_owners(self) -> Tuple[int, ...]:
        """Layers with a KV cache, in the order of the caches."""
        return tuple(i for i, l in enumerate(self.layers) if not l.mixer.recurrent)

    def cache_index(self, layer: int) -> int:
        return self.cache_owners.index(layer)

    @property
    def n_attn_layers(self) -> int:
        return len(self.cache_owners)

    @property
    def n_q_heads(self) -> int:
        return max([self.attn(i).heads for i in self.cache_owners] + [1])

    @property
    def n_kv_heads(self) -> int:
        return max([self.attn(i).kv_heads for i in self.cache_owners] + [1])

    def n_params(self) -> int:
        from .tobadra_layout import tensor_shapes
        return sum(math.prod(s) for s in tensor_shapes(self).values())

    # ---- config.json -----------------------------------------------------------------------
    @classmethod
    def from_json(cls, j: Dict, name: str = "tobadra", max_ctx: Optional[int] = None, shapes: Optional[Dict] = None) -> "TobadraConfig":
        """``shapes``: the checkpoint's tensor shapes, which hold the ranks of low-rank maps."""
        take(j, ("architecture", "width", "vocab", "norm", "canon", "logit_scale", "layers"), "configuration")
        take(j["norm"], ("eps",), "norm"), take(j["canon"], ("taps",), "canon")
        layers = []
        for i, l in enumerate(j["layers"]):
            l = take({"mlp": None, "weights_of": None, **l}, ("type", "mixer", "mlp", "weights_of"), f"layer {i}")
            m, f, src, where = l["mixer"], l["mlp"], l["weights_of"], f"layer {i} mixer"
            if l["type"] == "attention":
                m = SoftmaxAttnSpec.from_json(m, where, norm="none", half=True, windowed=True, bias=True, turned=True)
                if m.rot.scaling is not None:
                    raise ValueError(f"{where}: this design's rotations are not scaled")
            elif l["type"] == "lightning":
                m = LightningSpec.from_json(m, where)
            elif l["type"] == "channel_delta":
                own = _parameter_layer([x.get("weights_of") for x in j["layers"]], i)
                ranks = [(shapes or {}).get(f"l{own}.mix.{n}") for n in ("a1", "g1")]
                if None in ranks:
                    raise ValueError(f"{where}: the checkpoint does not have the maps whose shapes tell its ranks")
                m = ChannelDeltaSpec.from_json(m, where, *(r[0] for r in ranks))
            else:
                raise ValueError(f"layer {i}: unknown mixer type {l['type']!r}")
            if f is not None:
                if f.get("kind") not in ("dense", "moe"):
                    raise ValueError(f"layer {i}: unknown feed-forward kind {f.get('kind')!r}")
                f = DenseSpec.from_json(f, f"layer {i} mlp", "gelu") if f["kind"] == "dense" else MoeSpec.from_json_grouped(f, f"layer {i} mlp", "gelu_erf")
            layers.append(LayerSpec(m, f, None if src is None else int(src)))
        return cls(name=name, hidden=int(j["width"]), vocab=int(j["vocab"]), layers=tuple(layers), canon=int(j["canon"]["taps"]),
                   logit_scale=float(j["logit_scale"]), norm_eps=float(j["norm"]["eps"]), **({} if max_ctx is None else {"max_ctx": max_ctx}))

    @classmethod
    def from_dir(cls, j: Dict, path: str, name: str) -> "TobadraConfig":
        return cls.from_json(j, name=name, shapes=tensor_shapes_in(path))

    def to_json(self) -> Dict:
        layers = []
        for l in self.layers:
            layers.append({"type": l.mixer.type, "mixer": l.mixer.to_json(), "mlp": None if l.mlp is None else l.mlp.to_json()})
            if l.weights_of is not None:
                layers[-1]["weights_of"] = l.weights_of
        return {"architecture": self.architecture, "width": self.hidden, "vocab": self.vocab, "norm": {"eps": self.norm_eps},
                "canon": {"taps": self.canon}, "logit_scale": self.logit_scale, "layers": layers}


def tobadra_attention(heads, kv_heads, dim, vdim, scale, window, dims, base=10000.0) -> SoftmaxAttnSpec:
    """Windowed attention with biases whose values turn with their positions."""
    return SoftmaxAttnSpec(heads, kv_heads, dim, vdim, scale, RotarySpec(dims, base, None, True), "none", window, bias=True, turned=True)


def tobadra_moe(ff, experts, top, shared=0, scale=1.0, identity=0, groups=1, keep=1) -> MoeSpec:
    return MoeSpec(ff, experts, top, shared, "gelu_erf", False, shared > 0, RouterSpec(scale, identity, groups, keep))


def tobadra_tiny() -> TobadraConfig:
    """Smoke model: every mixer, shared parameters, both feed-forwards and none, byte vocabulary of 320."""
    moe, delta = tobadra_moe(40, 7, 2, 56, 1.3, 2, 3, 2), ChannelDeltaSpec(4, 2, 24, 16, 4, 12, 20)
    return TobadraConfig(
        name="tobadra-tiny", hidden=72, vocab=320, canon=3, logit_scale=0.5, norm_eps=1e-5, max_ctx=4096,
        layers=(LayerSpec(tobadra_attention(4, 2, 24, 20, 0.2, 24, 16), DenseSpec(100, "gelu")),
                LayerSpec(delta, moe), LayerSpec(LightningSpec(3, 16, 24, (0.7, 0.95, 0.995)), None),
                LayerSpec(delta, moe, weights_of=1)))


def tobadra_uniform(name: str, *, hidden: int, vocab: int, ff: int, expert_ff: int, experts: int, top: int, heads: int, kv_heads: int,
                    repeats: int, window: int, dim: int = 128, rank: int = 128, identity: int = 0, groups: int = 1, keep: int = 1, **kw) -> TobadraConfig:
    """A model of ``repeats`` x (channel delta, lightning, attention, channel delta) layers of one width; the first of the four has a
    dense feed-forward, the others experts and a shared one."""
    moe, layers = tobadra_moe(expert_ff, experts, top, expert_ff, 1.0, identity, groups, keep), []
    delta = ChannelDeltaSpec(heads, heads, dim, dim, 4, rank, rank)
    decay = tuple(1.0 - 2.0 ** (-4.0 - 6.0 * i / max(1, heads - 1)) for i in range(heads))
    for _ in range(repeats):
        layers += [LayerSpec(delta, DenseSpec(ff, "gelu")), LayerSpec(LightningSpec(heads, dim, dim, decay), moe),
                   LayerSpec(tobadra_attention(heads, kv_heads, dim, dim, dim ** -0.5, window, dim), moe), LayerSpec(delta, moe)]
    return TobadraConfig(name=name, hidden=hidden, vocab=vocab, layers=tuple(layers), canon=4, **kw)


def tobadra_small() -> TobadraConfig:
    """Four layers of a 1B-class width; profiler captures and GPU engine tests."""
    return tobadra_uniform("tobadra-small", hidden=2048, vocab=32768, ff=8192, expert_ff=1024, experts=32, top=4, heads=16, kv_heads=4,
                           repeats=1, window=1024, identity=8, groups=4, keep=2)


ARCHITECTURES = {c.architecture: c for c in (ZinutarConfig, FetotarConfig, DeluvikConfig, TobadraConfig)}

_REGISTRY = {
    "tobadra-tiny": tobadra_tiny, "tobadra-small": tobadra_small,
    "deluvik-tiny": deluvik_tiny, "deluvik-small": deluvik_small,
    "fetotar-tiny": fetotar_tiny, "fetotar-small": fetotar_small,
    "zinutar-tiny": zinutar_tiny, "zinutar-small": zinutar_small, "zinutar-8b": zinutar_8b,
    "qwen38-27b": qwen38_27b, "qwen36-27b": qwen36_27b, "tiny": tiny,
    "tiny-hybrid": tiny_hybrid, "small-gpu": small_gpu, "small-gpu-tp": small_gpu_tp,
    "tiny-agent": lambda: tiny(65536),
}


def config_from_dir(path: str):
    """The configuration a checkpoint directory describes in its ``config.json``: by ``architecture`` for designs
    whose file spells every size out, else by the registry name that ``save_checkpoint`` wrote."""
    with open(os.path.join(path, "config.json")) as f:
        j = json.load(f)
    arch = j.get("architecture")
    if arch in ARCHITECTURES:
        return ARCHITECTURES[arch].from_dir(j, path, os.path.basename(os.path.normpath(path)))
    if j.get("name") in _REGISTRY:
        return _REGISTRY[j["name"]]()
    raise ValueError(f"{path}/config.json names neither a known architecture ({sorted(ARCHITECTURES)}) nor a known model")


def get_config(name: str):
    """Configuration by registry name, or by a checkpoint directory that holds a ``config.json``."""
    if name in _REGISTRY:
        return _REGISTRY[name]()
    if os.path.exists(os.path.join(name, "config.json")):
        return config_from_dir(name)
    raise ValueError(f"unknown model {name!r}; known: {sorted(_REGISTRY)}, or a directory with a config.json")
