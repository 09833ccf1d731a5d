"""Shapes and memory layout of a Tobadra model: checkpoint tensors, served parameters, and what its layers keep per sequence.

Heads are padded with zero rows / columns to 16, everything a projection reads to 64, so every size of the configuration runs on the
same kernels.  Turned values keep their two halves at the halves of the padded head, so that a pair is always half a padded head
apart.  No counterpart in the reference.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, List, Tuple

from .deluvik_layout import AttnLayout, LayerLayout, MoeLayout
from .fetotar_layout import head_rows, pad, stream_width  # noqa: F401 - part of this module's surface
from .mixers import ChannelDeltaSpec, LightningSpec, MoeSpec, SoftmaxAttnSpec


# ---- served layout of a mixer: rows of its fused input projection, columns of its output projection --------------
@dataclass(frozen=True)
class LightningLayout:
    """``in`` rows: ``[q heads x dk | k heads x dk | v heads x dv | gate heads x dv]``; q, k and v pass silu."""
    spec: LightningSpec

    kind = "lightning"
    conv_c = 0
    taps = 1
    n_gates = 0
    norm_groups = 1

    @property
    def heads(self) -> int:
        return self.spec.heads

    @property
    def vdim(self) -> int:
        return self.spec.vdim

    @property
    def dk(self) -> int:
        return pad(self.spec.dim)

    @property
    def dv(self) -> int:
        return pad(self.spec.vdim)

    @property
    def k0(self) -> int:
        return self.heads * self.dk

    @property
    def v0(self) -> int:
        return 2 * self.heads * self.dk

    @property
    def g0(self) -> int:
        return self.v0 + self.heads * self.dv

    @property
    def n_in(self) -> int:
        return self.g0 + self.heads * self.dv

    @property
    def n_out(self) -> int:
        return pad(self.heads * self.dv, 64)

    @property
    def state_floats(self) -> int:
        return self.heads * self.dk * self.dv


@dataclass(frozen=True)
class DeltaLayout:
    """``in`` rows: ``[q kv_heads x dk | k kv_heads x dk | v heads x dv | decay map | gate map]``, then one fp32 write gate per head.
    The first ``conv_c`` columns pass the convolution.  Both maps go on from ``r`` columns to ``low`` rows: ``[gate heads x dv]``,
    then the fp32 decays ``[heads x dk]``."""
    spec: ChannelDeltaSpec

    kind = "delta"

    @property
    def heads(self) -> int:
        return self.spec.heads

    @property
    def kv_heads(self) -> int:
        return self.spec.kv_heads

    @property
    def per(self) -> int:
        """Heads that share a query / key head."""
        return self.spec.heads // self.spec.kv_heads

    @property
    def vdim(self) -> int:
        return self.spec.vdim

    @property
    def dk(self) -> int:
        return pad(self.spec.dim)

    @property
    def dv(self) -> int:
        return pad(self.spec.vdim)

    @property
    def taps(self) -> int:
        return self.spec.conv

    @property
    def k0(self) -> int:
        return self.kv_heads * self.dk

    @property
    def v0(self) -> int:
        return 2 * self.kv_heads * self.dk

    @property
    def conv_c(self) -> int:
        return self.v0 + self.heads * self.dv

    @property
    def r(self) -> int:
        return pad(max(self.spec.decay_rank, self.spec.gate_rank), 64)

    @property
    def a0(self) -> int:
        return self.conv_c

    @property
    def g0(self) -> int:
        return self.a0 + self.r

    @property
    def n_in(self) -> int:
        return self.g0 + self.r

    @property
    def n_low(self) -> int:
        """Rows of the output gate, before those of the decays."""
        return self.heads * self.dv

    @property
    def n_gates(self) -> int:
        return self.heads

    @property
    def norm_groups(self) -> int:
        return self.heads

    @property
    def n_out(self) -> int:
        return pad(self.heads * self.dv, 64)

    @property
    def state_floats(self) -> int:
        return self.heads * self.dk * self.dv


def layout_of(m):
    if isinstance(m, SoftmaxAttnSpec):
        return LayerLayout(AttnLayout(m), None)
    return LightningLayout(m) if isinstance(m, LightningSpec) else DeltaLayout(m)


def layouts(cfg) -> Tuple[object, ...]:
    return tuple(layout_of(l.mixer) for l in cfg.layers)


def gate_rows(l) -> int:
    """fp32 rows of a mixer's input projection, behind its ``n_in`` others."""
    return pad(getattr(l, "n_gates", 0))


@dataclass(frozen=True)
class InputLayout:
    """What the convolution on a mixer's input keeps per sequence: its last inputs."""
    layer: int
    conv_c: int
    taps: int

    kind = "input"
    state_floats = 0


def state_layouts(cfg) -> Tuple[object, ...]:
    """Every layer's input convolution, then the recurrent mixers' states."""
    w = stream_width(cfg)
    return tuple(InputLayout(i, w, cfg.canon) for i in range(cfg.n_layers)) + tuple(l for l in layouts(cfg) if not isinstance(l, LayerLayout))


# ---- feed-forwards -------------------------------------------------------------------------------------------
def router_rows(m: MoeSpec) -> int:
    """Rows of the fused router before those of the branch's gate: one per output, the shared expert's gate, padding."""
    return pad(m.outputs + 1)


# ---- checkpoint ----------------------------------------------------------------------------------------------
def _mixer_shapes(m, p: str, h: int) -> Dict[str, Tuple[int, ...]]:
    out: Dict[str, Tuple[int, ...]] = {}
    if isinstance(m, SoftmaxAttnSpec):
        for n, r in (("q", m.heads * m.dim), ("k", m.kv_heads * m.dim), ("v", m.kv_heads * m.vdim)):
            out[p + n], out[f"{p}{n}.b"] = (r, h), (r,)
        out[p + "o"], out[p + "o.b"] = (h, m.heads * m.vdim), (h,)
        return out
    if isinstance(m, LightningSpec):
        qk, v = m.heads * m.dim, m.heads * m.vdim
        return {p + "q": (qk, h), p + "k": (qk, h), p + "v": (v, h), p + "g": (v, h), p + "o": (h, v), p + "norm": (v,)}
    v = m.heads * m.vdim
    for n, r in (("q", m.kv_heads * m.dim), ("k", m.kv_heads * m.dim), ("v", v)):
        out[p + n], out[f"{p}{n}.conv"] = (r, h), (r, m.conv)
    out.update({p + "b": (m.heads, h), p + "A_log": (m.heads,), p + "norm": (m.vdim,), p + "a1": (m.decay_rank, h),
                p + "a2": (m.heads * m.dim, m.decay_rank), p + "dt_bias": (m.heads * m.dim,), p + "g1": (m.gate_rank, h),
                p + "g2": (v, m.gate_rank), p + "o": (h, v)})
    return out


def _ff_shapes(p: str, h: int, ff: int) -> Dict[str, Tuple[int, ...]]:
    return {p + "up": (ff, h), p + "down": (h, ff)}


def tensor_shapes(cfg) -> Dict[str, Tuple[int, ...]]:
    """Tensors of a checkpoint file (linear weights ``[out, in]``)."""
    h = cfg.hidden
    out: Dict[str, Tuple[int, ...]] = {"embed": (cfg.vocab, h), "embed.norm": (h,)}
    for i in cfg.owners:
        l, p = cfg.layers[i], f"l{i}."
        out[p + "norm1"] = out[p + "norm1b"] = (h,)
        out.update(_mixer_shapes(l.mixer, p + "mix.", h))
        out[p + "canon1"], out[p + "rg1"], out[p + "rg1.b"] = (h, cfg.canon), (h, h), (h,)
        if l.mlp is None:
            continue
        out[p + "norm2"] = out[p + "norm2b"] = out[p + "rg2.b"] = (h,)
        out[p + "rg2"] = (h, h)
        if not isinstance(l.mlp, MoeSpec):
            out.update(_ff_shapes(p + "mlp.", h, l.mlp.ff))
            continue
        for e in range(l.mlp.experts):
            out.update(_ff_shapes(f"{p}mlp.e{e}.", h, l.mlp.ff))
        out[p + "mlp.router"], out[p + "mlp.correction"] = (l.mlp.outputs, h), (l.mlp.outputs,)
        if l.mlp.shared:
            out.update(_ff_shapes(p + "mlp.shared.", h, l.mlp.shared))
            out[p + "mlp.shared.sg"] = (1, h)
    out["final.norm"] = (h,)
    return out


def param_shapes(cfg) -> Dict[str, Tuple[Tuple[int, ...], str]]:
    """Served parameters: name -> (shape, ``"w"`` for the compute dtype or ``"f32"``)."""
    w = stream_width(cfg)
    out: Dict[str, Tuple[Tuple[int, ...], str]] = {
        "embed": ((head_rows(cfg), w), "w"), "embed_norm": ((1, w), "f32"), "final_norm": ((1, w), "f32")}
    for i in cfg.owners:
        b, p = cfg.layers[i], f"L{i}."
        l = layout_of(b.mixer)
        out[p + "norm1"] = out[p + "norm1b"] = ((1, w), "f32")
        out[p + "canon"], out[p + "rg1_b"] = ((cfg.canon, w), "f32"), ((w,), "f32")
        out[p + "in"], out[p + "o"] = ((l.n_in + gate_rows(l) + w, w), "w"), ((w, l.n_out), "w")      # the mixer's rows, its branch's gate
        if isinstance(l, LayerLayout):
            out[p + "qkv_b"], out[p + "o_b"] = ((l.n_in,), "f32"), ((w,), "f32")
        elif l.kind == "lightning":
            out[p + "norm"] = ((l.heads * l.dv,), "f32")
        else:
            out[p + "norm"], out[p + "conv"] = ((l.dv,), "f32"), ((l.taps, l.conv_c), "f32")
            out[p + "low"] = ((l.n_low + l.heads * l.dk, l.r), "w")
            out[p + "dt_bias"], out[p + "a_log"] = ((l.heads * l.dk,), "f32"), ((l.heads,), "f32")
        if b.mlp is None:
            continue
        out[p + "norm2"] = out[p + "norm2b"] = ((1, w), "f32")
        out[p + "rg2_b"] = ((w,), "f32")
        if isinstance(b.mlp, MoeSpec):
            m = MoeLayout(b.mlp)
            out[p + "router"], out[p + "correction"] = ((router_rows(b.mlp) + w, w), "w"), ((pad(b.mlp.outputs, 8),), "f32")
            out[p + "up"], out[p + "down"] = ((m.n, m.ff, w), "w"), ((m.n, w, m.ff), "w")
        else:
            out[p + "up"], out[p + "down"] = ((pad(b.mlp.ff, 64) + w, w), "w"), ((w, pad(b.mlp.ff, 64)), "w")
    return out
