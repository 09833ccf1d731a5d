"""Shapes and memory layout of a Deluvik model: checkpoint tensors, served parameters, and what its layers keep per sequence.

Heads and the parts of a recurrence are padded with zero rows / columns to 16, everything a projection reads to 64, so every
size of the configuration runs on the same kernels.  No counterpart in the reference.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, List, Optional, Tuple

from .fetotar_layout import head_rows, pad, stream_width  # noqa: F401 - head_rows is part of this module's surface
from .mixers import LruSpec, MoeSpec, ParallelSpec, SoftmaxAttnSpec


# ---- served layout of a layer: rows of its fused input projection, columns of its output projection --------------
@dataclass(frozen=True)
class AttnLayout:
    """``in`` rows: ``[q heads x dk | k kv_heads x dk | v kv_heads x dv]``; without own keys only q, with tied values no v."""
    spec: SoftmaxAttnSpec

    @property
    def dk(self) -> int:
        return pad(self.spec.dim)

    @property
    def dv(self) -> int:
        return pad(self.spec.vdim)

    @property
    def own(self) -> bool:
        return self.spec.kv_from is None

    @property
    def k0(self) -> int:
        return self.spec.heads * self.dk

    @property
    def v0(self) -> int:
        """First column of the values: that of the keys where they are the values."""
        return self.k0 if self.spec.tied else self.k0 + self.spec.kv_heads * self.dk

    @property
    def n_in(self) -> int:
        return self.v0 + self.spec.kv_heads * self.dv if self.own else self.k0

    @property
    def conv_c(self) -> int:
        """Columns that pass the convolution."""
        return self.n_in if self.spec.conv else 0

    @property
    def taps(self) -> int:
        return max(1, self.spec.conv)

    @property
    def n_out(self) -> int:
        return self.spec.heads * self.dv


@dataclass(frozen=True)
class LruLayout:
    """``in`` rows: ``[gelu branch | recurrent branch]``, each ``blocks`` parts of ``pp`` rows; the recurrent branch passes the
    convolution."""
    spec: LruSpec

    @property
    def pp(self) -> int:
        return pad(self.spec.part)

    @property
    def width(self) -> int:
        return self.spec.blocks * self.pp

    @property
    def n_in(self) -> int:
        return 2 * self.width

    @property
    def n_out(self) -> int:
        return self.width


@dataclass(frozen=True)
class LayerLayout:
    attn: AttnLayout
    lru: Optional[LruLayout]
    attn_scale: float = 1.0
    lru_scale: float = 1.0

    @staticmethod
    def of(m) -> "LayerLayout":
        if isinstance(m, ParallelSpec):
            return LayerLayout(AttnLayout(m.left), LruLayout(m.right), m.left_scale, m.right_scale)
        return LayerLayout(AttnLayout(m), None)

    @property
    def n_in(self) -> int:
        return self.attn.n_in + (self.lru.n_in if self.lru else 0)

    @property
    def n_mid(self) -> int:
        """Columns between the two projections, without padding."""
        return self.attn.n_out + (self.lru.n_out if self.lru else 0)

    @property
    def n_out(self) -> int:
        return pad(self.n_mid, 64)


def layouts(cfg) -> Tuple[LayerLayout, ...]:
    return tuple(LayerLayout.of(l.mixer) for l in cfg.layers)


@dataclass(frozen=True)
class StateLayout:
    """What one layer keeps per sequence beside keys and values: ``state_floats`` fp32 values of a recurrence and the inputs of
    a convolution of ``taps`` over ``conv_c`` columns."""
    layer: int
    state_floats: int
    conv_c: int
    taps: int

    kind = "lru"

    def parts(self, rec):
        return [rec]


def state_layouts(cfg) -> Tuple[StateLayout, ...]:
    """In the order of the states; layers without any are left out."""
    out: List[StateLayout] = []
    for i, l in enumerate(layouts(cfg)):
        if l.lru is not None:
            out.append(StateLayout(i, l.lru.width, l.lru.width, l.lru.spec.conv))
        if l.attn.conv_c:
            out.append(StateLayout(i, 0, l.attn.conv_c, l.attn.taps))
    return tuple(out)


# ---- feed-forwards -------------------------------------------------------------------------------------------
@dataclass(frozen=True)
class MoeLayout:
    """Expert weights of one width ``ff``; the shared feed-forward is cut into ``pieces`` experts of that width that every token
    uses with weight one (a gated feed-forward is the sum of its column ranges)."""
    spec: MoeSpec

    @property
    def ff(self) -> int:
        return pad(self.spec.ff, 64)

    @property
    def pieces(self) -> int:
        return (self.spec.shared + self.ff - 1) // self.ff

    @property
    def n(self) -> int:
        return self.spec.experts + self.pieces

    @property
    def slots(self) -> int:
        """Experts a token uses."""
        return self.spec.top + self.pieces

    @property
    def router_rows(self) -> int:
        return pad(self.spec.experts, 8)


# ---- checkpoint ----------------------------------------------------------------------------------------------
def _attn_shapes(a: SoftmaxAttnSpec, p: str, h: int) -> Dict[str, Tuple[int, ...]]:
    rows = {"q": a.heads * a.dim}
    if a.kv_from is None:
        rows["k"] = a.kv_heads * a.dim
        if not a.tied:
            rows["v"] = a.kv_heads * a.vdim
    out: Dict[str, Tuple[int, ...]] = {}
    for n, r in rows.items():
        out[p + n] = (r, h)
        if n != "v":
            out[f"{p}{n}.norm"] = (a.dim if a.norm == "head" else r,)
        if a.conv:
            out[f"{p}{n}.conv"] = (r, a.conv)
    if a.sink:
        out[p + "sink"] = (a.heads,)
    out[p + "o"] = (h, a.heads * a.vdim)
    return out


def _lru_shapes(m: LruSpec, p: str, h: int) -> Dict[str, Tuple[int, ...]]:
    out: Dict[str, Tuple[int, ...]] = {}
    for n in ("y", "x"):
        out[p + n], out[f"{p}{n}.b"] = (m.width, h), (m.width,)
    out[p + "conv"], out[p + "conv.b"] = (m.width, m.conv), (m.width,)
    for n in ("ra", "ri"):
        out[p + n], out[f"{p}{n}.b"] = (m.blocks, m.part, m.part), (m.blocks, m.part)
    out[p + "lam"], out[p + "o"] = (m.width,), (h, m.width)
    return out


def _glu_shapes(p: str, h: int, ff: int) -> Dict[str, Tuple[int, ...]]:
    return {p + "gate": (ff, h), p + "up": (ff, h), p + "down": (h, ff)}


def tensor_shapes(cfg) -> Dict[str, Tuple[int, ...]]:
    """Tensors of a checkpoint file (linear weights ``[out, in]``)."""
    h = cfg.hidden
    out: Dict[str, Tuple[int, ...]] = {"embed": (cfg.vocab, h)}
    for i, l in enumerate(cfg.layers):
        p, m = f"l{i}.", l.mixer
        out[p + "norm1"] = (h,)
        if isinstance(m, ParallelSpec):
            out.update(_attn_shapes(m.left, p + "mix.left.", h))
            out.update(_lru_shapes(m.right, p + "mix.right.", h))
        else:
            out.update(_attn_shapes(m, p + "mix.", h))
        if l.mlp is None:
            continue
        out[p + "norm2"] = (h,)
        if isinstance(l.mlp, MoeSpec):
            for e in range(l.mlp.experts):
                out.update(_glu_shapes(f"{p}mlp.e{e}.", h, l.mlp.ff))
            if l.mlp.shared:
                out.update(_glu_shapes(p + "mlp.shared.", h, l.mlp.shared))
            out[p + "mlp.router"], out[p + "mlp.router.b"] = (l.mlp.experts, h), (l.mlp.experts,)
        else:
            out.update(_glu_shapes(p + "mlp.", h, l.mlp.ff))
    out["final.norm"], out["head"] = (h,), (cfg.vocab, h)
    return out


def param_shapes(cfg) -> Dict[str, Tuple[Tuple[int, ...], str]]:
    """Served parameters: name -> (shape, ``"w"`` for the compute dtype or ``"f32"``)."""
    w = stream_width(cfg)
    out: Dict[str, Tuple[Tuple[int, ...], str]] = {
        "embed": ((cfg.vocab, w), "w"), "lm_head": ((head_rows(cfg), w), "w"), "final_norm": ((1, w), "f32")}
    for i, (b, l) in enumerate(zip(cfg.layers, layouts(cfg))):
        p, a, s = f"L{i}.", l.attn, l.attn.spec
        out[p + "norm1"] = ((1, w), "f32")
        out[p + "in"], out[p + "o"] = ((l.n_in, w), "w"), ((w, l.n_out), "w")
        out[p + "q_norm"] = ((a.dk if s.norm == "head" else s.heads * a.dk,), "f32")
        if a.own:
            out[p + "k_norm"] = ((a.dk if s.norm == "head" else s.kv_heads * a.dk,), "f32")
        if s.conv:
            out[p + "conv"] = ((s.conv, a.conv_c), "f32")
        if s.sink:
            out[p + "sink"] = ((s.heads,), "f32")
        if l.lru is not None:
            r = l.lru
            out[p + "y_b"] = out[p + "x_b"] = out[p + "lru_conv_b"] = out[p + "lam"] = ((r.width,), "f32")
            out[p + "lru_conv"] = ((r.spec.conv, r.width), "f32")
            out[p + "gates"] = ((r.spec.blocks, 2 * r.pp, r.pp), "w")     # per part: recurrence gate rows, input gate rows
            out[p + "gates_b"] = ((r.spec.blocks, 2 * r.pp), "f32")
        if b.mlp is None:
            continue
        out[p + "norm2"] = ((1, w), "f32")
        if isinstance(b.mlp, MoeSpec):
            m = MoeLayout(b.mlp)
            out[p + "router"], out[p + "router_b"] = ((m.router_rows, w), "w"), ((m.router_rows,), "f32")
            out[p + "gate_up"] = ((m.n, 2 * m.ff, w), "w")                # per expert as below
            out[p + "down"] = ((m.n, w, m.ff), "w")
        else:
            out[p + "gate_up"] = ((2 * pad(b.mlp.ff, 64), w), "w")        # rows 2j = gate_j, 2j + 1 = up_j
            out[p + "down"] = ((w, pad(b.mlp.ff, 64)), "w")
    return out
