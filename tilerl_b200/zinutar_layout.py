"""Shapes and memory layout of a Zinutar model's parameters: what a checkpoint holds and what is served.

Every head and the stream are padded with zero rows / columns to the widths the kernels load.  No counterpart in the
reference.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, Tuple

from .config import BlockSpec, ZinutarConfig


def _pad(n: int, m: int) -> int:
    return (n + m - 1) // m * m


def stream_width(cfg: ZinutarConfig) -> int:
    """Columns of the stream and of every projection that reads it."""
    return _pad(cfg.hidden, 64)


def head_rows(cfg: ZinutarConfig) -> int:
    return _pad(cfg.vocab, 8)


@dataclass(frozen=True)
class BlockLayout:
    """Where a layer's pieces sit in its two fused projections.  ``in`` rows: ``[q heads x dk | k heads x dk |
    v heads x dv | up]``; ``out`` columns: ``[heads x dv | ff]``, both with padded widths."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    ff: int          # 0: no feed-forward

    @staticmethod
    def of(b: BlockSpec) -> "BlockLayout":
        a = b.mixer
        return BlockLayout(a.heads, a.kv_heads, a.dim, a.vdim, a.scale, 0 if b.mlp is None else b.mlp.ff)

    @property
    def dk(self) -> int:
        return _pad(self.dim, 16)

    @property
    def dv(self) -> int:
        return _pad(self.vdim, 16)

    @property
    def k0(self) -> int:
        return self.heads * self.dk

    @property
    def v0(self) -> int:
        return self.k0 + self.kv_heads * self.dk

    @property
    def up0(self) -> int:
        return self.v0 + self.kv_heads * self.dv

    @property
    def n_in(self) -> int:
        return self.up0 + (_pad(self.ff, 16) if self.ff else 0)

    @property
    def attn_cols(self) -> int:
        return self.heads * self.dv

    @property
    def n_out(self) -> int:
        return _pad(self.attn_cols + self.ff, 64)


def tensor_shapes(cfg: ZinutarConfig) -> Dict[str, Tuple[int, ...]]:
    """Tensors of a checkpoint file (linear weights ``[out, in]``)."""
    h = cfg.hidden
    out: Dict[str, Tuple[int, ...]] = {"embed": (cfg.vocab, h), "embed.norm": (h,)}
    for i, b in enumerate(cfg.layers):
        a, p = b.mixer, f"l{i}."
        out[p + "norm1"] = (h,)
        out[p + "mix.q"] = (a.heads * a.dim, h)
        out[p + "mix.k"] = (a.kv_heads * a.dim, h)
        out[p + "mix.v"] = (a.kv_heads * a.vdim, h)
        out[p + "mix.pb"] = (a.heads,)
        out[p + "mix.o"] = (h, a.heads * a.vdim)
        if b.mlp is not None:
            out[p + "mlp.up"] = (b.mlp.ff, h)
            out[p + "mlp.down"] = (h, b.mlp.ff)
            out[p + "mlp.act"] = (4,)
    out["final.norm"] = (h,)
    out["head"] = (cfg.vocab, h)
    return out


def param_shapes(cfg: ZinutarConfig) -> Dict[str, Tuple[Tuple[int, ...], str]]:
    """Served parameters: name -> (shape, ``"w"`` for the compute dtype or ``"f32"``)."""
    w = stream_width(cfg)
    out = {"embed": ((cfg.vocab, w), "w"), "embed_norm": ((w,), "f32"), "final_norm": ((w,), "f32"),
           "lm_head": ((head_rows(cfg), w), "w")}
    for i, b in enumerate(cfg.layers):
        l, p = BlockLayout.of(b), f"L{i}."
        out[p + "norm1"] = ((w,), "f32")
        out[p + "in"] = ((l.n_in, w), "w")
        out[p + "out"] = ((w, l.n_out), "w")
        out[p + "bias"] = ((l.heads,), "f32")
        if l.ff:
            out[p + "act"] = ((4,), "f32")
    return out
