"""Shapes and memory layout of a Fetotar model: checkpoint tensors, served parameters, and the state of its recurrent layers.

Heads and latents are padded with zero rows / columns to 16, everything a projection reads to 64, so every size of the
configuration runs on the same kernels.  No counterpart in the reference.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, Tuple

from .mixers import LatentAttnSpec, Mamba2Spec, MlstmSpec


def pad(n: int, m: int = 16) -> int:
    return (n + m - 1) // m * m


def stream_width(cfg) -> int:
    """Columns of the stream and of every projection that reads it."""
    return pad(cfg.hidden, 64)


def head_rows(cfg) -> int:
    return pad(cfg.vocab, 8)


# ---- served layout of each mixer: rows of its fused input projection, columns of its output projection ----------
@dataclass(frozen=True)
class LatentLayout:
    """``in`` rows: ``[query latent | kv latent | shared rotated key | gate heads x dv]``."""
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    window: int

    kind = "latent"
    n_gates = 0

    @staticmethod
    def of(m: LatentAttnSpec) -> "LatentLayout":
        return LatentLayout(m.heads, m.dim, m.rot_dim, m.vdim, m.q_rank, m.kv_rank, m.scale, m.window)

    @property
    def dk(self) -> int:
        return pad(self.dim)

    @property
    def rd(self) -> int:
        return pad(self.rot_dim)

    @property
    def dv(self) -> int:
        return pad(self.vdim)

    @property
    def kv(self) -> int:
        return pad(self.kv_rank)

    @property
    def c0(self) -> int:
        """First column of the kv latent (and padded width of the query latent)."""
        return pad(self.q_rank, 64)

    @property
    def kr0(self) -> int:
        return self.c0 + self.kv

    @property
    def g0(self) -> int:
        return self.kr0 + self.rd

    @property
    def n_in(self) -> int:
        return self.g0 + self.heads * self.dv

    @property
    def dq(self) -> int:
        """Width of one query head: unrotated part, rotated part."""
        return self.dk + self.rd

    @property
    def row(self) -> int:
        """Width of a cached row: latent, rotated key."""
        return self.kv + self.rd

    @property
    def n_out(self) -> int:
        return pad(self.heads * self.dv, 64)


@dataclass(frozen=True)
class MambaLayout:
    """``in`` rows: ``[x heads x dv | B groups x dk | C groups x dk | z heads x dv]``, then one fp32 step gate per head.
    The first ``conv_c`` columns pass the convolution."""
    heads: int
    vdim: int
    state: int
    groups: int
    taps: int
    norm_groups: int

    kind = "mamba2"

    @staticmethod
    def of(m: Mamba2Spec) -> "MambaLayout":
        return MambaLayout(m.heads, m.vdim, m.state, m.groups, m.conv, m.norm_groups)

    @property
    def dv(self) -> int:
        return pad(self.vdim)

    @property
    def dk(self) -> int:
        return pad(self.state)

    @property
    def k0(self) -> int:
        return self.heads * self.dv

    @property
    def q0(self) -> int:
        return self.k0 + self.groups * self.dk

    @property
    def conv_c(self) -> int:
        return self.q0 + self.groups * self.dk

    @property
    def g0(self) -> int:
        return self.conv_c

    @property
    def n_in(self) -> int:
        return self.g0 + self.heads * self.dv

    @property
    def n_gates(self) -> int:
        return self.heads

    @property
    def n_out(self) -> int:
        return pad(self.heads * self.dv, 64)

    @property
    def state_floats(self) -> int:
        return self.heads * self.dk * self.dv


@dataclass(frozen=True)
class MlstmLayout:
    """``in`` rows: ``[q heads x dk | k heads x dk | v heads x dv | gate heads x dv]``, then the fp32 input and forget
    gates per head.  The factor ``dim ** -0.5`` of the queries is applied in fp32 where they are read."""
    heads: int
    dim: int
    vdim: int
    cap: float

    kind = "mlstm"
    conv_c = 0
    taps = 1

    @staticmethod
    def of(m: MlstmSpec) -> "MlstmLayout":
        return MlstmLayout(m.heads, m.dim, m.vdim, m.gate_cap)

    @property
    def dk(self) -> int:
        return pad(self.dim)

    @property
    def dv(self) -> int:
        return pad(self.vdim)

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
    def n_gates(self) -> int:
        return 2 * self.heads

    @property
    def copies(self) -> int:
        """Copies of n and m a head keeps: one per slice of 32 value columns, so that no two blocks share one."""
        return (self.dv + 31) // 32

    @property
    def norm_groups(self) -> int:
        return self.heads

    @property
    def n_out(self) -> int:
        return pad(self.heads * self.dv, 64)

    @property
    def state_floats(self) -> int:
        """``S [heads, dk, dv]``, then the key sum ``n [heads, copies, dk]`` and the running maximum ``m [heads, copies]``."""
        return pad(self.heads * (self.dk * self.dv + self.copies * (self.dk + 1)), 4)


_LAYOUTS = {LatentAttnSpec: LatentLayout, Mamba2Spec: MambaLayout, MlstmSpec: MlstmLayout}


def layout_of(mixer):
    return _LAYOUTS[type(mixer)].of(mixer)


def layouts(cfg) -> Tuple[object, ...]:
    return tuple(layout_of(l.mixer) for l in cfg.layers)


def state_layouts(cfg) -> Tuple[object, ...]:
    """Layouts of the recurrent layers, in the order of their states."""
    return tuple(layout_of(m) for m in cfg.recurrent_mixers)


def side_width(cfg) -> int:
    """Columns between a token side input's two projections."""
    return pad(cfg.side_dim, 64)


def side_stride(cfg) -> int:
    """Columns of one layer in the served side embedding."""
    return pad(cfg.side_dim, 8)


# ---- checkpoint ----------------------------------------------------------------------------------------------
def _mixer_shapes(m, p: str, h: int) -> Dict[str, Tuple[int, ...]]:
    if isinstance(m, LatentAttnSpec):
        return {p + "dq": (m.q_rank, h), p + "dq.norm": (m.q_rank,), p + "uq": (m.heads * (m.dim + m.rot_dim), m.q_rank),
                p + "dkv": (m.kv_rank + m.rot_dim, h), p + "dkv.norm": (m.kv_rank,), p + "uk": (m.heads * m.dim, m.kv_rank),
                p + "uv": (m.heads * m.vdim, m.kv_rank), p + "g": (m.heads * m.vdim, h), p + "o": (h, m.heads * m.vdim)}
    if isinstance(m, Mamba2Spec):
        return {p + "in": (m.inner + m.channels + m.heads, h), p + "conv": (m.channels, m.conv), p + "conv.b": (m.channels,),
                p + "dt_bias": (m.heads,), p + "A_log": (m.heads,), p + "D": (m.heads,), p + "norm": (m.inner,), p + "o": (h, m.inner)}
    qk, v = m.heads * m.dim, m.heads * m.vdim
    return {p + "q": (qk, h), p + "k": (qk, h), p + "v": (v, h), p + "g": (v, h), p + "o": (h, v), p + "norm": (v,),
            p + "i": (m.heads, h), p + "i.b": (m.heads,), p + "f": (m.heads, h), p + "f.b": (m.heads,)}


def tensor_shapes(cfg) -> Dict[str, Tuple[int, ...]]:
    """Tensors of a checkpoint file (linear weights ``[out, in]``)."""
    h = cfg.hidden
    out: Dict[str, Tuple[int, ...]] = {"embed": (cfg.vocab, h), "side.embed": (cfg.vocab, cfg.n_layers * cfg.side_dim)}

    def norm(name: str) -> None:
        out[name] = out[name + ".b"] = (h,)
    for i, l in enumerate(cfg.layers):
        p = f"l{i}."
        norm(p + "norm1"), norm(p + "norm1b")
        out.update(_mixer_shapes(l.mixer, p + "mix.", h))
        if l.mlp is not None:
            norm(p + "norm2"), norm(p + "norm2b")
            out[p + "mlp.gate"] = out[p + "mlp.up"] = (l.mlp.ff, h)
            out[p + "mlp.down"] = (h, l.mlp.ff)
        out[p + "side.gate"], out[p + "side.proj"], out[p + "side.norm"] = (cfg.side_dim, h), (h, cfg.side_dim), (h,)
    norm("final.norm")
    out["head"] = (cfg.vocab, h)
    return out


def param_shapes(cfg) -> Dict[str, Tuple[Tuple[int, ...], str]]:
    """Served parameters: name -> (shape, ``"w"`` for the compute dtype or ``"f32"``)."""
    w = stream_width(cfg)
    out: Dict[str, Tuple[Tuple[int, ...], str]] = {
        "embed": ((cfg.vocab, w), "w"), "side_embed": ((cfg.vocab, cfg.n_layers * side_stride(cfg)), "w"),
        "lm_head": ((head_rows(cfg), w), "w"), "final_norm": ((2, w), "f32")}
    for i, b in enumerate(cfg.layers):
        l, p = layout_of(b.mixer), f"L{i}."
        out[p + "norm1"] = out[p + "norm1b"] = ((2, w), "f32")           # weight, bias
        out[p + "in"] = ((l.n_in + pad(l.n_gates, 8), w), "w")
        out[p + "o"] = ((w, l.n_out), "w")
        if l.kind == "latent":
            out[p + "q_norm"], out[p + "kv_norm"] = ((l.c0,), "f32"), ((l.kv,), "f32")
            out[p + "uq"] = ((l.heads * l.dq, l.c0), "w")
            out[p + "up"] = ((l.heads * (l.dk + l.dv), l.kv), "w")        # [key rows of every head ; value rows of every head]
        else:
            out[p + "norm"] = ((l.heads * l.dv,), "f32")
            out[p + "gate_b"] = ((l.n_gates,), "f32")
            if l.kind == "mamba2":
                out[p + "conv"], out[p + "conv_b"] = ((l.taps, l.conv_c), "f32"), ((l.conv_c,), "f32")
                out[p + "a_log"] = out[p + "skip"] = ((l.heads,), "f32")
        if b.mlp is not None:
            out[p + "norm2"] = out[p + "norm2b"] = ((2, w), "f32")
            out[p + "gate_up"] = ((2 * pad(b.mlp.ff, 64), w), "w")        # rows 2j = gate_j, 2j + 1 = up_j
            out[p + "down"] = ((w, pad(b.mlp.ff, 64)), "w")
        out[p + "side_gate"], out[p + "side_proj"] = ((side_width(cfg), w), "w"), ((w, side_width(cfg)), "w")
        out[p + "side_norm"] = ((1, w), "f32")
    return out
