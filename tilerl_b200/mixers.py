"""Sizes and constants of the mixers, feed-forwards and rotations that stream designs are put together from.

Every class is one mechanism with its constants as fields, checked on construction, and converts from and to the
dictionaries of a ``config.json``; a design's configuration lists them layer by layer.  No counterpart in the reference.
"""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Dict, Optional, Tuple


def take(d: Dict, known, where: str) -> Dict:
    """``d`` with exactly the keys ``known``; anything else is refused, so that nothing is silently left out."""
    if not isinstance(d, dict):
        raise ValueError(f"{where}: expected an object, got {d!r}")
    extra, lack = sorted(set(d) - set(known)), sorted(set(known) - set(d))
    if extra or lack:
        raise ValueError(f"{where}: " + "; ".join(([f"unknown keys {extra}"] if extra else []) + ([f"missing keys {lack}"] if lack else [])))
    return d


def _positive(what: str, *values) -> None:
    if min(values) <= 0:
        raise ValueError(f"{what}: sizes must be positive")


# ---- rotary positions ------------------------------------------------------------------------------------
@dataclass(frozen=True)
class YarnSpec:
    """Frequency scaling of a context extended ``factor`` times beyond ``original`` tokens: pairs that turn more than
    ``fast`` times over the original context keep their frequency, those below ``slow`` turns are slowed down by
    ``factor``, a linear ramp in between; cos and sin are multiplied by ``0.1 ln(factor) + 1``."""
    factor: float
    original: float
    fast: float
    slow: float

    def __post_init__(self) -> None:
        _positive("rotary scaling", self.factor, self.original, self.fast, self.slow)


@dataclass(frozen=True)
class RotarySpec:
    """Rotation of the first ``dims`` dimensions in neighbouring pairs (2i, 2i + 1)."""
    dims: int
    base: float
    scaling: Optional[YarnSpec] = None

    def __post_init__(self) -> None:
        if self.dims <= 0 or self.dims % 2 or self.base <= 1.0:
            raise ValueError(f"rotation needs an even number of dimensions and a base above 1: {self}")

    def frequencies(self) -> Tuple[float, ...]:
        """Radians per position of every pair."""
        plain = [self.base ** (-2.0 * i / self.dims) for i in range(self.dims // 2)]
        s = self.scaling
        if s is None:
            return tuple(plain)

        def dim_of(turns: float) -> float:      # (real-valued) dimension whose pair turns this often over `original`
            return self.dims * math.log(s.original / (2.0 * math.pi * turns)) / (2.0 * math.log(self.base))
        lo, hi = max(math.floor(dim_of(s.fast)), 0), min(math.ceil(dim_of(s.slow)), self.dims - 1)
        out = []
        for i, f in enumerate(plain):
            ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
            out.append(f / s.factor * ramp + f * (1.0 - ramp))
        return tuple(out)

    @property
    def amplitude(self) -> float:
        return 1.0 if self.scaling is None else 0.1 * math.log(self.scaling.factor) + 1.0

    @classmethod
    def from_json(cls, d: Dict, where: str) -> "RotarySpec":
        if "scaling" not in d or d["scaling"] is None:
            d = {k: v for k, v in d.items() if k != "scaling"}
            take(d, ("dims", "base"), where)
            return cls(int(d["dims"]), float(d["base"]))
        take(d, ("dims", "base", "scaling"), where)
        s = take(d["scaling"], ("factor", "original", "fast", "slow"), where + " scaling")
        return cls(int(d["dims"]), float(d["base"]),
                   YarnSpec(float(s["factor"]), float(s["original"]), float(s["fast"]), float(s["slow"])))

    def to_json(self) -> Dict:
        out: Dict = {"dims": self.dims, "base": self.base}
        if self.scaling is not None:
            s = self.scaling
            out["scaling"] = {"factor": s.factor, "original": s.original, "fast": s.fast, "slow": s.slow}
        return out


# ---- mixers ------------------------------------------------------------------------------------------------
@dataclass(frozen=True)
class LatentAttnSpec:
    """Softmax attention whose keys and values are linear maps of one cached latent of size ``kv_rank`` per token, plus
    one rotated key part of size ``rot_dim`` shared by all heads; queries go through a latent of size ``q_rank``.
    A query sees itself and the ``window - 1`` tokens before it; the output is gated by a sigmoid."""
    heads: int
    dim: int             # unrotated query / key dimensions per head
    rot_dim: int
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    window: int
    rot: RotarySpec

    type = "latent_attention"
    recurrent = False

    def __post_init__(self) -> None:
        _positive("latent attention", self.heads, self.dim, self.rot_dim, self.vdim, self.q_rank, self.kv_rank, self.window)
        if self.rot.dims > self.rot_dim:
            raise ValueError("more rotated dimensions than the rotated part has")

    @classmethod
    def from_json(cls, m: Dict, where: str) -> "LatentAttnSpec":
        take(m, ("heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank", "scale", "mask", "rot"), where)
        take(m["mask"], ("size",), where + " mask")
        return cls(int(m["heads"]), int(m["dim"]), int(m["rot_dim"]), int(m["vdim"]), int(m["q_rank"]), int(m["kv_rank"]),
                   float(m["scale"]), int(m["mask"]["size"]), RotarySpec.from_json(m["rot"], where + " rot"))

    def to_json(self) -> Dict:
        return {"heads": self.heads, "dim": self.dim, "rot_dim": self.rot_dim, "vdim": self.vdim, "q_rank": self.q_rank,
                "kv_rank": self.kv_rank, "scale": self.scale, "mask": {"size": self.window}, "rot": self.rot.to_json()}


@dataclass(frozen=True)
class Mamba2Spec:
    """State-space duality: per head a decayed sum of ``B x^T`` (``state`` x ``vdim``) read by ``C``; B and C are shared
    by the heads of a group, and x, B, C pass a short causal convolution of ``conv`` taps."""
    heads: int
    vdim: int
    state: int
    groups: int
    conv: int
    norm_groups: int

    type = "mamba2"
    recurrent = True

    def __post_init__(self) -> None:
        _positive("mamba2", self.heads, self.vdim, self.state, self.groups, self.conv, self.norm_groups)
        if self.heads % self.groups or (self.heads * self.vdim) % self.norm_groups:
            raise ValueError(f"mamba2: heads must divide into groups and inner width into norm groups: {self}")

    @property
    def inner(self) -> int:
        return self.heads * self.vdim

    @property
    def channels(self) -> int:
        return self.inner + 2 * self.groups * self.state

    @classmethod
    def from_json(cls, m: Dict, where: str) -> "Mamba2Spec":
        names = ("heads", "vdim", "state", "groups", "conv", "norm_groups")
        take(m, names, where)
        return cls(*(int(m[n]) for n in names))

    def to_json(self) -> Dict:
        return {n: getattr(self, n) for n in ("heads", "vdim", "state", "groups", "conv", "norm_groups")}


@dataclass(frozen=True)
class MlstmSpec:
    """Matrix memory with exponential gates: per head a decayed sum of ``k v^T`` (``dim`` x ``vdim``) and of ``k``,
    kept in range by a running maximum; gate pre-activations are soft-capped at ``gate_cap``."""
    heads: int
    dim: int
    vdim: int
    gate_cap: float

    type = "mlstm"
    recurrent = True

    def __post_init__(self) -> None:
        _positive("mlstm", self.heads, self.dim, self.vdim, self.gate_cap)

    @classmethod
    def from_json(cls, m: Dict, where: str) -> "MlstmSpec":
        take(m, ("heads", "dim", "vdim", "gate_cap"), where)
        return cls(int(m["heads"]), int(m["dim"]), int(m["vdim"]), float(m["gate_cap"]))

    def to_json(self) -> Dict:
        return {"heads": self.heads, "dim": self.dim, "vdim": self.vdim, "gate_cap": self.gate_cap}


MIXERS = {c.type: c for c in (LatentAttnSpec, Mamba2Spec, MlstmSpec)}


# ---- feed-forwards -----------------------------------------------------------------------------------------
@dataclass(frozen=True)
class ClampedGluSpec:
    """``W_down (g sigmoid(1.702 g) (u + 1))`` with ``g = min(W_gate h, limit)`` and ``u = W_up h`` clamped to
    ``[-limit, limit]``."""
    ff: int
    limit: float
    kind: str = "dense"

    def __post_init__(self) -> None:
        if self.kind != "dense":
            raise ValueError(f"unknown feed-forward kind {self.kind!r}")
        _positive("feed-forward", self.ff, self.limit)

    @classmethod
    def from_json(cls, f: Dict, where: str) -> "ClampedGluSpec":
        take(f, ("ff", "kind", "limit"), where)
        return cls(int(f["ff"]), float(f["limit"]), f["kind"])

    def to_json(self) -> Dict:
        return {"kind": self.kind, "ff": self.ff, "limit": self.limit}


@dataclass(frozen=True)
class LayerSpec:
    """One layer: a mixer and, unless ``mlp`` is None, a feed-forward after it."""
    mixer: object
    mlp: Optional[ClampedGluSpec] = None
