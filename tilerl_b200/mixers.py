"""Sizes and constants of the mixers, feed-forwards and rotations that stream designs are put together from.

Every class is one mechanism with its constants as fields, checked on construction, and converts from and to the
dictionaries of a ``config.json``; a design's configuration lists them layer by layer.  No counterpart in the reference.
"""
from __future__ import annotations

import math
from dataclasses import asdict, dataclass, fields
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
class BandScalingSpec:
    """Frequency scaling by wavelength bands: pairs that turn more than ``high`` times over ``original`` tokens keep their
    frequency, those that turn less than ``low`` times are slowed down by ``factor``, a linear blend in the number of turns in
    between."""
    factor: float
    low: float
    high: float
    original: float

    def __post_init__(self) -> None:
        _positive("rotary scaling", self.factor, self.low, self.high, self.original)
        if self.high < self.low:
            raise ValueError(f"rotary scaling: the bands overlap: {self}")

    def apply(self, f: float) -> float:
        turns = self.original * f / (2.0 * math.pi)
        if turns > self.high:
            return f
        if turns < self.low:
            return f / self.factor
        keep = (turns - self.low) / (self.high - self.low) if self.high > self.low else 1.0
        return (1.0 - keep) * f / self.factor + keep * f


@dataclass(frozen=True)
class RotarySpec:
    """Rotation of the first ``dims`` dimensions: in neighbouring pairs (2i, 2i + 1), or, with ``half``, of dimension i with
    dimension i + dims / 2."""
    dims: int
    base: float
    scaling: Optional[object] = None       # YarnSpec or BandScalingSpec
    half: bool = False

    def __post_init__(self) -> None:
        if self.dims <= 0 or self.dims % 2 or self.base <= 1.0:
            raise ValueError(f"rotation needs an even number of dimensions and a base above 1: {self}")

    def frequencies(self) -> Tuple[float, ...]:
        """Radians per position of every pair."""
        plain = [self.base ** (-2.0 * i / self.dims) for i in range(self.dims // 2)]
        s = self.scaling
        if s is None:
            return tuple(plain)
        if isinstance(s, BandScalingSpec):
            return tuple(s.apply(f) for f in plain)

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
        return 0.1 * math.log(self.scaling.factor) + 1.0 if isinstance(self.scaling, YarnSpec) else 1.0

    @classmethod
    def from_json(cls, d: Dict, where: str, scaling=YarnSpec, half: bool = False) -> "RotarySpec":
        """``scaling``: the class of the design's frequency scaling (used where the dictionary has one)."""
        if "scaling" not in d or d["scaling"] is None:
            d = {k: v for k, v in d.items() if k != "scaling"}
            take(d, ("dims", "base"), where)
            return cls(int(d["dims"]), float(d["base"]), None, half)
        take(d, ("dims", "base", "scaling"), where)
        names = [f.name for f in fields(scaling)]
        s = take(d["scaling"], names, where + " scaling")
        return cls(int(d["dims"]), float(d["base"]), scaling(*(float(s[n]) for n in names)), half)

    def to_json(self) -> Dict:
        out: Dict = {"dims": self.dims, "base": self.base}
        if self.scaling is not None:
            out["scaling"] = asdict(self.scaling)
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


@dataclass(frozen=True)
class SoftmaxAttnSpec:
    """Causal softmax attention of ``heads`` query heads over ``kv_heads`` key / value heads (contiguous groups).  Queries and
    keys are RMS-normalised with a weight, over the whole projection (``norm`` "all") or per head ("head"), or not ("none"),
    then rotated.  Optional: a ``window`` (a query sees itself and the ``window - 1`` tokens before it), a soft cap on scores
    (``cap``), a learned ``sink`` per head in the denominator, a short convolution of ``conv`` taps on every projection, values
    that are the projected keys (``tied``), keys and values of an earlier layer (``kv_from``), a ``bias`` on every projection,
    values that are ``turned`` by their position over the whole head and whose weighted sum is turned back by the query's."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot: RotarySpec
    norm: str = "all"
    window: Optional[int] = None
    cap: Optional[float] = None
    sink: bool = False
    conv: int = 0
    tied: bool = False
    kv_from: Optional[int] = None
    bias: bool = False
    turned: bool = False

    type = "attention"
    recurrent = False

    def __post_init__(self) -> None:
        _positive("attention", self.heads, self.kv_heads, self.dim, self.vdim)
        if self.heads % self.kv_heads:
            raise ValueError(f"attention needs heads a multiple of kv_heads: {self}")
        if self.rot.dims > self.dim:
            raise ValueError("more rotated dimensions than a head has")
        if self.norm not in ("all", "head", "none") or self.conv < 0 or (self.window is not None and self.window < 1) or \
                (self.cap is not None and self.cap <= 0):
            raise ValueError(f"attention: {self}")
        if self.tied and (self.dim != self.vdim or self.kv_from is not None):
            raise ValueError("values that are the keys have their size and their layer")
        if self.turned and (self.tied or not self.rot.half or self.vdim % 2):
            raise ValueError("turned values have an even size, are not the keys and turn in halves")

    def value_frequencies(self) -> Tuple[float, ...]:
        """Radians per position of every pair of a turned value (never scaled)."""
        return RotarySpec(self.vdim, self.rot.base).frequencies()

    @property
    def channels(self) -> int:
        """Columns of the layer's projections."""
        own = 0 if self.kv_from is not None else self.kv_heads * (self.dim + (0 if self.tied else self.vdim))
        return self.heads * self.dim + own

    def same_keys(self, other: "SoftmaxAttnSpec") -> bool:
        """The keys and values that ``other`` caches are what this layer reads."""
        return (self.heads, self.kv_heads, self.dim, self.vdim, self.rot) == (other.heads, other.kv_heads, other.dim, other.vdim, other.rot)

    @classmethod
    def from_json(cls, m: Dict, where: str, *, norm: str, half: bool, capped: bool = False, windowed: bool = False, conv: bool = False,
                  sink: bool = False, tied: bool = False, bias: bool = False, turned: bool = False) -> "SoftmaxAttnSpec":
        """The keyword arguments say which of the optional parts the design's mixer has."""
        m = dict(m)
        source = m.pop("kv_from", None) if conv else None
        take(m, ("heads", "kv_heads", "dim", "vdim", "scale", "rot") + capped * ("softcap",) + windowed * ("mask",) + conv * ("conv",), where)
        if windowed:
            take(m["mask"], ("size",), where + " mask")
        return cls(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), float(m["scale"]),
                   RotarySpec.from_json(m["rot"], where + " rot", BandScalingSpec, half), norm, int(m["mask"]["size"]) if windowed else None,
                   float(m["softcap"]) if capped else None, sink, int(m["conv"]) if conv else 0, tied, None if source is None else int(source),
                   bias, turned)

    def to_json(self) -> Dict:
        out: Dict = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "scale": self.scale,
                     "rot": self.rot.to_json()}
        for name, value in (("softcap", self.cap), ("conv", self.conv or None), ("kv_from", self.kv_from),
                            ("mask", None if self.window is None else {"size": self.window})):
            if value is not None:
                out[name] = value
        return out


@dataclass(frozen=True)
class LruSpec:
    """Gated linear recurrence of ``width`` channels (De et al., Griffin): a branch through a short convolution of ``conv``
    taps whose two gates are block-diagonal maps (``blocks`` equal parts), times a gelu branch."""
    width: int
    blocks: int
    conv: int

    def __post_init__(self) -> None:
        _positive("linear recurrence", self.width, self.blocks, self.conv)
        if self.width % self.blocks:
            raise ValueError(f"linear recurrence: the width must divide into the blocks: {self}")

    @property
    def part(self) -> int:
        return self.width // self.blocks

    @classmethod
    def from_json(cls, m: Dict, where: str) -> "LruSpec":
        take(m, ("width", "blocks", "conv"), where)
        return cls(int(m["width"]), int(m["blocks"]), int(m["conv"]))

    def to_json(self) -> Dict:
        return asdict(self)


@dataclass(frozen=True)
class LightningSpec:
    """Linear attention whose per-head sum of ``k v^T`` (``dim`` x ``vdim``) fades by a fixed factor a token (``decay``, one per
    head); queries, keys and values pass silu, the heads' outputs one RMS norm together and a sigmoid gate."""
    heads: int
    dim: int
    vdim: int
    decay: Tuple[float, ...]

    type = "lightning"
    recurrent = True

    def __post_init__(self) -> None:
        object.__setattr__(self, "decay", tuple(float(d) for d in self.decay))
        _positive("lightning", self.heads, self.dim, self.vdim)
        if len(self.decay) != self.heads or not all(0.0 < d <= 1.0 for d in self.decay):
            raise ValueError(f"lightning: one decay in (0, 1] per head: {self}")

    @classmethod
    def from_json(cls, m: Dict, where: str) -> "LightningSpec":
        take(m, ("heads", "dim", "vdim", "decay"), where)
        return cls(int(m["heads"]), int(m["dim"]), int(m["vdim"]), tuple(m["decay"]))

    def to_json(self) -> Dict:
        return {"heads": self.heads, "dim": self.dim, "vdim": self.vdim, "decay": list(self.decay)}


@dataclass(frozen=True)
class ChannelDeltaSpec:
    """Delta rule with one decay per key channel: per head a sum of ``k u^T`` (``dim`` x ``vdim``) whose rows fade on their own,
    ``u`` being the part of the value that the faded sum does not hold yet, scaled by a gate.  Queries and keys (``kv_heads``
    heads, shared by contiguous groups) and values pass a short convolution of ``conv`` taps; the decays and the output gate
    are maps of low rank (``decay_rank``, ``gate_rank``)."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int
    decay_rank: int
    gate_rank: int

    type = "channel_delta"
    recurrent = True

    def __post_init__(self) -> None:
        _positive("channel delta", self.heads, self.kv_heads, self.dim, self.vdim, self.conv, self.decay_rank, self.gate_rank)
        if self.heads % self.kv_heads:
            raise ValueError(f"channel delta needs heads a multiple of kv_heads: {self}")

    @classmethod
    def from_json(cls, m: Dict, where: str, decay_rank: int, gate_rank: int) -> "ChannelDeltaSpec":
        """The ranks are no part of the dictionary: a checkpoint's tensors have them."""
        names = ("heads", "kv_heads", "dim", "vdim", "conv")
        take(m, names, where)
        return cls(*(int(m[n]) for n in names), int(decay_rank), int(gate_rank))

    def to_json(self) -> Dict:
        return {n: getattr(self, n) for n in ("heads", "kv_heads", "dim", "vdim", "conv")}


@dataclass(frozen=True)
class ParallelSpec:
    """Two mixers that read the same row: ``left_scale`` attention + ``right_scale`` recurrence."""
    left: SoftmaxAttnSpec
    right: LruSpec
    left_scale: float
    right_scale: float


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
class GluSpec:
    """``W_down (act(W_gate h) * (W_up h))``."""
    ff: int
    act: str                  # "gelu" (its tanh form) or "silu"
    kind = "dense"

    def __post_init__(self) -> None:
        _positive("feed-forward", self.ff)
        if self.act not in ("gelu", "silu"):
            raise ValueError(f"unknown activation {self.act!r}")

    @classmethod
    def from_json(cls, f: Dict, where: str, act: str) -> "GluSpec":
        take(f, ("ff", "kind"), where)
        return cls(int(f["ff"]), act)

    def to_json(self) -> Dict:
        return {"kind": self.kind, "ff": self.ff}


@dataclass(frozen=True)
class DenseSpec:
    """``W_down act(W_up h)``."""
    ff: int
    act: str                  # "gelu" (its tanh form), "gelu_erf" or "silu"
    kind = "dense"

    def __post_init__(self) -> None:
        _positive("feed-forward", self.ff)
        if self.act not in ("gelu", "gelu_erf", "silu"):
            raise ValueError(f"unknown activation {self.act!r}")

    @classmethod
    def from_json(cls, f: Dict, where: str, act: str) -> "DenseSpec":
        take(f, ("ff", "kind"), where)
        return cls(int(f["ff"]), act)

    def to_json(self) -> Dict:
        return {"kind": self.kind, "ff": self.ff}


@dataclass(frozen=True)
class RouterSpec:
    """Choice by scores that are the softmax over all outputs, plus a learned correction that the weights (scores times ``scale``)
    do not see.  Outputs form ``groups`` equal groups of neighbours, of which the ``keep`` with the largest choice score can be
    chosen from; the last ``identity`` outputs stand for the input itself."""
    scale: float = 1.0
    identity: int = 0
    groups: int = 1
    keep: int = 1

    MAX_GROUPS = 64

    def check(self, experts: int, top: int) -> None:
        n = experts + self.identity
        if self.identity < 0 or not 1 <= self.keep <= self.groups <= self.MAX_GROUPS or n % self.groups or n // self.groups * self.keep < top:
            raise ValueError(f"router: {experts} experts, {top} chosen: {self}")


@dataclass(frozen=True)
class MoeSpec:
    """``experts`` feed-forwards of width ``ff`` (``gated`` or plain), of which a token uses ``top``; ``shared`` (0: none) is the width
    of one that every token uses, with weight one or (``shared_gate``) a sigmoid of the token's own.  Without ``router``, the
    experts with the largest router logits are chosen, weighted by the softmax over those."""
    ff: int
    experts: int
    top: int
    shared: int = 0
    act: str = "silu"
    gated: bool = True
    shared_gate: bool = False
    router: Optional[RouterSpec] = None
    kind = "moe"

    def __post_init__(self) -> None:
        _positive("experts", self.ff, self.experts, self.top)
        if self.top > self.outputs or self.shared < 0 or self.act not in (("gelu", "silu") if self.gated else ("gelu", "gelu_erf", "silu")):
            raise ValueError(f"experts: {self}")
        if self.router is not None:
            self.router.check(self.experts, self.top)

    @property
    def outputs(self) -> int:
        """Outputs of the router: experts, then the input itself."""
        return self.experts + (self.router.identity if self.router else 0)

    @classmethod
    def from_json(cls, f: Dict, where: str) -> "MoeSpec":
        f = take({"shared": None, **f}, ("kind", "expert", "router", "shared"), where)
        take(f["expert"], ("ff",), where + " expert"), take(f["router"], ("experts", "top"), where + " router")
        if f["shared"] is not None:
            take(f["shared"], ("ff",), where + " shared")
        return cls(int(f["expert"]["ff"]), int(f["router"]["experts"]), int(f["router"]["top"]),
                   0 if f["shared"] is None else int(f["shared"]["ff"]))

    @classmethod
    def from_json_grouped(cls, f: Dict, where: str, act: str) -> "MoeSpec":
        """Plain experts behind a :class:`RouterSpec`, the shared one gated."""
        f = take({"shared": None, **f}, ("kind", "expert", "router", "shared"), where)
        r = take({"identity": 0, "groups": {"count": 1, "keep": 1}, **f["router"]}, ("experts", "top", "scale", "identity", "groups"), where + " router")
        take(f["expert"], ("ff",), where + " expert"), take(r["groups"], ("count", "keep"), where + " groups")
        if f["shared"] is not None:
            take(f["shared"], ("ff",), where + " shared")
        return cls(int(f["expert"]["ff"]), int(r["experts"]), int(r["top"]), 0 if f["shared"] is None else int(f["shared"]["ff"]), act, False,
                   f["shared"] is not None, RouterSpec(float(r["scale"]), int(r["identity"]), int(r["groups"]["count"]), int(r["groups"]["keep"])))

    def to_json(self) -> Dict:
        r = self.router
        out: Dict = {"kind": self.kind, "expert": {"ff": self.ff}, "router": {"experts": self.experts, "top": self.top}}
        if r is not None:
            out["router"].update(scale=r.scale, identity=r.identity, groups={"count": r.groups, "keep": r.keep})
        if self.shared:
            out["shared"] = {"ff": self.shared}
        return out


@dataclass(frozen=True)
class LayerSpec:
    """One layer: a mixer and, unless ``mlp`` is None, a feed-forward after it.  ``weights_of``: the earlier layer whose parameters
    it uses (with a cache or state of its own)."""
    mixer: object
    mlp: Optional[object] = None
    weights_of: Optional[int] = None
