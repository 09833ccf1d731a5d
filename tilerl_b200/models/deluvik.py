"""Deluvik: layers of softmax attention (with sinks, score caps, shared keys or short convolutions) and of attention beside a
gated linear recurrence, with dense or mixture-of-experts feed-forwards (no counterpart in the reference).

Stream ``x`` (fp32); a sublayer reads the stream itself and only its output is normalised::

    x = embed[token]
    for each layer:
        x = x + rms(mixer(x)) * w1
        x = x + rms(feed_forward(x)) * w2                where the layer has one
    logits = cap tanh(W_head (rms(x) * w) / cap)

Every sublayer ends in one op that normalises the branch, adds it to the stream and rounds the next projection's input
(:meth:`join`).  A layer's mixers share one input and one output projection: the recurrence's columns stand beside the
attention's, each scaled before it is rounded (:mod:`tilerl_b200.deluvik_layout`).

Parameter names: ``embed``, ``final_norm``, ``lm_head`` and per layer ``L{i}.norm1|in|o|q_norm|k_norm|conv|sink``,
``y_b|x_b|lru_conv|lru_conv_b|gates|gates_b|lam``, ``norm2|gate_up|down`` and ``router|router_b``.
"""
from __future__ import annotations

from typing import Dict, Iterator, Sequence, Tuple

import torch

from ..config import DeluvikConfig
from ..deluvik_layout import MoeLayout, layouts, param_shapes, state_layouts, tensor_shapes
from ..mixers import MoeSpec, ParallelSpec
from .fetotar import _cols, _rows
from .zinutar import Dims


# ---- checkpoint tensors <-> served parameters -----------------------------------------------------
def _attn_places(a, p: str, t: str, params, h: int):
    s, w_in = a.spec, params[p + "in"][:, :h]
    pieces = [("q", 0, s.heads, s.dim, a.dk)]
    if a.own:
        pieces.append(("k", a.k0, s.kv_heads, s.dim, a.dk))
        if not s.tied:
            pieces.append(("v", a.v0, s.kv_heads, s.vdim, a.dv))
    for n, r0, heads, d, dp in pieces:
        yield t + n, _rows(w_in, r0, heads, d, dp), None
        if n != "v":
            norm = params[f"{p}{n}_norm"]
            yield f"{t}{n}.norm", (norm[:d] if s.norm == "head" else norm.view(heads, dp)[:, :d]), None
        if s.conv:
            yield f"{t}{n}.conv", _rows(params[p + "conv"].t(), r0, heads, d, dp), None
    if s.sink:
        yield t + "sink", params[p + "sink"], None
    yield t + "o", _cols(params[p + "o"][:h], s.heads, s.vdim, a.dv), None


def _lru_places(l, p: str, t: str, params, h: int):
    r, m = l.lru, l.lru.spec
    w_in, b, k, pp = params[p + "in"][:, :h], m.blocks, m.part, r.pp
    vec = lambda n: params[p + n].view(b, pp)[:, :k]
    for j, n in enumerate(("y", "x")):
        yield t + n, _rows(w_in, l.attn.n_in + j * r.width, b, k, pp), None
        yield f"{t}{n}.b", vec(n + "_b"), None
    yield t + "conv", _rows(params[p + "lru_conv"].t(), 0, b, k, pp), None
    yield t + "conv.b", vec("lru_conv_b"), None
    for j, n in enumerate(("ra", "ri")):
        yield t + n, params[p + "gates"][:, j * pp:j * pp + k, :k], None
        yield f"{t}{n}.b", params[p + "gates_b"][:, j * pp:j * pp + k], None
    yield t + "lam", vec("lam"), None
    o = params[p + "o"][:h, l.attn.n_out:l.n_mid]
    yield t + "o", o.unflatten(1, (b, pp))[:, :, :k], None


def _glu_places(t: str, gate_up, down, rows):
    """``rows``: (first, last + 1) of the tensors' feed-forward dimension that lie here (None: all)."""
    yield t + "gate", gate_up[0::2], rows
    yield t + "up", gate_up[1::2], rows
    yield t + "down", down, None if rows is None else (*rows, 1)


def places(cfg: DeluvikConfig, params: Dict[str, torch.Tensor]) -> Iterator[Tuple[str, torch.Tensor, Tuple[int, ...]]]:
    """``(checkpoint tensor, view of a served parameter that holds it, (first, last + 1[, dimension]) of the tensor)``: the
    one table behind loading and saving."""
    h = cfg.hidden
    yield "embed", params["embed"][:, :h], None
    yield "head", params["lm_head"][:cfg.vocab, :h], None
    yield "final.norm", params["final_norm"][0, :h], None
    for i, (b, l) in enumerate(zip(cfg.layers, layouts(cfg))):
        s, p = f"l{i}.", f"L{i}."
        both = isinstance(b.mixer, ParallelSpec)
        yield s + "norm1", params[p + "norm1"][0, :h], None
        yield from _attn_places(l.attn, p, s + ("mix.left." if both else "mix."), params, h)
        if both:
            yield from _lru_places(l, p, s + "mix.right.", params, h)
        if b.mlp is None:
            continue
        yield s + "norm2", params[p + "norm2"][0, :h], None
        gu, dn = params[p + "gate_up"], params[p + "down"]
        if not isinstance(b.mlp, MoeSpec):
            yield from _glu_places(s + "mlp.", gu[:2 * b.mlp.ff, :h], dn[:h, :b.mlp.ff], None)
            continue
        m = MoeLayout(b.mlp)
        yield s + "mlp.router", params[p + "router"][:b.mlp.experts, :h], None
        yield s + "mlp.router.b", params[p + "router_b"][:b.mlp.experts], None
        for e in range(b.mlp.experts):
            yield from _glu_places(f"{s}mlp.e{e}.", gu[e, :2 * b.mlp.ff, :h], dn[e, :h, :b.mlp.ff], None)
        for j in range(m.pieces):
            lo, hi = j * m.ff, min((j + 1) * m.ff, b.mlp.shared)
            e = b.mlp.experts + j
            yield from _glu_places(s + "mlp.shared.", gu[e, :2 * (hi - lo), :h], dn[e, :h, :hi - lo], (lo, hi))


def _part(t: torch.Tensor, piece) -> torch.Tensor:
    if piece is None:
        return t
    return t.narrow(piece[2] if len(piece) > 2 else 0, piece[0], piece[1] - piece[0])


def pack(cfg: DeluvikConfig, get, device, dtype) -> Dict[str, torch.Tensor]:
    """Checkpoint tensors (``get(name)``) -> served parameters on ``device``."""
    params = {n: torch.zeros(s, dtype=dtype if k == "w" else torch.float32, device=device)
              for n, (s, k) in param_shapes(cfg).items()}
    want = tensor_shapes(cfg)
    for name, view, piece in places(cfg, params):
        t = get(name)
        if tuple(t.shape) != want[name]:
            raise ValueError(f"{name}: shape {tuple(t.shape)}, the configuration says {want[name]}")
        view.copy_(_part(t.to(device), piece).reshape(view.shape))
    return params


def unpack(cfg: DeluvikConfig, params: Dict[str, torch.Tensor]) -> Dict[str, torch.Tensor]:
    """Served parameters -> checkpoint tensors (the inverse of :func:`pack`)."""
    out: Dict[str, torch.Tensor] = {}
    shapes = tensor_shapes(cfg)
    for name, view, piece in places(cfg, params):
        if piece is None:
            out[name] = view.reshape(shapes[name])
        else:
            t = out.setdefault(name, torch.zeros(shapes[name], dtype=view.dtype, device=view.device))
            dst = _part(t, piece)
            dst.copy_(view.reshape(dst.shape))
    return out


def random_tensor(name: str, shape, g: torch.Generator, device="cpu") -> torch.Tensor:
    """One checkpoint tensor of a random-init model: projections N(0, 0.02), norms 1, biases and sinks 0, decays between 0.9 and
    0.999 at full gates."""
    leaf = name.split(".")[-1]
    if leaf.startswith("norm"):
        return torch.ones(shape, device=device)
    if leaf in ("b", "sink"):
        return torch.zeros(shape, device=device)
    if leaf == "lam":
        rate = -torch.log(torch.empty(shape, device=device).uniform_(0.9, 0.999, generator=g)) / 8.0
        return torch.log(torch.expm1(rate))
    return torch.randn(shape, generator=g, device=device) * (0.3 if leaf == "conv" else 0.02)


class DeluvikModel:
    tp, tp_rank = 1, 0

    def __init__(self, cfg: DeluvikConfig, params: Dict[str, torch.Tensor]):
        self.cfg, self.params = cfg, params
        self.dims = Dims(cfg.n_q_heads, cfg.n_kv_heads)
        self.layouts = layouts(cfg)
        self.moe = [MoeLayout(b.mlp) if isinstance(b.mlp, MoeSpec) else None for b in cfg.layers]
        self.caches = [cfg.cache_index(i) for i in range(cfg.n_layers)]
        states = state_layouts(cfg)
        find = lambda i, lru: next((j for j, s in enumerate(states) if s.layer == i and (s.state_floats > 0) == lru), None)
        self.lru_state = [find(i, True) for i in range(cfg.n_layers)]
        self.conv_state = [find(i, False) for i in range(cfg.n_layers)]
        # radians per position of every rotated pair (fp64: angles are reduced before they are rounded)
        self.freqs = [torch.tensor(cfg.attn(i).rot.frequencies(), dtype=torch.float64, device=params["embed"].device)
                      for i in range(cfg.n_layers)]
        self.lora: Dict[str, object] = {}
        self.weights_version = 0
        if params["lm_head"].is_cuda:      # library products accumulate in fp32 and read fp32 operands whole
            torch.backends.cuda.matmul.allow_bf16_reduced_precision_reduction = False
            torch.backends.cuda.matmul.allow_tf32 = False

    @property
    def act_dtype(self) -> torch.dtype:
        return self.params["lm_head"].dtype

    @classmethod
    def from_tensors(cls, cfg: DeluvikConfig, get, device="cpu", dtype=torch.float32) -> "DeluvikModel":
        return cls(cfg, pack(cfg, get, torch.device(device), dtype))

    @classmethod
    def build_random(cls, cfg: DeluvikConfig, seed: int = 0, device="cpu", *, act_dtype=torch.float32) -> "DeluvikModel":
        g = torch.Generator(device=device).manual_seed(seed)
        shapes = tensor_shapes(cfg)
        kept: Dict[str, torch.Tensor] = {}        # tensors served in several pieces are drawn once

        def get(name):
            if name in kept:
                return kept[name]
            t = random_tensor(name, shapes[name], g, device)
            if ".shared." in name:
                for k in [k for k in kept if not k.startswith(name.split(".shared.")[0])]:
                    del kept[k]
                kept[name] = t
            return t
        return cls.from_tensors(cfg, get, device, act_dtype)

    def tensors(self) -> Iterator[Tuple[str, torch.Tensor]]:
        yield from unpack(self.cfg, self.params).items()

    # ---- serving forward --------------------------------------------------------------------
    def _mix(self, i: int, h, batch, ops, kv_pool, state_pool):
        """The mixers of layer ``i`` up to their output projection's input."""
        P, p, l, c = self.params, f"L{i}.", self.layouts[i], self.caches[i]
        eps = self.cfg.norm_eps
        proj = ops.project(h, P[p + "in"])
        w = {k: P.get(p + k) for k in ("q_norm", "k_norm", "conv")}
        q, mid = ops.attn_prep(proj, l, w, self.freqs[i], batch, kv_pool, c, state_pool, self.conv_state[i], eps)
        ops.softmax_attention(q, mid, l.attn, P.get(p + "sink"), l.attn_scale, batch, kv_pool, c)
        if l.lru is not None:
            w = {k: P[p + k] for k in ("y_b", "x_b", "lru_conv", "lru_conv_b", "gates", "gates_b", "lam")}
            ops.lru_mix(proj, mid, l, w, batch, state_pool, self.lru_state[i])
        return mid

    def forward(self, batch, ops, kv_pool, state_pool, *, last_only: bool = True, aux_layers: Sequence[int] = (),
                return_hidden: bool = False, rows=None):
        """Logits (fp32) of each sequence's last token, of every token (``last_only=False``) or of the token
        rows listed in ``rows``.  ``aux_layers``: also return the stream after those layers."""
        cfg, P = self.cfg, self.params
        eps, n = cfg.norm_eps, cfg.hidden
        x, h = ops.embed_stream(P["embed"], batch.token_ids, 1.0, None, eps, n)
        taps = {}
        for i, b in enumerate(cfg.layers):
            p = f"L{i}."
            end = P["final_norm"] if i + 1 == cfg.n_layers else None      # else the stream itself is the next input
            y = ops.project_f32(self._mix(i, h, batch, ops, kv_pool, state_pool), P[p + "o"])
            h = ops.join(x, y, P[p + "norm1"], None if b.mlp is not None else end, eps, n)
            if self.moe[i] is not None:
                rows_y = ops.experts(h, P[p + "router"], P[p + "router_b"], P[p + "gate_up"], P[p + "down"], self.moe[i])
                h = ops.join_experts(x, rows_y, P[p + "norm2"], end, eps, n)
            elif b.mlp is not None:
                y = ops.project_f32(ops.glu(h, P[p + "gate_up"], b.mlp.act), P[p + "down"])
                h = ops.join(x, y, P[p + "norm2"], end, eps, n)
            if i in aux_layers:
                taps[i] = x[:, :n].clone()
        if rows is not None:
            hs = h[rows] if len(rows) else None
        else:
            hs = h[batch.last_idx.long()] if last_only and batch.n_tokens != batch.n_seqs else h
        logits = None if hs is None else ops.project_logits(hs, P["lm_head"], cfg.logit_cap)[..., :cfg.vocab]
        if aux_layers or return_hidden:
            return logits, x[:, :n], taps
        return logits

    def served_bytes(self) -> int:
        return sum(v.numel() * v.element_size() for v in self.params.values())
