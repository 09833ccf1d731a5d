"""Tobadra: layers of windowed attention over turned values, lightning attention or a per-channel delta rule, with dense or
grouped-expert feed-forwards; every branch is gated by its input and normed before it joins the stream (no counterpart in the
reference).

Stream ``x`` (fp32), ``rms`` with a weight everywhere, ``conv`` a causal convolution over time per channel::

    x = rms(embed[token])
    for each layer:
        h = rms(x);  x = x + rms(mixer(h + conv(h)) * sigmoid(W_rg1 h + b))
        h = rms(x);  x = x + rms(feed_forward(h) * sigmoid(W_rg2 h + b))          where the layer has one
    logits = scale * embed . rms(x)

The rows of a branch's gate stand behind those of the mixer's input projection (which read the convolved row), behind a dense
feed-forward's up rows, or behind the router's; one op gates and norms a branch, adds it to the stream, norms the next input and, in
decode ticks, convolves it (:meth:`gated_join`).

Parameter names: ``embed``, ``embed_norm``, ``final_norm`` and per layer with parameters of its own
``L{i}.norm1|norm1b|canon|in|rg1_b|o``, the mixer's (``qkv_b|o_b``, ``norm``, ``conv|low|dt_bias|a_log``),
``norm2|norm2b|rg2_b|up|down`` and ``router|correction``.
"""
from __future__ import annotations

import math
from typing import Dict, Iterator, Sequence, Tuple

import torch

from ..config import TobadraConfig
from ..deluvik_layout import LayerLayout, MoeLayout
from ..mixers import MoeSpec
from ..tobadra_layout import gate_rows, layout_of, layouts, param_shapes, router_rows, state_layouts, stream_width, tensor_shapes
from .deluvik import _part
from .fetotar import _cols, _rows
from .zinutar import Dims


# ---- checkpoint tensors <-> served parameters -----------------------------------------------------
def _halves(dst: torch.Tensor, r0: int, heads: int, d: int, dp: int) -> torch.Tensor:
    """View ``[heads, 2, d / 2, columns]`` of the true rows of heads whose halves sit at the halves of ``dp`` padded rows."""
    return dst[r0:r0 + heads * dp].view(heads, 2, dp // 2, -1)[:, :, :d // 2]


def _mixer_places(l, p: str, t: str, params, h: int):
    w_in, w_o = params[p + "in"][:, :h], params[p + "o"][:h]
    if isinstance(l, LayerLayout):
        a, s, bias = l.attn, l.attn.spec, params[p + "qkv_b"][:, None]
        for n, rows, r0, heads, d, dp in (("q", _rows, 0, s.heads, s.dim, a.dk), ("k", _rows, a.k0, s.kv_heads, s.dim, a.dk),
                                          ("v", _halves, a.v0, s.kv_heads, s.vdim, a.dv)):
            yield t + n, rows(w_in, r0, heads, d, dp), None
            yield f"{t}{n}.b", rows(bias, r0, heads, d, dp), None
        yield t + "o", w_o[:, :a.n_out].view(h, s.heads, 2, a.dv // 2)[..., :s.vdim // 2], None
        yield t + "o.b", params[p + "o_b"][:h], None
        return
    s = l.spec
    yield t + "o", _cols(w_o, l.heads, l.vdim, l.dv), None
    if l.kind == "lightning":
        for n, r0, d, dp in (("q", 0, s.dim, l.dk), ("k", l.k0, s.dim, l.dk), ("v", l.v0, s.vdim, l.dv), ("g", l.g0, s.vdim, l.dv)):
            yield t + n, _rows(w_in, r0, l.heads, d, dp), None
        yield t + "norm", params[p + "norm"].view(l.heads, l.dv)[:, :l.vdim], None
        return
    for n, r0, heads, d, dp in (("q", 0, l.kv_heads, s.dim, l.dk), ("k", l.k0, l.kv_heads, s.dim, l.dk), ("v", l.v0, l.heads, s.vdim, l.dv)):
        yield t + n, _rows(w_in, r0, heads, d, dp), None
        yield f"{t}{n}.conv", _rows(params[p + "conv"].t(), r0, heads, d, dp), None
    yield t + "a1", w_in[l.a0:l.a0 + s.decay_rank], None
    yield t + "g1", w_in[l.g0:l.g0 + s.gate_rank], None
    yield t + "b", w_in[l.n_in:l.n_in + l.heads], None
    yield t + "a2", _rows(params[p + "low"][:, :s.decay_rank], l.n_low, l.heads, s.dim, l.dk), None
    yield t + "g2", _rows(params[p + "low"][:, :s.gate_rank], 0, l.heads, s.vdim, l.dv), None
    yield t + "dt_bias", params[p + "dt_bias"].view(l.heads, l.dk)[:, :s.dim], None
    yield t + "A_log", params[p + "a_log"], None
    yield t + "norm", params[p + "norm"][:l.vdim], None


def _ff_places(b, p: str, t: str, params, h: int):
    """(tensor, view, piece) of a feed-forward, and the first row of the branch's gate in its first projection."""
    up, down = params[p + "up"], params[p + "down"]
    if not isinstance(b, MoeSpec):
        yield t + "up", up[:b.ff, :h], None
        yield t + "down", down[:h, :b.ff], None
        return
    m = MoeLayout(b)
    yield t + "router", params[p + "router"][:b.outputs, :h], None
    yield t + "correction", params[p + "correction"][:b.outputs], None
    for e in range(b.experts):
        yield f"{t}e{e}.up", up[e, :b.ff, :h], None
        yield f"{t}e{e}.down", down[e, :h, :b.ff], None
    for j in range(m.pieces):
        lo, hi, e = j * m.ff, min((j + 1) * m.ff, b.shared), b.experts + j
        yield t + "shared.up", up[e, :hi - lo, :h], (lo, hi)
        yield t + "shared.down", down[e, :h, :hi - lo], (lo, hi, 1)
    if b.shared:
        yield t + "shared.sg", params[p + "router"][b.outputs:b.outputs + 1, :h], None


def places(cfg: TobadraConfig, params: Dict[str, torch.Tensor]) -> Iterator[Tuple[str, torch.Tensor, Tuple[int, ...]]]:
    """``(checkpoint tensor, view of a served parameter that holds it, (first, last + 1[, dimension]) of the tensor)``: the
    one table behind loading and saving."""
    h, w = cfg.hidden, stream_width(cfg)
    yield "embed", params["embed"][:cfg.vocab, :h], None
    yield "embed.norm", params["embed_norm"][0, :h], None
    yield "final.norm", params["final_norm"][0, :h], None
    for i in cfg.owners:
        b, s, p = cfg.layers[i], f"l{i}.", f"L{i}."
        gates = [("1", "in")] if b.mlp is None else [("1", "in"), ("2", "router" if isinstance(b.mlp, MoeSpec) else "up")]
        for n, at in gates:
            for leaf in ("norm" + n, f"norm{n}b"):
                yield s + leaf, params[p + leaf][0, :h], None
            yield f"{s}rg{n}", params[p + at][-w:][:h, :h], None
            yield f"{s}rg{n}.b", params[f"{p}rg{n}_b"][:h], None
        yield s + "canon1", params[p + "canon"].t()[:h], None
        yield from _mixer_places(layout_of(b.mixer), p, s + "mix.", params, h)
        if b.mlp is not None:
            yield from _ff_places(b.mlp, p, s + "mlp.", params, h)


def pack(cfg: TobadraConfig, get, device, dtype) -> Dict[str, torch.Tensor]:
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


def unpack(cfg: TobadraConfig, params: Dict[str, torch.Tensor]) -> Dict[str, torch.Tensor]:
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
    """One checkpoint tensor of a random-init model: projections N(0, 0.02), norms 1, biases 0, decays with A in 1..16 and small steps."""
    leaf = name.split(".")[-1]
    if leaf.startswith("norm"):
        return torch.ones(shape, device=device)
    if leaf in ("b", "correction") and len(shape) == 1:
        return torch.zeros(shape, device=device)
    if leaf == "A_log":
        return torch.log(torch.empty(shape, device=device).uniform_(1.0, 16.0, generator=g))
    if leaf == "dt_bias":
        return torch.empty(shape, device=device).uniform_(-6.0, -2.0, generator=g)
    return torch.randn(shape, generator=g, device=device) * (0.3 if leaf in ("conv", "canon1") else 0.02)


class TobadraModel:
    tp, tp_rank = 1, 0

    def __init__(self, cfg: TobadraConfig, params: Dict[str, torch.Tensor]):
        self.cfg, self.params = cfg, params
        dev = params["embed"].device
        self.dims = Dims(cfg.n_q_heads, cfg.n_kv_heads)
        self.layouts = layouts(cfg)
        self.moe = [MoeLayout(b.mlp) if isinstance(b.mlp, MoeSpec) else None for b in cfg.layers]
        states = state_layouts(cfg)
        recurrent = [i for i, l in enumerate(cfg.layers) if l.mixer.recurrent]
        self.states = [cfg.n_layers + recurrent.index(i) if i in recurrent else None for i in range(cfg.n_layers)]
        assert len(states) == cfg.n_layers + len(recurrent)
        self.final = params["final_norm"] * cfg.logit_scale
        f64 = lambda f: torch.tensor(f, dtype=torch.float64, device=dev)
        # what follows from the configuration or repeats a parameter: radians per position of every rotated pair (fp64: angles are
        # reduced before they are rounded), logarithms of fixed decays, a head's norm weight once per head
        self.freqs, self.value_freqs, self.log_decay, self.head_norm = [], [], [], []
        for i, (b, l) in enumerate(zip(cfg.layers, self.layouts)):
            m, attn, norm = b.mixer, not b.mixer.recurrent, params.get(f"L{cfg.source(i)}.norm")
            self.freqs.append(f64(m.rot.frequencies()) if attn else None)
            # (pairs of the padded head: those past the true ones hold zeros and do not turn)
            self.value_freqs.append(f64(m.value_frequencies() + (0.0,) * ((l.attn.dv - m.vdim) // 2)) if attn else None)
            self.log_decay.append(torch.tensor([math.log(d) for d in m.decay], dtype=torch.float32, device=dev) if m.type == "lightning" else None)
            self.head_norm.append(None if attn else norm if m.type == "lightning" else norm.repeat(m.heads))
        self.lora: Dict[str, object] = {}
        self.weights_version = 0
        if params["embed"].is_cuda:        # library products accumulate in fp32 and read fp32 operands whole
            torch.backends.cuda.matmul.allow_bf16_reduced_precision_reduction = False
            torch.backends.cuda.matmul.allow_tf32 = False

    @property
    def act_dtype(self) -> torch.dtype:
        return self.params["embed"].dtype

    @classmethod
    def from_tensors(cls, cfg: TobadraConfig, get, device="cpu", dtype=torch.float32) -> "TobadraModel":
        return cls(cfg, pack(cfg, get, torch.device(device), dtype))

    @classmethod
    def build_random(cls, cfg: TobadraConfig, seed: int = 0, device="cpu", *, act_dtype=torch.float32) -> "TobadraModel":
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
    def _mix(self, i: int, p: str, h, hc, batch, ops, kv_pool, state_pool):
        """The mixer of layer ``i`` up to its output projection's input, and its branch's gate before the sigmoid."""
        P, l, eps = self.params, self.layouts[i], self.cfg.norm_eps
        if isinstance(l, LayerLayout):
            c = self.cfg.cache_index(i)
            proj, _, z = ops.project_in(h, hc, P[p + "in"], l.n_in, 0)
            q, mid, turn = ops.turned_prep(proj, l, P[p + "qkv_b"], self.freqs[i], self.value_freqs[i], batch, kv_pool, c)
            ops.softmax_attention(q, mid, l.attn, None, 1.0, batch, kv_pool, c, turn)
            return mid, z
        if l.kind == "lightning":
            proj, _, z = ops.project_in(h, hc, P[p + "in"], l.n_in, 0, l.g0, "silu")
            return ops.lightning_mix(proj, self.log_decay[i], self.head_norm[i], l, batch, state_pool, self.states[i], eps), z
        proj, gates, z = ops.project_in(h, hc, P[p + "in"], l.n_in, gate_rows(l))
        w = {k: P[p + k] for k in ("conv", "low", "dt_bias", "a_log")}
        return ops.delta_mix(proj, gates, w, self.head_norm[i], l, batch, state_pool, self.states[i], eps), z

    def forward(self, batch, ops, kv_pool, state_pool, *, last_only: bool = True, aux_layers: Sequence[int] = (),
                return_hidden: bool = False, rows=None):
        """Logits (fp32) of each sequence's last token, of every token (``last_only=False``) or of the token
        rows listed in ``rows``.  ``aux_layers``: also return the stream after those layers."""
        cfg, P = self.cfg, self.params
        eps, n = cfg.norm_eps, cfg.hidden
        conv = lambda i: (P[f"L{cfg.source(i)}.canon"], batch, state_pool, i) if i < cfg.n_layers else None
        norm1 = lambda i: P[f"L{cfg.source(i)}.norm1"] if i < cfg.n_layers else self.final
        x, h, hc = ops.embed_normed(P["embed"], cfg.vocab, batch.token_ids, P["embed_norm"], norm1(0), eps, n, conv(0))
        taps = {}
        for i, b in enumerate(cfg.layers):
            p = f"L{cfg.source(i)}."
            mid, z = self._mix(i, p, h, hc, batch, ops, kv_pool, state_pool)
            y = ops.project_f32(mid, P[p + "o"])
            follow = (P[p + "norm2"], None) if b.mlp is not None else (norm1(i + 1), conv(i + 1))
            h, hc = ops.gated_join(x, y, P.get(p + "o_b"), z, P[p + "rg1_b"], P[p + "norm1b"], follow[0], eps, n, follow[1])
            if b.mlp is not None:
                last = (P[p + "norm2b"], norm1(i + 1), eps, n, conv(i + 1))
                if self.moe[i] is not None:
                    zr = ops.project_f32(h, P[p + "router"], "router")
                    branch = ops.routed_experts(h, zr, P[p + "correction"], P[p + "up"], P[p + "down"], self.moe[i])
                    h, hc = ops.gated_join_experts(x, branch, h, zr[:, router_rows(b.mlp):], P[p + "rg2_b"], *last)
                else:
                    mid, z = ops.up_act(h, P[p + "up"], P[p + "down"].shape[1], b.mlp.act)
                    h, hc = ops.gated_join(x, ops.project_f32(mid, P[p + "down"]), None, z, P[p + "rg2_b"], *last)
            if i in aux_layers:
                taps[i] = x[:, :n].clone()
        if rows is not None:
            hs = h[rows] if len(rows) else None
        else:
            hs = h[batch.last_idx.long()] if last_only and batch.n_tokens != batch.n_seqs else h
        logits = None if hs is None else ops.project_logits(hs, P["embed"])[..., :cfg.vocab]
        if aux_layers or return_hidden:
            return logits, x[:, :n], taps
        return logits

    def served_bytes(self) -> int:
        return sum(v.numel() * v.element_size() for v in self.params.values())
