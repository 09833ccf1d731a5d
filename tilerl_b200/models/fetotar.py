"""Fetotar: sandwich-normed layers of latent attention, Mamba-2 or mLSTM, with a per-layer token input (no counterpart
in the reference).

Stream ``x`` (fp32), ``LN`` a layer norm with weight and bias::

    x = embed[token] * embed_scale
    for each layer:
        x = x + LN(mixer(LN(x)))
        x = x + LN(W_down glu(W_gate LN(x), W_up LN(x)))                where the layer has a feed-forward
        x = x + rms(W_proj (gelu(W_side x) * side[token, layer])) * w
    logits = W_head LN(x)

Every sublayer ends in one op that normalises the branch, adds it to the stream and forms the next projection's input
(:meth:`join`); mixers are described by their layouts (:mod:`tilerl_b200.fetotar_layout`).

Parameter names: ``embed``, ``side_embed``, ``final_norm``, ``lm_head`` and per layer ``L{i}.norm1|norm1b|in|o``, the
mixer's own (``q_norm|kv_norm|uq|up``, ``norm|gate_b`` and ``conv|conv_b|a_log|skip``), ``norm2|norm2b|gate_up|down`` and
``side_gate|side_proj|side_norm``.
"""
from __future__ import annotations

from typing import Dict, Iterator, Sequence, Tuple

import torch

from ..config import FetotarConfig
from ..fetotar_layout import layouts, param_shapes, side_stride, tensor_shapes
from .zinutar import Dims


# ---- checkpoint tensors <-> served parameters -----------------------------------------------------
def _rows(dst: torch.Tensor, r0: int, heads: int, d: int, dp: int) -> torch.Tensor:
    """View ``[heads, d, columns]`` of the true rows of ``heads`` heads padded from ``d`` to ``dp`` rows."""
    return dst[r0:r0 + heads * dp].view(heads, dp, -1)[:, :d]


def _cols(dst: torch.Tensor, heads: int, d: int, dp: int) -> torch.Tensor:
    """View ``[rows, heads, d]`` of the true columns of ``heads`` heads padded from ``d`` to ``dp`` columns."""
    return dst[:, :heads * dp].view(dst.shape[0], heads, dp)[:, :, :d]


def places(cfg: FetotarConfig, params: Dict[str, torch.Tensor]) -> Iterator[Tuple[str, torch.Tensor, Tuple[int, int]]]:
    """``(checkpoint tensor, view of a served parameter that holds it, (first, last + 1 row of the tensor))``: the one
    table behind loading and saving."""
    h, sd = cfg.hidden, cfg.side_dim
    yield "embed", params["embed"][:, :h], None
    yield "side.embed", params["side_embed"].view(cfg.vocab, cfg.n_layers, side_stride(cfg))[:, :, :sd], None
    yield "head", params["lm_head"][:cfg.vocab, :h], None

    def norm(name: str, to: str):
        yield name, params[to][0, :h], None
        yield name + ".b", params[to][1, :h], None
    yield from norm("final.norm", "final_norm")
    for i, (b, l) in enumerate(zip(cfg.layers, layouts(cfg))):
        s, p = f"l{i}.", f"L{i}."
        w_in, w_o, m = params[p + "in"][:, :h], params[p + "o"][:h], s + "mix."
        yield from norm(s + "norm1", p + "norm1")
        yield from norm(s + "norm1b", p + "norm1b")
        yield m + "o", _cols(w_o, l.heads, l.vdim, l.dv), None
        if l.kind == "latent":
            yield m + "dq", w_in[:l.q_rank], None
            yield m + "dq.norm", params[p + "q_norm"][:l.q_rank], None
            yield m + "dkv", w_in[l.c0:l.c0 + l.kv_rank], (0, l.kv_rank)
            yield m + "dkv", w_in[l.kr0:l.kr0 + l.rot_dim], (l.kv_rank, l.kv_rank + l.rot_dim)
            yield m + "dkv.norm", params[p + "kv_norm"][:l.kv_rank], None
            yield m + "g", _rows(w_in, l.g0, l.heads, l.vdim, l.dv), None
            uq = params[p + "uq"].view(l.heads, l.dq, l.c0)[:, :, :l.q_rank]
            for hd in range(l.heads):
                r = hd * (l.dim + l.rot_dim)
                yield m + "uq", uq[hd, :l.dim], (r, r + l.dim)
                yield m + "uq", uq[hd, l.dk:l.dk + l.rot_dim], (r + l.dim, r + l.dim + l.rot_dim)
            up = params[p + "up"][:, :l.kv_rank]
            yield m + "uk", _rows(up, 0, l.heads, l.dim, l.dk), None
            yield m + "uv", _rows(up, l.heads * l.dk, l.heads, l.vdim, l.dv), None
        elif l.kind == "mamba2":
            inner, gn = l.heads * l.vdim, l.groups * l.state
            parts = ((l.g0, l.heads, l.vdim, l.dv), (0, l.heads, l.vdim, l.dv), (l.k0, l.groups, l.state, l.dk),
                     (l.q0, l.groups, l.state, l.dk), (l.n_in, l.heads, 1, 1))      # z, x, B, C, step gate
            r = 0
            for r0, heads, d, dp in parts:
                yield m + "in", _rows(w_in, r0, heads, d, dp), (r, r + heads * d)
                r += heads * d
            for leaf, dst in (("conv", params[p + "conv"].t()), ("conv.b", params[p + "conv_b"][:, None])):
                r = 0
                for (r0, heads, d, dp), n in zip(parts[1:4], (inner, gn, gn)):
                    yield m + leaf, _rows(dst, r0, heads, d, dp), (r, r + n)
                    r += n
            yield m + "dt_bias", params[p + "gate_b"], None
            yield m + "A_log", params[p + "a_log"], None
            yield m + "D", params[p + "skip"], None
            yield m + "norm", params[p + "norm"].view(l.heads, l.dv)[:, :l.vdim], None
        else:
            yield m + "q", _rows(w_in, 0, l.heads, l.dim, l.dk), None
            yield m + "k", _rows(w_in, l.k0, l.heads, l.dim, l.dk), None
            yield m + "v", _rows(w_in, l.v0, l.heads, l.vdim, l.dv), None
            yield m + "g", _rows(w_in, l.g0, l.heads, l.vdim, l.dv), None
            yield m + "i", w_in[l.n_in:l.n_in + l.heads], None
            yield m + "f", w_in[l.n_in + l.heads:l.n_in + 2 * l.heads], None
            yield m + "i.b", params[p + "gate_b"][:l.heads], None
            yield m + "f.b", params[p + "gate_b"][l.heads:], None
            yield m + "norm", params[p + "norm"].view(l.heads, l.dv)[:, :l.vdim], None
        if b.mlp is not None:
            yield from norm(s + "norm2", p + "norm2")
            yield from norm(s + "norm2b", p + "norm2b")
            gu = params[p + "gate_up"][:2 * b.mlp.ff, :h]
            yield s + "mlp.gate", gu[0::2], None
            yield s + "mlp.up", gu[1::2], None
            yield s + "mlp.down", params[p + "down"][:h, :b.mlp.ff], None
        yield s + "side.gate", params[p + "side_gate"][:sd, :h], None
        yield s + "side.proj", params[p + "side_proj"][:h, :sd], None
        yield s + "side.norm", params[p + "side_norm"][0, :h], None


def pack(cfg: FetotarConfig, get, device, dtype) -> Dict[str, torch.Tensor]:
    """Checkpoint tensors (``get(name)``) -> served parameters on ``device``."""
    params = {n: torch.zeros(s, dtype=dtype if k == "w" else torch.float32, device=device)
              for n, (s, k) in param_shapes(cfg).items()}
    want, last, name_of = tensor_shapes(cfg), None, None
    for name, view, rows in places(cfg, params):
        if name != name_of:                           # pieces of a tensor mostly follow each other: read it once
            last, name_of = get(name), name
            if tuple(last.shape) != want[name]:
                raise ValueError(f"{name}: shape {tuple(last.shape)}, the configuration says {want[name]}")
            last = last.to(device)
        view.copy_((last if rows is None else last[rows[0]:rows[1]]).reshape(view.shape))
    return params


def unpack(cfg: FetotarConfig, params: Dict[str, torch.Tensor]) -> Dict[str, torch.Tensor]:
    """Served parameters -> checkpoint tensors (the inverse of :func:`pack`)."""
    out: Dict[str, torch.Tensor] = {}
    shapes = tensor_shapes(cfg)
    for name, view, rows in places(cfg, params):
        if rows is None:
            out[name] = view.reshape(shapes[name])
        else:
            t = out.setdefault(name, torch.zeros(shapes[name], dtype=view.dtype, device=view.device))
            t[rows[0]:rows[1]] = view.reshape(t[rows[0]:rows[1]].shape)
    return out


def random_tensor(name: str, shape, g: torch.Generator, device="cpu") -> torch.Tensor:
    """One checkpoint tensor of a random-init model: projections N(0, 0.02), norms 1 with bias 0, decays as Mamba-2 and
    the mLSTM start with (A in 1..16, small steps, forget gates near one)."""
    leaf = name.split(".")[-1]
    if name.endswith((".norm.b", "norm1.b", "norm1b.b", "norm2.b", "norm2b.b", "conv.b", "i.b")):
        return torch.zeros(shape, device=device)
    if "norm" in leaf or leaf == "D":
        return torch.ones(shape, device=device)
    if leaf == "A_log":
        return torch.log(torch.empty(shape, device=device).uniform_(1.0, 16.0, generator=g))
    if leaf == "dt_bias":
        return torch.empty(shape, device=device).uniform_(-4.0, -2.0, generator=g)
    if name.endswith("f.b"):
        return torch.empty(shape, device=device).uniform_(3.0, 6.0, generator=g)
    return torch.randn(shape, generator=g, device=device) * (0.3 if leaf == "conv" else 0.02)


class FetotarModel:
    tp, tp_rank = 1, 0

    def __init__(self, cfg: FetotarConfig, params: Dict[str, torch.Tensor]):
        self.cfg, self.params = cfg, params
        self.dims = Dims(cfg.n_q_heads, cfg.n_kv_heads)
        self.layouts = layouts(cfg)
        self.caches = [cfg.cache_index(i) for i in range(cfg.n_layers)]
        # radians per position of every rotated pair (fp64: angles are reduced before they are rounded)
        self.freqs = [None if b.mixer.recurrent else
                      torch.tensor(b.mixer.rot.frequencies(), dtype=torch.float64, device=params["embed"].device) for b in cfg.layers]
        # the key maps once more, transposed per head [heads, latent, dim]: rows of the map of queries into the latent
        self.ukt = [None if l.kind != "latent" else
                    params[f"L{i}.up"][:l.heads * l.dk].view(l.heads, l.dk, l.kv).transpose(1, 2).contiguous() for i, l in enumerate(self.layouts)]
        self.lora: Dict[str, object] = {}
        self.weights_version = 0
        if params["lm_head"].is_cuda:      # library products accumulate in fp32 and read fp32 operands whole
            torch.backends.cuda.matmul.allow_bf16_reduced_precision_reduction = False
            torch.backends.cuda.matmul.allow_tf32 = False

    @property
    def act_dtype(self) -> torch.dtype:
        return self.params["lm_head"].dtype

    @classmethod
    def from_tensors(cls, cfg: FetotarConfig, get, device="cpu", dtype=torch.float32) -> "FetotarModel":
        return cls(cfg, pack(cfg, get, torch.device(device), dtype))

    @classmethod
    def build_random(cls, cfg: FetotarConfig, seed: int = 0, device="cpu", *, act_dtype=torch.float32) -> "FetotarModel":
        g = torch.Generator(device=device).manual_seed(seed)
        shapes = tensor_shapes(cfg)
        cache: Dict[str, torch.Tensor] = {}       # a tensor served in several pieces is drawn once

        def get(name):
            if name not in cache:
                cache.clear()
                cache[name] = random_tensor(name, shapes[name], g, device)
            return cache[name]
        return cls.from_tensors(cfg, get, device, act_dtype)

    def tensors(self) -> Iterator[Tuple[str, torch.Tensor]]:
        yield from unpack(self.cfg, self.params).items()

    # ---- serving forward --------------------------------------------------------------------
    def _mix(self, i: int, h, batch, ops, kv_pool, state_pool):
        """The mixer of layer ``i`` up to its output projection's input."""
        P, p, l, c = self.params, f"L{i}.", self.layouts[i], self.caches[i]
        eps = self.cfg.norm_eps
        proj, gates = ops.project_gates(h, P[p + "in"], l.n_in)
        if l.kind == "latent":
            rot = self.cfg.layers[i].mixer.rot
            q = ops.latent_prep(proj, l, P[p + "q_norm"], P[p + "kv_norm"], P[p + "uq"], self.freqs[i], rot, batch, kv_pool, c, eps)
            return ops.latent_attention(q, proj, P[p + "up"], self.ukt[i], l, self.freqs[i], rot, batch, kv_pool, c)
        w = {k: P.get(p + k) for k in ("norm", "gate_b", "conv", "conv_b", "a_log", "skip")}
        return ops.recurrent_mix(proj, gates, w, l, batch, state_pool, c, eps)

    def forward(self, batch, ops, kv_pool, state_pool, *, last_only: bool = True, aux_layers: Sequence[int] = (),
                return_hidden: bool = False, rows=None):
        """Logits (fp32) of each sequence's last token, of every token (``last_only=False``) or of the token
        rows listed in ``rows``.  ``aux_layers``: also return the stream after those layers."""
        cfg, P = self.cfg, self.params
        eps, n = cfg.norm_eps, cfg.hidden
        x, h = ops.embed_stream(P["embed"], batch.token_ids, cfg.embed_scale, P["L0.norm1"], eps, n)
        taps = {}
        for i, b in enumerate(cfg.layers):
            p = f"L{i}."
            y = ops.project_f32(self._mix(i, h, batch, ops, kv_pool, state_pool), P[p + "o"])
            h = ops.join(x, y, P[p + "norm1b"], P[p + "norm2"] if b.mlp is not None else None, eps, n)
            if b.mlp is not None:
                y = ops.project_f32(ops.clamped_glu(h, P[p + "gate_up"], b.mlp.limit), P[p + "down"])
                h = ops.join(x, y, P[p + "norm2b"], None, eps, n)
            s = ops.side_input(h, P[p + "side_gate"], P["side_embed"], batch.token_ids, i, cfg.side_dim)
            y = ops.project_f32(s, P[p + "side_proj"])
            h = ops.join(x, y, P[p + "side_norm"], P[f"L{i + 1}.norm1"] if i + 1 < cfg.n_layers else P["final_norm"], eps, n)
            if i in aux_layers:
                taps[i] = x[:, :n].clone()
        if rows is not None:
            hs = h[rows] if len(rows) else None
        else:
            hs = h[batch.last_idx.long()] if last_only and batch.n_tokens != batch.n_seqs else h
        logits = None if hs is None else ops.project_logits(hs, P["lm_head"])[..., :cfg.vocab]
        if aux_layers or return_hidden:
            return logits, x[:, :n], taps
        return logits

    def served_bytes(self) -> int:
        return sum(v.numel() * v.element_size() for v in self.params.values())
