"""Zinutar: a looped decoder of parallel blocks (no counterpart in the reference).

Stream ``x`` (fp32)::

    x0 = rms(embed[token]) * embed_norm                 the embedding output
    for each layer run:
        x  = x + x0                                     only on re-entry into the loop
        h  = rms(x) * norm1
        x  = x + W_o A(W_q h, W_k h, W_v h) + W_down P(W_up h)
    logits = W_head (rms(x) * final_norm)

``A`` is causal attention over RMS-normalised queries and keys whose weights are ``sigmoid(score * scale +
bias[head])``, not normalised over keys; ``P`` is PolyNorm (:func:`tilerl_b200.ops.ref.polynorm`).

Because both sublayers read the same ``h`` and add to the same ``x``, a layer is two projections: ``in`` holds
the rows of q, k, v and up under each other, ``out`` the columns of o and down side by side.  Every head and
the stream are padded with zero rows / columns to the widths the kernels load (:class:`~tilerl_b200.zinutar_layout.BlockLayout`), so any
size of the configuration runs on the same kernels.

Parameter names: ``embed``, ``embed_norm``, ``final_norm``, ``lm_head`` and per layer ``L{i}.norm1``,
``L{i}.in``, ``L{i}.out``, ``L{i}.bias``, ``L{i}.act``.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, Iterator, Sequence, Tuple

import torch

from ..config import ZinutarConfig
from ..zinutar_layout import BlockLayout, param_shapes, tensor_shapes


# ---- checkpoint tensors <-> served parameters -----------------------------------------------------
def _head_rows_into(dst: torch.Tensor, r0: int, w: torch.Tensor, heads: int, d: int, dp: int) -> None:
    dst[r0:r0 + heads * dp].view(heads, dp, -1)[:, :d, :w.shape[1]].copy_(w.view(heads, d, -1))


def pack(cfg: ZinutarConfig, get, device, dtype) -> Dict[str, torch.Tensor]:
    """Checkpoint tensors (``get(name)``) -> served parameters on ``device``."""
    params = {n: torch.zeros(s, dtype=dtype if k == "w" else torch.float32, device=device)
              for n, (s, k) in param_shapes(cfg).items()}
    want = tensor_shapes(cfg)

    def t(name: str) -> torch.Tensor:
        x = get(name)
        if tuple(x.shape) != want[name]:
            raise ValueError(f"{name}: shape {tuple(x.shape)}, the configuration says {want[name]}")
        return x.to(device)
    h = cfg.hidden
    params["embed"][:, :h].copy_(t("embed"))
    params["embed_norm"][:h].copy_(t("embed.norm"))
    params["final_norm"][:h].copy_(t("final.norm"))
    params["lm_head"][:cfg.vocab, :h].copy_(t("head"))
    for i, b in enumerate(cfg.layers):
        l, s, p = BlockLayout.of(b), f"l{i}.", f"L{i}."
        params[p + "norm1"][:h].copy_(t(s + "norm1"))
        params[p + "bias"].copy_(t(s + "mix.pb"))
        w_in, w_out = params[p + "in"], params[p + "out"]
        _head_rows_into(w_in, 0, t(s + "mix.q"), l.heads, l.dim, l.dk)
        _head_rows_into(w_in, l.k0, t(s + "mix.k"), l.kv_heads, l.dim, l.dk)
        _head_rows_into(w_in, l.v0, t(s + "mix.v"), l.kv_heads, l.vdim, l.dv)
        w_out[:h, :l.attn_cols].view(h, l.heads, l.dv)[:, :, :l.vdim].copy_(t(s + "mix.o").view(h, l.heads, l.vdim))
        if l.ff:
            w_in[l.up0:l.up0 + l.ff, :h].copy_(t(s + "mlp.up"))
            w_out[:h, l.attn_cols:l.attn_cols + l.ff].copy_(t(s + "mlp.down"))
            params[p + "act"].copy_(t(s + "mlp.act"))
    return params


def unpack(cfg: ZinutarConfig, params: Dict[str, torch.Tensor]) -> Dict[str, torch.Tensor]:
    """Served parameters -> checkpoint tensors (the inverse of :func:`pack`)."""
    h = cfg.hidden
    out = {"embed": params["embed"][:, :h], "embed.norm": params["embed_norm"][:h],
           "final.norm": params["final_norm"][:h], "head": params["lm_head"][:cfg.vocab, :h]}
    for i, b in enumerate(cfg.layers):
        l, s, p = BlockLayout.of(b), f"l{i}.", f"L{i}."
        w_in, w_out = params[p + "in"][:, :h], params[p + "out"][:h]

        def rows(r0, heads, d, dp):
            return w_in[r0:r0 + heads * dp].reshape(heads, dp, h)[:, :d].reshape(heads * d, h)
        out[s + "norm1"], out[s + "mix.pb"] = params[p + "norm1"][:h], params[p + "bias"]
        out[s + "mix.q"] = rows(0, l.heads, l.dim, l.dk)
        out[s + "mix.k"] = rows(l.k0, l.kv_heads, l.dim, l.dk)
        out[s + "mix.v"] = rows(l.v0, l.kv_heads, l.vdim, l.dv)
        out[s + "mix.o"] = w_out[:, :l.attn_cols].reshape(h, l.heads, l.dv)[:, :, :l.vdim].reshape(h, -1)
        if l.ff:
            out[s + "mlp.up"] = w_in[l.up0:l.up0 + l.ff]
            out[s + "mlp.down"] = w_out[:, l.attn_cols:l.attn_cols + l.ff]
            out[s + "mlp.act"] = params[p + "act"]
    return out


def random_tensor(name: str, shape, g: torch.Generator, device="cpu") -> torch.Tensor:
    """One checkpoint tensor of a random-init model: projections N(0, 0.02), norms 1, attention biases around
    ``-log`` of a context length, mild PolyNorm coefficients."""
    leaf = name.split(".")[-1]
    if "norm" in name:
        return torch.ones(shape, device=device)
    if leaf == "pb":
        return -5.0 + 0.5 * torch.randn(shape, generator=g, device=device)
    if leaf == "act":
        return torch.tensor([0.5, 0.3, 0.3, 0.1], device=device)
    return torch.randn(shape, generator=g, device=device) * 0.02


@dataclass(frozen=True)
class Dims:
    """What the engine and the graph runners read about head counts."""
    n_q: int
    n_kv: int
    gdn_nk: int = 0
    gdn_nv: int = 0


class ZinutarModel:
    tp, tp_rank = 1, 0

    def __init__(self, cfg: ZinutarConfig, params: Dict[str, torch.Tensor]):
        self.cfg, self.params = cfg, params
        self.dims = Dims(cfg.n_q_heads, cfg.n_kv_heads)
        self.layouts = [BlockLayout.of(b) for b in cfg.layers]
        self.runs = cfg.runs
        self.lora: Dict[str, object] = {}
        self.weights_version = 0
        if params["lm_head"].is_cuda:      # library products accumulate in fp32 and read fp32 operands whole
            torch.backends.cuda.matmul.allow_bf16_reduced_precision_reduction = False
            torch.backends.cuda.matmul.allow_tf32 = False

    @property
    def act_dtype(self) -> torch.dtype:
        return self.params["lm_head"].dtype

    @classmethod
    def from_tensors(cls, cfg: ZinutarConfig, get, device="cpu", dtype=torch.float32) -> "ZinutarModel":
        return cls(cfg, pack(cfg, get, torch.device(device), dtype))

    @classmethod
    def build_random(cls, cfg: ZinutarConfig, seed: int = 0, device="cpu", *, act_dtype=torch.float32) -> "ZinutarModel":
        g = torch.Generator(device=device).manual_seed(seed)
        shapes = tensor_shapes(cfg)
        return cls.from_tensors(cfg, lambda n: random_tensor(n, shapes[n], g, device), device, act_dtype)

    def tensors(self) -> Iterator[Tuple[str, torch.Tensor]]:
        yield from unpack(self.cfg, self.params).items()

    # ---- serving forward --------------------------------------------------------------------
    def forward(self, batch, ops, kv_pool, state_pool, *, last_only: bool = True, aux_layers: Sequence[int] = (),
                return_hidden: bool = False, rows=None):
        """Logits (fp32) of each sequence's last token, of every token (``last_only=False``) or of the token
        rows listed in ``rows``.  ``aux_layers``: also return the stream after the last run of those layers."""
        cfg, P = self.cfg, self.params
        eps = cfg.rms_eps
        x, x0 = ops.embed_norm(P["embed"], P["embed_norm"], batch.token_ids, eps, cfg.hidden,
                               keep=any(r.inject for r in self.runs))
        taps = {}
        for run in self.runs:
            p, l = f"L{run.layer}.", self.layouts[run.layer]
            if run.inject:
                ops.stream_add(x, x0)
            proj = ops.stream_linear(x, P[p + "norm1"], P[p + "in"], eps, cfg.hidden)
            mid = ops.block_mid(proj, P.get(p + "act"), l, batch, kv_pool, run.kv, eps)
            ops.sigmoid_attention(proj, mid, P[p + "bias"], l, batch, kv_pool, run.kv, eps)
            ops.stream_accumulate(mid, P[p + "out"], x)
            if run.layer in aux_layers:
                taps[run.layer] = x[:, :cfg.hidden].clone()
        if rows is not None:
            xs = x[rows] if len(rows) else None
        else:
            xs = x[batch.last_idx.long()] if last_only and batch.n_tokens != batch.n_seqs else x
        logits = None if xs is None else ops.stream_head(xs, P["final_norm"], P["lm_head"], eps, cfg.hidden)[..., :cfg.vocab]
        if aux_layers or return_hidden:
            return logits, x[:, :cfg.hidden], taps
        return logits

    def served_bytes(self) -> int:
        return sum(v.numel() * v.element_size() for v in self.params.values())
