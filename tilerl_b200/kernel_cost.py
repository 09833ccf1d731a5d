"""Declarative cost model: bytes and FLOPs of every kernel of a decode tick and of a
prefill, and the roofline bound they imply.

Every row is ``(name, count, bytes, flops, comm_bytes)`` for ONE rank; ``bound_seconds``
is ``max(bytes / hbm_bw, flops / peak, comm_bytes / nvlink_bw)`` summed over rows, which is
the floor a tick can reach if every kernel sat on its roofline.  The same table prices a
model without a GPU (``cli bench --kernels``) and normalises measured kernel times.

Parity: reference ``src/tilerl/kernel_cost.py`` -- ``TickShape:28``, ``_gemv:45``,
``_paged_attention_decode:92``, ``_gdn_decode_fused:107``, ``prefill_rows:239``,
``tick_rows:292``, ``sparse_indexer_rows:357``.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, List, Optional

from .config import ATTN, DeluvikConfig, FetotarConfig, ModelConfig, StreamDesign, TobadraConfig, ZinutarConfig
from .formats import FORMATS, nbytes
from .parallel.mesh import tp_dims


@dataclass(frozen=True)
class TickShape:
    batch: int = 1
    ctx: int = 512          # KV length attended per sequence
    width: int = 1          # tokens per sequence in the tick (speculative verify: W)
    tp: int = 1
    sparse_pages: int = 0   # >0: attention reads this many pages instead of ctx/16


@dataclass
class Row:
    name: str
    count: int
    bytes: float
    flops: float
    comm_bytes: float = 0.0

    def bound(self, hbm: float, peak: float, link: float) -> float:
        return self.count * max(self.bytes / hbm, self.flops / peak, self.comm_bytes / link if link else 0.0)


def _lin_format(cfg: ModelConfig) -> str:
    return {"nvfp4": "nvfp4", "fp8": "fp8_block", "bf16": "bf16"}[cfg.quant]


def _linear(name: str, count: int, m: int, n: int, k: int, fmt: str, comm: float = 0.0) -> Row:
    w = nbytes(fmt, (n, k))
    act = m * k * 2 + m * n * 2
    return Row(name, count, w + act, 2.0 * m * n * k, comm)


def _zinutar_rows(cfg: ZinutarConfig, m: int, pairs: float, kv_read: float, head_rows_m: int) -> List[Row]:
    """One forward of ``m`` tokens: ``pairs`` (query token, key) pairs, ``kv_read`` key tokens whose pages are read."""
    from .kv import kv_pages
    from .zinutar_layout import BlockLayout, head_rows, stream_width
    w = stream_width(cfg)
    rows = [Row("embedding + norm", 1, m * w * (2 + 4), 0)]
    for i in range(cfg.n_layers):
        runs = [r for r in cfg.runs if r.layer == i]
        if not runs:
            continue
        l, pg = BlockLayout.of(cfg.layers[i]), kv_pages(cfg, 2)[runs[0].kv]
        per_token = pg.n_kv * pg.nbytes / 16
        n = len(runs)
        rows += [Row(f"L{i} in (norm fused)", n, l.n_in * w * 2 + m * (w * 4 + l.n_in * 2), 2.0 * m * l.n_in * w),
                 Row(f"L{i} attn.kv write + polynorm", n, m * (per_token * 2 + 4.0 * l.ff), 0),
                 Row(f"L{i} attn.sigmoid", n, kv_read * per_token + m * l.heads * (l.dk + l.dv) * 2.0,
                     2.0 * pairs * l.heads * (l.dk + l.dv)),
                 Row(f"L{i} out (+stream)", n, l.n_out * w * 2 + m * (l.n_out * 2 + w * 8), 2.0 * m * l.n_out * w)]
    rows.append(Row("lm_head", 1, head_rows(cfg) * w * 2 + head_rows_m * (w * 4 + head_rows(cfg) * 4), 2.0 * head_rows_m * head_rows(cfg) * w))
    return rows


def _fetotar_rows(cfg: FetotarConfig, m: int, ctx: int, n_seqs: int, head_rows_m: int) -> List[Row]:
    """One forward of ``m`` tokens in ``n_seqs`` sequences that end at ``ctx`` tokens each."""
    from .fetotar_layout import head_rows, layout_of, pad, side_width, stream_width
    w, q = stream_width(cfg), m // n_seqs
    lin = lambda name, n, k, out=2: Row(name, 1, n * k * 2 + m * (k * 2 + n * out), 2.0 * m * n * k)
    rows = [Row("embedding + norm", 1, m * w * (2 + 4 + 2), 0)]
    for i, b in enumerate(cfg.layers):
        l = layout_of(b.mixer)
        rows.append(lin(f"L{i} in", l.n_in + pad(l.n_gates, 8), w))
        if l.kind == "latent":
            seen = sum(min(p + 1, l.window) for p in range(ctx - q, ctx))        # (query, key) pairs of one sequence
            keys = min(ctx, q + l.window - 1)
            rows += [Row(f"L{i} attn.latents into the cache", 1, m * (l.c0 + l.row) * 4.0, 0), lin(f"L{i} attn.queries", l.heads * l.dq, l.c0),
                     Row(f"L{i} attn.latent", 1, n_seqs * keys * l.row * 2 + m * l.heads * (l.dq + l.dv) * 2.0,
                         2.0 * n_seqs * seen * l.heads * (l.dq + l.dv)),
                     Row(f"L{i} attn.key / value maps", 1, l.heads * (l.dk + l.dv) * l.kv * 2.0, 2.0 * m * l.heads * (l.dk + l.dv) * l.kv)]
        else:
            rows.append(Row(f"L{i} {l.kind}.scan", 1, n_seqs * l.state_floats * 8.0 + m * (l.n_in * 2 + l.heads * l.dv * 6.0),
                            4.0 * m * l.heads * l.dk * l.dv))
        rows += [lin(f"L{i} o", w, l.n_out, 4), Row(f"L{i} joins", 2 + (b.mlp is not None), m * w * (4 + 8 + 2.0), 0)]
        if b.mlp is not None:
            ff = pad(b.mlp.ff, 64)
            rows += [lin(f"L{i} gate_up", 2 * ff, w), lin(f"L{i} down", w, ff, 4)]
        rows += [lin(f"L{i} side gate", side_width(cfg), w), lin(f"L{i} side proj", w, side_width(cfg), 4)]
    rows.append(Row("lm_head", 1, head_rows(cfg) * w * 2 + head_rows_m * (w * 2 + head_rows(cfg) * 4), 2.0 * head_rows_m * head_rows(cfg) * w))
    return rows


def _deluvik_rows(cfg: DeluvikConfig, m: int, ctx: int, n_seqs: int, head_rows_m: int) -> List[Row]:
    """One forward of ``m`` tokens in ``n_seqs`` sequences that end at ``ctx`` tokens each."""
    from .deluvik_layout import MoeLayout, head_rows, layouts, pad, stream_width
    from .mixers import MoeSpec
    w, q = stream_width(cfg), m // n_seqs
    lin = lambda name, n, k, out=2: Row(name, 1, n * k * 2 + m * (k * 2 + n * out), 2.0 * m * n * k)
    rows = [Row("embedding", 1, m * w * (2 + 4 + 2), 0)]
    for i, (b, l) in enumerate(zip(cfg.layers, layouts(cfg))):
        a, s = l.attn, l.attn.spec
        win = s.window or ctx
        seen = sum(min(p + 1, win) for p in range(ctx - q, ctx))                 # (query, key) pairs of one sequence
        keys = min(ctx, q + win - 1)
        rows += [lin(f"L{i} in", l.n_in, w), Row(f"L{i} attn.prep (norm, rotation, cache)", 1, m * a.n_in * 4.0, 0),
                 Row(f"L{i} attn.softmax", 1, n_seqs * keys * s.kv_heads * (a.dk + a.dv) * 2 + m * s.heads * (a.dk + a.dv) * 2.0,
                     2.0 * n_seqs * seen * s.heads * (a.dk + a.dv))]
        if l.lru is not None:
            r = l.lru
            gates = r.spec.blocks * 2 * r.pp * r.pp
            rows.append(Row(f"L{i} lru (gates, scan)", 1, gates * 2 + n_seqs * r.width * 8 + m * r.width * 6.0, 2.0 * m * gates))
        rows += [lin(f"L{i} o", w, l.n_out, 4), Row(f"L{i} joins", 1 + (b.mlp is not None), m * w * (4 + 8 + 2.0), 0)]
        if isinstance(b.mlp, MoeSpec):
            e = MoeLayout(b.mlp)
            used = e.pieces + e.spec.experts * (1.0 - (1.0 - e.spec.top / e.spec.experts) ** m)     # experts some token chooses
            rows.append(lin(f"L{i} router", e.router_rows, w, 4))
            for name, n, k, out in (("up", 2 * e.ff, w, 1), ("down", w, e.ff, 4)):
                rows.append(Row(f"L{i} experts {name}", 1, used * n * k * 2 + m * e.slots * (k * 2 + n * out), 2.0 * m * e.slots * n * k))
        elif b.mlp is not None:
            ff = pad(b.mlp.ff, 64)
            rows += [lin(f"L{i} gate_up", 2 * ff, w), lin(f"L{i} down", w, ff, 4)]
    rows.append(Row("lm_head", 1, head_rows(cfg) * w * 2 + head_rows_m * (w * 2 + head_rows(cfg) * 4), 2.0 * head_rows_m * head_rows(cfg) * w))
    return rows


def _tobadra_rows(cfg: TobadraConfig, m: int, ctx: int, n_seqs: int, head_rows_m: int) -> List[Row]:
    """One forward of ``m`` tokens in ``n_seqs`` sequences that end at ``ctx`` tokens each."""
    from .deluvik_layout import LayerLayout, MoeLayout
    from .mixers import MoeSpec
    from .tobadra_layout import gate_rows, head_rows, layouts, pad, router_rows, stream_width
    w, q = stream_width(cfg), m // n_seqs
    lin = lambda name, n, k, out=2: Row(name, 1, n * k * 2 + m * (k * 2 + n * out), 2.0 * m * n * k)
    rows = [Row("embedding, norm, convolution", 1, m * w * (2 + 4 + 4), 0)]
    for i, (b, l) in enumerate(zip(cfg.layers, layouts(cfg))):
        rows.append(lin(f"L{i} in, branch gate", l.n_in + gate_rows(l) + w, w))
        if isinstance(l, LayerLayout):
            a, s = l.attn, l.attn.spec
            seen = sum(min(p + 1, s.window) for p in range(ctx - q, ctx))            # (query, key) pairs of one sequence
            keys = min(ctx, q + s.window - 1)
            rows += [Row(f"L{i} attn.prep (bias, rotation, cache)", 1, m * a.n_in * 4.0, 0),
                     Row(f"L{i} attn.softmax", 1, n_seqs * keys * s.kv_heads * (a.dk + a.dv) * 2 + m * s.heads * (a.dk + a.dv) * 2.0,
                         2.0 * n_seqs * seen * s.heads * (a.dk + a.dv))]
        else:
            if l.kind == "delta":
                rows += [lin(f"L{i} delta.decays and gate", l.n_low + l.heads * l.dk, l.r, 3), Row(f"L{i} delta.prep", 1, m * (l.conv_c * 4.0 + l.heads * l.dk * 8), 0)]
            rows.append(Row(f"L{i} {l.kind}.scan", 1, n_seqs * l.state_floats * 8.0 + m * (l.n_in * 2 + l.heads * l.dv * 6.0),
                            (4.0 if l.kind == "lightning" else 6.0) * m * l.heads * l.dk * l.dv))
        rows += [lin(f"L{i} o", w, l.n_out, 4), Row(f"L{i} joins", 1 + (b.mlp is not None), m * w * (4 + 4 + 8 + 4.0), 0)]
        if isinstance(b.mlp, MoeSpec):
            e = MoeLayout(b.mlp)
            used = e.pieces + e.spec.experts * (1.0 - (1.0 - e.spec.top / e.spec.outputs) ** m)     # experts some token chooses
            slots = e.pieces + e.spec.top * e.spec.experts / e.spec.outputs                          # of a token, on average
            rows.append(lin(f"L{i} router, branch gate", router_rows(b.mlp) + w, w, 4))
            for name, n, k, out in (("up", e.ff, w, 2), ("down", w, e.ff, 4)):
                rows.append(Row(f"L{i} experts {name}", 1, used * n * k * 2 + m * slots * (k * 2 + n * out), 2.0 * m * slots * n * k))
        elif b.mlp is not None:
            ff = pad(b.mlp.ff, 64)
            rows += [lin(f"L{i} up, branch gate", ff + w, w), lin(f"L{i} down", w, ff, 4)]
    rows.append(Row("logits", 1, head_rows(cfg) * w * 2 + head_rows_m * (w * 2 + head_rows(cfg) * 4), 2.0 * head_rows_m * head_rows(cfg) * w))
    return rows


_STREAM_ROWS = {FetotarConfig: _fetotar_rows, DeluvikConfig: _deluvik_rows, TobadraConfig: _tobadra_rows}


def tick_rows(cfg: ModelConfig, s: TickShape) -> List[Row]:
    """One decode (or verify) tick on one TP rank."""
    if isinstance(cfg, StreamDesign):
        b, c = s.batch, s.ctx
        if type(cfg) in _STREAM_ROWS:
            return _STREAM_ROWS[type(cfg)](cfg, b * s.width, c, b, b * s.width)
        return _zinutar_rows(cfg, b * s.width, b * s.width * c, b * c, b * s.width)
    d = tp_dims(cfg, s.tp)
    m = s.batch * s.width
    h = cfg.hidden
    fmt = _lin_format(cfg)
    na, ng = cfg.n_attn_layers, cfg.n_gdn_layers
    ar = (s.tp - 1) * m * h * 4.0 if s.tp > 1 else 0.0      # one-shot all-reduce: fp32 partial to every peer
    rows = [Row("embedding", 1, m * h * 2 * 2, 0)]
    if na:
        hd = cfg.head_dim
        rows.append(_linear("attn.qkv (norm fused)", na, m, d.qkv_rows, h, fmt))
        kv_tokens = (s.sparse_pages * 16 if s.sparse_pages else s.ctx)
        kv_bytes = s.batch * kv_tokens * d.n_kv * hd * 2 * 2
        rows.append(Row("attn.prep + kv write", na, m * d.qkv_rows * 2 + m * d.n_kv * hd * 4, 0))
        rows.append(Row("attn.paged (split + combine)", na, kv_bytes + m * d.n_q * hd * 4,
                        4.0 * m * d.n_q * hd * kv_tokens))
        rows.append(_linear("attn.o (+residual, all-reduce)", na, m, h, d.n_q * hd, fmt, ar))
    if ng:
        gd = cfg.gdn_head_dim
        state = s.batch * d.gdn_nv * gd * gd * 4
        rows.append(_linear("gdn.in (norm fused)", ng, m, d.gdn_in_rows, h, fmt))
        rows.append(Row("gdn.step (state r/w)", ng, state * (1 + s.width) + m * d.gdn_in_rows * 2,
                        6.0 * m * d.gdn_nv * gd * gd))
        rows.append(_linear("gdn.out (+residual, all-reduce)", ng, m, h, d.gdn_nv * gd, fmt, ar))
    rows.append(_linear("mlp.gate_up (norm + swiglu fused)", cfg.n_layers, m, 2 * d.ffn, h, fmt))
    rows.append(_linear("mlp.down (+residual, all-reduce)", cfg.n_layers, m, h, d.ffn, fmt, ar))
    head_fmt = "nvfp4" if cfg.lm_head_quant == "nvfp4" else "bf16"
    rows.append(_linear("lm_head", 1, s.batch, d.vocab_local, h, head_fmt))
    rows.append(Row("argmax", 1, s.batch * d.vocab_local * 4, 0, (s.tp - 1) * s.batch * 8.0 if s.tp > 1 else 0))
    return rows


def prefill_rows(cfg: ModelConfig, tokens: int, tp: int = 1, terms: int = 2) -> List[Row]:
    """One prefill of ``tokens`` tokens (one sequence) on one TP rank; ``terms`` NVFP4
    activation terms per token multiply the tensor-core work."""
    if type(cfg) in _STREAM_ROWS:
        return _STREAM_ROWS[type(cfg)](cfg, tokens, tokens, 1, 1)
    if isinstance(cfg, StreamDesign):
        return _zinutar_rows(cfg, tokens, tokens * (tokens + 1) / 2, tokens, 1)
    d = tp_dims(cfg, tp)
    h, m = cfg.hidden, tokens
    fmt = _lin_format(cfg)
    na, ng = cfg.n_attn_layers, cfg.n_gdn_layers
    rs = 2.0 * (tp - 1) / tp * m * h * 2 if tp > 1 else 0.0     # reduce-scatter + all-gather of bf16 rows

    def lin(name, count, n, k, comm=0.0):
        r = _linear(name, count, m, n, k, fmt, comm)
        r.flops *= terms
        return r
    rows = [Row("embedding", 1, m * h * 4, 0)]
    if na:
        hd = cfg.head_dim
        rows += [lin("attn.qkv", na, d.qkv_rows, h),
                 Row("attn.causal", na, m * (d.n_q + 2 * d.n_kv) * hd * 2 * 2, 2.0 * m * m * d.n_q * hd),
                 lin("attn.o", na, h, d.n_q * hd, rs)]
    if ng:
        gd = cfg.gdn_head_dim
        rows += [lin("gdn.in", ng, d.gdn_in_rows, h),
                 Row("gdn.scan", ng, m * d.gdn_in_rows * 2 * 2 + d.gdn_nv * gd * gd * 8, 6.0 * m * d.gdn_nv * gd * gd),
                 lin("gdn.out", ng, h, d.gdn_nv * gd, rs)]
    rows += [lin("mlp.gate_up", cfg.n_layers, 2 * d.ffn, h), lin("mlp.down", cfg.n_layers, h, d.ffn, rs)]
    rows.append(_linear("lm_head (last token)", 1, 1, d.vocab_local, h, "bf16"))
    return rows


def sparse_indexer_rows(cfg: ModelConfig, ctx: int, batch: int = 1, tp: int = 1) -> List[Row]:
    d = tp_dims(cfg, tp)
    pages = ctx // 16
    b = batch * pages * d.n_kv * 2 * cfg.head_dim * 2
    return [Row("quest bounds + scores + top-k", cfg.n_attn_layers, b, 4.0 * batch * pages * d.n_q * cfg.head_dim)]


def bound_seconds(rows: List[Row], hbm_gbs: float, peak_tflops: float, nvlink_gbs: float = 770.0) -> float:
    return sum(r.bound(hbm_gbs * 1e9, peak_tflops * 1e12, nvlink_gbs * 1e9) for r in rows)


def tick_bytes(rows: List[Row]) -> float:
    return sum(r.count * r.bytes for r in rows)


def table(rows: List[Row], hbm_gbs: float, peak_tflops: float, nvlink_gbs: float = 770.0,
          measured_us: Optional[Dict[str, float]] = None) -> str:
    out = [f"{'kernel':40s} {'n':>4s} {'MB':>10s} {'GFLOP':>10s} {'bound us':>10s} {'meas us':>10s} {'frac':>6s}"]
    for r in rows:
        b = r.bound(hbm_gbs * 1e9, peak_tflops * 1e12, nvlink_gbs * 1e9) * 1e6
        meas = (measured_us or {}).get(r.name)
        out.append(f"{r.name:40s} {r.count:4d} {r.count * r.bytes / 1e6:10.2f} {r.count * r.flops / 1e9:10.2f} "
                   f"{b:10.1f} {meas if meas is not None else float('nan'):10.1f} "
                   f"{(b / meas) if meas else float('nan'):6.2f}")
    out.append(f"{'total':40s} {'':4s} {tick_bytes(rows) / 1e6:10.2f} {'':10s} "
               f"{bound_seconds(rows, hbm_gbs, peak_tflops, nvlink_gbs) * 1e6:10.1f}")
    return "\n".join(out)
