"""CUDA ops of decoders with an fp32 residual stream and parallel blocks (``models/zinutar.py``).

Mixed into :class:`tilerl_b200.ops.cuda.CudaOps`.  The activation type is that of the weights: bf16 (the serving
type) or fp32 (true fp32 everywhere: library products without TF32, fp32 kernels).

A layer is five launches in a decode tick: fused in-projection with the norm in its prologue, block middle (K / V
write, PolyNorm), attention, the sum of its splits, out-projection added to the stream.  More rows than the
weight-streaming projection serves take library products (``torch.mm``) between the same kernels.  No counterpart in the
reference.
"""
from __future__ import annotations

import torch

from . import native as N

# Rows the weight-streaming projection serves.  Decode ticks of 2048- and 4096-wide models, against library products in
# its place: 1 row 0.47 / 0.62 ms against 0.70 / 0.70, 4 rows 0.56 / 0.73 against 0.72 / 0.73, 8 rows even.
ROWS_MAX = 4
ROWS_NORM_MAX = 2       # rows whose norm it folds in (every block recomputes it)
EPI_STORE, EPI_STORE_F32, EPI_ADD_F32 = 0, 1, 2
SHORT_ROWS = 16         # (token, head of the group) rows of a sequence up to which attention splits keys over warps


class StreamOps:
    # ---- stream ----------------------------------------------------------------------
    def embed_norm(self, table, norm_w, ids, eps, n, keep):
        t, ld = ids.shape[0], table.shape[1]
        x = self.ws.get("stream", (t, ld), torch.float32)
        x0 = self.ws.get("stream0", (t, ld), torch.float32) if keep else None
        N.check(self.lib.trl_embed_norm(table.data_ptr(), ids.data_ptr(), norm_w.data_ptr(), x.data_ptr(), N.ptr(x0), t, ld, n,
                                        table.shape[0], eps, int(table.dtype == torch.float32), N.stream()), "embed_norm")
        N.count()
        return x, x0

    def stream_add(self, x, y):
        N.check(self.lib.trl_stream_add(x.data_ptr(), y.data_ptr(), x.numel(), N.stream()), "stream_add")
        N.count()

    def _stream_norm(self, x, norm_w, eps, n, dtype):
        t, ld = x.shape
        h = self.ws.get("stream_h", (t, ld), dtype)
        N.check(self.lib.trl_stream_norm(x.data_ptr(), norm_w.data_ptr(), h.data_ptr(), t, ld, n, eps,
                                         int(dtype == torch.float32), N.stream()), "stream_norm")
        N.count()
        return h

    def _linear_rows(self, x, w, y, epi, norm_w=None, eps=0.0, n=0):
        N.check(self.lib.trl_linear_rows(x.data_ptr(), x.stride(0), w.data_ptr(), N.ptr(norm_w), eps, n, y.data_ptr(),
                                         y.stride(0), x.shape[0], w.shape[0], w.shape[1], epi, N.stream()), "linear_rows")
        N.count()

    def _streams(self, rows: int, w) -> bool:
        """This many rows go through the weight-streaming projection."""
        return w.dtype == torch.bfloat16 and rows <= ROWS_MAX and rows <= self.lib.trl_linear_rows_max(w.shape[1])

    def _project(self, x, norm_w, w, eps, n, y, epi):
        """``y = norm(x) @ W^T`` from stream rows ``x``."""
        t = x.shape[0]
        if t <= ROWS_NORM_MAX and self._streams(t, w):
            self._linear_rows(x, w, y, epi, norm_w, eps, n)
            return y
        h = self._stream_norm(x, norm_w, eps, n, w.dtype)
        if self._streams(t, w):
            self._linear_rows(h, w, y, epi)
        elif y.dtype == w.dtype:
            torch.mm(h, w.t(), out=y)
        else:
            torch.mm(h, w.t(), out_dtype=y.dtype, out=y)
        return y

    def stream_linear(self, x, norm_w, w, eps, n):
        y = self.ws.get(f"block_proj_{w.dtype}", (x.shape[0], w.shape[0]), w.dtype)
        return self._project(x, norm_w, w, eps, n, y, EPI_STORE)

    def stream_head(self, x, norm_w, w, eps, n):
        logits = self.ws.get("logits", (x.shape[0], w.shape[0]), torch.float32)
        return self._project(x.contiguous(), norm_w, w, eps, n, logits, EPI_STORE_F32)

    def stream_accumulate(self, a, w, x):
        """``x += a @ W^T`` (fp32)."""
        if self._streams(a.shape[0], w):
            self._linear_rows(a, w, x, EPI_ADD_F32)
        elif w.dtype == torch.float32:
            x.addmm_(a, w.t())
        else:
            torch.addmm(x, a, w.t(), out_dtype=torch.float32, out=x)

    # ---- block -----------------------------------------------------------------------
    def block_mid(self, proj, act, l, batch, pool, kv_idx, eps):
        t = proj.shape[0]
        mid = self.ws.get(f"block_mid_{proj.dtype}", (t, l.n_out), proj.dtype)
        cache = pool.layer(kv_idx)
        N.check(self.lib.trl_block_mid(
            proj.data_ptr(), proj.stride(0), N.ptr(act), mid.data_ptr(), mid.stride(0), batch.slot_mapping.data_ptr(),
            cache.data_ptr(), cache.shape[0], t, l.k0, l.v0, l.up0, l.attn_cols, l.ff, l.kv_heads, l.dim, l.dk, l.dv, eps,
            int(proj.dtype == torch.float32), N.stream()), "block_mid")
        N.count()
        return mid

    def sigmoid_attention(self, proj, mid, bias, l, batch, pool, kv_idx, eps):
        """Attention output of every token into the first ``heads x dv`` columns of ``mid``."""
        cache, table = pool.layer(kv_idx), batch.block_table
        st = N.stream()
        if proj.dtype == torch.float32:
            N.check(self.lib.trl_sigmoid_attn_f32(
                proj.data_ptr(), proj.stride(0), cache.data_ptr(), cache.shape[0], table.data_ptr(), table.stride(0),
                batch.q_start.data_ptr(), batch.q_len.data_ptr(), batch.positions.data_ptr(), bias.data_ptr(), mid.data_ptr(),
                mid.stride(0), batch.n_seqs, batch.max_q_len, l.heads, l.kv_heads, l.dim, l.dk, l.dv, eps, l.scale, st),
                "sigmoid_attn_f32")
            N.count()
            return
        t, g = proj.shape[0], l.heads // l.kv_heads
        short = max(1, SHORT_ROWS // g)              # tokens of a sequence that fit the narrow row tile
        lens, kvs = batch.host_q_len, batch.host_kv_len
        classes = [(wide, [i for i, n in enumerate(lens) if (n > short) == bool(wide)]) for wide in (0, 1)]
        classes = [c for c in classes if c[1]]
        for wide, sel in classes:
            # alone, a launch takes every length: in a captured verify tick the lengths on the device are the true ones
            lo, hi = (1, 1 << 30) if len(classes) == 1 else ((short + 1, 1 << 30) if wide else (1, short))
            rows = self.lib.trl_sigmoid_attn_rows(l.dk, l.dv) if wide else 16
            tiles = max((lens[i] * g + rows - 1) // rows for i in sel)
            splits = self._sigmoid_splits(sum((lens[i] * g + rows - 1) // rows for i in sel) * l.kv_heads,
                                          max(kvs[i] for i in sel), wide, pool.pages[kv_idx].nbytes)
            part = self.ws.get("attn_part", (t * l.heads * splits * l.dv,), torch.float32) if splits > 1 else None
            N.check(self.lib.trl_sigmoid_attn(
                proj.data_ptr(), proj.stride(0), cache.data_ptr(), cache.shape[0], table.data_ptr(), table.stride(0),
                batch.q_start.data_ptr(), batch.q_len.data_ptr(), batch.positions.data_ptr(), batch.seq_ids.data_ptr(),
                bias.data_ptr(), mid.data_ptr(), mid.stride(0), N.ptr(part), t, batch.n_seqs, tiles,
                lo, hi, l.heads, l.kv_heads, l.dim, l.dk, l.dv, splits, wide, eps,
                l.scale, st), "sigmoid_attn")
            N.count(2 if splits > 1 else 1)

    def _sigmoid_splits(self, blocks: int, longest: int, wide: int, page_bytes: int) -> int:
        """Key splits that fill the GPU; a split holds at least 128 keys (256 for prompt tiles).  In a captured tick
        (``attn_splits`` set) the context may grow later: the kernel itself leaves splits without keys out."""
        per_sm = 1 if wide or 3 * 4 * page_bytes > 96 * 1024 else 2
        if not self.attn_splits:
            per_split = 256 if wide else 128
            longest = (longest + per_split - 1) // per_split
        else:
            longest = 64
        return max(1, min(64, longest, per_sm * self.sms // max(1, blocks)))
