"""CUDA ops of sandwich-normed stream designs (``models/fetotar.py``): joins, latent attention, decayed scans.

Mixed into :class:`tilerl_b200.ops.cuda.CudaOps` beside :class:`~tilerl_b200.ops.cuda_stream.StreamOps`, whose projections
they use.  The activation type is that of the weights: bf16 (the serving type) or fp32 (true fp32 everywhere).  No
counterpart in the reference.
"""
from __future__ import annotations

import ctypes

import torch

from . import native as N
from .cuda_stream import EPI_STORE, EPI_STORE_F32

MAMBA2, MLSTM, FIXED = 0, 1, 2
CONV_SILU, CONV_ADD = 1, 2
ACTS = {"silu": 1, "gelu": 2, "gelu_erf": 3}
GLU_CLAMPED = 0
GLU_ACTS = {"silu": 1, "gelu": 2}
MIX_ROWS_MAX = 8        # rows the weight-streaming projection serves
LATENT_SHORT = 32       # tokens of a sequence up to which attention runs in the latent (absorbed) form
SCAN_SHORT = 16         # tokens of a sequence up to which a scan goes token by token
CONV_FUSED = 2          # sequences of a decode tick up to which the scan convolves its columns itself
CHUNK_DK = 128          # state rows the chunked scan takes
MAX_SPLITS = 32         # shares of a window its keys are split into (a warp merges them)
PART_BYTES = 1 << 28    # most fp32 partial sums of split attention


class ScanArgs(ctypes.Structure):
    """``ScanArgs`` of ``csrc/scan.cuh``."""
    _fields_ = ([(n, ctypes.c_void_p) for n in ("rows", "gates", "gate_b", "a_log", "skip", "states", "cur", "keep_flags",
                                                "q_start", "q_len", "slots", "o")]
                + [(n, ctypes.c_long) for n in ("slot_stride", "plane_stride")]
                + [(n, ctypes.c_int) for n in ("ld", "q0", "k0", "v0", "ldg", "heads", "per", "dk", "dv", "min_len", "max_len")]
                + [(n, ctypes.c_float) for n in ("cap", "q_scale")]
                + [(n, ctypes.c_int) for n in ("taps", "channels", "ring_rows", "ring_ld")]
                + [(n, ctypes.c_void_p) for n in ("conv_w", "conv_b", "ring")] + [("ring_slot", ctypes.c_long), ("positions", ctypes.c_void_p)])


def _f32(t: torch.Tensor) -> int:
    return int(t.dtype == torch.float32)


def _norm_kind(norm) -> int:
    return 0 if norm is None else norm.shape[0]


class MixerOps:
    def _streams_mix(self, rows: int, w) -> bool:
        """This many rows go through the weight-streaming projection, whose epilogues save a launch each."""
        return w.dtype == torch.bfloat16 and rows <= MIX_ROWS_MAX and rows <= self.lib.trl_linear_rows_max(w.shape[1])

    # ---- stream ----------------------------------------------------------------------
    def _join(self, x, y, post, nxt, h, table, ids, scale, eps, n):
        t, ld = x.shape
        N.check(self.lib.trl_join(x.data_ptr(), N.ptr(y), N.ptr(post), _norm_kind(post), N.ptr(nxt), _norm_kind(nxt), h.data_ptr(),
                                  N.ptr(table), N.ptr(ids), scale, 0 if table is None else table.shape[0], t, ld, n, eps, _f32(h),
                                  N.stream()), "join")
        N.count()
        return h

    def embed_stream(self, table, ids, scale, norm, eps, n):
        t, ld = ids.shape[0], table.shape[1]
        x, h = self.ws.get("stream", (t, ld), torch.float32), self.ws.get(f"join_h_{table.dtype}", (t, ld), table.dtype)
        self._join_dtype = table.dtype
        return x, self._join(x, None, None, norm, h, table, ids, scale, eps, n)

    def join(self, x, y, post, nxt, eps, n):
        """``x += norm_post(y)``; returns ``norm_nxt(x)`` (or x rounded) as the next projection's input."""
        h = self.ws.get(f"join_h_{self._join_dtype}", tuple(x.shape), self._join_dtype)
        return self._join(x, y, post, nxt, h, None, None, 1.0, eps, n)

    def _mm(self, a, w, y):
        if y.dtype == w.dtype:
            torch.mm(a, w.t(), out=y)
        else:
            torch.mm(a, w.t(), out_dtype=y.dtype, out=y)
        return y

    def project_gates(self, h, w, n_in):
        t, ng = h.shape[0], w.shape[0] - n_in
        proj = self.ws.get(f"block_proj_{w.dtype}", (t, n_in), w.dtype)
        gates = self.ws.get("mix_gates", (t, max(ng, 1)), torch.float32)
        if self._streams_mix(t, w):
            N.check(self.lib.trl_linear_rows_split(h.data_ptr(), h.stride(0), w.data_ptr(), proj.data_ptr(), n_in, n_in, gates.data_ptr(),
                                                   max(ng, 1), t, w.shape[0], w.shape[1], N.stream()), "linear_rows_split")
            N.count()
            return proj, gates
        self._mm(h, w[:n_in], proj)
        if ng:
            self._mm(h, w[n_in:], gates)
        return proj, gates

    def project(self, h, w):
        """Projection rows in the compute type."""
        y = self.ws.get(f"block_proj_{w.dtype}", (h.shape[0], w.shape[0]), w.dtype)
        if self._streams_mix(h.shape[0], w):
            self._linear_rows(h, w, y, EPI_STORE)
            return y
        return self._mm(h, w, y)

    def project_f32(self, a, w, name="branch"):
        y = self.ws.get(name, (a.shape[0], w.shape[0]), torch.float32)
        if self._streams_mix(a.shape[0], w):
            self._linear_rows(a, w, y, EPI_STORE_F32)
            return y
        return self._mm(a, w, y)

    def project_logits(self, h, w, cap=0.0):
        """``cap``: logits are soft-capped there (0: not)."""
        logits = self.ws.get("logits", (h.shape[0], w.shape[0]), torch.float32)
        h = h.contiguous()
        if self._streams_mix(h.shape[0], w):
            if cap:
                N.check(self.lib.trl_linear_rows_cap(h.data_ptr(), h.stride(0), w.data_ptr(), logits.data_ptr(), logits.stride(0), h.shape[0],
                                                     w.shape[0], w.shape[1], cap, N.stream()), "linear_rows_cap")
                N.count()
            else:
                self._linear_rows(h, w, logits, EPI_STORE_F32)
            return logits
        self._mm(h, w, logits)
        if cap:
            N.check(self.lib.trl_soft_cap(logits.data_ptr(), logits.numel(), cap, N.stream()), "soft_cap")
            N.count()
        return logits

    def clamped_glu(self, h, w, limit):
        return self._glu(h, w, GLU_CLAMPED, limit)

    def glu(self, h, w, act):
        """Rows ``2j`` = gate, ``2j + 1`` = up of ``w``: ``act(gate) * up``."""
        return self._glu(h, w, GLU_ACTS[act], 0.0)

    def _glu(self, h, w, act: int, limit: float):
        t, n = h.shape[0], w.shape[0]
        out = self.ws.get(f"glu_{w.dtype}", (t, n // 2), w.dtype)
        if self._streams_mix(t, w):
            N.check(self.lib.trl_linear_rows_glu(h.data_ptr(), h.stride(0), w.data_ptr(), out.data_ptr(), n // 2, t, n, w.shape[1], act, limit,
                                                 N.stream()), "linear_rows_glu")
            N.count()
            return out
        gu = self._mm(h, w, self.ws.get(f"gate_up_{w.dtype}", (t, n), w.dtype))
        N.check(self.lib.trl_glu(gu.data_ptr(), out.data_ptr(), out.numel(), act, limit, _f32(w), N.stream()), "glu")
        N.count()
        return out

    def side_input(self, h, w, table, ids, layer, dim):
        t, n = h.shape[0], w.shape[0]
        out, off = self.ws.get(f"side_{w.dtype}", (t, n), w.dtype), layer * ((dim + 7) // 8 * 8)
        if self._streams_mix(t, w):
            N.check(self.lib.trl_linear_rows_side(h.data_ptr(), h.stride(0), w.data_ptr(), out.data_ptr(), n, t, n, w.shape[1], ids.data_ptr(),
                                                  table.data_ptr(), table.shape[1], off, dim, table.shape[0], N.stream()), "linear_rows_side")
            N.count()
            return out
        z = self._mm(h, w, self.ws.get(f"side_z_{w.dtype}", (t, n), w.dtype))
        N.check(self.lib.trl_side_input(z.data_ptr(), table.data_ptr(), ids.data_ptr(), out.data_ptr(), t, n, dim, table.shape[1],
                                        off, table.shape[0], _f32(w), N.stream()), "side_input")
        N.count()
        return out

    # ---- latent attention ----------------------------------------------------------------
    def latent_prep(self, proj, l, q_norm, kv_norm, uq, freqs, rot, batch, pool, idx, eps):
        t, cache, st = proj.shape[0], pool.layer(idx), N.stream()
        cq = self.ws.get(f"latent_cq_{proj.dtype}", (t, l.c0), proj.dtype)
        N.check(self.lib.trl_latent_prep(
            proj.data_ptr(), proj.stride(0), q_norm.data_ptr(), kv_norm.data_ptr(), freqs.data_ptr(), batch.positions.data_ptr(),
            batch.slot_mapping.data_ptr(), cq.data_ptr(), cache.data_ptr(), cache.shape[0], t, l.c0, l.kr0, l.q_rank, l.kv_rank, l.kv,
            l.rd, freqs.numel(), rot.amplitude, eps, _f32(proj), st), "latent_prep")
        q = self.ws.get(f"latent_q_{proj.dtype}", (t, uq.shape[0]), proj.dtype)
        if self._streams_mix(t, uq):
            self._linear_rows(cq, uq, q, EPI_STORE)
        else:
            self._mm(cq, uq, q)
        N.count()
        return q.view(t, l.heads, l.dq)

    def _latent_rope(self, q, l, freqs, rot, positions) -> None:
        N.check(self.lib.trl_latent_rope(q.data_ptr(), freqs.data_ptr(), positions.data_ptr(), q.shape[0], l.heads, l.dq, l.dk, freqs.numel(),
                                         rot.amplitude, _f32(q), N.stream()), "latent_rope")
        N.count()

    def latent_attention(self, q, proj, up, ukt, l, freqs, rot, batch, pool, idx):
        if proj.dtype == torch.bfloat16 and self.lib.trl_latent_mma_ok(l.dk, l.rd, l.dv, l.kv):
            return self._latent_mma(q, proj, up, ukt, l, freqs, rot, batch, pool, idx)
        self._latent_rope(q, l, freqs, rot, batch.positions)
        t, cache, table, dt, st = proj.shape[0], pool.layer(idx), batch.block_table, proj.dtype, N.stream()
        uk, uv = up[:l.heads * l.dk].view(l.heads, l.dk, l.kv), up[l.heads * l.dk:].view(l.heads, l.dv, l.kv)
        ql = self.ws.get(f"latent_ql_{dt}", (l.heads, t, l.kv), dt)
        oc = self.ws.get(f"latent_oc_{dt}", (l.heads, t, l.kv), dt)
        ov = self.ws.get(f"latent_ov_{dt}", (l.heads, t, l.dv), dt)
        torch.bmm(q.transpose(0, 1)[:, :, :l.dk], uk, out=ql)
        N.check(self.lib.trl_latent_attn(
            ql.data_ptr(), t * l.kv, l.kv, q.data_ptr(), l.dq, l.dk, cache.data_ptr(), l.kv, l.rd, cache.shape[0], table.data_ptr(),
            table.stride(0), batch.q_start.data_ptr(), batch.q_len.data_ptr(), batch.positions.data_ptr(), oc.data_ptr(), t * l.kv, l.kv,
            batch.n_seqs, batch.max_q_len, l.heads, l.window, l.scale, _f32(proj), st), "latent_attn")
        torch.bmm(oc, uv.transpose(1, 2), out=ov)
        out = self.ws.get(f"mix_out_{dt}", (t, l.n_out), dt)
        N.check(self.lib.trl_latent_gate(ov.data_ptr(), proj[:, l.g0:].data_ptr(), proj.stride(0), out.data_ptr(), l.n_out, t, l.heads,
                                         l.dv, _f32(proj), st), "latent_gate")
        N.count(2)
        return out

    def _latent_mma(self, q, proj, up, ukt, l, freqs, rot, batch, pool, idx):
        """Short sequences in the absorbed form (one pass over the cached latents for all heads), prompts over expanded
        keys and values."""
        t, cache, table, st = proj.shape[0], pool.layer(idx), batch.block_table, N.stream()
        lens, kvs, bf = batch.host_q_len, batch.host_kv_len, torch.bfloat16
        out = self.ws.get(f"mix_out_{bf}", (t, l.n_out), bf)
        starts = [0]
        for n in lens:
            starts.append(starts[-1] + n)
        short = [i for i, n in enumerate(lens) if n <= LATENT_SHORT]
        prompts = [i for i, n in enumerate(lens) if n > LATENT_SHORT]
        if prompts:
            self._latent_rope(q, l, freqs, rot, batch.positions)
        if short:
            ts = max(starts[i + 1] for i in short)                           # tokens up to the last short sequence's
            blocks = sum((lens[i] * l.heads + 15) // 16 for i in short)
            keys = min(l.window + LATENT_SHORT, table.shape[1] * 16 if self.attn_splits else max(kvs[i] for i in short))
            splits = max(1, min(MAX_SPLITS, (keys + 63) // 64 + 1, self.sms // blocks, PART_BYTES // (ts * l.heads * l.kv * 4)))
            ql = self.ws.get("latent_rows", (ts, l.heads, l.row), bf)
            part = self.ws.get("attn_part", (ts * l.heads * splits * l.kv,), torch.float32)
            ml = self.ws.get("attn_part_ml", (ts * l.heads * splits * 2,), torch.float32)
            N.check(self.lib.trl_latent_decode(
                q.data_ptr(), l.dq, l.dk, l.rd, ukt.data_ptr(), up[l.heads * l.dk:].data_ptr(), l.kv, l.dv, freqs.data_ptr(),
                0 if prompts else freqs.numel(), rot.amplitude, ql.data_ptr(), cache.data_ptr(), cache.shape[0], table.data_ptr(),
                table.stride(0), batch.q_start.data_ptr(), batch.q_len.data_ptr(), batch.positions.data_ptr(), batch.seq_ids.data_ptr(),
                part.data_ptr(), ml.data_ptr(), proj[:, l.g0:].data_ptr(), proj.stride(0), out.data_ptr(), l.n_out, ts, batch.n_seqs,
                max((lens[i] * l.heads + 15) // 16 for i in short), l.heads, splits, l.window, 1, LATENT_SHORT if prompts else 1 << 30, l.scale,
                st), "latent_decode")
            N.count(3)
        if prompts:
            los = [max(0, kvs[i] - lens[i] - l.window + 1) for i in prompts]
            n_keys = [kvs[i] - lo for i, lo in zip(prompts, los)]
            total, ldkv = sum(n_keys), l.heads * (l.dk + l.dv)
            c, kr = self.ws.get("latent_c", (total, l.kv), bf), self.ws.get("latent_kr", (total, l.rd), bf)
            o = 0
            for i, lo, n in zip(prompts, los, n_keys):
                N.check(self.lib.trl_latent_gather(cache.data_ptr(), cache.shape[0], table[i].data_ptr(), lo, n, l.kv, l.rd, c[o:].data_ptr(),
                                                   kr[o:].data_ptr(), st), "latent_gather")
                o += n
            kvx = self._mm(c, up, self.ws.get("latent_kvx", (total, ldkv), bf))
            o = 0
            for i, lo, n in zip(prompts, los, n_keys):
                q0 = starts[i]
                N.check(self.lib.trl_latent_prompt(
                    q[q0:].data_ptr(), l.dq, l.dk, l.rd, l.dv, kvx[o:].data_ptr(), ldkv, kr[o:].data_ptr(), proj[q0:, l.g0:].data_ptr(),
                    proj.stride(0), out[q0:].data_ptr(), l.n_out, batch.positions[q0:].data_ptr(), lens[i], lo, n, l.heads, l.window, l.scale,
                    st), "latent_prompt")
                o += n
            N.count(2 * len(prompts))
        return out

    # ---- recurrent mixers ------------------------------------------------------------------
    def _scan(self, a: ScanArgs, batch, kind: int, dt, st) -> None:
        """Prompts chunk by chunk on tensor cores, everything else token by token."""
        chunked = dt == torch.bfloat16 and a.dk <= CHUNK_DK and not a.keep_flags
        prompts = sum(n > SCAN_SHORT for n in batch.host_q_len) if chunked else 0
        if prompts:
            a.min_len = SCAN_SHORT + 1 if prompts < batch.n_seqs else 1
            narrow = int(prompts * a.heads * ((a.dv + 63) // 64) < self.sms)
            N.check(self.lib.trl_scan_chunk(ctypes.byref(a), batch.n_seqs, kind, narrow, st), "scan_chunk")
            N.count()
        if prompts < batch.n_seqs:
            a.min_len, a.max_len = 1, SCAN_SHORT if prompts else 1 << 30
            N.check(self.lib.trl_scan_serial(ctypes.byref(a), batch.n_seqs, kind, int(dt == torch.float32), st), "scan_serial")
            N.count()

    def recurrent_mix(self, proj, gates, w, l, batch, pool, idx, eps):
        t, dt, st = proj.shape[0], proj.dtype, N.stream()
        kind = MAMBA2 if l.kind == "mamba2" else MLSTM
        ring = pool.ring_view(idx, 0) if kind == MAMBA2 else None
        o = self.ws.get("scan_o", (t, l.heads * l.dv), torch.float32)
        a = ScanArgs()
        if kind == MAMBA2 and batch.max_q_len == 1 and batch.n_seqs <= CONV_FUSED and not batch.keep_steps:
            # a small decode tick: the scan convolves its own columns (every slice of a head its keys anew)
            rows = proj
            a.taps, a.channels, a.conv_w, a.conv_b = l.taps, l.conv_c, w["conv"].data_ptr(), w["conv_b"].data_ptr()
            a.ring, a.ring_slot, a.ring_rows, a.ring_ld = ring.data_ptr(), pool.ring.stride(0), pool.ring_rows, pool.ring.stride(1)
            a.positions = batch.positions.data_ptr()
        elif kind == MAMBA2:
            rows = self.ws.get(f"scan_conv_{dt}", (t, l.conv_c), dt)
            N.check(self.lib.trl_scan_conv(
                proj.data_ptr(), proj.stride(0), w["conv"].data_ptr(), w["conv_b"].data_ptr(), None, ring.data_ptr(), pool.ring.stride(0),
                pool.ring_rows, pool.ring.stride(1), batch.positions.data_ptr(), batch.seq_ids.data_ptr(), batch.q_start.data_ptr(),
                batch.state_slots.data_ptr(), rows.data_ptr(), t, l.conv_c, l.taps, CONV_SILU, _f32(proj), st), "scan_conv")
            N.count()
        if kind == MAMBA2:
            a.q0, a.k0, a.v0, a.per, a.q_scale, a.cap = l.q0, l.k0, 0, l.heads // l.groups, 1.0, 1.0
        else:
            rows = proj
            a.q0, a.k0, a.v0, a.per, a.q_scale, a.cap = 0, l.k0, l.v0, 1, l.dim ** -0.5, l.cap
        a.rows, a.ld, a.gates, a.ldg = rows.data_ptr(), rows.stride(0), gates.data_ptr(), gates.stride(0)
        a.gate_b, a.a_log, a.skip = w["gate_b"].data_ptr(), N.ptr(w["a_log"]), N.ptr(w["skip"])
        self._scan_state(a, o, l, batch, pool, idx)
        self._scan(a, batch, kind, dt, st)
        return self._scan_norm(o, proj[:, l.g0:], w["norm"], l, batch, pool, eps, kind, proj, ring)

    @staticmethod
    def _scan_state(a: ScanArgs, o, l, batch, pool, idx) -> None:
        a.states, a.slot_stride, a.plane_stride = pool.states.data_ptr() + 4 * pool.offsets[idx], pool.states.stride(0), pool.states.stride(1)
        a.cur, a.keep_flags = pool.cur.data_ptr(), N.ptr(batch.keep_flags) if batch.keep_steps else None
        a.q_start, a.q_len, a.slots = batch.q_start.data_ptr(), batch.q_len.data_ptr(), batch.state_slots.data_ptr()
        a.o, a.heads, a.dk, a.dv, a.min_len, a.max_len = o.data_ptr(), l.heads, l.dk, l.dv, 1, 1 << 30

    def _scan_norm(self, o, gate, norm, l, batch, pool, eps, kind: int, proj=None, ring=None):
        """Normed and gated output of a scan (``kind`` MAMBA2: a tick's convolution inputs ``proj`` go into the ring, too)."""
        t, dt = gate.shape[0], gate.dtype
        out = self.ws.get(f"mix_out_{dt}", (t, l.n_out), dt)
        N.check(self.lib.trl_scan_norm(
            o.data_ptr(), gate.data_ptr(), gate.stride(0), norm.data_ptr(), out.data_ptr(), l.n_out, t, l.heads, l.vdim, l.dv,
            l.norm_groups, eps, N.ptr(proj), N.ptr(ring), pool.ring.stride(0), pool.ring_rows, pool.ring.stride(1), l.conv_c,
            batch.positions.data_ptr(), batch.seq_ids.data_ptr(), batch.q_start.data_ptr(), batch.q_len.data_ptr(),
            batch.state_slots.data_ptr(), kind, _f32(gate), N.stream()), "scan_norm")
        N.count()
        return out
