"""CUDA ops of ``models/tobadra.py``: gated branches with a convolution on the next input, attention over turned values, lightning
attention, the per-channel delta rule, experts behind a grouped router.

Mixed into :class:`tilerl_b200.ops.cuda.CudaOps` beside :class:`~tilerl_b200.ops.cuda_blocks.BlockOps`, whose attention and experts
they use.  The activation type is that of the weights: bf16 (the serving type) or fp32 (true fp32 everywhere).  No counterpart in
the reference.
"""
from __future__ import annotations

import ctypes

import torch

from . import native as N
from .cuda_blocks import PrepArgs, _fields
from .cuda_mixers import ACTS, CONV_ADD, FIXED, MLSTM, ScanArgs, _f32, _norm_kind


class JoinArgs(ctypes.Structure):
    """``JoinArgs`` of ``csrc/join.cu``."""
    _fields_ = _fields("x y post next h table ids place weight own bias z z_b hc conv_w ring positions seq_ids state_slots ring_slot:l post_kind:i "
                       "next_kind:i V:i ld:i n:i slots:i y_bf16:i ldz:i taps:i ring_rows:i ring_ld:i scale:f eps:f")


class DeltaArgs(ctypes.Structure):
    """``DeltaArgs`` of ``csrc/delta.cuh``."""
    _fields_ = _fields("rows conv_w ring low dt_bias a_log gates q k v keep beta states cur keep_flags q_start q_len slots positions seq_ids o chunk "
                       "ring_slot:l slot_stride:l plane_stride:l ldp:i ldg:i k0:i v0:i channels:i taps:i ring_rows:i ring_ld:i write_ring:i heads:i "
                       "kv_heads:i dk:i dv:i min_len:i max_len:i q_scale:f")


class DeltaSel(ctypes.Structure):
    """``DeltaSel`` of ``csrc/delta_mma.cu``."""
    _fields_ = _fields("n:i c0:i nc:i pad:i") + [("seq", ctypes.c_int * 64)]


DELTA_SHORT = 16            # tokens of a sequence up to which the delta rule goes token by token
DELTA_DK = 128              # state rows its chunked form takes
DELTA_BYTES = 1 << 28       # most scratch of a launch's chunks


class GatedOps:
    # ---- joins ---------------------------------------------------------------------------
    def _join_conv(self, a: JoinArgs, x, h, post, nxt, eps, n, conv):
        """Runs the join; returns (h, h plus its convolution)."""
        t, ld = x.shape
        a.x, a.h, a.post, a.post_kind, a.next, a.next_kind = x.data_ptr(), h.data_ptr(), N.ptr(post), _norm_kind(post), N.ptr(nxt), _norm_kind(nxt)
        a.ld, a.n, a.eps, hc = ld, n, eps, None
        if conv is not None:
            w, batch, spool, idx = conv
            hc, ring = self.ws.get(f"join_hc_{h.dtype}", (t, ld), h.dtype), spool.ring_view(idx, 0)
            if batch.max_q_len == 1:           # a row's only reader of the ring is the block that writes it
                a.hc, a.conv_w, a.taps, a.ring, a.ring_slot = hc.data_ptr(), w.data_ptr(), w.shape[0], ring.data_ptr(), spool.ring.stride(0)
                a.ring_rows, a.ring_ld = spool.ring_rows, spool.ring.stride(1)
                a.positions, a.seq_ids, a.state_slots = batch.positions.data_ptr(), batch.seq_ids.data_ptr(), batch.state_slots.data_ptr()
        N.check(self.lib.trl_join_args(ctypes.byref(a), t, _f32(h), N.stream()), "join")
        N.count()
        if hc is not None and not a.taps:
            N.check(self.lib.trl_scan_conv(
                h.data_ptr(), ld, w.data_ptr(), None, None, ring.data_ptr(), spool.ring.stride(0), spool.ring_rows, spool.ring.stride(1),
                batch.positions.data_ptr(), batch.seq_ids.data_ptr(), batch.q_start.data_ptr(), batch.state_slots.data_ptr(), hc.data_ptr(), t, ld,
                w.shape[0], CONV_ADD, _f32(h), N.stream()), "scan_conv")
            N.count()
            self._ring_store(h, ld, ring, spool, batch)
        return h, hc

    def embed_normed(self, table, vocab, ids, post, nxt, eps, n, conv):
        """(stream, its normed row, that row convolved): the normed embedding."""
        t, ld, dt = ids.shape[0], table.shape[1], table.dtype
        self._join_dtype = dt
        x, h = self.ws.get("stream", (t, ld), torch.float32), self.ws.get(f"join_h_{dt}", (t, ld), dt)
        a = JoinArgs()
        a.table, a.ids, a.V, a.scale = table.data_ptr(), ids.data_ptr(), vocab, 1.0
        return (x, *self._join_conv(a, x, h, post, nxt, eps, n, conv))

    def gated_join(self, x, y, bias, z, z_b, post, nxt, eps, n, conv):
        """``x += norm_post((y + bias) sigmoid(z + z_b))``; returns (``norm_nxt(x)``, that row convolved)."""
        a = JoinArgs()
        a.y, a.bias, a.z, a.ldz, a.z_b = y.data_ptr(), N.ptr(bias), z.data_ptr(), z.stride(0), z_b.data_ptr()
        return self._join_conv(a, x, self.ws.get(f"join_h_{self._join_dtype}", tuple(x.shape), self._join_dtype), post, nxt, eps, n, conv)

    def gated_join_experts(self, x, branch, h, z, z_b, post, nxt, eps, n, conv):
        """The same with the weighted sum over a token's experts, and its own share of ``h``, as the branch."""
        y, place, weight = branch
        a = JoinArgs()
        a.y, a.y_bf16, a.place, a.weight, a.slots, a.own = y.data_ptr(), int(y.dtype == torch.bfloat16), place.data_ptr(), weight.data_ptr(), weight.shape[1], h.data_ptr()
        a.z, a.ldz, a.z_b = z.data_ptr(), z.stride(0), z_b.data_ptr()
        return self._join_conv(a, x, self.ws.get(f"join_h_{self._join_dtype}", tuple(x.shape), self._join_dtype), post, nxt, eps, n, conv)

    # ---- projections ---------------------------------------------------------------------
    def _streams_two(self, rows: int, w) -> bool:
        """The weight-streaming projection takes this many rows of two inputs."""
        return self._streams_mix(rows, w) and 2 * rows <= self.lib.trl_linear_rows_max(w.shape[1])

    def _linear_mix(self, x, x2, n_x2, w, y, n_split, y2, n_act=0, act=0) -> None:
        N.check(self.lib.trl_linear_rows_mix(x.data_ptr(), x.stride(0), N.ptr(x2), n_x2, w.data_ptr(), N.ptr(y), 0 if y is None else y.stride(0), n_split,
                                             N.ptr(y2), 0 if y2 is None else y2.stride(0), x.shape[0], w.shape[0], w.shape[1], n_act, act, N.stream()),
                "linear_rows_mix")
        N.count()

    def _act(self, z, n: int, act: int) -> None:
        N.check(self.lib.trl_act(z.data_ptr(), z.stride(0), z.shape[0], n, act, _f32(z), N.stream()), "act")
        N.count()

    def project_in(self, h, hc, w, n_in, n_gates, n_act=0, act="silu"):
        """(rows of the mixer, the first ``n_act`` through ``act``; fp32 rows of its gates; fp32 rows of its branch's gate): the last
        rows of ``w`` read ``h``, the others ``hc``."""
        t, n = h.shape[0], n_in + n_gates
        proj = self.ws.get(f"block_proj_{w.dtype}", (t, n_in), w.dtype)
        if self._streams_two(t, w):
            y2 = self.ws.get("in_gates", (t, w.shape[0] - n_in), torch.float32)
            self._linear_mix(hc, h, n, w, proj, n_in, y2, n_act, ACTS[act] if n_act else 0)
            return proj, y2[:, :n_gates], y2[:, n_gates:]
        z = self.ws.get("branch_gate", (t, w.shape[0] - n), torch.float32)
        gates = self.ws.get("mix_gates", (t, max(n_gates, 1)), torch.float32)
        self._mm(hc, w[:n_in], proj)
        if n_act:
            self._act(proj, n_act, ACTS[act])
        if n_gates:
            self._mm(hc, w[n_in:n], gates)
        self._mm(h, w[n:], z)
        return proj, gates, z

    def up_act(self, h, w, n, act):
        """(``act`` of the first ``n`` rows, the other rows in fp32)."""
        t = h.shape[0]
        up, z = self.ws.get(f"glu_{w.dtype}", (t, n), w.dtype), self.ws.get("branch_gate", (t, w.shape[0] - n), torch.float32)
        if self._streams_mix(t, w):
            self._linear_mix(h, None, 0, w, up, n, z, n, ACTS[act])
            return up, z
        self._mm(h, w[:n], up)
        self._act(up, n, ACTS[act])
        self._mm(h, w[n:], z)
        return up, z

    # ---- attention over turned values --------------------------------------------------------
    def turned_prep(self, proj, l, bias, freqs, vfreqs, batch, pool, idx):
        """Biased and turned queries ``[T, heads * dk]``; turned keys and values into the cache; the input of the output projection, its
        padding columns cleared; cos and sin of the values' turns."""
        al, s, t, dt = l.attn, l.attn.spec, proj.shape[0], proj.dtype
        q, mid = self.ws.get(f"attn_q_{dt}", (t, al.k0), dt), self.ws.get(f"mix_out_{dt}", (t, l.n_out), dt)
        turn = self.ws.get("attn_turn", (t, al.dv // 2, 2), torch.float32)
        a = PrepArgs()
        a.proj, a.ldp, a.heads, a.kv_heads, a.dim, a.dk, a.dv = proj.data_ptr(), proj.stride(0), s.heads, s.kv_heads, s.dim, al.dk, al.dv
        a.k0, a.v0, a.n_in, a.own, a.bias = al.k0, al.v0, al.n_in, 1, bias.data_ptr()
        a.freqs, a.n_pairs, a.half, a.vfreqs, a.turn = freqs.data_ptr(), freqs.numel(), 1, vfreqs.data_ptr(), turn.data_ptr()
        a.positions, a.seq_ids, a.q_start = batch.positions.data_ptr(), batch.seq_ids.data_ptr(), batch.q_start.data_ptr()
        a.slots, a.slot_mapping, a.q = batch.state_slots.data_ptr(), batch.slot_mapping.data_ptr(), q.data_ptr()
        cache = pool.layer(idx)
        a.pages, a.n_blocks, a.mid, a.ldm, a.pad0 = cache.data_ptr(), cache.shape[0], mid.data_ptr(), l.n_out, l.n_mid
        N.check(self.lib.trl_qkv_prep(ctypes.byref(a), t, _f32(proj), N.stream()), "qkv_prep")
        N.count()
        return q, mid, turn

    # ---- recurrent mixers ------------------------------------------------------------------
    def lightning_mix(self, proj, log_decay, norm, l, batch, pool, idx, eps):
        t = proj.shape[0]
        o = self.ws.get("scan_o", (t, l.heads * l.dv), torch.float32)
        a = ScanArgs()
        a.q0, a.k0, a.v0, a.per, a.q_scale, a.cap = 0, l.k0, l.v0, 1, 1.0, 1.0
        a.rows, a.ld, a.a_log = proj.data_ptr(), proj.stride(0), log_decay.data_ptr()
        self._scan_state(a, o, l, batch, pool, idx)
        self._scan(a, batch, FIXED, proj.dtype, N.stream())
        return self._scan_norm(o, proj[:, l.g0:], norm, l, batch, pool, eps, MLSTM)

    def delta_mix(self, proj, gates, w, norm, l, batch, pool, idx, eps):
        t, dt, st, low = proj.shape[0], proj.dtype, N.stream(), w["low"]
        f32 = lambda name, n: self.ws.get(name, (t, n), torch.float32)
        # output gate and decays from the two maps' columns
        z, keep = self.ws.get(f"delta_gate_{dt}", (t, l.n_low), dt), f32("delta_keep", l.heads * l.dk)
        if self._streams_two(t, low):
            self._linear_mix(proj[:, l.g0:], proj[:, l.a0:], l.n_low, low, z, l.n_low, keep)
        else:
            self._mm(proj[:, l.g0:l.n_in], low[:l.n_low], z)
            self._mm(proj[:, l.a0:l.g0], low[l.n_low:], keep)
        ring, single = pool.ring_view(idx, 0), batch.max_q_len == 1
        a = DeltaArgs()
        a.rows, a.ldp, a.conv_w, a.taps, a.channels, a.k0, a.v0 = proj.data_ptr(), proj.stride(0), w["conv"].data_ptr(), l.taps, l.conv_c, l.k0, l.v0
        a.ring, a.ring_slot, a.ring_rows, a.ring_ld, a.write_ring = ring.data_ptr(), pool.ring.stride(0), pool.ring_rows, pool.ring.stride(1), int(single)
        a.low, a.dt_bias, a.a_log, a.gates, a.ldg = keep.data_ptr(), w["dt_bias"].data_ptr(), w["a_log"].data_ptr(), gates.data_ptr(), gates.stride(0)
        a.states, a.slot_stride, a.plane_stride = pool.states.data_ptr() + 4 * pool.offsets[idx], pool.states.stride(0), pool.states.stride(1)
        a.cur, a.keep_flags = pool.cur.data_ptr(), N.ptr(batch.keep_flags) if batch.keep_steps else None
        a.q_start, a.q_len, a.slots, a.positions, a.seq_ids = (x.data_ptr() for x in (batch.q_start, batch.q_len, batch.state_slots, batch.positions, batch.seq_ids))
        a.heads, a.kv_heads, a.dk, a.dv, a.min_len, a.max_len, a.q_scale = l.heads, l.kv_heads, l.dk, l.dv, 1, 1 << 30, l.spec.dim ** -0.5
        if single and not batch.keep_steps and self.lib.trl_delta_step_ok(l.dk, l.dv):
            out = self.ws.get(f"mix_out_{dt}", (t, l.n_out), dt)
            N.check(self.lib.trl_delta_step(ctypes.byref(a), batch.n_seqs, z.data_ptr(), z.stride(0), norm.data_ptr(), out.data_ptr(), l.n_out, l.vdim, eps,
                                            _f32(proj), st), "delta_step")
            N.count()
            return out
        o, q, k, beta = f32("scan_o", l.heads * l.dv), f32("delta_q", l.k0), f32("delta_k", l.k0), f32("delta_beta", l.heads)
        v = self.ws.get(f"delta_v_{dt}", (t, l.heads * l.dv), dt)
        a.keep, a.q, a.k, a.v, a.beta, a.o = keep.data_ptr(), q.data_ptr(), k.data_ptr(), v.data_ptr(), beta.data_ptr(), o.data_ptr()
        N.check(self.lib.trl_delta_prep(ctypes.byref(a), t, _f32(proj), st), "delta_prep")
        N.count()
        if not single:
            self._ring_store(proj, l.conv_c, ring, pool, batch)
        self._delta_scan(a, batch, dt, st)
        return self._scan_norm(o, z, norm, l, batch, pool, eps, MLSTM)

    def _delta_scan(self, a: DeltaArgs, batch, dt, st) -> None:
        """Prompts chunk by chunk on tensor cores, everything else token by token."""
        lens, lib = batch.host_q_len, self.lib
        long = [i for i, n in enumerate(lens) if n > DELTA_SHORT] if dt == torch.bfloat16 and a.dk <= DELTA_DK and not a.keep_flags else []
        step = lib.trl_delta_chunk_tokens()
        for g in range(0, len(long), 64):
            seqs = long[g:g + 64]
            chunks = max((lens[i] + step - 1) // step for i in seqs)
            per = len(seqs) * a.heads * lib.trl_delta_record(a.dk, a.dv)
            nc = max(1, min(chunks, DELTA_BYTES // per))
            a.chunk = self.ws.get("delta_chunks", (nc * per // 4,), torch.float32).data_ptr()
            narrow = int(len(seqs) * a.heads * ((a.dv + 31) // 32) <= 2 * self.sms)          # (two blocks share an SM)
            for c0 in range(0, chunks, nc):
                sel = DeltaSel(len(seqs), c0, min(nc, chunks - c0), 0, (ctypes.c_int * 64)(*seqs))
                N.check(lib.trl_delta_chunk(ctypes.byref(a), ctypes.byref(sel), narrow, st), "delta_chunk")
                N.count(2)
        if len(long) < len(lens):
            a.min_len, a.max_len = 1, DELTA_SHORT if long else 1 << 30
            N.check(lib.trl_delta_serial(ctypes.byref(a), batch.n_seqs, int(dt == torch.float32), st), "delta_serial")
            N.count()

    # ---- experts -----------------------------------------------------------------------------
    def routed_experts(self, h, z, correction, up, down, m):
        """Outputs of a tick's experts, ordered by expert, with the place and weight of every token's (negative: its own row); ``z``: rows
        of the fused router."""
        return self._expert_rows(h, z, correction, up, down, m)
