"""CUDA ops of ``models/deluvik.py`` (and, as far as it has them, ``models/tobadra.py``): softmax attention with its preparation, gated linear recurrence, mixtures of experts.

Mixed into :class:`tilerl_b200.ops.cuda.CudaOps` beside :class:`~tilerl_b200.ops.cuda_mixers.MixerOps`, whose projections and joins
they use.  The activation type is that of the weights: bf16 (the serving type) or fp32 (true fp32 everywhere).  No counterpart in
the reference.
"""
from __future__ import annotations

import ctypes

import torch

from . import native as N
from .cuda_mixers import ACTS, GLU_ACTS, _f32
from .cuda_stream import SHORT_ROWS

P, I, L, F = ctypes.c_void_p, ctypes.c_int, ctypes.c_long, ctypes.c_float
MOE_UP, MOE_DOWN, MOE_ACT = 0, 1, 2
MOE_TC_MIN = 16         # tokens from which on experts run as tensor-core tiles
MOE_TILE = 8            # rows of a tile of the weight-streaming expert projections


def _fields(spec: str):
    """``"name name:type ..."``: pointers unless a type is given."""
    kinds = {"p": P, "i": I, "l": L, "f": F}
    return [(n, kinds[k or "p"]) for n, _, k in (x.partition(":") for x in spec.split())]


class PrepArgs(ctypes.Structure):
    """``PrepArgs`` of ``csrc/attn_softmax.cu``."""
    _fields_ = _fields("proj ldp:i heads:i kv_heads:i dim:i dk:i dv:i k0:i v0:i n_in:i own:i taps:i conv ring ring_slot:l ring_rows:i ring_ld:i "
                       "write_ring:i q_norm k_norm norm_all:i freqs n_pairs:i half:i eps:f positions seq_ids q_start slots slot_mapping q pages "
                       "n_blocks:i mid ldm:i pad0:i bias vfreqs turn")


class LruArgs(ctypes.Structure):
    """``LruArgs`` of ``csrc/lru.cu``."""
    _fields_ = _fields("y y_b u z gates_b lam gates conv conv_b x_b ring ring_slot:l states slot_stride:l plane_stride:l cur keep_flags q_start "
                       "q_len slots positions out ldp:i ldo:i T:i width:i pp:i taps:i ring_rows:i ring_ld:i factor:f")


class MoePlan(ctypes.Structure):
    """``MoePlanArgs`` of ``csrc/moe.cu``."""
    _fields_ = _fields("z bias ids weight place token items n_items T:i ldz:i experts:i top:i pieces:i tile:i max_items:i "
                       "outputs:i groups:i keep:i gate_col:i scale:f")


class BlockOps:
    # ---- softmax attention ---------------------------------------------------------------
    def _ring_store(self, rows, channels, ring, pool, batch) -> None:
        N.check(self.lib.trl_ring_store(
            rows.data_ptr(), rows.stride(0), ring.data_ptr(), pool.ring.stride(0), pool.ring_rows, pool.ring.stride(1), channels,
            batch.positions.data_ptr(), batch.seq_ids.data_ptr(), batch.q_start.data_ptr(), batch.q_len.data_ptr(), batch.state_slots.data_ptr(),
            rows.shape[0], _f32(rows), N.stream()), "ring_store")
        N.count()

    def attn_prep(self, proj, l, w, freqs, batch, pool, idx, spool, sidx, eps):
        """Convolved, normed and turned queries ``[T, heads * dk]``; keys and values of layers that have their own into the
        cache.  Also the input of the layer's output projection, its padding columns cleared."""
        al, s, t, dt = l.attn, l.attn.spec, proj.shape[0], proj.dtype
        q, mid = self.ws.get(f"attn_q_{dt}", (t, al.k0), dt), self.ws.get(f"mix_out_{dt}", (t, l.n_out), dt)
        a = PrepArgs()
        a.proj, a.ldp, a.heads, a.kv_heads, a.dim, a.dk, a.dv = proj.data_ptr(), proj.stride(0), s.heads, s.kv_heads, s.dim, al.dk, al.dv
        a.k0, a.v0, a.n_in, a.own, a.taps = al.k0, al.v0, al.n_in, int(al.own), s.conv
        single = batch.max_q_len == 1          # a row's only reader of the ring is the block that writes it
        if s.conv:
            ring = spool.ring_view(sidx, 0)
            a.conv, a.ring, a.ring_slot, a.ring_rows, a.ring_ld = (w["conv"].data_ptr(), ring.data_ptr(), spool.ring.stride(0), spool.ring_rows,
                                                                   spool.ring.stride(1))
            a.write_ring = int(single)
        a.q_norm, a.k_norm, a.norm_all, a.eps = w["q_norm"].data_ptr(), N.ptr(w["k_norm"]), int(s.norm == "all"), eps
        a.freqs, a.n_pairs, a.half = freqs.data_ptr(), freqs.numel(), int(s.rot.half)
        a.positions, a.seq_ids, a.q_start = batch.positions.data_ptr(), batch.seq_ids.data_ptr(), batch.q_start.data_ptr()
        a.slots, a.slot_mapping, a.q = batch.state_slots.data_ptr(), batch.slot_mapping.data_ptr(), q.data_ptr()
        cache = pool.layer(idx)
        a.pages, a.n_blocks, a.mid, a.ldm, a.pad0 = cache.data_ptr(), cache.shape[0], mid.data_ptr(), l.n_out, l.n_mid
        N.check(self.lib.trl_qkv_prep(ctypes.byref(a), t, _f32(proj), N.stream()), "qkv_prep")
        N.count()
        if s.conv and not single:
            self._ring_store(proj, al.n_in, ring, spool, batch)
        return q, mid

    def softmax_attention(self, q, mid, al, sink, factor, batch, pool, idx, turn=None):
        """Attention output of every token, times ``factor``, into the first columns of ``mid``; with ``turn`` (cos and sin per token
        and pair ``[T, dv / 2, 2]``) turned back first."""
        s, cache, table, lib = al.spec, pool.layer(idx), batch.block_table, self.lib
        t, g = q.shape[0], s.heads // s.kv_heads
        lens, kvs = batch.host_q_len, batch.host_kv_len
        if q.dtype == torch.float32 or not lib.trl_softmax_attn_ok(al.dk, al.dv):
            classes = [(2, list(range(len(lens))))]
        else:
            short = max(1, SHORT_ROWS // g)          # tokens of a sequence that fit the narrow row tile
            classes = [(wide, [i for i, n in enumerate(lens) if (n > short) == bool(wide)]) for wide in (0, 1)]
            classes = [c for c in classes if c[1]]
        for wide, sel in classes:
            # alone, a launch takes every length: in a captured verify tick the lengths on the device are the true ones
            lo, hi = (1, 1 << 30) if len(classes) == 1 else ((short + 1, 1 << 30) if wide else (1, short))
            rows = lib.trl_softmax_attn_rows(al.dk, al.dv) if wide == 1 else 16
            tiles, splits, part, ml = max((lens[i] * g + rows - 1) // rows for i in sel), 1, None, None
            if wide != 2:
                seen = lambda i: kvs[i] if s.window is None else min(kvs[i], s.window + 16 + rows // g)
                longest = max(seen(i) for i in sel)
                if self.attn_splits:                 # captured: the context may grow up to the window
                    longest = 1 << 20 if s.window is None else s.window + 16 + rows // g
                splits = self._softmax_splits(sum((lens[i] * g + rows - 1) // rows for i in sel) * s.kv_heads, longest, wide, pool.pages[idx].nbytes)
            if splits > 1:
                part = self.ws.get("attn_part", (t * s.heads * splits * al.dv,), torch.float32)
                ml = self.ws.get("attn_part_ml", (t * s.heads * splits * 2,), torch.float32)
            N.check(lib.trl_softmax_attn(
                q.data_ptr(), cache.data_ptr(), cache.shape[0], table.data_ptr(), table.stride(0), batch.q_start.data_ptr(),
                batch.q_len.data_ptr(), batch.positions.data_ptr(), batch.seq_ids.data_ptr(), N.ptr(sink), mid.data_ptr(), mid.stride(0),
                N.ptr(part), N.ptr(ml), t, batch.n_seqs, tiles, lo, hi, s.heads, s.kv_heads, al.dk, al.dv, splits, wide, s.window or 0,
                s.scale, s.cap or 0.0, factor, N.ptr(turn), _f32(q), N.stream()), "softmax_attn")
            N.count(2 if splits > 1 else 1)

    def _softmax_splits(self, blocks: int, longest: int, wide: int, page_bytes: int) -> int:
        """Key splits that fill the GPU; a split holds at least 128 keys (256 for prompt tiles).  The kernel itself leaves splits
        without keys out."""
        per_sm = 1 if wide or 3 * 4 * page_bytes > 96 * 1024 else 2
        per_split = 256 if wide else 128
        return max(1, min(64, (longest + per_split - 1) // per_split, per_sm * self.sms // max(1, blocks)))

    # ---- gated linear recurrence -----------------------------------------------------------
    def lru_mix(self, proj, mid, l, w, batch, spool, sidx):
        """Recurrence x gelu branch, times the layer's factor, into the columns of ``mid`` behind the attention's."""
        r, t, dt, y0, st = l.lru, proj.shape[0], proj.dtype, l.attn.n_in, N.stream()
        y, x, ring = proj[:, y0:y0 + r.width], proj[:, y0 + r.width:y0 + 2 * r.width], spool.ring_view(sidx, 0)
        a = LruArgs()
        a.y, a.y_b, a.gates_b, a.lam = y.data_ptr(), w["y_b"].data_ptr(), w["gates_b"].data_ptr(), w["lam"].data_ptr()
        a.states, a.slot_stride, a.plane_stride = spool.states.data_ptr() + 4 * spool.offsets[sidx], spool.states.stride(0), spool.states.stride(1)
        a.cur, a.q_start, a.q_len = spool.cur.data_ptr(), batch.q_start.data_ptr(), batch.q_len.data_ptr()
        a.slots, a.positions, a.out = batch.state_slots.data_ptr(), batch.positions.data_ptr(), mid[:, l.attn.n_out:].data_ptr()
        a.ldp, a.ldo, a.T, a.width, a.pp, a.taps, a.factor = proj.stride(0), mid.stride(0), t, r.width, r.pp, r.spec.conv, l.lru_scale
        a.ring_slot, a.ring_rows, a.ring_ld = spool.ring.stride(0), spool.ring_rows, spool.ring.stride(1)
        if batch.max_q_len == 1 and not batch.keep_steps:
            a.u, a.gates, a.conv, a.conv_b, a.x_b = (x.data_ptr(), w["gates"].data_ptr(), w["lru_conv"].data_ptr(), w["lru_conv_b"].data_ptr(),
                                                     w["x_b"].data_ptr())
            a.ring = ring.data_ptr()
            N.check(self.lib.trl_lru_step(ctypes.byref(a), batch.n_seqs, _f32(proj), st), "lru_step")
            N.count()
            return
        u = self.ws.get(f"scan_conv_{dt}", (t, r.width), dt)
        N.check(self.lib.trl_scan_conv(
            x.data_ptr(), proj.stride(0), w["lru_conv"].data_ptr(), w["lru_conv_b"].data_ptr(), w["x_b"].data_ptr(), ring.data_ptr(),
            spool.ring.stride(0), spool.ring_rows, spool.ring.stride(1), batch.positions.data_ptr(), batch.seq_ids.data_ptr(),
            batch.q_start.data_ptr(), batch.state_slots.data_ptr(), u.data_ptr(), t, r.width, r.spec.conv, 0, _f32(proj), st), "scan_conv")
        self._ring_store(x, r.width, ring, spool, batch)
        b = r.spec.blocks
        z = self.ws.get("lru_gates", (b, t, 2 * r.pp), torch.float32)
        ub, wb = u.view(t, b, r.pp).transpose(0, 1), w["gates"].transpose(1, 2)
        if dt == torch.float32:
            torch.bmm(ub, wb, out=z)
        else:
            torch.bmm(ub, wb, out_dtype=torch.float32, out=z)
        a.u, a.z, a.keep_flags = u.data_ptr(), z.data_ptr(), N.ptr(batch.keep_flags) if batch.keep_steps else None
        N.check(self.lib.trl_lru_scan(ctypes.byref(a), batch.n_seqs, _f32(proj), st), "lru_scan")
        N.count(2)

    # ---- experts -----------------------------------------------------------------------------
    def _moe_plan(self, h, router, router_b, m, tile: int):
        """Router, choice and order by expert of a tick's (token, expert) pairs, in tiles of at most ``tile`` rows."""
        return self._moe_order(self.project_f32(h, router, "moe_router"), router_b, m, tile)

    def _moe_order(self, z, bias, m, tile: int):
        """The same from router logits; with the spec's ``router``, ``bias`` is the correction of its choice."""
        t, s = z.shape[0], m.spec
        pairs = t * m.slots
        a = MoePlan()
        a.max_items = min(pairs, m.n) + pairs // tile
        ints = self.ws.get("moe_ints", (3 * pairs + 4,), torch.int32)
        weight, items = self.ws.get("moe_weight", (t, m.slots), torch.float32), self.ws.get("moe_items", (a.max_items, 4), torch.int32)
        n_items, ids, place, token = ints[:1], ints[4:4 + pairs], ints[4 + pairs:4 + 2 * pairs], ints[4 + 2 * pairs:]
        a.z, a.bias, a.ids, a.weight, a.place = z.data_ptr(), bias.data_ptr(), ids.data_ptr(), weight.data_ptr(), place.data_ptr()
        a.token, a.items, a.n_items = token.data_ptr(), items.data_ptr(), n_items.data_ptr()
        a.T, a.ldz, a.experts, a.top, a.pieces, a.tile = t, z.stride(0), s.experts, s.top, m.pieces, tile
        if s.router is not None:
            a.outputs, a.groups, a.keep, a.scale, a.gate_col = s.outputs, s.router.groups, s.router.keep, s.router.scale, s.outputs if s.shared_gate else -1
        N.check(self.lib.trl_moe_plan(ctypes.byref(a), N.stream()), "moe_plan")
        N.count(1 if t <= 64 else 2)
        return a, place, weight

    def _moe_rows(self, x, w, y, plan, kind: int, act: int, m) -> None:
        likely = min(plan.T * m.slots, m.n)
        N.check(self.lib.trl_moe_rows(x.data_ptr(), x.stride(0), w.data_ptr(), y.data_ptr(), y.stride(0), plan.items, plan.n_items, plan.token,
                                      w.shape[1], w.shape[2], kind, act, likely, _f32(w), N.stream()), "moe_rows")
        N.count()

    def experts(self, h, router, router_b, gate_up, down, m):
        """Outputs of a tick's experts, ordered by expert, with the place and weight of every token's
        (:meth:`join_experts` sums them)."""
        return self._expert_rows(h, self.project_f32(h, router, "moe_router"), router_b, gate_up, down, m)

    def _expert_rows(self, h, z, bias, up, down, m):
        pairs, dt, act = h.shape[0] * m.slots, h.dtype, m.spec.act
        kind, act = (MOE_UP, GLU_ACTS[act]) if m.spec.gated else (MOE_ACT, ACTS[act])
        if dt == torch.bfloat16 and h.shape[0] >= MOE_TC_MIN:
            return self._experts_tc(h, z, bias, up, down, m, kind, act)
        plan, place, weight = self._moe_order(z, bias, m, MOE_TILE)
        mid = self.ws.get(f"moe_mid_{dt}", (pairs, m.ff), dt)
        y = self.ws.get("moe_out", (pairs, down.shape[1]), torch.float32)
        self._moe_rows(h, up, mid, plan, kind, act, m)
        self._moe_rows(mid, down, y, plan, MOE_DOWN, 0, m)
        return y, place, weight

    def _experts_tc(self, h, z, bias, up, down, m, kind: int, act: int):
        """Many rows: tensor-core tiles of each expert's rows, gathered in order first; output rows in bf16."""
        pairs, w, bf, lib, st = h.shape[0] * m.slots, h.shape[1], torch.bfloat16, self.lib, N.stream()
        plan, place, weight = self._moe_order(z, bias, m, lib.trl_moe_tc_tile())
        rows, mid, y = (self.ws.get(n, (pairs, k), bf) for n, k in (("moe_rows", w), ("moe_mid_tc", m.ff), ("moe_out_tc", down.shape[1])))
        N.check(lib.trl_moe_gather(h.data_ptr(), h.stride(0), plan.token, rows.data_ptr(), pairs, w, st), "moe_gather")
        for x, wt, out, k, f in ((rows, up, mid, kind, act), (mid, down, y, MOE_DOWN, 0)):
            N.check(lib.trl_moe_tc(x.data_ptr(), wt.data_ptr(), out.data_ptr(), out.stride(0), plan.items, plan.n_items, pairs, wt.shape[0],
                                   wt.shape[1], wt.shape[2], k, f, st), "moe_tc")
        N.count(3)
        return y, place, weight

    def join_experts(self, x, branch, post, nxt, eps, n):
        """:meth:`join` with the weighted sum over a token's experts as the branch."""
        y, place, weight = branch
        t, ld = x.shape
        h = self.ws.get(f"join_h_{self._join_dtype}", (t, ld), self._join_dtype)
        N.check(self.lib.trl_join_experts(x.data_ptr(), y.data_ptr(), int(y.dtype == torch.bfloat16), place.data_ptr(), weight.data_ptr(), weight.shape[1], post.data_ptr(),
                                          post.shape[0], N.ptr(nxt), 0 if nxt is None else nxt.shape[0], h.data_ptr(), t, ld, n, eps, _f32(h),
                                          N.stream()), "join_experts")
        N.count()
        return h
