"""fp32 torch form of the stream designs' mechanisms (latent and softmax attention, decayed scans, delta rule, linear recurrence,
experts, norms, gates) and, on top of them, the op surface :class:`RefMixers` that ``models/fetotar.py``, ``models/deluvik.py`` and
``models/tobadra.py`` call; mixed into :class:`~tilerl_b200.ops.backend.RefOps`.  The CUDA twins are
:mod:`tilerl_b200.ops.cuda_mixers`, :mod:`tilerl_b200.ops.cuda_blocks` and :mod:`tilerl_b200.ops.cuda_gated`.  No counterpart in
the reference.
"""
from __future__ import annotations

import math

import torch
import torch.nn.functional as F

from . import ref
from .ref import KV_BLOCK


# ---- element-wise and norms --------------------------------------------------------------------------
def stream_norm(x, norm, eps: float, n: int):
    """``norm``: ``[2, width]`` weight and bias of a layer norm, ``[1, width]`` weight of an RMS norm, None for the row
    itself.  The first ``n`` columns count; columns past them come out as zeros (weights and biases are zero there)."""
    if norm is None:
        return x
    if norm.shape[0] == 1:
        return x * ref.rms_factor(x, n, eps)[:, None] * norm[0]
    mean = x[:, :n].sum(-1, keepdim=True) / n
    var = (x[:, :n] - mean).pow(2).sum(-1, keepdim=True) / n
    return (x - mean) * torch.rsqrt(var + eps) * norm[0] + norm[1]


def clamped_glu(gate_up, limit: float):
    """Rows ``2j`` = gate, ``2j + 1`` = up: ``g sigmoid(1.702 g) (u + 1)`` with ``g`` bounded above, ``u`` on both sides."""
    g, u = gate_up[..., 0::2].clamp(max=limit), gate_up[..., 1::2].clamp(-limit, limit)
    return g * torch.sigmoid(1.702 * g) * (u + 1.0)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z.pow(3))))


# ---- latent attention ----------------------------------------------------------------------------------
def rotate_pairs(x, positions, freqs, amplitude: float):
    """Turn the leading ``2 len(freqs)`` columns of ``x [T, ..., width]`` in neighbouring pairs."""
    ang = positions.to(torch.float64)[:, None] * freqs.to(positions.device)[None, :]
    shape = [x.shape[0]] + [1] * (x.dim() - 2) + [freqs.numel()]
    c, s = (ang.cos() * amplitude).float().view(shape), (ang.sin() * amplitude).float().view(shape)
    k = 2 * freqs.numel()
    u, v = x[..., 0:k:2], x[..., 1:k:2]
    out = x.clone()
    out[..., 0:k:2], out[..., 1:k:2] = u * c - v * s, v * c + u * s
    return out


def rotate_halves(x, positions, freqs):
    """Turn column i of ``x [T, ..., width]`` with column ``i + len(freqs)``; columns past ``2 len(freqs)`` stay."""
    n = freqs.numel()
    ang = positions.to(torch.float64)[:, None] * freqs.to(positions.device)[None, :]
    shape = [x.shape[0]] + [1] * (x.dim() - 2) + [n]
    c, s = ang.cos().float().view(shape), ang.sin().float().view(shape)
    u, v = x[..., :n], x[..., n:2 * n]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * n:]], -1)


def latent_write(cache, page, rows, slot_mapping):
    """Cached rows ``[T, width]`` into ``cache [blocks, 1, page bytes]``."""
    el, idx = cache.view(rows.dtype), page.index().to(rows.device)
    for t in range(rows.shape[0]):
        s = int(slot_mapping[t])
        if s >= 0:
            el[s // KV_BLOCK, 0, idx[s % KV_BLOCK]] = rows[t]


def latent_gather(cache, page, dtype, block_row, lo: int, hi: int):
    """Cached rows of positions ``lo .. hi - 1`` of one sequence, fp32."""
    first = lo // KV_BLOCK
    pages = cache[block_row[first:(hi + KV_BLOCK - 1) // KV_BLOCK].long()]
    rows = pages.view(dtype)[:, 0, page.index().to(cache.device)].float().reshape(-1, page.width)
    return rows[lo - first * KV_BLOCK:hi - first * KV_BLOCK]


def latent_attention(q, rows, kv: int, scale: float):
    """One query token over the rows it sees: ``q [heads, kv + rd]`` (the unrotated part already mapped into the latent),
    ``rows [n, kv + rd]``; softmax-weighted sum of the latents ``[heads, kv]``."""
    return torch.softmax(q @ rows.t() * scale, dim=-1) @ rows[:, :kv]


# ---- softmax attention over packed pages ----------------------------------------------------------------
def soft_cap(z, cap: float):
    return cap * torch.tanh(z / cap)


def softmax_attention(q, k, v, scale: float, cap=None, sink=None):
    """One query token over the keys it sees: ``q [heads, dk]``, ``k [n, kv_heads, dk]``, ``v [n, kv_heads, dv]``; ``sink
    [heads]`` counts in the denominator only."""
    hq, hkv = q.shape[0], k.shape[1]
    s = torch.einsum("hgd,nhd->hgn", q.view(hkv, hq // hkv, -1), k) * scale
    s = s if cap is None else soft_cap(s, cap)
    if sink is not None:
        s = torch.cat([s, sink.float().view(hkv, -1, 1)], -1)
    p = torch.softmax(s, dim=-1)[..., :k.shape[0]]
    return torch.einsum("hgn,nhd->hgd", p, v).reshape(hq, -1)


def weighted_norm(x, heads: int, d: int, weight, whole: bool, eps: float):
    """RMS norm of ``x [T, heads, dp]`` (``d`` true columns per head), over all heads at once or per head, times ``weight``."""
    n = heads * d if whole else d
    ss = x.pow(2).sum((-2, -1), keepdim=True) if whole else x.pow(2).sum(-1, keepdim=True)
    return x * torch.rsqrt(ss / n + eps) * (weight.view(heads, -1) if whole else weight)


# ---- linear recurrence, experts ---------------------------------------------------------------------------
def lru_step(state, u, r, i, lam):
    """``state, u [width]``, gate pre-activations ``r, i`` -> new state."""
    log_a = -8.0 * torch.sigmoid(r) * F.softplus(lam)
    return torch.exp(log_a) * state + torch.sqrt(-torch.expm1(2.0 * log_a)) * torch.sigmoid(i) * u


def activate(z, act: str):
    """"gelu" (its tanh form), "gelu_erf" or "silu"."""
    return gelu_tanh(z) if act == "gelu" else F.gelu(z) if act == "gelu_erf" else F.silu(z)


def choose(logits, top: int):
    """(experts ``[T, top]``, their weights): the largest logits (the first of equal ones), softmax over those."""
    best, idx = torch.sort(logits, dim=1, descending=True, stable=True)
    return idx[:, :top], torch.softmax(best[:, :top], dim=1)


def choose_grouped(z, correction, top: int, r):
    """(outputs ``[T, top]``, their weights): scores are the softmax over all outputs; the largest score plus correction among the
    outputs of the ``r.keep`` groups whose largest is largest."""
    s = torch.softmax(z, dim=1)
    c = s + correction
    t, n = c.shape
    best = c.view(t, r.groups, -1).amax(2)
    order = torch.sort(best, dim=1, descending=True, stable=True).indices[:, :r.keep]
    kept = torch.zeros_like(best, dtype=torch.bool).scatter_(1, order, True).repeat_interleave(n // r.groups, dim=1)
    idx = torch.sort(c.masked_fill(~kept, -math.inf), dim=1, descending=True, stable=True).indices[:, :top]
    return idx, s.gather(1, idx) * r.scale


# ---- decayed scans ---------------------------------------------------------------------------------------
def conv_rows(rows, taps, bias):
    """``rows [k, C]`` (oldest first), ``taps [k, C]`` -> silu of the depthwise convolution's newest output."""
    return F.silu((rows * taps).sum(0) + bias)


def mamba2_step(state, x, b, c, dt, a_log, skip):
    """``state [H, N, V]``; ``x [H, V]``, ``b, c [H, N]`` (groups expanded), ``dt [H]``."""
    s = torch.exp(-torch.exp(a_log) * dt)[:, None, None] * state + (dt[:, None] * b)[:, :, None] * x[:, None, :]
    return s, torch.einsum("hnv,hn->hv", s, c) + skip[:, None] * x


def mlstm_gates(raw, bias, cap: float):
    """Raw gates ``[..., 2H]`` -> (log input gate, log forget gate)."""
    z = cap * torch.tanh((raw + bias) / cap)
    h = raw.shape[-1] // 2
    return z[..., :h], F.logsigmoid(z[..., h:])


def mlstm_step(state, n, m, q, k, v, i, f):
    """``state [H, D, V]``, ``n [H, D]``, ``m [H]``."""
    new = torch.maximum(f + m, i)
    keep, add = torch.exp(f + m - new), torch.exp(i - new)
    s = keep[:, None, None] * state + (add[:, None] * k)[:, :, None] * v[:, None, :]
    n = keep[:, None] * n + add[:, None] * k
    den = torch.maximum((n * q).sum(-1).abs(), torch.exp(-new)) + 1e-6
    return s, n, new, torch.einsum("hdv,hd->hv", s, q) / den[:, None]


def unit_heads(x):
    """Vectors of length one along the last dimension."""
    return x * torch.rsqrt(x.pow(2).sum(-1, keepdim=True) + 1e-6)


def delta_step(state, q, k, v, log_keep, beta):
    """``state [H, D, V]``; ``q, k, log_keep [H, D]``, ``v [H, V]``, ``beta [H]``: fade every row, write what of the value is not there
    yet, read."""
    s = torch.exp(log_keep)[:, :, None] * state
    u = beta[:, None] * (v - torch.einsum("hdv,hd->hv", s, k))
    s = s + k[:, :, None] * u[:, None, :]
    return s, torch.einsum("hdv,hd->hv", s, q)


def grouped_rms(y, heads: int, vdim: int, dv: int, groups: int, eps: float):
    """RMS norm without a weight over ``groups`` equal parts of the true columns of ``y [T, heads * dv]``."""
    t = y.shape[0]
    v = y.view(t, heads, dv)[:, :, :vdim].reshape(t, groups, -1)
    out = torch.zeros_like(y)
    out.view(t, heads, dv)[:, :, :vdim] = (v * torch.rsqrt(v.pow(2).mean(-1, keepdim=True) + eps)).view(t, heads, vdim)
    return out


class RefMixers:
    """Ops of an fp32 stream with sandwich norms, and its mixers (mixed into RefOps: ``act_dtype``)."""

    # ---- stream ----------------------------------------------------------------------
    def embed_stream(self, table, ids, scale, norm, eps, n):
        """(stream, first normed row): the scaled embedding."""
        x = ref.embedding(table, ids) * scale
        return x, stream_norm(x, norm, eps, n).to(self.act_dtype)

    def join(self, x, y, post, nxt, eps, n):
        """``x += norm_post(y)``; the next projection's input ``norm_nxt(x)``."""
        x += stream_norm(y, post, eps, n)
        return stream_norm(x, nxt, eps, n).to(self.act_dtype)

    def project_gates(self, h, w, n_in):
        """(fused projection rows, fp32 gate rows)."""
        return ref.linear(h, w[:n_in]).to(self.act_dtype), ref.linear(h, w[n_in:])

    def project_f32(self, a, w, name="branch"):
        return ref.linear(a, w)

    def project_logits(self, h, w, cap=0.0):
        z = ref.linear(h, w)
        return soft_cap(z, cap) if cap else z

    def project(self, h, w):
        return ref.linear(h, w).to(self.act_dtype)

    def glu(self, h, w, act):
        """Rows ``2j`` = gate, ``2j + 1`` = up of ``w``: ``act(gate) * up``."""
        gu = ref.linear(h, w)
        return (activate(gu[:, 0::2], act) * gu[:, 1::2]).to(self.act_dtype)

    def clamped_glu(self, h, w, limit):
        return clamped_glu(ref.linear(h, w), limit).to(self.act_dtype)

    def side_input(self, h, w, table, ids, layer, dim):
        """``gelu(W h) * side[token, layer]``, zero past ``dim``."""
        z = ref.linear(h, w)
        stride = (dim + 7) // 8 * 8
        e = torch.zeros_like(z)
        e[:, :dim] = table[ids.long()][:, layer * stride:layer * stride + dim].float()
        return (gelu_tanh(z) * e).to(self.act_dtype)

    # ---- latent attention ----------------------------------------------------------------
    def latent_prep(self, proj, l, q_norm, kv_norm, uq, freqs, rot, batch, pool, idx, eps):
        """Normed latents and the rotated shared key into the cache; returns the query heads ``[T, heads, dk + rd]``, not
        turned yet."""
        t = proj.shape[0]
        cq = proj[:, :l.c0].float()
        cq = (cq * ref.rms_factor(cq, l.q_rank, eps)[:, None] * q_norm).to(self.act_dtype)
        c = proj[:, l.c0:l.kr0].float()
        c = c * ref.rms_factor(c, l.kv_rank, eps)[:, None] * kv_norm
        kr = rotate_pairs(proj[:, l.kr0:l.g0].float(), batch.positions, freqs, rot.amplitude)
        latent_write(pool.layer(idx), pool.pages[idx], torch.cat([c, kr], 1).to(pool.dtype), batch.slot_mapping)
        return ref.linear(cq, uq).view(t, l.heads, l.dq).to(self.act_dtype)

    def latent_attention(self, q, proj, up, ukt, l, freqs, rot, batch, pool, idx):
        """Gated attention output, padded to the output projection's columns."""
        t = proj.shape[0]
        uk, uv = up.float().split([l.heads * l.dk, l.heads * l.dv])
        uk, uv = uk.view(l.heads, l.dk, l.kv), uv.view(l.heads, l.dv, l.kv)
        qr = rotate_pairs(q[:, :, l.dk:].float(), batch.positions, freqs, rot.amplitude)
        ql = torch.cat([torch.einsum("thd,hdc->thc", q[:, :, :l.dk].float(), uk), qr], -1)
        out = torch.zeros(t, l.n_out, dtype=self.act_dtype, device=proj.device)
        for i in range(t):
            p = int(batch.positions[i])
            rows = latent_gather(pool.layer(idx), pool.pages[idx], pool.dtype, batch.block_table[int(batch.seq_ids[i])],
                                 max(0, p + 1 - l.window), p + 1)
            o = torch.einsum("hc,hdc->hd", latent_attention(ql[i], rows, l.kv, l.scale), uv).reshape(-1)
            out[i, :l.heads * l.dv] = (o * torch.sigmoid(proj[i, l.g0:l.n_in].float())).to(self.act_dtype)
        return out

    # ---- softmax attention ---------------------------------------------------------------
    def _conv_inputs(self, row, ring, pos: int, taps: int):
        """The last ``taps`` inputs (oldest first) of one sequence's convolution, ``row`` included; it goes into the ring."""
        ring[pos % ring.shape[0]] = row.to(ring.dtype)
        zero = torch.zeros_like(row, dtype=torch.float32)
        return torch.stack([ring[(pos - j) % ring.shape[0]].float() if pos >= j else zero for j in range(taps - 1, -1, -1)])

    def attn_prep(self, proj, l, w, freqs, batch, pool, idx, spool, sidx, eps):
        """Convolved, normed and turned queries ``[T, heads, dk]``; keys and values of layers that have their own into the
        cache.  Also the (zeroed) input of the layer's output projection."""
        a, s, t = l.attn, l.attn.spec, proj.shape[0]
        rows = proj[:, :a.n_in].float()
        if s.conv:
            rows = torch.stack([(self._conv_inputs(proj[i, :a.n_in], spool.ring_view(sidx, int(batch.state_slots[int(batch.seq_ids[i])])),
                                                   int(batch.positions[i]), s.conv) * w["conv"]).sum(0) for i in range(t)])
        turn = rotate_halves if s.rot.half else lambda x, p, f: rotate_pairs(x, p, f, 1.0)
        q = weighted_norm(rows[:, :a.k0].view(t, s.heads, a.dk), s.heads, s.dim, w["q_norm"], s.norm == "all", eps)
        if a.own:
            k = rows[:, a.k0:a.k0 + s.kv_heads * a.dk].view(t, s.kv_heads, a.dk)
            v = rows[:, a.v0:a.v0 + s.kv_heads * a.dv].view(t, s.kv_heads, a.dv)
            k = turn(weighted_norm(k, s.kv_heads, s.dim, w["k_norm"], s.norm == "all", eps), batch.positions, freqs)
            ref.packed_kv_write(pool.layer(idx), pool.pages[idx], k.to(pool.dtype), v.to(pool.dtype), batch.slot_mapping, eps)
        return turn(q, batch.positions, freqs).to(self.act_dtype), torch.zeros(t, l.n_out, dtype=self.act_dtype, device=proj.device)

    def softmax_attention(self, q, mid, a, sink, factor, batch, pool, idx, turn=None):
        """Attention output of every token, times ``factor``, into the first columns of ``mid``; with ``turn`` (cos and sin per token
        and pair ``[T, dv / 2, 2]``) turned back first."""
        s = a.spec
        for i in range(q.shape[0]):
            p = int(batch.positions[i])
            k, v = ref.packed_kv_gather(pool.layer(idx), pool.pages[idx], pool.dtype, batch.block_table[int(batch.seq_ids[i])], p + 1)
            lo = 0 if s.window is None else max(0, p + 1 - s.window)
            o = softmax_attention(q[i].float(), k[lo:], v[lo:], s.scale, s.cap, sink)
            if turn is not None:
                (x, y), (c, sn) = o.chunk(2, dim=1), turn[i].unbind(1)
                o = torch.cat([x * c + y * sn, y * c - x * sn], 1)
            mid[i, :a.n_out] = (o * factor).reshape(-1).to(self.act_dtype)

    # ---- gated linear recurrence -----------------------------------------------------------
    def lru_mix(self, proj, mid, l, w, batch, spool, sidx):
        """Recurrence x gelu branch, times the layer's factor, into the columns of ``mid`` behind the attention's."""
        r, t, y0 = l.lru, proj.shape[0], l.attn.n_in
        y = gelu_tanh(proj[:, y0:y0 + r.width].float() + w["y_b"])
        for q in range(batch.n_seqs):
            s0, n, slot = int(batch.q_start[q]), int(batch.q_len[q]), int(batch.state_slots[q])
            if n == 0:
                continue
            keep = bool(batch.keep_steps) and batch.keep_rows[q]
            live = spool.view(sidx, slot, int(spool.cur[slot]))[0]
            state = live.clone()
            for i in range(s0, s0 + n):
                pos = int(batch.positions[i])
                rows = self._conv_inputs(proj[i, y0 + r.width:y0 + 2 * r.width], spool.ring_view(sidx, slot), pos, r.spec.conv)
                rows[max(0, r.spec.conv - 1 - pos):] += w["x_b"]         # zeros before the start carry no bias
                u = ((rows * w["lru_conv"]).sum(0) + w["lru_conv_b"]).to(self.act_dtype).float()
                z = torch.einsum("bk,bjk->bj", u.view(r.spec.blocks, r.pp), w["gates"].float()) + w["gates_b"]
                state = lru_step(state, u, z[:, :r.pp].reshape(-1), z[:, r.pp:].reshape(-1), w["lam"])
                mid[i, l.attn.n_out:l.n_mid] = (state * y[i] * l.lru_scale).to(self.act_dtype)
                if keep:
                    spool.view(sidx, slot, i - s0)[0].copy_(state)
            if not keep:
                live.copy_(state)

    # ---- experts -----------------------------------------------------------------------------
    def experts(self, h, router, router_b, gate_up, down, m):
        """Weighted sum of the experts' outputs (the CUDA backend leaves the sum to :meth:`join_experts`)."""
        z = (ref.linear(h, router) + router_b)[:, :m.spec.experts]
        idx, weight = choose(z, m.spec.top)
        y = torch.zeros(h.shape[0], down.shape[1], dtype=torch.float32, device=h.device)
        for e in range(m.n):
            if e < m.spec.experts:
                rows, place = torch.nonzero(idx == e, as_tuple=True)
                scale = weight[rows, place][:, None]
            else:
                rows, scale = torch.arange(h.shape[0], device=h.device), 1.0
            if len(rows):
                y[rows] += scale * ref.linear(self.glu(h[rows], gate_up[e], m.spec.act), down[e])
        return y

    def join_experts(self, x, y, post, nxt, eps, n):
        return self.join(x, y, post, nxt, eps, n)

    # ---- gated branches with a convolution on the next input ----------------------------------
    def _input_conv(self, h, conv):
        """``h`` plus its causal convolution, or None without one (``conv``: taps, batch, state pool, index of the inputs kept)."""
        if conv is None:
            return None
        w, batch, spool, idx = conv
        out = torch.empty_like(h)
        for i in range(h.shape[0]):
            ring = spool.ring_view(idx, int(batch.state_slots[int(batch.seq_ids[i])]))
            out[i] = h[i] + (self._conv_inputs(h[i], ring, int(batch.positions[i]), w.shape[0]) * w).sum(0)
        return out.to(self.act_dtype)

    def embed_normed(self, table, vocab, ids, post, nxt, eps, n, conv):
        """(stream, its normed row, that row convolved): the normed embedding."""
        x = stream_norm(ref.embedding(table[:vocab], ids), post, eps, n)
        h = stream_norm(x, nxt, eps, n).to(self.act_dtype)
        return x, h, self._input_conv(h, conv)

    def gated_join(self, x, y, bias, z, z_b, post, nxt, eps, n, conv):
        """``x += norm_post((y + bias) sigmoid(z + z_b))``; returns (``norm_nxt(x)``, that row convolved)."""
        y = (y if bias is None else y + bias) * torch.sigmoid(z + z_b)
        h = self.join(x, y, post, nxt, eps, n)
        return h, self._input_conv(h, conv)

    def project_in(self, h, hc, w, n_in, n_gates, n_act=0, act="silu"):
        """(rows of the mixer, the first ``n_act`` through ``act``; fp32 rows of its gates; fp32 rows of its branch's gate): the last
        rows of ``w`` read ``h``, the others ``hc``."""
        n = n_in + n_gates
        proj = ref.linear(hc, w[:n_in])
        proj[:, :n_act] = activate(proj[:, :n_act], act)
        return proj.to(self.act_dtype), ref.linear(hc, w[n_in:n]), ref.linear(h, w[n:])

    def up_act(self, h, w, n, act):
        """(``act`` of the first ``n`` rows, the other rows in fp32)."""
        return activate(ref.linear(h, w[:n]), act).to(self.act_dtype), ref.linear(h, w[n:])

    def turned_prep(self, proj, l, bias, freqs, vfreqs, batch, pool, idx):
        """Biased and turned queries ``[T, heads, dk]``; turned keys and values into the cache; the input of the output projection;
        cos and sin of the values' turns."""
        a, s, t = l.attn, l.attn.spec, proj.shape[0]
        rows = proj.float() + bias
        q, k, v = (rows[:, c:c + h * d].reshape(t, h, d) for c, h, d in ((0, s.heads, a.dk), (a.k0, s.kv_heads, a.dk), (a.v0, s.kv_heads, a.dv)))
        q, k, v = (rotate_halves(x, batch.positions, f) for x, f in ((q, freqs), (k, freqs), (v, vfreqs)))
        ref.packed_kv_write(pool.layer(idx), pool.pages[idx], k.to(pool.dtype), v.to(pool.dtype), batch.slot_mapping, 0.0)
        ang = batch.positions.to(torch.float64)[:, None] * vfreqs.to(proj.device)[None, :]
        turn = torch.stack([ang.cos(), ang.sin()], -1).float()
        return q.to(self.act_dtype), torch.zeros(t, l.n_out, dtype=self.act_dtype, device=proj.device), turn

    def _scan_tokens(self, l, batch, spool, sidx, step):
        """``step(token, state, ring) -> (state, row)`` along every sequence; states move on in ``spool``."""
        y = torch.zeros(batch.n_tokens, l.heads * l.dv, dtype=torch.float32, device=batch.positions.device)
        for r in range(batch.n_seqs):
            s0, n, slot = int(batch.q_start[r]), int(batch.q_len[r]), int(batch.state_slots[r])
            if n == 0:
                continue
            keep = bool(batch.keep_steps) and batch.keep_rows[r]
            live = spool.view(sidx, slot, int(spool.cur[slot]))[0]
            state, ring = live.clone(), spool.ring_view(sidx, slot)
            for j in range(n):
                state, o = step(s0 + j, state, ring)
                y[s0 + j] = o.reshape(-1)
                if keep:
                    spool.view(sidx, slot, j)[0].copy_(state)
            if not keep:
                live.copy_(state)
        return y

    def _gated_heads(self, y, z, norm, l, eps):
        out = torch.zeros(y.shape[0], l.n_out, dtype=self.act_dtype, device=y.device)
        out[:, :l.heads * l.dv] = (grouped_rms(y, l.heads, l.vdim, l.dv, l.norm_groups, eps) * norm * torch.sigmoid(z.float())).to(self.act_dtype)
        return out

    def lightning_mix(self, proj, log_decay, norm, l, batch, spool, sidx, eps):
        keep = torch.exp(log_decay)[:, None, None]

        def step(t, s, ring):
            q, k, v = (proj[t, c:c + l.heads * d].float().view(l.heads, d) for c, d in ((0, l.dk), (l.k0, l.dk), (l.v0, l.dv)))
            s = keep * s + k[:, :, None] * v[:, None, :]
            return s, torch.einsum("hdv,hd->hv", s, q)
        return self._gated_heads(self._scan_tokens(l, batch, spool, sidx, step), proj[:, l.g0:], norm, l, eps)

    def delta_mix(self, proj, gates, w, norm, l, batch, spool, sidx, eps):
        a = ref.linear(proj[:, l.a0:l.g0], w["low"][l.n_low:]) + w["dt_bias"]
        log_keep = -torch.exp(w["a_log"])[None, :, None] * F.softplus(a).view(-1, l.heads, l.dk)
        beta = torch.sigmoid(gates[:, :l.heads].float())
        z = ref.linear(proj[:, l.g0:l.n_in], w["low"][:l.n_low])
        zero = torch.zeros(l.conv_c, device=proj.device)

        def step(t, s, ring):
            c = conv_rows(self._conv_inputs(proj[t, :l.conv_c], ring, int(batch.positions[t]), l.taps), w["conv"], zero).to(self.act_dtype).float()
            q, k = (unit_heads(c[o:o + l.k0].view(l.kv_heads, l.dk)).repeat_interleave(l.per, 0) for o in (0, l.k0))
            return delta_step(s, q * l.spec.dim ** -0.5, k, c[l.v0:].view(l.heads, l.dv), log_keep[t], beta[t])
        return self._gated_heads(self._scan_tokens(l, batch, spool, sidx, step), z, norm, l, eps)

    def routed_experts(self, h, z, correction, up, down, m):
        """Weighted sum of the chosen experts' outputs, the shared one and the input's own share; ``z``: rows of the fused router."""
        s = m.spec
        idx, weight = choose_grouped(z[:, :s.outputs], correction[:s.outputs], s.top, s.router)
        y = torch.zeros(h.shape[0], down.shape[1], dtype=torch.float32, device=h.device)
        for e in range(s.outputs + m.pieces):
            if e < s.outputs:
                rows, place = torch.nonzero(idx == e, as_tuple=True)
                scale = weight[rows, place][:, None]
            else:
                rows = torch.arange(h.shape[0], device=h.device)
                scale = torch.sigmoid(z[:, s.outputs])[:, None] if s.shared_gate else 1.0
            if not len(rows):
                continue
            if s.experts <= e < s.outputs:
                y[rows] += scale * h[rows].float()
                continue
            j = e if e < s.experts else e - s.outputs + s.experts
            y[rows] += scale * ref.linear(activate(ref.linear(h[rows], up[j]), s.act).to(self.act_dtype), down[j])
        return y

    def gated_join_experts(self, x, y, h, z, z_b, post, nxt, eps, n, conv):
        return self.gated_join(x, y, None, z, z_b, post, nxt, eps, n, conv)

    # ---- recurrent mixers ------------------------------------------------------------------
    def recurrent_mix(self, proj, gates, w, l, batch, pool, idx, eps):
        """Normed and gated output of a decayed scan; state and convolution inputs move on in ``pool``."""
        t, dev = proj.shape[0], proj.device
        y = torch.zeros(t, l.heads * l.dv, dtype=torch.float32, device=dev)
        gate = proj[:, l.g0:l.n_in].float()
        for r in range(batch.n_seqs):
            s0, n = int(batch.q_start[r]), int(batch.q_len[r])
            if n == 0:
                continue
            slot = int(batch.state_slots[r])
            keep = bool(batch.keep_steps) and batch.keep_rows[r]
            state = pool.view(idx, slot, int(pool.cur[slot]))
            parts = [a.clone() for a in state]
            ring = pool.ring_view(idx, slot)
            for j in range(n):
                tt = s0 + j
                if l.kind == "mamba2":
                    parts, y[tt] = self._mamba2_token(proj[tt], gates[tt], w, l, parts, ring, int(batch.positions[tt]))
                else:
                    parts, y[tt] = self._mlstm_token(proj[tt], gates[tt], w, l, parts)
                if keep:
                    for a, b in zip(pool.view(idx, slot, j), parts):
                        a.copy_(b)
            if not keep:
                for a, b in zip(state, parts):
                    a.copy_(b)
        if l.kind == "mamba2":
            y = y * F.silu(gate)
        y = grouped_rms(y, l.heads, l.vdim, l.dv, l.norm_groups, eps) * w["norm"]
        if l.kind == "mlstm":
            y = y * torch.sigmoid(gate)
        out = torch.zeros(t, l.n_out, dtype=self.act_dtype, device=dev)
        out[:, :l.heads * l.dv] = y.to(self.act_dtype)
        return out

    def _mamba2_token(self, row, gates, w, l, parts, ring, pos):
        rows = ring.shape[0]
        ring[pos % rows] = row[:l.conv_c].to(ring.dtype)
        taken = [ring[(pos - j) % rows].float() if pos >= j else torch.zeros(l.conv_c) for j in range(l.taps - 1, -1, -1)]
        c = conv_rows(torch.stack(taken), w["conv"], w["conv_b"]).to(self.act_dtype).float()
        per = l.heads // l.groups
        x = c[:l.k0].view(l.heads, l.dv)
        b, cc = (a.view(l.groups, l.dk).repeat_interleave(per, 0) for a in (c[l.k0:l.q0], c[l.q0:]))
        s, y = mamba2_step(parts[0], x, b, cc, F.softplus(gates[:l.heads].float() + w["gate_b"]), w["a_log"], w["skip"])
        return [s], y.reshape(-1)

    def _mlstm_token(self, row, gates, w, l, parts):
        row = row.float()
        q = row[:l.k0].view(l.heads, l.dk) * l.dim ** -0.5
        k, v = row[l.k0:l.v0].view(l.heads, l.dk), row[l.v0:l.g0].view(l.heads, l.dv)
        i, f = mlstm_gates(gates[:2 * l.heads].float(), w["gate_b"], l.cap)
        s, n, m, o = mlstm_step(parts[0], parts[1][:, 0], parts[2][:, 0], q, k, v, i, f)
        return [s, n[:, None].expand_as(parts[1]), m[:, None].expand_as(parts[2])], o.reshape(-1)
