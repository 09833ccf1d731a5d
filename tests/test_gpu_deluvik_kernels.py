"""The kernels of softmax attention on packed pages, the gated linear recurrence and the experts (csrc/attn_softmax.cu, lru.cu,
moe.cu, moe_tc.cu) against fp32 / fp64 torch, shape by shape: odd sizes, tile and page borders, splits, carried states."""
import math
from types import SimpleNamespace

import pytest
import torch

import deluvik_oracle as oracle
from tilerl_b200.deluvik_layout import AttnLayout, LayerLayout, LruLayout, MoeLayout, StateLayout, pad
from tilerl_b200.mixers import LruSpec, MoeSpec, RotarySpec, SoftmaxAttnSpec

pytestmark = pytest.mark.gpu


@pytest.fixture(scope="module")
def ops():
    from tilerl_b200.factory import make_ops
    return make_ops("cuda")


def _rel(a, b):
    a, b = a.double().cpu(), b.double().cpu()
    return float((a - b).abs().max() / b.abs().max().clamp_min(1e-30))


def _randn(*shape, seed=0, dtype=torch.float32):
    return torch.randn(*shape, device="cuda", generator=torch.Generator(device="cuda").manual_seed(seed)).to(dtype)


def _pool(specs, blocks, dtype):
    """A packed pool whose caches are those of ``specs``."""
    from tilerl_b200.config import DeluvikConfig
    from tilerl_b200.kv import PackedKvPool
    from tilerl_b200.mixers import LayerSpec
    cfg = DeluvikConfig(name="pool", hidden=16, vocab=16, layers=tuple(LayerSpec(s) for s in specs), logit_cap=1.0)
    pool = PackedKvPool(cfg, blocks, "cuda", dtype)
    pool.k.fill_(0xFF)                                       # not-a-number wherever nothing was written
    return pool


def _spec(heads, kv_heads, dim, vdim, window=None, cap=None, sink=False, conv=0, norm="all", half=True, dims=None, scale=0.2, tied=False):
    return SoftmaxAttnSpec(heads, kv_heads, dim, vdim, scale, RotarySpec(dims or dim // 2 * 2, 3000.0, None, half), norm, window, cap, sink, conv, tied)


def _batch(lens, starts, slots=None):
    """Sequences on interleaved pages out of order."""
    from tilerl_b200.batch import Batch
    order = torch.randperm(sum((n + s + 15) // 16 for n, s in zip(lens, starts)), generator=torch.Generator().manual_seed(3)).tolist()
    seqs = []
    for i, (n, s) in enumerate(zip(lens, starts)):
        k = (n + s + 15) // 16
        seqs.append(dict(tokens=[1] * n, start=s, blocks=[1 + order.pop() for _ in range(k)], slot=slots[i] if slots else i + 1))
    return Batch.build(seqs, "cuda"), sum(len(s["blocks"]) for s in seqs) + 1


# ---- softmax attention ----------------------------------------------------------------------------------------
SHAPES = [(1, 1, 16, 16), (6, 3, 40, 40), (7, 1, 64, 112), (3, 3, 20, 12), (20, 1, 128, 128), (4, 2, 256, 192), (8, 2, 128, 64), (5, 5, 72, 88)]


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 3e-6), (torch.bfloat16, 6e-3)])
@pytest.mark.parametrize("shape", SHAPES, ids=str)
@pytest.mark.parametrize("window,cap,sink", [(None, None, False), (37, None, True), (1, 3.0, False), (None, 4.0, True), (130, None, False)])
def test_attention_over_pages(ops, dtype, tol, shape, window, cap, sink):
    """Decoded tokens, a short portion and prompts in one batch, contexts from one token to hundreds, at page and tile borders."""
    from tilerl_b200.ops import ref
    s = _spec(*shape, window=window, cap=cap, sink=sink, scale=1.5 / shape[2] ** 0.5)
    al = AttnLayout(s)
    lens, starts = (1, 130, 3, 1, 65, 1, 1), (0, 37, 509, 640, 0, 127, 300)
    batch, blocks = _batch(lens, starts)
    pool = _pool([s], blocks, dtype)
    k, v, want, q_all = [], [], [], []
    factor = 0.8
    sk = _randn(s.heads, seed=9) + 1.0 if sink else None
    for i, (n, st) in enumerate(zip(lens, starts)):
        zero = lambda x, d: torch.nn.functional.pad(x.to(dtype), (0, pad(d) - d))
        q, kk, vv = (zero(_randn(r, h, d, seed=50 + 3 * i + j), d) for j, (r, h, d) in
                     enumerate(((n, s.heads, s.dim), (n + st, s.kv_heads, s.dim), (n + st, s.kv_heads, s.vdim))))
        where = torch.tensor([int(batch.block_table[i, p // 16]) * 16 + p % 16 for p in range(n + st)])
        ref.packed_kv_write(pool.layer(0), pool.pages[0], kk, vv, where, 0.0)
        full = torch.cat([torch.zeros(st, *q.shape[1:], dtype=dtype, device="cuda"), q])
        o = oracle.attend(full.double().cpu(), kk.double().cpu(), vv.double().cpu(), s.scale, window=window, cap=cap,
                          sink=None if sk is None else sk.double().cpu())[st:]
        want.append(factor * o.reshape(n, -1)), q_all.append(q.reshape(n, -1))
    q, want = torch.cat(q_all).contiguous(), torch.cat(want)
    for splits in (0, 4):
        ops.attn_splits = splits
        mid = torch.full((q.shape[0], al.n_out + 16), 7.0, dtype=dtype, device="cuda")
        ops.softmax_attention(q, mid, al, sk, factor, batch, pool, 0)
        ops.attn_splits = 0
        assert _rel(mid[:, :al.n_out], want) < tol and bool((mid[:, al.n_out:] == 7.0).all())


@pytest.mark.parametrize("n,start", [(1, 5000), (1, 2047), (2, 4095), (700, 2400)])
@pytest.mark.parametrize("window", [None, 1000])
def test_one_key_far_back(ops, n, start, window):
    """Long contexts over many splits: one score stands out, just inside the window, at split borders, at the start."""
    from tilerl_b200.ops import ref
    s = _spec(4, 2, 64, 64, window=window, sink=True, scale=1.0)
    al, dt = AttnLayout(s), torch.bfloat16
    batch, blocks = _batch((n,), (start,))
    pool = _pool([s], blocks, dt)
    total = n + start
    k, v, q = _randn(total, 2, 64, seed=1, dtype=dt) * 0.3, _randn(total, 2, 64, seed=2, dtype=dt), _randn(n, 4, 64, seed=3, dtype=dt) * 0.3
    sk = torch.zeros(4, device="cuda")
    where = torch.tensor([int(batch.block_table[0, p // 16]) * 16 + p % 16 for p in range(total)])
    for at in sorted({0, 17, total - 1000, total - 1001, total - 1002, total - 2, 1024, start - 1}):
        if at < 0 or at >= total:
            continue
        kk = k.clone()
        kk[at] = (q[-1].view(2, 2, 64)[:, 0].float() * 60.0 / q[-1].view(2, 2, 64)[:, 0].float().pow(2).sum(-1, keepdim=True)).to(dt)
        ref.packed_kv_write(pool.layer(0), pool.pages[0], kk, v, where, 0.0)
        lo = 0 if window is None else max(0, total - window)          # what the last query sees
        sc = torch.einsum("gxd,ngd->gxn", q[-1].float().view(2, 2, 64), kk[lo:].float()).reshape(4, -1)
        p = torch.softmax(torch.cat([sc, sk[:, None]], 1), 1)[:, :-1]
        want = torch.einsum("gxn,ngd->gxd", p.view(2, 2, -1), v[lo:].float()).reshape(-1)
        mid = torch.zeros(n, al.n_out, dtype=dt, device="cuda")
        ops.softmax_attention(q.reshape(n, -1).contiguous(), mid, al, sk, 1.0, batch, pool, 0)
        assert _rel(mid[-1], want) < 1e-2, at


PREPS = [_spec(3, 1, 20, 20, tied=True, sink=True, cap=9.0), _spec(6, 3, 56, 32, conv=4), _spec(5, 5, 24, 40, norm="head", half=False, dims=8, window=9),
         _spec(2, 1, 64, 16, conv=1, dims=32), _spec(16, 4, 128, 128, conv=3), _spec(4, 2, 40, 40, norm="head", half=True)]


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 2e-6), (torch.bfloat16, 6e-3)])
@pytest.mark.parametrize("s", PREPS, ids=lambda s: f"{s.norm}-{s.conv}-{s.heads}")
def test_preparation_in_portions(ops, dtype, tol, s):
    """Convolution over portion borders (prompts, two tokens, single ones), norm, rotation, pages."""
    from tilerl_b200.kv import RecurrentPool
    from tilerl_b200.ops import ref
    l = LayerLayout(AttnLayout(s), None)
    al, lens = l.attn, (90, 33)
    import tilerl_b200.kv as kv
    spool = RecurrentPool.__new__(RecurrentPool)
    real, kv.state_layouts = kv.state_layouts, lambda cfg: (StateLayout(0, 0, max(16, al.conv_c), al.taps),)
    try:
        spool.__init__(None, 4, "cuda", ring_dtype=dtype)
    finally:
        kv.state_layouts = real
    spool.ring.fill_(math.nan)
    zero = lambda x, h, d: torch.nn.functional.pad(x.view(-1, h, d), (0, pad(d) - d)).reshape(x.shape[0], -1)
    parts = [(s.heads, s.dim), (s.kv_heads, s.dim)] + ([] if s.tied else [(s.kv_heads, s.vdim)])
    w = {"q_norm": 1 + 0.3 * _randn(s.dim if s.norm == "head" else s.heads * s.dim, seed=1), "k_norm": 1 + 0.3 * _randn(s.dim if s.norm == "head" else s.kv_heads * s.dim, seed=2)}
    taps = [_randn(max(1, s.conv), h * d, seed=3 + i) for i, (h, d) in enumerate(parts)]
    served = {n: (torch.nn.functional.pad(t, (0, al.dk - s.dim)) if s.norm == "head" else zero(t[None], t.numel() // s.dim, s.dim)[0]).contiguous() for n, t in w.items()}
    served["conv"] = torch.cat([zero(t, h, d) for t, (h, d) in zip(taps, parts)], 1).contiguous() if s.conv else None
    freqs = torch.tensor(s.rot.frequencies(), dtype=torch.float64, device="cuda")
    raw = [[_randn(n, h * d, seed=20 + 5 * i + j).to(dtype) for j, (h, d) in enumerate(parts)] for i, n in enumerate(lens)]
    pos_of, got_q, want_q, kvs = [0, 0], [[], []], [], []
    blocks = [[3, 1, 7, 9, 2, 11], [5, 4, 6]]
    pool = _pool([s], 12, dtype)
    from tilerl_b200.batch import Batch
    for cut in ((40, 2), (1, 1), (2, 17), (1, 1), (46, 12)):
        seqs = [dict(tokens=[1] * c, start=pos_of[i], blocks=blocks[i], slot=2 - i) for i, c in enumerate(cut)]
        batch = Batch.build(seqs, "cuda")
        proj = torch.cat([torch.cat([zero(x[pos_of[i]:pos_of[i] + c], h, d) for x, (h, d) in zip(raw[i], parts)], 1) for i, c in enumerate(cut)]).contiguous()
        q, mid = ops.attn_prep(proj, l, served, freqs, batch, pool, 0, spool, 0, 1e-4)
        assert not mid[:, l.n_mid:].any()
        o = 0
        for i, c in enumerate(cut):
            got_q[i].append(q[o:o + c].clone())
            o, pos_of[i] = o + c, pos_of[i] + c
    for i, n in enumerate(lens):
        conv = [oracle.causal_conv(x.double().cpu(), t.double().cpu().T) if s.conv else x.double().cpu() for x, t in zip(raw[i], taps)]
        def normed(x, h, wt):
            x = x.view(n, h, s.dim)
            x = oracle.unit_rms(x, 1e-4) if s.norm == "head" else oracle.unit_rms(x.reshape(n, -1), 1e-4).view(n, h, s.dim)
            return oracle.rotate(x * (wt if s.norm == "head" else wt.view(h, s.dim)), s.rot.to_json(), s.rot.half)
        wq, wk = (w[k].double().cpu() for k in ("q_norm", "k_norm"))
        q = torch.cat(got_q[i]).view(n, s.heads, al.dk)
        assert _rel(q[:, :, :s.dim], normed(conv[0], s.heads, wq)) < tol and not q[:, :, s.dim:].any()
        k, v = ref.packed_kv_gather(pool.layer(0), pool.pages[0], dtype, torch.tensor(blocks[i], device="cuda"), n)
        assert _rel(k[:, :, :s.dim], normed(conv[1], s.kv_heads, wk)) < tol and not k[:, :, s.dim:].any()
        assert _rel(v[:, :, :s.vdim], (conv[1] if s.tied else conv[2]).view(n, s.kv_heads, s.vdim)) < tol and not v[:, :, s.vdim:].any()


# ---- gated linear recurrence -----------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype,tol", [(torch.float32, 1e-5), (torch.bfloat16, 2e-2)])
@pytest.mark.parametrize("spec", [LruSpec(48, 3, 4), LruSpec(60, 5, 2), LruSpec(512, 2, 4), LruSpec(40, 1, 1), LruSpec(640, 2, 6)], ids=lambda s: f"{s.width}-{s.blocks}-{s.conv}")
def test_recurrence_in_portions(ops, dtype, tol, spec):
    """Sequences of unequal length in portions and single tokens, on slots out of order; slow and fast channels."""
    from tilerl_b200.batch import Batch
    import tilerl_b200.kv as kv
    r = LruLayout(spec)
    attn = AttnLayout(_spec(1, 1, 16, 16))
    l = LayerLayout(attn, r, 1.0, 0.7)
    spool = kv.RecurrentPool.__new__(kv.RecurrentPool)
    real, kv.state_layouts = kv.state_layouts, lambda cfg: (StateLayout(0, r.width, r.width, spec.conv),)
    try:
        spool.__init__(None, 12, "cuda", ring_dtype=dtype)
    finally:
        kv.state_layouts = real
    spool.ring.fill_(math.nan)
    b, k = spec.blocks, spec.part
    spread = lambda x: torch.nn.functional.pad(x.reshape(*x.shape[:-1], b, k), (0, r.pp - k)).flatten(-2)
    full = {"y.b": _randn(spec.width, seed=1), "x.b": _randn(spec.width, seed=2), "conv": 0.6 * _randn(spec.width, spec.conv, seed=3), "conv.b": 0.3 * _randn(spec.width, seed=4),
            "lam": 3 * _randn(spec.width, seed=5) - 4, "ra": _randn(b, k, k, seed=6) * 2 / k ** 0.5, "ri": _randn(b, k, k, seed=7) * 2 / k ** 0.5,
            "ra.b": _randn(b, k, seed=8), "ri.b": _randn(b, k, seed=9)}
    full["ra"], full["ri"] = full["ra"].to(dtype).float(), full["ri"].to(dtype).float()
    w = {"y_b": spread(full["y.b"]), "x_b": spread(full["x.b"]), "lru_conv": spread(full["conv"].T).contiguous(), "lru_conv_b": spread(full["conv.b"]), "lam": spread(full["lam"])}
    w["gates"] = torch.zeros(b, 2 * r.pp, r.pp, dtype=dtype, device="cuda")
    w["gates_b"] = torch.zeros(b, 2 * r.pp, device="cuda")
    for j, n in enumerate(("ra", "ri")):
        w["gates"][:, j * r.pp:j * r.pp + k, :k] = full[n].to(dtype)
        w["gates_b"][:, j * r.pp:j * r.pp + k] = full[n + ".b"]
    lens = (200, 7, 150, 41, 9, 9, 9, 9, 9, 9)
    rows = [[_randn(n, spec.width, seed=30 + 2 * i + j).to(dtype) for j in range(2)] for i, n in enumerate(lens)]
    at, out = [0] * len(lens), [[] for _ in lens]
    cuts = [(130, 2, 1, 16, 2, 2, 2, 2, 2, 2), (1,) * 10, (2, 1, 100, 3, 1, 1, 1, 1, 1, 1), (1,) * 10, (66, 2, 47, 20, 4, 4, 4, 4, 4, 4)]
    for cut in cuts:
        batch = Batch.build([dict(tokens=[1] * c, start=at[i], blocks=[0] * 20, slot=10 - i) for i, c in enumerate(cut)], "cuda")
        proj = torch.cat([torch.cat([torch.full((c, attn.n_in), 9.0, device="cuda").to(dtype)] + [spread(x[at[i]:at[i] + c]) for x in rows[i]], 1) for i, c in enumerate(cut)])
        mid = torch.full((proj.shape[0], l.n_out), 5.0, dtype=dtype, device="cuda")
        ops.lru_mix(proj.contiguous(), mid, l, w, batch, spool, 0)
        assert bool((mid[:, :attn.n_out] == 5.0).all()) and bool((mid[:, l.n_mid:] == 5.0).all())
        o = 0
        for i, c in enumerate(cut):
            out[i].append(mid[o:o + c, attn.n_out:l.n_mid].clone())
            o, at[i] = o + c, at[i] + c
    d = {n: t.double().cpu() for n, t in full.items()}
    for i, n in enumerate(at):
        y, x = (t[:n].double().cpu() for t in rows[i])
        u = (oracle.causal_conv(x + d["x.b"], d["conv"]) + d["conv.b"]).to(dtype).double()
        s = oracle.scan_lru(u, oracle.block_gate(u, d["ra"], d["ra.b"]), oracle.block_gate(u, d["ri"], d["ri.b"]), d["lam"])
        want = 0.7 * s * oracle.gelu_tanh(y + d["y.b"])
        got = torch.cat(out[i]).view(n, b, r.pp)
        assert _rel(got[:, :, :k].reshape(n, -1), want) < tol and not got[:, :, k:].any(), i
        assert _rel(spool.states[10 - i, 0].view(b, r.pp)[:, :k].reshape(-1), s[-1]) < (1e-5 if dtype == torch.float32 else 2e-2)


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 2e-6), (torch.bfloat16, 6e-3)])
@pytest.mark.parametrize("taps,silu,biased", [(4, False, True), (3, True, False), (1, False, True), (6, False, False)])
def test_convolution_of_long_prompts(ops, dtype, tol, taps, silu, biased):
    """Sequences of unequal length whose borders fall anywhere, with and without earlier inputs."""
    from tilerl_b200.batch import Batch
    from tilerl_b200.ops import native as N
    ch, rows = 272, 16
    lens, starts = (333, 1, 2, 400, 17), (0, 5, 0, 2, 40)
    batch = Batch.build([dict(tokens=[1] * n, start=s, blocks=[0] * 40, slot=i) for i, (n, s) in enumerate(zip(lens, starts))], "cuda")
    t = sum(lens)
    w, b, pre = _randn(taps, ch, seed=1), _randn(ch, seed=2), _randn(ch, seed=3)
    proj, ring, out = torch.zeros(t, ch + 16, dtype=dtype, device="cuda"), torch.full((5, rows, ch), math.nan, dtype=dtype, device="cuda"), torch.zeros(t, ch, dtype=dtype, device="cuda")
    want, o = [], 0
    for i, (n, s) in enumerate(zip(lens, starts)):
        x = _randn(n + s, ch, seed=10 + i).to(dtype)
        proj[o:o + n, :ch], o = x[s:], o + n
        for p in range(max(0, s - rows), s):
            ring[i, p % rows] = x[p]
        x = x.double().cpu() + (pre.double().cpu() if biased else 0.0)
        y = (oracle.causal_conv(x, w.double().cpu().T) + b.double().cpu())[s:]
        want.append(oracle.silu(y) if silu else y)
    N.check(ops.lib.trl_scan_conv(proj.data_ptr(), proj.stride(0), w.data_ptr(), b.data_ptr(), pre.data_ptr() if biased else None, ring.data_ptr(), ring.stride(0),
                                  rows, ring.stride(1), batch.positions.data_ptr(), batch.seq_ids.data_ptr(), batch.q_start.data_ptr(),
                                  batch.state_slots.data_ptr(), out.data_ptr(), t, ch, taps, int(silu), int(dtype == torch.float32), N.stream()))
    assert _rel(out, torch.cat(want)) < tol


# ---- experts ----------------------------------------------------------------------------------------------------
MOES = [MoeSpec(24, 5, 2, 40), MoeSpec(64, 8, 8, 0), MoeSpec(192, 40, 6, 192), MoeSpec(100, 3, 1, 300), MoeSpec(256, 64, 4, 256)]


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 1e-5), (torch.bfloat16, 1.5e-2)])
@pytest.mark.parametrize("t", [1, 2, 9, 64, 65, 700])
@pytest.mark.parametrize("spec", MOES, ids=lambda s: f"{s.ff}-{s.experts}-{s.top}")
@pytest.mark.parametrize("hidden", [64, 448])
def test_experts(ops, dtype, tol, t, spec, hidden):
    m = MoeLayout(spec)
    h = _randn(t, hidden, seed=1, dtype=dtype)
    router, bias = torch.zeros(m.router_rows, hidden, device="cuda", dtype=dtype), torch.zeros(m.router_rows, device="cuda")
    router[:spec.experts], bias[:spec.experts] = _randn(spec.experts, hidden, seed=2).to(dtype), _randn(spec.experts, seed=3)
    gate_up, down = torch.zeros(m.n, 2 * m.ff, hidden, device="cuda", dtype=dtype), torch.zeros(m.n, hidden, m.ff, device="cuda", dtype=dtype)
    w = {"router": router[:spec.experts], "router.b": bias[:spec.experts]}
    for e in range(m.n):
        lo = (e - spec.experts) * m.ff
        ff = spec.ff if e < spec.experts else min(m.ff, spec.shared - lo)
        g, u, d = (_randn(*s, seed=10 + 3 * e + i) * 1.5 / s[1] ** 0.5 for i, s in enumerate(((ff, hidden), (ff, hidden), (hidden, ff))))
        gate_up[e, 0:2 * ff:2], gate_up[e, 1:2 * ff:2], down[e, :, :ff] = g.to(dtype), u.to(dtype), d.to(dtype)
        w[f"e{e}.gate"], w[f"e{e}.up"], w[f"e{e}.down"] = gate_up[e, 0:2 * ff:2], gate_up[e, 1:2 * ff:2], down[e, :, :ff]
    w = {n: x.double().cpu() for n, x in w.items()}
    x, post, nxt = _randn(t, hidden, seed=7), 1 + 0.2 * _randn(1, hidden, seed=8), 1 + 0.2 * _randn(1, hidden, seed=9)
    hd = h.double().cpu()
    want = oracle.experts(hd, w, "", {"router": {"experts": spec.experts, "top": spec.top}})
    for j in range(m.pieces):
        want += oracle.glu(hd, w, f"e{spec.experts + j}.", oracle.silu)
    want_x = x.double().cpu() + oracle.unit_rms(want, 1e-3) * post[0].double().cpu()
    ops._join_dtype = dtype
    branch = ops.experts(h, router, bias, gate_up, down, m)
    y, place, weight = branch
    got = (weight.double().cpu()[:, :, None] * y.double().cpu()[place.long().cpu().view(t, -1)]).sum(1)
    assert _rel(got, want) < tol
    hn = ops.join_experts(x, branch, post, nxt, 1e-3, hidden)
    assert _rel(x, want_x) < tol and _rel(hn, oracle.unit_rms(want_x, 1e-3) * nxt[0].double().cpu()) < tol


def test_experts_of_a_token_that_is_no_number(ops):
    """Such a row chooses different experts all the same and leaves the other rows alone."""
    m, dt = MoeLayout(MoeSpec(64, 6, 3, 64)), torch.bfloat16
    for t in (3, 80):
        h = _randn(t, 64, seed=1, dtype=dt)
        router, bias = _randn(m.router_rows, 64, seed=2, dtype=dt), _randn(m.router_rows, seed=3)
        gate_up, down = _randn(m.n, 2 * m.ff, 64, seed=4, dtype=dt) * 0.1, _randn(m.n, 64, m.ff, seed=5, dtype=dt) * 0.1
        sums = []
        for bad in (False, True):
            if bad:
                h[1] = math.nan
            y, place, weight = ops.experts(h, router, bias, gate_up, down, m)
            assert sorted(place.tolist()) == list(range(t * m.slots))
            sums.append((weight[:, :, None] * y[place.long().view(t, -1)]).sum(1).clone())
        keep = [i for i in range(t) if i != 1]
        assert _rel(sums[1][keep], sums[0][keep]) < 1e-5


# ---- epilogues --------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype,tol", [(torch.float32, 1e-5), (torch.bfloat16, 1.5e-2)])
@pytest.mark.parametrize("t", [1, 8, 9, 100])
@pytest.mark.parametrize("act", ["gelu", "silu"])
def test_glu_and_capped_logits(ops, dtype, tol, t, act):
    h, w = _randn(t, 192, seed=1, dtype=dtype), (_randn(256, 192, seed=2) * 2 / 192 ** 0.5).to(dtype)
    z = h.double() @ w.double().t()
    f = (lambda g: oracle.gelu_tanh(g)) if act == "gelu" else oracle.silu
    assert _rel(ops.glu(h, w, act), f(z[:, 0::2]) * z[:, 1::2]) < tol
    assert _rel(ops.project_logits(h, w, 3.0), oracle.soft_cap(z, 3.0)) < 2e-5
    assert _rel(ops.project(h, w), z) < (1e-5 if dtype == torch.float32 else 6e-3)
