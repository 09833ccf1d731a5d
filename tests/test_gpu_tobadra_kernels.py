"""The kernels of gated joins, dual-input projections, attention over turned values, fixed-decay and delta scans and grouped routing
(csrc/join.cu, linear_rows.cu, attn_softmax.cu, scan.cu, scan_mma.cu, delta.cu, delta_mma.cu, moe.cu) against fp64 torch, shape by
shape: odd sizes, tile, chunk and page borders, splits, carried states."""
import math

import pytest
import torch

import tobadra_oracle as oracle
from tilerl_b200.config import TobadraConfig, tobadra_attention, tobadra_moe
from tilerl_b200.deluvik_layout import MoeLayout
from tilerl_b200.mixers import ChannelDeltaSpec, LayerSpec, LightningSpec
from tilerl_b200.tobadra_layout import gate_rows, layout_of, pad, router_rows

pytestmark = pytest.mark.gpu
DTYPES = pytest.mark.parametrize("dtype,tol", [(torch.float32, 1e-5), (torch.bfloat16, 1.5e-2)])


@pytest.fixture(scope="module")
def ops():
    from tilerl_b200.factory import make_ops
    return make_ops("cuda")


def _rel(a, b):
    a, b = a.double().cpu(), b.double().cpu()
    return float((a - b).abs().max() / b.abs().max().clamp_min(1e-30))


def _randn(*shape, seed=0, dtype=torch.float32):
    return torch.randn(*shape, device="cuda", generator=torch.Generator(device="cuda").manual_seed(seed)).to(dtype)


def _cfg(mixer, taps=3, hidden=64):
    return TobadraConfig(name="one", hidden=hidden, vocab=16, layers=(LayerSpec(mixer),), canon=taps)


def _state_pool(cfg, slots, dtype):
    """A state pool that holds not-a-number wherever nothing was written."""
    from tilerl_b200.kv import RecurrentPool
    pool = RecurrentPool(cfg, slots, "cuda", ring_dtype=dtype)
    pool.ring.fill_(math.nan)
    return pool


def _batch(lens, starts=None, slots=None):
    from tilerl_b200.batch import Batch
    n = len(lens)
    starts, slots = starts or [0] * n, slots or [n - i for i in range(n)]
    rows = [-(-(a + b) // 16) for a, b in zip(starts, lens)]
    order = torch.randperm(sum(rows), generator=torch.Generator().manual_seed(3)).tolist()
    seqs = []
    for i in range(n):
        seqs.append(dict(tokens=[1] * lens[i], start=starts[i], blocks=[1 + order.pop() for _ in range(rows[i])], slot=slots[i]))
    return Batch.build(seqs, "cuda"), sum(rows) + 1


# ---- joins and the convolution on the next input ------------------------------------------------------------------
@DTYPES
@pytest.mark.parametrize("hidden", [40, 64, 1000, 2048, 4608])
@pytest.mark.parametrize("taps,cuts", [(3, ((1, 1), (5, 1), (1, 1), (200, 2), (1, 17))), (1, ((4, 1), (1, 1))), (6, ((2, 1), (1, 1), (2, 3), (1, 1), (1, 1)))])
def test_gated_joins_in_portions(ops, dtype, tol, hidden, taps, cuts):
    """The stream after the branch, the next row, and that row convolved over portion borders."""
    ld = pad(hidden, 64)
    cfg = _cfg(LightningSpec(1, 16, 16, (0.5,)), taps, hidden)
    pool = _state_pool(cfg, 4, dtype)
    full = lambda x: torch.nn.functional.pad(x, (0, ld - hidden)).contiguous()
    post, nxt = 1 + 0.3 * _randn(1, hidden, seed=1), 1 + 0.3 * _randn(1, hidden, seed=2)
    w, bias, z_b = 0.5 * _randn(taps, hidden, seed=3), _randn(hidden, seed=4), _randn(hidden, seed=5)
    ops._join_dtype = dtype
    at, seen = [0, 0], [[], []]
    for step, cut in enumerate(cuts):
        t = sum(cut)
        batch, _ = _batch(cut, at)
        x, y, z = (_randn(t, hidden, seed=10 * step + 6 + i) for i in range(3))
        xs, zs = full(x), full(z)
        conv = (full(w), batch, pool, 0)
        if step % 2:                                              # the branch as a token's experts, one of them its own row
            own = full(_randn(t, hidden, seed=77)).to(dtype)
            weight = torch.rand(t, 2, device="cuda", generator=torch.Generator(device="cuda").manual_seed(8))
            place = torch.stack([torch.randperm(t, generator=torch.Generator().manual_seed(9)), torch.full((t,), -1)], 1).int().cuda()
            branch = weight[:, :1].double() * y.double()[place[:, 0].long()] + weight[:, 1:].double() * own[:, :hidden].double()
            h, hc = ops.gated_join_experts(xs, (full(y), place, weight), own, zs, full(z_b), full(post), full(nxt), 1e-4, hidden, conv)
        else:
            branch = (y + bias).double()
            h, hc = ops.gated_join(xs, full(y), full(bias), zs, full(z_b), full(post), full(nxt), 1e-4, hidden, conv)
        branch = (branch * oracle.sigmoid((z + z_b).double())).cpu()
        want = x.double().cpu() + oracle.unit_rms(branch, 1e-4) * post[0].double().cpu()
        assert _rel(xs[:, :hidden], want) < 2e-5 and not xs[:, hidden:].any()
        assert _rel(h[:, :hidden], oracle.unit_rms(want, 1e-4) * nxt[0].double().cpu()) < max(tol / 2, 2e-5) and not h[:, hidden:].any()
        o = 0
        for i, n in enumerate(cut):
            seen[i].append(h[o:o + n, :hidden].double().cpu())
            rows = torch.cat(seen[i])
            want_c = rows + oracle.causal_conv(rows, w.double().cpu().T)
            assert _rel(hc[o:o + n, :hidden], want_c[-n:]) < max(tol / 2, 2e-5) and not hc[o:o + n, hidden:].any(), step
            o, at[i] = o + n, at[i] + n


@DTYPES
@pytest.mark.parametrize("t", [1, 3, 200])
def test_the_normed_embedding(ops, dtype, tol, t):
    hidden, vocab = 72, 50
    pool, ld = _state_pool(_cfg(LightningSpec(1, 16, 16, (0.5,)), 2, hidden), 3, dtype), 128
    full = lambda x: torch.nn.functional.pad(x, (0, ld - hidden)).contiguous()
    table, post, nxt, w = full(_randn(56, hidden, seed=1)).to(dtype), 1 + 0.3 * _randn(1, hidden, seed=2), 1 + 0.3 * _randn(1, hidden, seed=3), _randn(2, hidden, seed=4)
    ids = torch.arange(t, device="cuda", dtype=torch.int32) % vocab
    batch, _ = _batch([t])
    x, h, hc = ops.embed_normed(table, vocab, ids, full(post), full(nxt), 1e-5, hidden, (full(w), batch, pool, 0))
    want = oracle.unit_rms(table[ids.long(), :hidden].double().cpu(), 1e-5) * post[0].double().cpu()
    assert _rel(x[:, :hidden], want) < 2e-6
    rows = h[:, :hidden].double().cpu()
    assert _rel(rows, oracle.unit_rms(want, 1e-5) * nxt[0].double().cpu()) < tol
    assert _rel(hc[:, :hidden], rows + oracle.causal_conv(rows, w.double().cpu().T)) < tol


# ---- projections -----------------------------------------------------------------------------------------------
@DTYPES
@pytest.mark.parametrize("t", [1, 2, 7, 8, 9, 100])
@pytest.mark.parametrize("hidden,n_in,n_gates,n_act", [(64, 48, 0, 0), (192, 320, 16, 0), (448, 608, 0, 400), (2048, 1040, 32, 512)])
def test_projections_of_two_inputs(ops, dtype, tol, t, hidden, n_in, n_gates, n_act):
    h, hc = _randn(t, hidden, seed=1, dtype=dtype), _randn(t, hidden, seed=2, dtype=dtype)
    w = (_randn(n_in + n_gates + hidden, hidden, seed=3) * 2 / hidden ** 0.5).to(dtype)
    proj, gates, z = ops.project_in(h, hc, w, n_in, n_gates, n_act, "silu")
    a, b = hc.double().cpu() @ w[:n_in + n_gates].double().cpu().T, h.double().cpu() @ w[n_in + n_gates:].double().cpu().T
    want = torch.cat([oracle.silu(a[:, :n_act]), a[:, n_act:n_in]], 1)
    assert _rel(proj, want) < tol and _rel(z, b) < 2e-5
    assert not n_gates or _rel(gates[:, :n_gates], a[:, n_in:]) < 2e-5


@DTYPES
@pytest.mark.parametrize("t", [1, 8, 9, 100])
@pytest.mark.parametrize("act", ["gelu", "gelu_erf", "silu"])
def test_up_projection_with_activation(ops, dtype, tol, t, act):
    h, w = _randn(t, 192, seed=1, dtype=dtype), (_randn(256 + 192, 192, seed=2) * 3 / 192 ** 0.5).to(dtype)
    up, z = ops.up_act(h, w, 256, act)
    y = h.double().cpu() @ w.double().cpu().T
    f = {"gelu": oracle.gelu_tanh, "gelu_erf": oracle.gelu_erf, "silu": oracle.silu}[act]
    assert _rel(up, f(y[:, :256])) < tol and _rel(z, y[:, 256:]) < 2e-5


# ---- attention over turned values --------------------------------------------------------------------------------
SHAPES = [(4, 2, 24, 20), (6, 1, 40, 64), (3, 3, 16, 30), (20, 1, 128, 128), (8, 2, 64, 64), (4, 2, 256, 64), (2, 2, 64, 256), (4, 4, 80, 144)]


@DTYPES
@pytest.mark.parametrize("shape", SHAPES, ids=str)
@pytest.mark.parametrize("window", [1, 37, 130, 4000])
def test_attention_in_portions(ops, dtype, tol, shape, window):
    """Decoded tokens, short portions and prompts in one batch: biases, rotations, pages, the window, the turn back."""
    from tilerl_b200.kv import PackedKvPool
    H, G, d, dv = shape
    s = tobadra_attention(H, G, d, dv, 1.5 / d ** 0.5, window, d // 4 * 2, 700.0)
    l, cfg = layout_of(s), _cfg(s)
    al = l.attn
    m = s.to_json()
    freqs = torch.tensor(s.rot.frequencies(), dtype=torch.float64, device="cuda")
    vfreqs = torch.tensor(s.value_frequencies() + (0.0,) * ((al.dv - dv) // 2), dtype=torch.float64, device="cuda")
    lens = [170, 40, 400]
    raw = [[_randn(n, g * k, seed=20 + 3 * i + j).to(dtype) for j, (g, k) in enumerate(((H, d), (G, d), (G, dv)))] for i, n in enumerate(lens)]
    bias = [_randn(g * k, seed=60 + j) for j, (g, k) in enumerate(((H, d), (G, d), (G, dv)))]

    def served(x, j):
        g, k, kp = ((H, d, al.dk), (G, d, al.dk), (G, dv, al.dv))[j]
        x = x.view(*x.shape[:-1], g, k)
        if j == 2:
            x = torch.nn.functional.pad(x.unflatten(-1, (2, k // 2)), (0, (kp - k) // 2)).flatten(-2)
        else:
            x = torch.nn.functional.pad(x, (0, kp - k))
        return x.flatten(-2)
    b = torch.cat([served(x, j) for j, x in enumerate(bias)]).contiguous()
    full, blocks = _batch(lens)
    pool = PackedKvPool(cfg, blocks, "cuda", dtype)
    pool.k.fill_(0xFF)
    at, got = [0, 0, 0], [[], [], []]
    from tilerl_b200.batch import Batch
    for step, cut in enumerate(((130, 1, 17), (1, 1, 1), (2, 3, 300), (1, 1, 1), (36, 34, 81))):
        batch = Batch.build([dict(tokens=[1] * c, start=at[i], blocks=[int(x) for x in full.block_table[i]], slot=i) for i, c in enumerate(cut)], "cuda")
        proj = torch.cat([torch.cat([served(x[at[i]:at[i] + c], j) for j, x in enumerate(raw[i])], 1) for i, c in enumerate(cut)]).contiguous()
        q, mid, turn = ops.turned_prep(proj, l, b, freqs, vfreqs, batch, pool, 0)
        mid[:, :al.n_out].fill_(7.0)
        ops.attn_splits = step % 2 * 4
        ops.softmax_attention(q, mid, al, None, 1.0, batch, pool, 0, turn)
        ops.attn_splits = 0
        assert not mid[:, l.n_mid:].any()
        o = 0
        for i, c in enumerate(cut):
            got[i].append(mid[o:o + c, :al.n_out].clone())
            o, at[i] = o + c, at[i] + c
    for i, n in enumerate(at):
        q, k, v = ((x[:n].double().cpu() + bb.double().cpu()).view(n, g, -1) for x, bb, g in zip(raw[i], bias, (H, G, G)))
        q, k, v = oracle.turn_halves(q, 700.0, s.rot.dims), oracle.turn_halves(k, 700.0, s.rot.dims), oracle.turn_halves(v, 700.0, dv)
        want = oracle.turn_halves(oracle.attend(q, k, v, m["scale"], window), 700.0, dv, -1.0)
        o = torch.cat(got[i]).view(n, H, 2, al.dv // 2)
        assert _rel(o[..., :dv // 2].reshape(n, H, dv), want) < tol and not o[..., dv // 2:].any(), i


# ---- scans -----------------------------------------------------------------------------------------------------
CUTS = [(130, 2, 1, 16, 33), (1, 1, 1, 1, 1), (2, 17, 100, 3, 1), (1, 1, 1, 1, 1), (66, 40, 47, 20, 64)]


def _in_portions(ops, l, cfg, dtype, rows, gates, mix):
    """Runs ``mix(proj, gates, batch, pool)`` over the portions of CUTS; outputs and final states by sequence."""
    pool = _state_pool(cfg, 7, dtype)
    at, out = [0] * 5, [[] for _ in range(5)]
    for cut in CUTS:
        batch, _ = _batch(cut, at, [6, 2, 5, 1, 3])
        proj = torch.cat([rows[i][at[i]:at[i] + c] for i, c in enumerate(cut)]).contiguous()
        g = None if gates is None else torch.cat([gates[i][at[i]:at[i] + c] for i, c in enumerate(cut)]).contiguous()
        o, y = 0, mix(proj, g, batch, pool)
        assert not y[:, l.heads * l.dv:].any()
        for i, c in enumerate(cut):
            out[i].append(y[o:o + c, :l.heads * l.dv].clone())
            o, at[i] = o + c, at[i] + c
    return [torch.cat(x) for x in out], at, [pool.view(1, s, 0)[0] for s in (6, 2, 5, 1, 3)]


def _padded(x, heads, d, dp):
    return torch.nn.functional.pad(x.view(*x.shape[:-1], heads, d), (0, dp - d)).flatten(-2)


@DTYPES
@pytest.mark.parametrize("spec", [LightningSpec(3, 20, 36, (1.0, 0.05, 0.9)), LightningSpec(2, 64, 64, (0.5, 0.999)), LightningSpec(1, 128, 80, (0.98,)), LightningSpec(2, 144, 16, (0.7, 0.2))],
                         ids=lambda s: f"{s.heads}-{s.dim}-{s.vdim}")
def test_lightning_in_portions(ops, dtype, tol, spec):
    l, cfg = layout_of(spec), _cfg(spec)
    n, H = 300, spec.heads
    dims = ((spec.dim, l.dk), (spec.dim, l.dk), (spec.vdim, l.dv), (spec.vdim, l.dv))
    raw = [[_randn(n, H * d, seed=10 + 4 * i + j).to(dtype) for j, (d, _) in enumerate(dims)] for i in range(5)]
    rows = [torch.cat([_padded(x, H, d, dp) for x, (d, dp) in zip(r, dims)], 1) for r in raw]
    norm = 1 + 0.3 * _randn(H * spec.vdim, seed=5)
    ld = torch.tensor([math.log(x) for x in spec.decay], device="cuda")
    out, at, states = _in_portions(ops, l, cfg, dtype, rows, None, lambda p, g, b, pool: ops.lightning_mix(p, ld, _padded(norm, H, spec.vdim, l.dv), l, b, pool, 1, 1e-4))
    for i in range(5):
        q, k, v, z = (x[:at[i]].double().cpu() for x in raw[i])
        q, k, v = q.view(-1, H, spec.dim), k.view(-1, H, spec.dim), v.view(-1, H, spec.vdim)
        o = oracle.scan_fixed(q, k, v, torch.tensor(spec.decay, dtype=torch.float64)).reshape(at[i], -1)
        want = oracle.unit_rms(o, 1e-4) * norm.double().cpu() * oracle.sigmoid(z)
        got = out[i].view(at[i], H, l.dv)
        assert _rel(got[..., :spec.vdim].reshape(at[i], -1), want) < tol and not got[..., spec.vdim:].any(), i


DELTAS = [ChannelDeltaSpec(4, 2, 24, 20, 4, 12, 20), ChannelDeltaSpec(2, 2, 64, 64, 3, 64, 64), ChannelDeltaSpec(2, 1, 128, 128, 4, 16, 100), ChannelDeltaSpec(3, 3, 80, 144, 1, 8, 8),
          ChannelDeltaSpec(1, 1, 144, 32, 6, 8, 8)]


@DTYPES
@pytest.mark.parametrize("kind", ["plain", "hard"])
@pytest.mark.parametrize("spec", DELTAS, ids=lambda s: f"{s.heads}-{s.kv_heads}-{s.dim}-{s.vdim}-{s.conv}")
def test_delta_rule_in_portions(ops, dtype, tol, spec, kind):
    """``hard``: keys that repeat and full writes (the triangular system is far from the identity), decays from none to nearly all."""
    l, cfg = layout_of(spec), _cfg(spec)
    n, H, G, d, dv = 300, spec.heads, spec.kv_heads, spec.dim, spec.vdim
    hard = kind == "hard"
    parts = ((G, d, l.dk), (G, d, l.dk), (H, dv, l.dv))
    raw = [[_randn(n, h * k, seed=10 + 5 * i + j).to(dtype) for j, (h, k, _) in enumerate(parts)] for i in range(5)]
    if hard:
        for r in raw:
            r[1] = (r[1][:5].repeat(60, 1).float() + 0.1 * r[1].float()).to(dtype)
    low = [[_randn(n, k, seed=100 + 2 * i + j).to(dtype) for j, k in enumerate((spec.decay_rank, spec.gate_rank))] for i in range(5)]
    gates = [_randn(n, gate_rows(l), seed=200 + i) + (4.0 if hard else 0.0) for i in range(5)]
    zero = lambda x: torch.nn.functional.pad(x, (0, l.r - x.shape[1]))
    rows = [torch.cat([_padded(x, h, k, kp) for x, (h, k, kp) in zip(r, parts)] + [zero(x) for x in lo], 1) for r, lo in zip(raw, low)]
    conv = [0.6 * _randn(h * k, spec.conv, seed=300 + j) for j, (h, k, _) in enumerate(parts)]
    a2, g2 = ((_randn(H * k, r, seed=310 + j) / r ** 0.5).to(dtype) for j, (k, r) in enumerate(((d, spec.decay_rank), (dv, spec.gate_rank))))
    dt_bias, a_log, norm = (6.0 if hard else 2.0) * _randn(H * d, seed=320) - 3.0, _randn(H, seed=321), 1 + 0.3 * _randn(dv, seed=322)
    w = {"conv": torch.cat([_padded(c.T, h, k, kp) for c, (h, k, kp) in zip(conv, parts)], 1).contiguous(), "a_log": a_log,
         "dt_bias": _padded(dt_bias, H, d, l.dk).contiguous()}
    fill = lambda t, k, kp: torch.nn.functional.pad(t.view(H, k, -1), (0, l.r - t.shape[1], 0, kp - k)).reshape(H * kp, l.r)
    w["low"] = torch.cat([fill(g2, dv, l.dv), fill(a2, d, l.dk)]).contiguous()
    hn = _padded(norm.repeat(H), H, dv, l.dv).contiguous()
    out, at, states = _in_portions(ops, l, cfg, dtype, rows, gates, lambda p, g, b, pool: ops.delta_mix(p, g, w, hn, l, b, pool, 1, 1e-4))
    dbl = lambda t: t.double().cpu()
    for i in range(5):
        m = at[i]
        q, k, v = (oracle.silu(oracle.causal_conv(dbl(x[:m]), dbl(c))).to(dtype).double() for x, c in zip(raw[i], conv))
        q, k = (oracle.unit_length(x.view(m, G, d)).repeat_interleave(H // G, 1) for x in (q, k))
        step = oracle.softplus(dbl(low[i][0][:m]) @ dbl(a2).T + dbl(dt_bias)).view(m, H, d)
        g = torch.exp(-torch.exp(dbl(a_log))[None, :, None] * step)
        o = oracle.scan_delta(q * d ** -0.5, k, v.view(m, H, dv), g, oracle.sigmoid(dbl(gates[i][:m, :H])))
        z = oracle.sigmoid((dbl(low[i][1][:m]) @ dbl(g2).T).to(dtype).double())
        want = (oracle.unit_rms(o, 1e-4) * dbl(norm)).reshape(m, -1) * z
        got = out[i].view(m, H, l.dv)
        assert _rel(got[..., :dv].reshape(m, -1), want) < max(tol, 1e-4), i
        assert not got[..., dv:].any()


# ---- experts ----------------------------------------------------------------------------------------------------
MOES = [tobadra_moe(24, 5, 3, 40, 1.5, 1, 2, 1), tobadra_moe(64, 8, 8, 0, 0.7), tobadra_moe(192, 70, 8, 192, 2.0, 10, 40, 9), tobadra_moe(100, 2, 1, 300, 1.0, 6, 4, 2),
        tobadra_moe(256, 64, 4, 256, 1.0, 0, 64, 5)]


@DTYPES
@pytest.mark.parametrize("t", [1, 2, 9, 40, 65, 700])
@pytest.mark.parametrize("spec", MOES, ids=lambda s: f"{s.ff}-{s.experts}-{s.top}")
@pytest.mark.parametrize("hidden", [64, 448])
def test_grouped_experts(ops, dtype, tol, t, spec, hidden):
    m, r = MoeLayout(spec), spec.router
    h = _randn(t, hidden, seed=1, dtype=dtype)
    n = spec.outputs
    z = torch.full((t, router_rows(spec) + hidden), math.nan, device="cuda")
    z[:, :n + 1] = 1.5 * _randn(t, n + 1, seed=2)
    corr = torch.full((pad(n, 8),), math.nan, device="cuda")
    corr[:n] = 0.1 * _randn(n, seed=3) - 0.2
    up, down = torch.zeros(m.n, m.ff, hidden, device="cuda", dtype=dtype), torch.zeros(m.n, hidden, m.ff, device="cuda", dtype=dtype)
    w = {}
    for e in range(m.n):
        ff = spec.ff if e < spec.experts else min(m.ff, spec.shared - (e - spec.experts) * m.ff)
        up[e, :ff], down[e, :, :ff] = (_randn(ff, hidden, seed=10 + 2 * e) * 2 / hidden ** 0.5).to(dtype), (_randn(hidden, ff, seed=11 + 2 * e) * 1.5 / ff ** 0.5).to(dtype)
        w[f"e{e}.up"], w[f"e{e}.down"] = up[e, :ff].double().cpu(), down[e, :, :ff].double().cpu()
    hd, zd = h.double().cpu(), z[:, :n + 1].double().cpu()
    idx, weight = oracle.route(zd[:, :n], corr[:n].double().cpu(), {"groups": {"count": r.groups, "keep": r.keep}, "top": spec.top, "scale": r.scale})
    want = torch.zeros(t, hidden, dtype=torch.float64)
    for e in range(n):
        rows, place = torch.nonzero(idx == e, as_tuple=True)
        if len(rows):
            want[rows] += weight[rows, place][:, None] * (oracle.plain_ff(hd[rows], w, f"e{e}.", oracle.gelu_erf) if e < spec.experts else hd[rows])
    for j in range(m.pieces):
        want += oracle.sigmoid(zd[:, n:]) * oracle.plain_ff(hd, w, f"e{spec.experts + j}.", oracle.gelu_erf)
    y, place, weight = ops.routed_experts(h, z, corr, up, down, m)
    pl = place.long().cpu().view(t, -1)
    assert sorted(pl[pl >= 0].tolist()) == list(range(int((pl >= 0).sum())))
    assert torch.equal(pl < 0, torch.cat([idx >= spec.experts, torch.zeros(t, m.pieces, dtype=torch.bool)], 1))
    y, weight = y.double().cpu(), weight.double().cpu()
    got = sum(weight[:, j, None] * torch.where((pl[:, j] >= 0)[:, None], y[pl[:, j].clamp_min(0)], hd) for j in range(m.slots))
    assert _rel(got, want) < tol


def test_tokens_that_only_choose_themselves(ops):
    """No expert has a row, and none is left over from the tick before."""
    spec = tobadra_moe(64, 4, 2, 0, 1.0, 4, 2, 1)
    m, dt = MoeLayout(spec), torch.bfloat16
    up, down, corr = _randn(4, 64, 64, seed=1, dtype=dt), _randn(4, 64, 64, seed=2, dtype=dt), torch.zeros(8, device="cuda")
    for t in (1, 20, 100):
        h, z = _randn(t, 64, seed=3, dtype=dt), _randn(t, router_rows(spec) + 64, seed=4)
        ops.routed_experts(h, z, corr, up, down, m)
        z[:, 4:8] += 50.0
        _, place, weight = ops.routed_experts(h, z, corr, up, down, m)
        want = torch.softmax(z[:, 4:8], 1).topk(2, dim=1).values
        assert (place < 0).all() and torch.allclose(weight, want, atol=1e-5)


def test_a_token_that_is_no_number_leaves_the_others_alone(ops):
    spec = tobadra_moe(64, 6, 3, 64, 1.0, 2, 4, 2)
    m, dt = MoeLayout(spec), torch.bfloat16
    up, down, corr = _randn(m.n, 64, 64, seed=1, dtype=dt) * 0.1, _randn(m.n, 64, 64, seed=2, dtype=dt) * 0.1, torch.zeros(8, device="cuda")
    for t in (3, 80):
        h, z = _randn(t, 64, seed=3, dtype=dt), _randn(t, router_rows(spec) + 64, seed=4)
        sums = []
        for bad in (False, True):
            if bad:
                h[1], z[1] = math.nan, math.nan
            y, place, weight = ops.routed_experts(h, z, corr, up, down, m)
            pl = place.view(t, -1).long()
            assert int((pl[1] >= 0).sum()) >= 1 and sorted(pl[pl >= 0].tolist()) == list(range(int((pl >= 0).sum())))
            sums.append((weight[:, :, None] * torch.where((pl >= 0)[..., None], y[pl.clamp_min(0)].float(), h.float()[:, None])).sum(1).clone())
        keep = [i for i in range(t) if i != 1]
        assert _rel(sums[1][keep], sums[0][keep]) < 1e-5
