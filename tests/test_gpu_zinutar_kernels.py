"""The kernels of the fp32-stream ops (csrc/stream.cu, linear_rows.cu, attn_sigmoid.cu) against fp32 torch, shape by
shape: odd sizes, every row count, every tile variant of the attention, splits and page borders."""
import pytest
import torch

pytestmark = pytest.mark.gpu


@pytest.fixture(scope="module")
def ops():
    from tilerl_b200.factory import make_ops
    return make_ops("cuda")


def _rel(a, b):
    a, b = a.float(), b.float()
    return float((a - b).abs().max() / b.abs().max().clamp_min(1e-30))


@pytest.mark.parametrize("n,k", [(16, 64), (40, 128), (1000, 320), (4096, 2048), (24, 11264), (333 * 8, 64)])
@pytest.mark.parametrize("m", [1, 2, 3, 8, 9, 16])
def test_row_projection(ops, m, n, k):
    if m > ops.lib.trl_linear_rows_max(k):
        pytest.skip("more rows than shared memory holds")
    g = torch.Generator(device="cuda").manual_seed(m * 7 + n)
    w = (torch.randn(n, k, device="cuda", generator=g) / k ** 0.5).bfloat16()
    x = torch.randn(m, k, device="cuda", generator=g)
    nw = 1 + 0.2 * torch.randn(k, device="cuda", generator=g)
    true_k = k - 13
    x[:, true_k:], nw[true_k:] = 0, 0                           # stream padding
    want = x.bfloat16().float() @ w.float().t()
    y16, y32 = torch.empty(m, n, dtype=torch.bfloat16, device="cuda"), torch.empty(m, n, device="cuda")
    ops._linear_rows(x.bfloat16(), w, y16, 0)
    ops._linear_rows(x.bfloat16(), w, y32, 1)
    assert _rel(y16, want) < 6e-3 and _rel(y32, want) < 1e-5
    acc = torch.randn(m, n, device="cuda", generator=g)
    base = acc.clone()
    ops._linear_rows(x.bfloat16(), w, acc, 2)
    assert _rel(acc, base + want) < 1e-5
    h = (x * torch.rsqrt(x.pow(2).sum(-1, keepdim=True) / true_k + 1e-3) * nw)
    ops._linear_rows(x, w, y32, 1, nw, 1e-3, true_k)
    assert _rel(y32, h.bfloat16().float() @ w.float().t()) < 2e-3
    again = torch.empty_like(y32)
    ops._linear_rows(x, w, again, 1, nw, 1e-3, true_k)
    assert torch.equal(again, y32)                              # a run repeats bit for bit


def test_row_projection_refuses_what_does_not_fit(ops):
    from tilerl_b200.ops.native import KernelError
    k = 65536
    assert ops.lib.trl_linear_rows_max(k) < 2
    w = torch.zeros(16, k, dtype=torch.bfloat16, device="cuda")
    x, y = torch.zeros(2, k, dtype=torch.bfloat16, device="cuda"), torch.zeros(2, 16, device="cuda")
    with pytest.raises(KernelError):
        ops._linear_rows(x, w, y, 1)
    assert not ops._streams(2, w)


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 1e-6), (torch.bfloat16, 5e-3)])
@pytest.mark.parametrize("width", [50, 64, 2048, 9000])
def test_embedding_norm_and_stream_norm(ops, dtype, tol, width):
    ld = (width + 63) // 64 * 64
    g = torch.Generator(device="cuda").manual_seed(width)
    table = torch.zeros(37, ld, device="cuda")
    table[:, :width] = torch.randn(37, width, device="cuda", generator=g) * 3
    table = table.to(dtype)
    w = torch.zeros(ld, device="cuda")
    w[:width] = 1 + 0.3 * torch.randn(width, device="cuda", generator=g)
    ids = torch.tensor([0, 36, 5, 5], dtype=torch.int32, device="cuda")
    x, x0 = ops.embed_norm(table, w, ids, 1e-2, width, True)
    e = table.float()[ids.long()]
    norm = lambda v: v / torch.sqrt(v.pow(2).sum(-1, keepdim=True) / width + 1e-2) * w
    assert _rel(x, norm(e)) < 1e-6 and torch.equal(x, x0)
    ops.stream_add(x, x0)
    assert torch.equal(x, 2 * x0)
    x += torch.randn(4, 1, device="cuda", generator=g) * x
    assert _rel(ops._stream_norm(x, w, 1e-2, width, dtype), norm(x)) < tol
    assert ops.embed_norm(table, w, torch.tensor([99], dtype=torch.int32, device="cuda"), 1e-2, width, False)[0].abs().max() == 0
    assert ops.read_device_error()[0] == 2                      # an id outside the table: a zero row and the error word


def _layout(heads, kv, dim, vdim, scale, ff):
    from tilerl_b200.config import AttnSpec, BlockSpec, MlpSpec, ZinutarConfig
    from tilerl_b200.zinutar_layout import BlockLayout
    cfg = ZinutarConfig(name="k", hidden=64, vocab=8, layers=(BlockSpec(AttnSpec(heads, kv, dim, vdim, scale), MlpSpec(ff) if ff else None),))
    return cfg, BlockLayout.of(cfg.layers[0])


def _run(ops, cfg, l, lens, starts, dtype, seed=0, blocks=None):
    """Fill the pool with ``starts`` tokens per sequence, then one tick of ``lens``: (got, want) of ``block_mid`` and
    ``sigmoid_attention``, the wanted values by the reference backend on the same pool."""
    from tilerl_b200.batch import Batch
    from tilerl_b200.kv import PackedKvPool
    from tilerl_b200.ops.backend import RefOps
    g = torch.Generator().manual_seed(seed)
    per = max((s + n + 15) // 16 for s, n in zip(starts, lens))
    perm = (torch.randperm(len(lens) * per, generator=g) + 1).tolist()
    mine = [perm[i * per:(i + 1) * per] for i in range(len(lens))]
    pools = [PackedKvPool(cfg, len(perm) + 1, d, dtype=dtype) for d in ("cuda", "cpu")]
    pools[0].k.fill_(0xFF)                                      # NaN everywhere nothing was written
    bias = -2 + torch.randn(l.heads, generator=g)
    act = torch.tensor([0.7, -0.4, 0.9, 0.3])
    ref = RefOps(act_dtype=torch.float32)
    out = []
    for phase in (0, 1):
        n = starts if phase == 0 else lens
        seqs = [dict(tokens=[0] * n[i], start=0 if phase == 0 else starts[i], blocks=mine[i], slot=i + 1)
                for i in range(len(lens)) if n[i]]
        if not seqs:
            continue
        t = sum(len(s["tokens"]) for s in seqs)
        proj = torch.zeros(t, l.n_in)
        for a, h, d, dp in ((0, l.heads, l.dim, l.dk), (l.k0, l.kv_heads, l.dim, l.dk), (l.v0, l.kv_heads, l.vdim, l.dv)):
            proj[:, a:a + h * dp].view(t, h, dp)[:, :, :d] = torch.randn(t, h, d, generator=g)
        proj[:, l.up0:l.up0 + l.ff] = torch.randn(t, l.ff, generator=g) * 2
        proj = proj.to(dtype)
        b = [Batch.build(seqs, d) for d in ("cuda", "cpu")]
        pc = proj.cuda()
        mid = ops.block_mid(pc, act.cuda() if l.ff else None, l, b[0], pools[0], 0, 1e-4)
        pf = proj.float()
        want = ref.block_mid(pf, act if l.ff else None, l, b[1], pools[1], 0, 1e-4)
        if phase:
            ops.sigmoid_attention(pc, mid, bias.cuda(), l, b[0], pools[0], 0, 1e-4)
            ref.sigmoid_attention(pf, want, bias, l, b[1], pools[1], 0, 1e-4)
            out = [mid.float().cpu(), want]
    assert ops.read_device_error()[0] == 0
    return out


SHAPES = [(4, 2, 64, 64, 3.0, 96), (6, 2, 24, 40, 2.0, 100), (8, 1, 128, 128, 1.0, 0), (20, 1, 16, 96, 4.0, 40),
          (2, 2, 256, 256, 0.5, 20000), (4, 4, 256, 48, 0.5, 72), (3, 1, 80, 192, 1.0, 33), (5, 5, 8, 8, 6.0, 16),
          (3, 3, 40, 16, 2.0, 0)]


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 2e-5), (torch.bfloat16, 8e-3)])
@pytest.mark.parametrize("shape", SHAPES)
def test_block_middle_and_attention(ops, shape, dtype, tol):
    cfg, l = _layout(*shape)
    for lens, starts in (([1, 1, 1], [0, 15, 200]), ([5, 1, 40], [16, 64, 3]), ([150], [0]), ([2, 16], [33, 111]), ([70, 3, 1], [130, 0, 300])):
        got, want = _run(ops, cfg, l, lens, starts, dtype)
        a = l.attn_cols
        assert _rel(got[:, :a], want[:, :a]) < tol, (lens, starts)
        if l.n_out > a:
            assert _rel(got[:, a:], want[:, a:]) < tol
            assert torch.equal(got[:, a + l.ff:], torch.zeros_like(got[:, a + l.ff:]))


@pytest.mark.parametrize("splits", [0, 1, 3, 7, 64])
@pytest.mark.parametrize("shape", [(4, 2, 64, 64, 3.0, 16), (4, 1, 128, 128, 1.0, 16), (2, 1, 256, 256, 0.5, 16), (6, 2, 40, 24, 2.0, 16)])
def test_splits_change_nothing(ops, shape, splits, monkeypatch):
    """Every split count, in prompts and in decoding, around the ends of pages, tiles and splits."""
    cfg, l = _layout(*shape)
    if splits:
        monkeypatch.setattr(type(ops), "_sigmoid_splits", lambda *a, **k: splits)
    for start in (0, 62, 63, 64, 127, 128, 255, 256, 257, 511, 640):
        for n in (1, 2, 35):
            got, want = _run(ops, cfg, l, [n], [start], torch.bfloat16, seed=start + n)
            assert _rel(got[:, :l.attn_cols], want[:, :l.attn_cols]) < 8e-3, (start, n)
