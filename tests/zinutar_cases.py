"""Models and backends of the Zinutar tests."""
import pytest
import torch

import zinutar_oracle as oracle
from tilerl_b200.config import AttnSpec, BlockSpec, LoopSpec, MlpSpec, ZinutarConfig, zinutar_tiny

# per backend: device, compute dtype, largest relative error (rms over the vocabulary against the oracle)
BACKENDS = {"cpu": ("cpu", torch.float32, 2e-5), "cuda-f32": ("cuda", torch.float32, 2e-5),
            "cuda-bf16": ("cuda", torch.bfloat16, 3e-2)}
backends = pytest.mark.parametrize("backend", ["cpu", pytest.param("cuda-f32", marks=pytest.mark.gpu),
                                               pytest.param("cuda-bf16", marks=pytest.mark.gpu)])


def _cfg(name, **kw):
    return ZinutarConfig(name=name, max_ctx=4096, **kw)


CONFIGS = {
    # three sizes of layers, one without a feed-forward, a loop from the first layer on
    "tiny": zinutar_tiny(),
    # many query heads on one kv head, values wider than keys, one layer three times
    "mqa": _cfg("mqa", hidden=96, vocab=210, rms_eps=1e-3, loop=LoopSpec(1, 2, 3),
                layers=(BlockSpec(AttnSpec(6, 1, 32, 48, 0.4), MlpSpec(64)), BlockSpec(AttnSpec(20, 1, 16, 16, 0.5), MlpSpec(200)),
                        BlockSpec(AttnSpec(3, 3, 8, 20, 1.0), MlpSpec(40)))),
    # no loop, one head per group, head sizes that are no multiple of 16, no feed-forward at the end
    "mha": _cfg("mha", hidden=50, vocab=77, rms_eps=1e-6,
                layers=(BlockSpec(AttnSpec(3, 3, 20, 12, 0.7), MlpSpec(33)), BlockSpec(AttnSpec(2, 2, 72, 88, 0.1), None))),
    # a loop that runs once, one layer
    "one": _cfg("one", hidden=64, vocab=64, rms_eps=1e-5, loop=LoopSpec(0, 1, 1),
                layers=(BlockSpec(AttnSpec(1, 1, 16, 16, 0.25), MlpSpec(16)),)),
    # wide heads: the largest kernel tiles
    "wide": _cfg("wide", hidden=192, vocab=128, rms_eps=1e-5, loop=LoopSpec(0, 2, 2),
                 layers=(BlockSpec(AttnSpec(4, 2, 256, 192, 0.06), MlpSpec(320)), BlockSpec(AttnSpec(4, 1, 128, 128, 0.09), MlpSpec(64)))),
}


def random_weights(cfg, seed=0):
    """Checkpoint tensors with strong heads: scores and weights vary, nothing is equal to 1 or 0."""
    from tilerl_b200.zinutar_layout import tensor_shapes
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        leaf = name.split(".")[-1]
        t = torch.randn(shape, generator=g)
        if "norm" in name:
            t = 1.0 + 0.3 * t
        elif leaf == "pb":
            t = -3.0 + t
        elif leaf == "act":
            t = 0.6 + 0.3 * t
        else:
            t = t * (1.3 / shape[-1] ** 0.5)
        out[name] = t.to(torch.bfloat16).float()      # representable in every compute dtype
    return out


def build(cfg, weights, backend, *, max_tokens=1024, slots=4, graph=True, **kw):
    from tilerl_b200.factory import build_engine, make_ops
    from tilerl_b200.models.zinutar import ZinutarModel
    device, dtype, _ = BACKENDS[backend]
    model = ZinutarModel.from_tensors(cfg, weights.__getitem__, device, dtype)
    return build_engine(model, make_ops(device), device=device, blocks=max_tokens // 16 + 1, slots=slots, max_ctx=max_tokens,
                        graph=graph, prefix=kw.pop("prefix", False), **kw)


def tokens(cfg, n, seed=1):
    g = torch.Generator().manual_seed(seed)
    return torch.randint(0, cfg.vocab, (n,), generator=g).tolist()


def want_logits(cfg, weights, toks):
    return oracle.forward(cfg.to_json(), weights, toks)[0].float()


def rel_err(got, want):
    """Largest over positions: rms error over the vocabulary (means removed) / rms of the wanted logits."""
    got, want = got.detach().float().cpu(), want.float()
    assert got.shape == want.shape, (got.shape, want.shape)
    d = got - want
    d = d - d.mean(-1, keepdim=True)
    w = want - want.mean(-1, keepdim=True)
    e = d.pow(2).mean(-1).sqrt() / w.pow(2).mean().sqrt()
    return float(torch.nan_to_num(e, nan=float("inf")).max())


def feed_all(eng, key, toks, cuts, close=True):
    """Feed ``toks`` in portions of the sizes ``cuts`` (the last repeats); logits of every position."""
    out, at, i = [], 0, 0
    while at < len(toks):
        n = min(cuts[min(i, len(cuts) - 1)], len(toks) - at)
        last = at + n == len(toks)
        out.append(eng.feed([(key, toks[at:at + n], list(range(n)))], [key] if last and close else []).clone())
        at, i = at + n, i + 1
    return torch.cat(out)
