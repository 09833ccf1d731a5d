"""Models and helpers of the Deluvik tests."""
from dataclasses import replace

import torch

import deluvik_oracle as oracle
from fetotar_cases import TOL, close  # noqa: F401
from tilerl_b200.config import (DeluvikConfig, deluvik_attention, deluvik_conv_attention, deluvik_parallel, deluvik_tiny)
from tilerl_b200.mixers import BandScalingSpec, GluSpec, LayerSpec, LruSpec, MoeSpec, RotarySpec
from zinutar_cases import BACKENDS, backends, feed_all, rel_err, tokens  # noqa: F401

SCALED = BandScalingSpec(5.0, 0.5, 3.0, 90.0)


def rot(dims, base=2000.0, scaling=None):
    return RotarySpec(dims, base, scaling)


def tied(heads=3, kv_heads=1, dim=20, scale=0.25, cap=20.0, dims=None, **kw):
    return deluvik_attention(heads, kv_heads, dim, scale, cap, rot(dims or dim, **kw))


def conv(heads=4, kv_heads=2, dim=24, vdim=40, scale=0.2, taps=3, dims=16, kv_from=None):
    return deluvik_conv_attention(heads, kv_heads, dim, vdim, scale, taps, rot(dims), kv_from)


def both(window=19, heads=4, kv_heads=2, dim=24, vdim=12, lru=(44, 4, 3), scales=(0.7, 1.3), dims=8):
    return deluvik_parallel(*scales, LruSpec(*lru), heads, kv_heads, dim, vdim, 0.2, window, rot(dims))


def _cfg(name, layers, **kw):
    base = dict(hidden=56, vocab=90, logit_cap=12.0, norm_eps=1e-5, max_ctx=4096)
    return DeluvikConfig(name=name, layers=tuple(layers), **{**base, **kw})


CONFIGS = {
    "tiny": deluvik_tiny(),
    # one mixer each, every size its own, with each kind of feed-forward and none
    "tied": _cfg("tied", [LayerSpec(tied(scaling=SCALED), GluSpec(70, "gelu")), LayerSpec(tied(6, 3, 36, 0.5, 5.0, dims=12), MoeSpec(24, 5, 3, 50))]),
    "conv": _cfg("conv", [LayerSpec(conv(), MoeSpec(72, 7, 1, 0)), LayerSpec(conv(3, 3, 40, 16, 0.3, 5, 40)), LayerSpec(conv(kv_from=0)),
                          LayerSpec(conv(2, 1, 16, 16, 0.3, 1, 2), GluSpec(33, "gelu"))], hidden=70),
    "both": _cfg("both", [LayerSpec(both(), GluSpec(40, "gelu")), LayerSpec(both(7, 6, 1, 64, 80, (96, 1, 6), (1.0, -0.6), 64)),
                          LayerSpec(both(33, 2, 2, 16, 16, (30, 10, 1), (1.2, 0.5), 2), MoeSpec(130, 3, 3, 200))], vocab=131),
    # the order of layers turned round, two layers that read one layer's keys, a large eps, a window of one and one wider than any sequence
    "mixed": _cfg("mixed", [LayerSpec(conv(6, 2, 32, 48, 0.2, 4, 20), GluSpec(96, "gelu")), LayerSpec(both(1, lru=(64, 2, 4)), MoeSpec(20, 40, 6, 20)),
                            LayerSpec(conv(6, 2, 32, 48, 0.3, 2, 20, kv_from=0)), LayerSpec(tied(4, 2, 48, 0.15, 30.0, scaling=SCALED), MoeSpec(64, 4, 2, 0)),
                            LayerSpec(conv(6, 2, 32, 48, 0.1, 4, 20, kv_from=0), MoeSpec(33, 9, 2, 70)), LayerSpec(both(5000), GluSpec(48, "gelu"))],
                  norm_eps=1e-3, logit_cap=40.0, vocab=131),
    # wide heads, many of them on one key head, large parts: the largest tiles
    "wide": _cfg("wide", [LayerSpec(tied(20, 1, 128, 0.09, 40.0), MoeSpec(192, 6, 2, 192)), LayerSpec(both(70, 4, 2, 256, 128, (640, 2, 4), (0.5, 0.9), 128)),
                          LayerSpec(conv(4, 4, 64, 256, 0.1, 4, 64), GluSpec(320, "gelu"))], hidden=192),
}


def random_weights(cfg, seed=0):
    """Checkpoint tensors under which every mechanism moves the logits: uneven attention, sinks that take a share, decays from slow
    to fast, routers without close calls, branches that count without drowning the stream."""
    from tilerl_b200.deluvik_layout import tensor_shapes
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        leaf = name.split(".")[-1]
        t = torch.randn(shape, generator=g)
        if leaf in ("norm1", "norm2"):
            t = 0.5 + 0.15 * t
        elif leaf == "norm":
            t = 1.0 + 0.3 * t
        elif leaf == "sink":
            t = 1.0 + 1.5 * t
        elif leaf == "lam":
            t = 2.0 * t - 3.0                              # some channels remember for long, some forget at once
        elif name.endswith("router.b"):
            t = 0.5 * t
        elif leaf == "b":
            t = 0.4 * t
        elif leaf == "conv":
            t = 0.6 * t
        elif leaf == "router":
            t = t * (4.0 / shape[-1] ** 0.5)
        elif leaf == "embed":
            t = 1.2 * t
        else:
            t = t * (1.3 / shape[-1] ** 0.5)
        out[name] = t
    _clear_choices(cfg, out, g)
    return {n: t.to(torch.bfloat16).float() for n, t in out.items()}      # representable in every compute dtype


def _clear_choices(cfg, w, g, share=0.05, margin=1.2):
    """Routers without close calls, which rounding would turn round: a few columns of the stream that no branch writes to (their norm
    weights are zero) carry what mostly decides, drawn for every token until the last expert chosen stands clear of the next one."""
    moe = [(i, l.mlp) for i, l in enumerate(cfg.layers) if isinstance(l.mlp, MoeSpec)]
    if not moe:
        return
    r = 12
    for i, l in enumerate(cfg.layers):
        for n in (f"l{i}.norm1", f"l{i}.norm2"):
            if n in w:
                w[n][-r:] = 0.0
    for i, m in moe:
        t = w[f"l{i}.mlp.router"]
        t[:, :-r] *= share
        t[:, -r:] = torch.randn(t.shape[0], r, generator=g) * 4.0 / r ** 0.5
    open_ = torch.arange(cfg.vocab)
    for _ in range(4000):
        w["embed"][open_, -r:] = 1.2 * torch.randn(len(open_), r, generator=g)
        clear = torch.ones(len(open_), dtype=torch.bool)
        for i, m in moe:
            if m.top < m.experts:
                z = (w["embed"][open_, -r:] @ w[f"l{i}.mlp.router"][:, -r:].T + w[f"l{i}.mlp.router.b"]).sort(dim=1, descending=True).values
                clear &= z[:, m.top - 1] - z[:, m.top] > margin
        open_ = open_[~clear]
        if not len(open_):
            return
    raise AssertionError("no clear choice found")


def build(cfg, weights, backend, *, max_tokens=1024, slots=4, graph=True, **kw):
    from tilerl_b200.factory import build_engine, make_ops
    from tilerl_b200.models.deluvik import DeluvikModel
    device, dtype, _ = BACKENDS[backend]
    model = DeluvikModel.from_tensors(cfg, weights.__getitem__, device, dtype)
    return build_engine(model, make_ops(device), device=device, blocks=max_tokens // 16 + 1, slots=slots, max_ctx=max_tokens,
                        graph=graph, prefix=kw.pop("prefix", False), **kw)


def want_logits(cfg, weights, toks):
    return oracle.forward(cfg.to_json(), weights, toks)[0].float()


def needle_model(kind, window=None, heads=4, kv_heads=2, dim=32, sharp=18.0):
    """One attention layer (``kind``: tied, conv, shared, both) in which token 1 asks for token 2: that score stands far above every
    other, so the logits of a 1 show whether a 2 is among the keys it sees, and where a sink or a cap holds it back.  Only dimensions
    that do not turn ask."""
    free, taps = slice(8, dim), 1
    if kind == "tied":
        layers = [LayerSpec(deluvik_attention(heads, kv_heads, dim, 1.0, 60.0, rot(8)))]
    elif kind == "both":
        layers = [LayerSpec(deluvik_parallel(1.0, 0.3, LruSpec(24, 2, 2), heads, kv_heads, dim, 40, 1.0, window, rot(8)))]
    else:
        a = deluvik_conv_attention(heads, kv_heads, dim, 40, 1.0, taps, rot(8))
        layers = [LayerSpec(a)] + ([LayerSpec(replace(a, kv_from=0))] if kind == "shared" else [])
    cfg = _cfg("needle-" + kind, layers, hidden=96, logit_cap=50.0)
    w = random_weights(cfg, seed=11)
    last = len(layers) - 1
    pq, pk = (f"l{last}.mix.", "l0.mix.") if kind != "both" else ("l0.mix.left.", "l0.mix.left.")
    if kind == "shared":
        w["l0.norm1"] *= 0.01                               # the second layer sees the embeddings, nearly
    for p, n in ((pq, "q"), (pk, "k")):
        w[p + n + ".norm"] = torch.ones_like(w[p + n + ".norm"])
        if f"{p}{n}.conv" in w:
            w[f"{p}{n}.conv"] = torch.ones_like(w[f"{p}{n}.conv"])
    e1, e2 = (w["embed"][i] / w["embed"][i].norm() for i in (1, 2))
    e1 = e1 - (e1 @ e2) * e2
    e1 = e1 / e1.norm()
    q, k = w[pq + "q"].view(heads, dim, -1), w[pk + "k"].view(kv_heads, dim, -1)
    g = torch.Generator().manual_seed(5)
    for h in range(kv_heads):
        mark = torch.randn(dim - 8, generator=g)
        mark = mark / mark.norm()
        k[h, free] += torch.outer(mark, e2)                 # weak enough that the norm leaves other tokens' keys alone
        for i in range(h * heads // kv_heads, (h + 1) * heads // kv_heads):
            q[i] *= 0.05
            q[i, free] += sharp * torch.outer(mark, e1)
    return cfg, {n: t.to(torch.bfloat16).float() for n, t in w.items()}
