"""Models and helpers of the Tobadra tests."""
import torch

import tobadra_oracle as oracle
from fetotar_cases import TOL, close  # noqa: F401
from tilerl_b200.config import TobadraConfig, tobadra_attention, tobadra_moe, tobadra_tiny
from tilerl_b200.mixers import ChannelDeltaSpec, DenseSpec, LayerSpec, LightningSpec, MoeSpec
from zinutar_cases import BACKENDS, backends, feed_all, rel_err, tokens  # noqa: F401


def attn(window=19, heads=4, kv_heads=2, dim=24, vdim=36, scale=0.2, dims=16, base=700.0):
    return tobadra_attention(heads, kv_heads, dim, vdim, scale, window, dims, base)


def delta(heads=4, kv_heads=2, dim=24, vdim=20, conv=4, ranks=(12, 20)):
    return ChannelDeltaSpec(heads, kv_heads, dim, vdim, conv, *ranks)


def dense(ff):
    return DenseSpec(ff, "gelu")


def _cfg(name, layers, **kw):
    base = dict(hidden=56, vocab=90, canon=3, logit_scale=0.7, norm_eps=1e-5, max_ctx=4096)
    return TobadraConfig(name=name, layers=tuple(layers), **{**base, **kw})


CONFIGS = {
    "tiny": tobadra_tiny(),
    # one mixer each, every size its own, with each kind of feed-forward and none
    "attention": _cfg("attention", [LayerSpec(attn(), tobadra_moe(24, 5, 3, 50, 0.8, 1, 2, 1)), LayerSpec(attn(1, 6, 1, 40, 16, 0.15, 40)),
                                    LayerSpec(attn(33, 3, 3, 16, 50, 0.3, 2, 50.0), dense(70)), LayerSpec(attn(5000, 2, 2, 20, 20, 0.3, 20), dense(33))], hidden=70),
    "lightning": _cfg("lightning", [LayerSpec(LightningSpec(3, 20, 36, (0.5, 0.9, 1.0)), dense(40)), LayerSpec(LightningSpec(1, 64, 16, (0.97,))),
                                    LayerSpec(LightningSpec(5, 16, 16, (1.0, 0.05, 0.3, 0.99, 0.8)), tobadra_moe(130, 3, 3, 200, 2.0))], vocab=131, canon=1),
    "delta": _cfg("delta", [LayerSpec(delta(), dense(40)), LayerSpec(delta(6, 1, 40, 64, 1, (70, 3))), LayerSpec(delta(3, 3, 16, 16, 2, (5, 130)), tobadra_moe(20, 9, 1, 0, 1.0, 3, 4, 3)),
                            LayerSpec(delta(2, 2, 72, 40, 6))], vocab=77, canon=2),
    # every mixer, parameters used again (by an earlier layer, too), many groups, all chosen from one, wide shared experts, large eps
    "mixed": _cfg("mixed", [LayerSpec(delta(4, 4, 32, 48), tobadra_moe(20, 19, 3, 20, 1.4, 5, 12, 3), weights_of=3), LayerSpec(attn(30), dense(96)),
                            LayerSpec(LightningSpec(4, 32, 24, (0.6, 0.9, 0.98, 0.999)), tobadra_moe(64, 6, 2, 300, 0.5, 2, 2, 1)),
                            LayerSpec(delta(4, 4, 32, 48), tobadra_moe(20, 19, 3, 20, 1.4, 5, 12, 3)), LayerSpec(attn(30), dense(96), weights_of=1),
                            LayerSpec(LightningSpec(4, 32, 24, (0.6, 0.9, 0.98, 0.999)), tobadra_moe(64, 6, 2, 300, 0.5, 2, 2, 1), weights_of=2)],
                  norm_eps=1e-3, logit_scale=2.5, vocab=131, canon=5),
    # wide heads, many of them on one key head, no expert but the input chosen most of the time: the largest tiles
    "wide": _cfg("wide", [LayerSpec(attn(70, 20, 1, 128, 128, 0.09, 128), tobadra_moe(192, 2, 2, 192, 1.0, 6, 4, 3)), LayerSpec(delta(2, 1, 128, 128, 4, (64, 64))),
                          LayerSpec(LightningSpec(2, 128, 256, (0.9, 0.99)), dense(320)), LayerSpec(attn(47, 4, 2, 256, 64, 0.06, 64)),
                          LayerSpec(delta(1, 1, 256, 48, 3, (16, 16)))], hidden=192),
}


def random_weights(cfg, seed=0):
    """Checkpoint tensors under which every mechanism moves the logits: uneven attention, biases, decays from slow to fast, gates away
    from one half, routers without close calls, branches that count without drowning the stream."""
    from tilerl_b200.tobadra_layout import tensor_shapes
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        leaf = name.split(".")[-1]
        t = torch.randn(shape, generator=g)
        if leaf in ("norm1b", "norm2b"):
            t = 0.4 + 0.1 * t
        elif leaf.startswith("norm"):
            t = 1.0 + 0.25 * t
        elif leaf == "A_log":
            t = t
        elif leaf == "dt_bias":
            t = 2.0 * t - 3.0                              # some channels remember for long, some forget at once
        elif leaf == "correction":
            t = 0.1 * t
        elif leaf == "b" and len(shape) == 1:
            t = 0.5 * t
        elif leaf in ("conv", "canon1"):
            t = 0.5 * t
        elif leaf == "embed":
            t = 1.2 * t
        else:
            t = t * (1.3 / shape[-1] ** 0.5)
        out[name] = t
    _clear_choices(cfg, out, g)
    return {n: t.to(torch.bfloat16).float() for n, t in out.items()}      # representable in every compute dtype


def _clear_choices(cfg, w, g, share=0.05, margin=0.025):
    """Routers without close calls, which rounding would turn round: a few columns of the stream that no branch writes to (their norm
    weights are zero) carry what mostly decides.  They are drawn for every token until its choice stays the same, and clear, whatever
    the size of the rest of the row."""
    moe = [(i, cfg.layers[i].mlp) for i in cfg.owners if isinstance(cfg.layers[i].mlp, MoeSpec)]
    if not moe:
        return
    r = 8
    for i in cfg.owners:
        for n in (f"l{i}.norm1b", f"l{i}.norm2b"):
            if n in w:
                w[n][-r:] = 0.0
    for i, m in moe:
        t = w[f"l{i}.mlp.router"]
        t[:, :-r] *= share
        t[:, -r:] = torch.randn(t.shape[0], r, generator=g) * 1.5 / r ** 0.5
    open_ = torch.arange(cfg.vocab)
    for _ in range(20000):
        w["embed"][open_, -r:] = 1.2 * torch.randn(len(open_), r, generator=g)
        x = w["embed"][open_]
        x = x / x.pow(2).mean(1, keepdim=True).sqrt() * w["embed.norm"]
        clear = torch.ones(len(open_), dtype=torch.bool)
        for i, m in moe:
            first = None
            for size in (0.9, 1.2, 1.6, 2.1):
                h = (x / size * w[f"l{i}.norm2"])[:, -r:]
                s = torch.softmax(h @ w[f"l{i}.mlp.router"][:, -r:].T, 1) + w[f"l{i}.mlp.correction"]
                q = m.router
                best = s.view(len(x), q.groups, -1).amax(2).sort(dim=1, descending=True)
                if q.keep < q.groups:
                    clear &= best.values[:, q.keep - 1] - best.values[:, q.keep] > margin
                kept = torch.zeros(len(x), q.groups, dtype=torch.bool).scatter_(1, best.indices[:, :q.keep], True)
                c = s.masked_fill(~kept.repeat_interleave(m.outputs // q.groups, 1), -1e9).sort(dim=1, descending=True)
                if m.top < m.outputs:
                    clear &= c.values[:, m.top - 1] - c.values[:, m.top] > margin
                now = c.indices[:, :m.top].sort(dim=1).values
                clear &= (now == (now if first is None else first)).all(1)
                first = now if first is None else first
        open_ = open_[~clear]
        if not len(open_):
            return
    raise AssertionError("no clear choice found")


def build(cfg, weights, backend, *, max_tokens=1024, slots=4, graph=True, **kw):
    from tilerl_b200.factory import build_engine, make_ops
    from tilerl_b200.models.tobadra import TobadraModel
    device, dtype, _ = BACKENDS[backend]
    model = TobadraModel.from_tensors(cfg, weights.__getitem__, device, dtype)
    return build_engine(model, make_ops(device), device=device, blocks=max_tokens // 16 + 1, slots=slots, max_ctx=max_tokens,
                        graph=graph, prefix=kw.pop("prefix", False), **kw)


def want_logits(cfg, weights, toks):
    return oracle.forward(cfg.to_json(), weights, toks)[0].float()


def needle_model(window, heads=4, kv_heads=2, dim=32, vdim=40, score=25.0):
    """One attention layer in which token 1 asks for token 2: that score stands far above every other, so the logits of a 1 show
    whether a 2 is among the keys it sees.  Only dimensions that do not turn ask."""
    cfg = _cfg("needle", [LayerSpec(tobadra_attention(heads, kv_heads, dim, vdim, 1.0, window, 8))], hidden=96)
    w = random_weights(cfg, seed=11)
    for n in ("embed.norm", "l0.norm1"):
        w[n] = torch.ones_like(w[n])
    w["l0.norm1b"] = torch.ones_like(w["l0.norm1b"])
    w["l0.canon1"] *= 0.02
    h = w["embed"] / w["embed"].pow(2).mean(1, keepdim=True).sqrt()
    e1, e2 = h[1] / h[1].norm(), h[2] / h[2].norm()
    e1 = e1 - (e1 @ e2) * e2
    e1 = e1 / e1.norm()
    q, k = w["l0.mix.q"].view(heads, dim, -1), w["l0.mix.k"].view(kv_heads, dim, -1)
    q *= 0.05
    k *= 0.3
    w["l0.mix.q.b"] *= 0.1
    g = torch.Generator().manual_seed(5)
    for i in range(kv_heads):
        mark = torch.randn(dim - 8, generator=g)
        mark = mark / mark.norm()
        k[i, 8:] += torch.outer(mark, e2)
        for j in range(i * heads // kv_heads, (i + 1) * heads // kv_heads):
            q[j, 8:] += score / 96.0 * torch.outer(mark, e1)
    return cfg, {n: t.to(torch.bfloat16).float() for n, t in w.items()}
