"""Models and helpers of the Fetotar tests."""
import torch

import fetotar_oracle as oracle
from tilerl_b200.config import FetotarConfig, fetotar_tiny
from tilerl_b200.mixers import ClampedGluSpec, LatentAttnSpec, LayerSpec, Mamba2Spec, MlstmSpec, RotarySpec, YarnSpec
from zinutar_cases import BACKENDS, backends, feed_all, rel_err, tokens  # noqa: F401

TOL = {"cpu": 5e-4, "cuda-f32": 5e-4, "cuda-bf16": 6e-2}      # relative error of a position (rms over the vocabulary)


def close(got, want, backend):
    """Every position within the tolerance; in bf16 nine of ten, and none far off: a branch that comes out near zero is
    normalised up again with its rounding."""
    got, want = got.detach().float().cpu(), want.float()
    d, w = got - want, want - want.mean(-1, keepdim=True)
    e = ((d - d.mean(-1, keepdim=True)).pow(2).mean(-1) / w.pow(2).mean()).sqrt()
    e = torch.nan_to_num(e, nan=float("inf")).sort().values
    if "bf16" not in backend:
        return bool(e[-1] < TOL[backend])
    return bool(e[-1] < 16 * TOL[backend] and (len(e) < 10 or e[int(0.9 * (len(e) - 1))] < TOL[backend]))


def rot(dims, base=1000.0, scaled=True):
    return RotarySpec(dims, base, YarnSpec(3.0, 48.0, 6.0, 0.5) if scaled else None)


def attn(heads=3, dim=20, rot_dim=12, vdim=24, q_rank=30, kv_rank=28, window=19, scale=0.3, **kw):
    return LatentAttnSpec(heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, window, rot(rot_dim, **kw))


def _cfg(name, layers, **kw):
    base = dict(hidden=56, vocab=90, side_dim=12, embed_scale=0.8, norm_eps=1e-5, max_ctx=4096)
    return FetotarConfig(name=name, layers=tuple(layers), **{**base, **kw})


CONFIGS = {
    "tiny": fetotar_tiny(),
    # one mixer each, without and with a feed-forward; every size its own
    "attention": _cfg("attention", [LayerSpec(attn(), ClampedGluSpec(70, 0.9)), LayerSpec(attn(1, 16, 2, 40, 16, 64, 33, 0.5, scaled=False))]),
    "mamba2": _cfg("mamba2", [LayerSpec(Mamba2Spec(4, 12, 20, 2, 3, 3)), LayerSpec(Mamba2Spec(3, 40, 72, 1, 5, 1), ClampedGluSpec(48, 4.0)),
                              LayerSpec(Mamba2Spec(2, 24, 8, 2, 1, 4))], hidden=70, side_dim=7),
    "mlstm": _cfg("mlstm", [LayerSpec(MlstmSpec(2, 40, 72, 6.0), ClampedGluSpec(33, 2.5)), LayerSpec(MlstmSpec(5, 8, 12, 20.0))], embed_scale=1.0),
    # the order of layers turned round, norms with a large eps, a window of one and one wider than any sequence
    "mixed": _cfg("mixed", [LayerSpec(attn(2, 32, 16, 16, 64, 48, 1)), LayerSpec(MlstmSpec(3, 16, 16, 9.0)), LayerSpec(Mamba2Spec(6, 16, 16, 3, 4, 2), ClampedGluSpec(64, 1.2)),
                            LayerSpec(attn(4, 24, 8, 20, 24, 40, 5000), ClampedGluSpec(40, 3.0))], norm_eps=1e-3, vocab=131),
    # wide heads and latents: the largest tiles
    "wide": _cfg("wide", [LayerSpec(MlstmSpec(2, 128, 128, 15.0)), LayerSpec(attn(6, 128, 64, 128, 192, 512, 70, 0.07), ClampedGluSpec(160, 7.0)),
                          LayerSpec(Mamba2Spec(4, 64, 128, 2, 4, 1)), LayerSpec(MlstmSpec(1, 240, 200, 15.0))], hidden=192, side_dim=64),
}


def random_weights(cfg, seed=0):
    """Checkpoint tensors under which every mechanism moves the logits: decays from slow to fast, gates on both sides of
    their caps, biases away from zero."""
    from tilerl_b200.fetotar_layout import tensor_shapes
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        leaf = name.split(".")[-1]
        t = torch.randn(shape, generator=g)
        if name.endswith(".f.b"):
            t = 3.0 + 3.0 * t                              # some heads remember for long, some forget at once
        elif name.endswith(".i.b"):
            t = 2.0 * t
        elif name.endswith(("norm1b", "norm2b", "side.norm")):
            t = 0.4 + 0.1 * t                              # a branch counts, and does not drown the stream
        elif leaf == "b":
            t = 0.15 * t                                   # norm and convolution biases
        elif "norm" in leaf or leaf == "D":
            t = 1.0 + 0.3 * t
        elif leaf == "A_log":
            t = 1.5 * t - 1.0
        elif leaf == "dt_bias":
            t = t - 1.0
        elif leaf == "conv":
            t = 0.6 * t
        elif leaf in ("gate", "up") and "mlp" in name:
            t = t * (2.0 / shape[-1] ** 0.5)               # reaches the clamps
        elif leaf == "uq":
            t = t * (2.0 / shape[-1] ** 0.5)               # uneven attention
        else:
            t = t * (1.3 / shape[-1] ** 0.5)
        out[name] = t.to(torch.bfloat16).float()           # representable in every compute dtype
    return out


def build(cfg, weights, backend, *, max_tokens=1024, slots=4, graph=True, **kw):
    from tilerl_b200.factory import build_engine, make_ops
    from tilerl_b200.models.fetotar import FetotarModel
    device, dtype, _ = BACKENDS[backend]
    model = FetotarModel.from_tensors(cfg, weights.__getitem__, device, dtype)
    return build_engine(model, make_ops(device), device=device, blocks=max_tokens // 16 + 1, slots=slots, max_ctx=max_tokens,
                        graph=graph, prefix=kw.pop("prefix", False), **kw)


def want_logits(cfg, weights, toks):
    return oracle.forward(cfg.to_json(), weights, toks)[0].float()


def needle_model(window, heads=2, dim=32, rot_dim=16, vdim=32, kv_rank=48, turned=False):
    """One attention layer in which token 1 asks for token 2: that score stands far above every other, so the logits of a
    1 show whether a 2 is among the keys it sees.  ``turned``: the rotated part asks as well, for a key at the query's own
    place, without outweighing the other part."""
    cfg = _cfg("needle", [LayerSpec(LatentAttnSpec(heads, dim, rot_dim, vdim, 64, kv_rank, 1.0, window, rot(rot_dim)))], hidden=96)
    w = random_weights(cfg, seed=11)
    eps = cfg.norm_eps
    d = {k: t.double() for k, t in w.items()}
    h = oracle.layer_norm(oracle.embedding(cfg.to_json(), d, [1, 2]), d["l0.norm1"], d["l0.norm1.b"], eps)
    cq = oracle.unit_rms(h[0] @ d["l0.mix.dq"].T, eps) * d["l0.mix.dq.norm"]
    c = oracle.unit_rms(h[1] @ d["l0.mix.dkv"][:kv_rank].T, eps) * d["l0.mix.dkv.norm"]
    k2 = (d["l0.mix.uk"] @ c).view(heads, dim)
    uq = w["l0.mix.uq"].view(heads, dim + rot_dim, 64)
    uq *= 0.02
    for hd in range(heads):
        uq[hd, :dim] += (14.0 * torch.outer(k2[hd] / (k2[hd] @ k2[hd]), cq / (cq @ cq))).float()
        if not turned:
            uq[hd, dim:] = 0.0
    w = {k: t.to(torch.bfloat16).float() for k, t in w.items()}
    return cfg, w
