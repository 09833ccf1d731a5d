"""Fetotar beside the hybrid model at equal size: throughput of whole models and the kernels of a layer against their
rooflines.

    python bench.py --design fetotar [--only throughput|kernels]

The closest existing model is the hybrid with Gated-DeltaNet and attention layers (two to one, as the recurrent and the
attention layers here): same width, depth, vocabulary, head size of the recurrent layers and feed-forward width.  Both have
random-init weights and run in the format each is served in (bf16 weights here, NVFP4 there); single kernels of both are
timed on bf16 weights, with the L2 flushed before each, as a fraction of the measured copy bandwidth or bf16 GEMM rate.
"""
from __future__ import annotations

import argparse
import json
import statistics

import torch

from .zinutar import throughput

SIZES = {     # hidden, recurrent / latent heads, ff, query latent, repeats of (mLSTM, attention, Mamba-2), window
    "2048": (2048, 16, 6144, 768, 4, 1024),
    "4096": (4096, 32, 9728, 1536, 3, 1024),
}
VOCAB = 32768


def configs(size: str):
    from ..config import ATTN, GDN, ModelConfig, fetotar_uniform
    h, heads, ff, qr, rep, window = SIZES[size]
    f = fetotar_uniform(f"fetotar-{size}", hidden=h, vocab=VOCAB, ff=ff, heads=heads, repeats=rep, window=window, q_rank=qr)
    m = ModelConfig(name=f"hybrid-{size}", hidden=h, ffn=ff, vocab=VOCAB, layer_types=(GDN, ATTN, GDN) * rep, n_q_heads=h // 256,
                    n_kv_heads=max(1, h // 1024), head_dim=256, rotary_dim=64, rope_theta=1e6, attn_gated=True, gdn_k_heads=heads // 2,
                    gdn_v_heads=heads, gdn_head_dim=128, quant="nvfp4")
    return {"fetotar": f, "hybrid": m}


def kernels(size: str, reps: int, hbm_gbs: float, tflops: float):
    """Kernels of one layer of both designs at the same shapes."""
    from dataclasses import replace

    from ..batch import Batch
    from ..config import ATTN, GDN
    from ..factory import build_model, make_ops
    from ..fetotar_layout import pad
    from ..kv import make_kv_pool, make_state_pool
    cf, ch = configs(size)["fetotar"], configs(size)["hybrid"]
    cf = replace(cf, layers=cf.layers[:3])
    h, heads, ff, _, _, window = SIZES[size]
    ops, dev = make_ops("cuda"), "cuda"
    model = build_model(cf, dev, seed=0, ops=ops)
    lm, la, lb = model.layouts
    P, eps, rot = model.params, cf.norm_eps, cf.layers[1].mixer.rot
    bf = lambda *s: (torch.randn(*s, device=dev) * 0.5).to(torch.bfloat16)
    flush = torch.empty(1 << 28, dtype=torch.uint8, device=dev)
    rows = []

    def time_us(fn) -> float:
        out = []
        for i in range(3 + reps):
            flush.fill_(i & 1)
            a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            a.record()
            fn()
            b.record()
            torch.cuda.synchronize()
            if i >= 3:
                out.append(a.elapsed_time(b) * 1e3)
        return statistics.median(out)

    def row(what, design, fn, nbytes, flops=0.0):
        us = time_us(fn)
        mem, tc = nbytes / hbm_gbs * 1e-3, flops / tflops * 1e-6
        rows.append({"what": what, "design": design, "us": round(us, 2), "bound": "memory" if mem >= tc else "tensor",
                     "of_measured": round(max(mem, tc) / us, 4)})

    # ---- projections
    norm = torch.ones(h, device=dev)
    n_in, wp = lm.n_in, 2 * pad(ff, 64)
    w_in, w_gu, w_dn = P["L0.in"], P["L0.gate_up"], P["L0.down"]
    for m in (1, 8, 2048):
        hb, x, a, y = bf(m, h), torch.randn(m, h, device=dev), bf(m, pad(ff, 64)), torch.randn(m, h, device=dev)
        row(f"in projection {m} rows", "fetotar", lambda: ops.project_gates(hb, w_in, n_in), w_in.numel() * 2 + m * (h + n_in) * 2, 2.0 * m * w_in.numel())
        row(f"in projection {m} rows", "hybrid", lambda: ops.norm_linear(hb, norm, w_in[:n_in], eps), w_in.numel() * 2 + m * (h + n_in) * 2, 2.0 * m * w_in.numel())
        row(f"gate / up {m} rows", "fetotar", lambda: ops.clamped_glu(hb, w_gu, 7.0), w_gu.numel() * 2 + m * (h + wp // 2) * 2, 2.0 * m * w_gu.numel())
        row(f"gate / up {m} rows", "hybrid", lambda: ops.norm_linear(hb, norm, w_gu, eps), w_gu.numel() * 2 + m * (h + wp) * 2, 2.0 * m * w_gu.numel())
        row(f"down {m} rows", "fetotar", lambda: ops.project_f32(a, w_dn), w_dn.numel() * 2 + m * (a.shape[1] * 2 + h * 4), 2.0 * m * w_dn.numel())
        row(f"down {m} rows", "hybrid", lambda: ops.linear_residual(a, w_dn, hb), w_dn.numel() * 2 + m * (a.shape[1] * 2 + h * 4), 2.0 * m * w_dn.numel())
        ops._join_dtype = torch.bfloat16
        row(f"elementwise {m} rows: join", "fetotar", lambda: ops.join(x, y, P["L0.norm1b"], P["L0.norm2"], eps, h), m * h * (4 + 8 + 2))
        row(f"elementwise {m} rows: norm", "hybrid", lambda: ops._rmsnorm(hb, norm, eps), m * h * 4)
    # ---- mixers
    gd = ch.gdn_head_dim
    glp = {"conv": torch.randn(ch.gdn_conv_dim, 4, device=dev), "dt_bias": torch.zeros(heads, device=dev), "a_log": torch.zeros(heads, device=dev),
           "gdn_norm": torch.ones(gd, device=dev)}
    alp = {"q_norm": torch.ones(256, device=dev), "k_norm": torch.ones(256, device=dev)}
    nq, nkv = ch.n_q_heads, ch.n_kv_heads
    for b, n, ctx in ((1, 1, 4096), (16, 1, 4096), (64, 1, 4096), (1, 2048, 2048), (1, 8192, 8192), (4, 2048, 4096)):
        per = ctx // 16 + 2
        seqs = [dict(tokens=[1] * n, start=ctx - n, blocks=list(range(1 + i * per, 1 + (i + 1) * per)), slot=i + 1) for i in range(b)]
        batch, t = Batch.build(seqs, dev), b * n
        what = f"{b} x {n} at {ctx}"
        pool = make_state_pool(cf, b + 1, dev)
        gpool = make_state_pool(replace(ch, layer_types=(GDN,)), b + 1, dev)
        for l, i, p in ((lm, 0, "L0."), (lb, 1, "L2.")):
            proj, gates = bf(t, l.n_in), torch.randn(t, pad(l.n_gates, 8), device=dev)
            w = {k: P.get(p + k) for k in ("norm", "gate_b", "conv", "conv_b", "a_log", "skip")}
            # state read and written, projected rows read, output written
            by = b * l.state_floats * 8 + t * (l.n_in * 2 + l.n_out * 2)
            row(f"recurrent mixer {what}", f"fetotar {l.kind}", lambda: ops.recurrent_mix(proj, gates, w, l, batch, pool, i, eps), by,
                4.0 * t * l.heads * l.dk * l.dv)
        inp = bf(t, ch.gdn_in_rows)
        row(f"recurrent mixer {what}", "hybrid gdn", lambda: ops.gdn(inp, glp, batch, gpool, 0, ch, heads // 2, heads),
            b * heads * gd * gd * 8 + t * (ch.gdn_in_rows * 2 + heads * gd * 2), 6.0 * t * heads * gd * gd)
        kv = make_kv_pool(replace(cf, layers=cf.layers[1:2]), b * per + 1, dev)
        kv.k.view(torch.bfloat16).normal_()
        proj, q = bf(t, la.n_in), bf(t, la.heads, la.dq)
        seen = b * sum(min(p + 1, window) for p in range(ctx - n, ctx))
        keys = b * min(ctx, n + window - 1)
        # cached rows and the maps read once, queries and gates read, output written; scores and sums over expanded heads
        by = keys * la.row * 2 + P["L1.up"].numel() * 2 + t * la.heads * (la.dq + 2 * la.dv) * 2
        fl = 2.0 * seen * la.heads * (la.dq + la.dv) + 2.0 * t * P["L1.up"].numel()
        row(f"attention {what}", "fetotar", lambda: ops.latent_attention(q, proj, P["L1.up"], model.ukt[1], la, model.freqs[1], rot, batch, kv, 0), by, fl)
        pa = make_kv_pool(replace(ch, layer_types=(ATTN,)), b * per + 1, dev)
        pa.k.normal_(), pa.v.normal_()
        qkv = bf(t, ch.qkv_rows)
        pairs = b * sum(range(ctx - n + 1, ctx + 1))
        row(f"attention {what}", "hybrid", lambda: ops.attention(qkv, alp, batch, pa, 0, ch, nq, nkv),
            b * ctx * nkv * 256 * 4 + t * nq * 256 * 6, 4.0 * pairs * nq * 256)
        del kv, pa, pool, gpool
    return rows


def main(argv=None):
    ap = argparse.ArgumentParser(prog="tilerl_b200.suites.fetotar")
    ap.add_argument("--sizes", default="2048,4096")
    ap.add_argument("--only", default=None, choices=["throughput", "kernels"])
    ap.add_argument("--reps", type=int, default=7)
    ap.add_argument("--ticks", type=int, default=32)
    args = ap.parse_args(argv)
    from ..calibration import load_peaks
    pk = load_peaks()
    out = {"suite": "fetotar", "dtype": "fetotar bf16 weights, hybrid NVFP4 weights, bf16 KV", "data": "synthetic (random-init weights, random tokens)",
           "peaks": {"hbm_gbs": pk.hbm_gbs, "bf16_tflops": pk.bf16_tflops}, "throughput": [], "kernels": {}}
    for size in args.sizes.split(","):
        if args.only != "kernels":
            for cfg in configs(size).values():
                out["throughput"] += throughput(cfg, (512, 2048, 8192), ((1, 2048), (8, 2048), (16, 2048), (64, 2048)), args.ticks, args.reps)
                torch.cuda.empty_cache()
        if args.only != "throughput":
            out["kernels"][size] = kernels(size, args.reps, pk.hbm_gbs, pk.bf16_tflops)
            torch.cuda.empty_cache()
    print(json.dumps(out))
