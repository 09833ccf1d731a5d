"""Tobadra beside the hybrid model at equal size: throughput of whole models and the kernels of a layer against their rooflines.

    python bench.py --design tobadra [--only throughput|kernels]

The closest existing model is the hybrid with three Gated-DeltaNet layers (for two per-channel delta layers and a lightning layer) per
attention layer: same width, depth, vocabulary, query and key / value widths, and as many feed-forward weights per token (chosen
experts and the shared one).  Both have random-init weights and run in the format each is served in (bf16 weights here, NVFP4 there);
single kernels of both are timed on bf16 weights, with the L2 flushed before each, as a fraction of the measured copy bandwidth or
bf16 GEMM rate.
"""
from __future__ import annotations

import argparse
import json
from dataclasses import replace

import torch

from .deluvik import Rows
from .zinutar import throughput

SIZES = {     # hidden, heads, kv heads (of 128), dense ff = (top + 1) expert ff, expert ff, experts, identity, top, repeats of four layers, window
    "2048": (2048, 16, 4, 6144, 1024, 32, 8, 5, 3, 1024),
    "4096": (4096, 32, 8, 9216, 1536, 32, 8, 5, 2, 1024),
}
VOCAB = 32768


def configs(size: str):
    from ..config import ATTN, GDN, ModelConfig, tobadra_uniform
    h, heads, kvh, ff, eff, n_exp, own, top, rep, window = SIZES[size]
    t = tobadra_uniform(f"tobadra-{size}", hidden=h, vocab=VOCAB, ff=ff, expert_ff=eff, experts=n_exp, top=top, heads=heads, kv_heads=kvh,
                        repeats=rep, window=window, identity=own, groups=4, keep=2)
    m = ModelConfig(name=f"hybrid-{size}", hidden=h, ffn=ff * 2 // 3, vocab=VOCAB, layer_types=(GDN, GDN, ATTN, GDN) * rep, n_q_heads=heads // 2,
                    n_kv_heads=kvh // 2, head_dim=256, rotary_dim=64, rope_theta=1e6, attn_gated=False, gdn_k_heads=heads,
                    gdn_v_heads=heads, gdn_head_dim=128, quant="nvfp4")
    return {"tobadra": t, "hybrid": m}


def kernels(size: str, reps: int, hbm_gbs: float, tflops: float):
    """Kernels of one layer of both designs at the same shapes."""
    from ..batch import Batch
    from ..config import ATTN, GDN
    from ..factory import build_model, make_ops
    from ..kv import make_kv_pool, make_state_pool
    from ..ops import native as N
    from ..tobadra_layout import gate_rows, router_rows
    ct, ch = configs(size)["tobadra"], configs(size)["hybrid"]
    ct = replace(ct, layers=ct.layers[:4])
    h, heads, kvh, ff, eff, n_exp, own, top, _, window = SIZES[size]
    ops, dev = make_ops("cuda"), "cuda"
    model = build_model(ct, dev, seed=0, ops=ops)
    P, eps, moe = model.params, ct.norm_eps, model.moe[1]
    bf = lambda *s: (torch.randn(*s, device=dev) * 0.5).to(torch.bfloat16)
    r = Rows(reps, hbm_gbs, tflops)
    norm = torch.ones(h, device=dev)
    ops._join_dtype = torch.bfloat16
    D, L, A = (model.layouts[i] for i in (0, 1, 2))

    # ---- projections, feed-forwards, joins
    w_in, w_up, w_dn, w_r = P["L1.in"], P["L0.up"], P["L0.down"], P["L1.router"]
    w_gu = bf(2 * ch.ffn, h)
    w_hd = bf(h, ch.ffn)
    pool0 = make_state_pool(ct, 65, dev)
    for m in (1, 8, 64, 2048, 8192):
        hb, x, a, y, z = bf(m, h), torch.randn(m, h, device=dev), bf(m, ff), torch.randn(m, h, device=dev), torch.randn(m, h, device=dev)
        n_in = w_in.shape[0]
        if m != 64:
            by, fl = n_in * h * 2 + m * (2 * h + n_in + h) * 2, 2.0 * m * n_in * h
            r.add(f"in projection and branch gate {m} rows", "tobadra", lambda: ops.project_in(hb, hb, w_in, L.n_in, 0, L.g0, "silu"), by, fl)
            r.add(f"in projection {m} rows", "hybrid", lambda: ops.norm_linear(hb, norm, w_in, eps), by, fl)
            by, fl = w_up.numel() * 2 + m * (h + ff + 2 * h) * 2, 2.0 * m * w_up.numel()
            r.add(f"up, activation and branch gate {m} rows", "tobadra", lambda: ops.up_act(hb, w_up, ff, "gelu"), by, fl)
            r.add(f"gate / up {m} rows (without activation)", "hybrid", lambda: ops.norm_linear(hb, norm, w_gu, eps), w_gu.numel() * 2 + m * (h + 2 * ch.ffn) * 2,
                  2.0 * m * w_gu.numel())
            by, fl = w_dn.numel() * 2 + m * (ff * 2 + h * 4), 2.0 * m * w_dn.numel()
            r.add(f"down {m} rows", "tobadra", lambda: ops.project_f32(a, w_dn), by, fl)
            ah = bf(m, ch.ffn)
            r.add(f"down {m} rows", "hybrid", lambda: ops.linear_residual(ah, w_hd, hb), w_hd.numel() * 2 + m * (ch.ffn + 2 * h) * 2, 2.0 * m * w_hd.numel())
        # the experts this input really uses: their weights once, input, middle and output rows once
        zr = ops.project_f32(hb, w_r, "router").clone()
        branch = ops.routed_experts(hb, zr, P["L1.correction"], P["L1.up"], P["L1.down"], moe)
        place = branch[1].view(m, moe.slots)
        pairs = int((place >= 0).sum())
        s = torch.softmax(zr[:, :moe.spec.outputs], 1).view(m, 4, -1)
        best = s.amax(2).topk(2, 1).indices
        kept = torch.zeros(m, 4, dtype=torch.bool, device=dev).scatter_(1, best, True)
        chosen = s.masked_fill(~kept[:, :, None], -1).view(m, -1).topk(top, 1).indices
        used = int(chosen[chosen < n_exp].unique().numel()) + moe.pieces
        per = 2 * moe.ff * h
        by, fl = used * per * 2 + w_r.numel() * 2 + m * h * 2 + pairs * (moe.ff * 2 + h * 2), 2.0 * (pairs * per + m * w_r.numel())

        def experts():
            zz = ops.project_f32(hb, w_r, "router")
            return ops.routed_experts(hb, zz, P["L1.correction"], P["L1.up"], P["L1.down"], moe)
        r.add(f"experts {m} rows (router and branch gate to weighted rows)", "tobadra", experts, by, fl)
        ah = bf(m, ch.ffn)
        r.add(f"experts {m} rows: dense gate / up and down (without activation)", "hybrid",
              lambda: (ops.norm_linear(hb, norm, w_gu, eps), ops.linear_residual(ah, w_hd, hb)), (w_gu.numel() + w_hd.numel()) * 2 + m * (2 * h + 3 * ch.ffn) * 2,
              2.0 * m * (w_gu.numel() + w_hd.numel()))
        n = min(m, 64)
        lens = [m // n] * n if m <= 64 else [m]
        batch = Batch.build([dict(tokens=[1] * k, start=64, blocks=list(range(1, 3 + (64 + k) // 16)), slot=i + 1) for i, k in enumerate(lens)], dev)
        conv = (P["L1.canon"], batch, pool0, 1)
        bias = torch.zeros(h, device=dev)
        r.add(f"join {m} rows", "tobadra", lambda: ops.gated_join(x, y, None, z, bias, P["L1.norm1b"], P["L1.norm2"], eps, h, None), m * h * (4 + 4 + 8 + 2))
        r.add(f"join and input convolution {m} rows", "tobadra", lambda: ops.gated_join(x, y, None, z, bias, P["L1.norm1b"], P["L1.norm2"], eps, h, conv),
              m * h * (4 + 4 + 8 + 4))
        r.add(f"join of experts and input convolution {m} rows", "tobadra",
              lambda: ops.gated_join_experts(x, branch, hb, z, bias, P["L1.norm2b"], P["L1.norm1"], eps, h, conv),
              pairs * h * branch[0].element_size() + m * h * (2 + 4 + 8 + 4))
        r.add(f"join {m} rows: norm", "hybrid", lambda: ops._rmsnorm(hb, norm, eps), m * h * 4)

    # ---- mixers
    gd = ch.gdn_head_dim
    glp = {"conv": torch.randn(ch.gdn_conv_dim, 4, device=dev), "dt_bias": torch.zeros(heads, device=dev), "a_log": torch.zeros(heads, device=dev),
           "gdn_norm": torch.ones(gd, device=dev)}
    alp = {"q_norm": torch.ones(256, device=dev), "k_norm": torch.ones(256, device=dev)}
    nq, nkv = ch.n_q_heads, ch.n_kv_heads
    dw = {k: P["L0." + k] for k in ("conv", "low", "dt_bias", "a_log")}
    for b, n, ctx in ((1, 1, 1024), (16, 1, 1024), (64, 1, 1024), (64, 1, 4096), (1, 512, 512), (1, 2048, 2048), (1, 8192, 8192), (4, 2048, 4096)):
        pages = ctx // 16 + 2
        seqs = [dict(tokens=[1] * n, start=ctx - n, blocks=list(range(1 + i * pages, 1 + (i + 1) * pages)), slot=i + 1) for i in range(b)]
        batch, t = Batch.build(seqs, dev), b * n
        what = f"{b} x {n} at {ctx}"
        pool, gpool = make_state_pool(ct, b + 1, dev), make_state_pool(replace(ch, layer_types=(GDN,)), b + 1, dev)
        kv = make_kv_pool(ct, b * pages + 1, dev)
        kv.k.view(torch.bfloat16).normal_()
        al, s = A.attn, A.attn.spec
        proj, kv_cols = bf(t, A.n_in), s.kv_heads * (al.dk + al.dv)
        prep = lambda: ops.turned_prep(proj, A, P["L2.qkv_b"], model.freqs[2], model.value_freqs[2], batch, kv, 0)
        r.add(f"preparation {what}", "tobadra", prep, t * (al.n_in + al.k0 + kv_cols) * 2)
        q, mid, turn = prep()
        seen = b * sum(min(p + 1, window) for p in range(ctx - n, ctx))
        keys = b * min(ctx, n + window - 1)
        r.add(f"attention {what}: window, turned", "tobadra", lambda: ops.softmax_attention(q, mid, al, None, 1.0, batch, kv, 0, turn),
              keys * kv_cols * 2 + t * s.heads * (al.dk + al.dv) * 2, 2.0 * seen * s.heads * (al.dk + al.dv))
        state = b * heads * gd * gd * 8
        lp = bf(t, L.n_in)
        r.add(f"recurrent mixer {what}: lightning", "tobadra", lambda: ops.lightning_mix(lp, model.log_decay[1], model.head_norm[1], L, batch, pool, model.states[1], eps),
              state + t * (L.n_in * 2 + heads * gd * 2), 4.0 * t * heads * gd * gd)
        dp, gates = bf(t, D.n_in), torch.randn(t, gate_rows(D), device=dev)
        low = dw["low"]
        r.add(f"recurrent mixer {what}: delta (with its low-rank maps)", "tobadra",
              lambda: ops.delta_mix(dp, gates, dw, model.head_norm[0], D, batch, pool, model.states[0], eps),
              state + low.numel() * 2 + t * (D.n_in * 2 + heads * gd * 2), 6.0 * t * heads * gd * gd + 2.0 * t * low.numel())
        inp = bf(t, ch.gdn_in_rows)
        r.add(f"recurrent mixer {what}: gdn", "hybrid", lambda: ops.gdn(inp, glp, batch, gpool, 0, ch, heads, heads),
              state + t * (ch.gdn_in_rows * 2 + heads * gd * 2), 6.0 * t * heads * gd * gd)
        pa = make_kv_pool(replace(ch, layer_types=(ATTN,)), b * pages + 1, dev)
        pa.k.normal_(), pa.v.normal_()
        qkv = bf(t, ch.qkv_rows)
        qb, (kc, vc) = bf(t, nq * 256), pa.layer(0)

        def hprep():
            N.check(ops.lib.trl_attn_prep(qkv.data_ptr(), qkv.stride(0), alp["q_norm"].data_ptr(), alp["k_norm"].data_ptr(), batch.positions.data_ptr(),
                                          batch.slot_mapping.data_ptr(), qb.data_ptr(), kc.data_ptr(), vc.data_ptr(), t, nq, nkv, 256, ch.rotary_dim,
                                          ch.rope_theta, eps, 0, kc.shape[0], N.stream()))
        r.add(f"preparation {what}", "hybrid", hprep, t * (2 * ch.qkv_rows) * 2)
        pairs = b * sum(range(ctx - n + 1, ctx + 1))
        r.add(f"attention {what}: with preparation", "hybrid", lambda: ops.attention(qkv, alp, batch, pa, 0, ch, nq, nkv),
              b * ctx * nkv * 256 * 4 + t * nq * 256 * 6, 4.0 * pairs * nq * 256)
        del kv, pa, pool, gpool
    return r.rows


def main(argv=None):
    ap = argparse.ArgumentParser(prog="tilerl_b200.suites.tobadra")
    ap.add_argument("--sizes", default="2048,4096")
    ap.add_argument("--only", default=None, choices=["throughput", "kernels"])
    ap.add_argument("--reps", type=int, default=7)
    ap.add_argument("--ticks", type=int, default=32)
    args = ap.parse_args(argv)
    from ..calibration import load_peaks
    pk = load_peaks()
    out = {"suite": "tobadra", "dtype": "tobadra bf16 weights, hybrid NVFP4 weights, bf16 KV", "data": "synthetic (random-init weights, random tokens)",
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
