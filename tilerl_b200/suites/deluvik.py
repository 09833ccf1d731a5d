"""Deluvik beside the hybrid model at equal size: throughput of whole models and the kernels of a layer against their rooflines.

    python bench.py --design deluvik [--only throughput|kernels]

The closest existing model is the hybrid with one Gated-DeltaNet layer (for the linear recurrence) per three attention layers: same
width, depth, vocabulary, query and key / value widths, and as many feed-forward weights per token (top experts and the shared
one).  Both have random-init weights and run in the format each is served in (bf16 weights here, NVFP4 there); single kernels of both
are timed on bf16 weights, with the L2 flushed before each, as a fraction of the measured copy bandwidth or bf16 GEMM rate.
"""
from __future__ import annotations

import argparse
import json
import statistics
from dataclasses import replace

import torch

from .zinutar import throughput

SIZES = {     # hidden, heads, kv heads (of 128), dense ff = (top + 1) expert ff, expert ff, experts, top, repeats of four layers, window
    "2048": (2048, 16, 4, 5120, 1024, 32, 4, 3, 1024),
    "4096": (4096, 32, 8, 7680, 1536, 32, 4, 2, 1024),
}
VOCAB = 32768


def configs(size: str):
    from ..config import ATTN, GDN, ModelConfig, deluvik_uniform
    h, heads, kvh, ff, eff, n_exp, top, rep, window = SIZES[size]
    d = deluvik_uniform(f"deluvik-{size}", hidden=h, vocab=VOCAB, ff=ff, expert_ff=eff, experts=n_exp, top=top, heads=heads, kv_heads=kvh,
                        repeats=rep, window=window)
    m = ModelConfig(name=f"hybrid-{size}", hidden=h, ffn=ff, vocab=VOCAB, layer_types=(GDN, ATTN, ATTN, ATTN) * rep, n_q_heads=heads // 2,
                    n_kv_heads=kvh // 2, head_dim=256, rotary_dim=64, rope_theta=1e6, attn_gated=False, gdn_k_heads=heads // 2,
                    gdn_v_heads=heads, gdn_head_dim=128, quant="nvfp4")
    return {"deluvik": d, "hybrid": m}


class Rows:
    """Timed launches as fractions of their rooflines."""

    def __init__(self, reps: int, hbm_gbs: float, tflops: float):
        self.reps, self.hbm, self.tf, self.rows = reps, hbm_gbs, tflops, []
        self.flush = torch.empty(1 << 28, dtype=torch.uint8, device="cuda")

    def add(self, what: str, design: str, fn, nbytes: float, flops: float = 0.0) -> None:
        out = []
        for i in range(3 + self.reps):
            self.flush.fill_(i & 1)
            a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            a.record()
            fn()
            b.record()
            torch.cuda.synchronize()
            if i >= 3:
                out.append(a.elapsed_time(b) * 1e3)
        us = statistics.median(out)
        mem, tc = nbytes / self.hbm * 1e-3, flops / self.tf * 1e-6
        self.rows.append({"what": what, "design": design, "us": round(us, 2), "bound": "memory" if mem >= tc else "tensor",
                          "of_measured": round(max(mem, tc) / us, 4)})


def kernels(size: str, reps: int, hbm_gbs: float, tflops: float):
    """Kernels of one layer of both designs at the same shapes."""
    from ..batch import Batch
    from ..config import ATTN, GDN
    from ..factory import build_model, make_ops
    from ..kv import make_kv_pool, make_state_pool
    from ..ops import native as N
    cd, ch = configs(size)["deluvik"], configs(size)["hybrid"]
    cd = replace(cd, layers=cd.layers[:4])
    h, heads, kvh, ff, eff, n_exp, top, _, window = SIZES[size]
    ops, dev = make_ops("cuda"), "cuda"
    model = build_model(cd, dev, seed=0, ops=ops)
    P, eps, moe = model.params, cd.norm_eps, model.moe[1]
    bf = lambda *s: (torch.randn(*s, device=dev) * 0.5).to(torch.bfloat16)
    r = Rows(reps, hbm_gbs, tflops)
    norm = torch.ones(h, device=dev)
    ops._join_dtype = torch.bfloat16

    # ---- projections, feed-forwards, joins
    w_in, w_gu, w_dn, n_in = P["L1.in"], P["L3.gate_up"], P["L3.down"], P["L1.in"].shape[0]
    for m in (1, 8, 64, 2048, 8192):
        hb, x, a, y = bf(m, h), torch.randn(m, h, device=dev), bf(m, ff), torch.randn(m, h, device=dev)
        if m != 64:
            by, fl = n_in * h * 2 + m * (h + n_in) * 2, 2.0 * m * n_in * h
            r.add(f"in projection {m} rows", "deluvik", lambda: ops.project(hb, w_in), by, fl)
            r.add(f"in projection {m} rows", "hybrid", lambda: ops.norm_linear(hb, norm, w_in, eps), by, fl)
            by, fl = w_gu.numel() * 2 + m * (h + ff) * 2, 2.0 * m * w_gu.numel()
            r.add(f"dense gate / up {m} rows", "deluvik", lambda: ops.glu(hb, w_gu, "gelu"), by, fl)
            r.add(f"dense gate / up {m} rows (without activation)", "hybrid", lambda: ops.norm_linear(hb, norm, w_gu, eps), by + m * ff * 2, fl)
            by, fl = w_dn.numel() * 2 + m * (ff * 2 + h * 4), 2.0 * m * w_dn.numel()
            r.add(f"dense down {m} rows", "deluvik", lambda: ops.project_f32(a, w_dn), by, fl)
            r.add(f"dense down {m} rows", "hybrid", lambda: ops.linear_residual(a, w_dn, hb), by, fl)
        # the experts this input really uses: their weights once, input, gated and output rows once
        z = (hb.float() @ P["L1.router"][:n_exp].float().t())
        used = int(torch.topk(z, top, dim=1).indices.unique().numel()) + moe.pieces
        per = 2 * moe.ff * h + h * moe.ff
        by, fl = used * per * 2 + m * h * 2 + m * moe.slots * (moe.ff * 2 + h * 2), 2.0 * m * moe.slots * per
        r.add(f"experts {m} rows (router to weighted rows)", "deluvik", lambda: ops.experts(hb, P["L1.router"], P["L1.router_b"], P["L1.gate_up"], P["L1.down"], moe), by, fl)
        r.add(f"experts {m} rows: dense gate / up and down (without activation)", "hybrid",
              lambda: (ops.norm_linear(hb, norm, w_gu, eps), ops.linear_residual(a, w_dn, hb)), (w_gu.numel() + w_dn.numel()) * 2 + m * (2 * h + 3 * ff) * 2,
              2.0 * m * (w_gu.numel() + w_dn.numel()))
        branch = ops.experts(hb, P["L1.router"], P["L1.router_b"], P["L1.gate_up"], P["L1.down"], moe)
        r.add(f"join {m} rows", "deluvik", lambda: ops.join(x, y, P["L1.norm1"], None, eps, h), m * h * (4 + 8 + 2))
        r.add(f"join of experts {m} rows", "deluvik", lambda: ops.join_experts(x, branch, P["L1.norm2"], None, eps, h),
              m * h * (moe.slots * branch[0].element_size() + 8 + 2))
        r.add(f"join {m} rows: norm", "hybrid", lambda: ops._rmsnorm(hb, norm, eps), m * h * 4)
        if m >= 64:
            tile = ops.lib.trl_moe_tc_tile()
            plan, _, _ = ops._moe_plan(hb, P["L1.router"], P["L1.router_b"], moe, tile)
            pairs = m * moe.slots
            xs, mid, out = bf(pairs, h), bf(pairs, moe.ff), bf(pairs, h)
            for what, x_, w_, o_, kind in (("up", xs, P["L1.gate_up"], mid, 0), ("down", mid, P["L1.down"], out, 1)):
                def go():
                    N.check(ops.lib.trl_moe_tc(x_.data_ptr(), w_.data_ptr(), o_.data_ptr(), o_.stride(0), plan.items, plan.n_items, pairs, w_.shape[0],
                                               w_.shape[1], w_.shape[2], kind, 1, N.stream()))
                r.add(f"experts {m} rows: {what} product alone", "deluvik", go, used * w_.shape[1] * w_.shape[2] * 2 + (x_.numel() + o_.numel()) * 2,
                      2.0 * pairs * w_.shape[1] * w_.shape[2])

    # ---- mixers
    gd = ch.gdn_head_dim
    glp = {"conv": torch.randn(ch.gdn_conv_dim, 4, device=dev), "dt_bias": torch.zeros(heads, device=dev), "a_log": torch.zeros(heads, device=dev),
           "gdn_norm": torch.ones(gd, device=dev)}
    alp = {"q_norm": torch.ones(256, device=dev), "k_norm": torch.ones(256, device=dev)}
    nq, nkv = ch.n_q_heads, ch.n_kv_heads
    lp = model.layouts[0]
    lw = {k: P["L0." + k] for k in ("y_b", "x_b", "lru_conv", "lru_conv_b", "gates", "gates_b", "lam")}
    for b, n, ctx in ((1, 1, 4096), (16, 1, 4096), (64, 1, 4096), (1, 1, 32768), (1, 2048, 2048), (1, 8192, 8192), (4, 2048, 4096)):
        pages = ctx // 16 + 2
        seqs = [dict(tokens=[1] * n, start=ctx - n, blocks=list(range(1 + i * pages, 1 + (i + 1) * pages)), slot=i + 1) for i in range(b)]
        batch, t = Batch.build(seqs, dev), b * n
        what = f"{b} x {n} at {ctx}"
        pool, gpool = make_state_pool(cd, b + 1, dev), make_state_pool(replace(ch, layer_types=(GDN,)), b + 1, dev)
        kv = make_kv_pool(cd, b * pages + 1, dev)
        kv.k.view(torch.bfloat16).normal_()
        for i, name in ((0, "window"), (1, "convolution"), (3, "tied, cap, sink")):
            l, s = model.layouts[i], model.layouts[i].attn.spec
            al = l.attn
            proj = bf(t, l.n_in)
            w = {k: P.get(f"L{i}.{k}") for k in ("q_norm", "k_norm", "conv")}
            kv_cols = s.kv_heads * (al.dk + al.dv)
            r.add(f"preparation {what}: {name}", "deluvik",
                  lambda: ops.attn_prep(proj, l, w, model.freqs[i], batch, kv, model.caches[i], pool, model.conv_state[i], eps), t * (al.n_in + al.k0 + kv_cols) * 2)
            q, mid = bf(t, al.k0), bf(t, l.n_out)
            win = s.window or ctx
            seen = b * sum(min(p + 1, win) for p in range(ctx - n, ctx))
            keys = b * min(ctx, n + win - 1)
            r.add(f"attention {what}: {name}", "deluvik",
                  lambda: ops.softmax_attention(q, mid, al, P.get(f"L{i}.sink"), 1.0, batch, kv, model.caches[i]),
                  keys * kv_cols * 2 + t * s.heads * (al.dk + al.dv) * 2, 2.0 * seen * s.heads * (al.dk + al.dv))
        rl = lp.lru
        proj, mid, gates = bf(t, lp.n_in), bf(t, lp.n_out), rl.spec.blocks * 2 * rl.pp * rl.pp
        r.add(f"recurrence {what}", "deluvik", lambda: ops.lru_mix(proj, mid, lp, lw, batch, pool, model.lru_state[0]),
              gates * 2 + b * rl.width * 8 + t * rl.width * 6, 2.0 * t * gates)
        inp = bf(t, ch.gdn_in_rows)
        r.add(f"recurrence {what}: gdn", "hybrid", lambda: ops.gdn(inp, glp, batch, gpool, 0, ch, heads // 2, heads),
              b * heads * gd * gd * 8 + t * (ch.gdn_in_rows * 2 + heads * gd * 2), 6.0 * t * heads * gd * gd)
        pa = make_kv_pool(replace(ch, layer_types=(ATTN,)), b * pages + 1, dev)
        pa.k.normal_(), pa.v.normal_()
        qkv = bf(t, ch.qkv_rows)
        qb, (kc, vc) = bf(t, nq * 256), pa.layer(0)

        def prep():
            N.check(ops.lib.trl_attn_prep(qkv.data_ptr(), qkv.stride(0), alp["q_norm"].data_ptr(), alp["k_norm"].data_ptr(), batch.positions.data_ptr(),
                                          batch.slot_mapping.data_ptr(), qb.data_ptr(), kc.data_ptr(), vc.data_ptr(), t, nq, nkv, 256, ch.rotary_dim,
                                          ch.rope_theta, eps, 0, kc.shape[0], N.stream()))
        r.add(f"preparation {what}", "hybrid", prep, t * (2 * ch.qkv_rows) * 2)
        pairs = b * sum(range(ctx - n + 1, ctx + 1))
        r.add(f"attention {what}: with preparation", "hybrid", lambda: ops.attention(qkv, alp, batch, pa, 0, ch, nq, nkv),
              b * ctx * nkv * 256 * 4 + t * nq * 256 * 6, 4.0 * pairs * nq * 256)
        del kv, pa, pool, gpool
    return r.rows


def main(argv=None):
    ap = argparse.ArgumentParser(prog="tilerl_b200.suites.deluvik")
    ap.add_argument("--sizes", default="2048,4096")
    ap.add_argument("--only", default=None, choices=["throughput", "kernels"])
    ap.add_argument("--reps", type=int, default=7)
    ap.add_argument("--ticks", type=int, default=32)
    args = ap.parse_args(argv)
    from ..calibration import load_peaks
    pk = load_peaks()
    out = {"suite": "deluvik", "dtype": "deluvik bf16 weights, hybrid NVFP4 weights, bf16 KV", "data": "synthetic (random-init weights, random tokens)",
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
