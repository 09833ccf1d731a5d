"""Zinutar beside the hybrid model's attention-only form at equal size: throughput of whole models and the kernels
of a layer against their rooflines.

    python bench.py --design zinutar [--only throughput|kernels]

Both models have random-init weights, the same width, heads, head size, depth, vocabulary and parameter count (the
hybrid's SwiGLU has three matrices of two thirds the width).  Whole models run in the format each is served in:
bf16 weights here, NVFP4 (0.56 bytes a weight) there; the kernels of both are timed on bf16 weights.  Throughput: device time (CUDA events) of a whole
prompt, and of captured decode ticks replayed back to back.  Kernels: single launches with the L2 flushed before
each, median of the repetitions, as a fraction of the measured copy bandwidth or bf16 GEMM rate.
"""
from __future__ import annotations

import argparse
import json
import statistics

import torch

SIZES = {     # hidden, query heads, kv heads, head size, ff (two matrices), ffn (three matrices), layers
    "2048": (2048, 8, 2, 256, 9216, 6144, 12),
    "4096": (4096, 16, 4, 256, 14592, 9728, 8),
}
VOCAB = 32768


def configs(size: str):
    from ..config import ATTN, ModelConfig, zinutar_uniform
    h, nq, nkv, d, ff, ffn, n = SIZES[size]
    z = zinutar_uniform(f"zinutar-{size}", hidden=h, vocab=VOCAB, n_layers=n, heads=nq, kv_heads=nkv, dim=d, ff=ff)
    a = ModelConfig(name=f"attention-{size}", hidden=h, ffn=ffn, vocab=VOCAB, layer_types=(ATTN,) * n, n_q_heads=nq,
                    n_kv_heads=nkv, head_dim=d, rotary_dim=64, rope_theta=1e6, attn_gated=False, quant="nvfp4")
    return {"zinutar": z, "attention": a}


def _build(cfg, max_ctx: int, slots: int):
    from ..factory import build_engine, build_model, make_ops
    ops = make_ops("cuda")
    model = build_model(cfg, "cuda", seed=0, ops=ops)
    pages = slots * (max_ctx // 16 + 2)
    return build_engine(model, ops, blocks=pages + 1, slots=slots, max_ctx=max_ctx, prefix=False)


def _events(fn, reps: int, warm: int = 3) -> float:
    """Median device milliseconds of ``fn``."""
    out = []
    for i in range(warm + reps):
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record()
        fn()
        b.record()
        torch.cuda.synchronize()
        if i >= warm:
            out.append(a.elapsed_time(b))
    return statistics.median(out)


def throughput(cfg, prompts, decodes, ticks: int, reps: int):
    """``prompts``: tokens of one sequence; ``decodes``: (sequences, context) pairs."""
    from ..batch import Batch
    need = max(list(prompts) + [c for _, c in decodes]) + 2 * ticks + 32
    slots = max([b for b, _ in decodes] + [1])
    per = need // 16 + 1
    eng = _build(cfg, per * 16, slots)
    g = torch.Generator().manual_seed(0)
    seq = lambda i, toks, start: dict(tokens=toks, start=start, blocks=list(range(1 + i * per, 1 + (i + 1) * per)), slot=i + 1)
    toks = torch.randint(0, cfg.vocab, (max(prompts),), generator=g).tolist()
    rows = []
    for n in prompts:
        batch = Batch.build([seq(0, toks[:n], 0)], "cuda")
        ms = _events(lambda: eng.ops.argmax(eng.model.forward(batch, eng.ops, eng.kv, eng.states)), reps)
        rows.append({"model": cfg.name, "phase": "prefill", "tokens": n, "ms": round(ms, 3), "tok_s": round(n / ms * 1e3)})
    for b, ctx in decodes:
        bk = eng.graph.bucket(b)
        seqs = [seq(i, [5 + i], ctx) for i in range(b)]

        def run():
            for _ in range(ticks):
                bk.graph.replay()
        best = []
        for i in range(3 + reps):
            bk.fill(seqs)
            bk.dev.copy_(bk.host)
            bk.hist_n.zero_()
            best.append(_events(run, 1, 0))
        ms = statistics.median(best[3:]) / ticks
        rows.append({"model": cfg.name, "phase": "decode", "sequences": b, "context": ctx, "ms": round(ms, 4),
                     "tok_s": round(b / ms * 1e3), "kernels": bk.kernels})
    return rows


def kernels(size: str, reps: int, hbm_gbs: float, tflops: float):
    """Kernels of one layer of both designs at the same shapes."""
    from ..batch import Batch
    from ..factory import make_ops
    from ..kv import make_kv_pool
    from ..zinutar_layout import BlockLayout
    h, nq, nkv, d, ff, ffn, _ = SIZES[size]
    cz, ca = configs(size)["zinutar"], configs(size)["attention"]
    l = BlockLayout.of(cz.layers[0])
    ops, dev = make_ops("cuda"), "cuda"
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
        ideal = max(nbytes / hbm_gbs * 1e-3, flops / tflops * 1e-6)
        rows.append({"what": what, "design": design, "us": round(us, 2), "bound": "memory" if nbytes / hbm_gbs * 1e-3 >= flops / tflops * 1e-6
                     else "tensor", "of_measured": round(ideal / us, 3)})

    norm = torch.ones(h, device=dev)
    wi, wo = bf(l.n_in, h), bf(h, l.n_out)
    for m in (1, 8, 16, 2048):
        x, xb, a = torch.randn(m, h, device=dev), bf(m, h), bf(m, l.n_out)
        fl, by = 2.0 * m * h, m * h * 2
        row(f"in projection {m} rows", "zinutar", lambda: ops.stream_linear(x, norm, wi, 1e-5, h), l.n_in * h * 2 + by * 2 + m * l.n_in * 2, fl * l.n_in)
        row(f"in projection {m} rows", "attention", lambda: ops.norm_linear(xb, norm, wi, 1e-5), l.n_in * h * 2 + by + m * l.n_in * 2, fl * l.n_in)
        row(f"out projection {m} rows", "zinutar", lambda: ops.stream_accumulate(a, wo, x), l.n_out * h * 2 + m * l.n_out * 2 + by * 4, fl * l.n_out)
        row(f"out projection {m} rows", "attention", lambda: ops.linear_residual(a, wo, xb), l.n_out * h * 2 + m * l.n_out * 2 + by * 2, fl * l.n_out)
    lp = {"q_norm": torch.ones(d, device=dev), "k_norm": torch.ones(d, device=dev)}
    bias = torch.full((nq,), -6.0, device=dev)
    act = torch.tensor([0.5, 0.3, 0.3, 0.1], device=dev)
    for b, n, ctx in ((1, 1, 16384), (1, 1, 65536), (8, 1, 8192), (64, 1, 2048), (1, 2048, 2048), (1, 8192, 8192), (1, 512, 16384)):
        per = ctx // 16 + 2
        seqs = [dict(tokens=[1] * n, start=ctx - n, blocks=list(range(1 + i * per, 1 + (i + 1) * per)), slot=i + 1) for i in range(b)]
        batch = Batch.build(seqs, dev)
        t = b * n
        pz, pa = make_kv_pool(_one_layer(cz), b * per + 1, dev), make_kv_pool(_one_layer(ca), b * per + 1, dev)
        pa.k.normal_(), pa.v.normal_()
        proj, qkv = bf(t, l.n_in), bf(t, (nq + 2 * nkv) * d)
        mid = ops.block_mid(proj, act, l, batch, pz, 0, 1e-5)
        pairs = b * sum(range(ctx - n + 1, ctx + 1))
        kv_bytes = b * ctx * nkv * d * 4 + t * nq * d * 4
        what = f"attention {b} x {n} at {ctx}"
        row(what, "zinutar", lambda: ops.sigmoid_attention(proj, mid, bias, l, batch, pz, 0, 1e-5), kv_bytes, 4.0 * pairs * nq * d)
        row(what, "attention", lambda: ops.attention(qkv, lp, batch, pa, 0, ca, nq, nkv), kv_bytes, 4.0 * pairs * nq * d)
        if n > 1:
            kvw = t * nkv * d * 8
            row(f"elementwise {t} tokens: block middle", "zinutar", lambda: ops.block_mid(proj, act, l, batch, pz, 0, 1e-5), t * ff * 4 + kvw)
            gu, out = bf(t, 2 * ffn), bf(t, ffn)
            from ..ops import native as N
            row(f"elementwise {t} tokens: SwiGLU", "attention", lambda: N.check(ops.lib.trl_swiglu(gu.data_ptr(), out.data_ptr(), out.numel(), N.stream())), t * ffn * 6)
            x, xb = torch.randn(t, h, device=dev), bf(t, h)
            row(f"elementwise {t} tokens: norm", "zinutar", lambda: ops._stream_norm(x, norm, 1e-5, h, torch.bfloat16), t * h * 6)
            row(f"elementwise {t} tokens: norm", "attention", lambda: ops._rmsnorm(xb, norm, 1e-5), t * h * 4)
        del pz, pa
    return rows


def _one_layer(cfg):
    from dataclasses import replace
    return replace(cfg, layers=cfg.layers[:1]) if hasattr(cfg, "layers") else replace(cfg, layer_types=cfg.layer_types[:1])


def main(argv=None):
    ap = argparse.ArgumentParser(prog="tilerl_b200.suites.zinutar")
    ap.add_argument("--sizes", default="2048,4096")
    ap.add_argument("--only", default=None, choices=["throughput", "kernels"])
    ap.add_argument("--reps", type=int, default=7)
    ap.add_argument("--ticks", type=int, default=32)
    args = ap.parse_args(argv)
    from ..calibration import load_peaks
    pk = load_peaks()
    out = {"suite": "zinutar", "dtype": "zinutar bf16 weights, attention NVFP4 weights, bf16 KV", "data": "synthetic (random-init weights, random tokens)",
           "peaks": {"hbm_gbs": pk.hbm_gbs, "bf16_tflops": pk.bf16_tflops}, "throughput": [], "kernels": {}}
    for size in args.sizes.split(","):
        if args.only != "kernels":
            for cfg in configs(size).values():
                out["throughput"] += throughput(cfg, (512, 2048, 8192), ((1, 2048), (8, 2048), (16, 2048), (1, 32768)), args.ticks, args.reps)
                torch.cuda.empty_cache()
        if args.only != "throughput":
            out["kernels"][size] = kernels(size, args.reps, pk.hbm_gbs, pk.bf16_tflops)
            torch.cuda.empty_cache()
    print(json.dumps(out))
