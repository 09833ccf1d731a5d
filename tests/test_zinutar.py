"""Zinutar through the framework's engine (pools, scheduler, captured ticks) against the plain oracle of
``zinutar_oracle.py``: every schedule of the same tokens gives the same logits, on the CPU reference backend and on
the GPU in fp32 and bf16."""
import json
import math

import pytest
import torch

import zinutar_oracle as oracle
from tilerl_b200.config import AttnSpec, BlockSpec, LoopSpec, MlpSpec, ZinutarConfig, config_from_dir, get_config
from tilerl_b200.engine import SamplingParams, StepLimits
from zinutar_cases import BACKENDS, CONFIGS, backends, build, feed_all, random_weights, rel_err, tokens, want_logits


# ---- mechanisms on their own (reference backend functions against the oracle) ---------------------------
def test_polynorm_against_the_oracle_and_by_hand():
    from tilerl_b200.ops import ref
    z = torch.randn(5, 37, generator=torch.Generator().manual_seed(0)) * 3
    coef = torch.tensor([0.7, -0.4, 1.3, 0.25])
    got = ref.polynorm(z, coef, 1e-3)
    assert torch.allclose(got, oracle.poly_act(z.double(), coef.double(), 1e-3).float(), atol=2e-6)
    # two equal magnitudes: every power is its own root mean square
    z = torch.tensor([[2.0, -2.0]])
    assert torch.allclose(ref.polynorm(z, torch.tensor([1.0, 10.0, 100.0, 0.5]), 0.0), torch.tensor([[111.5, -90.5]]))


def test_sigmoid_attention_is_a_plain_sum_over_keys():
    from tilerl_b200.ops import ref
    g = torch.Generator().manual_seed(1)
    q, k, v = torch.randn(6, 8, generator=g), torch.randn(9, 2, 8, generator=g), torch.randn(9, 2, 5, generator=g)
    bias = torch.randn(6, generator=g)
    got = ref.sigmoid_attention(q, k, v, bias, 0.3)
    for h in range(6):
        s = (k[:, h // 3] @ q[h]) * 0.3 + bias[h]
        assert torch.allclose(got[h], (torch.sigmoid(s)[:, None] * v[:, h // 3]).sum(0), atol=1e-6)
    # the same keys twice count twice: no normalisation over keys
    twice = ref.sigmoid_attention(q, torch.cat([k, k]), torch.cat([v, v]), bias, 0.3)
    assert torch.allclose(twice, 2 * got, atol=1e-5)


@pytest.mark.parametrize("itemsize", [2, 4])
@pytest.mark.parametrize("dim,vdim", [(16, 16), (20, 88), (128, 40), (256, 256)])
def test_packed_pages_place_every_element_once(dim, vdim, itemsize):
    from tilerl_b200.kv import KvPage
    pg = KvPage(3, dim, vdim, itemsize)
    byte = lambda idx, size: (idx.reshape(-1, 1) * size + torch.arange(size)).reshape(-1)
    used = torch.cat([byte(pg.k_index(), itemsize), byte(pg.v_index(), itemsize), byte(pg.rms_index(), 4)])
    spare = range(pg.rms_offset + 64, pg.v_offset)
    assert sorted(used.tolist() + list(spare)) == list(range(pg.nbytes))      # every other byte of the page once
    assert pg.nbytes % 128 == 0 and pg.v_offset % 128 == 0
    # eight rows at one chunk index fall into different 16-byte bank groups when a row is a multiple of 128 bytes
    for c in range(pg.k_chunks if pg.k_chunks % 8 == 0 else 0):
        groups = (pg.k_index()[:8, c * 16 // itemsize] * itemsize // 16) % 8
        assert len(set(groups.tolist())) == 8


def test_packed_pool_round_trip_and_tiers():
    from tilerl_b200.kv import PackedKvPool
    from tilerl_b200.ops import ref
    cfg = CONFIGS["mha"]
    pool = PackedKvPool(cfg, 5, dtype=torch.float32)
    g = torch.Generator().manual_seed(2)
    for i, pg in enumerate(pool.pages):
        k = torch.nn.functional.pad(torch.randn(20, pg.n_kv, pg.dim, generator=g), (0, pg.pad(pg.dim) - pg.dim))
        v = torch.nn.functional.pad(torch.randn(20, pg.n_kv, pg.vdim, generator=g), (0, pg.pad(pg.vdim) - pg.vdim))
        slots = torch.tensor([3 * 16 + j for j in range(16)] + [16 + j for j in range(4)])
        ref.packed_kv_write(pool.layer(i), pg, k, v, slots, cfg.rms_eps)
        kk, vv = ref.packed_kv_gather(pool.layer(i), pg, pool.dtype, torch.tensor([3, 1]), 20)
        assert torch.equal(vv, v)
        assert torch.allclose(kk[..., :pg.dim], oracle.rms(k[..., :pg.dim].double(), cfg.rms_eps).float(), atol=1e-6)
    before = pool.k.clone()
    a, b = pool.read_block(3)
    assert list(a.shape) == pool.page_shape and a.numel() + b.numel() == pool.block_bytes()
    for i in range(len(pool.pages)):
        pool.layer(i)[3].zero_()
    pool.write_block(3, a, b)
    assert torch.equal(pool.k, before)


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_fused_parameters_hold_every_tensor_and_only_zeros_besides(name):
    from tilerl_b200.models.zinutar import ZinutarModel
    cfg = CONFIGS[name]
    w = random_weights(cfg)
    m = ZinutarModel.from_tensors(cfg, w.__getitem__, "cpu", torch.float32)
    for k, t in m.tensors():
        assert torch.equal(t, w[k]), k
    total = sum(float(t.double().pow(2).sum()) for t in w.values())
    assert math.isclose(sum(float(t.double().pow(2).sum()) for t in m.params.values()), total, rel_tol=1e-9)
    assert cfg.n_params() == sum(t.numel() for t in w.values())


def test_execution_order_and_caches():
    cfg = CONFIGS["mqa"]
    assert [(r.layer, r.kv, r.inject) for r in cfg.runs] == [(0, 0, False), (1, 1, False), (1, 2, True), (1, 3, True), (2, 4, False)]
    for c in CONFIGS.values():
        j = c.to_json()
        assert [(r.layer, r.inject) for r in c.runs] == oracle.execution_order(len(j["layers"]), j.get("loop"))
        assert [r.kv for r in c.runs] == list(range(c.n_attn_layers))
        assert ZinutarConfig.from_json(json.loads(json.dumps(j)), name=c.name, max_ctx=c.max_ctx) == c


def test_configuration_refuses_what_it_does_not_know():
    j = CONFIGS["one"].to_json()
    for edit in (lambda d: d["layers"][0].update(type="conv"), lambda d: d["layers"][0]["mixer"].update(window=4),
                 lambda d: d["layers"][0]["mlp"].update(kind="moe"), lambda d: d["layers"][0]["mixer"].update(heads=3, kv_heads=2),
                 lambda d: d.update(loop={"start": 0, "stop": 2, "times": 1})):
        bad = json.loads(json.dumps(j))
        edit(bad)
        with pytest.raises(ValueError):
            ZinutarConfig.from_json(bad)
    with pytest.raises(ValueError):
        get_config("no-such-model")


# ---- schedules ---------------------------------------------------------------------------------------
@backends
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_whole_prompt_matches_the_oracle(backend, name):
    cfg = CONFIGS[name]
    w = random_weights(cfg)
    eng = build(cfg, w, backend)
    for n in (1, 2, 15, 16, 17, 64, 150):
        toks = tokens(cfg, n, seed=n)
        assert rel_err(feed_all(eng, "a", toks, [n]), want_logits(cfg, w, toks)) < BACKENDS[backend][2], n
    assert eng.kv.used_blocks == 0 and eng.states.free_slots == 4


@backends
@pytest.mark.parametrize("name", ["tiny", "mqa", "mha", "wide"])
@pytest.mark.parametrize("cuts", [[1], [2], [3, 1, 2, 5], [17, 15, 1, 16], [64, 3, 64], [130, 1]])
def test_portions_and_token_by_token_match_the_oracle(backend, name, cuts):
    cfg = CONFIGS[name]
    w = random_weights(cfg, seed=3)
    toks = tokens(cfg, 147, seed=7)
    got = feed_all(build(cfg, w, backend), "a", toks, cuts)
    assert rel_err(got, want_logits(cfg, w, toks)) < BACKENDS[backend][2]


@backends
def test_layer_outputs_match_the_oracle(backend):
    from tilerl_b200.batch import Batch
    from tilerl_b200.models.zinutar import ZinutarModel
    cfg = CONFIGS["tiny"]
    w = random_weights(cfg, seed=5)
    eng = build(cfg, w, backend)
    toks = tokens(cfg, 40)
    _, states = oracle.forward(cfg.to_json(), w, toks)
    batch = Batch.build([dict(tokens=toks, start=0, blocks=[1, 2, 3], slot=1)], eng.device)
    _, x, taps = eng.model.forward(batch, eng.ops, eng.kv, eng.states, aux_layers=(0, 1, 2))
    last = {r.layer: i for i, r in enumerate(cfg.runs)}
    for layer, t in taps.items():
        want = states[last[layer]].float()
        assert float((t.cpu().float() - want).abs().max() / want.abs().max()) < BACKENDS[backend][2], layer
    assert torch.equal(x, taps[2])


@backends
def test_mixed_batches_of_unequal_requests_equal_each_alone(backend):
    """Portions of some requests beside single tokens of others; requests pause, end and start again, so pages and
    slots change hands."""
    cfg = CONFIGS["mqa"]
    w = random_weights(cfg, seed=4)
    eng = build(cfg, w, backend, max_tokens=4 * 128)
    lens = {"a": 120, "b": 33, "c": 1, "d": 90, "e": 64, "f": 47}
    toks = {k: tokens(cfg, n, seed=ord(k)) for k, n in lens.items()}
    got, at = {k: [] for k in lens}, {k: 0 for k in lens}
    g = torch.Generator().manual_seed(9)
    live, todo = [], list(lens)
    while live or todo:
        while todo and len(live) < 4:
            live.append(todo.pop(0))
        entries, end = [], []
        for k in list(live):
            if int(torch.randint(0, 5, (1,), generator=g)) == 0 and len(live) > 1:
                continue                                      # left out of this step
            n = min(lens[k] - at[k], [1, 1, 2, 7, 16, 31][int(torch.randint(0, 6, (1,), generator=g))])
            entries.append((k, toks[k][at[k]:at[k] + n], list(range(n))))
        if not entries:
            continue
        for k, t, _ in entries:
            at[k] += len(t)
            if at[k] == lens[k]:
                end.append(k)
                live.remove(k)
        out, o = eng.feed(entries, end).clone(), 0
        for k, t, _ in entries:
            got[k].append(out[o:o + len(t)])
            o += len(t)
    for k in lens:
        assert rel_err(torch.cat(got[k]), want_logits(cfg, w, toks[k])) < BACKENDS[backend][2], k
    assert eng.kv.used_blocks == 0


@backends
def test_freed_pages_and_slots_carry_nothing_over(backend):
    """The pool is filled with NaN bytes before and between requests: nothing a request reads was left by another."""
    cfg = CONFIGS["tiny"]
    w = random_weights(cfg, seed=6)
    eng = build(cfg, w, backend, max_tokens=256)
    for i, n in enumerate((100, 37, 130)):
        eng.kv.k.fill_(0xFF)
        toks = tokens(cfg, n, seed=20 + i)
        assert rel_err(feed_all(eng, i, toks, [50, 1, 1, 3, 16, 1]), want_logits(cfg, w, toks)) < BACKENDS[backend][2]


def needle_model(heads=2, kv_heads=1, dim=32, vdim=32):
    """One layer in which token 1 asks for token 2: that score stands far above every other, whose weights are
    e^-12 and less, so the logits of a 1 count the 2s it sees."""
    cfg = ZinutarConfig(name="needle", hidden=96, vocab=90, max_ctx=4096, rms_eps=1e-5,
                        layers=(BlockSpec(AttnSpec(heads, kv_heads, dim, vdim, 1.0), MlpSpec(24)),))
    w = random_weights(cfg, seed=11)
    x = oracle.embedding_output({k: t.double() for k, t in w.items()}, [1, 2], cfg.rms_eps)
    h = oracle.rms(x, cfg.rms_eps) * w["l0.norm1"].double()
    k2 = w["l0.mix.k"][:dim].double() @ h[1]
    for head in range(heads):
        rows = slice(head * dim, (head + 1) * dim)
        w["l0.mix.q"][rows] += (8.0 * torch.outer(k2, h[0]) / (h[0] @ h[0])).float()
    w["l0.mix.pb"].fill_(-0.75 * dim)
    w = {k: t.to(torch.bfloat16).float() for k, t in w.items()}
    return cfg, w


@backends
@pytest.mark.parametrize("decode", [False, True])
def test_a_far_key_is_seen_at_every_place(backend, decode):
    """The wanted key first of all, on both sides of page and tile borders, right before the query and as the query's
    own neighbour -- asked for from a prompt and from a decoded token."""
    cfg, w = needle_model()
    eng = build(cfg, w, backend, max_tokens=1024)
    n = 700
    filler = [3 + t % (cfg.vocab - 3) for t in tokens(cfg, n, seed=31)]
    base = want_logits(cfg, w, filler[:-1] + [1])[-1:]
    places = [0, 1, 15, 16, 17, 63, 64, 127, 128, 255, 256, 511, 512, 639, 640, n - 17, n - 3, n - 2]
    for at in places:
        toks = list(filler)
        toks[at], toks[n - 1] = 2, 1
        want = want_logits(cfg, w, toks)[-1:]
        assert rel_err(want, base) > 0.3                       # the key shows
        cut = n - 1 if decode else 650
        if cut:
            eng.feed([("a", toks[:cut], [])])
        got = eng.feed([("a", toks[cut:], [n - 1 - cut])], ["a"])
        assert rel_err(got, want) < BACKENDS[backend][2], at


@backends
def test_future_keys_stay_out_and_repeats_count(backend):
    cfg, w = needle_model(heads=4, kv_heads=2, dim=24, vdim=40)
    eng = build(cfg, w, backend)
    toks = [3 + t % (cfg.vocab - 3) for t in tokens(cfg, 200, seed=33)]
    for i in (10, 20, 47, 48, 150):
        toks[i] = 2
    for i in (9, 11, 47 - 1, 49, 149, 199):
        toks[i] = 1                                            # sees 0, 1, 2, 4, 4 and 5 of them
    want = want_logits(cfg, w, toks)
    for cuts in ([200], [48, 1, 1, 100], [2], [11, 38, 1]):
        assert rel_err(feed_all(eng, "a", toks, cuts), want) < BACKENDS[backend][2], cuts


@backends
def test_long_decoding_through_the_cache(backend):
    cfg = CONFIGS["one"]
    w = random_weights(cfg, seed=8)
    toks = tokens(cfg, 420, seed=40)
    eng = build(cfg, w, backend)
    assert rel_err(feed_all(eng, "a", toks, [20, 1]), want_logits(cfg, w, toks)) < BACKENDS[backend][2]
    if eng.graph is not None and eng.graph.enabled:
        assert eng.counters["graph_ticks"] == 400              # decoded in captured ticks


# ---- generation through the scheduler --------------------------------------------------------------------
def _greedy_ok(cfg, w, prompt, out, tol):
    """Every generated token is the oracle's best one, or within the backend's rounding of it."""
    lg = want_logits(cfg, w, prompt + out)
    for i, t in enumerate(out):
        row = lg[len(prompt) + i - 1]
        assert float(row.max() - row[t]) <= 4 * tol * float(row.std()), i


@backends
@pytest.mark.parametrize("limit", [512, 24])
def test_greedy_generation_through_the_scheduler(backend, limit):
    cfg = CONFIGS["tiny"]
    w = random_weights(cfg, seed=12)
    eng = build(cfg, w, backend, limits=StepLimits(max_batch=3, max_batched_tokens=limit, prefill_align=8))
    prompts = [tokens(cfg, n, seed=50 + n) for n in (3, 70, 41, 16, 1)]
    lens = (20, 7, 12, 20, 5)
    for p, n, r in zip(prompts, lens, eng.generate(prompts, [SamplingParams(max_tokens=n, ignore_eos=True) for n in lens])):
        assert len(r.tokens) == n
        _greedy_ok(cfg, w, p, r.tokens, BACKENDS[backend][2])
    assert eng.kv.used_blocks == 0 and eng.counters["mixed_ticks"] > 0


@backends
def test_preemption_and_prefix_reuse_give_the_same_tokens(backend):
    cfg = CONFIGS["tiny"]
    w = random_weights(cfg, seed=13)
    prompts = [tokens(cfg, n, seed=60 + n) for n in (40, 50, 60)]
    sp = SamplingParams(max_tokens=40, ignore_eos=True)
    eng = build(cfg, w, backend, max_tokens=208)               # not enough pages for all three to the end
    small = eng.generate(prompts, sp)
    assert eng.counters["preempted"] > 0
    for p, r in zip(prompts, small):
        _greedy_ok(cfg, w, p, r.tokens, BACKENDS[backend][2])
    eng = build(cfg, w, backend, prefix=True)
    first = eng.generate([prompts[2]], sp)[0]
    again = eng.generate([prompts[2] + [5]], sp)[0]
    assert first.cached_tokens == 0 and again.cached_tokens == 48
    _greedy_ok(cfg, w, prompts[2] + [5], again.tokens, BACKENDS[backend][2])


@backends
def test_sampling_is_seeded_and_speculative_windows_change_nothing(backend):
    from tilerl_b200.spec import ConstantDrafter
    cfg = CONFIGS["tiny"]
    w = random_weights(cfg, seed=14)
    p = [tokens(cfg, 30, seed=70)]
    eng = build(cfg, w, backend)
    sp = SamplingParams(max_tokens=12, temperature=0.8, top_p=0.9, top_k=40, seed=5, ignore_eos=True)
    assert eng.generate(p, sp)[0].tokens == eng.generate(p, sp)[0].tokens
    spec = build(cfg, w, backend, drafter=ConstantDrafter(7), spec_width=4)
    out = spec.generate(p, SamplingParams(max_tokens=12, ignore_eos=True))[0].tokens
    assert spec.counters["verify_ticks"] > 0
    _greedy_ok(cfg, w, p[0], out, BACKENDS[backend][2])


def test_feed_refuses_bad_steps_and_leaves_nothing_behind():
    cfg = CONFIGS["one"]
    eng = build(cfg, random_weights(cfg), "cpu", max_tokens=64)
    for bad in ([("a", [], [])], [("a", [cfg.vocab], [])], [("a", [1, 2], [2])], [("a", [1], []), ("a", [2], [])]):
        with pytest.raises(ValueError):
            eng.feed(bad)
    with pytest.raises(ValueError):
        eng.feed([("a", [1], [])], ["b"])
    assert eng.kv.used_blocks == 0 and eng.states.free_slots == 4
    assert eng.feed([("a", [1, 2], [])], ["a"]) is None
    from tilerl_b200.kv import PoolExhausted
    with pytest.raises(PoolExhausted):
        eng.feed([("a", [1] * 100, [])])


# ---- registry, checkpoint, command line -------------------------------------------------------------------
def _save(tmp_path, cfg, w):
    from tilerl_b200.checkpoint import save_checkpoint
    from tilerl_b200.models.zinutar import ZinutarModel
    save_checkpoint(ZinutarModel.from_tensors(cfg, w.__getitem__, "cpu", torch.float32), str(tmp_path))
    return str(tmp_path)


def test_checkpoint_round_trip_and_missing_tensor(tmp_path):
    from tilerl_b200.checkpoint import CheckpointError
    from tilerl_b200.factory import build_model
    cfg = CONFIGS["mha"]
    w = random_weights(cfg)
    d = _save(tmp_path, cfg, w)
    assert config_from_dir(d).to_json() == cfg.to_json()
    m = build_model(d)
    assert all(torch.equal(t, w[k]) for k, t in m.tensors())
    from safetensors.torch import load_file, save_file
    t = load_file(d + "/model.safetensors")
    t.pop("l1.mix.pb")
    save_file(t, d + "/model.safetensors")
    with pytest.raises(CheckpointError):
        build_model(d)


def test_command_line_generates_from_a_directory(tmp_path, capsys):
    from tilerl_b200 import cli
    cfg = CONFIGS["tiny"]
    d = _save(tmp_path / "m", cfg, random_weights(cfg, seed=15))
    (tmp_path / "p.txt").write_text("hello\nworld\n")
    assert cli.main(["generate", "--model", d, "--prompts", str(tmp_path / "p.txt"), "--out", str(tmp_path / "o"),
                     "--max-tokens", "4", "--device", "cpu"]) == 0
    rows = [json.loads(l) for l in (tmp_path / "o" / "part-000.jsonl").read_text().splitlines()]
    assert [r["prompt"] for r in rows] == ["hello", "world"]
    capsys.readouterr()
    assert cli.main(["bench", "--model", "zinutar-tiny", "--device", "cpu", "--prompt-len", "12", "--gen", "3"]) == 0
    assert json.loads(capsys.readouterr().out)[0]["decode_tok_s"] > 0
    for flags in (["serve", "--dry-run"], ["bench", "--kernels"]):
        assert cli.main([flags[0], "--model", "zinutar-8b", *flags[1:]]) == 0
        assert "attn" in capsys.readouterr().out or flags[0] == "serve"
    with pytest.raises(SystemExit):
        cli.main(["train", "--model", "zinutar-tiny", "--device", "cpu"])


@backends
def test_trace_replay_program(backend, tmp_path):
    """Steps on standard input, logits in files: the program a user replays a trace with."""
    import io
    from tilerl_b200.replay import open_engine, replay
    cfg = CONFIGS["mqa"]
    w = random_weights(cfg, seed=16)
    d = _save(tmp_path / "m", cfg, w)
    device, dtype, tol = BACKENDS[backend]
    ta, tb = tokens(cfg, 30, seed=80), tokens(cfg, 9, seed=81)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": ta[:20], "want": [3, 19]}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": tb[:8], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "b", "tokens": tb[8:], "want": [0]}, {"id": "a", "tokens": ta[20:], "want": [9, 0]}],
              "end": ["a", "b"]}]
    out = io.StringIO()
    eng = open_engine(d, dtype, 128, device)
    assert eng.kv.num_blocks == 128 // 16 + 1 and eng.states.free_slots == 4
    assert replay(eng, [json.dumps(s) for s in steps], str(tmp_path), out) == 3
    assert out.getvalue().split() == ["done", "0", "done", "1", "done", "2"]
    assert not (tmp_path / "1.f32").exists() and eng.kv.used_blocks == 0
    la, lb = want_logits(cfg, w, ta), want_logits(cfg, w, tb)
    import numpy as np
    for n, want in ((0, la[[3, 19]]), (2, torch.stack([lb[8], la[29], la[20]]))):
        got = torch.from_numpy(np.fromfile(str(tmp_path / f"{n}.f32"), dtype="<f4").reshape(-1, cfg.vocab).copy())
        assert rel_err(got, want) < tol
