"""Fetotar through the framework's engine (pools, scheduler, captured ticks) against the plain oracle of
``fetotar_oracle.py``: every schedule of the same tokens gives the same logits, on the CPU reference backend and on
the GPU in fp32 and bf16."""
import json
import math

import pytest
import torch

import fetotar_oracle as oracle
from fetotar_cases import (BACKENDS, CONFIGS, TOL, attn, backends, build, close, feed_all, needle_model, random_weights, rel_err, rot, tokens,
                           want_logits)
from tilerl_b200.config import FetotarConfig, config_from_dir, get_config
from tilerl_b200.engine import SamplingParams, StepLimits
from tilerl_b200.mixers import ClampedGluSpec, LatentAttnSpec, LayerSpec, Mamba2Spec, MlstmSpec, RotarySpec, YarnSpec


# ---- mechanisms on their own (reference backend functions against the oracle) ---------------------------
def _g(seed):
    return torch.Generator().manual_seed(seed)


@pytest.mark.parametrize("spec", [RotarySpec(16, 10000.0), RotarySpec(32, 500.0, YarnSpec(8.0, 64.0, 4.0, 1.0)), RotarySpec(2, 100.0, YarnSpec(2.0, 16.0, 2.0, 1.0)),
                                  RotarySpec(12, 50.0, YarnSpec(40.0, 4096.0, 32.0, 1.0)), RotarySpec(8, 1e6, YarnSpec(1.0, 128.0, 32.0, 1.0))])
def test_rotation_frequencies_and_pairs(spec):
    from tilerl_b200.ops.ref_mixers import rotate_pairs
    want, amp = oracle.rotary_frequencies(spec.to_json())
    assert spec.amplitude == amp and all(math.isclose(a, b, rel_tol=1e-12) for a, b in zip(spec.frequencies(), want))
    x = torch.randn(6, 3, spec.dims + 4, generator=_g(0))
    pos = [0, 1, 5, 63, 1000, 70001]
    got = rotate_pairs(x, torch.tensor(pos), torch.tensor(spec.frequencies(), dtype=torch.float64), spec.amplitude)
    assert torch.allclose(got.double(), oracle.rotate(x.double(), pos, spec.to_json()), atol=1e-6)
    assert torch.equal(got[..., spec.dims:], x[..., spec.dims:])


def test_rotation_by_hand():
    plain = RotarySpec(4, 100.0)
    assert plain.frequencies() == (1.0, 0.1) and plain.amplitude == 1.0
    scaled = RotarySpec(4, 100.0, YarnSpec(10.0, 2 * math.pi * 10, 10.0, 1.0))     # turns 10 -> dimension 0, turns 1 -> dimension 1
    assert all(math.isclose(a, b) for a, b in zip(scaled.frequencies(), (1.0, 0.01)))
    assert math.isclose(scaled.amplitude, 1.0 + 0.1 * math.log(10.0))


def test_norms_glu_and_gelu_against_the_oracle():
    from tilerl_b200.ops import ref_mixers as m
    x, w, b = (torch.randn(s, generator=_g(i)) for i, s in enumerate([(5, 37), (37,), (37,)]))
    pad = lambda t: torch.nn.functional.pad(t, (0, 27))
    got = m.stream_norm(pad(x + 3.0), torch.stack([pad(w), pad(b)]), 1e-3, 37)
    assert torch.allclose(got[:, :37], oracle.layer_norm((x + 3.0).double(), w.double(), b.double(), 1e-3).float(), atol=1e-5)
    assert not got[:, 37:].any()
    got = m.stream_norm(pad(x), pad(w)[None], 1e-3, 37)
    assert torch.allclose(got[:, :37], (oracle.unit_rms(x.double(), 1e-3) * w).float(), atol=1e-5)
    gu = 3.0 * torch.randn(4, 20, generator=_g(5))
    assert torch.allclose(m.clamped_glu(gu, 1.1), oracle.clamped_glu(gu[:, 0::2], gu[:, 1::2], 1.1), atol=1e-6)
    assert torch.allclose(m.clamped_glu(torch.tensor([[9.0, -9.0]]), 2.0), torch.tensor([[2.0 / (1 + math.exp(-3.404)) * -1.0]]))
    assert torch.allclose(m.gelu_tanh(gu), torch.nn.functional.gelu(gu, approximate="tanh"), atol=1e-6)


def test_scan_steps_against_the_oracle():
    from tilerl_b200.ops import ref_mixers as m
    g, n, h, d, v = _g(3), 40, 3, 7, 5
    x, b, c = torch.randn(n, h, v, generator=g), torch.randn(n, 1, d, generator=g), torch.randn(n, 1, d, generator=g)
    dt, a, skip = torch.rand(n, h, generator=g), torch.randn(h, generator=g), torch.randn(h, generator=g)
    s, out = torch.zeros(h, d, v), []
    for t in range(n):
        s, y = m.mamba2_step(s, x[t], b[t].expand(h, d), c[t].expand(h, d), dt[t], a, skip)
        out.append(y)
    assert torch.allclose(torch.stack(out).double(), oracle.scan_mamba2(x.double(), b.double(), c.double(), dt.double(), a.double(), skip.double()), atol=1e-4)
    q, k = torch.randn(n, h, d, generator=g), torch.randn(n, h, d, generator=g)
    raw = 6.0 * torch.randn(n, 2 * h, generator=g)
    i, f = m.mlstm_gates(raw, torch.zeros(2 * h), 5.0)
    assert float(i.abs().max()) <= 5.0 and float(f.max()) < 0.0
    st, out = (torch.zeros(h, d, v), torch.zeros(h, d), torch.zeros(h)), []
    for t in range(n):
        *st, o = m.mlstm_step(*st, q[t], k[t], x[t], i[t], f[t])
        out.append(o)
    assert torch.allclose(torch.stack(out).double(), oracle.scan_mlstm(q.double(), k.double(), x.double(), i.double(), f.double()), rtol=1e-4, atol=1e-4)


def test_the_running_maximum_of_the_matrix_memory_starts_at_zero():
    """One token with a strongly negative input gate: with m = max(f, i) from m_0 = 0 its contribution stays far below the
    floor exp(-m), where a start at minus infinity would normalise it away."""
    from tilerl_b200.ops.ref_mixers import mlstm_step
    one = torch.ones(1, 1)
    _, _, m, o = mlstm_step(torch.zeros(1, 1, 1), torch.zeros(1, 1), torch.zeros(1), one, one, one, torch.tensor([-8.0]), torch.tensor([-0.5]))
    assert math.isclose(float(m), -0.5) and math.isclose(float(o), math.exp(-7.5) / (math.exp(0.5) + 1e-6), rel_tol=1e-5)


@pytest.mark.parametrize("itemsize", [2, 4])
@pytest.mark.parametrize("kv,rd", [(16, 16), (48, 32), (512, 64), (96, 16)])
def test_latent_pages_place_every_element_once(kv, rd, itemsize):
    from tilerl_b200.kv import LatentPage
    pg = LatentPage(kv, rd, itemsize)
    assert sorted(pg.index().reshape(-1).tolist()) == list(range(pg.nbytes // itemsize)) and pg.nbytes == 16 * (kv + rd) * itemsize
    for c in range(pg.chunks if pg.chunks % 8 == 0 else 0):       # eight rows at one chunk: eight bank groups
        assert len(set((pg.index()[:8, c * 16 // itemsize] * itemsize // 16 % 8).tolist())) == 8


def test_latent_pool_round_trip_and_tiers():
    from tilerl_b200.kv import PackedKvPool
    from tilerl_b200.ops import ref_mixers as m
    pool = PackedKvPool(CONFIGS["mixed"], 5, dtype=torch.float32)
    assert len(pool.pages) == 2
    for i, pg in enumerate(pool.pages):
        rows = torch.randn(20, pg.width, generator=_g(i))
        m.latent_write(pool.layer(i), pg, rows, torch.tensor([3 * 16 + j for j in range(16)] + [16 + j for j in range(4)]))
        for lo, hi in ((0, 20), (3, 17), (16, 20), (15, 16)):
            assert torch.equal(m.latent_gather(pool.layer(i), pg, pool.dtype, torch.tensor([3, 1]), lo, hi), rows[lo:hi])
    before = pool.k.clone()
    a, b = pool.read_block(3)
    assert list(a.shape) == pool.page_shape and a.numel() + b.numel() == pool.block_bytes()
    pool.layer(0)[3].zero_(), pool.layer(1)[3].zero_()
    pool.write_block(3, a, b)
    assert torch.equal(pool.k, before)


def test_state_pool_slots_planes_and_snapshots():
    from tilerl_b200.kv import PoolExhausted, RecurrentPool
    pool = RecurrentPool(CONFIGS["wide"], 3, planes=4, ring_dtype=torch.float32)
    assert pool.recurrent and pool.ring_rows >= 4 + 3
    s = pool.alloc_slot()
    parts = [p for i in range(3) for p in pool.view(i, s, 2)]
    assert len({p.data_ptr() for p in parts}) == len(parts)
    for j, p in enumerate(parts):
        p.fill_(float(j + 1))
    assert pool.states[s, 2].unique().numel() <= len(parts) + 1 and not pool.states[s, 0].any()
    pool.ring[s].fill_(2.0)
    pool.select_step(s, 2)
    snap = pool.snapshot(s)
    other = pool.alloc_slot()
    with pytest.raises(PoolExhausted):
        pool.alloc_slot()
    pool.restore(other, snap)
    assert torch.equal(pool.states[other, 0], pool.states[s, 2]) and torch.equal(pool.ring[other], pool.ring[s])
    pool.release(s)
    assert pool.alloc_slot() == s and not pool.states[s].any() and not pool.ring[s].any()


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_served_parameters_hold_every_tensor_and_only_zeros_besides(name):
    from tilerl_b200.models.fetotar import FetotarModel
    cfg = CONFIGS[name]
    w = random_weights(cfg)
    m = FetotarModel.from_tensors(cfg, w.__getitem__, "cpu", torch.float32)
    got = dict(m.tensors())
    assert set(got) == set(w)
    for k, t in got.items():
        assert torch.equal(t, w[k]), k
    total = sum(float(t.double().pow(2).sum()) for t in w.values())
    assert math.isclose(sum(float(t.double().pow(2).sum()) for t in m.params.values()), total, rel_tol=1e-9)
    assert cfg.n_params() == sum(t.numel() for t in w.values())
    assert FetotarConfig.from_json(json.loads(json.dumps(cfg.to_json())), name=cfg.name, max_ctx=cfg.max_ctx) == cfg


def test_configuration_refuses_what_it_does_not_know():
    j = CONFIGS["mixed"].to_json()
    edits = (lambda d: d["layers"][0].update(type="attention"), lambda d: d["layers"][0]["mixer"].update(sinks=4), lambda d: d.update(loop={}),
             lambda d: d["layers"][2]["mlp"].update(kind="moe"), lambda d: d["layers"][2]["mixer"].update(groups=4),
             lambda d: d["layers"][2]["mixer"].update(norm_groups=5), lambda d: d["layers"][1]["mixer"].pop("gate_cap"),
             lambda d: d["layers"][0]["mixer"]["rot"].update(dims=64), lambda d: d["layers"][0]["mixer"]["rot"]["scaling"].update(kind="x"),
             lambda d: d["layers"][0]["mixer"]["mask"].update(size=0))
    for edit in edits:
        bad = json.loads(json.dumps(j))
        edit(bad)
        with pytest.raises(ValueError):
            FetotarConfig.from_json(bad)
    assert get_config("fetotar-tiny").n_attn_layers == 1


# ---- schedules ---------------------------------------------------------------------------------------
@backends
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_whole_prompt_matches_the_oracle(backend, name):
    cfg = CONFIGS[name]
    w = random_weights(cfg)
    eng = build(cfg, w, backend)
    for n in (1, 2, 15, 17, 64, 65, 150):
        toks = tokens(cfg, n, seed=n)
        assert close(feed_all(eng, "a", toks, [n]), want_logits(cfg, w, toks), backend), n
    assert eng.kv.used_blocks == 0 and eng.states.free_slots == 4


@backends
@pytest.mark.parametrize("name", ["tiny", "attention", "mamba2", "mlstm", "mixed", "wide"])
@pytest.mark.parametrize("cuts", [[1], [2], [3, 1, 2, 5], [17, 15, 1, 16], [64, 3, 64], [130, 1]])
def test_portions_and_token_by_token_match_the_oracle(backend, name, cuts):
    cfg = CONFIGS[name]
    w = random_weights(cfg, seed=3)
    toks = tokens(cfg, 147, seed=7)
    got = feed_all(build(cfg, w, backend), "a", toks, cuts)
    assert close(got, want_logits(cfg, w, toks), backend)


@backends
def test_layer_outputs_match_the_oracle(backend):
    from tilerl_b200.batch import Batch
    cfg = CONFIGS["mixed"]
    w = random_weights(cfg, seed=5)
    eng = build(cfg, w, backend)
    toks = tokens(cfg, 40)
    _, states = oracle.forward(cfg.to_json(), w, toks)
    batch = Batch.build([dict(tokens=toks, start=0, blocks=[1, 2, 3], slot=eng.states.alloc_slot())], eng.device)
    _, x, taps = eng.model.forward(batch, eng.ops, eng.kv, eng.states, aux_layers=tuple(range(cfg.n_layers)))
    for layer, t in taps.items():
        want = states[layer].float()
        assert float((t.cpu().float() - want).abs().max() / want.abs().max()) < 3 * TOL[backend], layer
    assert torch.equal(x, taps[cfg.n_layers - 1])


@backends
@pytest.mark.parametrize("name", ["tiny", "mixed"])
def test_mixed_batches_of_unequal_requests_equal_each_alone(backend, name):
    """Portions of some requests beside single tokens of others; requests pause, end and start again, so pages and
    slots change hands."""
    cfg = CONFIGS[name]
    w = random_weights(cfg, seed=4)
    eng = build(cfg, w, backend, max_tokens=4 * 128)
    lens = {"a": 120, "b": 33, "c": 1, "d": 90, "e": 64, "f": 47}
    toks = {k: tokens(cfg, n, seed=ord(k)) for k, n in lens.items()}
    got, at = {k: [] for k in lens}, {k: 0 for k in lens}
    g = _g(9)
    live, todo = [], list(lens)
    while live or todo:
        while todo and len(live) < 4:
            live.append(todo.pop(0))
        entries, end = [], []
        for k in list(live):
            if int(torch.randint(0, 5, (1,), generator=g)) == 0 and len(live) > 1:
                continue                                      # left out of this step
            n = min(lens[k] - at[k], [1, 1, 2, 7, 16, 31, 70][int(torch.randint(0, 7, (1,), generator=g))])
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
        assert close(torch.cat(got[k]), want_logits(cfg, w, toks[k]), backend), k
    assert eng.kv.used_blocks == 0 and eng.states.free_slots == 4


@backends
def test_freed_pages_and_slots_carry_nothing_over(backend):
    """Pages, states and rings are filled with NaN before and between requests: nothing a request reads was left by another."""
    cfg = CONFIGS["mixed"]
    w = random_weights(cfg, seed=6)
    eng = build(cfg, w, backend, max_tokens=256)
    for i, n in enumerate((100, 37, 130)):
        eng.kv.k.fill_(0xFF)
        eng.states.states.fill_(math.nan), eng.states.ring.fill_(math.nan)
        eng.states.cur.fill_(0)
        toks = tokens(cfg, n, seed=20 + i)
        assert close(feed_all(eng, i, toks, [50, 1, 1, 3, 16, 1]), want_logits(cfg, w, toks), backend)


@backends
@pytest.mark.parametrize("turned", [False, True])
@pytest.mark.parametrize("decode", [False, True])
@pytest.mark.parametrize("window", [1, 2, 16, 47, 64, 130])
def test_window_edges(backend, decode, window, turned):
    """The wanted key just inside and just outside the window, first of all, at page borders, right before the query --
    asked for from a prompt, from a short portion and from a decoded token."""
    cfg, w = needle_model(window, turned=turned)
    eng = build(cfg, w, backend, max_tokens=512)
    n = 200
    filler = [3 + t % (cfg.vocab - 3) for t in tokens(cfg, n, seed=31)]
    base = want_logits(cfg, w, filler[:-1] + [1])[-1:]
    at_edge = {n - window: True, n - 1 - window: False}             # the oldest key in sight, the one before it
    for at in sorted({max(0, n - 2), max(0, n - window), max(0, n - 1 - window), max(0, n - 2 - window), max(0, n + 1 - window), 0, 127, 128, 159, 160, 191, 192}):
        if at >= n - 1:
            continue
        toks = list(filler)
        toks[at], toks[n - 1] = 2, 1
        want = want_logits(cfg, w, toks)[-1:]
        if at in at_edge:
            assert (rel_err(want, base) > 0.2) == at_edge[at], (window, at)      # the key shows, or does not
        for cut in ((n - 1,) if decode else (0, n - 2, 150)):
            if cut:
                eng.feed([("a", toks[:cut], [])])
            got = eng.feed([("a", toks[cut:], [n - 1 - cut])], ["a"])
            assert close(got, want, backend), (at, cut)


@backends
def test_the_first_tokens_of_a_sequence(backend):
    """Zeros before the start for the convolution, the empty state, a window that is not full: every length from one on."""
    cfg = CONFIGS["tiny"]
    w = random_weights(cfg, seed=21)
    eng = build(cfg, w, backend)
    toks = tokens(cfg, 30, seed=77)
    want = want_logits(cfg, w, toks)
    for n in range(1, 9):
        got = eng.feed([("a", toks[:n], list(range(n)))]).clone()
        rest = eng.feed([("a", toks[n:], list(range(30 - n)))], ["a"])
        assert close(torch.cat([got, rest]), want, backend), n


@backends
@pytest.mark.parametrize("name", ["mamba2", "mlstm"])
def test_a_state_remembers_a_far_token(backend, name):
    """Slow decays: a token far back changes the logits at the end, over portion borders and through long decoding."""
    cfg = CONFIGS[name]
    w = random_weights(cfg, seed=13)
    for k in w:
        if k.endswith("A_log"):
            w[k] = torch.full_like(w[k], -7.0)
        if k.endswith("f.b"):
            w[k] = torch.full_like(w[k], 16.0)
    n = 260
    toks = tokens(cfg, n, seed=14)
    other = list(toks)
    other[3] = (toks[3] + 1) % cfg.vocab
    want, changed = want_logits(cfg, w, toks), want_logits(cfg, w, other)
    assert rel_err(changed[-1:], want[-1:]) > 8e-3
    eng = build(cfg, w, backend)
    for cuts in ([n], [64, 64, 64, 3], [37, 100, 1, 2, 100], [200, 1]):
        got, moved = feed_all(eng, "a", toks, cuts), feed_all(eng, "b", other, cuts)
        assert close(got, want, backend) and close(moved, changed, backend), cuts
        d = (moved[-1] - got[-1]).float().cpu()
        assert rel_err(d[None], (changed - want)[-1:]) < (0.02 if "bf16" not in backend else 1.5), cuts


@backends
def test_long_decoding_through_cache_and_state(backend):
    cfg = CONFIGS["tiny"]
    w = random_weights(cfg, seed=8)
    toks = tokens(cfg, 300, seed=40)
    eng = build(cfg, w, backend)
    assert close(feed_all(eng, "a", toks, [20, 1]), want_logits(cfg, w, toks), backend)
    if eng.graph is not None and eng.graph.enabled:
        assert eng.counters["graph_ticks"] == 280              # decoded in captured ticks


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
        _greedy_ok(cfg, w, p, r.tokens, TOL[backend])
    assert eng.kv.used_blocks == 0 and eng.counters["mixed_ticks"] > 0


@backends
def test_preemption_and_prefix_reuse_give_the_same_tokens(backend):
    """A prefix hit adopts pages and the recurrent snapshot taken at the same boundary."""
    cfg = CONFIGS["tiny"]
    w = random_weights(cfg, seed=13)
    prompts = [tokens(cfg, n, seed=60 + n) for n in (40, 50, 60)]
    sp = SamplingParams(max_tokens=40, ignore_eos=True)
    eng = build(cfg, w, backend, max_tokens=208)               # not enough pages for all three to the end
    small = eng.generate(prompts, sp)
    assert eng.counters["preempted"] > 0
    for p, r in zip(prompts, small):
        _greedy_ok(cfg, w, p, r.tokens, TOL[backend])
    eng = build(cfg, w, backend, prefix=True)
    first = eng.generate([prompts[2]], sp)[0]
    again = eng.generate([prompts[2] + [5]], sp)[0]
    assert first.cached_tokens == 0 and again.cached_tokens == 48
    _greedy_ok(cfg, w, prompts[2] + [5], again.tokens, TOL[backend])


@backends
def test_sampling_is_seeded_and_speculative_windows_change_nothing(backend):
    """A verify tick keeps the state after every token of its window; a rejected draft leaves nothing behind."""
    from tilerl_b200.spec import ConstantDrafter
    cfg = CONFIGS["tiny"]
    w = random_weights(cfg, seed=14)
    p = [tokens(cfg, 30, seed=70)]
    eng = build(cfg, w, backend)
    sp = SamplingParams(max_tokens=12, temperature=0.8, top_p=0.9, top_k=40, seed=5, ignore_eos=True)
    assert eng.generate(p, sp)[0].tokens == eng.generate(p, sp)[0].tokens
    for draft in (7, eng.generate(p, SamplingParams(max_tokens=2, ignore_eos=True))[0].tokens[1]):
        spec = build(cfg, w, backend, drafter=ConstantDrafter(draft), spec_width=4)
        out = spec.generate(p, SamplingParams(max_tokens=24, ignore_eos=True))[0].tokens
        assert spec.counters["verify_ticks"] > 0
        _greedy_ok(cfg, w, p[0], out, TOL[backend])


# ---- registry, checkpoint, command line -------------------------------------------------------------------
def _save(tmp_path, cfg, w):
    from tilerl_b200.checkpoint import save_checkpoint
    from tilerl_b200.models.fetotar import FetotarModel
    save_checkpoint(FetotarModel.from_tensors(cfg, w.__getitem__, "cpu", torch.float32), str(tmp_path))
    return str(tmp_path)


def test_checkpoint_round_trip_and_bad_tensors(tmp_path):
    from safetensors.torch import load_file, save_file
    from tilerl_b200.checkpoint import CheckpointError
    from tilerl_b200.factory import build_model
    cfg = CONFIGS["mixed"]
    w = random_weights(cfg)
    d = _save(tmp_path, cfg, w)
    assert config_from_dir(d).to_json() == cfg.to_json()
    assert all(torch.equal(t, w[k]) for k, t in build_model(d).tensors())
    t = load_file(d + "/model.safetensors")
    for edit in (lambda x: x.pop("l2.mix.conv.b"), lambda x: x.update({"l1.mix.q": x["l1.mix.q"][1:].contiguous()})):
        bad = dict(t)
        edit(bad)
        save_file(bad, d + "/model.safetensors")
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
    assert cli.main(["bench", "--model", "fetotar-tiny", "--device", "cpu", "--prompt-len", "12", "--gen", "3"]) == 0
    assert json.loads(capsys.readouterr().out)[0]["decode_tok_s"] > 0
    for flags in (["serve", "--dry-run"], ["bench", "--kernels"]):
        assert cli.main([flags[0], "--model", "fetotar-small", *flags[1:]]) == 0
        assert "attn" in capsys.readouterr().out or flags[0] == "serve"
    with pytest.raises(SystemExit):
        cli.main(["train", "--model", "fetotar-tiny", "--device", "cpu"])


@backends
def test_trace_replay_program(backend, tmp_path):
    """Steps on standard input, logits in files: the program a user replays a trace with."""
    import io
    import numpy as np
    from tilerl_b200.replay import open_engine, replay
    cfg = CONFIGS["mixed"]
    w = random_weights(cfg, seed=16)
    d = _save(tmp_path / "m", cfg, w)
    device, dtype, _ = BACKENDS[backend]
    ta, tb = tokens(cfg, 30, seed=80), tokens(cfg, 9, seed=81)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": ta[:20], "want": [3, 19]}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": tb[:8], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "b", "tokens": tb[8:], "want": [0]}, {"id": "a", "tokens": ta[20:], "want": [9, 0]}],
              "end": ["a", "b"]}]
    out = io.StringIO()
    eng = open_engine(d, dtype, 128, device)
    assert replay(eng, [json.dumps(s) for s in steps], str(tmp_path), out) == 3
    assert out.getvalue().split() == ["done", "0", "done", "1", "done", "2"]
    assert not (tmp_path / "1.f32").exists() and eng.kv.used_blocks == 0
    la, lb = want_logits(cfg, w, ta), want_logits(cfg, w, tb)
    for n, want in ((0, la[[3, 19]]), (2, torch.stack([lb[8], la[29], la[20]]))):
        got = torch.from_numpy(np.fromfile(str(tmp_path / f"{n}.f32"), dtype="<f4").reshape(-1, cfg.vocab).copy())
        assert close(got, want, backend)
