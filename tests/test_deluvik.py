"""Deluvik through the framework's engine (pools, scheduler, captured ticks) against the plain oracle of ``deluvik_oracle.py``:
every schedule of the same tokens gives the same logits, on the CPU reference backend and on the GPU in fp32 and bf16."""
import json
import math

import pytest
import torch

import deluvik_oracle as oracle
from deluvik_cases import (BACKENDS, CONFIGS, SCALED, TOL, backends, both, build, close, conv, feed_all, needle_model, random_weights, rel_err,
                           rot, tied, tokens, want_logits)
from tilerl_b200.config import DeluvikConfig, config_from_dir, get_config
from tilerl_b200.engine import SamplingParams, StepLimits
from tilerl_b200.mixers import BandScalingSpec, GluSpec, LayerSpec, LruSpec, MoeSpec, RotarySpec, SoftmaxAttnSpec


# ---- mechanisms on their own (reference backend functions against the oracle) ---------------------------
def _g(seed):
    return torch.Generator().manual_seed(seed)


def _r(*shape, seed=0):
    return torch.randn(*shape, generator=_g(seed))


@pytest.mark.parametrize("half", [False, True])
@pytest.mark.parametrize("spec", [RotarySpec(16, 10000.0), RotarySpec(2, 100.0), RotarySpec(40, 800.0, SCALED), RotarySpec(12, 50.0, BandScalingSpec(8.0, 1.0, 4.0, 512.0)),
                                  RotarySpec(8, 1e6, BandScalingSpec(2.0, 1.0, 1.0, 64.0))])
def test_rotation_frequencies_and_layouts(spec, half):
    from tilerl_b200.ops.ref_mixers import rotate_halves, rotate_pairs
    j = spec.to_json()
    want = oracle.rotary_frequencies(j) if spec.scaling is None or spec.scaling.high > spec.scaling.low else spec.frequencies()
    assert spec.amplitude == 1.0 and all(math.isclose(a, b, rel_tol=1e-12) for a, b in zip(spec.frequencies(), want))
    if spec.scaling is not None and spec.scaling.high == spec.scaling.low:
        return
    x, f = _r(6, 3, spec.dims + 5), torch.tensor(spec.frequencies(), dtype=torch.float64)
    for first in (0, 63, 70001):
        pos = torch.arange(first, first + 6)
        got = rotate_halves(x, pos, f) if half else rotate_pairs(x, pos, f, 1.0)
        assert torch.allclose(got.double(), oracle.rotate(x.double(), j, half, first), atol=1e-6)
        assert torch.equal(got[..., spec.dims:], x[..., spec.dims:])


def test_band_scaling_by_hand():
    s = BandScalingSpec(10.0, 1.0, 4.0, 2.0 * math.pi * 100.0)        # a frequency f turns 100 f times over the original context
    assert s.apply(0.05) == 0.05 and s.apply(0.005) == 0.0005 and math.isclose(s.apply(0.025), 0.5 * 0.025 / 10 + 0.5 * 0.025)


def test_attention_with_cap_and_sink_by_hand():
    from tilerl_b200.ops.ref_mixers import softmax_attention
    q, k, v = torch.tensor([[2.0, 0.0]]), torch.tensor([[[3.0, 0.0]], [[0.0, 1.0]]]), torch.tensor([[[1.0]], [[5.0]]])
    s0, s1 = 4.0 * math.tanh(0.5 * 6.0 / 4.0), 0.0
    den = math.exp(s0) + math.exp(s1) + math.exp(0.7)                  # the sink is neither scaled nor capped, and has no value
    got = softmax_attention(q, k, v, 0.5, 4.0, torch.tensor([0.7]))
    assert math.isclose(float(got), (math.exp(s0) + 5.0 * math.exp(s1)) / den, rel_tol=1e-6)


@pytest.mark.parametrize("cap,sink", [(None, False), (3.0, False), (None, True), (6.0, True)])
def test_attention_against_the_oracle(cap, sink):
    from tilerl_b200.ops.ref_mixers import softmax_attention
    q, k, v, s = _r(9, 6, 10, seed=1), _r(9, 2, 10, seed=2), _r(9, 2, 7, seed=3), _r(6, seed=4) if sink else None
    want = oracle.attend(q.double(), k.double(), v.double(), 0.6, cap=cap, sink=None if s is None else s.double())
    for i in range(9):
        assert torch.allclose(softmax_attention(q[i], k[:i + 1], v[:i + 1], 0.6, cap, s).double(), want[i], atol=1e-5)


def test_norms_over_the_projection_and_per_head():
    from tilerl_b200.ops.ref_mixers import weighted_norm
    x, w = _r(4, 3, 10, seed=1), _r(30, seed=2)
    x[:, :, 7:] = 0.0                                                   # padding columns
    true = x[:, :, :7].reshape(4, 21).double()
    got = weighted_norm(x, 3, 7, w, True, 1e-3)[:, :, :7].reshape(4, 21)
    assert torch.allclose(got.double(), oracle.unit_rms(true, 1e-3) * w.view(3, 10)[:, :7].reshape(21).double(), atol=1e-6)
    got = weighted_norm(x, 3, 7, w[:10], False, 1e-3)[:, :, :7]
    assert torch.allclose(got.double(), oracle.unit_rms(x[:, :, :7].double(), 1e-3) * w[:7].double(), atol=1e-6)


def test_recurrence_against_the_oracle():
    from tilerl_b200.ops.ref_mixers import lru_step
    n, u, r, i, lam = 50, _r(50, 12, seed=1), 3 * _r(50, 12, seed=2), 3 * _r(50, 12, seed=3), 4 * _r(12, seed=4) - 4
    s, out = torch.zeros(12), []
    for t in range(n):
        s = lru_step(s, u[t], r[t], i[t], lam)
        out.append(s)
    want = oracle.scan_lru(u.double(), oracle.sigmoid(r.double()), oracle.sigmoid(i.double()), lam.double())
    assert torch.allclose(torch.stack(out).double(), want, atol=1e-5)
    a = math.exp(-8.0 * 0.5 * math.log1p(math.exp(0.3)))               # by hand: both gates at one half
    got = lru_step(torch.tensor([2.0]), torch.tensor([1.5]), torch.zeros(1), torch.zeros(1), torch.tensor([0.3]))
    assert math.isclose(float(got), 2.0 * a + math.sqrt(1.0 - a * a) * 0.5 * 1.5, rel_tol=1e-6)


def test_choice_of_experts_against_the_oracle():
    from tilerl_b200.ops.ref_mixers import activate, choose
    h, w, b = _r(20, 8, seed=1), _r(6, 8, seed=2), _r(6, seed=3)
    for top in (1, 2, 6):
        idx, weight = choose(h @ w.T + b, top)
        want = oracle.route(h.double(), {"router": w.double(), "router.b": b.double()}, "", top)
        assert torch.equal(idx, want[0]) and torch.allclose(weight.double(), want[1], atol=1e-6)
    assert choose(torch.tensor([[1.0, 2.0, 2.0]]), 2)[0].tolist() == [[1, 2]]
    assert torch.allclose(activate(h, "silu"), torch.nn.functional.silu(h)) and torch.allclose(activate(h, "gelu"), oracle.gelu_tanh(h))


# ---- pages, states, parameters, configuration ------------------------------------------------------------
@pytest.mark.parametrize("itemsize", [2, 4])
@pytest.mark.parametrize("dk,dv", [(16, 16), (48, 32), (128, 256), (80, 16)])
def test_pages_without_factors_place_every_element_once(dk, dv, itemsize):
    from tilerl_b200.kv import KvPage
    pg = KvPage(2, dk, dv, itemsize, False)
    places = sorted(pg.k_index().reshape(-1).tolist() + pg.v_index().reshape(-1).tolist())
    assert places == list(range(pg.nbytes // itemsize)) and pg.nbytes == 16 * (dk + dv) * itemsize


def test_layers_that_share_keys_have_one_cache():
    from tilerl_b200.kv import PackedKvPool
    cfg = CONFIGS["mixed"]
    assert [cfg.cache_index(i) for i in range(6)] == [0, 1, 0, 2, 0, 3]
    pool = PackedKvPool(cfg, 5, dtype=torch.float32)
    assert len(pool.pages) == 4 and (pool.pages[0].dim, pool.pages[0].vdim) == (32, 48)


def test_state_pool_holds_vectors_and_convolution_inputs():
    from tilerl_b200.kv import make_state_pool
    cfg = CONFIGS["mixed"]
    pool = make_state_pool(cfg, 3, planes=4, ring_dtype=torch.float32)
    assert pool.recurrent and pool.ring_rows >= 4 + 3
    # (layer, recurrent values, convolved columns): parts and heads are padded to 16
    assert [(l.layer, l.state_floats, l.conv_c) for l in pool.layouts] == [(0, 0, 352), (1, 64, 64), (2, 0, 192), (4, 0, 192), (5, 64, 64)]
    s = pool.alloc_slot()
    for j in range(5):
        pool.ring_view(j, s).fill_(float(j + 1))
        for p in pool.view(j, s, 2):
            p.fill_(float(j + 1))
    for j in range(5):
        assert pool.ring_view(j, s).unique().tolist() == [float(j + 1)]
        assert all(not p.numel() or p.unique().tolist() == [float(j + 1)] for p in pool.view(j, s, 2))
    assert not pool.states[s, 0].any()


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_served_parameters_hold_every_tensor_and_only_zeros_besides(name):
    from tilerl_b200.models.deluvik import DeluvikModel
    cfg = CONFIGS[name]
    w = random_weights(cfg)
    m = DeluvikModel.from_tensors(cfg, w.__getitem__, "cpu", torch.float32)
    got = dict(m.tensors())
    assert set(got) == set(w)
    for k, t in got.items():
        assert torch.equal(t, w[k]), k
    total = sum(float(t.double().pow(2).sum()) for t in w.values())
    assert math.isclose(sum(float(t.double().pow(2).sum()) for t in m.params.values()), total, rel_tol=1e-9)
    assert cfg.n_params() == sum(t.numel() for t in w.values())
    assert DeluvikConfig.from_json(json.loads(json.dumps(cfg.to_json())), name=cfg.name, max_ctx=cfg.max_ctx) == cfg
    again = DeluvikModel.build_random(cfg, seed=3)
    assert set(dict(again.tensors())) == set(w)


def test_configuration_refuses_what_it_does_not_know():
    j = CONFIGS["mixed"].to_json()
    edits = (lambda d: d["layers"][0].update(type="latent_attention"), lambda d: d["layers"][0]["mixer"].update(sinks=4), lambda d: d.update(loop={}),
             lambda d: d["layers"][0]["mlp"].update(kind="switch"), lambda d: d["layers"][1]["mixer"]["right"].update(blocks=7),
             lambda d: d["layers"][1]["mixer"].pop("left_scale"), lambda d: d["layers"][1]["mixer"]["left"]["mask"].update(size=0),
             lambda d: d["layers"][2]["mixer"].update(kv_from=3), lambda d: d["layers"][2]["mixer"].update(kv_from=4), lambda d: d["layers"][4]["mixer"].update(kv_from=2),
             lambda d: d["layers"][2]["mixer"].update(kv_heads=3), lambda d: d["layers"][2]["mixer"]["rot"].update(base=7.0), lambda d: d.pop("logit_softcap"),
             lambda d: d["layers"][3]["mixer"].update(vdim=32), lambda d: d["layers"][3]["mixer"].pop("softcap"), lambda d: d["layers"][3]["mixer"]["rot"].update(dims=64),
             lambda d: d["layers"][3]["mixer"]["rot"]["scaling"].update(fast=2), lambda d: d["layers"][1]["mlp"]["router"].update(top=41),
             lambda d: d["layers"][1]["mlp"].pop("expert"))
    for edit in edits:
        bad = json.loads(json.dumps(j))
        edit(bad)
        with pytest.raises(ValueError):
            DeluvikConfig.from_json(bad)
    assert get_config("deluvik-tiny").n_attn_layers == 3
    with pytest.raises(ValueError):
        SoftmaxAttnSpec(3, 2, 16, 16, 1.0, rot(8))


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
@pytest.mark.parametrize("name", sorted(CONFIGS))
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
@pytest.mark.parametrize("name", ["tiny", "mixed", "both"])
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
@pytest.mark.parametrize("decode", [False, True])
@pytest.mark.parametrize("window", [1, 2, 16, 47, 64, 130])
def test_window_edges(backend, decode, window):
    """The wanted key just inside and just outside the window, first of all, at page borders, right before the query --
    asked for from a prompt, from a short portion and from a decoded token."""
    cfg, w = needle_model("both", window)
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
        if at in at_edge and at < n - 2:                             # (the convolution shows the last token as well)
            assert (rel_err(want, base) > 0.2) == at_edge[at], (window, at)      # the key shows, or does not
        for cut in ((n - 1,) if decode else (0, n - 2, 150)):
            if cut:
                eng.feed([("a", toks[:cut], [])])
            got = eng.feed([("a", toks[cut:], [n - 1 - cut])], ["a"])
            assert close(got, want, backend), (at, cut)


@backends
@pytest.mark.parametrize("kind", ["tied", "conv", "shared"])
def test_one_far_key_among_hundreds(backend, kind):
    """Without a window every key stays in reach: the wanted one at the start, at page and tile borders, near the end."""
    cfg, w = needle_model(kind)
    eng = build(cfg, w, backend, max_tokens=1024)
    n = 530
    filler = [3 + t % (cfg.vocab - 3) for t in tokens(cfg, n, seed=32)]
    base = want_logits(cfg, w, filler[:-1] + [1])[-1:]
    for at in (0, 1, 15, 16, 127, 128, 255, 400, 511, 512, n - 3):
        toks = list(filler)
        toks[at], toks[n - 1] = 2, 1
        want = want_logits(cfg, w, toks)[-1:]
        assert rel_err(want, base) > 0.2
        for cut in (0, n - 1, n - 2, 300):
            if cut:
                eng.feed([("a", toks[:cut], [])])
            got = eng.feed([("a", toks[cut:], [n - 1 - cut])], ["a"])
            assert close(got, want, backend), (at, cut)


@backends
@pytest.mark.parametrize("kind", ["tied", "conv"])
def test_a_sink_takes_its_share(backend, kind):
    """A sink far below, level with and far above the best score."""
    cfg, w = needle_model(kind)
    toks = [3 + t % (cfg.vocab - 3) for t in tokens(cfg, 70, seed=33)]
    toks[20], toks[-1] = 2, 1
    seen = []
    for sink in (-30.0, 20.0, 80.0):
        w["l0.mix.sink"] = torch.full_like(w["l0.mix.sink"], sink)
        want = want_logits(cfg, w, toks)
        seen.append(want[-1:])
        eng = build(cfg, w, backend, max_tokens=256)
        assert close(feed_all(eng, "a", toks, [69, 1]), want, backend), sink
    assert rel_err(seen[2], seen[0]) > 0.2


@backends
def test_the_first_tokens_of_a_sequence(backend):
    """Zeros before the start for the convolutions, the empty state, a window that is not full: every length from one on."""
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
def test_a_state_remembers_a_far_token(backend):
    """Slow decays: a token far back changes the logits at the end, over portion borders and through long decoding."""
    cfg = DeluvikConfig(name="far", hidden=56, vocab=90, logit_cap=30.0, layers=(LayerSpec(both(4, lru=(48, 2, 3), scales=(0.1, 1.0))),))
    w = random_weights(cfg, seed=13)
    w["l0.mix.right.lam"] = torch.full_like(w["l0.mix.right.lam"], -9.0)
    w["l0.norm1"] *= 3.0
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
    """A prefix hit adopts pages and the snapshot of states and convolution inputs taken at the same boundary."""
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
    from tilerl_b200.models.deluvik import DeluvikModel
    save_checkpoint(DeluvikModel.from_tensors(cfg, w.__getitem__, "cpu", torch.float32), str(tmp_path))
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
    for edit in (lambda x: x.pop("l1.mix.right.conv.b"), lambda x: x.update({"l1.mlp.e3.up": x["l1.mlp.e3.up"][1:].contiguous()})):
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
    assert cli.main(["bench", "--model", "deluvik-tiny", "--device", "cpu", "--prompt-len", "12", "--gen", "3"]) == 0
    assert json.loads(capsys.readouterr().out)[0]["decode_tok_s"] > 0
    for flags in (["serve", "--dry-run"], ["bench", "--kernels"]):
        assert cli.main([flags[0], "--model", "deluvik-small", *flags[1:]]) == 0
        assert "attn" in capsys.readouterr().out or flags[0] == "serve"
    with pytest.raises(SystemExit):
        cli.main(["train", "--model", "deluvik-tiny", "--device", "cpu"])


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
