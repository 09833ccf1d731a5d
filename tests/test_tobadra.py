"""Tobadra through the framework's engine (pools, scheduler, captured ticks) against the plain oracle of ``tobadra_oracle.py``:
every schedule of the same tokens gives the same logits, on the CPU reference backend and on the GPU in fp32 and bf16."""
import json
import math

import pytest
import torch

import tobadra_oracle as oracle
from tobadra_cases import (BACKENDS, CONFIGS, TOL, _cfg, attn, backends, build, close, delta, feed_all, needle_model, random_weights, rel_err,
                           tokens, want_logits)
from tilerl_b200.config import TobadraConfig, config_from_dir, get_config
from tilerl_b200.engine import SamplingParams, StepLimits
from tilerl_b200.mixers import ChannelDeltaSpec, DenseSpec, LayerSpec, LightningSpec, MoeSpec, RouterSpec


@pytest.fixture(autouse=True, scope="module")
def _one_thread():
    """The reference backend's operations are too small to share among threads."""
    n = torch.get_num_threads()
    torch.set_num_threads(1)
    yield
    torch.set_num_threads(n)


# ---- mechanisms on their own (reference backend functions against the oracle) ---------------------------
def _g(seed):
    return torch.Generator().manual_seed(seed)


def _r(*shape, seed=0):
    return torch.randn(*shape, generator=_g(seed))


@pytest.mark.parametrize("dims,base", [(16, 10000.0), (2, 100.0), (40, 50.0)])
def test_rotation_of_keys_and_values(dims, base):
    from tilerl_b200.ops.ref_mixers import rotate_halves
    x = _r(6, 3, dims + 6)
    f = torch.tensor(attn(dims=dims, dim=dims, vdim=dims, base=base).value_frequencies(), dtype=torch.float64)
    for first in (0, 63, 70001):
        pos = torch.arange(first, first + 6)
        assert torch.allclose(rotate_halves(x, pos, f).double(), oracle.turn_halves(x.double(), base, dims, first=first), atol=1e-6)
        back = oracle.turn_halves(oracle.turn_halves(x.double(), base, dims, first=first), base, dims, -1.0, first)
        assert torch.allclose(back, x.double())
    assert attn(dims=4, dim=8, vdim=6, base=8.0).value_frequencies() == (1.0, 8.0 ** (-2 / 6), 8.0 ** (-4 / 6))


def test_turned_values_see_distances_only():
    """The weighted sum of turned values, turned back, is the same when every position moves by the same amount."""
    v, p = _r(7, 1, 12, seed=1).double(), torch.softmax(_r(7, seed=2).double(), 0)
    outs = []
    for first in (0, 40):
        s = torch.einsum("j,jhd->hd", p, oracle.turn_halves(v, 90.0, 12, first=first))
        outs.append(oracle.turn_halves(s[None], 90.0, 12, -1.0, first + 6))
    assert torch.allclose(outs[0], outs[1])


def test_attention_against_the_oracle():
    from tilerl_b200.ops.ref_mixers import softmax_attention
    q, k, v = _r(9, 6, 10, seed=1), _r(9, 2, 10, seed=2), _r(9, 2, 7, seed=3)
    for window in (1, 4, 50):
        want = oracle.attend(q.double(), k.double(), v.double(), 0.6, window)
        for i in range(9):
            lo = max(0, i + 1 - window)
            assert torch.allclose(softmax_attention(q[i], k[lo:i + 1], v[lo:i + 1], 0.6).double(), want[i], atol=1e-5)


def test_delta_rule_against_the_oracle():
    from tilerl_b200.ops.ref_mixers import delta_step, unit_heads
    n, q, v, b = 40, _r(40, 3, 8, seed=1), _r(40, 3, 5, seed=3), torch.sigmoid(_r(40, 3, seed=4))
    k, lg = unit_heads(_r(40, 3, 8, seed=2)), -torch.nn.functional.softplus(_r(40, 3, 8, seed=5) - 2)
    s, out = torch.zeros(3, 8, 5), []
    for t in range(n):
        s, o = delta_step(s, q[t], k[t], v[t], lg[t], b[t])
        out.append(o)
    want = oracle.scan_delta(q.double(), k.double(), v.double(), lg.double().exp(), b.double())
    assert torch.allclose(torch.stack(out).double(), want, atol=1e-5)
    # by hand: a full write replaces what the key finds; the read-out sees it; rows fade on their own
    s = torch.tensor([[[3.0], [5.0]]])
    s, o = delta_step(s, torch.tensor([[1.0, 1.0]]), torch.tensor([[1.0, 0.0]]), torch.tensor([[7.0]]), torch.tensor([[0.5, 0.2]]).log(), torch.ones(1))
    assert torch.allclose(s, torch.tensor([[[7.0], [1.0]]])) and math.isclose(float(o), 8.0, rel_tol=1e-6)
    assert torch.allclose(unit_heads(torch.tensor([3e-4, 4e-4])), torch.tensor([3e-4, 4e-4]) / math.sqrt(25e-8 + 1e-6))


def test_fixed_decay_by_hand():
    q, k, v = torch.ones(2, 1, 1), torch.ones(2, 1, 1), torch.tensor([[[2.0]], [[3.0]]])
    assert oracle.scan_fixed(q, k, v, torch.tensor([0.5])).flatten().tolist() == [2.0, 4.0]


ROUTERS = [(6, 2, RouterSpec(1.5, 2, 2, 1)), (12, 4, RouterSpec(0.7, 0, 4, 2)), (5, 1, RouterSpec(1.0, 3, 1, 1)), (70, 8, RouterSpec(2.0, 10, 40, 9)), (4, 4, RouterSpec())]


@pytest.mark.parametrize("experts,top,r", ROUTERS, ids=str)
def test_choice_of_experts_against_the_oracle(experts, top, r):
    from tilerl_b200.ops.ref_mixers import choose_grouped
    n = experts + r.identity
    z, c = 2 * _r(30, n, seed=1), 0.2 * _r(n, seed=2) - 0.3                # (most choice scores are negative)
    idx, weight = choose_grouped(z, c, top, r)
    j = {"groups": {"count": r.groups, "keep": r.keep}, "top": top, "scale": r.scale}
    want = oracle.route(z.double(), c.double(), j)
    assert torch.equal(idx, want[0]) and torch.allclose(weight.double(), want[1], atol=1e-6)
    assert (idx < n).all() and all(len(set(row.tolist())) == top for row in idx)


def test_router_by_hand():
    """The correction moves the choice and not the weight; a group counts by its best output; others cannot be chosen."""
    from tilerl_b200.ops.ref_mixers import choose_grouped
    z = torch.log(torch.tensor([[0.4, 0.1, 0.3, 0.2]]))
    got = choose_grouped(z, torch.zeros(4), 2, RouterSpec(2.0, 0, 2, 1))
    assert got[0].tolist() == [[0, 1]] and torch.allclose(got[1], torch.tensor([[0.8, 0.2]]))
    got = choose_grouped(z, torch.tensor([0.0, 0.0, -0.9, 0.5]), 2, RouterSpec(1.0, 0, 2, 1))
    assert got[0].tolist() == [[3, 2]] and torch.allclose(got[1], torch.tensor([[0.2, 0.3]]))
    got = choose_grouped(z, torch.tensor([-0.9, -0.9, -0.9, -0.9]), 2, RouterSpec(1.0, 0, 2, 2))
    assert got[0].tolist() == [[0, 2]]


def test_activations():
    from tilerl_b200.ops.ref_mixers import activate
    z = 3 * _r(50)
    for name, f in (("gelu", oracle.gelu_tanh), ("gelu_erf", oracle.gelu_erf), ("silu", oracle.silu)):
        assert torch.allclose(activate(z, name).double(), f(z.double()), atol=1e-6)
    assert float((oracle.gelu_erf(z.double()) - oracle.gelu_tanh(z.double())).abs().max()) > 1e-4


# ---- pages, states, parameters, configuration ------------------------------------------------------------
def test_attention_layers_have_caches_and_the_others_states():
    from tilerl_b200.kv import PackedKvPool, make_state_pool
    cfg = CONFIGS["mixed"]
    assert cfg.cache_owners == (1, 4) and cfg.owners == (1, 2, 3) and [cfg.source(i) for i in range(6)] == [3, 1, 2, 3, 1, 2]
    assert len(PackedKvPool(cfg, 5, dtype=torch.float32).pages) == 2
    pool = make_state_pool(cfg, 3, planes=4, ring_dtype=torch.float32)
    assert pool.recurrent and pool.ring_rows >= 4 + 4
    # every layer's input convolution, then the states: heads are padded to 16, the stream to 64
    assert [(l.kind, l.state_floats, l.conv_c) for l in pool.layouts] == 6 * [("input", 0, 64)] + [
        ("delta", 4 * 32 * 48, 448), ("lightning", 4 * 32 * 32, 0), ("delta", 4 * 32 * 48, 448), ("lightning", 4 * 32 * 32, 0)]
    s = pool.alloc_slot()
    for j, l in enumerate(pool.layouts):
        pool.ring_view(j, s).fill_(float(j + 1))
        if l.state_floats:
            pool.view(j, s, 2)[0].fill_(float(j + 1))
    for j, l in enumerate(pool.layouts):
        assert not l.conv_c or pool.ring_view(j, s).unique().tolist() == [float(j + 1)]
        assert not l.state_floats or pool.view(j, s, 2)[0].unique().tolist() == [float(j + 1)]
    assert not pool.states[s, 0].any()


def _again(cfg):
    from tilerl_b200.tobadra_layout import tensor_shapes
    return TobadraConfig.from_json(json.loads(json.dumps(cfg.to_json())), name=cfg.name, max_ctx=cfg.max_ctx, shapes=tensor_shapes(cfg))


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_served_parameters_hold_every_tensor_and_only_zeros_besides(name):
    from tilerl_b200.models.tobadra import TobadraModel
    cfg = CONFIGS[name]
    w = random_weights(cfg)
    m = TobadraModel.from_tensors(cfg, w.__getitem__, "cpu", torch.float32)
    got = dict(m.tensors())
    assert set(got) == set(w)
    for k, t in got.items():
        assert torch.equal(t, w[k]), k
    total = sum(float(t.double().pow(2).sum()) for t in w.values())
    assert math.isclose(sum(float(t.double().pow(2).sum()) for t in m.params.values()), total, rel_tol=1e-9)
    assert cfg.n_params() == sum(t.numel() for t in w.values())
    assert _again(cfg) == cfg
    again = TobadraModel.build_random(cfg, seed=3)
    assert set(dict(again.tensors())) == set(w)


def test_parameters_used_by_way_of_another_layer():
    cfg = CONFIGS["mixed"]
    j = cfg.to_json()
    j["layers"].append({**json.loads(json.dumps(j["layers"][0])), "weights_of": 0})            # layer 0 uses those of layer 3
    from tilerl_b200.tobadra_layout import tensor_shapes
    more = TobadraConfig.from_json(j, shapes=tensor_shapes(cfg))
    assert more.source(6) == 3 and more.owners == cfg.owners and tensor_shapes(more) == tensor_shapes(cfg)
    j["layers"][3]["weights_of"] = 6
    with pytest.raises(ValueError):
        TobadraConfig.from_json(j, shapes=tensor_shapes(cfg))


def test_configuration_refuses_what_it_does_not_know():
    from tilerl_b200.tobadra_layout import tensor_shapes
    cfg = CONFIGS["mixed"]
    j, shapes = cfg.to_json(), tensor_shapes(cfg)
    edits = (lambda d: d["layers"][1].update(type="latent_attention"), lambda d: d["layers"][1]["mixer"].update(sinks=4), lambda d: d.update(loop={}),
             lambda d: d["layers"][1]["mlp"].update(kind="switch"), lambda d: d["layers"][2]["mixer"].update(heads=3), lambda d: d["layers"][2]["mixer"]["decay"].append(0.5),
             lambda d: d["layers"][5]["mixer"].update(decay=[0.6, 0.9, 0.98, 1.5]), lambda d: d["layers"][1]["mixer"]["mask"].update(size=0),
             lambda d: d["layers"][0].update(weights_of=0), lambda d: d["layers"][0].update(weights_of=2), lambda d: d["layers"][4].update(weights_of=9),
             lambda d: d["layers"][1]["mixer"].update(kv_heads=3), lambda d: d["layers"][1]["mixer"]["rot"].update(dims=64), lambda d: d.pop("logit_scale"),
             lambda d: d["layers"][4]["mixer"].update(vdim=35), lambda d: d["layers"][3]["mixer"].pop("conv"), lambda d: d["canon"].update(taps=0),
             lambda d: d["layers"][1]["mixer"]["rot"].update(scaling={"factor": 2, "low": 1, "high": 4, "original": 64}),
             lambda d: d["layers"][3]["mlp"]["router"].update(top=49), lambda d: d["layers"][3]["mlp"]["router"]["groups"].update(keep=13),
             lambda d: d["layers"][3]["mlp"]["router"]["groups"].update(count=7), lambda d: d["layers"][3]["mlp"]["router"].pop("scale"),
             lambda d: d["layers"][3]["mlp"].pop("expert"))
    for edit in edits:
        bad = json.loads(json.dumps(j))
        edit(bad)
        with pytest.raises(ValueError):
            TobadraConfig.from_json(bad, shapes=shapes)
    with pytest.raises(ValueError):
        TobadraConfig.from_json(j)                                  # the ranks are not in the file
    assert get_config("tobadra-tiny").n_attn_layers == 1
    with pytest.raises(ValueError):
        attn(vdim=21)
    with pytest.raises(ValueError):
        MoeSpec(8, 4, 2, act="gelu_erf")                            # gated experts have no exact gelu
    with pytest.raises(ValueError):
        ChannelDeltaSpec(4, 3, 8, 8, 2, 4, 4)


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
@pytest.mark.parametrize("name", ["tiny", "mixed", "delta"])
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
    cfg, w = needle_model(window)
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
        if at in at_edge and at < n - 3:                             # (the input's convolution shows the last tokens as well)
            assert (rel_err(want, base) > 0.2) == at_edge[at], (window, at)      # the key shows, or does not
        for cut in ((n - 1,) if decode else (0, n - 2, 150)):
            if cut:
                eng.feed([("a", toks[:cut], [])])
            got = eng.feed([("a", toks[cut:], [n - 1 - cut])], ["a"])
            assert close(got, want, backend), (at, cut)


@backends
def test_one_far_key_among_hundreds(backend):
    """A wide window: the wanted key at the start, at page and tile borders, near the end."""
    cfg, w = needle_model(600)
    eng = build(cfg, w, backend, max_tokens=1024)
    n = 530
    filler = [3 + t % (cfg.vocab - 3) for t in tokens(cfg, n, seed=32)]
    base = want_logits(cfg, w, filler[:-1] + [1])[-1:]
    for at in (0, 15, 16, 127, 400, 511, n - 4):
        toks = list(filler)
        toks[at], toks[n - 1] = 2, 1
        want = want_logits(cfg, w, toks)[-1:]
        assert rel_err(want, base) > 0.2
        for cut in (0, n - 1, 300):
            if cut:
                eng.feed([("a", toks[:cut], [])])
            got = eng.feed([("a", toks[cut:], [n - 1 - cut])], ["a"])
            assert close(got, want, backend), (at, cut)


@backends
def test_the_values_turn(backend):
    """What a far key brings depends on how far it is: the same two tokens at other distances give other logits."""
    cfg, w = needle_model(600)
    eng = build(cfg, w, backend, max_tokens=256)
    seen = []
    for at in (10, 40):
        toks = [3 + t % (cfg.vocab - 3) for t in tokens(cfg, 90, seed=33)]
        toks[at], toks[-1] = 2, 1
        want = want_logits(cfg, w, toks)
        seen.append(want[-1:])
        assert close(feed_all(eng, "a", toks, [89, 1]), want, backend)
    assert rel_err(seen[1], seen[0]) > 0.2


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
@pytest.mark.parametrize("kind", ["lightning", "delta"])
def test_a_state_remembers_a_far_token(backend, kind):
    """Slow decays: a token far back changes the logits at the end, over portion borders and through long decoding."""
    mixer = LightningSpec(3, 24, 32, (1.0, 0.9995, 0.999)) if kind == "lightning" else delta(3, 3, 48, 32, 2)
    cfg = _cfg("far", [LayerSpec(mixer)])
    w = random_weights(cfg, seed=13)
    w["l0.norm1b"] = torch.ones_like(w["l0.norm1b"])
    if kind == "delta":                                     # nothing fades; writes are weak, so that they do not push each other out
        w["l0.mix.A_log"] = torch.full_like(w["l0.mix.A_log"], -9.0)
        w["l0.mix.b"] *= 0.2
    n = 260
    toks = tokens(cfg, n, seed=14)
    toks = [t if t != 5 else 6 for t in toks]
    for i in range(3, 13):
        toks[i] = 5
    other = [7 if t == 5 else t for t in toks]
    want, changed = want_logits(cfg, w, toks), want_logits(cfg, w, other)
    moved_by = rel_err(changed[-1:], want[-1:])
    assert moved_by > 0.01, moved_by
    eng = build(cfg, w, backend)
    for cuts in ([n], [64, 64, 64, 3], [37, 100, 1, 2, 100], [200, 1]):
        got, moved = feed_all(eng, "a", toks, cuts), feed_all(eng, "b", other, cuts)
        assert close(got, want, backend) and close(moved, changed, backend), cuts
        d = (moved[-1] - got[-1]).float().cpu()
        assert rel_err(d[None], (changed - want)[-1:]) < (0.02 if "bf16" not in backend else 1.0), cuts


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
    from tilerl_b200.models.tobadra import TobadraModel
    save_checkpoint(TobadraModel.from_tensors(cfg, w.__getitem__, "cpu", torch.float32), str(tmp_path))
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
    for edit in (lambda x: x.pop("l3.mix.k.conv"), lambda x: x.update({"l3.mlp.e3.up": x["l3.mlp.e3.up"][1:].contiguous()})):
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
    assert cli.main(["bench", "--model", "tobadra-tiny", "--device", "cpu", "--prompt-len", "12", "--gen", "3"]) == 0
    assert json.loads(capsys.readouterr().out)[0]["decode_tok_s"] > 0
    for flags in (["serve", "--dry-run"], ["bench", "--kernels"]):
        assert cli.main([flags[0], "--model", "tobadra-small", *flags[1:]]) == 0
        assert "attn" in capsys.readouterr().out or flags[0] == "serve"
    with pytest.raises(SystemExit):
        cli.main(["train", "--model", "tobadra-tiny", "--device", "cpu"])


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
