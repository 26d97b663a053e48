"""The Puposun configuration, description and plain statement, and whole models on the CPU with the plain kernel
statements in the kernels' place."""
from __future__ import annotations

import copy
import math

import pytest
import torch

import kernel_refs
import plain_puposun as pp
from helpers import cut, random_tokens, rel_err
from inferrs_b200.config.base import ConfigError
from inferrs_b200.engine.batch import StepEntry
from inferrs_b200.engine.loading import spec_from_config
from inferrs_b200.engine.model import ModelError, cache_needs, check_schedule, declared_tensors, side_state_needs
from inferrs_b200.engine.runner import ModelRunner
from inferrs_b200.parts.registry import part_class
from inferrs_b200.parts.spec import looped_schedule
from inferrs_b200.runtime import Runtime
from puposun_cases import CASE_A, CASE_B, CASE_C, CASE_D, CASES, experts, full, make_weights, model, random_case, windowed


def test_description_takes_every_size_from_the_configuration():
    spec, cfg = spec_from_config(CASE_A)
    assert spec.architecture == "Puposun" and spec.vocab_size == 211 and len(spec.layers) == 5 and spec.streams is None
    assert spec.embedding_scale == 3.0 and spec.logit_softcap == 9.0 and spec.lm_head == "head"
    assert [layer.arrangement for layer in spec.layers] == ["parallel"] * 5
    m = [layer.mixer for layer in spec.layers]
    assert [(x.n_heads, x.n_kv_heads, x.head_dim) for x in m] == [(6, 2, 24), (4, 4, 16), (6, 3, 32), (5, 1, 16), (8, 2, 40)]
    assert [(x.window, x.keep_first) for x in m] == [(23, 5), (17, 19), (None, 0), (None, 0), (40, 3)]
    assert [x.score_cap for x in m] == [None, None, 7.0, 30.0, None]
    assert [x.sink_score for x in m] == [None, None, 0.0, 0.0, None]
    assert all(x.value_is_key and x.v_proj is None for x in m)
    assert [x.head_gate for x in m] == ["l0.mix.g", "l1.mix.g", None, None, "l4.mix.g"]
    assert [x.o_bias for x in m] == [None, None, "l2.mix.o.b", "l3.mix.o.b", None]
    assert [(x.position.kind, x.position.rot_dim, x.position.theta) for x in m[1:3]] == [
        ("rotary_scaled_interleaved", 8, 500.0), ("rotary_scaled", 32, 100000.0)]
    f = [layer.ffn for layer in spec.layers]
    assert f[1] is None and [(x.top, len(x.experts), x.inner, x.groups, x.groups_keep, x.route_scale) for x in f if x] == [
        (2, 6, 40, 3, 2, 1.5), (3, 9, 24, 3, 1, 0.7), (1, 4, 72, 0, 0, 2.0), (4, 8, 16, 4, 3, 1.0)]
    assert all(len(layer.sublayers) == 1 or layer.sublayers[1].norm is None for layer in spec.layers)


def test_layers_are_passed_again_with_caches_of_their_own():
    spec, _ = spec_from_config(CASE_A)
    assert [e.layer for e in spec.schedule] == [0, 1, 2, 3, 1, 2, 3, 1, 2, 3, 4]
    assert [e.cache for e in spec.schedule] == list(range(11))
    assert [k for k, e in enumerate(spec.schedule) if e.add_embedding] == [4, 7]
    assert [e.layer for e in spec_from_config(CASE_B)[0].schedule] == [0]
    assert [(e.layer, e.add_embedding) for e in looped_schedule(3, 0, 1, 2, True)] == [(0, False), (0, True), (1, False), (2, False)]
    no_loop = copy.deepcopy(CASE_A)
    no_loop["loop"] = None
    assert [e.layer for e in spec_from_config(no_loop)[0].schedule] == [0, 1, 2, 3, 4]
    kv, states = cache_needs(spec)
    assert states == {} and side_state_needs(spec) == {} and sorted(kv) == list(range(11))
    assert (kv[4].n_kv_heads, kv[4].head_dim, kv[4].window, kv[4].keep_first, kv[4].planes) == (4, 16, 17, 19, 2)
    assert kv[1] == kv[4] == kv[7] and kv[2] == kv[5] == kv[8]


def test_tensor_names_and_shapes():
    spec, _ = spec_from_config(CASE_A)
    t = {d.name: tuple(d.shape) for d in declared_tensors(spec)}
    assert t["embed"] == t["head"] == (211, 96) and t["final.norm"] == t["l0.norm1"] == (96,) and "l0.norm2" not in t
    assert t["l0.mix.q"] == (144, 96) and t["l0.mix.k"] == (48, 96) and t["l0.mix.o"] == (96, 144) and t["l0.mix.g"] == (6, 96)
    assert t["l2.mix.q.b"] == (192,) and t["l2.mix.k.b"] == (96,) and t["l2.mix.o.b"] == (96,) and "l2.mix.g" not in t
    assert "l0.mix.q.b" not in t and not any(n.endswith(".v") for n in t)
    assert t["l2.mlp.e8.gate"] == t["l2.mlp.e8.up"] == (24, 96) and t["l2.mlp.e8.down"] == (96, 24)
    assert t["l2.mlp.router"] == (9, 96) and t["l2.mlp.correction"] == (9,) and "l1.mlp.router" not in t


@pytest.mark.parametrize("change,message", [
    (lambda c: c.pop("norm"), "lacks the keys"),
    (lambda c: c.pop("embedding"), "lacks the keys"),
    (lambda c: c["norm"].update(eps=0), "must be positive"),
    (lambda c: c["norm"].update(groups=2), "must be an object with 'eps'"),
    (lambda c: c["embedding"].update(norm=1), "must be an object with 'scale'"),
    (lambda c: c.update(logit_softcap=0), "logit_softcap must be positive"),
    (lambda c: c["loop"].update(stop=6), "the loop runs layers"),
    (lambda c: c["loop"].update(start=4), "the loop runs layers"),
    (lambda c: c["loop"].update(times=0), "the loop runs layers"),
    (lambda c: c["loop"].pop("times"), "'loop' must be"),
    (lambda c: c["layers"][1].update(type="attention_3"), "is not one of"),
    (lambda c: c["layers"][1].update(norm=2), "must be an object with"),
    (lambda c: c["layers"][1]["mixer"].update(softcap=3.0), "unknown or missing"),
    (lambda c: c["layers"][2]["mixer"].update(mask={"size": 3}), "unknown or missing"),
    (lambda c: c["layers"][2]["mixer"].update(softcap=-1.0), "softcap must be positive"),
    (lambda c: c["layers"][1]["mixer"].pop("scale"), "unknown or missing"),
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=3), "not a multiple"),
    (lambda c: c["layers"][1]["mixer"].update(vdim=8), "values are the keys"),
    (lambda c: c["layers"][1]["mixer"]["mask"].update(size=0), "positive 'size'"),
    (lambda c: c["layers"][1]["mixer"]["mask"].update(keep_first=-1), "positive 'size'"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=18), "even 'dims'"),
    (lambda c: c["layers"][0]["mlp"].update(kind="dense"), "kind 'moe'"),
    (lambda c: c["layers"][0]["mlp"]["expert"].update(ff=0), "positive 'ff'"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=7), "0 < top <= experts"),
    (lambda c: c["layers"][0]["mlp"]["router"].pop("scale"), "0 < top <= experts"),
    (lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(count=4), "equal groups"),
    (lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(keep=4), "equal groups"),
    (lambda c: c["layers"][2]["mlp"]["router"].update(top=4), "must hold the 4"),
])
def test_configurations_that_are_refused(change, message):
    c = copy.deepcopy(CASE_A)
    change(c)
    with pytest.raises(ConfigError, match=message):
        spec_from_config(c)


def test_an_unknown_key_at_the_top_is_named_and_ignored(capsys):
    spec, _ = spec_from_config(dict(CASE_A, seed=4))
    assert len(spec.layers) == 5 and "seed" in capsys.readouterr().err


def test_optional_keys_may_be_absent():
    c = copy.deepcopy(CASE_A)
    c["logit_softcap"] = None
    del c["layers"][2]["mixer"]["softcap"], c["layers"][2]["mixer"]["rot"], c["layers"][0]["mixer"]["mask"]
    spec, _ = spec_from_config(c)
    assert spec.logit_softcap is None and spec.layers[2].mixer.score_cap is None
    assert spec.layers[2].mixer.position.kind == "none" and spec.layers[0].mixer.window is None


def test_the_embedding_can_be_added_again_only_where_a_norm_takes_it():
    from dataclasses import replace
    spec, _ = spec_from_config(CASE_A)
    check_schedule(spec)
    with pytest.raises(ModelError, match="adds the embedding"):
        check_schedule(replace(spec, streams=2))
    odd = replace(spec.layers[1], arrangement="gated_residual")
    with pytest.raises(ModelError, match="adds the embedding"):
        check_schedule(replace(spec, layers=(spec.layers[0], odd) + spec.layers[2:]))


# ---------------------------------------------------------------------------------------------------
# the plain statement's own mechanisms, each against its definition written out number by number
# ---------------------------------------------------------------------------------------------------
def test_plain_rotations_turn_the_right_pairs():
    x = torch.arange(1.0, 9.0).view(1, 1, 8)
    pos, base, dims = torch.tensor([3]), 50.0, 6
    halves, neighbours = pp.rotate_halves(x, pos, base, dims)[0, 0], pp.rotate_neighbours(x, pos, base, dims)[0, 0]
    for i in range(3):
        a = 3 * base ** (-2 * i / 6)
        for out, (p, q) in ((halves, (i, i + 3)), (neighbours, (2 * i, 2 * i + 1))):
            u, v = float(x[0, 0, p]), float(x[0, 0, q])
            assert math.isclose(float(out[p]), u * math.cos(a) - v * math.sin(a), rel_tol=1e-5, abs_tol=1e-5)
            assert math.isclose(float(out[q]), v * math.cos(a) + u * math.sin(a), rel_tol=1e-5, abs_tol=1e-5)
    assert torch.equal(halves[6:], x[0, 0, 6:]) and torch.equal(neighbours[6:], x[0, 0, 6:])


def test_plain_masks_and_shares():
    see = pp.sees_window_and_first(9, 3, 2)
    assert [j for j in range(9) if see[7, j]] == [0, 1, 5, 6, 7] and [j for j in range(9) if see[1, j]] == [0, 1]
    assert [j for j in range(9) if pp.sees_window_and_first(9, 3, 0)[7, j]] == [5, 6, 7]
    s = torch.tensor([[0.3, -2.0, 1.1]])
    see = torch.tensor([[True, True, False]])
    total = 1.0 + math.exp(0.3) + math.exp(-2.0)
    assert torch.allclose(pp.shares_beside_a_zero_score(s, see), torch.tensor([[math.exp(0.3) / total, math.exp(-2.0) / total, 0.0]]))
    assert torch.allclose(pp.shares_beside_a_zero_score(s + 200, see).sum(), torch.tensor(1.0))
    assert math.isclose(float(pp.squashed(torch.tensor(50.0), 4.0)), 4.0, rel_tol=1e-6)


def test_plain_choice_of_experts():
    s = torch.tensor([[0.9, 0.1, 0.5, 0.6, 0.2, 0.3]])
    c = torch.tensor([-2.0, 0.0, -0.5, -0.4, 0.0, 0.0])
    # choice scores: -1.1, 0.1 | 0.0, 0.2 | 0.2, 0.3: the groups' worths are -1.0, 0.2, 0.5
    assert pp.chosen_experts(s, c, 2, {"count": 3, "keep": 1}) == [[5, 4]]
    assert pp.chosen_experts(s, c, 3, {"count": 3, "keep": 2})[0][0] == 5
    assert 0 not in pp.chosen_experts(s, c, 4, {"count": 3, "keep": 2})[0]
    # a negative choice score still beats an excluded expert
    assert set(pp.chosen_experts(s, c, 2, {"count": 3, "keep": 1})[0]) == {4, 5}
    low = c - 5.0
    assert set(pp.chosen_experts(s, low, 2, {"count": 3, "keep": 1})[0]) == {4, 5}
    assert pp.chosen_experts(s, torch.zeros(6), 2, None) == [[0, 3]]


def test_plain_order_of_layer_runs():
    assert pp.layer_runs(CASE_A) == [(0, False), (1, False), (2, False), (3, False), (1, True), (2, False), (3, False), (1, True),
                                     (2, False), (3, False), (4, False)]
    assert pp.layer_runs(CASE_B) == [(0, False)]


# ---------------------------------------------------------------------------------------------------
# tables and parts
# ---------------------------------------------------------------------------------------------------
def test_rotation_tables_are_made_in_double_precision():
    spec, _ = spec_from_config(CASE_C)
    p = spec.layers[1].mixer.position
    part = part_class("position", p)(p, Runtime(device=torch.device("cpu"), dtype=torch.float32))
    cos, sin, dims = part.tables()
    want_cos, want_sin = pp.angles(torch.arange(512), p.theta, p.rot_dim)
    assert dims == 32 and part.interleaved
    assert float((cos - want_cos).abs().max()) < 1e-7 and float((sin - want_sin).abs().max()) < 1e-7


# ---------------------------------------------------------------------------------------------------
# whole models: cache, schedule, batches and the block's joined products, without a GPU
# ---------------------------------------------------------------------------------------------------
def make_runner(case, w, n_pages, max_requests=3, page_size=16):
    spec, _ = spec_from_config(case)
    rt = Runtime(device=torch.device("cpu"), dtype=torch.float32)
    return ModelRunner(spec, dict(w), rt, page_size=page_size, n_pages=n_pages, max_requests=max_requests)


@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
def test_cuttings_and_batches_on_the_cpu(monkeypatch, name):
    kernel_refs.install(monkeypatch)
    case, w = CASES[name], make_weights(CASES[name], 5)
    toks = random_tokens(52, case["vocab"], seed=2)
    other = random_tokens(30, case["vocab"], seed=3)
    want, want_other = pp.forward(case, w, toks), pp.forward(case, w, other)
    page_size = 4 if name == "A" else 16
    runner = make_runner(case, w, n_pages=104 // page_size + 2, page_size=page_size)
    runner.admit("a")
    assert rel_err(runner.step([StepEntry("a", toks, list(range(52)))]), want) < 1e-4
    runner.release("a")
    runner.admit("b")
    runner.admit("c")
    at, o_at, rows, o_rows = 0, 0, [], []
    for n in cut(52, [7, 2, 13, 1, 1, 2]):
        entries = [StepEntry("b", toks[at:at + n], list(range(n)))]
        if o_at < 30:
            entries.append(StepEntry("c", other[o_at:o_at + 5], list(range(5))))
        out = runner.step(entries)
        rows.append(out[:n])
        o_rows.append(out[n:])
        at, o_at = at + n, o_at + 5
        runner.manager.check_invariants()
    assert rel_err(torch.cat(rows), want) < 1e-4 and rel_err(torch.cat(o_rows), want_other) < 1e-4


@pytest.mark.parametrize("seed", range(10))
def test_configurations_drawn_at_random_on_the_cpu(monkeypatch, seed):
    kernel_refs.install(monkeypatch)
    case = random_case(seed)
    w = make_weights(case, 50 + seed)
    toks = random_tokens(60, case["vocab"], seed=seed)
    want = pp.forward(case, w, toks)
    runner = make_runner(case, w, n_pages=4, max_requests=1)
    runner.admit(0)
    rows, at = [], 0
    for n in cut(60, [19, 2, 1, 11]):
        rows.append(runner.step([StepEntry(0, toks[at:at + n], list(range(n)))]))
        at += n
    assert rel_err(torch.cat(rows), want) < 1e-4


def test_sublayers_that_do_not_join_their_products_run_one_by_one(monkeypatch):
    kernel_refs.install(monkeypatch)
    from inferrs_b200.parts.attention import Attention
    case, w = CASE_A, make_weights(CASE_A, 6)
    monkeypatch.setattr(Attention, "joins_products", lambda self: False)
    toks = random_tokens(40, case["vocab"], seed=4)
    runner = make_runner(case, w, n_pages=8)
    assert not any(b.joined for b in runner.model.blocks)
    runner.admit(0)
    got = runner.step([StepEntry(0, toks, list(range(40)))])
    # (an output bias is added to the sub-layer's own rows then)
    assert rel_err(got, pp.forward(case, w, toks)) < 1e-4
