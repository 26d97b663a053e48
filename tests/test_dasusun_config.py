"""The Dasusun configuration, description and plain statement, without a GPU."""
from __future__ import annotations

import copy
import math

import pytest
import torch

import plain_dasusun as pd
from dasusun_cases import CASE_A, CASE_B, CASE_D, CASES, latent, make_weights, model
from helpers import random_tokens, rel_err
from inferrs_b200.config.base import ConfigError
from inferrs_b200.engine.loading import spec_from_config
from inferrs_b200.engine.model import ModelError, cache_needs, check_schedule, declared_tensors, side_state_needs
from inferrs_b200.parts.registry import part_class
from inferrs_b200.parts.spec import DepthAverageSpec
from inferrs_b200.runtime import Runtime


def test_description_takes_every_size_from_the_configuration():
    spec, cfg = spec_from_config(CASE_A)
    assert spec.architecture == "Dasusun" and spec.vocab_size == 211 and len(spec.layers) == 4 and spec.streams is None
    assert [layer.arrangement for layer in spec.layers] == ["sandwich"] * 4
    assert [layer.depth_average.results for layer in spec.layers] == [2, 3, 4, 5]
    assert spec.lm_head == spec.embedding == "embed" and spec.final_norm.weight_offset == 1.0
    m = [layer.mixer for layer in spec.layers]
    assert [x.window for x in m] == [23, 50, None, 31] and all(x.gate_proj is None for x in m)
    assert (m[0].n_heads, m[0].key_dim, m[0].rot_dim, m[0].value_dim, m[0].q_rank, m[0].kv_rank) == (6, 24, 12, 20, 36, 40)
    assert m[0].scale == 0.17 and m[0].eps == 1e-5
    assert m[0].position.scaling == (4.0, 64.0, 32.0, 1.0) and m[1].position.scaling is None
    assert m[0].position.rot_dim == 12 and m[0].position.theta == 10000.0 and m[3].position.theta == 10000.0
    assert [layer.ffn.inner if layer.ffn else None for layer in spec.layers] == [72, None, 50, 136]
    first = spec.layers[0].sublayers
    assert first[0].input_conv.taps == 4 and first[0].input_conv.width == 96 and first[1].input_conv is None
    assert all(s.norm.weight_offset == s.post_norm.weight_offset == 1.0 for layer in spec.layers for s in layer.sublayers)
    assert [s.layer_scale for s in first] == ["l0.ls1", "l0.ls2"] and len(spec.layers[1].sublayers) == 1


def test_caches_and_states():
    spec, _ = spec_from_config(CASE_A)
    kv, states = cache_needs(spec)
    assert states == {} and sorted(kv) == [0, 1, 2, 3]
    # one plane: the latent padded to 32 numbers and the rotated part padded to 16
    assert [(kv[i].planes, kv[i].n_kv_heads, kv[i].head_dim, kv[i].window) for i in range(4)] == \
        [(1, 1, 64 + 16, 23), (1, 1, 64 + 16, 50), (1, 1, 96 + 16, None), (1, 1, 32 + 32, 31)]
    side = side_state_needs(spec)
    assert sorted(cid for cid, _ in side) == [0, 1, 2, 3] and all(need.shape == (3 * 96,) for need in side.values())
    assert side_state_needs(spec_from_config(CASE_B)[0]) == {}      # one tap keeps nothing


def test_tensor_names_and_shapes():
    spec, _ = spec_from_config(CASE_A)
    t = {d.name: tuple(d.shape) for d in declared_tensors(spec)}
    assert t["embed"] == (211, 96) and "head" not in t and t["final.norm"] == (96,)
    assert t["l0.mix.dq"] == (36, 96) and t["l0.mix.dq.norm"] == (36,) and t["l0.mix.uq"] == (6 * 36, 36)
    assert t["l0.mix.dkv"] == (52, 96) and t["l0.mix.dkv.norm"] == (40,)
    assert t["l0.mix.uk"] == (144, 40) and t["l0.mix.uv"] == (120, 40) and t["l0.mix.o"] == (96, 120)
    assert t["l0.mlp.up"] == (72, 96) and t["l0.mlp.down"] == (96, 72) and "l0.mlp.gate" not in t
    assert t["l0.canon1"] == (96, 4) and [t[f"l{i}.dwa"] for i in range(4)] == [(2,), (3,), (4,), (5,)]
    assert all(t[f"l0.{n}"] == (96,) for n in ("norm1", "norm1b", "ls1", "norm2", "norm2b", "ls2"))
    assert not any(f"l1.{n}" in t for n in ("norm2", "norm2b", "ls2", "mlp.up"))
    # weight files that hold some of a second sub-layer's tensors for a layer without one: declared, and nothing runs
    spec2, _ = spec_from_config(CASE_A, tensor_shapes={"l1.norm2": (96,), "l1.ls2": (96,)})
    assert {d.name for d in declared_tensors(spec2)} - set(t) == {"l1.norm2", "l1.ls2"}
    assert len(spec2.layers[1].sublayers) == 1


@pytest.mark.parametrize("change,message", [
    (lambda c: c.pop("norm"), "lacks the keys"),
    (lambda c: c.pop("canon"), "lacks the keys"),
    (lambda c: c["canon"].update(taps=0), "positive 'taps'"),
    (lambda c: c["norm"].update(eps=0), "must be positive"),
    (lambda c: c["norm"].update(groups=2), "'norm' must be"),
    (lambda c: c["layers"][1].update(type="attention"), "is not 'latent_attention'"),
    (lambda c: c["layers"][1].update(loop=2), "must be an object with"),
    (lambda c: c["layers"][1]["mixer"].update(gate=True), "unknown or missing"),
    (lambda c: c["layers"][1]["mixer"].pop("scale"), "unknown or missing"),
    (lambda c: c["layers"][1]["mixer"].pop("rot"), "unknown or missing"),
    (lambda c: c["layers"][1]["mixer"].update(q_rank=0), "must be positive"),
    (lambda c: c["layers"][1]["mixer"]["mask"].update(size=0), "positive 'size'"),
    (lambda c: c["layers"][1]["mixer"]["mask"].update(first=4), "positive 'size'"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=7), "even 'dims'"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=10), "even 'dims'"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(base=1.0), "'base' above 1"),
    (lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].pop("slow"), "rot.scaling must give"),
    (lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].update(factor=-1.0), "rot.scaling must give"),
    (lambda c: c["layers"][0]["mlp"].update(kind="gated"), "of kind 'dense'"),
    (lambda c: c["layers"][0]["mlp"].update(ff=0), "of kind 'dense'"),
    (lambda c: c.update(eos_token_id=211), "inside the vocabulary"),
])
def test_configurations_that_are_refused(change, message):
    c = copy.deepcopy(CASE_A)
    change(c)
    with pytest.raises(ConfigError, match=message):
        spec_from_config(c)


def test_unknown_key_at_the_top_is_named_and_ignored(capsys):
    spec_from_config(dict(CASE_B, seed=5))
    assert "['seed']" in capsys.readouterr().err


def test_random_weights_cover_every_declared_tensor():
    from inferrs_b200.weights.random_init import random_weights
    spec, _ = spec_from_config(CASE_D)
    w = random_weights(declared_tensors(spec), 3, torch.float32, torch.device("cpu"))
    assert set(w) == {d.name for d in declared_tensors(spec)}
    assert abs(float(w["l0.norm1"].mean())) < 0.05 and abs(float(w["l0.ls1"].mean()) - 1.0) < 0.2
    assert bool(torch.isfinite(pd.forward(CASE_D, w, random_tokens(9, 77, seed=1))).all())


def test_the_rotation_tables_follow_the_stretch():
    """The product's tables against the plain frequencies: a stretch in the middle of the pairs, one that leaves every
    pair as it is, one that reaches every pair, none."""
    rt = Runtime(torch.device("cpu"), torch.float32)
    for case in CASES.values():
        for layer, described in zip(case["layers"], spec_from_config(case)[0].layers):
            pos = described.mixer.position
            cos, sin, dims = part_class("position", pos)(pos, rt).tables()
            f, factor = pd.frequencies(layer["mixer"]["rot"])
            p = torch.tensor([0, 1, 7, 100, min(4000, cos.shape[0] - 1)])
            ang = p.double()[:, None] * f[None, :]
            assert dims == layer["mixer"]["rot"]["dims"]
            assert float((cos[p].double() - torch.cos(ang) * factor).abs().max()) < 1e-6
            assert float((sin[p].double() - torch.sin(ang) * factor).abs().max()) < 1e-6


def test_an_average_over_depth_that_does_not_fit_the_schedule_is_refused():
    from dataclasses import replace
    spec, _ = spec_from_config(CASE_A)
    layers = list(spec.layers)
    layers[1] = replace(layers[1], depth_average=DepthAverageSpec(weight="l1.dwa", results=4))
    with pytest.raises(ModelError, match="averages the 3 results"):
        check_schedule(replace(spec, layers=tuple(layers)))
    with pytest.raises(ModelError, match="averages the 3 results"):      # a layer that runs twice
        check_schedule(replace(spec, schedule=(spec.schedule[0],) + spec.schedule))


# ---- the plain statement itself: every mechanism moves the logits as it should -----------------------------------
@pytest.mark.parametrize("name", ["l0.norm1", "l0.norm1b", "l0.ls1", "l2.norm2", "l2.norm2b", "l2.ls2", "l0.canon1", "l1.dwa",
                                  "l2.mix.dq.norm", "l2.mix.dkv.norm", "final.norm", "l2.mix.uk", "l0.mix.uv"])
def test_every_tensor_of_the_plain_statement_moves_the_logits(name):
    case, w = CASE_A, make_weights(CASE_A, 3)
    toks = random_tokens(40, case["vocab"], seed=2)
    base = pd.forward(case, w, toks)[-1]
    w2 = dict(w)
    bump = torch.zeros_like(w[name])
    bump.view(-1)[::2] = 0.3
    w2[name] = w[name] + bump
    assert float((pd.forward(case, w2, toks)[-1] - base).abs().max()) > 1e-3


def test_plain_layer_sees_its_window_and_no_further():
    """One layer alone: a token beyond the window changes nothing, the last one inside it does; the convolution in
    front of the mixer reaches taps - 1 tokens further."""
    case = model(50, 32, 1e-5, 3, [latent(2, 8, 4, 8, 16, 16, 0.3, 100.0, 9)])
    w = make_weights(case, 4)
    toks = random_tokens(40, 50, seed=5)
    base = pd.forward(case, w, toks)[-1]
    reach = 9 + 2
    for back, seen in ((reach - 1, True), (reach, False), (reach + 5, False)):
        t2 = list(toks)
        t2[39 - back] = (t2[39 - back] + 7) % 50
        assert (float((pd.forward(case, w, t2)[-1] - base).abs().max()) > 1e-6) == seen, back


def test_plain_rotation_depends_on_distance_alone_and_the_stretch_slows_pairs():
    rot = {"base": 1000.0, "dims": 8, "scaling": {"factor": 4.0, "original": 64, "fast": 4.0, "slow": 0.5}}
    g = torch.Generator().manual_seed(1)
    q, k = torch.randn(1, 1, 8, generator=g).double(), torch.randn(1, 1, 8, generator=g).double()
    dot = lambda i, j: float((pd.rotate(q, torch.tensor([i]), rot) * pd.rotate(k, torch.tensor([j]), rot)).sum())   # noqa: E731
    assert abs(dot(30, 20) - dot(130, 120)) < 1e-9 and abs(dot(30, 20) - dot(30, 21)) > 1e-3
    f, factor = pd.frequencies(rot)
    plain, one = pd.frequencies({"base": 1000.0, "dims": 8})
    assert one == 1.0 and abs(factor - (0.1 * math.log(4.0) + 1.0)) < 1e-12
    ratio = f / plain
    assert float(ratio[0]) == 1.0 and abs(float(ratio[-1]) - 0.25) < 1e-12 and bool((ratio[1:] <= ratio[:-1]).all())


def test_plain_average_over_depth_and_centred_norm():
    rows = [torch.randn(3, 4) for _ in range(3)]
    assert torch.allclose(pd.depth_average(rows, torch.tensor([0.0, 0.0, 1.0])), rows[2])
    assert torch.allclose(pd.depth_average(rows, torch.tensor([1.0, -2.0, 0.5])), rows[0] - 2 * rows[1] + 0.5 * rows[2])
    x = torch.randn(5, 8)
    assert torch.allclose(pd.centred_norm(x, torch.zeros(8), 1e-6), pd.divided_by_rms(x, 1e-6))
    assert rel_err(pd.centred_norm(x, torch.full((8,), -1.0), 1e-6) + x, x) == 0.0


def test_plain_convolution_starts_from_zeros():
    x, w = torch.randn(5, 2), torch.tensor([[0.5, -1.0, 2.0], [1.0, 0.0, 0.0]])
    y = pd.causal_conv(x, w)
    assert torch.allclose(y[0], torch.tensor([2.0, 0.0]) * x[0])
    assert torch.allclose(y[4], torch.stack([0.5 * x[2, 0] - x[3, 0] + 2 * x[4, 0], x[2, 1]]))


@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
def test_float64_bounds_float32(name):
    case, w = CASES[name], make_weights(CASES[name], 9)
    toks = random_tokens(24, case["vocab"], seed=1)
    assert rel_err(pd.forward(case, w, toks), pd.forward(case, w, toks, torch.float64)) < 5e-5
