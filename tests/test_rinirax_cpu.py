"""Rinirax without a GPU: configuration, tensor names, what its layers ask of the cache manager, the
frequency table, and the plain implementation's mechanisms on hand-made inputs."""

from __future__ import annotations

import math

import pytest
import torch

import rinirax_configs as rc
import rinirax_plain as plain
from mlx_omnia_b200.config.hydrate import ConfigError
from mlx_omnia_b200.kernels import ops
from mlx_omnia_b200.parts.base import KVSpec, PartSpec, Runtime
from mlx_omnia_b200.parts.blocks import ParallelBlock
from mlx_omnia_b200.parts.feedforward import RoutedExperts
from mlx_omnia_b200.parts.model import DecoderModel
from mlx_omnia_b200.parts.positions import Rotary
from mlx_omnia_b200.registry import resolve_architecture

F64 = torch.float64


def _model(name):
    raw = rc.config(name)
    architecture = resolve_architecture(raw)
    return raw, architecture, rc.tensors(name), DecoderModel(architecture.model_spec(architecture.parse(raw)))


@pytest.mark.parametrize("name", sorted(rc.CONFIGS))
def test_names_and_shapes_match_the_random_checkpoint(name):
    raw, architecture, drawn, model = _model(name)
    declared = model.tensors()
    assert {architecture.tensor_name(k) for k in drawn} == set(declared)
    for k, t in drawn.items():
        assert tuple(t.shape) == tuple(declared[architecture.tensor_name(k)].shape), k
    for i, layer in enumerate(raw["layers"]):
        assert drawn[f"l{i}.dwa"].shape == (i + 2,)
        if layer["type"] == "attention":
            reads = "kv_from" in layer["mixer"]
            for part in ("k", "v"):
                for suffix in ("", ".b", ".conv"):
                    assert (f"l{i}.mix.{part}{suffix}" in drawn) == (not reads)
        assert (f"l{i}.mlp.act" in drawn) == (layer["mlp"] is not None and layer["mlp"]["kind"] == "dense")


def test_what_the_layers_ask_of_the_cache():
    _, _, _, model = _model("S")
    needs = model.cache_needs()
    assert needs[0].kv == KVSpec(((2, 40), (2, 40))) and needs[0].state["conv"].shape == (3, 6 * 32 + 2 * 32 + 2 * 40)
    assert needs[1].kv is None and needs[1].state.shape == (72,)
    assert needs[2].kv == KVSpec(((1, 48),), 9) and needs[2].state is None
    assert needs[3].kv is None and needs[3].reads == 0 and needs[3].state["conv"].shape == (1, 4 * 32)
    _, _, _, model = _model("W")
    needs = model.cache_needs()
    assert needs[0].kv == KVSpec(((1, 26),)) and needs[1].kv == KVSpec(((3, 16), (3, 16)))
    _, _, _, model = _model("T")
    assert model.cache_needs()[4].state["conv"].shape[0] == 1  # a single tap keeps no inputs; the slot has a row


def test_named_errors():
    architecture = resolve_architecture(rc.config("S"))

    def broken(change):
        raw = rc.config("S")
        change(raw)
        return raw

    for change, word in [(lambda c: c["layers"][3]["mixer"].update(kv_from=1), "kv_from"),
                         (lambda c: c["layers"][3]["mixer"].update(kv_from=3), "kv_from"),
                         (lambda c: c["layers"][3]["mixer"]["rot"].update(base=301.0), "kv_from"),
                         (lambda c: c["layers"][0]["mixer"].update(kv_heads=4), "heads"),
                         (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=18), "dims"),
                         (lambda c: c["layers"][2]["mixer"].pop("q_rank"), "q_rank"),
                         (lambda c: c["layers"][2]["mixer"]["rot"]["scaling"].pop("slow"), "slow"),
                         (lambda c: c["layers"][2]["mixer"]["mask"].update(size=0), "size"),
                         (lambda c: c["layers"][0]["mlp"]["router"].update(top=7), "experts"),
                         (lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(count=5), "groups"),
                         (lambda c: c["layers"][2]["mlp"].update(kind="other"), "unknown kind"),
                         (lambda c: c["layers"][1].update(type="other"), "unknown type"),
                         (lambda c: c.pop("vocab"), "vocab")]:
        with pytest.raises(ConfigError, match=word):
            architecture.parse(broken(change))


@pytest.mark.parametrize("dims,base,scaling", [(48, 3e5, (6.0, 1024, 20.0, 2.0)), (6, 100.0, None), (16, 500.0, (8.0, 64, 16.0, 0.5)),
                                               (64, 10000.0, (40.0, 4096, 32.0, 1.0)), (8, 20.0, (3.0, 16, 1.0, 1.0))])
def test_the_frequency_table(dims, base, scaling):
    part = Rotary(dims, base, "half", scaling)
    part.load({}, Runtime(torch.float32, torch.device("cpu")))
    keys = dict(zip(("factor", "original", "fast", "slow"), scaling)) if scaling else None
    f, amount = plain.frequencies(dims, base, keys, F64)
    assert torch.equal(part.table(), f.to(torch.float32)) and part.amount == pytest.approx(amount, rel=1e-15)
    if scaling:
        unscaled = plain.frequencies(dims, base, None, F64)[0]
        assert bool((f <= unscaled * (1 + 1e-12)).all()) and float((f / unscaled).min()) >= 1 / scaling[0] - 1e-12
    with pytest.raises(ValueError):
        Rotary(dims, base, "half", (0.0, 1.0, 1.0, 1.0))


def test_mixers_that_do_not_scale_the_turn_refuse_it():
    from mlx_omnia_b200.parts.base import MIXERS

    scaled = PartSpec("rotary", {"dims": 4, "theta": 100.0, "scaling": (2.0, 64.0, 8.0, 1.0)})
    for spec in (PartSpec("gqa_attention", {"hidden": 16, "heads": 2, "kv_heads": 1, "head_dim": 8, "scale": 1.0, "position": scaled}),
                 PartSpec("sink_window_attention", {"hidden": 16, "heads": 2, "kv_heads": 1, "dim": 8, "vdim": 8, "scale": 1.0,
                                                    "position": scaled}),
                 PartSpec("gated_state_attention", {"hidden": 16, "heads": 2, "dim": 8, "vdim": 8, "norm_eps": 1e-5,
                                                    "decay": (0.5, 0.9), "position": scaled})):
        with pytest.raises(ValueError, match="cosine"):
            MIXERS.build(spec)


def test_a_depth_average_fits_its_model():
    norm = PartSpec("layer_norm", {"size": 8, "eps": 1e-5})
    mixer = PartSpec("min_gru", {"hidden": 8, "width": 4})
    assert "dwa" not in ParallelBlock(mixer, None, norm).tensors()
    assert ParallelBlock(mixer, None, norm, 2, 3).tensors()["dwa"].shape == (3,)
    with pytest.raises(ValueError, match="depth"):
        ParallelBlock(mixer, None, norm, 4, 3)
    with pytest.raises(ValueError, match="groups"):
        RoutedExperts(8, 4, 6, 3, groups=3, keep_groups=1)


def test_the_recurrence_over_a_cut_in_closed_form_and_at_its_ends():
    g = torch.Generator().manual_seed(1)
    z, u = (torch.randn(23, 5, generator=g, dtype=F64) * 2 for _ in range(2))
    whole = plain.min_gru_states(z, u)
    first = plain.min_gru_states(z[:9], u[:9])
    assert torch.allclose(torch.cat([first, plain.min_gru_states(z[9:], u[9:], first[-1])]), whole)
    keep, cand = torch.sigmoid(-z), torch.where(u >= 0, u + 0.5, torch.sigmoid(u))
    want = sum(keep[j + 1: 12].prod(0) * torch.sigmoid(z[j]) * cand[j] for j in range(12))
    assert torch.allclose(whole[11], want)
    near = plain.min_gru_states(torch.full((1, 2), 50.0, dtype=F64), torch.tensor([[1e-12, -1e-12]], dtype=F64))
    assert torch.allclose(near, torch.full((1, 2), 0.5, dtype=F64))  # the candidate is continuous at zero


def test_two_equal_maps_leave_one_minus_lambda():
    g = torch.Generator().manual_seed(2)
    q, k, v = (torch.randn(7, 1, *s, generator=g, dtype=F64) for s in ((2, 4), (2, 4), (6,)))
    q[:, :, 1], k[:, :, 1] = q[:, :, 0], k[:, :, 0]
    one = plain.softmax_map(q[:, 0, 0], k[:, 0, 0], v[:, 0], 0.5)
    got = plain.differential_heads(q, k, v, 0.5, 3.0, 0.2, 0.0)[:, 0]
    assert torch.allclose(got, -plain.rms(one, 0.0) * 0.8)  # one - 3 one = -2 one, its size normed away


def test_a_window_sees_its_first_position_and_not_the_one_before():
    g = torch.Generator().manual_seed(3)
    T, w = 20, 6
    q, k, v = (torch.randn(T, d, generator=g, dtype=F64) for d in (4, 4, 3))
    base = plain.softmax_map(q, k, v, 1.0, w)
    for j in (0, 7):
        moved = v.clone()
        moved[j] += 1.0
        changed = ((plain.softmax_map(q, k, moved, 1.0, w) - base).abs().amax(-1) > 0).nonzero().flatten().tolist()
        assert changed == list(range(j, j + w))


def test_groups_are_ranked_by_their_two_best_and_others_cannot_be_chosen():
    r = {"experts": 6, "top": 2, "groups": {"count": 3, "keep": 1}, "scale": 2.0}
    s = torch.tensor([[0.9, 0.1, 0.6, 0.55, 0.2, 0.3]], dtype=F64)
    z = torch.log(s / (1 - s))
    chosen, w = plain.route(z, torch.zeros(6), r)
    assert sorted(chosen[0].tolist()) == [2, 3]  # 0.6 + 0.55 beats 0.9 + 0.1: the largest expert is not chosen
    assert torch.allclose(w.sum(), torch.tensor(2.0, dtype=F64))
    # Choice scores below zero: what is shut out is minus infinity, not zero.
    chosen, w = plain.route(z, torch.full((6,), -5.0), r)
    assert sorted(chosen[0].tolist()) == [2, 3]
    correction = torch.tensor([0.0, 0.0, 0.0, 0.0, 1.0, 1.0])
    chosen, w = plain.route(z, correction, r)
    assert sorted(chosen[0].tolist()) == [4, 5]  # chosen by the corrected score, weighted by the score itself
    assert torch.allclose(w[0].sort().values, torch.tensor([0.8, 1.2], dtype=F64))


def test_xielu_is_continuous_and_has_its_slopes():
    p, q = torch.tensor(0.3, dtype=F64), torch.tensor(-0.7, dtype=F64)
    z = torch.tensor([-1e-6, 0.0, 1e-6], dtype=F64, requires_grad=True)
    y = plain.xielu(z, p, q)
    assert torch.allclose(y, 0.5 * z, atol=1e-11)
    y.sum().backward()
    assert torch.allclose(z.grad, torch.full((3,), 0.5, dtype=F64), atol=1e-5)
    big = plain.xielu(torch.tensor([3.0, -30.0], dtype=F64), p, q)
    assert big[0] == pytest.approx(math.log1p(math.exp(0.3)) * 9 + 1.5)
    assert big[1] == pytest.approx((0.5 + math.log1p(math.exp(-0.7))) * 29.0 - 15.0)


def test_the_segments_a_portion_is_cut_into():
    for longest, channels, requests in [(1, 64, 1), (17, 32, 3), (2048, 2048, 1), (100000, 40, 1), (300, 4096, 64)]:
        warps, cluster = ops.mingru_segments(longest, channels, requests, 148)
        assert 1 <= warps <= ops.MINGRU_MAX_WARPS and cluster in (1, 2, 4, 8)
    assert ops.mingru_segments(2048, 2048, 1, 148) == (16, 8) and ops.mingru_segments(300, 4096, 64, 148)[1] == 1
