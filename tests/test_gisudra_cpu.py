"""Gisudra without a GPU: configuration, tensor names, what its layers ask of the cache manager, the plans
made on the host, and the plain implementation's mechanisms on hand-made inputs."""

from __future__ import annotations

import math

import pytest
import torch

import gisudra_configs as gc
import gisudra_plain as plain
from mlx_omnia_b200.config.hydrate import ConfigError
from mlx_omnia_b200.kernels import ops
from mlx_omnia_b200.parts.attention import LatentAttention, SinkWindowAttention
from mlx_omnia_b200.parts.base import KVSpec, PartSpec
from mlx_omnia_b200.parts.blocks import PreNormBlock
from mlx_omnia_b200.parts.feedforward import GLUMLP, RoutedExperts
from mlx_omnia_b200.parts.model import DecoderModel
from mlx_omnia_b200.parts.recurrent import StateSpace
from mlx_omnia_b200.registry import resolve_architecture

F64 = torch.float64


def _model(name):
    raw = gc.config(name)
    architecture = resolve_architecture(raw)
    return raw, architecture, gc.tensors(name), DecoderModel(architecture.model_spec(architecture.parse(raw)))


@pytest.mark.parametrize("name", sorted(gc.CONFIGS))
def test_names_and_shapes_match_the_random_checkpoint(name):
    raw, architecture, drawn, model = _model(name)
    declared = model.tensors()
    assert {architecture.tensor_name(k) for k in drawn} == set(declared)
    for k, t in drawn.items():
        assert tuple(t.shape) == tuple(declared[architecture.tensor_name(k)].shape), k
    for i, layer in enumerate(raw["layers"]):
        assert (f"l{i}.norm2" in drawn) == (layer["mlp"] is not None)
        assert (f"l{i}.mix.vmix" in drawn) == bool(layer["mixer"].get("v_mix"))
        if layer["type"] == "mamba2":
            m = layer["mixer"]
            assert drawn[f"l{i}.mix.in"].shape[0] == 2 * m["heads"] * m["vdim"] + 2 * m["groups"] * m["state"] + m["heads"]


def test_what_the_layers_ask_of_the_cache():
    _, _, _, model = _model("G")
    needs = model.cache_needs()
    assert needs[0].kv == KVSpec(((2, 16), (2, 24)), 11, keep_first=5) and needs[0].state is None
    assert needs[1].kv is None and needs[1].state["S"].shape == (6, 24, 20) and needs[1].state["conv"].shape == (1, 6 * 20 + 96)
    assert needs[2].kv == KVSpec(((4, 16), (4, 16)), 30) and needs[3].kv == KVSpec(((1, 48),), 9)
    _, _, _, model = _model("H")
    needs = model.cache_needs()
    assert needs[5].kv == KVSpec(((2, 32), (2, 32)))  # no mask: every position is seen
    _, _, _, model = _model("J")
    assert model.cache_needs()[1].state["conv"].shape[0] == 1  # a single tap keeps no inputs; the slot has a row


def test_which_layers_mix_values():
    _, architecture, _, model = _model("G")
    assert [getattr(b.mixer, "value_mix", None) for b in model.blocks] == ["source", None, None, None, "mixed", "mixed"]
    raw = gc.config("G")
    raw["layers"][0]["mixer"]["v_mix"] = False
    model = DecoderModel(architecture.model_spec(architecture.parse(raw)))
    assert [getattr(b.mixer, "value_mix", None) for b in model.blocks] == [None, None, None, None, "source", "mixed"]


def test_named_errors():
    architecture = resolve_architecture(gc.config("G"))

    def broken(change):
        raw = gc.config("G")
        change(raw)
        return raw

    for change, word in [(lambda c: c["layers"][4]["mixer"].update(vdim=16), "mixes values"),
                         (lambda c: c["layers"][0]["mixer"].update(kv_heads=4), "heads"),
                         (lambda c: c["layers"][0]["mixer"]["mask"].update(size=0), "size"),
                         (lambda c: c["layers"][0]["mixer"]["mask"].update(keep_first=-1), "keep_first"),
                         (lambda c: c["layers"][1]["mixer"].update(groups=4), "groups"),
                         (lambda c: c["layers"][1]["mixer"].update(norm_groups=7), "norm groups"),
                         (lambda c: c["layers"][1]["mixer"].pop("state"), "state"),
                         (lambda c: c["layers"][3]["mixer"]["rot"].update(dims=10), "dims"),
                         (lambda c: c["layers"][3]["mixer"]["rot"].pop("base"), "base"),
                         (lambda c: c["layers"][0]["mlp"]["router"].update(top=7), "experts"),
                         (lambda c: c["layers"][0]["mlp"]["shared"].pop("ff"), "ff"),
                         (lambda c: c["layers"][1]["mlp"].update(kind="other"), "unknown kind"),
                         (lambda c: c["layers"][1].update(type="other"), "unknown type"),
                         (lambda c: c.pop("vocab"), "vocab")]:
        with pytest.raises(ConfigError, match=word):
            architecture.parse(broken(change))


def test_parts_refuse_what_they_do_not_do():
    with pytest.raises(ValueError, match="value_mix"):
        SinkWindowAttention(16, 2, 1, 8, 8, 1.0, bias=True, value_mix="mixed")
    with pytest.raises(ValueError, match="gated"):
        LatentAttention(16, 2, 8, 4, 8, 16, 1.0, 1e-5, PartSpec("rotary", {"dims": 4, "theta": 10.0}), gated="heads")
    with pytest.raises(ValueError, match="taps"):
        StateSpace(16, 2, 8, 8, 1, ops.SSD_MAX_TAPS + 1, 1, 1e-5)
    with pytest.raises(ValueError, match="groups"):
        StateSpace(16, 3, 8, 8, 2, 4, 1, 1e-5)
    with pytest.raises(ValueError, match="shared"):
        RoutedExperts(16, 8, 4, 2, shared_gate=True)
    with pytest.raises(ValueError, match="activation"):
        GLUMLP(16, 8, "silu2")
    block = PreNormBlock(PartSpec("state_space", {"hidden": 8, "heads": 1, "vdim": 8, "state": 4, "groups": 1, "conv": 2,
                                                  "norm_groups": 1, "norm_eps": 1e-5}), None,
                         {"norm1": PartSpec("rms_norm", {"size": 8, "eps": 1e-5})}, norm_names=("norm1", "norm2"))
    assert set(block.norms) == {"norm1"} and "norm1.weight" in block.tensors()


def test_columns_of_the_single_token_kernel():
    for requests, heads, dv in [(1, 1, 5), (1, 64, 64), (4, 24, 64), (64, 64, 128), (2, 3, 30), (1, 2, 256)]:
        cols = ops.ssd_step_columns(requests, heads, dv, 148)
        assert 1 <= cols <= dv and (dv % 4 or cols % 4 == 0)
    assert ops.ssd_step_columns(64, 64, 128, 148) == 128 and ops.ssd_step_columns(1, 8, 128, 148) == 16


def test_columns_of_the_chunked_kernel():
    bf16 = torch.bfloat16
    assert ops.ssd_chunk_columns(1, 64, 64, 128, bf16, 148) == 32 and ops.ssd_chunk_columns(1, 16, 64, 128, bf16, 148) == 16
    assert ops.ssd_chunk_columns(8, 64, 48, 16, bf16, 148) == 16  # heads of 48 do not come in 32
    for dv, N, dtype in [(64, 128, torch.float32), (64, 24, bf16), (24, 64, bf16), (64, 512, bf16)]:
        assert ops.ssd_chunk_columns(1, 64, dv, N, dtype, 148) == 0


# ---- the plain implementation's mechanisms ---------------------------------------------------


def test_the_state_space_recurrence_over_a_cut_and_in_closed_form():
    g = torch.Generator().manual_seed(1)
    T, H, dv, G, N = 19, 4, 3, 2, 5
    x, B, C = (torch.randn(T, *s, generator=g, dtype=F64) for s in ((H, dv), (G, N), (G, N)))
    dt = plain.softplus(torch.randn(T, H, generator=g, dtype=F64))
    A_log, D = torch.randn(H, generator=g), torch.randn(H, generator=g)
    y, S = plain.state_space(x, B, C, dt, A_log, D)
    first, S9 = plain.state_space(x[:9], B[:9], C[:9], dt[:9], A_log, D)
    rest, S_cut = plain.state_space(x[9:], B[9:], C[9:], dt[9:], A_log, D, S9)
    assert torch.allclose(torch.cat([first, rest]), y) and torch.allclose(S_cut, S)
    # In closed form: y_t = sum_j exp(-A sum_(j < i <= t) dt_i) dt_j (C_t . B_j) x_j + D x_t.
    t, h = 12, 3
    A = float(torch.exp(A_log[h].double()))
    want = D[h].double() * x[t, h] + sum(math.exp(-A * float(dt[j + 1: t + 1, h].sum())) * dt[j, h] * (C[t, 1] @ B[j, 1]) * x[j, h]
                                         for j in range(t + 1))
    assert torch.allclose(y[t, h], want)


def test_norm_groups_are_normed_by_themselves_behind_the_gate():
    g = torch.Generator().manual_seed(2)
    y, z, w = (torch.randn(3, 12, generator=g, dtype=F64) for _ in range(3))
    got = plain.gated_group_norm(y, z, 3, 1e-5, w[0])
    part = (y * plain.silu(z))[:, 4:8]
    assert torch.allclose(got[:, 4:8], part / torch.sqrt((part ** 2).mean(-1, keepdim=True) + 1e-5) * w[0, 4:8])


def test_a_window_with_kept_first_tokens():
    sees = plain.visible(12, {"size": 4, "keep_first": 2})
    assert sees[9].nonzero().flatten().tolist() == [0, 1, 6, 7, 8, 9] and sees[1].nonzero().flatten().tolist() == [0, 1]
    assert plain.visible(5, {"size": 1})[3].nonzero().flatten().tolist() == [3]
    assert int(plain.visible(5, None).sum()) == 15


def test_values_mix_with_the_first_layers_own():
    v, first = torch.ones(2, 1, 3, dtype=F64), torch.full((2, 1, 3), 5.0, dtype=F64)
    assert torch.allclose(plain.mixed_values(v, first, torch.tensor(0.25)), torch.full_like(v, 2.0))
    assert plain.mixed_values(v, None, torch.tensor(0.25)) is v


def test_the_router_weighs_the_chosen_logits_only():
    chosen, w = plain.route(torch.tensor([[1.0, 3.0, -200.0, 2.0]], dtype=F64), 2)
    assert chosen[0].tolist() == [1, 3] and torch.allclose(w[0], torch.softmax(torch.tensor([3.0, 2.0], dtype=F64), 0))


def test_the_two_gelus():
    z = torch.linspace(-4, 4, 33, dtype=F64)
    assert torch.allclose(plain.gelu_erf(z), torch.nn.functional.gelu(z))
    assert torch.allclose(plain.gelu_tanh(z), torch.nn.functional.gelu(z, approximate="tanh"))
    assert float((plain.gelu_erf(z) - plain.gelu_tanh(z)).abs().max()) > 1e-4


def test_the_convolution_reaches_back_and_has_a_bias():
    u = torch.zeros(6, 1, dtype=F64)
    u[2] = 1.0
    y = plain.causal_conv(u, torch.tensor([[3.0, 2.0, 1.0]]), torch.tensor([10.0]))
    assert y.flatten().tolist() == [10.0, 10.0, 11.0, 12.0, 13.0, 10.0]


def test_interleaved_rotation_keeps_products_of_equal_distance():
    g = torch.Generator().manual_seed(3)
    x = torch.randn(1, 1, 8, generator=g, dtype=F64).expand(9, 1, 8)
    y = plain.rotate(x, 50.0, 6)[:, 0]
    assert torch.allclose(y[2] @ y[5], y[4] @ y[7]) and torch.equal(y[:, 6:], x[:, 0, 6:])
    assert not torch.allclose(y[2] @ y[5], y[2] @ y[6])
