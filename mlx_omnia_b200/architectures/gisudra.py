"""Gisudra as configuration, parts and tensor names.

A pre-norm decoder whose layers carry, in any order the configuration lists, one of three mixers:
`attention`, a grouped-query attention without positions over a sliding window and a number of kept first
tokens, queries and keys normed per head, values mixed with those of the first such layer of the pass, the
output gated element by element; `latent_attention`, a sliding-window attention over a low-rank latent cache
with interleaved rotation and the same kind of gate; `mamba2`, a state-space recurrence behind a short
convolution, gated and normed in groups. The feed-forward is dense (gated, with the tanh form of GELU) or a
mixture of ungated experts with the exact GELU, weighted by a softmax over the chosen logits, beside a shared
expert with a gate of its own; a layer may have none. Everything here is data for the generic engine.

config.json keys: `architecture` ("Gisudra"), `vocab`, `width`, `norm.eps`, and `layers`: a list of {`type`,
`mixer`, `mlp`} with `mixer` = {heads, kv_heads, dim, vdim, scale, mask? {size, keep_first?}, v_mix?} |
{heads, dim, rot_dim, vdim, kv_rank, scale, rot {base, dims}, mask? {size}} | {heads, vdim, state, groups, conv,
norm_groups}, and `mlp` = null | {kind: "dense", ff} | {kind: "moe", expert {ff}, router {experts, top},
shared? {ff}}.
Tensor names: `embed`, `head`, `final.norm`, and per layer i `l<i>.norm1|norm2`; `l<i>.mix.q|k|v|q.norm|k.norm|
vmix|g|o`, or `l<i>.mix.q|dkv|dkv.norm|uk|uv|g|o`, or `l<i>.mix.in|conv|conv.b|dt_bias|A_log|D|norm|o`;
`l<i>.mlp.gate|up|down`, or `l<i>.mlp.router|router.b`, `l<i>.mlp.e<j>.up|down`, `l<i>.mlp.shared.up|down|sg`.
"""

from __future__ import annotations

import re
from dataclasses import dataclass
from typing import Any

import torch

from mlx_omnia_b200.config.hydrate import ConfigError
from mlx_omnia_b200.parts.base import PartSpec
from mlx_omnia_b200.parts.model import LayerSpec, ModelSpec, ScheduleEntry
from mlx_omnia_b200.registry import Architecture, register_architecture

ATTENTION, LATENT, STATE_SPACE = "attention", "latent_attention", "mamba2"
DENSE, EXPERTS = "dense", "moe"


@dataclass(frozen=True)
class GisudraAttention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int | None
    keep_first: int
    v_mix: bool


@dataclass(frozen=True)
class GisudraLatent:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    scale: float
    rot_base: float
    rot_dims: int
    window: int | None


@dataclass(frozen=True)
class GisudraStateSpace:
    heads: int
    vdim: int
    state: int
    groups: int
    conv: int
    norm_groups: int


@dataclass(frozen=True)
class GisudraDense:
    ff: int


@dataclass(frozen=True)
class GisudraExperts:
    ff: int
    experts: int
    top: int
    shared_ff: int | None


@dataclass(frozen=True)
class GisudraConfig:
    vocab: int
    width: int
    norm_eps: float
    mixers: tuple[GisudraAttention | GisudraLatent | GisudraStateSpace, ...]
    feed_forwards: tuple[GisudraDense | GisudraExperts | None, ...]

    def value_source(self) -> int | None:
        """The first layer that mixes values, whose own values the later ones mix in."""
        return next((i for i, m in enumerate(self.mixers) if isinstance(m, GisudraAttention) and m.v_mix), None)


def _need(raw: Any, key: str, where: str):
    if not isinstance(raw, dict) or key not in raw:
        raise ConfigError(f"Gisudra: {where} lacks the key {key!r}")
    return raw[key]


def _sizes(raw: dict, where: str, *keys: str) -> list[int]:
    values = [int(_need(raw, key, where)) for key in keys]
    for key, value in zip(keys, values):
        if value < 1:
            raise ConfigError(f"Gisudra: {where}.{key} must be at least 1, got {value}")
    return values


def _window(raw: dict, where: str) -> int | None:
    mask = raw.get("mask")
    return None if mask is None else _sizes(mask, where + ".mask", "size")[0]


def _attention(raw: dict, where: str) -> GisudraAttention:
    heads, kv_heads, dim, vdim = _sizes(raw, where, "heads", "kv_heads", "dim", "vdim")
    if heads % kv_heads:
        raise ConfigError(f"Gisudra: {where}: {heads} heads do not divide into {kv_heads} key/value heads")
    window = _window(raw, where)
    keep_first = 0 if window is None else int(raw["mask"].get("keep_first") or 0)
    if keep_first < 0:
        raise ConfigError(f"Gisudra: {where}.mask.keep_first must not be negative, got {keep_first}")
    return GisudraAttention(heads, kv_heads, dim, vdim, float(_need(raw, "scale", where)), window, keep_first,
                            bool(raw.get("v_mix", False)))


def _latent(raw: dict, where: str) -> GisudraLatent:
    heads, dim, rot_dim, vdim, kv_rank = _sizes(raw, where, "heads", "dim", "rot_dim", "vdim", "kv_rank")
    rot = _need(raw, "rot", where)
    dims = _sizes(rot, where + ".rot", "dims")[0]
    if dims % 2 or dims > rot_dim:
        raise ConfigError(f"Gisudra: {where}.rot.dims must be even and at most {rot_dim}, got {dims}")
    return GisudraLatent(heads, dim, rot_dim, vdim, kv_rank, float(_need(raw, "scale", where)),
                         float(_need(rot, "base", where + ".rot")), dims, _window(raw, where))


def _state_space(raw: dict, where: str) -> GisudraStateSpace:
    m = GisudraStateSpace(*_sizes(raw, where, "heads", "vdim", "state", "groups", "conv", "norm_groups"))
    if m.heads % m.groups or m.heads * m.vdim % m.norm_groups:
        raise ConfigError(f"Gisudra: {where}: {m.heads} heads of {m.vdim} do not divide into {m.groups} groups and "
                          f"{m.norm_groups} norm groups")
    return m


def _feed_forward(raw: dict | None, where: str) -> GisudraDense | GisudraExperts | None:
    if raw is None:
        return None
    kind = _need(raw, "kind", where)
    if kind == DENSE:
        return GisudraDense(*_sizes(raw, where, "ff"))
    if kind != EXPERTS:
        raise ConfigError(f"Gisudra: {where} has the unknown kind {kind!r}")
    experts, top = _sizes(_need(raw, "router", where), where + ".router", "experts", "top")
    if top > experts:
        raise ConfigError(f"Gisudra: {where}.router: {top} of {experts} experts")
    shared = raw.get("shared")
    return GisudraExperts(*_sizes(_need(raw, "expert", where), where + ".expert", "ff"), experts, top,
                          None if shared is None else _sizes(shared, where + ".shared", "ff")[0])


_MIXERS = {ATTENTION: _attention, LATENT: _latent, STATE_SPACE: _state_space}


def parse(raw: dict[str, Any]) -> GisudraConfig:
    if raw.get("architecture") != "Gisudra":
        raise ConfigError(f"expected architecture 'Gisudra', got {raw.get('architecture')!r}")
    mixers, feed_forwards = [], []
    for index, layer in enumerate(_need(raw, "layers", "config.json")):
        where = f"layers[{index}]"
        kind, mixer = _need(layer, "type", where), _need(layer, "mixer", where)
        if kind not in _MIXERS:
            raise ConfigError(f"Gisudra: {where} has the unknown type {kind!r}")
        mixers.append(_MIXERS[kind](mixer, where + ".mixer"))
        feed_forwards.append(_feed_forward(layer.get("mlp"), where + ".mlp"))
    if not mixers:
        raise ConfigError("Gisudra: no layers")
    vocab, width = _sizes(raw, "config.json", "vocab", "width")
    config = GisudraConfig(vocab, width, float(_need(_need(raw, "norm", "config.json"), "eps", "norm")), tuple(mixers),
                           tuple(feed_forwards))
    source = config.value_source()
    for index, m in enumerate(mixers):
        if isinstance(m, GisudraAttention) and m.v_mix and (m.kv_heads, m.vdim) != (mixers[source].kv_heads, mixers[source].vdim):
            raise ConfigError(f"Gisudra: layers[{index}] mixes values of {m.kv_heads} x {m.vdim} with layer {source}'s of "
                              f"{mixers[source].kv_heads} x {mixers[source].vdim}")
    return config


def _norm(config: GisudraConfig) -> PartSpec:
    return PartSpec("rms_norm", {"size": config.width, "eps": config.norm_eps, "weight": "plain"})


def _mixer_spec(config: GisudraConfig, index: int) -> PartSpec:
    m = config.mixers[index]
    if isinstance(m, GisudraStateSpace):
        return PartSpec("state_space", {"hidden": config.width, "heads": m.heads, "vdim": m.vdim, "state": m.state,
                                        "groups": m.groups, "conv": m.conv, "norm_groups": m.norm_groups,
                                        "norm_eps": config.norm_eps})
    if isinstance(m, GisudraAttention):
        mix = None if not m.v_mix else "source" if index == config.value_source() else "mixed"
        return PartSpec("sink_window_attention", {
            "hidden": config.width, "heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "scale": m.scale,
            "window": m.window, "keep_first": m.keep_first, "norm_eps": config.norm_eps, "gated": True, "value_mix": mix})
    position = PartSpec("rotary", {"dims": m.rot_dims, "theta": m.rot_base, "pairing": "interleaved"})
    return PartSpec("latent_attention", {
        "hidden": config.width, "heads": m.heads, "dim": m.dim, "rot_dim": m.rot_dim, "vdim": m.vdim, "kv_rank": m.kv_rank,
        "scale": m.scale, "norm_eps": config.norm_eps, "position": position, "sink": False, "gated": "values",
        "window": m.window})


def _feed_forward_spec(config: GisudraConfig, f) -> PartSpec | None:
    if f is None:
        return None
    if isinstance(f, GisudraDense):
        return PartSpec("glu_mlp", {"hidden": config.width, "inner": f.ff, "activation": "gelu_tanh"})
    return PartSpec("routed_experts", {"hidden": config.width, "inner": f.ff, "experts": f.experts, "top": f.top,
                                       "correction": False, "scoring": "chosen", "router_bias": True, "unit": "gelu_erf",
                                       "shared_inner": f.shared_ff, "shared_gate": f.shared_ff is not None})


def model_spec(config: GisudraConfig) -> ModelSpec:
    layers = []
    for index, f in enumerate(config.feed_forwards):
        names = ("norm1", "norm2")
        layers.append(LayerSpec(PartSpec("pre_norm", {
            "mixer": _mixer_spec(config, index), "feed_forward": _feed_forward_spec(config, f),
            "norms": {name: _norm(config) for name in names}, "norm_names": names, "mixer_name": "mix",
            "feed_forward_name": "mlp"}), f"l{index}"))
    return ModelSpec(
        embedding=PartSpec("token_embedding", {"vocab": config.vocab, "hidden": config.width}),
        layers=tuple(layers),
        schedule=tuple(ScheduleEntry(i) for i in range(len(layers))),
        final_norm=_norm(config),
        head=PartSpec("lm_head", {"vocab": config.vocab, "hidden": config.width}),
        embedding_prefix="embed", final_norm_prefix="final.norm", head_prefix="head",
    )


_WEIGHT = re.compile(r"^(embed|head|final\.norm|l\d+\.norm[12])$")


def tensor_name(file_name: str) -> str:
    """The file's names are the model's, but for the parts that call their one tensor `weight`."""
    return file_name + ".weight" if _WEIGHT.match(file_name) else file_name


def random_tensors(config: GisudraConfig, seed: int) -> dict[str, torch.Tensor]:
    """Float32 tensors under the checkpoint's names, drawn on the CPU in a fixed order from one
    generator: matrices N(0, gain / sqrt(fan_in)); norm weights around one; biases, decays and
    step sizes of a size that makes every mechanism count."""
    g = torch.Generator().manual_seed(seed)

    def normal(*shape: int, std: float = 1.0) -> torch.Tensor:
        return torch.randn(*shape, generator=g, dtype=torch.float32) * std

    def matrix(rows: int, cols: int, gain: float = 1.0) -> torch.Tensor:
        return normal(rows, cols, std=gain * cols ** -0.5)

    def weight(size: int) -> torch.Tensor:
        return 1.0 + normal(size, std=0.1)

    D = config.width
    out = {"embed": normal(config.vocab, D), "head": matrix(config.vocab, D)}
    for i, (m, f) in enumerate(zip(config.mixers, config.feed_forwards)):
        p = f"l{i}."
        q = p + "mix."
        out[p + "norm1"] = weight(D)
        if isinstance(m, GisudraStateSpace):
            inner, channels = m.heads * m.vdim, m.heads * m.vdim + 2 * m.groups * m.state
            out[q + "in"] = matrix(inner + channels + m.heads, D, gain=1.5)
            out[q + "conv"] = normal(channels, m.conv, std=0.5 * m.conv ** -0.5) + torch.eye(m.conv)[-1] * 0.7
            out[q + "conv.b"] = normal(channels, std=0.2)
            # Decays exp(-exp(A_log) dt) from about a half to nearly one a token.
            out[q + "dt_bias"], out[q + "A_log"] = normal(m.heads) - 2.0, normal(m.heads, std=0.7)
            out[q + "D"], out[q + "norm"] = normal(m.heads, std=0.5), weight(inner)
            out[q + "o"] = matrix(D, inner)
        elif isinstance(m, GisudraAttention):
            out[q + "q"], out[q + "k"] = matrix(m.heads * m.dim, D), matrix(m.kv_heads * m.dim, D)
            out[q + "v"], out[q + "g"] = matrix(m.kv_heads * m.vdim, D), matrix(m.heads * m.vdim, D)
            out[q + "q.norm"], out[q + "k.norm"] = weight(m.dim), weight(m.dim)
            if m.v_mix:
                out[q + "vmix"] = normal(1, std=0.2)[0] + 0.4
            out[q + "o"] = matrix(D, m.heads * m.vdim)
        else:
            out[q + "q"] = matrix(m.heads * (m.dim + m.rot_dim), D, gain=2.0)
            out[q + "dkv"], out[q + "dkv.norm"] = matrix(m.kv_rank + m.rot_dim, D), weight(m.kv_rank)
            out[q + "uk"], out[q + "uv"] = matrix(m.heads * m.dim, m.kv_rank, gain=2.0), matrix(m.heads * m.vdim, m.kv_rank)
            out[q + "g"], out[q + "o"] = matrix(m.heads * m.vdim, D), matrix(D, m.heads * m.vdim)
        if f is None:
            continue
        q = p + "mlp."
        out[p + "norm2"] = weight(D)
        if isinstance(f, GisudraDense):
            out[q + "gate"], out[q + "up"], out[q + "down"] = matrix(f.ff, D), matrix(f.ff, D), matrix(D, f.ff)
            continue
        out[q + "router"], out[q + "router.b"] = matrix(f.experts, D, gain=2.0), normal(f.experts, std=0.3)
        units = [(f"e{e}", f.ff) for e in range(f.experts)]
        if f.shared_ff is not None:
            units.append(("shared", f.shared_ff))
            out[q + "shared.sg"] = matrix(1, D)
        for name, inner in units:
            out[q + name + ".up"], out[q + name + ".down"] = matrix(inner, D, gain=1.5), matrix(D, inner)
    out["final.norm"] = weight(D)
    return out


ARCHITECTURE = Architecture(
    name="gisudra",
    config_class=GisudraConfig,
    parse=parse,
    model_spec=model_spec,
    tensor_name=tensor_name,
    random_tensors=random_tensors,
)

register_architecture(ARCHITECTURE, "Gisudra", "gisudra")
