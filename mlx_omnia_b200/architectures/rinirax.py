"""Rinirax as configuration, parts and tensor names.

A decoder of parallel blocks (one layer norm; the mixer and the feed-forward both read its output and are
added together) whose residual is, after every layer, a learned average of the embedding output and all
layers' results so far. Its layers carry, in any order the configuration lists, one of three mixers:
`attention`, a differential attention (two softmax maps a head over the same values, their difference
normed) with biased projections behind short convolutions and interleaved rotation, which may read an
earlier layer's keys and values; `latent_attention`, a sliding-window attention over a low-rank latent
cache whose queries come through a latent too, rotated half-split with YaRN's frequencies; `mingru`, a
gated recurrence over channels whose gates read the current token only. The feed-forward is dense with
xIELU, or a mixture of gated experts chosen by corrected sigmoid scores within the best groups of
experts; a layer may have none. Everything here is data for the generic engine.

config.json keys: `architecture` ("Rinirax"), `vocab`, `width`, `norm.eps`, and `layers`: a list of {`type`,
`mixer`, `mlp`} with `mixer` = {heads, kv_heads, dim, vdim, scale, diff, conv, rot? {base, dims}, kv_from?} |
{heads, dim, rot_dim, vdim, kv_rank, q_rank, scale, rot {base, dims, scaling? {factor, original, fast, slow}},
mask? {size}} | {width}, and `mlp` = null | {kind: "dense", ff} | {kind: "moe", expert {ff}, router {experts,
top, groups? {count, keep}, scale?}}.
Tensor names: `embed`, `head`, `final.norm`, `final.norm.b`, and per layer i `l<i>.norm1`, `l<i>.norm1.b`,
`l<i>.dwa`; `l<i>.mix.q|k|v` with `.b` and `.conv`, `.lq1|lk1|lq2|lk2|o`, or `l<i>.mix.dq|dq.norm|uq|dkv|
dkv.norm|uk|uv|o`, or `l<i>.mix.z|z.b|x|x.b|g|o`; `l<i>.mlp.up|down|act`, or `l<i>.mlp.router|correction`,
`l<i>.mlp.e<j>.gate|up|down`.
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

ATTENTION, LATENT, RECURRENT = "attention", "latent_attention", "mingru"
DENSE, EXPERTS = "dense", "moe"


@dataclass(frozen=True)
class RiniraxRotation:
    base: float
    dims: int
    scaling: tuple[float, float, float, float] | None = None  # factor, original, fast, slow


@dataclass(frozen=True)
class RiniraxAttention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    diff: float
    conv: int
    rot: RiniraxRotation | None
    kv_from: int | None


@dataclass(frozen=True)
class RiniraxLatent:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    q_rank: int
    scale: float
    rot: RiniraxRotation
    window: int | None


@dataclass(frozen=True)
class RiniraxRecurrent:
    width: int


@dataclass(frozen=True)
class RiniraxDense:
    ff: int


@dataclass(frozen=True)
class RiniraxExperts:
    ff: int
    experts: int
    top: int
    groups: int
    keep: int
    scale: float


@dataclass(frozen=True)
class RiniraxConfig:
    vocab: int
    width: int
    norm_eps: float
    mixers: tuple[RiniraxAttention | RiniraxLatent | RiniraxRecurrent, ...]
    feed_forwards: tuple[RiniraxDense | RiniraxExperts | None, ...]


def _need(raw: Any, key: str, where: str):
    if not isinstance(raw, dict) or key not in raw:
        raise ConfigError(f"Rinirax: {where} lacks the key {key!r}")
    return raw[key]


def _sizes(raw: dict, where: str, *keys: str) -> list[int]:
    values = [int(_need(raw, key, where)) for key in keys]
    for key, value in zip(keys, values):
        if value < 1:
            raise ConfigError(f"Rinirax: {where}.{key} must be at least 1, got {value}")
    return values


def _rotation(rot: dict | None, dim: int, where: str) -> RiniraxRotation | None:
    if rot is None:
        return None
    dims = int(_need(rot, "dims", where))
    if dims % 2 or not 0 <= dims <= dim:
        raise ConfigError(f"Rinirax: {where}.dims must be even and at most {dim}, got {dims}")
    if dims == 0:
        return None
    scaling = rot.get("scaling")
    if scaling is not None:
        scaling = tuple(float(_need(scaling, key, where + ".scaling")) for key in ("factor", "original", "fast", "slow"))
    return RiniraxRotation(float(_need(rot, "base", where)), dims, scaling)


def _attention(raw: dict, where: str, index: int, earlier: list) -> RiniraxAttention:
    heads, kv_heads, dim, vdim, conv = _sizes(raw, where, "heads", "kv_heads", "dim", "vdim", "conv")
    if heads % kv_heads:
        raise ConfigError(f"Rinirax: {where}: {heads} heads do not divide into {kv_heads} key/value heads")
    mixer = RiniraxAttention(heads, kv_heads, dim, vdim, float(_need(raw, "scale", where)), float(_need(raw, "diff", where)),
                             conv, _rotation(raw.get("rot"), dim, where + ".rot"), raw.get("kv_from"))
    if mixer.kv_from is not None:
        source = earlier[mixer.kv_from] if 0 <= mixer.kv_from < index else None
        if not isinstance(source, RiniraxAttention) or source.kv_from is not None:
            raise ConfigError(f"Rinirax: {where}.kv_from {mixer.kv_from} names no earlier attention with keys of its own")
        if (source.kv_heads, source.dim, source.vdim, source.rot) != (kv_heads, dim, vdim, mixer.rot):
            raise ConfigError(f"Rinirax: {where}.kv_from: layer {mixer.kv_from} keeps keys of other sizes or another rotation")
    return mixer


def _latent(raw: dict, where: str) -> RiniraxLatent:
    heads, dim, rot_dim, vdim, kv_rank, q_rank = _sizes(raw, where, "heads", "dim", "rot_dim", "vdim", "kv_rank", "q_rank")
    rot = _rotation(_need(raw, "rot", where), rot_dim, where + ".rot")
    if rot is None:
        raise ConfigError(f"Rinirax: {where}.rot.dims must be positive")
    mask = raw.get("mask")
    window = None if mask is None else _sizes(mask, where + ".mask", "size")[0]
    return RiniraxLatent(heads, dim, rot_dim, vdim, kv_rank, q_rank, float(_need(raw, "scale", where)), rot, window)


def _feed_forward(raw: dict | None, where: str) -> RiniraxDense | RiniraxExperts | None:
    if raw is None:
        return None
    kind = _need(raw, "kind", where)
    if kind == DENSE:
        return RiniraxDense(*_sizes(raw, where, "ff"))
    if kind != EXPERTS:
        raise ConfigError(f"Rinirax: {where} has the unknown kind {kind!r}")
    router = _need(raw, "router", where)
    experts, top = _sizes(router, where + ".router", "experts", "top")
    groups, keep = 1, 1
    if router.get("groups") is not None:
        groups, keep = _sizes(router["groups"], where + ".router.groups", "count", "keep")
    if experts % groups or keep > groups or top > keep * (experts // groups):
        raise ConfigError(f"Rinirax: {where}.router: {top} of {experts} experts in {groups} groups of which {keep} are kept")
    return RiniraxExperts(*_sizes(_need(raw, "expert", where), where + ".expert", "ff"), experts, top, groups, keep,
                          float(router.get("scale", 1.0)))


def parse(raw: dict[str, Any]) -> RiniraxConfig:
    if raw.get("architecture") != "Rinirax":
        raise ConfigError(f"expected architecture 'Rinirax', got {raw.get('architecture')!r}")
    mixers, feed_forwards = [], []
    for index, layer in enumerate(_need(raw, "layers", "config.json")):
        where = f"layers[{index}]"
        kind, mixer = _need(layer, "type", where), _need(layer, "mixer", where)
        if kind == ATTENTION:
            mixers.append(_attention(mixer, where + ".mixer", index, mixers))
        elif kind == LATENT:
            mixers.append(_latent(mixer, where + ".mixer"))
        elif kind == RECURRENT:
            mixers.append(RiniraxRecurrent(*_sizes(mixer, where + ".mixer", "width")))
        else:
            raise ConfigError(f"Rinirax: {where} has the unknown type {kind!r}")
        feed_forwards.append(_feed_forward(layer.get("mlp"), where + ".mlp"))
    if not mixers:
        raise ConfigError("Rinirax: no layers")
    vocab, width = _sizes(raw, "config.json", "vocab", "width")
    return RiniraxConfig(vocab, width, float(_need(_need(raw, "norm", "config.json"), "eps", "norm")), tuple(mixers),
                         tuple(feed_forwards))


def _norm(config: RiniraxConfig) -> PartSpec:
    return PartSpec("layer_norm", {"size": config.width, "eps": config.norm_eps})


def _mixer_spec(config: RiniraxConfig, m) -> PartSpec:
    if isinstance(m, RiniraxRecurrent):
        return PartSpec("min_gru", {"hidden": config.width, "width": m.width})
    if isinstance(m, RiniraxAttention):
        position = None if m.rot is None else PartSpec("rotary", {"dims": m.rot.dims, "theta": m.rot.base,
                                                                  "pairing": "interleaved", "scaling": m.rot.scaling})
        return PartSpec("differential_attention", {
            "hidden": config.width, "heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "scale": m.scale,
            "diff": m.diff, "conv": m.conv, "norm_eps": config.norm_eps, "position": position, "own_kv": m.kv_from is None})
    position = PartSpec("rotary", {"dims": m.rot.dims, "theta": m.rot.base, "pairing": "half", "scaling": m.rot.scaling})
    return PartSpec("latent_attention", {
        "hidden": config.width, "heads": m.heads, "dim": m.dim, "rot_dim": m.rot_dim, "vdim": m.vdim, "kv_rank": m.kv_rank,
        "q_rank": m.q_rank, "scale": m.scale, "norm_eps": config.norm_eps, "position": position, "sink": False,
        "gated": False, "window": m.window})


def _feed_forward_spec(config: RiniraxConfig, f) -> PartSpec | None:
    if f is None:
        return None
    if isinstance(f, RiniraxDense):
        return PartSpec("dense_mlp", {"hidden": config.width, "inner": f.ff, "activation": "xielu"})
    return PartSpec("routed_experts", {"hidden": config.width, "inner": f.ff, "experts": f.experts, "top": f.top,
                                       "scoring": "sigmoid", "groups": f.groups, "keep_groups": f.keep, "normalise": True,
                                       "weight_scale": f.scale})


def model_spec(config: RiniraxConfig) -> ModelSpec:
    depth = len(config.mixers)
    layers, schedule = [], []
    for index, (m, f) in enumerate(zip(config.mixers, config.feed_forwards)):
        layers.append(LayerSpec(PartSpec("parallel", {
            "mixer": _mixer_spec(config, m), "feed_forward": _feed_forward_spec(config, f), "norm": _norm(config),
            "averaged": index + 1, "depth": depth}), f"l{index}"))
        schedule.append(ScheduleEntry(index, getattr(m, "kv_from", None)))
    return ModelSpec(
        embedding=PartSpec("token_embedding", {"vocab": config.vocab, "hidden": config.width}),
        layers=tuple(layers),
        schedule=tuple(schedule),
        final_norm=_norm(config),
        head=PartSpec("lm_head", {"vocab": config.vocab, "hidden": config.width}),
        embedding_prefix="embed", final_norm_prefix="final.norm", head_prefix="head",
    )


_WEIGHT = re.compile(r"^(embed|head|final\.norm|l\d+\.norm1)$")
_BIAS = re.compile(r"^(final\.norm|l\d+\.norm1)\.b$")


def tensor_name(file_name: str) -> str:
    """The file's names are the model's, but for the parts that call their tensors `weight` and `bias`."""
    if _WEIGHT.match(file_name):
        return file_name + ".weight"
    return file_name[:-1] + "bias" if _BIAS.match(file_name) else file_name


def random_tensors(config: RiniraxConfig, seed: int) -> dict[str, torch.Tensor]:
    """Float32 tensors under the checkpoint's names, drawn on the CPU in a fixed order from one
    generator: matrices N(0, gain / sqrt(fan_in)); norm weights around one; biases, corrections, lambdas
    and averages of a size that makes every mechanism count."""
    g = torch.Generator().manual_seed(seed)

    def normal(*shape: int, std: float = 1.0) -> torch.Tensor:
        return torch.randn(*shape, generator=g, dtype=torch.float32) * std

    def matrix(rows: int, cols: int, gain: float = 1.0) -> torch.Tensor:
        return normal(rows, cols, std=gain * cols ** -0.5)

    D = config.width
    out = {"embed": normal(config.vocab, D), "head": matrix(config.vocab, D)}
    for i, (m, f) in enumerate(zip(config.mixers, config.feed_forwards)):
        p = f"l{i}."
        out[p + "norm1"], out[p + "norm1.b"] = 1.0 + normal(D, std=0.1), normal(D, std=0.1)
        out[p + "dwa"] = torch.cat([normal(i + 1, std=0.3), 0.7 + normal(1, std=0.1)])
        q = p + "mix."
        if isinstance(m, RiniraxRecurrent):
            for name in ("z", "x", "g"):
                out[q + name] = matrix(m.width, D, gain=2.0)
            out[q + "z.b"], out[q + "x.b"] = normal(m.width) - 1.5, normal(m.width, std=0.3)
            out[q + "o"] = matrix(D, m.width)
        elif isinstance(m, RiniraxAttention):
            rows = {"q": m.heads * 2 * m.dim}
            if m.kv_from is None:
                rows |= {"k": m.kv_heads * 2 * m.dim, "v": m.kv_heads * m.vdim}
            for name, count in rows.items():
                out[q + name], out[q + name + ".b"] = matrix(count, D, gain=1.5), normal(count, std=0.3)
                out[q + name + ".conv"] = normal(count, m.conv, std=0.5 * m.conv ** -0.5) + torch.eye(m.conv)[-1] * 0.7
            for name in ("lq1", "lk1", "lq2", "lk2"):
                out[q + name] = normal(m.dim, std=0.5 * m.dim ** -0.25)
            out[q + "o"] = matrix(D, m.heads * m.vdim)
        else:
            qd = m.dim + m.rot_dim
            out[q + "dq"], out[q + "dq.norm"] = matrix(m.q_rank, D), 1.0 + normal(m.q_rank, std=0.1)
            out[q + "uq"] = matrix(m.heads * qd, m.q_rank, gain=2.0)
            out[q + "dkv"], out[q + "dkv.norm"] = matrix(m.kv_rank + m.rot_dim, D), 1.0 + normal(m.kv_rank, std=0.1)
            out[q + "uk"], out[q + "uv"] = matrix(m.heads * m.dim, m.kv_rank, gain=2.0), matrix(m.heads * m.vdim, m.kv_rank)
            out[q + "o"] = matrix(D, m.heads * m.vdim)
        q = p + "mlp."
        if isinstance(f, RiniraxDense):
            out[q + "up"], out[q + "down"], out[q + "act"] = matrix(f.ff, D), matrix(D, f.ff), normal(2, std=0.5)
        elif f is not None:
            out[q + "router"], out[q + "correction"] = matrix(f.experts, D, gain=2.0), normal(f.experts, std=0.3)
            for e in range(f.experts):
                out[q + f"e{e}.gate"], out[q + f"e{e}.up"] = matrix(f.ff, D, gain=2.0), matrix(f.ff, D, gain=2.0)
                out[q + f"e{e}.down"] = matrix(D, f.ff)
    out["final.norm"], out["final.norm.b"] = 1.0 + normal(D, std=0.1), normal(D, std=0.1)
    return out


ARCHITECTURE = Architecture(
    name="rinirax",
    config_class=RiniraxConfig,
    parse=parse,
    model_spec=model_spec,
    tensor_name=tensor_name,
    random_tensors=random_tensors,
)

register_architecture(ARCHITECTURE, "Rinirax", "rinirax")
