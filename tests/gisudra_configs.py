"""Tiny Gisudra configurations for the tests, and their random weights as a checkpoint would hold them
(rounded to bfloat16). Their sizes are unlike one another on purpose."""

from __future__ import annotations

import copy
import json
from pathlib import Path

import torch

from mlx_omnia_b200.registry import resolve_architecture


def _attention(heads, kv_heads, dim, vdim, scale, size=None, keep_first=None, v_mix=None):
    mixer = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if size is not None:
        mixer["mask"] = {"size": size} | ({} if keep_first is None else {"keep_first": keep_first})
    if v_mix is not None:
        mixer["v_mix"] = v_mix
    return {"type": "attention", "mixer": mixer}


def _latent(heads, dim, rot_dim, vdim, kv_rank, scale, base, size, dims=None):
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank,
                                                  "scale": scale, "rot": {"base": base, "dims": dims or rot_dim},
                                                  "mask": {"size": size}}}


def _mamba(heads, vdim, state, groups, conv, norm_groups):
    return {"type": "mamba2", "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv,
                                        "norm_groups": norm_groups}}


def _moe(layer, ff, experts, top, shared):
    layer["mlp"] = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}, "shared": {"ff": shared}}
    return layer


def _dense(layer, ff):
    layer["mlp"] = {"kind": "dense", "ff": ff}
    return layer


def _bare(layer):
    layer["mlp"] = None
    return layer


CONFIGS = {
    # attention first; a layer between the mixing ones that mixes nothing; values wider than keys; two groups of B
    # and C, three norm groups, two taps; a layer without a feed-forward
    "G": {"architecture": "Gisudra", "vocab": 139, "width": 96, "norm": {"eps": 1e-5},
          "layers": [_moe(_attention(6, 2, 16, 24, 0.3, 11, 5, True), 24, 6, 3, 40),
                     _dense(_mamba(6, 20, 24, 2, 2, 3), 56),
                     _bare(_attention(4, 4, 16, 16, 0.25, 30, 0, False)),
                     _moe(_latent(3, 24, 8, 20, 40, 0.2, 5000.0, 9), 32, 5, 2, 24),
                     _moe(_attention(4, 2, 8, 24, 0.4, 17, 3, True), 16, 7, 4, 16),
                     _dense(_attention(2, 2, 32, 24, 0.2, 6, 1, True), 48)]},
    # heads of 64 and 32 over pages of 16 (the tensor-core kernels in bfloat16), a latent of 64 + 32, a state of 64;
    # every expert for every token, so that no choice can fall the other way in bfloat16
    "H": {"architecture": "Gisudra", "vocab": 211, "width": 128, "norm": {"eps": 1e-6},
          "layers": [_dense(_mamba(4, 32, 64, 1, 4, 1), 96),
                     _moe(_latent(4, 32, 32, 48, 64, 0.11, 20000.0, 33), 32, 4, 4, 64),
                     _moe(_attention(4, 2, 64, 64, 0.2, 25, 7, True), 32, 3, 3, 32),
                     _moe(_mamba(2, 64, 32, 2, 3, 2), 40, 2, 2, 96),
                     _dense(_attention(6, 2, 64, 64, 0.15, 50, 20, True), 64),
                     _bare(_attention(2, 2, 32, 32, 0.2))]},
    # nothing a multiple of eight, one head, one group, one tap, one expert, one row of state
    "J": {"architecture": "Gisudra", "vocab": 101, "width": 100, "norm": {"eps": 1e-4},
          "layers": [_moe(_latent(5, 12, 6, 10, 20, 0.3, 100.0, 14, 4), 20, 1, 1, 12),
                     _dense(_mamba(3, 7, 5, 3, 1, 7), 36),
                     _moe(_attention(3, 3, 5, 7, 0.5, 1, 2, True), 12, 9, 4, 28),
                     _bare(_mamba(1, 30, 1, 1, 5, 5)),
                     _moe(_attention(6, 3, 9, 7, 0.3, 4, 6, True), 12, 4, 2, 20),
                     _bare(_mamba(5, 6, 13, 1, 9, 1))]},
}


def config(name: str) -> dict:
    return copy.deepcopy(CONFIGS[name])


def tensors(name_or_raw, seed: int = 0) -> dict[str, torch.Tensor]:
    """Random weights under the checkpoint's names, rounded to bfloat16."""
    raw = config(name_or_raw) if isinstance(name_or_raw, str) else name_or_raw
    architecture = resolve_architecture(raw)
    drawn = architecture.random_tensors(architecture.parse(raw), seed)
    return {k: t.to(torch.bfloat16).float() for k, t in drawn.items()}


def prompt(length: int, vocab: int, seed: int) -> list[int]:
    g = torch.Generator().manual_seed(900 + seed)
    return torch.randint(0, vocab, (length,), generator=g).tolist()


def write_folder(folder: Path, raw: dict, weights: dict[str, torch.Tensor]) -> None:
    """A model folder as the loader reads it: config.json and bfloat16 tensors."""
    from safetensors.torch import save_file

    folder.mkdir(parents=True, exist_ok=True)
    save_file({k: t.to(torch.bfloat16).contiguous() for k, t in weights.items()}, str(folder / "model.safetensors"))
    (folder / "config.json").write_text(json.dumps(raw))
