"""Tiny Rinirax configurations for the tests, and their random weights as a checkpoint would hold them
(rounded to bfloat16). Their sizes are unlike one another on purpose."""

from __future__ import annotations

import copy
import json
from pathlib import Path

import torch

from mlx_omnia_b200.registry import resolve_architecture


def _attention(heads, kv_heads, dim, vdim, scale, diff, conv, dims, base, kv_from=None):
    mixer = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "diff": diff, "conv": conv,
             "rot": {"base": base, "dims": dims}}
    if kv_from is not None:
        mixer["kv_from"] = kv_from
    return {"type": "attention", "mixer": mixer}


def _latent(heads, dim, rot_dim, vdim, kv_rank, q_rank, scale, base, window, scaling=None):
    mixer = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank,
             "scale": scale, "rot": {"base": base, "dims": rot_dim}}
    if window is not None:
        mixer["mask"] = {"size": window}
    if scaling is not None:
        mixer["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return {"type": "latent_attention", "mixer": mixer}


def _gru(width):
    return {"type": "mingru", "mixer": {"width": width}}


def _moe(layer, ff, experts, top, count, keep, scale):
    layer["mlp"] = {"kind": "moe", "expert": {"ff": ff},
                    "router": {"experts": experts, "top": top, "groups": {"count": count, "keep": keep}, "scale": scale}}
    return layer


def _dense(layer, ff):
    layer["mlp"] = {"kind": "dense", "ff": ff}
    return layer


def _bare(layer):
    layer["mlp"] = None
    return layer


CONFIGS = {
    # attention first, values wider than a head's two maps, a rotation over half a map, four taps; a layer
    # without a feed-forward; a latent behind the generic kernel with a short window; a reader with other
    # query heads than the layer it reads from; two of four groups of experts kept
    "S": {"architecture": "Rinirax", "vocab": 149, "width": 96, "norm": {"eps": 1e-5},
          "layers": [_moe(_attention(6, 2, 16, 40, 0.3, 0.2, 4, 8, 300.0), 24, 12, 3, 4, 2, 2.0),
                     _bare(_gru(72)),
                     _dense(_latent(3, 24, 8, 20, 40, 28, 0.2, 5000.0, 9, (4.0, 64, 8.0, 1.5)), 56),
                     _moe(_attention(4, 2, 16, 40, 0.25, 0.6, 2, 8, 300.0, kv_from=0), 16, 6, 2, 1, 1, 0.7),
                     _moe(_gru(40), 40, 8, 2, 4, 3, 1.3)]},
    # rows of 64 over pages of 16 (the tensor-core attention kernels in bfloat16), a latent of 64 + 32 on the
    # tensor cores with a window of 33; every expert for every token, so that no choice can fall the other
    # way in bfloat16 and every row of logits can be held to the tolerance
    "T": {"architecture": "Rinirax", "vocab": 211, "width": 128, "norm": {"eps": 1e-6},
          "layers": [_dense(_latent(4, 32, 32, 16, 64, 48, 0.11, 20000.0, 33, (8.0, 256, 16.0, 0.5)), 96),
                     _moe(_attention(4, 2, 32, 64, 0.2, 0.35, 3, 32, 9000.0), 32, 4, 4, 2, 2, 1.5),
                     _moe(_gru(128), 32, 3, 3, 1, 1, 1.0),
                     _bare(_attention(4, 2, 32, 64, 0.18, 0.5, 3, 32, 9000.0, kv_from=1)),
                     _dense(_attention(2, 1, 32, 48, 0.22, 0.1, 1, 16, 700.0), 64)]},
    # nothing a multiple of eight: odd maps, odd values, a latent of 20 with 6 rotated, no frequency scaling and
    # no window, one head, one group of one key head, a single expert, one layer that reads a later one's neighbour
    "W": {"architecture": "Rinirax", "vocab": 101, "width": 100, "norm": {"eps": 1e-5},
          "layers": [_moe(_latent(5, 12, 6, 10, 20, 12, 0.3, 100.0, None), 20, 1, 1, 1, 1, 0.8),
                     _dense(_attention(3, 3, 5, 7, 0.5, 0.4, 5, 4, 40.0), 36),
                     _moe(_attention(3, 3, 5, 7, 0.4, 0.3, 2, 4, 40.0, kv_from=1), 12, 9, 4, 3, 3, 1.1),
                     _bare(_gru(30)),
                     _moe(_attention(1, 1, 9, 20, 0.3, 0.15, 2, 8, 1000.0), 12, 4, 2, 4, 2, 1.0)]},
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
    g = torch.Generator().manual_seed(700 + seed)
    return torch.randint(0, vocab, (length,), generator=g).tolist()


def write_folder(folder: Path, raw: dict, weights: dict[str, torch.Tensor]) -> None:
    """A model folder as the loader reads it: config.json and bfloat16 tensors."""
    from safetensors.torch import save_file

    folder.mkdir(parents=True, exist_ok=True)
    save_file({k: t.to(torch.bfloat16).contiguous() for k, t in weights.items()}, str(folder / "model.safetensors"))
    (folder / "config.json").write_text(json.dumps(raw))
