"""Small Fusanex configurations for the tests, and folders with weights made so that every mechanism matters.

'mixed'   a gated recurrence first (three blocks, four taps), grouped attention with values of their own size beside time mixing, a
          recurrence of one block and three taps without a feed-forward, a second pair of mixers without a query temperature, as
          many key/value heads as query heads and a negative factor; 2 of 6 + 2 experts, rows normed in four groups
'odd'     sizes in no step of 4 or 8 (width 50 in five groups, blocks of 10 channels, two taps, heads of 10 and 6, time mixing heads of
          10, 3 + 2 experts of 14 with 3 chosen, a shared expert of 10)
'bare'    what a file may leave out is left out: no embedding factor, no groups, no temperature, no factors, no identity experts, no
          shared expert; a convolution of one tap, every expert chosen, a layer with a pair of mixers first
'heads64' attention heads of 64 elements on the tensor-core kernels, time mixing heads of 64, blocks of 64 channels on the tensor cores,
          a query temperature that changes every 8 positions
"""
from __future__ import annotations

import copy
import json
import os

import torch
from safetensors.torch import save_file


def _lru(width, blocks, conv):
    return {"width": width, "blocks": blocks, "conv": conv}


def _par(left, right, left_scale=None, right_scale=None):
    m = {"left": left, "right": right}
    if left_scale is not None:
        m["left_scale"] = left_scale
    if right_scale is not None:
        m["right_scale"] = right_scale
    return m


def _att(heads, kv, dim, vdim=None, scale=None, temp=None):
    m = {"heads": heads, "dim": dim}
    if kv is not None:
        m["kv_heads"] = kv
    if vdim is not None:
        m["vdim"] = vdim
    if scale is not None:
        m["scale"] = scale
    if temp is not None:
        m["q_temp"] = {"coef": temp[0], "every": temp[1]}
    return m


def _mix(heads, dim, rank):
    return {"heads": heads, "dim": dim, "rank": rank}


def _moe(experts, top, ff, limit, identity=None, shared=None):
    m = {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}
    if identity is not None:
        m["router"]["identity"] = identity
    if shared is not None:
        m["shared"] = {"ff": shared[0], "limit": shared[1]}
    return m


MIXED = {
    "architecture": "Fusanex", "vocab": 200, "width": 64, "embedding": {"scale": 6.0}, "norm": {"eps": 1e-5, "groups": 4},
    "layers": [
        {"type": "rglru", "mixer": _lru(48, 3, 4), "mlp": _moe(6, 2, 40, 1.5, 2, (24, 0.7))},
        {"type": "parallel", "mixer": _par(_att(4, 2, 16, 24, 0.3, (0.7, 16)), _mix(2, 24, 12), 0.8, 0.4), "mlp": _moe(6, 2, 40, 1.5, 2, (24, 0.7))},
        {"type": "rglru", "mixer": _lru(64, 1, 3), "mlp": None},
        {"type": "parallel", "mixer": _par(_att(2, None, 16), _mix(3, 16, 8), 0.7, -0.6), "mlp": _moe(4, 1, 32, 2.0, 1, (40, 1.0))},
        {"type": "rglru", "mixer": _lru(32, 4, 4), "mlp": _moe(5, 3, 24, 1.0, 3)},
    ],
}

ODD = {
    "architecture": "Fusanex", "vocab": 77, "width": 50, "embedding": {"scale": 2.5}, "norm": {"eps": 1e-6, "groups": 5},
    "layers": [
        {"type": "parallel", "mixer": _par(_att(5, 1, 10, 6, 0.35, (0.4, 5)), _mix(3, 10, 5), 0.5, 0.9), "mlp": _moe(3, 3, 14, 0.8, 2, (10, 1.3))},
        {"type": "rglru", "mixer": _lru(30, 3, 2), "mlp": _moe(3, 1, 14, 0.8, 1, (6, 2.0))},
        {"type": "rglru", "mixer": _lru(21, 1, 5), "mlp": _moe(3, 2, 9, 1.2)},
    ],
}

BARE = {
    "architecture": "Fusanex", "vocab": 90, "width": 40, "norm": {"eps": 1e-5},
    "layers": [
        {"type": "parallel", "mixer": _par(_att(3, 3, 16), _mix(2, 8, 4)), "mlp": _moe(2, 2, 24, 1.0)},
        {"type": "rglru", "mixer": _lru(24, 1, 1), "mlp": None},
        {"type": "parallel", "mixer": _par(_att(2, 1, 8, None, None), _mix(1, 16, 8), 1.0, 0.5), "mlp": None},
    ],
}

HEADS64 = {
    "architecture": "Fusanex", "vocab": 120, "width": 128, "embedding": {"scale": 4.0}, "norm": {"eps": 1e-6, "groups": 2},
    "layers": [
        {"type": "parallel", "mixer": _par(_att(6, 2, 64, None, 0.125, (0.5, 8)), _mix(2, 64, 16), 0.6, 0.7), "mlp": _moe(4, 2, 64, 1.0, 2, (32, 1.0))},
        {"type": "rglru", "mixer": _lru(128, 2, 4), "mlp": _moe(4, 1, 64, 1.0, 1, (64, 1.0))},
        {"type": "parallel", "mixer": _par(_att(4, 4, 64, None, 0.125), _mix(1, 64, 8), 0.9, 0.3), "mlp": _moe(6, 3, 32, 1.0)},
    ],
}

CONFIGS = {"mixed": MIXED, "odd": ODD, "bare": BARE, "heads64": HEADS64}
SEEDS = {"mixed": 51, "odd": 52, "bare": 53, "heads64": 54}


def shaped_weights(cfg: dict, seed: int) -> dict:
    """Random tensors by name.  Matrices N(0, 0.1); gains of all norms around one; the recurrences' forgetting rates and the time
    mixing's decays spread from fast to very slow; blends inside (0, 1); gates, routers and corrections large enough to decide."""
    from wllm_b200.weights import random_tensors
    tensors = random_tensors(cfg, seed, dtype=torch.float32, std=0.1, vector_std=0.3)
    g = torch.Generator().manual_seed(seed + 1000)
    for key, t in tensors.items():
        if key.endswith(("norm", "norm1", "norm2")):
            tensors[key] = 1.0 + t
        elif ".mu." in key:
            tensors[key] = torch.rand(t.shape, generator=g)
        elif key.endswith(".lam"):
            tensors[key] = torch.rand(t.shape, generator=g) * 6.0 - 6.5
        elif key.endswith(".w0"):
            tensors[key] = torch.rand(t.shape, generator=g) * 6.0 - 5.0
        elif key.endswith((".mix.conv", ".mix.ra", ".mix.ri", ".router", ".w1", ".w2")):
            tensors[key] = t * 4.0
        elif key.endswith(".right.u"):
            tensors[key] = t * 3.0
        elif key.endswith((".mix.o", ".left.o", ".right.o", ".down", ".gate", ".up")):
            tensors[key] = t * 2.0
        elif key.endswith(".correction"):
            tensors[key] = t * 0.5
    return tensors


def write_tensors(folder: str, cfg: dict, tensors: dict, dtype=torch.bfloat16) -> str:
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w", encoding="utf-8") as f:
        json.dump(cfg, f)
    save_file({k: v.to(dtype).contiguous() for k, v in tensors.items()}, os.path.join(folder, "model.safetensors"))
    return folder


def write_folder(folder: str, name: str, dtype=torch.bfloat16) -> str:
    cfg = copy.deepcopy(CONFIGS[name])
    return write_tensors(folder, cfg, shaped_weights(cfg, SEEDS[name]), dtype)
