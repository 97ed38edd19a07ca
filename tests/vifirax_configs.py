"""Small Vifirax configurations for the tests, and folders with weights made so that every mechanism matters.

'mixed'      a state space with grouped B and C rows and three norm groups, a delta rule with fewer query/key than value heads, an
             attention layer whose values have a size of their own, a second one on its keys and values with more query heads and a
             scale of its own (dense and routed feed-forwards, a layer without one), a second state space with one group
'odd'        sizes in no step of 4 or 8 (width 50, heads of 10 and 6, states of 7 rows, low-rank maps of ranks 5 and 3, parts of 15, a
             feed-forward of 14, 3 experts, convolutions of 2 and 5 taps), a turn over 6 of 10 elements whose bands meet at once
'bare'       what a file may leave out is left out: no turn, no factor on the logits, one group everywhere; convolutions of one tap (no
             inputs kept), every expert chosen (top = experts), layers that begin with attention
'heads64'    attention heads of 64 elements with values of the same size and the whole head turned, unscaled frequencies in one
             layer and scaled ones in the next, a state of 128 rows, delta heads of 64 by 64, 12 experts
'recurrent'  no attention at all: no pages, only state
"""
from __future__ import annotations

import copy
import json
import os

import torch
from safetensors.torch import save_file


def _rot(dims, base, factor=None, original=None, fast=None, slow=None):
    rot = {"dims": dims, "base": base}
    if factor is not None:
        rot["scaling"] = {"factor": factor, "original": original, "fast": fast, "slow": slow}
    return rot


def _att(heads, kv, dim, vdim=None, scale=None, rot=None, kv_from=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim}
    for key, value in (("vdim", vdim), ("scale", scale), ("rot", rot), ("kv_from", kv_from)):
        if value is not None:
            m[key] = value
    return {"type": "attention", "mixer": m}


def _ssm(heads, vdim, state, conv, groups=None, norm_groups=None):
    m = {"heads": heads, "vdim": vdim, "state": state, "conv": conv}
    if groups is not None:
        m["groups"] = groups
    if norm_groups is not None:
        m["norm_groups"] = norm_groups
    return {"type": "mamba2", "mixer": m}


def _delta(heads, kv, dim, vdim, conv, decay_rank, gate_rank):
    return {"type": "channel_delta", "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "conv": conv, "decay_rank": decay_rank,
                                               "gate_rank": gate_rank}}


def _with(layer, mlp):
    return {**layer, "mlp": mlp}


def _ff(n):
    return {"kind": "dense", "ff": n}


def _moe(experts, top, ff):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


NEAR = _rot(12, 500.0, 3.0, 64, 8.0, 1.0)          # bands that differ within a few hundred positions

MIXED = {
    "architecture": "Vifirax", "vocab": 200, "width": 64, "norm": {"eps": 1e-5}, "logit_scale": 0.6,
    "layers": [
        _with(_ssm(4, 24, 16, 4, 2, 3), _moe(6, 2, 40)),
        _with(_delta(4, 2, 16, 24, 3, 8, 16), _ff(48)),
        _with(_att(4, 2, 32, 24, 0.3, NEAR), None),
        _with(_att(8, 2, 32, 24, 0.22, NEAR, 2), _moe(5, 3, 32)),
        _with(_ssm(6, 16, 24, 3, 1, 1), _ff(56)),
    ],
}

ODD = {
    "architecture": "Vifirax", "vocab": 77, "width": 50, "norm": {"eps": 1e-6}, "logit_scale": 1.7,
    "layers": [
        _with(_att(5, 1, 10, 6, 0.35, _rot(6, 50.0, 5.0, 20, 3.0, 2.9)), _moe(3, 1, 14)),
        _with(_delta(3, 1, 10, 6, 5, 5, 3), _ff(14)),
        _with(_ssm(3, 10, 7, 2, 3, 2), _moe(3, 2, 14)),
        _with(_att(2, 1, 10, 6, 0.5, _rot(6, 50.0, 5.0, 20, 3.0, 2.9), 0), _ff(30)),
    ],
}

BARE = {
    "architecture": "Vifirax", "vocab": 90, "width": 40, "norm": {"eps": 1e-5},
    "layers": [
        _with(_att(3, 3, 16), _moe(2, 2, 24)),
        _with(_delta(2, 2, 8, 8, 1, 4, 4), None),
        _with(_ssm(2, 8, 8, 1), _ff(24)),
    ],
}

HEADS64 = {
    "architecture": "Vifirax", "vocab": 120, "width": 64, "norm": {"eps": 1e-6}, "logit_scale": 0.5,
    "layers": [
        _with(_ssm(4, 64, 128, 4, 2, 4), _ff(64)),
        _with(_att(6, 2, 64, None, 0.125, _rot(64, 10000.0)), _moe(12, 4, 32)),
        _with(_delta(2, 1, 64, 64, 4, 16, 24), _ff(64)),
        _with(_att(4, 4, 64, None, None, _rot(64, 10000.0, 8.0, 256, 16.0, 2.0)), _moe(4, 1, 64)),
        _with(_att(8, 4, 64, None, 0.2, _rot(64, 10000.0, 8.0, 256, 16.0, 2.0), 3), _ff(40)),
    ],
}

RECURRENT = {
    "architecture": "Vifirax", "vocab": 100, "width": 48, "norm": {"eps": 1e-5}, "logit_scale": 0.8,
    "layers": [
        _with(_delta(4, 4, 16, 16, 4, 8, 8), _ff(32)),
        _with(_ssm(3, 16, 16, 4, 1, 3), _moe(4, 2, 24)),
    ],
}

CONFIGS = {"mixed": MIXED, "odd": ODD, "bare": BARE, "heads64": HEADS64, "recurrent": RECURRENT}
SEEDS = {"mixed": 61, "odd": 62, "bare": 63, "heads64": 64, "recurrent": 65}


def write_folder(folder: str, name: str, dtype=torch.bfloat16) -> str:
    """config.json and model.safetensors.  Matrices N(0, 0.1); the norms behind the sublayers around zero, plain gains around
    one; steps and decays such that heads and channels forget within a few and within hundreds of tokens; biases large enough to
    matter; the routers' biases two apart and their products of order one, so that the choice follows both and seldom nearly ties (a tie that
    the rounded input breaks the other way is carried on by the recurrences behind it); the embedding of order one (it is the head too)."""
    from wllm_b200.weights import random_tensors
    cfg = copy.deepcopy(CONFIGS[name])
    tensors = random_tensors(cfg, SEEDS[name], dtype=torch.float32, std=0.1, vector_std=0.3)
    g = torch.Generator().manual_seed(SEEDS[name] + 1000)
    kinds = {f"l{i}.": layer["type"] for i, layer in enumerate(cfg["layers"])}
    for key, t in tensors.items():
        kind = kinds.get(key.split(".")[0] + ".")
        if key.endswith((".q.norm", ".k.norm", ".mix.norm")):
            tensors[key] = 1.0 + t
        elif key.endswith((".norm1", ".norm2")):
            tensors[key] = t - 0.3
        elif key.endswith((".q.b", ".k.b", ".v.b", ".o.b")):
            tensors[key] = t * 2.0
        elif key.endswith(".conv"):
            tensors[key] = t * 5.0
        elif key.endswith((".mix.b", ".mix.g", ".a1", ".a2", ".g1", ".g2")):
            tensors[key] = t * 4.0
        elif key.endswith(".router"):
            tensors[key] = t * 1.3
        elif key.endswith(".router.b"):
            tensors[key] = (torch.randperm(len(t), generator=g) - 0.5 * len(t)) * 2.0
        elif key.endswith(".A_log"):
            tensors[key] = torch.rand(t.shape, generator=g) * 2.0 - 1.0
        elif key.endswith(".dt_bias"):
            tensors[key] = torch.rand(t.shape, generator=g) * 5.0 - 5.0 if kind == "channel_delta" else torch.rand(t.shape, generator=g) * 4.0 - 4.0
        elif key.endswith(".D"):
            tensors[key] = 1.0 + t
        elif key == "embed":
            tensors[key] = t * 10.0
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w", encoding="utf-8") as f:
        json.dump(cfg, f)
    save_file({k: v.to(dtype).contiguous() for k, v in tensors.items()}, os.path.join(folder, "model.safetensors"))
    return folder
