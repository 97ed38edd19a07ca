"""Vifirax configuration, read from its own config.json keys.

    architecture     "Vifirax"
    vocab, width     sizes of the vocabulary and of the residual stream
    norm.eps         the eps of every root-mean-square norm of the model
    logit_scale      factor on the logits (absent: 1)
    layers[i]        {"type": "attention" | "mamba2" | "channel_delta", "mixer": {...}, "mlp": {...} or null}

Mixer `attention`: heads, kv_heads (default heads), dim, vdim (default dim), scale (default dim^-1/2), rot {dims, base, scaling {factor,
original, fast, slow} (absent: frequencies as they are)} (absent: nothing turns), kv_from (an earlier attention layer whose keys and
values the layer reads; absent: its own).
Mixer `mamba2`: heads, vdim, state, groups (default 1), conv (taps), norm_groups (default 1).
Mixer `channel_delta`: heads, kv_heads (default heads), dim, vdim, conv (taps), decay_rank and gate_rank (ranks of the two low-rank
maps; absent: the checkpoint's).
mlp: {"kind": "dense", "ff": n} or {"kind": "moe", "expert": {"ff": n}, "router": {"experts": E, "top": k}}.
Whatever a config.json leaves out does not exist.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass

from .base import ConfigError, ConfigReader

MIXER_TYPES = ("attention", "mamba2", "channel_delta")


def _grouped(r: ConfigReader, sub: ConfigReader, where: str) -> dict:
    heads = sub.integer("heads")
    kv = sub.integer("kv_heads", default=heads)
    if heads and kv and heads % kv:
        r.complain(f"{where}: {heads} heads are no multiple of {kv} kv_heads")
    return {"heads": heads, "kv_heads": kv}


def _rotation(r: ConfigReader, raw, where: str, dim):
    sub = r.nested(raw, where)
    if sub is None:
        return None
    out = {"dims": sub.integer("dims", minimum=0), "base": sub.number("base")}
    if out["dims"] is not None and (out["dims"] % 2 or (dim and out["dims"] > dim)):
        r.complain(f"{where}: dims {out['dims']} must be even and at most dim {dim}")
    if raw.get("scaling") is not None:
        scaling = r.nested(raw["scaling"], where + ".scaling")
        if scaling is not None:
            out["scaling"] = {k: scaling.number(k) for k in ("factor", "original", "fast", "slow")}
            if out["base"] == 1.0:
                r.complain(f"{where}: scaled frequencies need a base other than 1")
            r.absorb(scaling)
    r.absorb(sub)
    return out


def _mixer(r: ConfigReader, kind: str, raw, where: str) -> dict:
    sub = r.nested(raw, where)
    if sub is None:
        return {}
    if kind == "attention":
        out = _grouped(r, sub, where)
        dim = sub.integer("dim")
        out.update(dim=dim, vdim=sub.integer("vdim", default=dim),
                   scale=sub.number("scale", default=(float(dim) ** -0.5 if dim else None), positive=False))
        if raw.get("rot") is not None:
            out["rot"] = _rotation(r, raw["rot"], where + ".rot", dim)
        if raw.get("kv_from") is not None:
            out["kv_from"] = sub.integer("kv_from", minimum=0)
    elif kind == "mamba2":
        out = {"heads": sub.integer("heads"), "vdim": sub.integer("vdim"), "state": sub.integer("state"),
               "groups": sub.integer("groups", default=1), "conv": sub.integer("conv"), "norm_groups": sub.integer("norm_groups", default=1)}
        h, v, g, parts = (out[k] for k in ("heads", "vdim", "groups", "norm_groups"))
        if h and g and h % g:
            r.complain(f"{where}: {h} heads are no multiple of {g} groups")
        if h and v and parts and (h * v) % parts:
            r.complain(f"{where}: rows of {h} x {v} cannot be cut into {parts} norm_groups")
    else:
        out = _grouped(r, sub, where)
        out.update(dim=sub.integer("dim"), vdim=sub.integer("vdim"), conv=sub.integer("conv"))
        for key in ("decay_rank", "gate_rank"):
            if raw.get(key) is not None:
                out[key] = sub.integer(key)
    r.absorb(sub)
    return out


def _mlp(r: ConfigReader, raw, where: str):
    if raw is None:
        return None
    if not isinstance(raw, dict) or raw.get("kind") not in ("dense", "moe"):
        r.complain(f"{where}.kind must be 'dense' or 'moe' (or mlp null)")
        return None
    if raw["kind"] == "dense":
        sub = ConfigReader(raw, where)
        out = {"kind": "dense", "ff": sub.integer("ff")}
        r.absorb(sub)
        return out
    expert, router = r.nested(raw.get("expert"), where + ".expert"), r.nested(raw.get("router"), where + ".router")
    out = {"kind": "moe", "expert": {}, "router": {}}
    if expert is not None:
        out["expert"] = {"ff": expert.integer("ff")}
        r.absorb(expert)
    if router is not None:
        out["router"] = {"experts": router.integer("experts"), "top": router.integer("top")}
        r.absorb(router)
        e, top = out["router"]["experts"], out["router"]["top"]
        if e and top and top > e:
            r.complain(f"{where}.router: top {top} of {e} experts")
    return out


def _check_source(r: ConfigReader, layers: list, i: int, at: str) -> None:
    """The layer whose keys and values layer i reads: an earlier attention layer with projections of its own and the same heads."""
    m = layers[i]["mixer"]
    j = m["kv_from"]
    if not 0 <= j < i or layers[j].get("type") != "attention" or layers[j]["mixer"].get("kv_from") is not None:
        r.complain(f"{at}.mixer.kv_from {j} must name an earlier attention layer with keys and values of its own")
        return
    mine, theirs = (tuple(x.get(k) for k in ("kv_heads", "dim", "vdim")) for x in (m, layers[j]["mixer"]))
    if mine != theirs:
        r.complain(f"{at}.mixer: key/value heads {mine} cannot be read from layer {j}, which has {theirs}")


@dataclass(frozen=True)
class VifiraxConfig:
    vocab: int
    width: int
    eps: float
    logit_scale: float
    layers: tuple            # of checked layer dictionaries (see the module's text)

    architecture = "Vifirax"

    @classmethod
    def from_dict(cls, raw: dict, where: str = "config.json") -> "VifiraxConfig":
        r = ConfigReader(raw, where)
        vocab, width = r.integer("vocab"), r.integer("width")
        scale = r.number("logit_scale", default=1.0, positive=False)
        eps = None
        norm = r.nested(raw.get("norm"), "norm")
        if norm is not None:
            eps = norm.number("eps")
            r.absorb(norm)
        layers = raw.get("layers")
        if not isinstance(layers, list) or not layers:
            r.complain("'layers' must be a list with at least one layer")
            layers = []
        checked = []
        for i, layer in enumerate(layers):
            at = f"layers[{i}]"
            if not isinstance(layer, dict) or layer.get("type") not in MIXER_TYPES:
                r.complain(f"{at}.type must be one of {', '.join(MIXER_TYPES)}")
                checked.append({})
                continue
            checked.append({"type": layer["type"], "mixer": _mixer(r, layer["type"], layer.get("mixer"), at + ".mixer"),
                            "mlp": _mlp(r, layer.get("mlp"), at + ".mlp")})
            if checked[i]["mixer"].get("kv_from") is not None:
                _check_source(r, checked, i, at)
        r.finish()
        return cls(vocab=vocab, width=width, eps=eps, logit_scale=scale, layers=tuple(checked))

    def to_dict(self) -> dict:
        return {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.eps},
                "logit_scale": self.logit_scale, "layers": copy.deepcopy(list(self.layers))}


__all__ = ["VifiraxConfig", "ConfigError"]
