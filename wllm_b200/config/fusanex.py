"""Fusanex configuration, read from its own config.json keys.

    architecture     "Fusanex"
    vocab, width     sizes of the vocabulary and of the residual stream
    embedding.scale  factor on the token's embedding row (absent: 1)
    norm.eps         the eps of every root-mean-square norm of the model
    norm.groups      equal parts of a row that are normed by themselves (absent: 1)
    layers[i]        {"type": "rglru" | "parallel", "mixer": {...}, "mlp": {...} or null}

Mixer `rglru`: width (channels of the recurrence), blocks (equal parts of them with gate maps of their own), conv (taps).
Mixer `parallel`: left {heads, kv_heads (default heads), dim, vdim (default dim), scale (default dim^-1/2), q_temp {coef, every} (absent:
queries are not scaled by position)}, right {heads, dim, rank (of the decay's low-rank map; absent: the checkpoint's)}, left_scale, right_scale
(default 1).
mlp: {"kind": "moe", "expert": {"ff": n, "limit": l}, "router": {"experts": E, "top": k, "identity": m (absent: 0)},
"shared": {"ff": n, "limit": l} (absent: no shared expert)}.
Whatever a config.json leaves out does not exist.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass

from .base import ConfigError, ConfigReader

MIXER_TYPES = ("rglru", "parallel")


def _sub(r: ConfigReader, raw, where: str):
    if not isinstance(raw, dict):
        r.complain(f"{where} must be an object")
        return None
    return ConfigReader(raw, where)


def _take(r: ConfigReader, sub: ConfigReader) -> None:
    r.problems.extend(f"{sub.where}: {p}" for p in sub.problems)
    sub.problems = []


def _left(r: ConfigReader, raw, where: str) -> dict:
    sub = _sub(r, raw, where)
    if sub is None:
        return {}
    heads = sub.integer("heads")
    kv = sub.integer("kv_heads", default=heads)
    if heads and kv and heads % kv:
        r.complain(f"{where}: {heads} heads are no multiple of {kv} kv_heads")
    dim = sub.integer("dim")
    out = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": sub.integer("vdim", default=dim),
           "scale": sub.number("scale", default=(float(dim) ** -0.5 if dim else None), positive=False)}
    if raw.get("q_temp") is not None:
        temp = _sub(r, raw["q_temp"], where + ".q_temp")
        if temp is not None:
            out["q_temp"] = {"coef": temp.number("coef", positive=False), "every": temp.integer("every")}
            _take(r, temp)
    _take(r, sub)
    return out


def _right(r: ConfigReader, raw, where: str) -> dict:
    sub = _sub(r, raw, where)
    if sub is None:
        return {}
    out = {"heads": sub.integer("heads"), "dim": sub.integer("dim")}
    rank = sub.optional_integer("rank")
    if rank is not None:
        out["rank"] = rank
        if rank < 1:
            r.complain(f"{where}: rank {rank} must be >= 1")
    _take(r, sub)
    return out


def _mixer(r: ConfigReader, kind: str, raw, where: str) -> dict:
    sub = _sub(r, raw, where)
    if sub is None:
        return {}
    if kind == "rglru":
        out = {"width": sub.integer("width"), "blocks": sub.integer("blocks"), "conv": sub.integer("conv")}
        if out["width"] and out["blocks"] and out["width"] % out["blocks"]:
            r.complain(f"{where}: width {out['width']} is no multiple of {out['blocks']} blocks")
    else:
        out = {"left": _left(r, raw.get("left"), where + ".left"), "left_scale": sub.number("left_scale", default=1.0, positive=False),
               "right": _right(r, raw.get("right"), where + ".right"), "right_scale": sub.number("right_scale", default=1.0, positive=False)}
    _take(r, sub)
    return out


def _unit(r: ConfigReader, raw, where: str) -> dict:
    sub = _sub(r, raw, where)
    if sub is None:
        return {}
    out = {"ff": sub.integer("ff"), "limit": sub.number("limit")}
    _take(r, sub)
    return out


def _mlp(r: ConfigReader, raw, where: str):
    if raw is None:
        return None
    if not isinstance(raw, dict) or raw.get("kind") != "moe":
        r.complain(f"{where}.kind must be 'moe' (or mlp null)")
        return None
    out = {"kind": "moe", "expert": _unit(r, raw.get("expert"), where + ".expert"), "router": {}}
    router = _sub(r, raw.get("router"), where + ".router")
    if router is not None:
        out["router"] = {"experts": router.integer("experts"), "top": router.integer("top"), "identity": router.integer("identity", default=0, minimum=0)}
        _take(r, router)
        e, m, top = out["router"]["experts"], out["router"]["identity"], out["router"]["top"]
        if e and top and m is not None and top > e + m:
            r.complain(f"{where}.router: top {top} of {e + m} experts")
    if raw.get("shared") is not None:
        out["shared"] = _unit(r, raw["shared"], where + ".shared")
    return out


@dataclass(frozen=True)
class FusanexConfig:
    vocab: int
    width: int
    embedding_scale: float
    eps: float
    norm_groups: int
    layers: tuple            # of checked layer dictionaries (see the module's text)

    architecture = "Fusanex"

    @classmethod
    def from_dict(cls, raw: dict, where: str = "config.json") -> "FusanexConfig":
        r = ConfigReader(raw, where)
        vocab, width = r.integer("vocab"), r.integer("width")
        eps, groups, scale = None, 1, 1.0
        norm = _sub(r, raw.get("norm"), "norm")
        if norm is not None:
            eps, groups = norm.number("eps"), norm.integer("groups", default=1)
            _take(r, norm)
            if width and groups and width % groups:
                r.complain(f"norm.groups: width {width} is no multiple of {groups} groups")
        if raw.get("embedding") is not None:
            emb = _sub(r, raw["embedding"], "embedding")
            if emb is not None:
                scale = emb.number("scale", default=1.0, positive=False)
                _take(r, emb)
        layers = raw.get("layers")
        if not isinstance(layers, list) or not layers:
            r.complain("'layers' must be a list with at least one layer")
            layers = []
        checked = []
        for i, layer in enumerate(layers):
            at = f"layers[{i}]"
            if not isinstance(layer, dict) or layer.get("type") not in MIXER_TYPES:
                r.complain(f"{at}.type must be one of {', '.join(MIXER_TYPES)}")
                continue
            checked.append({"type": layer["type"], "mixer": _mixer(r, layer["type"], layer.get("mixer"), at + ".mixer"),
                            "mlp": _mlp(r, layer.get("mlp"), at + ".mlp")})
        r.finish()
        return cls(vocab=vocab, width=width, embedding_scale=scale, eps=eps, norm_groups=groups, layers=tuple(checked))

    def to_dict(self) -> dict:
        return {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "embedding": {"scale": self.embedding_scale},
                "norm": {"eps": self.eps, "groups": self.norm_groups}, "layers": copy.deepcopy(list(self.layers))}


__all__ = ["FusanexConfig", "ConfigError"]
