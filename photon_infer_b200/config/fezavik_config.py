"""Typed configuration of the Fezavik decoder, read from the keys of its ``config.json``.

Nested like the file: ``architecture``, ``vocab``, ``width``, ``norm.eps`` and ``layers`` (one object per layer: ``type`` names the
mixer, ``mixer`` holds its sizes and constants, ``mlp`` its feed-forward or null).  Every size and constant is read here;
errors name the key.  What the file leaves out does not exist (no window, no rotation, no identity experts).

Mixers:

* ``attention``: ``heads``, ``kv_heads``, ``dim`` (queries and keys), ``vdim`` (values), ``scale``, optional ``rot`` (``base``,
  ``dims``: rotated numbers of a head, pairs of neighbours; optional ``scaling``: ``factor``, ``low``, ``high``, ``original``),
  optional ``mask.size`` (the window);
* ``latent_attention``: ``heads``, ``dim`` and ``rot_dim`` (unrotated and rotated numbers of a query or key), ``vdim``, ``kv_rank`` and
  ``q_rank`` (latents), ``scale``, ``rot`` (``base``, ``dims``: rotated numbers of the ``rot_dim`` part, paired in halves), optional
  ``mask.size``;
* ``hgrn2``: ``heads``, ``dim``, ``vdim``.

Feed-forward ``kind`` ``moe``: ``expert.ff``, ``router.experts``, ``router.top``, optional ``router.identity`` (experts that return
their input).  Optional top-level ``max_positions`` bounds a request's length.
"""
from __future__ import annotations

import copy
import dataclasses
from typing import Any, Dict, Optional, Tuple

from .nested import bad, num, obj

MIXER_TYPES = ("attention", "latent_attention", "hgrn2")
DEFAULT_MAX_POSITIONS = 131072


def _check_rot(m: Dict[str, Any], where: str, most: int, most_name: str, default_dims: Optional[int] = None) -> Optional[Dict[str, Any]]:
    rot = obj(m, "rot", where, required=default_dims is not None)
    if rot is None:
        return None
    at = where + ".rot"
    out: Dict[str, Any] = {"base": num(rot, "base", at, float), "dims": num(rot, "dims", at, default=default_dims)}
    if out["dims"] % 2 or out["dims"] > most:
        raise bad(f"'{at}.dims' must be even and at most {most_name}")
    scaling = obj(rot, "scaling", at)
    if scaling is not None:
        out["scaling"] = {k: num(scaling, k, at + ".scaling", float) for k in ("factor", "low", "high", "original")}
        if not out["scaling"]["low"] < out["scaling"]["high"]:
            raise bad(f"'{at}.scaling.low' must be below '{at}.scaling.high'")
    return out


def _check_mixer(kind: str, m: Any, where: str) -> Dict[str, Any]:
    if not isinstance(m, dict):
        raise bad(f"'{where}' must be an object")
    out: Dict[str, Any] = {k: num(m, k, where) for k in ("heads", "dim")}
    out["vdim"] = num(m, "vdim", where, default=out["dim"])
    if kind == "hgrn2":
        return out
    if kind == "attention":
        out["kv_heads"] = num(m, "kv_heads", where, default=out["heads"])
        if out["heads"] % out["kv_heads"]:
            raise bad(f"'{where}.heads' must be a multiple of '{where}.kv_heads'")
        rot = _check_rot(m, where, out["dim"], "dim")
    else:
        out.update({k: num(m, k, where) for k in ("rot_dim", "kv_rank", "q_rank")})
        rot = _check_rot(m, where, out["rot_dim"], "rot_dim", default_dims=out["rot_dim"])
    if rot is not None:
        out["rot"] = rot
    out["scale"] = num(m, "scale", where, float)
    mask = obj(m, "mask", where)
    if mask is not None:
        out["mask"] = {"size": num(mask, "size", where + ".mask")}
    return out


def _check_mlp(m: Any, where: str) -> Optional[Dict[str, Any]]:
    if m is None:
        return None
    if not isinstance(m, dict):
        raise bad(f"'{where}' must be an object or null")
    if m.get("kind") != "moe":
        raise bad(f"key '{where}.kind' must be 'moe', got {m.get('kind')!r}")
    r = obj(m, "router", where, required=True)
    at = where + ".router"
    router = {"experts": num(r, "experts", at), "top": num(r, "top", at)}
    if r.get("identity") is not None:
        router["identity"] = num(r, "identity", at, positive=False)
        if router["identity"] < 0:
            raise bad(f"key '{at}.identity' must not be negative")
    if router["top"] > router["experts"] + router.get("identity", 0):
        raise bad(f"'{at}.top' cannot exceed the number of experts, identity experts included")
    e = obj(m, "expert", where, required=True)
    return {"kind": "moe", "expert": {"ff": num(e, "ff", where + ".expert")}, "router": router}


@dataclasses.dataclass(frozen=True)
class FezavikLayer:
    type: str
    mixer: Dict[str, Any]
    mlp: Optional[Dict[str, Any]]


@dataclasses.dataclass(frozen=True)
class FezavikConfig:
    architecture: str
    vocab: int
    width: int
    norm_eps: float
    layers: Tuple[FezavikLayer, ...]
    max_positions: int = DEFAULT_MAX_POSITIONS

    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "FezavikConfig":
        name = d.get("architecture")
        if not isinstance(name, str):
            archs = d.get("architectures")
            if not isinstance(archs, list) or not archs or not isinstance(archs[0], str):
                raise bad("key 'architecture' must name the model class")
            name = archs[0]
        layers_in = d.get("layers")
        if not isinstance(layers_in, list) or not layers_in:
            raise bad("key 'layers' must be a non-empty list")
        layers = []
        for i, l in enumerate(layers_in):
            where = f"layers[{i}]"
            if not isinstance(l, dict) or l.get("type") not in MIXER_TYPES:
                raise bad(f"'{where}.type' must be one of {', '.join(MIXER_TYPES)}")
            layers.append(FezavikLayer(l["type"], _check_mixer(l["type"], l.get("mixer"), where + ".mixer"),
                                       _check_mlp(l.get("mlp"), where + ".mlp")))
        norm = obj(d, "norm", "config", required=True)
        return cls(architecture=name, vocab=num(d, "vocab", "config"), width=num(d, "width", "config"),
                   norm_eps=num(norm, "eps", "norm", float), layers=tuple(layers),
                   max_positions=num(d, "max_positions", "config", default=DEFAULT_MAX_POSITIONS))

    def to_dict(self) -> Dict[str, Any]:
        d: Dict[str, Any] = {
            "architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
            "layers": [{"type": l.type, "mixer": copy.deepcopy(l.mixer), "mlp": copy.deepcopy(l.mlp)} for l in self.layers],
        }
        if self.max_positions != DEFAULT_MAX_POSITIONS:
            d["max_positions"] = self.max_positions
        return d
