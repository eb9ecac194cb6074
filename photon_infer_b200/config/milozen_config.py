"""Typed configuration of the Milozen decoder, read from the keys of its ``config.json``.

Nested like the file: ``architecture``, ``vocab``, ``width``, ``streams`` (parallel residual streams), ``norm.eps``, optional
``embedding.scale`` (default 1), and ``layers`` (one object per layer: ``type`` names the mixer, ``mixer`` holds its sizes
and constants, ``mlp`` its feed-forward or null).  Every size and constant is read here; errors name the key.  What the
file leaves out does not exist (no window, no feed-forward).

Mixer ``latent_attention``: ``heads``, ``dim`` and ``rot_dim`` (unrotated and rotated numbers of a query or key), ``vdim``,
``kv_rank`` and ``q_rank`` (latents), ``scale``, ``rot`` (``base``, ``dims``: rotated numbers of the ``rot_dim`` part, paired with
their neighbours), optional ``mask.size`` (the window), optional ``kv_from`` (an earlier layer whose cached latent and
rotated key part this one reads).

Feed-forward ``kind`` ``dense``: ``ff``.  ``kind`` ``moe``: ``expert.ff``, ``expert.limit`` (the bound of the experts'
activation), ``router.experts``, ``router.top``.  Optional top-level ``max_positions`` bounds a request's length.
"""
from __future__ import annotations

import copy
import dataclasses
from typing import Any, Dict, Optional, Tuple

from .nested import bad, num, obj

MIXER_TYPES = ("latent_attention",)
DEFAULT_MAX_POSITIONS = 131072


def _check_mixer(m: Any, where: str, index: int, before) -> Dict[str, Any]:
    if not isinstance(m, dict):
        raise bad(f"'{where}' must be an object")
    out: Dict[str, Any] = {k: num(m, k, where) for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank", "q_rank")}
    out["scale"] = num(m, "scale", where, float)
    rot = obj(m, "rot", where, required=True)
    out["rot"] = {"base": num(rot, "base", where + ".rot", float),
                  "dims": num(rot, "dims", where + ".rot", default=out["rot_dim"])}
    if out["rot"]["dims"] % 2 or out["rot"]["dims"] > out["rot_dim"]:
        raise bad(f"'{where}.rot.dims' must be even and at most rot_dim")
    mask = obj(m, "mask", where)
    if mask is not None:
        out["mask"] = {"size": num(mask, "size", where + ".mask")}
    if m.get("kv_from") is not None:
        src = num(m, "kv_from", where, positive=False)
        if not 0 <= src < index or "kv_from" in before[src].mixer:
            raise bad(f"'{where}.kv_from' must name an earlier layer that has a latent of its own")
        for key in ("kv_rank", "rot_dim", "rot"):
            if before[src].mixer[key] != out[key]:
                raise bad(f"'{where}.{key}' must equal that of layer {src}, whose latent it reads")
        out["kv_from"] = src
    return out


def _check_mlp(m: Any, where: str) -> Optional[Dict[str, Any]]:
    if m is None:
        return None
    if not isinstance(m, dict):
        raise bad(f"'{where}' must be an object or null")
    kind = m.get("kind")
    if kind == "dense":
        return {"kind": "dense", "ff": num(m, "ff", where)}
    if kind != "moe":
        raise bad(f"key '{where}.kind' must be 'dense' or 'moe', got {kind!r}")
    r = obj(m, "router", where, required=True)
    router = {"experts": num(r, "experts", where + ".router"), "top": num(r, "top", where + ".router")}
    if router["top"] > router["experts"]:
        raise bad(f"'{where}.router.top' cannot exceed the number of experts")
    e = obj(m, "expert", where, required=True)
    return {"kind": "moe", "expert": {"ff": num(e, "ff", where + ".expert"), "limit": num(e, "limit", where + ".expert", float)},
            "router": router}


@dataclasses.dataclass(frozen=True)
class MilozenLayer:
    type: str
    mixer: Dict[str, Any]
    mlp: Optional[Dict[str, Any]]


@dataclasses.dataclass(frozen=True)
class MilozenConfig:
    architecture: str
    vocab: int
    width: int
    streams: int
    norm_eps: float
    layers: Tuple[MilozenLayer, ...]
    embedding_scale: float = 1.0
    max_positions: int = DEFAULT_MAX_POSITIONS

    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "MilozenConfig":
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
            layers.append(MilozenLayer(l["type"], _check_mixer(l.get("mixer"), where + ".mixer", i, layers),
                                       _check_mlp(l.get("mlp"), where + ".mlp")))
        norm = obj(d, "norm", "config", required=True)
        emb = obj(d, "embedding", "config") or {}
        return cls(architecture=name, vocab=num(d, "vocab", "config"), width=num(d, "width", "config"),
                   streams=num(d, "streams", "config"), norm_eps=num(norm, "eps", "norm", float), layers=tuple(layers),
                   embedding_scale=num(emb, "scale", "embedding", float, positive=False, default=1.0),
                   max_positions=num(d, "max_positions", "config", default=DEFAULT_MAX_POSITIONS))

    def to_dict(self) -> Dict[str, Any]:
        d: Dict[str, Any] = {
            "architecture": self.architecture, "vocab": self.vocab, "width": self.width, "streams": self.streams,
            "norm": {"eps": self.norm_eps}, "embedding": {"scale": self.embedding_scale},
            "layers": [{"type": l.type, "mixer": copy.deepcopy(l.mixer), "mlp": copy.deepcopy(l.mlp)} for l in self.layers],
        }
        if self.max_positions != DEFAULT_MAX_POSITIONS:
            d["max_positions"] = self.max_positions
        return d
