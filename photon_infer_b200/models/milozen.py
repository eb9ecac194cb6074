"""The Milozen decoder as a ``ModelSpec``.

Embedding rows times ``embedding.scale`` enter ``streams`` parallel residual streams, all equal at first.  Every sublayer
reads a learned mixture of the streams through a layer norm (weight, no bias) and writes its output back into all of them,
which are mixed with each other at the same time (``parts/hyper.py``).  The mixer is attention over a cached latent with
neighbouring rotation pairs, a window and an output gate (``parts/latent_attention.py``); a layer may read an earlier
layer's cached rows.  The feed-forward is dense with silu gates, a mixture of experts with bounded activations whose
routing score multiplies the expert's input (``parts/moe.py``), or absent.  At the end the streams are summed, normed and
multiplied with the embedding table.

Tensor names: ``embed``, ``final.norm``, and per layer ``l<i>.norm1``, ``l<i>.norm2``, ``l<i>.hc1.*``, ``l<i>.hc2.*``,
``l<i>.mix.*``, ``l<i>.mlp.*``.
"""
from __future__ import annotations

from typing import Optional

from ..config.milozen_config import MilozenConfig
from ..config.registry import register_architecture
from .spec import LayerSpec, ModelSpec, PartSpec, RunEntry

#: slope of the sigmoid in the experts' gate, ``g * sigmoid(1.702 g)``
EXPERT_GATE_SLOPE = 1.702


def _window(m: dict) -> Optional[int]:
    return (m.get("mask") or {}).get("size")


def _cache_window(cfg: MilozenConfig, index: int) -> Optional[int]:
    """Rows that layer ``index`` must keep: the largest window among itself and the layers that read its pages."""
    sizes = [_window(cfg.layers[index].mixer)]
    sizes += [_window(l.mixer) for l in cfg.layers if l.mixer.get("kv_from") == index]
    return None if any(s is None for s in sizes) else max(sizes)


def _mixer(cfg: MilozenConfig, index: int) -> PartSpec:
    m = cfg.layers[index].mixer
    own = m.get("kv_from") is None
    return PartSpec("latent_attention",
                    dict(hidden_size=cfg.width, heads=m["heads"], dim=m["dim"], rot_dim=m["rot_dim"], vdim=m["vdim"],
                         kv_rank=m["kv_rank"], q_rank=m["q_rank"], scale=m["scale"], eps=cfg.norm_eps,
                         rot_base=m["rot"]["base"], rot_dims=m["rot"]["dims"], rot_interleaved=True, window=_window(m),
                         cache_window=_cache_window(cfg, index) if own else "own", own_kv=own, output_gate=True), "mix.")


def _feed_forward(cfg: MilozenConfig, mlp: Optional[dict]) -> Optional[PartSpec]:
    if mlp is None:
        return None
    if mlp["kind"] == "dense":
        return PartSpec("gated", dict(hidden_size=cfg.width, intermediate_size=mlp["ff"], activation="silu",
                                      names=("gate", "up", "down")), "mlp.")
    return PartSpec("moe", dict(hidden_size=cfg.width, experts=mlp["router"]["experts"], top=mlp["router"]["top"],
                                expert_size=mlp["expert"]["ff"], activation="clamped_swish", act_limit=mlp["expert"]["limit"],
                                act_slope=EXPERT_GATE_SLOPE, router_bias=False, scoring="sigmoid", weight_input=True), "mlp.")


def build_milozen_spec(cfg: MilozenConfig) -> ModelSpec:
    norm = lambda name: PartSpec("layer_norm", {"size": cfg.width, "eps": cfg.norm_eps, "weight_name": name, "bias_name": None})
    connect = lambda prefix: PartSpec("hyper", {"streams": cfg.streams}, prefix)
    layers, run, ignored = [], [], []
    for i, l in enumerate(cfg.layers):
        ff = _feed_forward(cfg, l.mlp)
        layers.append(LayerSpec(block=PartSpec("hyper_pre_norm", {}), norm1=norm("norm1"), mixer=_mixer(cfg, i),
                                norm2=norm("norm2") if ff is not None else None, feed_forward=ff, prefix=f"l{i}.",
                                connect1=connect("hc1."), connect2=connect("hc2.") if ff is not None else None))
        run.append(RunEntry(i, kv_from=l.mixer.get("kv_from")))
        if ff is None:                          # files may carry the unused second norm and connection of such a layer
            ignored += [f"l{i}.norm2", f"l{i}.hc2.*"]
    return ModelSpec(hidden_size=cfg.width, vocab_size=cfg.vocab, max_position=cfg.max_positions, embedding_name="embed",
                     head_name=None, final_norm=norm("final.norm"), position_encodings={}, layers=layers, run=run,
                     embedding_scale=cfg.embedding_scale, ignored_tensors=tuple(ignored))


register_architecture("Milozen", MilozenConfig, build_milozen_spec, replace=True)
