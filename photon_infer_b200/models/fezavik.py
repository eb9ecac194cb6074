"""The Fezavik decoder as a ``ModelSpec``.

Layers with an RMS norm before and behind every sublayer: ``x <- x + norm1b(mixer(norm1(x)))``, then ``x <- x +
norm2b(ff(norm2(x)))``.  The mixer is grouped-query attention with queries and keys normed over their whole projections,
neighbouring rotation pairs with stretched frequencies, a window and a learned sink (``parts/normed_attention.py``); attention
over a cached latent with a window, a learned sink and one output gate per head (``parts/latent_attention.py``); or linear
attention whose forget gate also decides what is written (``parts/hgrn2.py``).  The feed-forward is a mixture of gated experts
behind a softmax router whose choice has a correction and whose last outputs may be identity experts (``parts/moe.py``), or
absent.  A final RMS norm and an untied output head.

Tensor names: ``embed``, ``head``, ``final.norm``, and per layer ``l<i>.norm1``, ``l<i>.norm1b``, ``l<i>.norm2``, ``l<i>.norm2b``,
``l<i>.mix.*``, ``l<i>.mlp.*``.
"""
from __future__ import annotations

from typing import Optional

from ..config.fezavik_config import FezavikConfig, FezavikLayer
from ..config.registry import register_architecture
from .spec import LayerSpec, ModelSpec, PartSpec, RunEntry


def _scaling(rot: dict) -> Optional[dict]:
    s = rot.get("scaling")
    return None if s is None else {"factor": s["factor"], "low_freq_factor": s["low"], "high_freq_factor": s["high"],
                                   "original_max_position_embeddings": s["original"]}


def _mixer(cfg: FezavikConfig, layer: FezavikLayer) -> PartSpec:
    m = layer.mixer
    params = dict(hidden_size=cfg.width, eps=cfg.norm_eps)
    if layer.type == "hgrn2":
        return PartSpec("hgrn2", dict(params, heads=m["heads"], dim=m["dim"], vdim=m["vdim"]), "mix.")
    rot = m.get("rot") or {}
    params.update(scale=m["scale"], window=(m.get("mask") or {}).get("size"), rot_scaling=_scaling(rot))
    if layer.type == "latent_attention":
        return PartSpec("latent_attention",
                        dict(params, heads=m["heads"], dim=m["dim"], rot_dim=m["rot_dim"], vdim=m["vdim"], kv_rank=m["kv_rank"],
                             q_rank=m["q_rank"], rot_base=rot["base"], rot_dims=rot["dims"], output_gate="head", sink=True), "mix.")
    return PartSpec("normed_attention",
                    dict(params, n_q_heads=m["heads"], n_kv_heads=m["kv_heads"], head_dim=m["dim"], value_dim=m["vdim"],
                         norm_weight=True, norm_scope="row", rot_dims=rot.get("dims", 0), rot_base=rot.get("base", 10000.0),
                         rot_interleaved=True, sink="learned"), "mix.")


def _feed_forward(cfg: FezavikConfig, mlp: Optional[dict]) -> Optional[PartSpec]:
    if mlp is None:
        return None
    r = mlp["router"]
    return PartSpec("moe", dict(hidden_size=cfg.width, experts=r["experts"], top=r["top"], expert_size=mlp["expert"]["ff"],
                                activation="silu", router_bias=False, scoring="softmax_raw", correction=True,
                                identity=r.get("identity", 0)), "mlp.")


def build_fezavik_spec(cfg: FezavikConfig) -> ModelSpec:
    norm = lambda name: PartSpec("rms_norm", {"size": cfg.width, "eps": cfg.norm_eps, "weight_name": name})
    layers, ignored = [], []
    for i, l in enumerate(cfg.layers):
        ff = _feed_forward(cfg, l.mlp)
        second = lambda name: norm(name) if ff is not None else None
        layers.append(LayerSpec(block=PartSpec("sandwich", {}), norm1=norm("norm1"), mixer=_mixer(cfg, l), norm2=second("norm2"),
                                feed_forward=ff, prefix=f"l{i}.", post1=norm("norm1b"), post2=second("norm2b")))
        if ff is None:                          # files may carry the unused second pair of norms of such a layer
            ignored += [f"l{i}.norm2", f"l{i}.norm2b"]
    return ModelSpec(hidden_size=cfg.width, vocab_size=cfg.vocab, max_position=cfg.max_positions, embedding_name="embed",
                     head_name="head", final_norm=norm("final.norm"), position_encodings={}, layers=layers,
                     run=[RunEntry(i) for i in range(len(layers))], ignored_tensors=tuple(ignored))


register_architecture("Fezavik", FezavikConfig, build_fezavik_spec, replace=True)
