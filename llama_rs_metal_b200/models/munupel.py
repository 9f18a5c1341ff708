"""The Munupel decoder as a plan of parts.

Layers are parallel: one layer norm (weight and bias) whose output both sublayers read, x <- x + mixer(h) + ff(h),
h = norm1(x), or the mixer alone. Two kinds of mixer, both softmax attention with grouped key heads, a split-half
rotation of a part of each head, values of their own width and a sigmoid gate on the heads ahead of the output
projection: `attention`, with biases on all projections, capped scores, a rotation whose slow frequencies are
stretched and whose cosines and sines have a magnitude, keys visible inside the query's chunk of positions, and a
gate per head and value dimension; `attention_2`, without biases, with a sliding window beside kept first keys, a
sink per head in the softmax's denominator, and one gate per head. The feed-forward is dense (a SiLU gate). A
layer may run another layer's tensors on a cache entry of its own. The head is a matrix of its own behind the
model's last norm.

Checkpoint names: `embed`, `head`, `final.norm`, and per layer i with tensors of its own `l<i>.norm1`, `l<i>.mix.*`,
`l<i>.mlp.*`; a bias is its tensor's name + `.b`.
"""
from __future__ import annotations

from ..config.munupel import MunupelConfig
from ..parts.base import LayerSpec, ModelPlan, PartSpec, ScheduleEntry
from ..registry import register_architecture

MAX_POSITIONS = 1 << 20  # the design names no limit


def _rotation(m):
    if m.rot is None:
        return None
    params = dict(head_dim=m.dim, rotary_dim=m.rot.dims, theta=m.rot.base)
    if m.rot.scaling is not None:
        factor, original, fast, slow = m.rot.scaling
        params.update(scaling="yarn", factor=factor, original_max_position_embeddings=original, fast_turns=fast,
                      slow_turns=slow)
    return PartSpec("rope", params)


def _shared(config: MunupelConfig, m) -> dict:
    return dict(hidden_size=config.width, num_heads=m.heads, num_kv_heads=m.kv_heads, head_dim=m.dim, value_dim=m.vdim,
                position=_rotation(m), scale=m.scale)


def _weights(p: str) -> dict:
    return {f"{own}_proj.weight": p + own for own in ("q", "k", "v", "g", "o")}


def _chunked(config: MunupelConfig, m, p: str) -> PartSpec:
    names = {**_weights(p), **{f"{own}_proj.bias": f"{p}{own}.b" for own in ("q", "k", "v", "o")}}
    return PartSpec("attention", dict(_shared(config, m), bias=True, output_bias=True, score_cap=m.softcap, chunk=m.span,
                                      gate="element"), names=names)


def _windowed(config: MunupelConfig, m, p: str) -> PartSpec:
    names = {**_weights(p), "sinks": p + "sink"}
    return PartSpec("attention", dict(_shared(config, m), sinks=True, window=m.span, keep_first=m.keep_first, gate="head"),
                    names=names)


MIXERS = {"attention": _chunked, "attention_2": _windowed}


def munupel_plan(config: MunupelConfig) -> ModelPlan:
    def norm(name: str) -> PartSpec:
        return PartSpec("layer_norm", dict(size=config.width, eps=config.eps), names={"weight": name, "bias": name + ".b"})

    layers, number = [], {}  # number: layer of the configuration -> layer of the plan, for those with tensors
    for i, layer in enumerate(config.layers):
        if config.owner(i) != i:
            continue
        p = f"l{i}."
        parts = dict(mixer=MIXERS[layer.kind](config, layer.mixer, p + "mix."), norm=norm(p + "norm1"))
        if layer.ff is not None:
            parts["feed_forward"] = PartSpec(
                "gated_mlp", dict(hidden_size=config.width, intermediate_size=layer.ff, activation="silu"),
                names={f"{own}_proj.weight": f"{p}mlp.{own}" for own in ("gate", "up", "down")})
        number[i] = len(layers)
        layers.append(LayerSpec("parallel" if layer.ff is not None else "parallel_mixer", parts=parts))
    schedule = tuple(ScheduleEntry(layer=number[config.owner(i)], cache=i) for i in range(len(config.layers)))
    return ModelPlan(
        hidden_size=config.width, vocab_size=config.vocab, max_positions=MAX_POSITIONS, embedding_name="embed",
        layers=tuple(layers), schedule=schedule, final_norm=norm("final.norm"), head_name="head")


register_architecture("Munupel", MunupelConfig, munupel_plan, model_types=("munupel",))
