"""The Tolurax decoder as a plan of parts.

Layers are pre-norm with layer norms that have a weight and no bias: x <- x + mixer(canon(norm1(x))), then
x <- x + ff(norm2(x)) (or nothing), where canon(h) = h + conv(h) with a short causal convolution over time
per channel. Two kinds of mixer: `delta`, a gated delta rule with one decay per head behind short
convolutions, gated by SiLU; `parallel`, a weighted sum of windowed attention without a softmax (sigmoid
weights with an offset per head, a norm per query and key head, a rotation whose slow frequencies are
stretched, a sigmoid gate per head and value dimension) and a time mix (a matrix state with a decay per key
channel computed from the input, a bonus for the current token, each projection reading its own mix with
the previous token). The feed-forward is dense (a SiLU gate). A run of layers may loop: it runs several
times in a row with the same weights, every pass with cache entries of its own, and before every pass the
stream x becomes W [x; x0], x0 being the embedding's output. The head is a matrix of its own behind the
model's last norm; logits are soft-capped.

Checkpoint names: `embed`, `head`, `final.norm`, `loop.in`, and per layer i `l<i>.norm1`, `l<i>.norm2`,
`l<i>.canon1`, `l<i>.mix.*`, `l<i>.mlp.*`; a convolution's taps are its matrix's name + `.conv`, a head
norm's weight + `.norm`; the parallel mixer's two sides are under `.left` and `.right`.
"""
from __future__ import annotations

from ..config.tolurax import ToluraxConfig
from ..parts.base import LayerSpec, ModelPlan, PartSpec, ScheduleEntry, looped_runs
from ..registry import register_architecture

MAX_POSITIONS = 1 << 20   # the design names no limit
UNIT_EPS = 1e-6           # under the root of the delta rule's unit vectors


def _delta(config: ToluraxConfig, m, p: str) -> PartSpec:
    names = {f"{own}_proj.weight": p + own for own in ("q", "k", "v", "b", "a", "g", "o")}
    names.update({f"{own}_conv.weight": p + own + ".conv" for own in ("q", "k", "v")})
    names.update({"A_log": p + "A_log", "dt_bias": p + "dt_bias", "norm.weight": p + "norm"})
    return PartSpec("head_decay_delta_rule", dict(
        hidden_size=config.width, num_heads=m.heads, num_kv_heads=m.kv_heads, head_dim=m.dim, value_dim=m.vdim,
        conv_taps=m.conv, eps=config.eps, unit_eps=UNIT_EPS), names=names)


def _attention(config: ToluraxConfig, m) -> PartSpec:
    position = None
    if m.rot is not None:
        params = dict(head_dim=m.dim, rotary_dim=m.rot.dims, theta=m.rot.base)
        if m.rot.scaling is not None:
            factor, low, high, original = m.rot.scaling
            params.update(scaling="llama3", factor=factor, low_freq_factor=low, high_freq_factor=high,
                          original_max_position_embeddings=original)
        position = PartSpec("rope", params)
    return PartSpec("attention", dict(
        hidden_size=config.width, num_heads=m.heads, num_kv_heads=m.kv_heads, head_dim=m.dim, value_dim=m.vdim,
        position=position, scale=m.scale, window=m.window, weights="sigmoid", gate=True, head_weight_eps=config.eps))


def _attention_names(p: str) -> dict:
    names = {f"{own}_proj.weight": p + own for own in ("q", "k", "v", "g", "o")}
    names.update({"q_head_norm.weight": p + "q.norm", "k_head_norm.weight": p + "k.norm", "score_offset": p + "pb"})
    return names


def _time_mix(config: ToluraxConfig, m) -> PartSpec:
    return PartSpec("time_mix", dict(hidden_size=config.width, num_heads=m.heads, head_dim=m.dim, eps=config.eps,
                                     decay_rank=m.decay_rank))


def _time_mix_names(p: str) -> dict:
    names = {f"{own}_proj.weight": p + own for own in ("r", "k", "v", "g", "o")}
    names.update({f"{own}_mix": p + "mu." + own for own in ("r", "k", "v", "g", "w")})
    names.update({"w_down.weight": p + "w1", "w_up.weight": p + "w2", "w_bias": p + "w0", "bonus": p + "u",
                  "norm.weight": p + "norm"})
    return names


def _parallel(config: ToluraxConfig, m, p: str) -> PartSpec:
    names = {"left." + own: full for own, full in _attention_names(p + "left.").items()}
    names.update({"right." + own: full for own, full in _time_mix_names(p + "right.").items()})
    return PartSpec("parallel", dict(left=_attention(config, m.left), right=_time_mix(config, m.right),
                                     left_scale=m.left_scale, right_scale=m.right_scale), names=names)


MIXERS = {"delta": _delta, "parallel": _parallel}


def tolurax_plan(config: ToluraxConfig) -> ModelPlan:
    def norm(name: str) -> PartSpec:
        return PartSpec("layer_norm", dict(size=config.width, eps=config.eps, bias=False), names={"weight": name})

    layers = []
    for i, layer in enumerate(config.layers):
        p = f"l{i}."
        parts = dict(mixer=MIXERS[layer.kind](config, layer.mixer, p + "mix."), mixer_norm=norm(p + "norm1"))
        if layer.ff is not None:
            parts.update(feed_forward=PartSpec(
                "gated_mlp", dict(hidden_size=config.width, intermediate_size=layer.ff, activation="silu"),
                names={f"{own}_proj.weight": f"{p}mlp.{own}" for own in ("gate", "up", "down")}),
                feed_forward_norm=norm(p + "norm2"))
        layers.append(LayerSpec("pre_norm" if layer.ff is not None else "pre_norm_mixer", parts=parts,
                                options=dict(hidden_size=config.width, input_taps=config.canon_taps),
                                names={"input_conv": p + "canon1"}))
    schedule = tuple(ScheduleEntry(layer=i, cache=n, join_embedding=starts is not None)
                     for n, (i, starts) in enumerate(looped_runs(len(layers), config.loop_start, config.loop_stop,
                                                                 config.loop_times)))
    return ModelPlan(
        hidden_size=config.width, vocab_size=config.vocab, max_positions=MAX_POSITIONS,
        embedding_name="embed", layers=tuple(layers), schedule=schedule,
        final_norm=norm("final.norm"), head_name="head", logit_softcap=config.logit_softcap,
        stream_join="loop.in" if config.loops else None)


register_architecture("Tolurax", ToluraxConfig, tolurax_plan, model_types=("tolurax",))
