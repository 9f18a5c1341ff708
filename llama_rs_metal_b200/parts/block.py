"""Arrangements of a layer's parts."""
from __future__ import annotations

from typing import Dict, Optional

import torch

from ..errors import InvalidError
from ..kernels import ops
from ..registry import register_block
from ..weights.loader import TensorSpec
from .base import Block, CompositeRequest, StateRequest
from .linear import LinearWeight, SplitLinear
from .mlp import GatedMLP
from .norm import StreamCast

STREAM_ITSELF = StreamCast()  # what a block whose sublayers read the stream itself has for an entry norm


class _PreNormBlock(Block):
    """Pre-norm sublayers. With `input_taps` n > 0 a mixer reads h + conv(h) instead of its norm's output
    h: a causal convolution over time per channel (tensor `input_conv`, [hidden_size, n], the last
    column the current token's, no bias); the last n - 1 rows h of every sequence are state of the
    layer, kept beside the mixer's own."""

    graph_safe = True

    def __init__(self, hidden_size: int = 0, input_taps: int = 0, **parts):
        super().__init__(**parts)
        self.hidden_size, self.input_taps = int(hidden_size), int(input_taps)
        if self.input_taps < 0 or (self.input_taps and self.hidden_size <= 0):
            raise InvalidError("an input convolution has positive taps and the layer's width")
        self.taps: Optional[torch.Tensor] = None

    @property
    def folds_pending_on_entry(self) -> bool:
        return self.mixer_norm.folds_pending

    def tensors(self) -> Dict[str, TensorSpec]:
        return {"input_conv": TensorSpec((self.hidden_size, self.input_taps))} if self.input_taps else {}

    def bind(self, weights, runtime) -> None:
        if self.input_taps:
            # [taps, width]: the kernels read one tap of many channels at a time
            self.taps = weights["input_conv"].to(torch.float32).t().contiguous()

    def cache_request(self):
        request = self.mixer.cache_request()
        if self.input_taps <= 1:
            return request
        return CompositeRequest((request, StateRequest((self.input_taps - 1, self.hidden_size), torch.float32)))

    def _mixer_input(self, hidden, ctx, cache):
        """(what the mixer reads, the mixer's part of the layer's cache)."""
        if not self.input_taps:
            return self.mixer_norm.forward(hidden, ctx), cache
        tails = None
        if self.input_taps > 1:
            if cache is None or not ctx.entry.writes_cache:
                raise InvalidError("a layer with an input convolution keeps state of its own")
            cache, last = cache
            tails = last.state
        return self.mixer_norm.forward_conv(hidden, ctx, self.taps, tails), cache


@register_block("pre_norm")
class PreNormBlock(_PreNormBlock):
    """hidden += mixer(norm(hidden)); hidden += feed_forward(norm(hidden))
    (crates/model-runtime/src/execute.rs:24,196-199,236)."""

    def forward(self, hidden, ctx, cache):
        after = ctx.next_folds_pending  # what comes after this block (the model says)
        x, cache = self._mixer_input(hidden, ctx, cache)
        # the mixer's output goes straight into the second norm: if that norm adds pending
        # partial sums itself, the mixer's last product may leave its K slices unadded
        ctx.may_defer = self.feed_forward_norm.folds_pending
        hidden = self.mixer.forward(x, ctx, cache, residual=hidden)
        ctx.may_defer = False
        x = self.feed_forward_norm.forward(hidden, ctx)
        ctx.may_defer = after
        hidden = self.feed_forward.forward(x, ctx, residual=hidden)
        ctx.may_defer = False
        return hidden


@register_block("pre_norm_mixer")
class PreNormMixerBlock(_PreNormBlock):
    """hidden += mixer(norm(hidden)): a layer without a feed-forward."""

    roles = {"mixer": "mixer", "mixer_norm": "norm"}

    def forward(self, hidden, ctx, cache):
        after = ctx.next_folds_pending
        x, cache = self._mixer_input(hidden, ctx, cache)
        ctx.may_defer = after
        hidden = self.mixer.forward(x, ctx, cache, residual=hidden)
        ctx.may_defer = False
        return hidden


class _ParallelBlock(Block):
    """One norm whose output every sublayer reads: hidden += mixer(x) + feed_forward(x), x = norm(hidden).

    Where the mixer can make its mixed heads from one product of its input (Mixer.projection, mix_projected), the
    sublayers are joined under bfloat16: one product makes the mixer's projection and the gated values of the
    feed-forward, the latter into the row that the mixed heads are then written beside, and one product with
    [W_down | W_out] makes both outputs and their sum. A bias of the mixer's output then rides in the norm's pass
    over the stream (Norm.forward_add)."""

    graph_safe = True

    @property
    def folds_pending_on_entry(self) -> bool:
        return self.norm.folds_pending


@register_block("parallel")
class ParallelBlock(_ParallelBlock):
    """A mixer and a feed-forward side by side on the same input."""

    roles = {"mixer": "mixer", "feed_forward": "feed_forward", "norm": "norm"}

    def __init__(self, **parts):
        super().__init__(**parts)
        self.into: Optional[SplitLinear] = None  # [projection | gate and up]
        self.out: Optional[LinearWeight] = None  # [down | mixer's output]
        self.inner = 0                           # columns of gated values in the joined row

    def bind(self, weights, runtime) -> None:
        # (a block is bound behind its parts)
        mixer, ff = self.mixer, self.feed_forward
        if runtime.dtype != torch.bfloat16 or mixer.projection is None or mixer.mixed_width is None \
                or not isinstance(ff, GatedMLP) or not ff.gates_in_product:
            return
        four = (mixer.projection.weight, mixer.out.weight, ff.gate_up.weight, ff.down.weight)
        if any(w.dtype != torch.bfloat16 for w in four) or any(n % 8 for n in (four[0].shape[1], mixer.mixed_width)):
            return  # the products' kernels want rows of whole 16-byte pieces
        self.inner = ff.intermediate_size
        self.into = SplitLinear(four[0], four[2])
        self.out = LinearWeight(torch.cat([four[3], four[1]], dim=1))
        mixer.give_up_products()
        ff.gate_up = ff.down = None

    def _joined(self, hidden, ctx, cache, after: bool):
        if self.mixer.output_bias is not None:
            x = self.norm.forward_add(hidden, ctx, self.mixer.output_bias)
        else:
            x = self.norm.forward(hidden, ctx)
        row = ops._activation(x.shape[0], self.inner + self.mixer.mixed_width, x.dtype, x.device)
        projected = self.into(x, row)
        self.mixer.mix_projected(projected, ctx, cache, row, self.inner)
        ctx.may_defer = after
        hidden = self.out(row, epilogue=ops.ADD, out=hidden, ctx=ctx)
        ctx.may_defer = False
        return hidden

    def forward(self, hidden, ctx, cache):
        after = ctx.next_folds_pending
        if self.into is not None:
            return self._joined(hidden, ctx, cache, after)
        x = self.norm.forward(hidden, ctx)
        hidden = self.mixer.forward(x, ctx, cache, residual=hidden)
        ctx.may_defer = after
        hidden = self.feed_forward.forward(x, ctx, residual=hidden)
        ctx.may_defer = False
        return hidden


@register_block("parallel_mixer")
class ParallelMixerBlock(_ParallelBlock):
    """The same for a layer without a feed-forward."""

    roles = {"mixer": "mixer", "norm": "norm"}

    def forward(self, hidden, ctx, cache):
        after = ctx.next_folds_pending
        x = self.norm.forward(hidden, ctx)
        ctx.may_defer = after
        hidden = self.mixer.forward(x, ctx, cache, residual=hidden)
        ctx.may_defer = False
        return hidden


class _ScaledPreNormBlock(Block):
    """Pre-norm sublayers whose outputs enter the stream under a factor per channel:
    hidden += mult * scale * sublayer(norm(hidden)), with `scale` a stored vector per sublayer
    (`layer_scale`; tensors `mixer_scale`, `feed_forward_scale`) and `mult` one number for the model.
    A sublayer's output stays float32 up to the addition. With `token_shift` the mixer reads
    h + (h' - h) * shift instead of its norm's output h, h' being the previous token's h (zeros for
    a sequence's first token; tensor `shift`); the last h of every sequence is state of the layer,
    kept beside the mixer's own. The pass that adds a sublayer's output also applies the norm that
    comes next (the feed-forward's, or the next block's first norm when that block takes it, handed
    over through StepContext.normed)."""

    graph_safe = True

    def __init__(self, hidden_size: int, residual_mult: float = 1.0, layer_scale: bool = False,
                 token_shift: bool = False, **parts):
        super().__init__(**parts)
        self.hidden_size, self.residual_mult = int(hidden_size), float(residual_mult)
        self.layer_scale, self.token_shift = bool(layer_scale), bool(token_shift)
        self.factors: Dict[str, torch.Tensor] = {}
        self.shift: Optional[torch.Tensor] = None

    @property
    def folds_pending_on_entry(self) -> bool:
        return self.mixer_norm.folds_pending

    def tensors(self) -> Dict[str, TensorSpec]:
        out = {}
        if self.layer_scale:
            out.update({role + "_scale": TensorSpec((self.hidden_size,)) for role in ("mixer", "feed_forward")
                        if role in self.parts})
        if self.token_shift:
            out["shift"] = TensorSpec((self.hidden_size,))
        return out

    def bind(self, weights, runtime) -> None:
        for role in ("mixer", "feed_forward"):
            if role in self.parts:
                scale = weights[role + "_scale"].to(torch.float32) if self.layer_scale else \
                    torch.ones(self.hidden_size, dtype=torch.float32, device=runtime.device)
                self.factors[role] = (scale * self.residual_mult).contiguous()
        if self.token_shift:
            self.shift = weights["shift"].to(torch.float32).contiguous()

    def cache_request(self):
        request = self.mixer.cache_request()
        if not self.token_shift:
            return request
        return CompositeRequest((request, StateRequest((1, self.hidden_size), torch.float32)))

    @property
    def entry_norm(self):
        return self.mixer_norm

    def _add(self, hidden, y, role, then, ctx):
        """hidden += factor * y; returns then.forward(hidden) of the updated stream (None without `then`)."""
        from .norm import RMSNorm
        if isinstance(then, RMSNorm) and then.weight is not None and ctx.pending is None:
            return ops.scaled_add_norm_(hidden, y, self.factors[role], then.weight, then.eps, ctx.runtime.dtype)
        ops.scaled_add_(hidden, y, self.factors[role])
        return then.forward(hidden, ctx) if then is not None else None

    def _mixer_half(self, hidden, ctx, cache, then):
        x = ctx.take_normed(self.mixer_norm)
        if x is None:
            x = self.mixer_norm.forward(hidden, ctx)
        if self.token_shift:
            if cache is None or not ctx.entry.writes_cache:
                raise InvalidError("a layer with token shift keeps state of its own")
            cache, last = cache
            x = ops.token_shift(x, self.shift, last.state, ctx.cu_seqlens, ctx.seq_of_token, ctx.slots)
        y = self.mixer.forward(x, ctx, cache, residual=None)
        return self._add(hidden, y, "mixer", then, ctx)


@register_block("scaled_pre_norm")
class ScaledPreNormBlock(_ScaledPreNormBlock):
    """A mixer and a feed-forward, each behind a norm, each added under its factor."""

    def forward(self, hidden, ctx, cache):
        following = ctx.next_entry_norm
        x = self._mixer_half(hidden, ctx, cache, self.feed_forward_norm)
        y = self.feed_forward.forward(x, ctx, residual=None)
        normed = self._add(hidden, y, "feed_forward", following, ctx)
        ctx.normed = (following, normed) if following is not None else None
        return hidden


@register_block("scaled_pre_norm_mixer")
class ScaledPreNormMixerBlock(_ScaledPreNormBlock):
    """The same for a layer without a feed-forward."""

    roles = {"mixer": "mixer", "mixer_norm": "norm"}

    def forward(self, hidden, ctx, cache):
        following = ctx.next_entry_norm
        normed = self._mixer_half(hidden, ctx, cache, following)
        ctx.normed = (following, normed) if following is not None else None
        return hidden


class _SandwichBlock(Block):
    """Norms on both sides of every sublayer, and a factor on what a sublayer adds:
    hidden += mult * post_norm(sublayer(pre_norm(hidden))). The sublayer's output stays float32
    up to its norm. The post-norm's pass also applies the norm that comes next (the
    feed-forward's pre-norm, or the next block's first norm when that block takes it)."""

    graph_safe = True

    def __init__(self, residual_mult: float = 1.0, **parts):
        super().__init__(**parts)
        self.residual_mult = float(residual_mult)

    @property
    def entry_norm(self):
        return self.mixer_norm

    def _mixer_half(self, hidden, ctx, cache, then):
        x = ctx.take_normed(self.mixer_norm)
        if x is None:
            x = self.mixer_norm.forward(hidden, ctx)
        y = self.mixer.forward(x, ctx, cache, residual=None)
        return self.mixer_post_norm.add_into(hidden, y, ctx, self.residual_mult, then)


@register_block("sandwich_norm")
class SandwichNormBlock(_SandwichBlock):
    """A mixer and a feed-forward, each between two norms."""

    roles = {"mixer": "mixer", "feed_forward": "feed_forward", "mixer_norm": "norm", "mixer_post_norm": "norm",
             "feed_forward_norm": "norm", "feed_forward_post_norm": "norm"}

    def forward(self, hidden, ctx, cache):
        following = ctx.next_entry_norm
        x = self._mixer_half(hidden, ctx, cache, self.feed_forward_norm)
        y = self.feed_forward.forward(x, ctx, residual=None)
        normed = self.feed_forward_post_norm.add_into(hidden, y, ctx, self.residual_mult, following)
        ctx.normed = (following, normed) if following is not None else None
        return hidden


@register_block("sandwich_norm_mixer")
class SandwichNormMixerBlock(_SandwichBlock):
    """A mixer between two norms: a layer without a feed-forward."""

    roles = {"mixer": "mixer", "mixer_norm": "norm", "mixer_post_norm": "norm"}

    def forward(self, hidden, ctx, cache):
        following = ctx.next_entry_norm
        normed = self._mixer_half(hidden, ctx, cache, following)
        ctx.normed = (following, normed) if following is not None else None
        return hidden


class _PostNormBlock(Block):
    """A norm on each sublayer's output only, and a factor on what it adds:
    hidden += mult * post_norm(sublayer(hidden)). The sublayers read the stream itself (its rounding
    under bfloat16 activations, which the pass of the norm before writes beside the float32 row);
    a sublayer's output stays float32 up to its norm. While a sublayer runs, ctx.stream is the
    float32 stream its input is the rounding of."""

    graph_safe = True

    def __init__(self, residual_mult: float = 1.0, **parts):
        super().__init__(**parts)
        self.residual_mult = float(residual_mult)

    @property
    def entry_norm(self):
        return STREAM_ITSELF

    def _mixer_half(self, hidden, ctx, cache, then):
        x = ctx.take_normed(STREAM_ITSELF)
        if x is None:
            x = STREAM_ITSELF.forward(hidden, ctx)
        ctx.stream = hidden
        y = self.mixer.forward(x, ctx, cache, residual=None)
        return self.mixer_post_norm.add_into(hidden, y, ctx, self.residual_mult, then)


@register_block("post_norm")
class PostNormBlock(_PostNormBlock):
    """A mixer and a feed-forward, each with a norm behind it."""

    roles = {"mixer": "mixer", "feed_forward": "feed_forward", "mixer_post_norm": "norm",
             "feed_forward_post_norm": "norm"}

    def forward(self, hidden, ctx, cache):
        following = ctx.next_entry_norm
        x = self._mixer_half(hidden, ctx, cache, STREAM_ITSELF)
        y = self.feed_forward.forward(x, ctx, residual=None)
        normed = self.feed_forward_post_norm.add_into(hidden, y, ctx, self.residual_mult, following)
        ctx.stream = None
        ctx.normed = (following, normed) if following is not None else None
        return hidden


@register_block("post_norm_mixer")
class PostNormMixerBlock(_PostNormBlock):
    """A mixer with a norm behind it: a layer without a feed-forward."""

    roles = {"mixer": "mixer", "mixer_post_norm": "norm"}

    def forward(self, hidden, ctx, cache):
        following = ctx.next_entry_norm
        normed = self._mixer_half(hidden, ctx, cache, following)
        ctx.stream = None
        ctx.normed = (following, normed) if following is not None else None
        return hidden
