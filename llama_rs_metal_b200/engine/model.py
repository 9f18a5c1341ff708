"""A decoder put together from a plan: embedding, scheduled blocks, final norm, head."""
from __future__ import annotations

from typing import Dict, List, Optional

import torch

from ..errors import InvalidError
from ..kernels import ops
from ..parts.base import Block, ModelPlan, PartSpec
from ..parts.linear import LinearWeight
from ..registry import BLOCKS, FEED_FORWARDS, MIXERS, NORMS, build_part

FAMILIES = {"mixer": (MIXERS, "mixer"), "feed_forward": (FEED_FORWARDS, "feed-forward"), "norm": (NORMS, "norm")}
from ..runtime import Runtime
from ..weights.loader import TensorSpec


def _full_names(spec: PartSpec, part) -> Dict[str, str]:
    """own tensor name -> checkpoint name, for one part."""
    return {own: spec.names.get(own, spec.prefix + own) for own in part.tensors()}


class DecoderModel:
    """Owns the parts of one model and runs them over a step's packed tokens.

    It knows nothing of Llama: which parts there are, their sizes, their tensor
    names and the order of layers all come from the plan.
    """

    def __init__(self, plan: ModelPlan, runtime: Runtime):
        self.plan, self.runtime = plan, runtime
        self.blocks: List[Block] = []
        self._names: List[Dict[str, Dict[str, str]]] = []
        self._block_names: List[Dict[str, str]] = []
        for layer in plan.layers:
            if layer.block not in BLOCKS:
                raise InvalidError(f"block kind {layer.block!r} is not registered")
            block_class = BLOCKS[layer.block]
            # the block says which roles a layer of its kind has, and of which family each is
            parts = {}
            for role, family in block_class.roles.items():
                if role not in layer.parts:
                    raise InvalidError(f"a {layer.block!r} layer needs a part for the role {role!r}")
                if family not in FAMILIES:
                    raise InvalidError(f"block {layer.block!r}: role {role!r} has unknown family {family!r}")
                table, label = FAMILIES[family]
                parts[role] = build_part(table, layer.parts[role], label)
            unknown = sorted(set(layer.parts) - set(parts))
            if unknown:
                raise InvalidError(f"a {layer.block!r} layer has no role {', '.join(unknown)}")
            self.blocks.append(block_class(**parts, **layer.options))
            self._names.append({role: _full_names(layer.parts[role], part) for role, part in parts.items()})
            # tensors the arrangement itself owns (a factor per channel on what a sublayer adds, ...)
            self._block_names.append({own: layer.names.get(own, own) for own in self.blocks[-1].tensors()})
        self.final_norm = build_part(NORMS, plan.final_norm, "norm")
        self._final_names = _full_names(plan.final_norm, self.final_norm)
        self.embedding: Optional[torch.Tensor] = None
        self.stream_offsets: Optional[torch.Tensor] = None  # float32 [rows, hidden]
        self.head: Optional[LinearWeight] = None
        # the two halves of the plan's stream_join matrix: W [x; x0] = W_x x + W_0 x0, of which the second
        # term is the same for every pass of a step
        self.join_stream: Optional[LinearWeight] = None
        self.join_embedding: Optional[LinearWeight] = None
        self.unexpected_tensors: tuple = ()  # stored names the loader skipped (set by the loader's caller)
        self._check_schedule()

    # -- schedule and cache --------------------------------------------------------
    def _check_schedule(self) -> None:
        writers = {}
        for position, entry in enumerate(self.plan.schedule):
            if not 0 <= entry.layer < len(self.blocks):
                raise InvalidError(f"schedule names layer {entry.layer}, the model has {len(self.blocks)}")
            if entry.add_offset is not None:
                rows = self.plan.stream_offsets[1] if self.plan.stream_offsets is not None else 0
                if not 0 <= entry.add_offset < rows:
                    raise InvalidError(f"schedule entry {position} adds offset {entry.add_offset} of {rows}")
            if entry.join_embedding and self.plan.stream_join is None:
                raise InvalidError(f"schedule entry {position} joins the embedding, the plan has no matrix for it")
            if entry.writes_cache:
                if entry.cache in writers:
                    raise InvalidError(f"cache entry {entry.cache} is written by two schedule entries")
                writers[entry.cache] = position
            elif entry.cache not in writers:
                raise InvalidError(f"schedule entry {position} reads cache entry {entry.cache} before it is written")
        if sorted(writers) != list(range(len(writers))):
            raise InvalidError("cache entries must be numbered 0..n-1")

    def cache_requests(self) -> list:
        """What each cache entry's writing layer asks of the cache (index = cache entry)."""
        out = {}
        for entry in self.plan.schedule:
            if entry.writes_cache:
                out[entry.cache] = self.blocks[entry.layer].cache_request()
        return [out[i] for i in range(len(out))]

    @property
    def graph_safe(self) -> bool:
        """True when every part only enqueues device work, so a decode step can be a CUDA graph."""
        parts = [self.final_norm]
        for block in self.blocks:
            parts += [block, *block.parts.values()]
        return all(p.graph_safe for p in parts)

    # -- weights ---------------------------------------------------------------------
    def tensor_specs(self) -> Dict[str, TensorSpec]:
        plan = self.plan
        specs = {plan.embedding_name: TensorSpec((plan.vocab_size, plan.hidden_size))}
        if plan.head_name is not None:
            specs[plan.head_name] = TensorSpec((plan.vocab_size, plan.hidden_size))
        if plan.stream_offsets is not None:
            specs[plan.stream_offsets[0]] = TensorSpec((plan.stream_offsets[1], plan.hidden_size))
        if plan.stream_join is not None:
            specs[plan.stream_join] = TensorSpec((plan.hidden_size, 2 * plan.hidden_size))
        for block, names, own_names in zip(self.blocks, self._names, self._block_names):
            for role, mapping in names.items():
                part_specs = getattr(block, role).tensors()
                for own, full in mapping.items():
                    specs[full] = part_specs[own]
            block_specs = block.tensors()
            for own, full in own_names.items():
                specs[full] = block_specs[own]
        for own, full in self._final_names.items():
            specs[full] = self.final_norm.tensors()[own]
        return specs

    def bind(self, tensors: Dict[str, torch.Tensor]) -> None:
        """Hand every part its tensors (already on the device, in their kept precision)."""
        rt = self.runtime
        self.embedding = tensors[self.plan.embedding_name].contiguous()
        head = self.embedding if self.plan.head_name is None else tensors[self.plan.head_name]
        self.head = LinearWeight(head)
        if self.plan.stream_offsets is not None:  # added to the float32 stream: kept in float32
            self.stream_offsets = tensors[self.plan.stream_offsets[0]].to(torch.float32).contiguous()
        if self.plan.stream_join is not None:
            both, h = tensors[self.plan.stream_join], self.plan.hidden_size
            self.join_stream, self.join_embedding = LinearWeight(both[:, :h]), LinearWeight(both[:, h:])
        for block, names, own_names in zip(self.blocks, self._names, self._block_names):
            for role, mapping in names.items():
                getattr(block, role).bind({own: tensors[full] for own, full in mapping.items()}, rt)
            block.bind({own: tensors[full] for own, full in own_names.items()}, rt)
        self.final_norm.bind({own: tensors[full] for own, full in self._final_names.items()}, rt)

    # -- forward ---------------------------------------------------------------------
    def forward(self, ctx, cache) -> torch.Tensor:
        """float32 logits [len(ctx.wanted_rows), vocab] for one step."""
        x = self._hidden_of_wanted_rows(ctx, cache)
        if x is None:
            return torch.empty((0, self.plan.vocab_size), dtype=torch.float32, device=self.runtime.device)
        logits = self.head(x, out_dtype=torch.float32)
        if self.plan.logit_scale is not None:
            ops.scale_(logits, self.plan.logit_scale)
        if self.plan.logit_softcap is not None:
            ops.softcap_(logits, self.plan.logit_softcap)
        return logits

    def forward_pick(self, ctx, cache, temperature=None, seed: int = 0, keys=None) -> torch.Tensor:
        """int32 [len(ctx.wanted_rows)]: the token chosen at each wanted place, for a caller that
        wants no logits (generation): greedy when `temperature` is None, else a draw from
        softmax(logits / temperature) keyed per row by `keys` (int64). The head product chooses in
        its epilogue where a kernel can (crates/model-runtime/src/execute.rs:238-247 pairs the head
        with the GPU argmax the same way). -1 marks a row with a non-finite logit."""
        x = self._hidden_of_wanted_rows(ctx, cache)
        if x is None:
            return torch.empty((0,), dtype=torch.int32, device=self.runtime.device)
        scale, cap = self.plan.logit_scale, self.plan.logit_softcap
        if scale is not None and (scale <= 0 or cap is not None):
            logits = ops.scale_(self.head(x, out_dtype=torch.float32), scale)
            if cap is not None:
                ops.softcap_(logits, cap)
            return ops.argmax_rows(logits) if temperature is None else \
                ops.sample_gumbel_rows(logits, temperature, seed, keys)
        if temperature is not None and scale is not None:
            temperature = temperature / scale  # (s z) / T = z / (T / s)
        return self.head.pick(x, temperature, seed, keys, softcap=cap)

    def _hidden_of_wanted_rows(self, ctx, cache) -> Optional[torch.Tensor]:
        """Embedding, the scheduled blocks and the final norm on the wanted rows; None when no
        row is wanted (the cache is filled all the same)."""
        plan = self.plan
        # what dispatchers kept belongs to one run of the step: a context that runs again (a
        # captured step, once before and once under capture) must compute it again from its arrays
        ctx.scratch.clear()
        ctx.fresh_kv.clear()
        ctx.normed = None
        hidden = ops.embed_rows(self.embedding, ctx.token_ids, plan.embedding_scale)
        wanted = ctx.wanted_rows.numel() > 0
        schedule = plan.schedule
        embedded = hidden.clone() if any(entry.add_embedding for entry in schedule) else None
        joined = None  # W_0 x0 of the stream's join, made once
        if any(entry.join_embedding for entry in schedule):
            joined = self.join_embedding(ops.cast(hidden, self.runtime.dtype), out_dtype=torch.float32)
        for i, entry in enumerate(schedule):
            ctx.entry = entry
            view = cache.view(entry.cache) if cache is not None else None
            # may this block's last product leave its K slices for the next reader of the stream?
            if i + 1 < len(schedule):
                following = self.blocks[schedule[i + 1].layer]
                ctx.next_folds_pending = following.folds_pending_on_entry
                # a block may hand the next one its stream already passed through that block's
                # first norm (nothing may be added to the stream in between)
                ctx.next_entry_norm = following.entry_norm \
                    if schedule[i + 1].add_offset is None and not schedule[i + 1].add_embedding \
                    and not schedule[i + 1].join_embedding else None
                # a join takes pending sums along with the stream it reads
                ctx.next_folds_pending |= schedule[i + 1].join_embedding
            else:
                ctx.next_folds_pending = wanted and self.final_norm.folds_pending
                ctx.next_entry_norm = None
            if entry.join_embedding:
                # x <- W_x x + W_0 x0: the stream leaves in the activation type and is replaced by the second
                # term, into which the product of the first is added
                x = ops.stream_swap_(hidden, joined, self.runtime.dtype, ctx.take_pending())
                hidden = self.join_stream(x, epilogue=ops.ADD, out=hidden)
            if entry.add_embedding:
                hidden = ops.add_(ctx.settle(hidden), embedded)
            if entry.add_offset is not None:
                hidden = ops.add_row_(hidden, self.stream_offsets[entry.add_offset])
            hidden = self.blocks[entry.layer].forward(hidden, ctx, view)
            if ctx.pending is not None and not ctx.next_folds_pending:
                ctx.settle(hidden)  # a block left sums its successor cannot add itself
        ctx.entry = None
        ctx.next_folds_pending = False
        if not wanted:
            ctx.take_pending()
            return None
        # the head runs only on the rows whose logits are wanted
        # (crates/model-runtime/src/execute.rs:238-247 does it for the last row)
        return self.final_norm.forward(hidden, ctx, rows=ctx.wanted_rows)
