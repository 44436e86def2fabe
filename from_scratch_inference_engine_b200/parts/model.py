"""A decoder model assembled from a `ModelSpec`: embedding, blocks in run order, final
norm and output head."""

from __future__ import annotations

from typing import Dict, List, Optional

import torch

from ..cache.manager import CacheNeed
from ..config.spec import ModelSpec
from ..kernels import ops
from ..weights.loader import check_tensors, to_runtime_dtype
from ..weights.tensor_spec import TensorSpec
from .base import LayerCache, StateNeed, build_part
from .norm import StreamNorm, StreamUpdate


class DecoderModel:
    """Embedding (times `embedding_scale`, then through `embedding_norm` where the model has one)
    -> blocks in the order of `spec.schedule`, an inlet
    before the calls that name one -> final norm -> head, times `logit_scale`, capped by
    `logit_softcap * tanh(. / logit_softcap)` where a cap is given.  With `spec.streams` the residual
    is that many streams, every one the embedding output at the start; the final norm reads their sum.

    The run order is data: entry i of the schedule runs block `layer` on cache entry
    `cache` (its own by default).  A block named twice runs twice with the same weights;
    a call with writes_cache=False attends over keys another call stored.
    Reference wiring: src/model/model.cpp:159-281.
    """

    def __init__(self, spec: ModelSpec):
        self.spec = spec
        self.schedule = spec.resolved_schedule()
        self.blocks = [build_part("arrangement",
                                  _arrangement_spec(layer, spec.streams), layer.prefix) for layer in spec.layers]
        self.final_norm = build_part("norm", spec.final_norm, spec.final_norm_prefix)
        self.embedding_norm = None if spec.embedding_norm is None else \
            build_part("norm", spec.embedding_norm, spec.embedding_norm_prefix)
        self.inlets = [build_part("inlet", part, prefix) for part, prefix in spec.inlets]
        self.inlet_before = [call.inlet for call in spec.schedule]
        if spec.streams and (self.inlets or not isinstance(self.final_norm, StreamNorm)):
            raise ValueError("a model of several residual streams takes no inlets, and a final norm that reads "
                             "several streams")
        self.embedding: Optional[torch.Tensor] = None
        self.head: Optional[torch.Tensor] = None
        self.runtime = None

    # ------------------------------------------------------------------ tensors
    def tensor_specs(self) -> List[TensorSpec]:
        spec = self.spec
        shape = (spec.vocab_size, spec.hidden_size)
        specs = [TensorSpec(spec.embedding_name, shape)]
        if spec.head_name is not None:
            specs.append(TensorSpec(spec.head_name, shape))
        else:
            # a tied head may be stored a second time; it must then equal the embedding
            specs.append(TensorSpec("lm_head.weight", shape, optional=True,
                                    same_as=spec.embedding_name))
        specs += self.final_norm.tensor_specs()
        if self.embedding_norm is not None:
            specs += self.embedding_norm.tensor_specs()
        for inlet in self.inlets:
            specs += inlet.tensor_specs()
        for block in self.blocks:
            specs += block.tensor_specs()
        return specs

    def bind(self, tensors: Dict[str, torch.Tensor], runtime) -> None:
        """Check `tensors` (host or device, any stored dtype) against the declarations, move
        them to the runtime's device and dtypes, and hand each part its own."""
        specs = self.tensor_specs()
        check_tensors(specs, tensors)
        by_name = {s.name: s for s in specs}
        placed = {}
        for name, tensor in tensors.items():
            spec = by_name[name]
            if spec.optional and spec.same_as:
                continue
            placed[name] = to_runtime_dtype(tensor, spec, runtime.dtype).to(runtime.device)
        self.runtime = runtime
        self.embedding = placed[self.spec.embedding_name].contiguous()
        self.head = (placed[self.spec.head_name].contiguous()
                     if self.spec.head_name is not None else self.embedding)
        runtime.prepare_weight(self.head)
        self.final_norm.bind(placed, runtime)
        if self.embedding_norm is not None:
            self.embedding_norm.bind(placed, runtime)
        for inlet in self.inlets:
            inlet.bind(placed, runtime)
        for block in self.blocks:
            block.bind(placed, runtime)

    # -------------------------------------------------------------------- needs
    @property
    def capturable(self) -> bool:
        """Whether a step launches the same kernels whatever the data (every part says so)."""
        return self.final_norm.capturable and all(block.capturable for block in self.blocks) \
            and all(inlet.capturable for inlet in self.inlets) \
            and (self.embedding_norm is None or self.embedding_norm.capturable)

    def cache_needs(self) -> List[Optional[CacheNeed]]:
        """Need of each cache entry (index = position in the run order); None where the
        entry is not written by its own call or the mixer keeps no keys."""
        needs: List[Optional[CacheNeed]] = [None] * len(self.schedule)
        for index, (layer, entry, writes) in enumerate(self.schedule):
            need = self.blocks[layer].mixer.cache_need()
            if writes:
                needs[entry] = need
            elif need != needs[entry]:
                # a reader with another window: the entry keeps what either can still see
                if need is None or needs[entry] is None:
                    raise ValueError(f"schedule entry {index} reads cache entry {entry} whose "
                                     f"layout {needs[entry]} differs from its own {need}")
                try:
                    needs[entry] = needs[entry].covering(need)
                except ValueError as error:
                    raise ValueError(f"schedule entry {index} reads cache entry {entry}: "
                                     f"{error}") from None
        return needs

    def state_needs(self) -> List[Optional[StateNeed]]:
        """State each call of the run order keeps per request (None for most mixers)."""
        return [self.blocks[layer].mixer.state_need() for layer, _, _ in self.schedule]

    # ------------------------------------------------------------------ forward
    def forward(self, ctx, caches: List[LayerCache], want_rows: Optional[torch.Tensor]):
        """Run the step's tokens; returns float32 logits [len(want_rows), vocab] (None if
        nothing is wanted).  `caches[i]` belongs to call i of the run order."""
        rt = self.runtime
        hidden = self.spec.hidden_size
        x = rt.buffer("model.residual", ctx.num_tokens, hidden, torch.float32)
        scale = self.spec.embedding_scale
        if self.embedding_norm is None:
            ops.embed_gather(ctx.token_ids, self.embedding, x, ctx.error, scale)
        else:           # the normed rows, still 32-bit, are the stream
            rows = rt.buffer("model.embedding_rows", ctx.num_tokens, hidden, torch.float32)
            ops.embed_gather(ctx.token_ids, self.embedding, rows, ctx.error, scale)
            x = self.embedding_norm.forward(rows, None, tag="model.residual", out_dtype=torch.float32)
        delta = None
        if self.spec.streams:             # every stream starts as x; they exist once a layer has changed them
            delta = StreamUpdate(start=x)
            x = rt.buffer("model.streams", ctx.num_tokens, self.spec.streams * hidden, torch.float32)
            x = x.view(ctx.num_tokens, self.spec.streams, hidden)
        x0 = None
        if self.inlets:                   # the embedding output, for the inlets that read it
            x0 = rt.buffer("model.embedding_output", ctx.num_tokens, hidden, torch.float32)
            ops.embed_gather(ctx.token_ids, self.embedding, x0, ctx.error, scale)
        ctx.residual_copy = None          # x in the compute dtype, where an arrangement keeps one
        for index, (layer, _, _) in enumerate(self.schedule):
            if self.inlet_before[index] is not None:
                x, delta = self.inlets[self.inlet_before[index]].forward(ctx, x, delta, x0), None
                ctx.residual_copy = None
            delta = self.blocks[layer].forward(ctx, x, delta, caches[index])
        if want_rows is None or want_rows.numel() == 0:
            return None
        if self.spec.streams:
            y = self.final_norm.over_streams(x, delta, None, rows=want_rows, write_x=False)
        else:
            y = self.final_norm.forward(x, delta, rows=want_rows, write_x=False)
        # the logits live where the last step's lived: whoever gets them reads them (or queues
        # what reads them on this stream) before the next step runs
        logits = rt.linear_f32_out(y, self.head, "model.logits")
        if self.spec.logit_scale != 1.0 or self.spec.logit_softcap > 0.0:
            ops.logit_cap(logits, self.spec.logit_scale, self.spec.logit_softcap)
        return logits


def _arrangement_spec(layer, streams: int):
    from ..config.spec import PartSpec
    return PartSpec(layer.arrangement, {"layer": layer, "streams": streams} if streams else {"layer": layer})


def tensor_specs(spec: ModelSpec) -> List[TensorSpec]:
    """Every tensor a model of this spec reads from a checkpoint (no device needed)."""
    return DecoderModel(spec).tensor_specs()
