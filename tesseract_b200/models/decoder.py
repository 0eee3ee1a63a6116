"""A decoder-only model assembled from a :class:`ModelSpec`.

The builder looks every part kind up in the registries, asks the parts which checkpoint
tensors they expect, and wires them in the order the spec's ``run_order`` gives.  The
forward pass walks that list: embedding, then for each run entry the named layer with
the entry's cache binding, then the final norm and the head on the wanted rows only
(intermediate prompt portions that want no logits skip both, as in
src/cuda/dense_decoder.rs:784-787).
"""

from __future__ import annotations

from typing import Dict, List, Mapping, Optional, Sequence

import torch

from .. import kernels
from ..config.spec import LayerSpec, ModelSpec, PartSpec
from ..parts import (BLOCKS, EMBEDDINGS, FEED_FORWARDS, HEADS, INJECTIONS, MIXERS, NORMS, RESIDUAL_GATES, STREAM_MIXINGS, TOKEN_INPUTS, Block, CacheBinding, DeferredNorm,
                     ResidualStream, Runtime, StepContext)
from ..weights.loader import ExpectedTensor


def _part_specs(spec: ModelSpec):
    """Yield ``(registry, PartSpec)`` for every weight-bearing part of the model."""
    yield EMBEDDINGS, spec.embedding
    for layer in spec.layers:
        block_cls = BLOCKS.get(layer.block)
        norms = layer.norms
        for role in block_cls.norm_roles(with_feed_forward=layer.feed_forward is not None):
            if role not in norms:
                raise ValueError(f"block '{layer.block}' needs a norm for role '{role}'")
        for role in sorted(norms):
            yield NORMS, norms[role]
        yield MIXERS, layer.mixer
        if layer.feed_forward is not None:
            yield FEED_FORWARDS, layer.feed_forward
        if layer.token_input is not None:
            if not block_cls.accepts_token_input:
                raise ValueError(f"block '{layer.block}' takes no token input")
            yield TOKEN_INPUTS, layer.token_input
        if layer.residual_gates is not None:
            if not block_cls.accepts_residual_gates:
                raise ValueError(f"block '{layer.block}' takes no residual gates")
            yield RESIDUAL_GATES, layer.residual_gates
        if layer.stream_mixing is not None:
            if not block_cls.accepts_stream_mixing:
                raise ValueError(f"block '{layer.block}' takes no stream mixing")
            yield STREAM_MIXINGS, layer.stream_mixing
    for injection in spec.injections:
        yield INJECTIONS, injection
    yield NORMS, spec.final_norm
    yield HEADS, spec.head


def expected_tensors(spec: ModelSpec) -> Dict[str, ExpectedTensor]:
    """Every checkpoint tensor the model reads, by name."""
    out: Dict[str, ExpectedTensor] = {}
    for registry, part in _part_specs(spec):
        for name, want in registry.get(part.kind).expected_tensors(part).items():
            if name in out and out[name] != want:
                raise ValueError(f"tensor '{name}' is expected with two shapes: {out[name]} and {want}")
            out[name] = want
    return out


def tensor_roles(spec: ModelSpec):
    """Yield ``(part class, PartSpec, role, checkpoint name, ExpectedTensor)`` once per distinct tensor."""
    seen = set()
    for registry, part in _part_specs(spec):
        cls = registry.get(part.kind)
        expected = cls.expected_tensors(part)
        for role, name in part.weights.items():
            if name in seen or name not in expected:
                continue
            seen.add(name)
            yield cls, part, role, name, expected[name]


class DecoderModel:
    def __init__(self, spec: ModelSpec, tensors: Mapping[str, torch.Tensor], runtime: Runtime):
        spec.validate()
        self.spec = spec
        self.runtime = runtime

        def build(registry, part: PartSpec, **extra):
            cls = registry.get(part.kind)
            mine = {role: tensors[name] for role, name in part.weights.items()}
            return cls(part, mine, runtime, **extra)

        self.embedding = build(EMBEDDINGS, spec.embedding)
        self.layers: List[Block] = []
        for layer in spec.layers:
            block_cls = BLOCKS.get(layer.block)
            norms = {role: build(NORMS, part) for role, part in layer.norms.items()}
            mixer = build(MIXERS, layer.mixer)
            feed_forward = build(FEED_FORWARDS, layer.feed_forward) if layer.feed_forward is not None else None
            extras = {}
            if layer.token_input is not None:
                extras["token_input"] = build(TOKEN_INPUTS, layer.token_input)
            if layer.residual_gates is not None:
                extras["residual_gates"] = build(RESIDUAL_GATES, layer.residual_gates)
            if layer.stream_mixing is not None:
                extras["stream_mixing"] = build(STREAM_MIXINGS, layer.stream_mixing)
            self.layers.append(block_cls(norms, mixer, feed_forward, **extras))
        self.injections = [build(INJECTIONS, part) for part in spec.injections]
        self.final_norm = build(NORMS, spec.final_norm)
        # A head that names the embedding's checkpoint tensor (tied embeddings) gets the same host tensor, and the
        # runtime hands it the device copy that the embedding made: tying is a matter of tensor names alone.
        self.head = build(HEADS, spec.head)
        runtime.forget_uploads()

    # ------------------------------------------------------------------ cache description
    def cache_needs(self) -> List[Optional[object]]:
        """For each run entry: its mixer's cache need, or ``None`` if it keeps no cache of its own; behind them, if the
        embedding keeps something per request, its need (the embedding's binding is then the last one)."""
        needs: List[Optional[object]] = []
        for index, entry in enumerate(self.spec.run_order):
            need = self.layers[entry.layer].mixer.cache_need()
            if entry.cache_of is not None:
                other = self.layers[self.spec.run_order[entry.cache_of].layer].mixer.cache_need()
                if other != need:
                    raise ValueError(f"run entry {index} reads the cache of entry {entry.cache_of}, "
                                     f"whose geometry {other} differs from its own {need}")
                needs.append(None)
            else:
                needs.append(need)
        own = self.embedding.cache_need()
        return needs if own is None else needs + [own]

    def cache_sources(self) -> List[Optional[int]]:
        """For each of :meth:`cache_needs`: the earlier one whose cache it reads, or ``None``."""
        sources = [entry.cache_of for entry in self.spec.run_order]
        return sources if self.embedding.cache_need() is None else sources + [None]

    # ------------------------------------------------------------------ forward
    def _embed(self, ctx: StepContext, bindings: Sequence[Optional[CacheBinding]]) -> torch.Tensor:
        token_ids = ctx.token_ids[:ctx.num_rows]
        if self.embedding.takes_context:
            own = bindings[len(self.spec.run_order)] if self.embedding.cache_need() is not None else None
            return self.embedding.forward(token_ids, ctx=ctx, cache=own)
        if self.embedding.takes_positions:
            return self.embedding.forward(token_ids, positions=ctx.positions[:ctx.num_rows])
        return self.embedding.forward(token_ids)

    def forward(self, ctx: StepContext, bindings: Sequence[Optional[CacheBinding]],
                want_rows: Optional[torch.Tensor], want_every_row: bool = False) -> Optional[torch.Tensor]:
        """Run the step's rows; return float32 logits ``[len(want_rows), vocab]`` or ``None``.
        ``want_every_row``: the caller knows that ``want_rows`` is ``0 .. num_rows - 1`` (a decode step), so the
        rows need not be gathered before the head."""
        ctx.carried.clear()
        hidden = self._embed(ctx, bindings)
        stream = ResidualStream(hidden, None)
        order = self.spec.run_order
        # the embedding output that injections read: rows of their own, since blocks add into the stream in place
        origin = None
        if any(injection.reads_origin for injection in self.injections):
            # (an embedding with a state of its own runs once a step)
            origin = hidden.clone() if self.embedding.takes_context else self._embed(ctx, bindings)
        wants_logits = want_rows is not None and want_rows.numel() > 0
        every_row = wants_logits and want_every_row and want_rows.numel() == ctx.num_rows
        for index, entry in enumerate(order):
            block = self.layers[entry.layer]
            if entry.inject is not None:
                stream = self.injections[entry.inject].forward(stream, origin, ctx)
            if not block.accepts_next_norm:
                stream = block.forward(stream, ctx, bindings[index])
                continue
            # the norm that will consume what this block returns: the next block's first one, or the final norm if
            # it runs on every row (on a few wanted rows it runs after they have been picked out); None where an
            # injection changes the stream in between
            if index + 1 < len(order):
                next_norm = self.layers[order[index + 1].layer].entry_norm() if order[index + 1].inject is None else None
            else:
                next_norm = self.final_norm if every_row else None
            stream = block.forward(stream, ctx, bindings[index], next_norm=next_norm)
        if not wants_logits:
            return None
        return self.logits_at(stream, want_rows, every_row)

    def logits_at(self, stream: ResidualStream, want_rows: torch.Tensor, every_row: bool = False) -> torch.Tensor:
        count = want_rows.numel()
        width = stream.residual.shape[1]
        if every_row and stream.prepared is not None and stream.prepared.norm is self.final_norm:
            return self.head.forward(stream.prepared if self.head.accepts_deferred_norm else stream.prepared.materialize())
        pending = [stream.update, stream.update_b]
        if every_row:
            residual = stream.residual[:count]
            pending = [None if u is None else u[:count] for u in pending]
        else:
            residual = torch.empty((count, width), dtype=stream.residual.dtype, device=stream.residual.device)
            kernels.gather_rows(want_rows, stream.residual, residual)
            for index, update in enumerate(pending):
                if update is not None:
                    pending[index] = kernels.gather_rows(want_rows, update, torch.empty((count, update.shape[1]), dtype=update.dtype,
                                                                                 device=update.device))
        final = DeferredNorm(self.final_norm, residual, pending[0], pending[1])
        return self.head.forward(final if self.head.accepts_deferred_norm else final.materialize())
