"""Token embedding (a row gather, src/cuda/kernels.rs:10-24) and the output head.

The head multiplies the normalised hidden rows by the ``[vocab, hidden]`` matrix
(src/cuda/dense_decoder.rs:824-831) and returns 32-bit logits.  With tied embeddings the
model description names one checkpoint tensor for both parts, and both keep one device copy.
"""

from __future__ import annotations

from typing import Dict, Mapping, Optional

import torch

from .. import kernels
from ..config.spec import PartSpec
from ..weights.loader import ExpectedTensor
from .base import EMBEDDINGS, HEADS, Embedding, Head, Runtime, StateNeed
from .linear import BestOfRows, Linear


@EMBEDDINGS.register("token_embedding")
class TokenEmbedding(Embedding):
    """params: ``vocab_size, hidden_size``, optional ``stream`` (``"float32"``: the rows come out in 32-bit whatever
    the run dtype, for a model whose residual stream is kept in 32-bit), optional ``scale`` (the rows are multiplied
    by it, in 32-bit: needs the 32-bit stream); weights: ``table``."""

    graph_safe = True

    def __init__(self, spec: PartSpec, tensors: Mapping[str, torch.Tensor], runtime: Runtime):
        super().__init__(spec, tensors, runtime)
        self.vocab_size = int(spec.params["vocab_size"])
        self.hidden_size = int(spec.params["hidden_size"])
        self.table = runtime.matrix(tensors["table"])
        stream = spec.params.get("stream")
        if stream not in (None, "float32"):
            raise ValueError(f"an embedding's stream is the run dtype or 'float32', got '{stream}'")
        self.widen = stream == "float32" and self.table.dtype != torch.float32
        self.scale = float(spec.params.get("scale") or 1.0)
        if self.scale != 1.0 and stream != "float32":
            raise ValueError("a scaled embedding feeds a residual stream kept in 32-bit (stream='float32')")

    @classmethod
    def expected_tensors(cls, spec: PartSpec) -> Dict[str, ExpectedTensor]:
        p = spec.params
        return {spec.weights["table"]: ExpectedTensor((int(p["vocab_size"]), int(p["hidden_size"])))}

    def forward(self, token_ids: torch.Tensor, out: Optional[torch.Tensor] = None) -> torch.Tensor:
        if self.scale != 1.0:
            if out is None:
                out = torch.empty((token_ids.numel(), self.hidden_size), dtype=torch.float32, device=self.table.device)
            return kernels.embedding_scaled(token_ids, self.table, out, self.scale)
        if self.widen:
            if out is None:
                out = torch.empty((token_ids.numel(), self.hidden_size), dtype=torch.float32, device=self.table.device)
            return kernels.embedding_widen(token_ids, self.table, out)
        if out is None:
            out = torch.empty((token_ids.numel(), self.hidden_size), dtype=self.table.dtype, device=self.table.device)
        return kernels.embedding(token_ids, self.table, out)


@EMBEDDINGS.register("positioned_embedding")
class PositionedEmbedding(Embedding):
    """A token's row plus a learned row for its position, normed: ``rms(table[token] + positions[p]) * weight`` over
    ``groups`` equal consecutive parts of the row, as the 32-bit start of a residual stream kept in 32-bit.

    params: ``vocab_size, hidden_size, max_positions, groups, eps``; weights: ``table``, ``positions``, ``weight``."""

    graph_safe = True
    takes_positions = True

    def __init__(self, spec: PartSpec, tensors: Mapping[str, torch.Tensor], runtime: Runtime):
        super().__init__(spec, tensors, runtime)
        p = spec.params
        self.hidden_size = int(p["hidden_size"])
        self.groups = int(p.get("groups") or 1)
        self.eps = float(p["eps"])
        if self.groups < 1 or self.hidden_size % self.groups:
            raise ValueError(f"a norm over {self.groups} groups needs a size that they divide, got {self.hidden_size}")
        self.table = runtime.matrix(tensors["table"])
        self.positions = runtime.matrix(tensors["positions"])
        self.weight = runtime.vector_f32(tensors["weight"])

    @classmethod
    def expected_tensors(cls, spec: PartSpec) -> Dict[str, ExpectedTensor]:
        p, w = spec.params, spec.weights
        hidden = int(p["hidden_size"])
        return {w["table"]: ExpectedTensor((int(p["vocab_size"]), hidden)),
                w["positions"]: ExpectedTensor((int(p["max_positions"]), hidden)), w["weight"]: ExpectedTensor((hidden,))}

    @classmethod
    def random_tensor(cls, spec, role, shape, generator) -> torch.Tensor:
        noise = torch.randn(shape, generator=generator, dtype=torch.float32)
        return 1.0 + noise * 0.1 if role == "weight" else noise * (0.3 if role == "positions" else 1.0)

    def forward(self, token_ids: torch.Tensor, positions: torch.Tensor, out: Optional[torch.Tensor] = None) -> torch.Tensor:
        if out is None:
            out = torch.empty((token_ids.numel(), self.hidden_size), dtype=torch.float32, device=self.table.device)
        return kernels.embedding_norm(token_ids, positions, self.table, self.positions, self.weight, self.groups, self.eps, out)


@EMBEDDINGS.register("bigram_embedding")
class BigramEmbedding(Embedding):
    """A token's row plus a row for the pair it forms with the token in front: ``table[token] + pairs[(token in front * mul_prev +
    token * mul_cur) mod buckets]``, or the last row of ``pairs`` for a sequence's first token.  The rows come out in 32-bit,
    ``copies`` times side by side (a stream kept as several copies starts with equal ones).

    params: ``vocab_size, hidden_size, buckets, mul_prev, mul_cur``, optional ``copies``; weights: ``table``, ``pairs``
    ``[buckets + 1, hidden]``.  A request's last token is state in its slot: a step's first token of a request pairs with it."""

    graph_safe = True
    takes_context = True

    def __init__(self, spec: PartSpec, tensors: Mapping[str, torch.Tensor], runtime: Runtime):
        super().__init__(spec, tensors, runtime)
        p = spec.params
        self.hidden_size = int(p["hidden_size"])
        self.buckets = int(p["buckets"])
        self.mul_prev, self.mul_cur = int(p["mul_prev"]), int(p["mul_cur"])
        self.copies = int(p.get("copies") or 1)
        if self.buckets < 1 or self.copies < 1:
            raise ValueError("bigram_embedding needs at least one bucket and one copy")
        self.table = runtime.matrix(tensors["table"])
        self.pairs = runtime.matrix(tensors["pairs"])

    @classmethod
    def expected_tensors(cls, spec: PartSpec) -> Dict[str, ExpectedTensor]:
        p, w = spec.params, spec.weights
        hidden = int(p["hidden_size"])
        return {w["table"]: ExpectedTensor((int(p["vocab_size"]), hidden)),
                w["pairs"]: ExpectedTensor((int(p["buckets"]) + 1, hidden))}

    @classmethod
    def random_tensor(cls, spec, role, shape, generator) -> torch.Tensor:
        return torch.randn(shape, generator=generator, dtype=torch.float32) * (0.5 if role == "pairs" else 1.0)

    def cache_need(self) -> StateNeed:
        return StateNeed((1,), torch.int32)

    def forward(self, token_ids: torch.Tensor, ctx, cache, out: Optional[torch.Tensor] = None) -> torch.Tensor:
        if cache is None or cache.storage is None:
            raise RuntimeError("bigram_embedding needs a state binding")
        if out is None:
            out = torch.empty((token_ids.numel(), self.copies * self.hidden_size), dtype=torch.float32, device=self.table.device)
        return kernels.bigram_embedding(token_ids, ctx.positions, ctx.seq_of_row, ctx.row_start, ctx.state_slots, self.table,
                                        self.pairs, cache.storage, out, self.copies, self.mul_prev, self.mul_cur)


@HEADS.register("lm_head")
class LMHead(Head):
    """params: ``vocab_size, hidden_size``, optional ``scale`` (the logits are multiplied by it); weights: ``weight``.
    Returns float32 logits."""

    graph_safe = True

    def __init__(self, spec: PartSpec, tensors: Mapping[str, torch.Tensor], runtime: Runtime):
        super().__init__(spec, tensors, runtime)
        self.vocab_size = int(spec.params["vocab_size"])
        self.hidden_size = int(spec.params["hidden_size"])
        self.proj = Linear(tensors["weight"], runtime)     # the embedding's device copy if both name one tensor
        # per-CTA best logit of each row, left by the product when it is the weight-streaming kernel (at most 16
        # rows): the sampler then need not read the logits again to find a row's best token
        self.scale = float(spec.params.get("scale") or 1.0)
        # (scaled logits are scaled behind the product, so the product's own best-of-row values would not be theirs)
        self.best = BestOfRows(runtime.device) if not runtime.is_float32 and self.scale == 1.0 else None

    @classmethod
    def expected_tensors(cls, spec: PartSpec) -> Dict[str, ExpectedTensor]:
        p = spec.params
        return {spec.weights["weight"]: ExpectedTensor((int(p["vocab_size"]), int(p["hidden_size"])))}

    accepts_deferred_norm = True

    def forward(self, x, out: Optional[torch.Tensor] = None) -> torch.Tensor:
        from .base import DeferredNorm

        if self.best is not None:
            self.best.valid = False
        if isinstance(x, DeferredNorm):
            logits = self.proj.forward_normed(x, float32_out=True, best=self.best)
            if logits is not None:
                return logits if self.scale == 1.0 else kernels.scale_rows(logits, self.scale)
            x = x.materialize()
        logits = self.proj.forward(x, out=out, float32_out=True, best=self.best)
        return logits if self.scale == 1.0 else kernels.scale_rows(logits, self.scale)

    def argmax_partials(self):
        """``(values, indices)`` that the last ``forward`` left for the sampler, or None if it left none."""
        return self.best.buffers if self.best is not None and self.best.valid else None
