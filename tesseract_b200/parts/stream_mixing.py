"""How the copies of a stream kept as several copies meet around a sublayer.

``hyper_connections``: with ``x_1 .. x_s`` the copies and ``y`` the result of a sublayer (which read a weighted sum of the copies
through its norm, ``mixed_streams_rms_norm``),

    x_t <- sum_s mix[s, t] x_s + out[t] * y            all at once, from the old copies

``mix`` ``[s, s]`` and ``out`` ``[s]`` are the sublayer's own.  This part holds the tensors; the mixing itself and the following
norm are the block's fused kernel.
"""

from __future__ import annotations

from typing import Dict, Mapping

import torch

from ..config.spec import PartSpec
from ..weights.loader import ExpectedTensor
from .base import STREAM_MIXINGS, Runtime, StreamMixing

_SUBLAYERS = ("mixer", "feed_forward")


@STREAM_MIXINGS.register("hyper_connections")
class HyperConnections(StreamMixing):
    """params: ``streams``, ``feed_forward`` (bool: whether the layer has one); weights: ``mixer_mix, mixer_out`` and, with a
    feed-forward, ``feed_forward_mix, feed_forward_out``."""

    graph_safe = True

    def __init__(self, spec: PartSpec, tensors: Mapping[str, torch.Tensor], runtime: Runtime):
        super().__init__(spec, tensors, runtime)
        self.streams = int(spec.params["streams"])
        self.sublayers = _SUBLAYERS if spec.params.get("feed_forward") else _SUBLAYERS[:1]
        self._mix = {w: runtime.vector_f32(tensors[w + "_mix"]) for w in self.sublayers}
        self._share = {w: runtime.vector_f32(tensors[w + "_out"]) for w in self.sublayers}

    @classmethod
    def expected_tensors(cls, spec: PartSpec) -> Dict[str, ExpectedTensor]:
        s, w = int(spec.params["streams"]), spec.weights
        out = {}
        for which in (_SUBLAYERS if spec.params.get("feed_forward") else _SUBLAYERS[:1]):
            out[w[which + "_mix"]] = ExpectedTensor((s, s))
            out[w[which + "_out"]] = ExpectedTensor((s,))
        return out

    @classmethod
    def random_tensor(cls, spec, role, shape, generator) -> torch.Tensor:
        noise = torch.randn(shape, generator=generator, dtype=torch.float32)
        if role.endswith("_mix"):
            return torch.eye(shape[0]) * 0.8 + noise * 0.15
        return 1.0 + noise * 0.2

    def mix(self, which: str) -> torch.Tensor:
        return self._mix[which]

    def share(self, which: str) -> torch.Tensor:
        return self._share[which]
