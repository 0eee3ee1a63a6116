"""Recurrent mixers: fixed-size state per request instead of pages.

``mingru``: a gated recurrence whose gates read only the current token, so that within a step it is an affine scan
per channel.  With ``h`` the mixer's input,

    z_t = sigmoid(Wz h_t + bz)                       the update gate, ``width`` channels
    c_t = u_t + 1/2  if u_t >= 0  else sigmoid(u_t)   with u_t = Wx h_t + bx, the candidate
    S_t = (1 - z_t) * S_(t-1) + z_t * c_t            element by element, S_(-1) = 0
    y_t = Wo (S_t * silu(Wg h_t))

The three input projections are one product whose result is kept in 32-bit; biases, activations, the recurrence
and the output gate are 32-bit inside one kernel; ``S`` lives in the request's state slot as float32.

``rglru``: a real-gated linear recurrent unit behind a short convolution, beside a second branch that gates its output,

    y_t = gelu_tanh(Wy h_t + by)                      u_t = conv(Wx h + bx)_t + bc     causal, per channel, ``taps`` inputs
    r_t = sigmoid(Ra_b u_t + ba),  i_t = sigmoid(Ri_b u_t + bi)      square matrices over each of ``blocks`` runs of channels
    log a_t = -8 r_t softplus(lam)
    S_t = a_t * S_(t-1) + sqrt(1 - a_t^2) * i_t * u_t                element by element, S_(-1) = 0
    out_t = Wo (S_t * y_t)

The two input projections are one product; the convolution is a kernel of its own whose last ``taps - 1`` inputs are part of
the request's state (32-bit); the gates' matrices are one block-diagonal product whose kernel leaves ``a_t`` and what enters
the state, in 32-bit, for the scan, or takes the step itself where every sequence brings one row.
"""

from __future__ import annotations

from typing import Dict, Mapping

import torch

from .. import kernels
from ..config.spec import PartSpec
from ..weights.loader import ExpectedTensor
from .base import MIXERS, DeferredNorm, Mixer, Runtime, StateNeed, StepContext
from .linear import Linear


@MIXERS.register("mingru")
class MinGRU(Mixer):
    """params: ``hidden_size, width``, optional ``stream``; weights: ``z, z_bias, x, x_bias, g, o``."""

    graph_safe = True

    def __init__(self, spec: PartSpec, tensors: Mapping[str, torch.Tensor], runtime: Runtime):
        super().__init__(spec, tensors, runtime)
        p = spec.params
        self.hidden_size = int(p["hidden_size"])
        self.width = int(p["width"])
        self.stream_f32 = p.get("stream") == "float32"
        self.in_proj = Linear(torch.cat([tensors["z"], tensors["x"], tensors["g"]], dim=0), runtime)
        self.o_proj = Linear(tensors["o"], runtime)
        self.bias_z = runtime.vector_f32(tensors["z_bias"])
        self.bias_x = runtime.vector_f32(tensors["x_bias"])

    @classmethod
    def expected_tensors(cls, spec: PartSpec) -> Dict[str, ExpectedTensor]:
        p, w = spec.params, spec.weights
        hidden, width = int(p["hidden_size"]), int(p["width"])
        return {
            w["z"]: ExpectedTensor((width, hidden)), w["z_bias"]: ExpectedTensor((width,)),
            w["x"]: ExpectedTensor((width, hidden)), w["x_bias"]: ExpectedTensor((width,)),
            w["g"]: ExpectedTensor((width, hidden)), w["o"]: ExpectedTensor((hidden, width)),
        }

    @classmethod
    def random_tensor(cls, spec, role, shape, generator) -> torch.Tensor:
        if role.endswith("_bias"):
            return torch.randn(shape, generator=generator, dtype=torch.float32) * 0.5
        return torch.randn(shape, generator=generator, dtype=torch.float32) * (shape[-1] ** -0.5)

    def products(self):
        """``(name, Linear, epilogue)`` of the mixer's matrix products, for the printed kernel plan."""
        from .. import plan

        return [("z/x/gate", self.in_proj, plan.F32), ("o", self.o_proj, plan.F32 if self.stream_f32 else plan.BF16)]

    def cache_need(self) -> StateNeed:
        return StateNeed((self.width,), torch.float32)

    def forward(self, x, ctx: StepContext, cache):
        if isinstance(x, DeferredNorm):
            x = x.materialize()
        if cache is None or cache.storage is None:
            raise RuntimeError("mingru needs a state binding")
        proj = self.in_proj.forward(x, float32_out=True)        # gates and candidate enter the recurrence in 32-bit
        gated = torch.empty((proj.shape[0], self.width), dtype=self.runtime.dtype, device=proj.device)
        kernels.gated_recurrence(proj, self.bias_z, self.bias_x, cache.storage, gated, ctx.row_start, ctx.state_slots,
                                 num_seqs=ctx.num_seqs, max_new=ctx.max_new)
        return self.o_proj.forward(gated, float32_out=self.stream_f32)


@MIXERS.register("rglru")
class RGLRU(Mixer):
    """params: ``hidden_size, width, blocks, conv_taps``, optional ``stream``; weights: ``y, y_bias, x, x_bias, conv``
    (``[width, taps]``), ``conv_bias, r, r_bias, i, i_bias`` (``[blocks, size, size]`` and ``[blocks, size]``), ``decay``
    (``[width]``), ``o``."""

    graph_safe = True      # reads only device-side metadata of the step (and its shape)

    def __init__(self, spec: PartSpec, tensors: Mapping[str, torch.Tensor], runtime: Runtime):
        super().__init__(spec, tensors, runtime)
        p = spec.params
        self.hidden_size = int(p["hidden_size"])
        self.width = int(p["width"])
        self.blocks = int(p["blocks"])
        self.conv_taps = int(p["conv_taps"])
        self.stream_f32 = p.get("stream") == "float32"
        if self.blocks < 1 or self.width % self.blocks:
            raise ValueError(f"rglru: {self.blocks} blocks do not divide {self.width} channels")
        if self.conv_taps < 1:
            raise ValueError("rglru: the short convolution takes at least one tap")
        self.in_proj = Linear(torch.cat([tensors["y"], tensors["x"]], dim=0), runtime)
        self.o_proj = Linear(tensors["o"], runtime)
        self.y_bias = runtime.vector_f32(tensors["y_bias"])
        self.x_bias = runtime.vector_f32(tensors["x_bias"])
        # [taps, width]: tap j of every channel side by side, as the kernel reads them
        self.taps = tensors["conv"].to(device=runtime.device, dtype=torch.float32).t().contiguous()
        self.conv_bias = runtime.vector_f32(tensors["conv_bias"])
        # the rows of the two matrices of a block alternate: the kernel's neighbouring sums are r and i of one channel
        gates = torch.stack([tensors["r"], tensors["i"]], dim=2).flatten(1, 2)
        self.gates = gates.to(device=runtime.device, dtype=runtime.dtype).contiguous()
        self.r_bias = runtime.vector_f32(tensors["r_bias"]).reshape(-1)
        self.i_bias = runtime.vector_f32(tensors["i_bias"]).reshape(-1)
        decay = tensors["decay"].to(torch.float64)
        self.rate = (-8.0 * torch.nn.functional.softplus(decay)).to(device=runtime.device, dtype=torch.float32).contiguous()

    @classmethod
    def expected_tensors(cls, spec: PartSpec) -> Dict[str, ExpectedTensor]:
        p, w = spec.params, spec.weights
        hidden, width, blocks = int(p["hidden_size"]), int(p["width"]), int(p["blocks"])
        size = width // max(1, blocks)
        return {
            w["y"]: ExpectedTensor((width, hidden)), w["y_bias"]: ExpectedTensor((width,)),
            w["x"]: ExpectedTensor((width, hidden)), w["x_bias"]: ExpectedTensor((width,)),
            w["conv"]: ExpectedTensor((width, int(p["conv_taps"]))), w["conv_bias"]: ExpectedTensor((width,)),
            w["r"]: ExpectedTensor((blocks, size, size)), w["r_bias"]: ExpectedTensor((blocks, size)),
            w["i"]: ExpectedTensor((blocks, size, size)), w["i_bias"]: ExpectedTensor((blocks, size)),
            w["decay"]: ExpectedTensor((width,)), w["o"]: ExpectedTensor((hidden, width)),
        }

    @classmethod
    def random_tensor(cls, spec, role, shape, generator) -> torch.Tensor:
        noise = torch.randn(shape, generator=generator, dtype=torch.float32)
        if role.endswith("_bias"):
            return noise * 0.3
        if role == "decay":            # decays between nothing remembered and nothing forgotten
            return torch.rand(shape, generator=generator, dtype=torch.float32) * 6.0 - 6.0
        if role == "conv":
            return noise * 0.5
        return noise * (shape[-1] ** -0.5)

    def products(self):
        """``(name, Linear, epilogue)`` of the mixer's matrix products, for the printed kernel plan."""
        from .. import plan

        return [("y/x", self.in_proj, plan.BF16), ("o", self.o_proj, plan.F32 if self.stream_f32 else plan.BF16)]

    def cache_need(self):
        state = StateNeed((self.width,), torch.float32)
        if self.conv_taps == 1:
            return state
        return (state, StateNeed((self.conv_taps - 1, self.width), torch.float32))

    def forward(self, x, ctx: StepContext, cache):
        if isinstance(x, DeferredNorm):
            x = x.materialize()
        state, inputs = cache if isinstance(cache, tuple) else (cache, None)
        if state is None or state.storage is None or (self.conv_taps > 1 and (inputs is None or inputs.storage is None)):
            raise RuntimeError("rglru needs a binding for its state and, with more than one tap, for its convolution's inputs")
        if not state.writes:
            raise NotImplementedError("rglru keeps a state of its own: a run entry cannot read another entry's")
        proj = self.in_proj.forward(x)
        rows = proj.shape[0]
        y, before = proj[:, :self.width], proj[:, self.width:]
        u = torch.empty((rows, self.width), dtype=proj.dtype, device=proj.device)
        kernels.short_conv(before, self.x_bias, self.taps, self.conv_bias, None if inputs is None else inputs.storage, u,
                           ctx.positions, ctx.seq_of_row, ctx.row_start, ctx.seq_begin, ctx.state_slots,
                           num_seqs=ctx.num_seqs, single=ctx.max_new == 1)
        gated = torch.empty((rows, self.width), dtype=proj.dtype, device=proj.device)
        kernels.rglru(u, self.gates, self.r_bias, self.i_bias, self.rate, y, self.y_bias, state.storage, gated, ctx.row_start,
                      ctx.state_slots, num_seqs=ctx.num_seqs, max_new=ctx.max_new)
        return self.o_proj.forward(gated, float32_out=self.stream_f32)
