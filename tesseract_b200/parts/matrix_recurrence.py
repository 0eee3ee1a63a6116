"""Recurrent mixers whose state is a matrix per head (fixed-size state per request instead of pages).

With ``h`` the mixer's input, per head ``S_t = a_t S_(t-1) + k_t u_t^T``, read by a query: ``S_t^T q_t``; the decay ``a_t`` is one number per
head and token.  ``S`` lives in the request's state slot in 32-bit and starts at zero.  Three kinds.

``state_space`` (Mamba-2): ``[z | x | B | C | dt] = W_in h``; ``x``, ``B`` and ``C`` pass a short causal convolution per channel with a bias and
SiLU; head ``n`` uses the ``B`` and ``C`` of group ``n // (heads / groups)``;

    dt = softplus(dt + dt_bias)      S_t = exp(-exp(A_log) dt) S_(t-1) + dt B_t x_t^T      y_t = S_t^T C_t + D x_t
    out = Wo (rms(y * silu(z)) * w)                          the root mean square over each of ``norm_groups`` parts of the row

``matrix_memory`` (the matrix memory of xLSTM): ``q, k, v, g`` projections of ``h``, ``q`` times ``key_dim^(-1/2)``, two gate logits a head,

    i = c tanh((Wi h + bi) / c)      f = log sigmoid(c tanh((Wf h + bf) / c))      m_t = max(f + m_(t-1), i), m_(-1) = 0
    S_t = e^(f + m_(t-1) - m_t) S_(t-1) + e^(i - m_t) k v^T      n_t the same with k alone
    o_t = S_t^T q / (max(|n_t . q|, e^(-m_t)) + 1e-6)            out = Wo (rms per head(o) * w * sigmoid(g))

``gated_delta`` (the gated delta rule): ``q, k`` (of ``num_kv_heads`` heads) and ``v`` pass short causal convolutions without bias and
SiLU; ``q`` and ``k`` become unit vectors per head, ``q`` times ``key_dim^(-1/2)``,

    beta = sigmoid(Wb h)      a = exp(-exp(A_log) softplus(Wa h + dt_bias))
    S <- a S      u = beta (v - S^T k)      S <- S + k u^T      o = S^T q          out = Wo (rms per head(o) * w * silu(g))

Per mixer: one product for everything that may be 16-bit, one small product for the gate logits, which stay 32-bit; the
convolution with its SiLU (``short_conv``; its last ``taps - 1`` inputs are state too); one kernel for gates, unit vectors, recurrence
and read-out, a sequence's rows one after the other with the state in registers, everything in 32-bit; one kernel for the norm
and the output gate; the output product, in 32-bit for a residual stream kept in 32-bit.
"""

from __future__ import annotations

from typing import Dict, Mapping, Optional

import torch

from .. import kernels, plan
from ..config.spec import PartSpec
from ..weights.loader import ExpectedTensor
from .base import MIXERS, DeferredNorm, Mixer, Runtime, StateNeed, StepContext
from .linear import Linear


class _MatrixMixer(Mixer):
    """What the three kinds share: products, convolution, recurrence, norm."""

    graph_safe = True      # reads only device-side metadata of the step (and its shape)
    recurrence: int

    def _prepare(self, runtime: Runtime, *, wide: torch.Tensor, gates: torch.Tensor, out: torch.Tensor, stream: Optional[str],
                 taps: Optional[torch.Tensor] = None, conv_bias: Optional[torch.Tensor] = None) -> None:
        self.stream_f32 = stream == "float32"
        self.in_proj = Linear(wide, runtime)
        self.gate_proj = Linear(gates, runtime)
        self.o_proj = Linear(out, runtime)
        # [taps, channels]: tap j of every channel side by side, as the kernel reads them
        self.taps = None if taps is None else taps.to(device=runtime.device, dtype=torch.float32).t().contiguous()
        self.conv_bias = None if conv_bias is None else runtime.vector_f32(conv_bias)
        self.o_width = self.num_heads * self.value_dim

    @staticmethod
    def _rate(a_log: torch.Tensor, runtime: Runtime) -> torch.Tensor:
        """``-exp(A_log)``, taken in 64-bit and rounded once."""
        return (-torch.exp(a_log.to(torch.float64))).to(device=runtime.device, dtype=torch.float32).contiguous()

    def products(self):
        """``(name, Linear, epilogue)`` of the mixer's matrix products, for the printed kernel plan."""
        return [("in", self.in_proj, plan.BF16), ("gates", self.gate_proj, plan.F32),
                ("o", self.o_proj, plan.F32 if self.stream_f32 else plan.BF16)]

    def cache_need(self):
        shape = kernels.matrix_state_shape(self.recurrence, self.num_heads, self.key_dim, self.value_dim)
        needs = [StateNeed(shape, torch.float32)]
        if self.recurrence == kernels.MATRIX_MEMORY:
            needs.append(StateNeed(shape[:2], torch.float32))                 # the running maximum, a copy per value column
        if self.taps is not None and self.taps.shape[0] > 1:
            needs.append(StateNeed((self.taps.shape[0] - 1, self.taps.shape[1]), torch.float32))
        return tuple(needs) if len(needs) > 1 else needs[0]

    def _bindings(self, cache):
        cache = cache if isinstance(cache, tuple) else (cache,)
        need = self.cache_need()
        count = len(need) if isinstance(need, tuple) else 1
        if len(cache) != count or any(c is None or c.storage is None for c in cache):
            raise RuntimeError(f"{self.kind} needs {count} state binding(s)")
        if any(not c.writes for c in cache):
            raise NotImplementedError(f"{self.kind} keeps a state of its own: a run entry cannot read another entry's")
        return [c.storage for c in cache]

    def _convolve(self, rows: torch.Tensor, state: Optional[torch.Tensor], ctx: StepContext) -> torch.Tensor:
        out = torch.empty((rows.shape[0], rows.shape[1]), dtype=rows.dtype, device=rows.device)
        return kernels.short_conv(rows, None, self.taps, self.conv_bias, state, out, ctx.positions, ctx.seq_of_row,
                                  ctx.row_start, ctx.seq_begin, ctx.state_slots, num_seqs=ctx.num_seqs,
                                  single=ctx.max_new == 1, activation=True)

    def _recur(self, rows, offsets, gates, per_head, state, ctx: StepContext, qk_heads: int, **more) -> torch.Tensor:
        out = torch.empty((rows.shape[0], self.o_width), dtype=torch.float32, device=rows.device)
        return kernels.matrix_recurrence(self.recurrence, rows, offsets, gates, per_head, state, out, ctx.row_start,
                                         ctx.state_slots, num_seqs=ctx.num_seqs, heads=self.num_heads, qk_heads=qk_heads,
                                         dim=self.key_dim, vdim=self.value_dim, max_new=ctx.max_new, **more)

    def _finish(self, v, gate, *, groups: int, size: int, gate_kind: int, aux=None) -> torch.Tensor:
        normed = torch.empty((v.shape[0], self.o_width), dtype=gate.dtype, device=gate.device)
        kernels.recurrence_norm(v, gate, self.norm_weight, normed, groups=groups, size=size, eps=self.eps, gate_kind=gate_kind,
                                aux=aux)
        return self.o_proj.forward(normed, float32_out=self.stream_f32)

    @classmethod
    def random_tensor(cls, spec, role, shape, generator) -> torch.Tensor:
        noise = torch.randn(shape, generator=generator, dtype=torch.float32)
        if role == "norm":
            return 1.0 + noise * 0.1
        if role == "conv_bias":
            return noise * 0.2
        if role in ("i_bias", "dt_bias"):
            return noise * 0.5
        if role == "f_bias":                  # forget gates from nearly closed to nearly open
            return noise * 2.0 + 2.0
        if role in ("a_log", "skip"):
            return noise * 0.7
        if role.endswith("conv"):
            return noise * 0.5
        return noise * (shape[-1] ** -0.5)


def _sizes(p, *names):
    return tuple(int(p[name]) for name in names)


@MIXERS.register("state_space")
class StateSpace(_MatrixMixer):
    """params: ``hidden_size, num_heads, value_dim, state`` (rows of the state matrix), ``groups, norm_groups, conv_taps, eps``,
    optional ``stream``; weights: ``in`` ``[2 * inner + 2 * groups * state + heads, hidden]`` with ``inner = heads * value_dim``, ``conv``
    ``[inner + 2 * groups * state, taps]``, ``conv_bias``, ``dt_bias``, ``a_log``, ``skip`` (``[heads]`` each), ``norm`` ``[inner]``, ``o``."""

    recurrence = kernels.STATE_SPACE

    def __init__(self, spec: PartSpec, tensors: Mapping[str, torch.Tensor], runtime: Runtime):
        super().__init__(spec, tensors, runtime)
        p = spec.params
        self.hidden_size, self.num_heads, self.value_dim, self.key_dim, self.groups, self.norm_groups, self.conv_taps = _sizes(
            p, "hidden_size", "num_heads", "value_dim", "state", "groups", "norm_groups", "conv_taps")
        self.eps = float(p["eps"])
        if self.num_heads % self.groups or (self.num_heads * self.value_dim) % self.norm_groups or self.conv_taps < 1:
            raise ValueError("state_space: groups divide the heads, norm groups the row, and the convolution has a tap")
        if self.key_dim > 1024:
            raise ValueError("the recurrence kernel takes states of up to 1024 rows a head")
        rows = tensors["in"]
        self._prepare(runtime, wide=rows[:-self.num_heads], gates=rows[-self.num_heads:], out=tensors["o"], stream=p.get("stream"),
                      taps=tensors["conv"], conv_bias=tensors["conv_bias"])
        self.per_head = (self._rate(tensors["a_log"], runtime), runtime.vector_f32(tensors["dt_bias"]),
                         runtime.vector_f32(tensors["skip"]))
        self.norm_weight = runtime.vector_f32(tensors["norm"])

    @classmethod
    def expected_tensors(cls, spec: PartSpec) -> Dict[str, ExpectedTensor]:
        p, w = spec.params, spec.weights
        hidden, heads, dv, n, groups, taps = _sizes(p, "hidden_size", "num_heads", "value_dim", "state", "groups", "conv_taps")
        inner, channels = heads * dv, heads * dv + 2 * groups * n
        return {w["in"]: ExpectedTensor((inner + channels + heads, hidden)), w["conv"]: ExpectedTensor((channels, taps)),
                w["conv_bias"]: ExpectedTensor((channels,)), w["dt_bias"]: ExpectedTensor((heads,)),
                w["a_log"]: ExpectedTensor((heads,)), w["skip"]: ExpectedTensor((heads,)), w["norm"]: ExpectedTensor((inner,)),
                w["o"]: ExpectedTensor((hidden, inner))}

    def forward(self, x, ctx: StepContext, cache):
        if isinstance(x, DeferredNorm):
            x = x.materialize()
        state, *inputs = self._bindings(cache)
        proj, dt = self.in_proj.forward(x), self.gate_proj.forward(x, float32_out=True)
        inner, width = self.o_width, self.groups * self.key_dim
        u = self._convolve(proj[:, inner:], inputs[0] if inputs else None, ctx)
        y = self._recur(u, (inner + width, inner, 0), dt, self.per_head, state, ctx, self.groups)
        return self._finish(y, proj[:, :inner], groups=self.norm_groups, size=inner // self.norm_groups,
                            gate_kind=kernels.NORM_GATE_SILU_FIRST)


@MIXERS.register("matrix_memory")
class MatrixMemory(_MatrixMixer):
    """params: ``hidden_size, num_heads, key_dim, value_dim, gate_cap, eps``, optional ``stream``; weights: ``q, k, v, g, i, f, i_bias,
    f_bias, norm`` (``[heads * value_dim]``), ``o``."""

    recurrence = kernels.MATRIX_MEMORY

    def __init__(self, spec: PartSpec, tensors: Mapping[str, torch.Tensor], runtime: Runtime):
        super().__init__(spec, tensors, runtime)
        p = spec.params
        self.hidden_size, self.num_heads, self.key_dim, self.value_dim = _sizes(p, "hidden_size", "num_heads", "key_dim", "value_dim")
        self.eps, self.cap = float(p["eps"]), float(p["gate_cap"])
        if not self.cap > 0.0:
            raise ValueError("matrix_memory: gate_cap must be positive")
        if self.key_dim > 1024:
            raise ValueError("the recurrence kernel takes keys of up to 1024 numbers a head")
        self._prepare(runtime, wide=torch.cat([tensors["q"], tensors["k"], tensors["v"], tensors["g"]], dim=0),
                      gates=torch.cat([tensors["i"], tensors["f"]], dim=0), out=tensors["o"], stream=p.get("stream"))
        self.per_head = (runtime.vector_f32(tensors["i_bias"]), runtime.vector_f32(tensors["f_bias"]))
        self.norm_weight = runtime.vector_f32(tensors["norm"])

    @classmethod
    def expected_tensors(cls, spec: PartSpec) -> Dict[str, ExpectedTensor]:
        p, w = spec.params, spec.weights
        hidden, heads, d, dv = _sizes(p, "hidden_size", "num_heads", "key_dim", "value_dim")
        return {w["q"]: ExpectedTensor((heads * d, hidden)), w["k"]: ExpectedTensor((heads * d, hidden)),
                w["v"]: ExpectedTensor((heads * dv, hidden)), w["g"]: ExpectedTensor((heads * dv, hidden)),
                w["i"]: ExpectedTensor((heads, hidden)), w["f"]: ExpectedTensor((heads, hidden)),
                w["i_bias"]: ExpectedTensor((heads,)), w["f_bias"]: ExpectedTensor((heads,)),
                w["norm"]: ExpectedTensor((heads * dv,)), w["o"]: ExpectedTensor((hidden, heads * dv))}

    def forward(self, x, ctx: StepContext, cache):
        if isinstance(x, DeferredNorm):
            x = x.materialize()
        state, running = self._bindings(cache)
        proj, gates = self.in_proj.forward(x), self.gate_proj.forward(x, float32_out=True)
        width = self.num_heads * self.key_dim
        aux = torch.empty((proj.shape[0], self.num_heads, 2), dtype=torch.float32, device=proj.device)
        o = self._recur(proj, (0, width, 2 * width), gates, self.per_head, state, ctx, self.num_heads, running=running, aux=aux,
                        cap=self.cap, q_scale=self.key_dim ** -0.5)
        return self._finish(o, proj[:, 2 * width + self.o_width:], groups=self.num_heads, size=self.value_dim,
                            gate_kind=kernels.NORM_GATE_SIGMOID, aux=aux)


@MIXERS.register("gated_delta")
class GatedDelta(_MatrixMixer):
    """params: ``hidden_size, num_heads, num_kv_heads, key_dim, value_dim, conv_taps, eps``, optional ``stream``; weights: ``q, k, v, g``,
    ``q_conv, k_conv, v_conv`` (``[channels, taps]``), ``a, b`` (``[heads, hidden]``), ``a_log, dt_bias`` (``[heads]``), ``norm``
    (``[value_dim]``, shared by the heads), ``o``."""

    recurrence = kernels.DELTA_RULE

    def __init__(self, spec: PartSpec, tensors: Mapping[str, torch.Tensor], runtime: Runtime):
        super().__init__(spec, tensors, runtime)
        p = spec.params
        self.hidden_size, self.num_heads, self.num_kv_heads, self.key_dim, self.value_dim, self.conv_taps = _sizes(
            p, "hidden_size", "num_heads", "num_kv_heads", "key_dim", "value_dim", "conv_taps")
        self.eps = float(p["eps"])
        if self.num_heads % self.num_kv_heads or self.conv_taps < 1:
            raise ValueError("gated_delta: q/k heads divide the heads, and the convolution has a tap")
        if self.key_dim > 1024:
            raise ValueError("the recurrence kernel takes keys of up to 1024 numbers a head")
        self._prepare(runtime, wide=torch.cat([tensors["q"], tensors["k"], tensors["v"], tensors["g"]], dim=0),
                      gates=torch.cat([tensors["a"], tensors["b"]], dim=0), out=tensors["o"], stream=p.get("stream"),
                      taps=torch.cat([tensors["q_conv"], tensors["k_conv"], tensors["v_conv"]], dim=0))
        self.per_head = (self._rate(tensors["a_log"], runtime), runtime.vector_f32(tensors["dt_bias"]))
        self.norm_weight = runtime.vector_f32(tensors["norm"])

    @classmethod
    def expected_tensors(cls, spec: PartSpec) -> Dict[str, ExpectedTensor]:
        p, w = spec.params, spec.weights
        hidden, heads, kv, d, dv, taps = _sizes(p, "hidden_size", "num_heads", "num_kv_heads", "key_dim", "value_dim", "conv_taps")
        return {w["q"]: ExpectedTensor((kv * d, hidden)), w["k"]: ExpectedTensor((kv * d, hidden)),
                w["v"]: ExpectedTensor((heads * dv, hidden)), w["g"]: ExpectedTensor((heads * dv, hidden)),
                w["q_conv"]: ExpectedTensor((kv * d, taps)), w["k_conv"]: ExpectedTensor((kv * d, taps)),
                w["v_conv"]: ExpectedTensor((heads * dv, taps)),
                w["a"]: ExpectedTensor((heads, hidden)), w["b"]: ExpectedTensor((heads, hidden)),
                w["a_log"]: ExpectedTensor((heads,)), w["dt_bias"]: ExpectedTensor((heads,)),
                w["norm"]: ExpectedTensor((dv,)), w["o"]: ExpectedTensor((hidden, heads * dv))}

    def forward(self, x, ctx: StepContext, cache):
        if isinstance(x, DeferredNorm):
            x = x.materialize()
        state, *inputs = self._bindings(cache)
        proj, gates = self.in_proj.forward(x), self.gate_proj.forward(x, float32_out=True)
        width = self.num_kv_heads * self.key_dim
        channels = 2 * width + self.o_width
        u = self._convolve(proj[:, :channels], inputs[0] if inputs else None, ctx)
        o = self._recur(u, (0, width, 2 * width), gates, self.per_head, state, ctx, self.num_kv_heads,
                        q_scale=self.key_dim ** -0.5)
        return self._finish(o, proj[:, channels:], groups=self.num_heads, size=self.value_dim, gate_kind=kernels.NORM_GATE_SILU)
