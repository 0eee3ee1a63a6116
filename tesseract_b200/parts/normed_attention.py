"""Grouped-query attention whose queries and keys are brought to unit root mean square after the rotation.

Per row ``h`` (the mixer's input):

* one fused product gives the queries (``num_heads * key_dim``), keys (``num_kv_heads * key_dim``) and values
  (``num_kv_heads * value_dim``); query head ``i`` reads kv head ``i // (num_heads / num_kv_heads)``;
* the position encoding (``rotary_blend``, rotate-half layout) turns the first ``dims`` numbers of every query and
  key head; with ``qk_norm_eps`` every query and key head is then divided by ``sqrt(mean(head^2) + qk_norm_eps)``
  (no weight); rotated, normalised keys and the values go into the request's pages;
* with ``projection_norm_eps`` the norm stands in front of the rotation and runs over the whole projection instead: all heads'
  queries over their one root mean square, times a weight per number, and the keys likewise; with ``values_from_keys`` there
  is no value projection and a token's values are its keys as projected, before norm and rotation;
* every row attends over the keys its mask lets it see: ``causal`` (all up to its own position), ``window`` (its own
  and the ``size - 1`` positions before it; older pages go back to the pool), ``blocks`` (the positions are cut into consecutive
  blocks of ``size`` from 0, and a row sees its own block up to itself) or ``window_pooled``: the window and, for
  every block of ``pool`` positions that ends in front of it (blocks are counted from position 0; block ``b`` is seen
  from position ``p`` if ``(b + 1) * pool <= p - size + 1``), one key and one value that are the averages of the block's
  keys and values as the pages hold them; so for up to ``pool - 1`` steps a token is visible neither by itself nor through
  its block.  The averages live in pages of their own (an entry a block) and are written by the step that brings a
  block's last token.  A ``window`` may also keep the first ``keep_first`` positions of the sequence, which every row goes
  on seeing (their pages stay; older pages behind the window go back to the pool).  Scores ``(q . k) * scale``, with ``softcap`` then ``softcap * tanh(score / softcap)``, the softmax
  and the weights are 32-bit; with ``sink`` the denominator also holds ``exp`` of a learned number per query head; with
  ``distance_bias`` the score of the key ``n`` positions back loses ``w * ln(1 + r * n)``, two numbers per query head;
* with ``head_gate`` a head's output is multiplied by the sigmoid of one number that a projection of ``h`` gives it;
* with ``bias`` the three projections add a bias each, with ``output_bias`` the output projection does;
* values may be mixed across layers: a part with ``value_mix`` ``"first"`` leaves its values in the step
  (``StepContext.carried``), a later one with ``"mix"`` stores ``(1 - x) v + x v_first`` instead of its own values ``v``, ``x``
  one learned number (the first part's values of the same token are rows of the same step, so nothing is cached for it);
* the output projection's result comes out in 32-bit for a residual stream kept in 32-bit (``stream`` = ``"float32"``).

Rotation, normalisation and the cache write are one kernel; the attention kernel is the one the other mixers with
keys and values of separate widths use, or, for bfloat16 steps of many rows and head sizes it is built for, the
tensor-core kernel with the same masks and 32-bit scores and weights (the kernel plan decides).
"""

from __future__ import annotations

from typing import Dict, Mapping

import torch

from .. import kernels, plan
from ..config.spec import PartSpec
from ..weights.loader import ExpectedTensor
from .base import (MIXERS, POSITION_ENCODINGS, DeferredNorm, Mixer, PagedKeyValueNeed, PooledBlocksNeed, Runtime,
                   StepContext)
from .linear import Linear

_MASKS = {"causal": kernels.MASK_CAUSAL, "window": kernels.MASK_WINDOW, "window_pooled": kernels.MASK_WINDOW_POOLED,
          "blocks": kernels.MASK_BLOCKS}


@MIXERS.register("normed_attention")
class NormedAttention(Mixer):
    """params: ``hidden_size, num_heads, num_kv_heads, key_dim, value_dim, scale``, ``mask`` (``{"kind": "causal" |
    "window" | "blocks" | "window_pooled", "size": n, "pool": P, "keep_first": k}``), ``qk_norm_eps`` (None: queries and keys stay as
    rotated), optional ``softcap``, ``sink`` (bool), ``bias`` (bool), ``output_bias`` (bool), ``distance_bias`` (bool),
    ``value_mix`` (``"first"`` | ``"mix"``), ``projection_norm_eps``, ``values_from_keys`` (bool), ``head_gate`` (bool), ``stream``.  weights:
    ``q, k, v, o`` (no ``v`` with ``values_from_keys``), with ``projection_norm_eps`` ``q_norm`` and ``k_norm`` (as wide as the
    projections), with ``head_gate`` ``g`` ``[num_heads, hidden]``, with ``bias`` also ``q_bias, k_bias,
    v_bias``, with ``output_bias`` ``o_bias``, with ``sink`` ``sink`` ``[num_heads]``, with ``distance_bias`` ``distance_weight``
    and ``distance_rate`` (``[num_heads]`` each), to mix ``value_mix`` (one number).  children: ``position``."""

    graph_safe = True      # reads only device-side metadata of the step (and its shape)

    def __init__(self, spec: PartSpec, tensors: Mapping[str, torch.Tensor], runtime: Runtime):
        super().__init__(spec, tensors, runtime)
        p = spec.params
        self.hidden_size = int(p["hidden_size"])
        self.num_heads = int(p["num_heads"])
        self.num_kv_heads = int(p["num_kv_heads"])
        self.key_dim = int(p["key_dim"])
        self.value_dim = int(p["value_dim"])
        self.scale = float(p["scale"])
        mask = dict(p.get("mask") or {"kind": "causal"})
        if mask.get("kind") not in _MASKS:
            raise ValueError(f"mask kind must be one of {sorted(_MASKS)}, got {mask.get('kind')!r}")
        self.mask_kind = mask["kind"]
        self.mask_size = int(mask.get("size") or 0)
        if self.mask_kind != "causal" and self.mask_size < 1:
            raise ValueError(f"a '{self.mask_kind}' mask needs a positive size")
        self.pool = int(mask.get("pool") or 0)
        if self.mask_kind == "window_pooled" and self.pool < 1:
            raise ValueError("a 'window_pooled' mask needs a positive pool")
        self.keep_first = int(mask.get("keep_first") or 0)
        if self.keep_first < 0 or (self.keep_first and self.mask_kind != "window"):
            raise ValueError("keep_first is a number of positions that a 'window' mask keeps")
        self.softcap = float(p.get("softcap") or 0.0)
        if self.softcap < 0.0:
            raise ValueError("softcap must not be negative")
        self.sinks = runtime.vector_f32(tensors["sink"]) if p.get("sink") else None
        self.distance_bias = None
        if p.get("distance_bias"):
            if self.mask_kind == "window_pooled":
                raise ValueError("averaged blocks have no distance: a distance bias goes with the other masks")
            self.distance_bias = (runtime.vector_f32(tensors["distance_weight"]), runtime.vector_f32(tensors["distance_rate"]))
        self.value_mix = p.get("value_mix")
        if self.value_mix not in (None, "first", "mix"):
            raise ValueError(f"value_mix is 'first', 'mix' or absent, got {self.value_mix!r}")
        self.mix = runtime.vector_f32(tensors["value_mix"]).reshape(1) if self.value_mix == "mix" else None
        self.biased = bool(p.get("bias"))
        eps = p.get("qk_norm_eps")
        self.unit_norm = eps is not None
        self.qk_norm_eps = float(eps) if eps is not None else 0.0
        eps = p.get("projection_norm_eps")
        self.projection_norm_eps = float(eps) if eps is not None else None
        self.values_from_keys = bool(p.get("values_from_keys"))
        self.projection_norm = None
        if self.projection_norm_eps is not None:
            if self.biased or self.unit_norm or self.value_mix is not None:
                raise ValueError("a norm over the whole projection goes with no biases, no unit norm and no mixed values")
            self.projection_norm = torch.cat([tensors["q_norm"], tensors["k_norm"]]).to(
                device=runtime.device, dtype=torch.float32).contiguous()
        elif self.values_from_keys:
            raise ValueError("keys that are values come with a norm over the whole projection")
        if self.values_from_keys and self.key_dim != self.value_dim:
            raise ValueError("keys that are values have the values' width")
        self.head_gated = bool(p.get("head_gate"))
        self.stream_f32 = p.get("stream") == "float32"
        if self.num_heads % self.num_kv_heads:
            raise ValueError("num_heads must be a multiple of num_kv_heads")
        if not (1 <= self.key_dim <= 1024 and 1 <= self.value_dim <= 512):
            raise ValueError("the attention kernel takes keys of up to 1024 and values of up to 512 numbers a head")
        self.q_width = self.num_heads * self.key_dim
        self.o_width = self.num_heads * self.value_dim
        # (the biases are added by the kernel behind the product, in 32-bit, in front of its rotation)
        self.in_bias = None
        if self.biased:
            self.in_bias = torch.cat([tensors["q_bias"], tensors["k_bias"], tensors["v_bias"]]).to(
                device=runtime.device, dtype=torch.float32).contiguous()
        wide = [tensors["q"], tensors["k"]] + ([] if self.values_from_keys else [tensors["v"]])
        self.gate_offset = sum(t.shape[0] for t in wide)
        if self.head_gated:
            wide.append(tensors["g"])
            missing = -(self.gate_offset + self.num_heads) % 8      # (rows of zeros, so that projected rows start on 16 bytes)
            if missing:
                wide.append(torch.zeros((missing, self.hidden_size), dtype=tensors["g"].dtype))
        self.in_proj = Linear(torch.cat(wide, dim=0), runtime)
        self.o_proj = Linear(tensors["o"], runtime, bias=tensors["o_bias"] if p.get("output_bias") else None)
        position_spec = spec.children.get("position") or PartSpec.make("none")
        self.position = POSITION_ENCODINGS.get(position_spec.kind)(position_spec, {}, runtime)
        if self.position.kind not in ("rotary_blend", "none"):
            raise ValueError(f"normed_attention rotates halves or not at all, got position encoding '{self.position.kind}'")
        self.rot_dims = int(getattr(self.position, "dims", 0))
        self.inv_freq = getattr(self.position, "half_inv_freq", None)
        self.amplitude = float(getattr(self.position, "amplitude", 1.0))
        if self.rot_dims > self.key_dim:
            raise ValueError("the rotation covers more numbers than a key has")

    @classmethod
    def expected_tensors(cls, spec: PartSpec) -> Dict[str, ExpectedTensor]:
        p, w = spec.params, spec.weights
        hidden, d, dv = int(p["hidden_size"]), int(p["key_dim"]), int(p["value_dim"])
        heads, kv = int(p["num_heads"]), int(p["num_kv_heads"])
        out = {
            w["q"]: ExpectedTensor((heads * d, hidden)),
            w["k"]: ExpectedTensor((kv * d, hidden)),
            w["o"]: ExpectedTensor((hidden, heads * dv)),
        }
        if not p.get("values_from_keys"):
            out[w["v"]] = ExpectedTensor((kv * dv, hidden))
        if p.get("projection_norm_eps") is not None:
            out.update({w["q_norm"]: ExpectedTensor((heads * d,)), w["k_norm"]: ExpectedTensor((kv * d,))})
        if p.get("head_gate"):
            out[w["g"]] = ExpectedTensor((heads, hidden))
        if p.get("bias"):
            out.update({w["q_bias"]: ExpectedTensor((heads * d,)), w["k_bias"]: ExpectedTensor((kv * d,)),
                        w["v_bias"]: ExpectedTensor((kv * dv,))})
        if p.get("output_bias"):
            out[w["o_bias"]] = ExpectedTensor((hidden,))
        if p.get("sink"):
            out[w["sink"]] = ExpectedTensor((heads,))
        if p.get("distance_bias"):
            out.update({w["distance_weight"]: ExpectedTensor((heads,)), w["distance_rate"]: ExpectedTensor((heads,))})
        if p.get("value_mix") == "mix":
            out[w["value_mix"]] = ExpectedTensor(())
        return out

    @classmethod
    def random_tensor(cls, spec, role, shape, generator) -> torch.Tensor:
        if role.endswith("_bias"):
            return torch.randn(shape, generator=generator, dtype=torch.float32) * 0.3
        if role in ("distance_weight", "distance_rate", "value_mix"):
            return torch.rand(shape, generator=generator, dtype=torch.float32) * 0.5 + 0.1
        if role.endswith("_norm"):
            return 1.0 + torch.randn(shape, generator=generator, dtype=torch.float32) * 0.1
        if role == "sink":
            return torch.randn(shape, generator=generator, dtype=torch.float32)
        return torch.randn(shape, generator=generator, dtype=torch.float32) * (shape[-1] ** -0.5)

    def products(self):
        """``(name, Linear, epilogue)`` of the mixer's matrix products, for the printed kernel plan."""
        from .. import plan

        name = "q/k" + ("" if self.values_from_keys else "/v") + ("/gate" if self.head_gated else "")
        return [(name, self.in_proj, plan.BF16), ("o", self.o_proj, plan.F32 if self.stream_f32 else plan.BF16)]

    def cache_need(self):
        if self.mask_kind == "window_pooled":
            # the tokens of a block stay until the block is averaged, although the window may have passed them
            return (PagedKeyValueNeed(num_kv_heads=self.num_kv_heads, key_dim=self.key_dim, value_dim=self.value_dim,
                                      window=self.mask_size, hold=self.pool),
                    PooledBlocksNeed(num_kv_heads=self.num_kv_heads, key_dim=self.key_dim, value_dim=self.value_dim,
                                     pool=self.pool))
        return PagedKeyValueNeed(num_kv_heads=self.num_kv_heads, key_dim=self.key_dim, value_dim=self.value_dim,
                                 window=self.mask_size if self.mask_kind == "window" else None,
                                 block=self.mask_size if self.mask_kind == "blocks" else None, keep_first=self.keep_first)

    def attention_choice(self, rows: int) -> str:
        """The attention kernel of a step of ``rows`` rows (all three know the cap, the learned sink and pooled blocks)."""
        return plan.masked_attention(self.runtime.dtype, rows, self.key_dim, self.value_dim,
                                     heads_per_kv=self.num_heads // self.num_kv_heads)

    def forward(self, x, ctx: StepContext, cache):
        if isinstance(x, DeferredNorm):
            x = x.materialize()
        pooled = None
        if self.mask_kind == "window_pooled":
            if not isinstance(cache, tuple) or len(cache) != 2:
                raise RuntimeError("a pooled window needs two cache bindings: the tokens' pages and the blocks'")
            cache, pooled = cache
        if cache is None or cache.storage is None:
            raise RuntimeError("normed_attention needs a paged key/value cache binding")
        if not cache.writes:
            raise NotImplementedError("normed_attention keeps a cache of its own: a run entry cannot read another entry's")
        group = ctx.groups[cache.group]
        proj = self.in_proj.forward(x)
        rows = proj.shape[0]
        q = torch.empty((rows, self.q_width), dtype=proj.dtype, device=proj.device)
        across = {}
        if self.value_mix == "first":
            across["leave_values"] = torch.empty((rows, self.num_kv_heads * self.value_dim), dtype=torch.float32,
                                                 device=proj.device)
            ctx.carried["first_values"] = across["leave_values"]
        elif self.value_mix == "mix":
            first = ctx.carried.get("first_values")
            if first is None or first.shape != (rows, self.num_kv_heads * self.value_dim):
                raise RuntimeError("a mixer that mixes values needs an earlier layer's values of the same width in the step")
            across["mix_values"] = (first, self.mix)
        if self.projection_norm is not None:
            kernels.row_norm_rope_cache(proj, q, cache.storage, ctx.positions, ctx.seq_of_row, group.block_table, self.inv_freq,
                                        self.projection_norm, amplitude=self.amplitude, heads=self.num_heads,
                                        kv_heads=self.num_kv_heads, dim=self.key_dim, vdim=self.value_dim,
                                        rot_dims=self.rot_dims, eps=self.projection_norm_eps, page_size=cache.page_size,
                                        values_from_keys=self.values_from_keys)
        else:
            kernels.rope_norm_cache(proj, q, cache.storage, ctx.positions, ctx.seq_of_row, group.block_table, self.inv_freq,
                                    amplitude=self.amplitude, heads=self.num_heads, kv_heads=self.num_kv_heads,
                                    dim=self.key_dim, vdim=self.value_dim, rot_dims=self.rot_dims,
                                    unit_norm=self.unit_norm, eps=self.qk_norm_eps, page_size=cache.page_size,
                                    bias=self.in_bias, **across)
        extras = {"sinks": self.sinks, "softcap": self.softcap, "keep_first": self.keep_first,
                  "distance_bias": self.distance_bias,
                  "head_gate": proj[:, self.gate_offset:self.gate_offset + self.num_heads] if self.head_gated else None}
        if pooled is not None:
            pool_table = ctx.groups[pooled.group].block_table
            kernels.pool_blocks(cache.storage, pooled.storage, ctx.positions, ctx.seq_of_row, group.block_table, pool_table,
                                kv_heads=self.num_kv_heads, dim=self.key_dim, vdim=self.value_dim,
                                page_size=cache.page_size, pool=self.pool)
            extras["pooled"] = (pooled.storage, pool_table, self.pool)
        attended = torch.empty((rows, self.o_width), dtype=proj.dtype, device=proj.device)
        choice = self.attention_choice(rows)
        if choice == "attention_rows_mma":
            kernels.attention_rows_mma(q, attended, cache.storage, ctx.positions, ctx.seq_of_row, group.block_table,
                                       heads=self.num_heads, kv_heads=self.num_kv_heads, dim=self.key_dim,
                                       vdim=self.value_dim, page_size=cache.page_size, mask_kind=_MASKS[self.mask_kind],
                                       mask_size=self.mask_size, scale=self.scale, **extras)
        elif choice == "attention_prompt_mma":
            kernels.attention_prompt_mma(q, attended, cache.storage, ctx.positions, ctx.row_start, group.block_table,
                                         num_seqs=ctx.num_seqs, heads=self.num_heads, kv_heads=self.num_kv_heads,
                                         dim=self.key_dim, vdim=self.value_dim, page_size=cache.page_size,
                                         mask_kind=_MASKS[self.mask_kind], mask_size=self.mask_size, scale=self.scale,
                                         **extras)
        else:
            kernels.attention_masked(q, None, attended, cache.storage, ctx.positions, ctx.seq_of_row, group.block_table,
                                     heads=self.num_heads, kv_heads=self.num_kv_heads, dim=self.key_dim,
                                     vdim=self.value_dim, page_size=cache.page_size, mask_kind=_MASKS[self.mask_kind],
                                     mask_size=self.mask_size, sink=False, scale=self.scale, **extras)
        return self.o_proj.forward(attended, float32_out=self.stream_f32)
