"""Tibivik: configuration -> model description.

A pre-norm decoder over a residual stream kept as ``streams`` 32-bit copies that are mixed around every sublayer
(``hyper_connected`` block with ``hyper_connections``; its norms read a weighted sum of the copies); a run of layers may be walked
several times, each walk with a cache and state of its own.  A token's row is its embedding plus a row for the pair it forms with the
token in front (``bigram_embedding``).  Three mixers: ``state_space`` (Mamba-2), and two kinds of ``parallel_mixers``: ``normed_attention``
over a sliding window whose keys, as projected, are also its values, with a norm over the whole projections, a rotation and a learned
sink, beside ``matrix_memory`` (xLSTM); and ``normed_attention`` within chunks of the sequence, with biases, a learned sink and a gate per
head, beside ``gated_delta`` (the gated delta rule).  The feed-forward is ``gated_mlp`` (SiLU) or absent.  The head is the embedding
table.  Tensor names: ``embed``, ``bigram``, ``final.norm`` and per layer ``l<i>.norm1/2``, ``l<i>.hc1/2.{in,out,mix}``, ``l<i>.mix.*``,
``l<i>.mlp.{gate,up,down}``.
"""

from __future__ import annotations

from ..config.registry import Architecture, register_architecture
from ..config.spec import LayerSpec, ModelSpec, PartSpec, RunEntry
from ..parts.parallel_mixers import ParallelMixers
from .tibivik_config import (TibivikConfig, TibivikDelta, TibivikMemory, TibivikParallel, TibivikStateSpace)

STREAM = "float32"       # the copies of the stream are 32-bit in every run dtype


def _state_space(cfg: TibivikConfig, m: TibivikStateSpace, mix: str) -> PartSpec:
    return PartSpec.make(
        "state_space",
        {"hidden_size": cfg.width, "num_heads": m.heads, "value_dim": m.vdim, "state": m.state, "groups": m.groups,
         "norm_groups": m.norm_groups, "conv_taps": m.taps, "eps": cfg.norm_eps, "stream": STREAM},
        {"in": mix + "in", "conv": mix + "conv", "conv_bias": mix + "conv.b", "dt_bias": mix + "dt_bias", "a_log": mix + "A_log",
         "skip": mix + "D", "norm": mix + "norm", "o": mix + "o"})


def _shared_key_attention(cfg: TibivikConfig, m, mix: str) -> PartSpec:
    position = {}
    if m.rotation is not None:
        position = {"position": PartSpec.make("rotary_blend", {"head_dim": m.dim, "dims": m.rotation.dims,
                                                               "base": m.rotation.base, "scaling": None})}
    return PartSpec.make(
        "normed_attention",
        {"hidden_size": cfg.width, "num_heads": m.heads, "num_kv_heads": m.kv_heads, "key_dim": m.dim, "value_dim": m.vdim,
         "scale": m.scale, "mask": (("kind", "window"), ("size", m.size)), "projection_norm_eps": cfg.norm_eps,
         "values_from_keys": True, "sink": True, "stream": STREAM},
        {"q": mix + "q", "k": mix + "k", "q_norm": mix + "q.norm", "k_norm": mix + "k.norm", "sink": mix + "sink", "o": mix + "o"},
        position)


def _chunk_attention(cfg: TibivikConfig, m, mix: str) -> PartSpec:
    return PartSpec.make(
        "normed_attention",
        {"hidden_size": cfg.width, "num_heads": m.heads, "num_kv_heads": m.kv_heads, "key_dim": m.dim, "value_dim": m.vdim,
         "scale": m.scale, "mask": (("kind", "blocks"), ("size", m.size)), "bias": True, "sink": True, "head_gate": True,
         "stream": STREAM},
        {"q": mix + "q", "k": mix + "k", "v": mix + "v", "q_bias": mix + "q.b", "k_bias": mix + "k.b", "v_bias": mix + "v.b",
         "sink": mix + "sink", "g": mix + "g", "o": mix + "o"})


def _matrix_memory(cfg: TibivikConfig, m: TibivikMemory, mix: str) -> PartSpec:
    return PartSpec.make(
        "matrix_memory",
        {"hidden_size": cfg.width, "num_heads": m.heads, "key_dim": m.dim, "value_dim": m.vdim, "gate_cap": m.gate_cap,
         "eps": cfg.norm_eps, "stream": STREAM},
        {"q": mix + "q", "k": mix + "k", "v": mix + "v", "g": mix + "g", "i": mix + "i", "i_bias": mix + "i.b", "f": mix + "f",
         "f_bias": mix + "f.b", "norm": mix + "norm", "o": mix + "o"})


def _gated_delta(cfg: TibivikConfig, m: TibivikDelta, mix: str) -> PartSpec:
    return PartSpec.make(
        "gated_delta",
        {"hidden_size": cfg.width, "num_heads": m.heads, "num_kv_heads": m.kv_heads, "key_dim": m.dim, "value_dim": m.vdim,
         "conv_taps": m.taps, "eps": cfg.norm_eps, "stream": STREAM},
        {"q": mix + "q", "k": mix + "k", "v": mix + "v", "g": mix + "g", "q_conv": mix + "q.conv", "k_conv": mix + "k.conv",
         "v_conv": mix + "v.conv", "a": mix + "a", "b": mix + "b", "a_log": mix + "A_log", "dt_bias": mix + "dt_bias",
         "norm": mix + "norm", "o": mix + "o"})


def _mixer(cfg: TibivikConfig, m, mix: str) -> PartSpec:
    if isinstance(m, TibivikStateSpace):
        return _state_space(cfg, m, mix)
    assert isinstance(m, TibivikParallel)
    if isinstance(m.right, TibivikMemory):
        children = {"left": _shared_key_attention(cfg, m.left, mix + "left."), "right": _matrix_memory(cfg, m.right, mix + "right.")}
    else:
        children = {"left": _chunk_attention(cfg, m.left, mix + "left."), "right": _gated_delta(cfg, m.right, mix + "right.")}
    return PartSpec.make("parallel_mixers", {"hidden_size": cfg.width, "left_scale": m.left_scale, "right_scale": m.right_scale},
                         ParallelMixers.lifted_weights(children), children)


def tibivik_spec(cfg: TibivikConfig) -> ModelSpec:
    def norm(weight: str, **more: str) -> PartSpec:
        return PartSpec.make("mixed_streams_rms_norm", {"size": cfg.width, "streams": cfg.streams, "eps": cfg.norm_eps},
                             dict(more, weight=weight))

    layers = []
    for index, layer in enumerate(cfg.layers):
        prefix = f"l{index}."
        norms = {"input": norm(prefix + "norm1", take=prefix + "hc1.in")}
        mixing = {"mixer_mix": prefix + "hc1.mix", "mixer_out": prefix + "hc1.out"}
        feed_forward = None
        if layer.ff is not None:
            feed_forward = PartSpec.make("gated_mlp", {"hidden_size": cfg.width, "intermediate_size": layer.ff, "activation": "silu",
                                                       "bias": False, "stream": STREAM},
                                         {role: f"{prefix}mlp.{role}" for role in ("gate", "up", "down")})
            norms["post_mixer"] = norm(prefix + "norm2", take=prefix + "hc2.in")
            mixing.update({"feed_forward_mix": prefix + "hc2.mix", "feed_forward_out": prefix + "hc2.out"})
        stream_mixing = PartSpec.make("hyper_connections", {"streams": cfg.streams, "feed_forward": layer.ff is not None}, mixing)
        layers.append(LayerSpec.make("hyper_connected", _mixer(cfg, layer.mixer, prefix + "mix."), feed_forward, norms,
                                     stream_mixing=stream_mixing))
    sizes = {"vocab_size": cfg.vocab, "hidden_size": cfg.width}
    return ModelSpec(
        architecture=TibivikConfig.ARCHITECTURE,
        hidden_size=cfg.width,
        vocab_size=cfg.vocab,
        max_positions=1 << 30,           # the design sets no limit; positions are 32-bit
        embedding=PartSpec.make("bigram_embedding", dict(sizes, buckets=cfg.buckets, mul_prev=cfg.mul_prev, mul_cur=cfg.mul_cur,
                                                         copies=cfg.streams), {"table": "embed", "pairs": "bigram"}),
        layers=tuple(layers),
        run_order=tuple(RunEntry(index) for index in cfg.run_order()),
        final_norm=norm("final.norm"),
        head=PartSpec.make("lm_head", sizes, {"weight": "embed"}),
    )


def tibivik_ignorable_tensors(cfg: TibivikConfig):
    """Tensors a checkpoint may hold that this model does not read: what belongs to the feed-forward of a layer without
    one."""
    names = []
    for index, layer in enumerate(cfg.layers):
        if layer.ff is None:
            names += [f"l{index}.norm2", f"l{index}.hc2.in", f"l{index}.hc2.out", f"l{index}.hc2.mix"]
    return names


def tibivik_kernel_libraries(cfg: TibivikConfig, dtype: str):
    """The kernel files a Tibivik model of this run dtype calls: a first call compiles these and no others."""
    shared = ["elementwise", "hyper_streams", "matrix_recurrence", "sampling"]
    pairs = [layer.mixer for layer in cfg.layers if isinstance(layer.mixer, TibivikParallel)]
    if any(layer.ff is not None for layer in cfg.layers):
        shared.append("pointwise")
    if pairs:
        shared += ["rope_norm_cache", "attention_masked"]
    if any(isinstance(layer.mixer, TibivikStateSpace) for layer in cfg.layers) or any(isinstance(m.right, TibivikDelta) for m in pairs):
        shared.append("short_conv")
    if dtype != "float32":
        import torch

        from .. import kernels

        if any(kernels.attention_prompt_mma_supported(torch.bfloat16, m.left.dim, m.left.vdim) for m in pairs):
            shared.append("attention_prompt_mma")     # (head sizes the tensor-core attention takes)
    return shared + (["gemm_f32"] if dtype == "float32" else ["decode_linear", "skinny_tcgen05"])


register_architecture(Architecture(
    name=TibivikConfig.ARCHITECTURE,
    read_config=TibivikConfig.from_dict,
    build_spec=tibivik_spec,
    ignorable_tensors=tibivik_ignorable_tensors,
    kernel_libraries=tibivik_kernel_libraries,
))
