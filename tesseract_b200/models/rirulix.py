"""Rirulix: configuration -> model description.

A decoder over a 32-bit stream whose layers are listed one by one and whose sublayers are normed on both sides
(``sandwich`` block; every norm of the model is ``grouped_rms_norm`` over ``norm.groups`` parts of the row).  The stream starts
from a token's row plus a learned row for its position, normed (``positioned_embedding``).  Two mixers: ``normed_attention``
without a norm of queries and keys or a rotation (biases on all four projections, a sliding window that keeps the first
tokens, a learned distance bias per head, values mixed with the first such layer's) and ``rglru`` (a real-gated linear
recurrent unit behind a short convolution, gated by a second branch).  The feed-forward is ``routed_experts`` (sigmoid
scores that weigh the experts' inputs, clamped gated experts, a gated shared expert) or absent.  The head is a matrix of
its own.  Tensor names: ``embed``, ``pos``, ``embed.norm``, ``head``, ``final.norm`` and per layer ``l<i>.norm{1,1b,2,2b}``,
``l<i>.mix.*``, ``l<i>.mlp.*``.
"""

from __future__ import annotations

from ..config.registry import Architecture, register_architecture
from ..config.spec import LayerSpec, ModelSpec, PartSpec, RunEntry
from .rirulix_config import RirulixAttention, RirulixConfig, RirulixExperts, RirulixRecurrence

STREAM = "float32"       # the residual sum is 32-bit in every run dtype
GATE_SLOPE = 1.702       # an expert's gate is g * sigmoid(1.702 g)


def _attention(cfg: RirulixConfig, index: int, m: RirulixAttention, mix: str) -> PartSpec:
    weights = {"q": mix + "q", "k": mix + "k", "v": mix + "v", "o": mix + "o", "q_bias": mix + "q.b", "k_bias": mix + "k.b",
               "v_bias": mix + "v.b", "o_bias": mix + "o.b", "distance_weight": mix + "r1", "distance_rate": mix + "r2"}
    value_mix = None
    if m.v_mix:
        value_mix = "first" if index == cfg.first_mixing_layer() else "mix"
    if value_mix == "mix":
        weights["value_mix"] = mix + "vmix"
    return PartSpec.make(
        "normed_attention",
        {"hidden_size": cfg.width, "num_heads": m.heads, "num_kv_heads": m.kv_heads, "key_dim": m.dim, "value_dim": m.vdim,
         "scale": m.scale, "mask": (("keep_first", m.keep_first), ("kind", "window"), ("size", m.window)), "bias": True,
         "output_bias": True, "distance_bias": True, "value_mix": value_mix, "stream": STREAM},
        weights)


def _recurrence(cfg: RirulixConfig, m: RirulixRecurrence, mix: str) -> PartSpec:
    return PartSpec.make(
        "rglru", {"hidden_size": cfg.width, "width": m.width, "blocks": m.blocks, "conv_taps": m.taps, "stream": STREAM},
        {"y": mix + "y", "y_bias": mix + "y.b", "x": mix + "x", "x_bias": mix + "x.b", "conv": mix + "conv",
         "conv_bias": mix + "conv.b", "r": mix + "ra", "r_bias": mix + "ra.b", "i": mix + "ri", "i_bias": mix + "ri.b",
         "decay": mix + "lam", "o": mix + "o"})


def _experts(cfg: RirulixConfig, mlp: RirulixExperts, prefix: str) -> PartSpec:
    weights = {"router": prefix + "router"}
    for e in range(mlp.experts):
        weights.update({f"gate.{e}": f"{prefix}e{e}.gate", f"up.{e}": f"{prefix}e{e}.up", f"down.{e}": f"{prefix}e{e}.down"})
    if mlp.shared_ff:
        weights.update({"shared_gate": prefix + "shared.gate", "shared_up": prefix + "shared.up",
                        "shared_down": prefix + "shared.down", "shared_weight": prefix + "shared.sg"})
    return PartSpec.make(
        "routed_experts",
        {"hidden_size": cfg.width, "num_experts": mlp.experts, "top_k": mlp.top, "expert_size": mlp.ff,
         "shared_size": mlp.shared_ff, "scoring": "sigmoid", "weigh": "input", "expert_form": "gated_clamped",
         "limit": mlp.limit, "shared_limit": mlp.shared_limit, "slope": GATE_SLOPE, "gated_shared": mlp.shared_ff is not None,
         "stream": STREAM},
        weights)


def rirulix_spec(cfg: RirulixConfig) -> ModelSpec:
    def norm(name: str) -> PartSpec:
        return PartSpec.make("grouped_rms_norm", {"size": cfg.width, "groups": cfg.norm_groups, "eps": cfg.norm_eps},
                             {"weight": name})

    layers = []
    for index, layer in enumerate(cfg.layers):
        prefix = f"l{index}."
        if isinstance(layer.mixer, RirulixAttention):
            mixer = _attention(cfg, index, layer.mixer, prefix + "mix.")
        else:
            mixer = _recurrence(cfg, layer.mixer, prefix + "mix.")
        norms = {"pre_mixer": norm(prefix + "norm1"), "post_mixer": norm(prefix + "norm1b")}
        feed_forward = None
        if layer.mlp is not None:
            feed_forward = _experts(cfg, layer.mlp, prefix + "mlp.")
            norms.update({"pre_feed_forward": norm(prefix + "norm2"), "post_feed_forward": norm(prefix + "norm2b")})
        layers.append(LayerSpec.make("sandwich", mixer, feed_forward, norms))
    sizes = {"vocab_size": cfg.vocab, "hidden_size": cfg.width}
    return ModelSpec(
        architecture=RirulixConfig.ARCHITECTURE,
        hidden_size=cfg.width,
        vocab_size=cfg.vocab,
        max_positions=cfg.max_positions,
        embedding=PartSpec.make("positioned_embedding", dict(sizes, max_positions=cfg.max_positions, groups=cfg.norm_groups,
                                                             eps=cfg.norm_eps),
                                {"table": "embed", "positions": "pos", "weight": "embed.norm"}),
        layers=tuple(layers),
        run_order=tuple(RunEntry(index) for index in range(len(layers))),
        final_norm=norm("final.norm"),
        head=PartSpec.make("lm_head", sizes, {"weight": "head"}),
    )


def rirulix_ignorable_tensors(cfg: RirulixConfig):
    """Tensors a checkpoint may hold that this model does not read: the mixing number of an attention layer that mixes
    nothing (the first one with ``v_mix`` among them) and the feed-forward's norms of a layer without one."""
    names = []
    for index, layer in enumerate(cfg.layers):
        if isinstance(layer.mixer, RirulixAttention) and (not layer.mixer.v_mix or index == cfg.first_mixing_layer()):
            names.append(f"l{index}.mix.vmix")
        if layer.mlp is None:
            names += [f"l{index}.norm2", f"l{index}.norm2b"]
    return names


def rirulix_kernel_libraries(cfg: RirulixConfig, dtype: str):
    """The kernel files a Rirulix model of this run dtype calls: a first call compiles these and no others."""
    shared = ["elementwise", "norm", "sandwich_norm", "pointwise", "sampling"]
    attentions = [layer.mixer for layer in cfg.layers if isinstance(layer.mixer, RirulixAttention)]
    if attentions:
        shared += ["rope_norm_cache", "attention_masked"]
    if any(isinstance(layer.mixer, RirulixRecurrence) for layer in cfg.layers):
        shared += ["short_conv", "rglru"]
    if any(layer.mlp is not None for layer in cfg.layers):
        shared.append("experts")
    if dtype != "float32":
        import torch

        from .. import kernels

        if any(kernels.attention_prompt_mma_supported(torch.bfloat16, m.dim, m.vdim) for m in attentions):
            shared.append("attention_prompt_mma")     # (head sizes the tensor-core attention takes)
    return shared + (["gemm_f32"] if dtype == "float32" else ["decode_linear", "skinny_tcgen05"])


register_architecture(Architecture(
    name=RirulixConfig.ARCHITECTURE,
    read_config=RirulixConfig.from_dict,
    build_spec=rirulix_spec,
    ignorable_tensors=rirulix_ignorable_tensors,
    kernel_libraries=rirulix_kernel_libraries,
))
