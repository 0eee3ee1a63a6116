"""A plain, slow Rirulix in float64: whole sequences, one function per mechanism, nothing shared with the package.

``forward(config, tensors, tokens)`` takes the dictionary of ``config.json``, a mapping from tensor name to a numpy
array, and one sequence's token ids; it returns the logits of every position and the stream behind every layer.
``store`` is applied wherever a serving path may keep numbers in 16 bits between two of its kernels (normed rows,
projected rows, cached keys and values, what enters an output product); the default keeps float64, and ``bfloat16``
measures what such rounding alone does to a result.
"""

from __future__ import annotations

import math

import numpy as np


def identity(x):
    return x


def bfloat16(x):
    """``x`` rounded to bfloat16 and widened again."""
    import torch

    return torch.from_numpy(np.ascontiguousarray(x, dtype=np.float64)).to(torch.bfloat16).to(torch.float64).numpy()


def load_folder(folder):
    """``(config, {name: float64 array})`` of a model folder, read with a parser of its own."""
    import json
    import os
    import struct

    import torch

    with open(os.path.join(folder, "config.json")) as handle:
        config = json.load(handle)
    raw = open(os.path.join(folder, "model.safetensors"), "rb").read()
    (size,) = struct.unpack("<Q", raw[:8])
    header = json.loads(raw[8:8 + size])
    kinds = {"BF16": torch.bfloat16, "F32": torch.float32, "F16": torch.float16}
    tensors = {}
    for name, entry in header.items():
        if name == "__metadata__":
            continue
        first, last = entry["data_offsets"]
        flat = torch.frombuffer(bytearray(raw[8 + size + first:8 + size + last]), dtype=kinds[entry["dtype"]])
        tensors[name] = flat.to(torch.float64).numpy().reshape(entry["shape"])
    return config, tensors


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def softplus(z):
    return np.logaddexp(0.0, z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def grouped_rms_norm(x, weight, groups, eps):
    """Every row in ``groups`` equal consecutive parts, each over its own root mean square; the whole times ``weight``."""
    parts = x.reshape(x.shape[0], groups, -1)
    return (parts / np.sqrt(np.mean(parts * parts, axis=-1, keepdims=True) + eps)).reshape(x.shape) * weight


def embed(config, tensors, tokens):
    tokens = np.asarray(tokens)
    x = tensors["embed"][tokens] + tensors["pos"][np.arange(len(tokens))]
    return grouped_rms_norm(x, tensors["embed.norm"], config["norm"]["groups"], config["norm"]["eps"])


# ----------------------------------------------------------------------------- mixers


def causal_convolution(u, taps, bias):
    """``y[t, c] = bias[c] + sum_j taps[c, j] u[t - J + 1 + j, c]``, zeros in front of the first row."""
    T, J = u.shape[0], taps.shape[1]
    padded = np.concatenate([np.zeros((J - 1, u.shape[1])), u])
    return sum(padded[j:j + T] * taps[:, j] for j in range(J)) + bias


def recurrence_gates(w, u, blocks):
    """``(r, i)`` of every row: per block of channels a square matrix and a bias each, through a sigmoid."""
    size = u.shape[1] // blocks
    r, i = np.empty_like(u), np.empty_like(u)
    for b in range(blocks):
        part = slice(b * size, (b + 1) * size)
        r[:, part] = sigmoid(u[:, part] @ w["ra"][b].T + w["ra.b"][b])
        i[:, part] = sigmoid(u[:, part] @ w["ri"][b].T + w["ri.b"][b])
    return r, i


def gated_linear_recurrence(u, r, i, lam, state=None):
    """``S_t = a_t S_(t-1) + sqrt(1 - a_t^2) i_t u_t`` with ``log a_t = -8 r_t softplus(lam)``; ``(all S, last S)``."""
    log_a = -8.0 * r * softplus(lam)
    a, enters = np.exp(log_a), np.sqrt(-np.expm1(2.0 * log_a)) * i * u
    S = np.zeros(u.shape[1]) if state is None else state.copy()
    out = np.empty_like(u)
    for t in range(u.shape[0]):
        S = a[t] * S + enters[t]
        out[t] = S
    return out, S


def rglru(m, w, h, store=identity):
    """``m``: the mixer's entry of the configuration; ``w``: name -> array with the layer's ``mix.`` prefix removed."""
    y = gelu_tanh(store(h @ w["y"].T) + w["y.b"])
    u = store(causal_convolution(store(h @ w["x"].T) + w["x.b"], w["conv"], w["conv.b"]))
    r, i = recurrence_gates(w, u, m["blocks"])
    S, _ = gated_linear_recurrence(u, r, i, w["lam"])
    return store(S * y) @ w["o"].T


def attention(m, w, h, first_values=None, store=identity):
    """``(output, values before any mixing)``.  ``first_values`` ``[T, G * dv]``: mixed into this layer's values."""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    size, kept = m["mask"]["size"], m["mask"].get("keep_first", 0)
    q = store(store(h @ w["q"].T) + w["q.b"]).reshape(T, H, d)
    k = store(store(h @ w["k"].T) + w["k.b"]).reshape(T, G, d)
    own = store(h @ w["v"].T) + w["v.b"]
    v = own if first_values is None else (1.0 - w["vmix"]) * own + w["vmix"] * first_values
    v = store(v).reshape(T, G, dv)
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    seen = (j <= i) & ((i - j < size) | (j < kept))
    distance = np.maximum(i - j, 0)
    out = np.zeros((T, H, dv))
    for head in range(H):
        g = head // (H // G)
        scores = (q[:, head] @ k[:, g].T) * m["scale"] - w["r1"][head] * np.log1p(w["r2"][head] * distance)
        scores = np.where(seen, scores, -np.inf)
        weights = np.exp(scores - scores.max(axis=1, keepdims=True))
        out[:, head] = (weights / weights.sum(axis=1, keepdims=True)) @ v[:, g]
    return store(out.reshape(T, H * dv)) @ w["o"].T + w["o.b"], own


# ----------------------------------------------------------------------------- feed-forward


def clamped_expert(w, prefix, h, limit, store=identity):
    g = np.minimum(store(h @ w[prefix + "gate"].T), limit)
    u = np.clip(store(h @ w[prefix + "up"].T), -limit, limit)
    return store(g * sigmoid(1.702 * g) * (u + 1.0)) @ w[prefix + "down"].T


def route(router, logits, gaps=None):
    """``(chosen experts, weights)`` of one row.  ``gaps`` (a list) receives how far, in logits, the last chosen expert was
    from the best one not chosen."""
    scores = sigmoid(logits)
    ranked = sorted(range(router["experts"]), key=lambda e: (-logits[e], e))
    chosen = ranked[:router["top"]]
    if gaps is not None and router["top"] < router["experts"]:
        gaps.append(logits[chosen[-1]] - logits[ranked[router["top"]]])
    return chosen, scores[chosen]


def expert_feed_forward(mlp, w, h, store=identity, close_calls=None):
    """Every chosen expert reads the row times its weight.  ``close_calls`` (a dictionary) receives, per row, the smallest
    gap of its routing decision (see :func:`route`)."""
    out = np.zeros((h.shape[0], w["e0.down"].shape[0]))
    logits = h @ w["router"].T
    for t in range(h.shape[0]):
        gaps = []
        chosen, weights = route(mlp["router"], logits[t], gaps)
        if close_calls is not None and gaps:
            close_calls[t] = min(close_calls.get(t, math.inf), min(gaps))
        for e, weight in zip(chosen, weights):
            out[t] += clamped_expert(w, f"e{e}.", weight * h[t:t + 1], mlp["expert"]["limit"], store)[0]
    if mlp.get("shared"):
        out += clamped_expert(w, "shared.", h, mlp["shared"]["limit"], store) * sigmoid(h @ w["shared.sg"].T)
    return out


# ----------------------------------------------------------------------------- the model


def layer_forward(config, tensors, index, x, first_values, store=identity, close_calls=None):
    """``(stream behind the layer, values that later layers mix in)``; ``first_values`` is None up to the first layer
    that keeps some."""
    layer, prefix = config["layers"][index], f"l{index}."
    w = {name[len(prefix):]: a for name, a in tensors.items() if name.startswith(prefix)}
    mix = {name[4:]: a for name, a in w.items() if name.startswith("mix.")}

    def norm(name, rows):
        return grouped_rms_norm(rows, w[name], config["norm"]["groups"], config["norm"]["eps"])

    h = store(norm("norm1", x))
    if layer["type"] == "rglru":
        mixed = rglru(layer["mixer"], mix, h, store)
    elif layer["type"] == "attention":
        mixes = bool(layer["mixer"].get("v_mix"))
        mixed, own = attention(layer["mixer"], mix, h, first_values if mixes else None, store)
        if mixes and first_values is None:
            first_values = own
    else:
        raise ValueError(layer["type"])
    x = x + norm("norm1b", mixed)
    mlp = layer.get("mlp")
    if mlp is not None:
        h = store(norm("norm2", x))
        feed = {name[4:]: a for name, a in w.items() if name.startswith("mlp.")}
        x = x + norm("norm2b", expert_feed_forward(mlp, feed, h, store, close_calls))
    return x, first_values


def forward(config, tensors, tokens, store=identity, close_calls=None):
    """``(logits [T, vocab], [stream behind layer 0, 1, ...])``.  ``close_calls`` (a dictionary) receives, per position, the
    smallest gap by which a router of any layer decided."""
    x, first_values, streams = embed(config, tensors, tokens), None, []
    for index in range(len(config["layers"])):
        x, first_values = layer_forward(config, tensors, index, x, first_values, store, close_calls)
        streams.append(x.copy())
    last = grouped_rms_norm(x, tensors["final.norm"], config["norm"]["groups"], config["norm"]["eps"])
    return store(last) @ tensors["head"].T, streams
