"""A plain, slow Tibivik in float64: whole sequences, one function per mechanism, nothing shared with the package.

``forward(config, tensors, tokens)`` takes the dictionary of ``config.json``, a mapping from tensor name to a numpy
array, and one sequence's token ids; it returns the logits of every position and the stream (the sum of its copies) behind
every layer run.  ``store`` is applied wherever a serving path may keep numbers in 16 bits between two of its kernels
(normed rows, projected rows, convolved rows, cached keys and values, what enters an output product); the default keeps
float64, and ``bfloat16`` measures what such rounding alone does to a result.
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
    kinds = {"BF16": torch.bfloat16, "F32": torch.float32, "F16": torch.float16, "I32": torch.int32}
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


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, z)


def log_sigmoid(z):
    return -np.logaddexp(0.0, -z)


def over_rms(x, eps):
    """``x`` over its root mean square along the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def bigram_rows(config, tokens):
    """Which row of the pair table every token adds: a hash of the token in front and the token, or the row behind all
    buckets for a token with none in front."""
    b = config["embedding"]["bigram"]
    rows = [b["buckets"]]
    for before, token in zip(tokens[:-1], tokens[1:]):
        rows.append((int(before) * b["mul_prev"] + int(token) * b["mul_cur"]) % b["buckets"])
    return rows


def embed(config, tensors, tokens):
    return tensors["embed"][np.asarray(tokens)] + tensors["bigram"][bigram_rows(config, list(tokens))]


# ----------------------------------------------------------------------------- attention


def rotate_halves(x, dims, base, first=0):
    """Number ``i`` turns with number ``i + dims / 2`` by ``p * base^(-2i / dims)``; ``x`` ``[T, heads, d]``, row 0 at
    position ``first``."""
    half = dims // 2
    p = first + np.arange(x.shape[0])
    angle = p[:, None] * np.array([base ** (-2.0 * i / dims) for i in range(half)])[None, :]
    c, s = np.cos(angle)[:, None, :], np.sin(angle)[:, None, :]
    u, v = x[..., :half], x[..., half:dims]
    return np.concatenate([u * c - v * s, v * c + u * s, x[..., dims:]], axis=-1)


def window_mask(T, size):
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    return (j <= i) & (i - j < size)


def chunk_mask(T, size):
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    return (j <= i) & (i // size == j // size)


def attend(q, k, v, seen, scale, sinks):
    """``[T, H, d]`` queries over ``[T, G, d]`` keys and ``[T, G, dv]`` values; ``sinks[h]`` is one more logit of head ``h``'s
    softmax that carries nothing."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    out = np.zeros((T, H, v.shape[2]))
    for head in range(H):
        g = head // (H // G)
        scores = np.where(seen, (q[:, head] @ k[:, g].T) * scale, -np.inf)
        top = np.maximum(scores.max(axis=1, keepdims=True), sinks[head])
        weights = np.exp(scores - top)
        out[:, head] = (weights / (weights.sum(axis=1, keepdims=True) + np.exp(sinks[head] - top))) @ v[:, g]
    return out


def shared_kv_attention(m, w, h, eps, store=identity):
    """A window over keys whose projection, before its norm and rotation, is also the value."""
    T = h.shape[0]
    H, G, d = m["heads"], m["kv_heads"], m["dim"]
    raw_q, raw_k = store(h @ w["q"].T), store(h @ w["k"].T)
    q = (over_rms(raw_q, eps) * w["q.norm"]).reshape(T, H, d)
    k = (over_rms(raw_k, eps) * w["k.norm"]).reshape(T, G, d)
    rot = m.get("rot")
    if rot:
        q, k = rotate_halves(q, rot["dims"], rot["base"]), rotate_halves(k, rot["dims"], rot["base"])
    out = attend(store(q), store(k), raw_k.reshape(T, G, d), window_mask(T, m["mask"]["size"]), m["scale"], w["sink"])
    return store(out.reshape(T, -1)) @ w["o"].T


def chunk_attention(m, w, h, store=identity):
    """Within chunks of the sequence, biased projections, a gate per head on the output."""
    T = h.shape[0]
    H, G = m["heads"], m["kv_heads"]
    q = store(store(h @ w["q"].T) + w["q.b"]).reshape(T, H, -1)
    k = store(store(h @ w["k"].T) + w["k.b"]).reshape(T, G, -1)
    v = store(store(h @ w["v"].T) + w["v.b"]).reshape(T, G, -1)
    out = attend(q, k, v, chunk_mask(T, m["mask"]["size"]), m["scale"], w["sink"])
    out = out * sigmoid(h @ w["g"].T)[:, :, None]
    return store(out.reshape(T, -1)) @ w["o"].T


# ----------------------------------------------------------------------------- recurrences


def causal_convolution(u, taps, bias=0.0):
    """``y[t, c] = bias[c] + sum_j taps[c, j] u[t - J + 1 + j, c]``, zeros in front of the first row."""
    T, J = u.shape[0], taps.shape[1]
    padded = np.concatenate([np.zeros((J - 1, u.shape[1])), u])
    return sum(padded[j:j + T] * taps[:, j] for j in range(J)) + bias


def matrix_memory(q, k, v, log_i, log_f, state=None):
    """``q, k`` ``[T, H, d]``, ``v`` ``[T, H, dv]``, gates ``[T, H]``; ``(outputs, last (S, n, m))``."""
    T, H, d = q.shape
    S, n, m = (np.zeros((H, d, v.shape[2])), np.zeros((H, d)), np.zeros(H)) if state is None else [a.copy() for a in state]
    out = np.empty(v.shape)
    for t in range(T):
        new = np.maximum(log_f[t] + m, log_i[t])
        keep, write = np.exp(log_f[t] + m - new), np.exp(log_i[t] - new)
        m = new
        S = keep[:, None, None] * S + write[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + write[:, None] * k[t]
        weight = np.maximum(np.abs(np.sum(n * q[t], axis=1)), np.exp(-m)) + 1e-6
        out[t] = np.einsum("hdv,hd->hv", S, q[t]) / weight[:, None]
    return out, (S, n, m)


def mlstm(m, w, h, eps, store=identity):
    T = h.shape[0]
    H, d, cap = m["heads"], m["dim"], m["gate_cap"]
    q = store(h @ w["q"].T).reshape(T, H, d) * d ** -0.5
    k = store(h @ w["k"].T).reshape(T, H, d)
    v = store(h @ w["v"].T).reshape(T, H, -1)
    log_i = cap * np.tanh((h @ w["i"].T + w["i.b"]) / cap)
    log_f = log_sigmoid(cap * np.tanh((h @ w["f"].T + w["f.b"]) / cap))
    o, _ = matrix_memory(q, k, v, log_i, log_f)
    rows = over_rms(o, eps).reshape(T, -1) * w["norm"] * sigmoid(store(h @ w["g"].T))
    return store(rows) @ w["o"].T


def gated_delta(q, k, v, beta, decay, state=None):
    """``q, k`` ``[T, H, d]`` (a copy per head), ``v`` ``[T, H, dv]``, ``beta`` and ``decay`` ``[T, H]``; ``(outputs, last S)``."""
    T, H, d = q.shape
    S = np.zeros((H, d, v.shape[2])) if state is None else state.copy()
    out = np.empty(v.shape)
    for t in range(T):
        S = decay[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - np.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out[t] = np.einsum("hdv,hd->hv", S, q[t])
    return out, S


def unit(x):
    return x / np.sqrt(np.sum(x * x, axis=-1, keepdims=True) + 1e-6)


def delta_mixer(m, w, h, eps, store=identity):
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (store(silu(causal_convolution(store(h @ w[name].T), w[name + ".conv"]))) for name in "qkv")
    q = np.repeat(unit(q.reshape(T, G, d)) * d ** -0.5, H // G, axis=1)
    k = np.repeat(unit(k.reshape(T, G, d)), H // G, axis=1)
    beta = sigmoid(h @ w["b"].T)
    decay = np.exp(-np.exp(w["A_log"]) * softplus(h @ w["a"].T + w["dt_bias"]))
    o, _ = gated_delta(q, k, v.reshape(T, H, dv), beta, decay)
    rows = (over_rms(o, eps) * w["norm"]).reshape(T, -1) * silu(store(h @ w["g"].T))
    return store(rows) @ w["o"].T


def state_space(x, B, C, dt, A_log, D, state=None):
    """``x`` ``[T, H, dv]``, ``B, C`` ``[T, H, N]`` (a copy per head), ``dt`` ``[T, H]``; ``(outputs, last S)``."""
    T, H, dv = x.shape
    S = np.zeros((H, B.shape[2], dv)) if state is None else state.copy()
    out = np.empty(x.shape)
    for t in range(T):
        keep = np.exp(-np.exp(A_log) * dt[t])
        S = keep[:, None, None] * S + (dt[t][:, None] * B[t])[:, :, None] * x[t][:, None, :]
        out[t] = np.einsum("hnv,hn->hv", S, C[t]) + D[:, None] * x[t]
    return out, S


def mamba2(m, w, h, eps, store=identity):
    T = h.shape[0]
    H, dv, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * dv
    rows = h @ w["in"].T
    z, xbc, dt = store(rows[:, :inner]), store(rows[:, inner:2 * inner + 2 * G * N]), rows[:, 2 * inner + 2 * G * N:]
    xbc = store(silu(causal_convolution(xbc, w["conv"], w["conv.b"])))
    x = xbc[:, :inner].reshape(T, H, dv)
    B = np.repeat(xbc[:, inner:inner + G * N].reshape(T, G, N), H // G, axis=1)
    C = np.repeat(xbc[:, inner + G * N:].reshape(T, G, N), H // G, axis=1)
    y, _ = state_space(x, B, C, softplus(dt + w["dt_bias"]), w["A_log"], w["D"])
    gated = (y.reshape(T, inner) * silu(z)).reshape(T, m["norm_groups"], -1)
    return store(over_rms(gated, eps).reshape(T, inner) * w["norm"]) @ w["o"].T


# ----------------------------------------------------------------------------- layers


def side(w, name):
    return {key[len(name) + 1:]: a for key, a in w.items() if key.startswith(name + ".")}


def mixer_forward(kind, m, w, h, eps, store=identity):
    if kind == "mamba2":
        return mamba2(m, w, h, eps, store)
    if kind == "parallel":
        left = shared_kv_attention(m["left"], side(w, "left"), h, eps, store)
        right = mlstm(m["right"], side(w, "right"), h, eps, store)
    elif kind == "parallel_2":
        left = chunk_attention(m["left"], side(w, "left"), h, store)
        right = delta_mixer(m["right"], side(w, "right"), h, eps, store)
    else:
        raise ValueError(kind)
    return m["left_scale"] * left + m["right_scale"] * right


def gated_feed_forward(w, h, store=identity):
    return store(silu(store(h @ w["gate"].T)) * store(h @ w["up"].T)) @ w["down"].T


def connect(streams, w, q, sublayer):
    """One sublayer over ``[s, T, width]`` copies of the stream: it reads a weighted sum of them, and every copy becomes a
    weighted sum of the old copies plus its share of the result."""
    u = np.einsum("s,stw->tw", w[f"hc{q}.in"], streams)
    y = sublayer(u)
    return np.einsum("sr,stw->rtw", w[f"hc{q}.mix"], streams) + w[f"hc{q}.out"][:, None, None] * y[None]


def layer_forward(config, tensors, index, streams, store=identity):
    layer, prefix, eps = config["layers"][index], f"l{index}.", config["norm"]["eps"]
    w = {name[len(prefix):]: a for name, a in tensors.items() if name.startswith(prefix)}
    streams = connect(streams, w, 1, lambda u: mixer_forward(
        layer["type"], layer["mixer"], side(w, "mix"), store(over_rms(u, eps) * w["norm1"]), eps, store))
    if layer.get("mlp") is not None:
        streams = connect(streams, w, 2, lambda u: gated_feed_forward(
            side(w, "mlp"), store(over_rms(u, eps) * w["norm2"]), store))
    return streams


def run_order(config):
    """Layer indices in the order they run."""
    count, loop = len(config["layers"]), config.get("loop")
    if not loop:
        return list(range(count))
    looped = list(range(loop["start"], loop["stop"]))
    return list(range(loop["start"])) + looped * loop["times"] + list(range(loop["stop"], count))


def forward(config, tensors, tokens, store=identity):
    """``(logits [T, vocab], [stream behind every layer run])``."""
    x = embed(config, tensors, tokens)
    streams = np.repeat(x[None], config["streams"], axis=0)
    runs = []
    for index in run_order(config):
        streams = layer_forward(config, tensors, index, streams, store)
        runs.append(streams.sum(axis=0))
    last = over_rms(runs[-1], config["norm"]["eps"]) * tensors["final.norm"]
    return store(last) @ tensors["embed"].T, runs
