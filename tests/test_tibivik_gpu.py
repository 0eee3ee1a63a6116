"""Tibivik on the GPU against the plain implementation (``tests/plain/tibivik.py``).

First every mechanism alone (its kernel or part against the plain function, with inputs made so that a fault shows: one key
that dominates, at a window's or a chunk's first position and one before it, at page borders; sinks that take most of a softmax;
a recurrence that remembers one token over hundreds of steps; slots that held another request), then whole tiny models with
random weights under every way of cutting the work: whole prompts, token-by-token decoding, portions down to two tokens, mixed
batches with slots and pages used again, long decoding while windows and chunks move over decoded tokens, and greedy
generation through the package's own entry point and scheduler.
"""

import numpy as np
import pytest
import torch

from tests.helpers import (GREEDY_MARGIN, max_live_tokens, random_tokens, replay, trace_mixed, trace_portions,
                           trace_tail, trace_whole)
from tests.plain import tibivik as plain
from tests.tibivik_models import LENGTHS, TINY_TIBIVIK, random_config

pytestmark = pytest.mark.gpu

REL = {"float32": 5e-5, "bfloat16": 3e-2}
TOL = {torch.float32: 2e-5, torch.bfloat16: 3e-2}
# In bfloat16 a result may also differ by this many times what rounding to bfloat16 alone moves in the plain computation
# (``store=plain.bfloat16``): the package rounds at other places than the plain functions do, so the two are two draws of
# that noise, and in these tiny models single positions amplify it.
NOISE = 4.0
# In float32 a result may differ by this many times what rounding every weight to 32-bit once more moves in the plain model
# (``reweighed``): tiny random models hold spots (a head whose output its own norm divides by almost nothing, say) that
# amplify any rounding; a lost key, a stale state or a reach one off moves a logit by percents.
NOISE_32 = 6.0


def reweighed(tensors, seed):
    """The tensors with every number off by some half a unit in the last place of a 32-bit float."""
    rng = np.random.default_rng(seed)
    return {name: a * (1.0 + 6e-8 * rng.standard_normal(a.shape)) for name, a in tensors.items()}


def dev():
    return torch.device("cuda", 0)


def runtime(dtype):
    from tesseract_b200.parts import Runtime

    return Runtime(dtype, dev())


def close(got, want, tol, what="", noise=0.0):
    got = got.detach().cpu().double().numpy() if isinstance(got, torch.Tensor) else np.asarray(got, dtype=np.float64)
    want = np.asarray(want, dtype=np.float64)
    assert np.isfinite(got).all(), what
    worst = float(np.abs(got - want).max())
    assert worst <= max(tol * max(1.0, float(np.abs(want).max())), NOISE * noise), f"{what}: {worst}"


def i32(values):
    return torch.tensor(list(values), dtype=torch.int32, device=dev())


def step_of(parts, tables=(), page=16):
    """A step of several sequences: ``parts`` is a list of (first position, rows, slot); ``tables``: per cache group one block
    table per sequence (or None)."""
    from tesseract_b200.parts import GroupView, StepContext

    counts = [n for _, n, _ in parts]
    starts = [0] + list(np.cumsum(counts))
    return StepContext(
        num_rows=starts[-1], num_seqs=len(parts), token_ids=i32([0] * starts[-1]),
        positions=i32([p for begin, n, _ in parts for p in range(begin, begin + n)]),
        seq_of_row=i32([s for s, n in enumerate(counts) for _ in range(n)]), row_start=i32(starts),
        seq_begin=i32([begin for begin, _, _ in parts]), state_slots=i32([slot for _, _, slot in parts]),
        groups=[GroupView(torch.tensor(t, dtype=torch.int32, device=dev()) if t is not None else None, page) for t in tables],
        host_new=counts, host_begin=[begin for begin, _, _ in parts], host_slots=[slot for _, _, slot in parts],
        max_new=max(counts), max_context=max(begin + n for begin, n, _ in parts))


def bf16(t):
    return t.to(torch.bfloat16)


def as_plain(tensors):
    return {name: t.double().numpy() for name, t in tensors.items()}


def portions_of(cut, T):
    if cut == "prompt":
        return [(0, T)]
    if cut == "decode":
        return [(0, 10)] + [(p, p + 1) for p in range(10, T)]
    if cut == "twos":
        return [(p, min(p + 2, T)) for p in range(0, T, 2)]
    if cut == "groups":
        return [(p, min(p + 20, T)) for p in range(0, T, 20)]
    edges = list(range(0, T, 37)) + [T]
    return list(zip(edges[:-1], edges[1:]))


# ----------------------------------------------------------------------------- the copies of the stream


@pytest.mark.parametrize("width,streams", [(5, 3), (42, 5), (64, 1), (64, 2), (96, 3), (256, 4), (4096, 4), (5120, 2), (40, 6), (24, 7),
                                           (32, 8), (48, 9), (8, 20)])
@pytest.mark.parametrize("out_dtype", [torch.float32, torch.bfloat16])
def test_copies_are_mixed_and_the_next_norm_taken(width, streams, out_dtype):
    """One kernel around a sublayer: no, one or two results taken in, with and without the norm behind; the copies differ by
    orders of magnitude, so one that is read after it was renewed would show."""
    from tesseract_b200 import kernels

    g = torch.Generator().manual_seed(width + streams)
    rows, eps = 7, 1e-5
    copies = torch.randn(rows, streams, width, generator=g) * torch.logspace(-1, 1, streams)[None, :, None]
    a, b = torch.randn(rows, width, generator=g), torch.randn(rows, width, generator=g)
    mix, share, take = (torch.randn(*shape, generator=g) for shape in ((streams, streams), (streams,), (streams,)))
    weight = torch.rand(width, generator=g) + 0.5
    on = [t.to(dev()) for t in (mix, share, take, weight, a, b)]
    for update in (None, (on[4], 0.7, None, 0.0), (on[4], 0.7, on[5], -1.3)):
        new = copies.double().numpy()
        if update is not None:
            y = 0.7 * a.double().numpy() + (-1.3 * b.double().numpy() if update[2] is not None else 0.0)
            new = (np.einsum("rsw,st->rtw", new, mix.double().numpy()) + share.double().numpy()[None, :, None] * y[:, None])
        u = np.einsum("rsw,s->rw", new, take.double().numpy())
        want = plain.over_rms(u, eps) * weight.double().numpy()
        for with_norm in (True, False):
            residual = copies.reshape(rows, -1).to(dev())
            out = torch.empty(rows, width, dtype=out_dtype, device=dev()) if with_norm else None
            kernels.mixed_streams_norm(residual, update, on[0], on[1], on[2] if with_norm else None, on[3] if with_norm else None, out,
                                       streams, eps)
            close(residual, new.reshape(rows, -1), 3e-6, "copies")
            if with_norm:
                close(out, want, 2e-5 if out_dtype == torch.float32 else 1e-2, "normed rows")


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width,copies,vocab,buckets,mul_prev,mul_cur", [(24, 1, 50, 1, 3, 4), (42, 3, 77, 97, 101, 12345),
                                                                          (256, 4, 300, 4096, 31, 7), (8, 2, 2 ** 17, 65537, 2 ** 40 + 1, 10 ** 9)])
def test_pairs_of_tokens_across_portions_and_slots(dtype, width, copies, vocab, buckets, mul_prev, mul_cur):
    """The first token of a request has nothing in front, whatever its slot held; the first token of a portion pairs with the
    last one of the portion before."""
    from tesseract_b200.config.spec import PartSpec
    from tesseract_b200.parts import EMBEDDINGS, CacheBinding

    g = torch.Generator().manual_seed(width)
    tensors = {"table": bf16(torch.randn(vocab, width, generator=g)), "pairs": bf16(torch.randn(buckets + 1, width, generator=g))}
    spec = PartSpec.make("bigram_embedding", {"vocab_size": vocab, "hidden_size": width, "buckets": buckets, "mul_prev": mul_prev,
                                              "mul_cur": mul_cur, "copies": copies}, {"table": "t", "pairs": "p"})
    part = EMBEDDINGS.get(spec.kind)(spec, tensors, runtime(dtype))
    config = {"embedding": {"bigram": {"buckets": buckets, "mul_prev": mul_prev, "mul_cur": mul_cur}}}
    requests = {slot: random_tokens(vocab, n, seed=slot) for slot, n in ((0, 30), (2, 9), (3, 17))}
    requests[0][0] = vocab - 1
    want = {slot: plain.embed(config, {"embed": tensors["table"].double().numpy(), "bigram": tensors["pairs"].double().numpy()}, tokens)
            for slot, tokens in requests.items()}
    cache = CacheBinding(group=0, storage=torch.full((5, 1), 3, dtype=torch.int32, device=dev()))
    at = {slot: 0 for slot in requests}
    for sizes in ((1, 2, 5), (7, 1, 1), (1, 1, 1), (2, 5, 9), (19, 0, 1)):
        parts, ids, rows = [], [], []
        for (slot, tokens), n in zip(requests.items(), sizes):
            if n:
                parts.append((at[slot], n, slot))
                ids += tokens[at[slot]:at[slot] + n]
                rows.append(want[slot][at[slot]:at[slot] + n])
                at[slot] += n
        got = part.forward(i32(ids), ctx=step_of(parts), cache=cache)
        rows = np.concatenate(rows)
        close(got, np.tile(rows[:, None], (1, copies, 1)).reshape(rows.shape[0], -1), 1e-6)
    assert at == {0: 30, 2: 9, 3: 17}


# ----------------------------------------------------------------------------- recurrences


RECURRENCES = {"state_space": ("mamba2", {"in": "in", "conv": "conv", "conv_bias": "conv.b", "dt_bias": "dt_bias", "a_log": "A_log", "skip": "D",
                                          "norm": "norm", "o": "o"}),
               "matrix_memory": ("mlstm", {"q": "q", "k": "k", "v": "v", "g": "g", "i": "i", "i_bias": "i.b", "f": "f", "f_bias": "f.b",
                                           "norm": "norm", "o": "o"}),
               "gated_delta": ("delta_mixer", {"q": "q", "k": "k", "v": "v", "g": "g", "q_conv": "q.conv", "k_conv": "k.conv", "v_conv": "v.conv",
                                               "a": "a", "b": "b", "a_log": "A_log", "dt_bias": "dt_bias", "norm": "norm", "o": "o"})}
CASES = [("state_space", {"heads": 6, "vdim": 12, "state": 20, "groups": 2, "norm_groups": 3, "conv": 3}),
         ("state_space", {"heads": 1, "vdim": 5, "state": 3, "groups": 1, "norm_groups": 1, "conv": 1}),
         ("state_space", {"heads": 4, "vdim": 64, "state": 128, "groups": 4, "norm_groups": 2, "conv": 4}),
         ("state_space", {"heads": 2, "vdim": 400, "state": 300, "groups": 1, "norm_groups": 1, "conv": 6}),
         ("state_space", {"heads": 3, "vdim": 33, "state": 530, "groups": 3, "norm_groups": 9, "conv": 2}),
         ("matrix_memory", {"heads": 3, "dim": 16, "vdim": 20, "gate_cap": 9.0}),
         ("matrix_memory", {"heads": 1, "dim": 7, "vdim": 31, "gate_cap": 3.0}),
         ("matrix_memory", {"heads": 2, "dim": 128, "vdim": 64, "gate_cap": 15.0}),
         ("matrix_memory", {"heads": 2, "dim": 90, "vdim": 100, "gate_cap": 40.0}),
         ("gated_delta", {"heads": 6, "kv_heads": 3, "dim": 12, "vdim": 20, "conv": 3}),
         ("gated_delta", {"heads": 2, "kv_heads": 2, "dim": 5, "vdim": 7, "conv": 1}),
         ("gated_delta", {"heads": 4, "kv_heads": 1, "dim": 128, "vdim": 32, "conv": 4}),
         ("gated_delta", {"heads": 4, "kv_heads": 2, "dim": 200, "vdim": 48, "conv": 2}),
         ("gated_delta", {"heads": 2, "kv_heads": 1, "dim": 260, "vdim": 9, "conv": 5})]


def recurrence_part(dtype, kind, m, hidden, eps, seed=None, tensors=None):
    """``(part, plain tensors, plain function)``; tensors are drawn by the part class unless given."""
    from tesseract_b200.config.spec import PartSpec
    from tesseract_b200.parts import MIXERS

    names = {"heads": "num_heads", "vdim": "value_dim", "dim": "key_dim", "kv_heads": "num_kv_heads", "conv": "conv_taps"}
    params = {names.get(key, key): value for key, value in m.items()}
    function, roles = RECURRENCES[kind]
    spec = PartSpec.make(kind, dict(params, hidden_size=hidden, eps=eps, stream="float32"), roles)
    cls = MIXERS.get(kind)
    if tensors is None:
        g = torch.Generator().manual_seed(seed)
        expected = cls.expected_tensors(spec)
        tensors = {name: bf16(cls.random_tensor(spec, role, expected[name].shape, g)) for role, name in roles.items()}
    part = cls(spec, {role: tensors[name] for role, name in roles.items()}, runtime(dtype))
    return part, as_plain(tensors), getattr(plain, function)


def states_of(part, slots=4, fill=0.0):
    """Bindings of the part's states; slots hold ``fill`` (a slot is zeroed when it is handed out, the others must not matter)."""
    from tesseract_b200.parts import CacheBinding

    needs = part.cache_need()
    needs = needs if isinstance(needs, tuple) else (needs,)
    made = tuple(CacheBinding(group=i, storage=torch.full((slots, *n.shape), fill, dtype=n.dtype, device=dev())) for i, n in enumerate(needs))
    return made if len(made) > 1 else made[0]


def hand_out(bindings, slot):
    for b in (bindings if isinstance(bindings, tuple) else (bindings,)):
        b.storage[slot].zero_()


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("kind,m", CASES)
def test_recurrences_in_portions_and_batches_over_used_slots(dtype, kind, m):
    hidden, eps, T = 40, 1e-4, 131
    part, w, function = recurrence_part(dtype, kind, m, hidden, eps, seed=len(str(m)))
    g = torch.Generator().manual_seed(5)
    rows = {slot: bf16(torch.randn(T, hidden, generator=g)) for slot in (0, 2, 3)}
    want = {slot: function(m, w, h.double().numpy(), eps) for slot, h in rows.items()}
    noise = 0.0
    if dtype == torch.bfloat16:
        noise = max(float(np.abs(function(m, w, h.double().numpy(), eps, store=plain.bfloat16) - want[slot]).max()) for slot, h in rows.items())
    bindings = states_of(part, fill=7.0)
    got = {slot: [] for slot in rows}
    at = {slot: 0 for slot in rows}
    for slot in rows:
        hand_out(bindings, slot)
    plan = [(2, 1, 33), (1, 1, 1), (5, 40, 2), (17, 16, 1), (1, 1, 1), (33, 2, 2), (2, 17, 15), (70, 53, 76)]
    for sizes in plan:
        parts = [(at[slot], n, slot) for slot, n in zip(rows, sizes)]
        x = torch.cat([rows[slot][begin:begin + n] for begin, n, slot in parts])
        out = part.forward(x.to(dtype).to(dev()), step_of(parts), bindings)
        done = 0
        for begin, n, slot in parts:
            got[slot].append(out[done:done + n])
            at[slot] += n
            done += n
    assert all(n == T for n in at.values())
    for slot in rows:
        close(torch.cat(got[slot]), want[slot], TOL[dtype], f"{kind} slot {slot}", noise)
    whole = part.forward(rows[2].to(dtype).to(dev()), step_of([(0, T, 1)]), states_of(part))
    close(whole, want[2], TOL[dtype], "whole", noise)


@pytest.mark.parametrize("kind,m", [c for c in CASES if c[1].get("conv", 4) > 1])
def test_cuts_of_the_recurrence_differ_by_rounding(kind, m):
    """The recurrence kernel itself on 32-bit rows: groups of rows begin where a portion begins, and single rows take a kernel of
    their own; results and states agree to a few roundings, and cuts at multiples of a group bit for bit."""
    from tesseract_b200 import kernels

    codes = {"state_space": kernels.STATE_SPACE, "matrix_memory": kernels.MATRIX_MEMORY, "gated_delta": kernels.DELTA_RULE}
    code, heads, vdim = codes[kind], m["heads"], m["vdim"]
    dim, qk = m.get("dim", m.get("state")), m.get("kv_heads", m.get("groups", heads))
    g = torch.Generator().manual_seed(11)
    T = 75
    rows = torch.randn(T, 2 * qk * dim + heads * vdim, generator=g).to(dev())
    gates = torch.randn(T, 2 * heads, generator=g).to(dev())
    vectors = [(-torch.rand(heads, generator=g)).to(dev()) for _ in range(3 if kind == "state_space" else 2)]
    shape = kernels.matrix_state_shape(code, heads, dim, vdim)

    def run(cut):
        state, running = torch.zeros(2, *shape, device=dev()), torch.zeros(2, *shape[:2], device=dev())
        out, aux = torch.empty(T, heads * vdim, device=dev()), torch.zeros(T, heads, 2, device=dev())
        for lo, hi in portions_of(cut, T):
            kernels.matrix_recurrence(code, rows[lo:hi], (0, qk * dim, 2 * qk * dim), gates[lo:hi], vectors, state, out[lo:hi], i32([0, hi - lo]),
                                      i32([1]), num_seqs=1, heads=heads, qk_heads=qk, dim=dim, vdim=vdim, max_new=hi - lo, q_scale=0.3, cap=5.0,
                                      running=running if kind == "matrix_memory" else None,
                                      aux=aux[lo:hi] if kind == "matrix_memory" else None)
        return out, aux, state

    first = run("prompt")
    assert not first[2][0].any(), "a slot of another request was touched"
    for cut in ("decode", "twos", "portions", "groups"):
        for one, other in zip(first, run(cut)):
            assert torch.isfinite(other).all()
            if cut == "groups":
                assert torch.equal(one, other)
            else:
                assert float((one - other).abs().max()) <= 2e-5 * max(1.0, float(one.abs().max())), cut


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("kind", ["state_space", "matrix_memory", "gated_delta"])
def test_recurrences_remember_one_token_over_hundreds(dtype, kind):
    """One token writes; 520 silent ones follow; the last one asks.  With decays near one its value must still be there."""
    hidden, T, eps = 24, 524, 1e-6
    m = {"state_space": {"heads": 2, "vdim": 8, "state": 8, "groups": 1, "norm_groups": 1, "conv": 2},
         "matrix_memory": {"heads": 2, "dim": 8, "vdim": 8, "gate_cap": 12.0},
         "gated_delta": {"heads": 2, "kv_heads": 1, "dim": 8, "vdim": 8, "conv": 2}}[kind]
    part, w, function = recurrence_part(torch.float32, kind, m, hidden, eps, seed=3)
    tensors = {name: torch.from_numpy(a).float() for name, a in w.items()}
    if kind == "state_space":
        tensors["A_log"][:], tensors["dt_bias"][:], tensors["D"][:], tensors["conv.b"][:] = -7.0, -1.0, 0.0, 0.0
    elif kind == "gated_delta":
        tensors["A_log"][:], tensors["dt_bias"][:] = -7.0, -1.0
    else:
        tensors["f.b"][:], tensors["i.b"][:] = 11.0, 0.0
        tensors["f"].zero_()
    tensors = {name: bf16(t) for name, t in tensors.items()}
    g = torch.Generator().manual_seed(1)
    h = torch.zeros(T, hidden)                              # (a silent token's key is zero: it writes and erases nothing)
    h[3] = torch.randn(hidden, generator=g) * 2.0
    h[T - 1] = torch.randn(hidden, generator=g)
    h = bf16(h)
    want = function(m, as_plain(tensors), h.double().numpy(), eps)
    forgotten = h.clone()
    forgotten[3] = h[2]
    assert np.abs(function(m, as_plain(tensors), forgotten.double().numpy(), eps)[T - 1] - want[T - 1]).max() > 0.2, "the case is not sharp"
    noise = 0.0
    if dtype == torch.bfloat16:
        noise = float(np.abs(function(m, as_plain(tensors), h.double().numpy(), eps, store=plain.bfloat16) - want)[[3, T - 1]].max())
    part, _, _ = recurrence_part(dtype, kind, m, hidden, eps, tensors=tensors)
    for cut in ("prompt", "portions", "decode"):
        bindings = states_of(part)
        got = torch.cat([part.forward(h[lo:hi].to(dtype).to(dev()), step_of([(lo, hi - lo, 1)]), bindings) for lo, hi in portions_of(cut, T)])
        close(got[[3, T - 1]], want[[3, T - 1]], 1e-4 if dtype == torch.float32 else 3e-2, cut, noise)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("groups,size", [(3, 7), (1, 64), (4, 96), (2, 300), (1, 5000), (1, 9000), (16, 128), (5, 513)])
@pytest.mark.parametrize("kind", ["sigmoid", "silu", "silu first"])
def test_norms_and_gates_behind_a_recurrence(dtype, groups, size, kind):
    from tesseract_b200 import kernels

    g = torch.Generator().manual_seed(size)
    rows, eps = 5, 1e-4
    v = torch.randn(rows, groups, size, generator=g) * torch.logspace(-2, 1, groups)[None, :, None]
    gate, shared = bf16(torch.randn(rows, groups * size, generator=g)), torch.rand(size, generator=g) + 0.5
    own = torch.rand(groups * size, generator=g) + 0.5
    aux = torch.stack([torch.randn(rows, groups, generator=g) * 3.0, torch.randn(rows, groups, generator=g)], dim=-1)
    z = gate.double().numpy().reshape(rows, groups, size)
    for weight, with_aux in ((shared, False), (own, True)):
        x = v.double().numpy()
        if with_aux:
            a = aux.double().numpy()
            x = x / (np.maximum(np.abs(a[..., 0]), np.exp(-a[..., 1])) + 1e-6)[..., None]
        w = weight.double().numpy().reshape(-1, size)
        want = plain.over_rms(x * plain.silu(z), eps) * w if kind == "silu first" else \
            plain.over_rms(x, eps) * w * (plain.sigmoid(z) if kind == "sigmoid" else plain.silu(z))
        out = torch.empty(rows, groups * size, dtype=dtype, device=dev())
        code = {"sigmoid": kernels.NORM_GATE_SIGMOID, "silu": kernels.NORM_GATE_SILU, "silu first": kernels.NORM_GATE_SILU_FIRST}[kind]
        wide = torch.zeros(rows, groups * size + 3, dtype=dtype, device=dev())       # gate rows of another stride
        for rows_of_gate in (gate.to(dtype).to(dev()), wide[:, :groups * size].copy_(gate.to(dev()))):
            kernels.recurrence_norm(v.reshape(rows, -1).to(dev()), rows_of_gate, weight.to(dev()), out, groups=groups, size=size, eps=eps,
                                    gate_kind=code, aux=aux.to(dev()) if with_aux else None)
            close(out, want.reshape(rows, -1), 5e-6 if dtype == torch.float32 else 1e-2, kind)


# ----------------------------------------------------------------------------- attention


def attention_case(kind, heads, kv_heads, d, dv, size, T, seed):
    """Tensors, input rows and marked (row, key) pairs of an attention in which queries read one slice of the input and keys
    another, so that a marked row's query points along its key and nowhere else."""
    g = torch.Generator().manual_seed(seed)
    width = 2 * d + 8
    tensors = {"q": torch.zeros(heads * d, width), "k": torch.zeros(kv_heads * d, width),
               "o": torch.randn(width, heads * dv, generator=g) * 0.3, "sink": torch.randn(heads, generator=g) * 2.0 + 3.0}
    for head in range(heads):
        tensors["q"][head * d:(head + 1) * d, d:2 * d] = torch.eye(d)
    for head in range(kv_heads):
        tensors["k"][head * d:(head + 1) * d, :d] = torch.eye(d)
    m = {"heads": heads, "kv_heads": kv_heads, "dim": d, "vdim": dv, "mask": {"size": size}, "scale": 12.0 / d}
    if kind == "window":
        m["scale"] *= 2.0                              # (the turned half of a head no longer lines up)
        tensors.update({"q.norm": torch.rand(heads * d, generator=g) * 0.5 + 0.75, "k.norm": torch.rand(kv_heads * d, generator=g) * 0.5 + 0.75})
        m["rot"] = {"dims": d // 4 * 2, "base": 1e6}
    else:
        tensors.update({"v": torch.randn(kv_heads * dv, width, generator=g) * 0.3, "q.b": torch.randn(heads * d, generator=g) * 0.1,
                        "k.b": torch.randn(kv_heads * d, generator=g) * 0.1, "v.b": torch.randn(kv_heads * dv, generator=g) * 0.3,
                        "g": torch.randn(heads, width, generator=g) * 0.5})
    tensors = {n: bf16(t) for n, t in tensors.items()}
    h = torch.randn(T, width, generator=g)
    pairs = []

    def mark(row, key):
        if 0 <= key <= row < T and all(row != r for r, _ in pairs):
            pairs.append((row, key))

    if size >= T:                                          # all is seen
        for row, key in ((T - 1, 0), (T - 2, 3), (300, 44), (257, 0), (200, 100), (64, 63)):
            mark(row, key)
    elif kind == "window":
        for row, back in zip([T - 1, T - 2, 300, 257, 256, 200, 150, 64, 48, size - 1, size],
                             [size - 1, size, size - 1, size, 0, 16, size - 1, size, size - 1, size - 1, size]):
            mark(row, row - back)
    else:
        for at in range(0, T, size):                   # the chunk's first position from its last row, and the one before from others
            mark(min(at + size, T) - 1, at)
            mark(at + size // 2, at - 1)
            mark(at, at - 1)
    for row, key in pairs:
        h[row, d:2 * d] = h[key, :d].clone()
    return tensors, bf16(h).float(), m, pairs


def attention_part(dtype, kind, width, m, tensors, eps):
    from tesseract_b200.config.spec import PartSpec
    from tesseract_b200.parts import MIXERS

    params = {"hidden_size": width, "num_heads": m["heads"], "num_kv_heads": m["kv_heads"], "key_dim": m["dim"], "value_dim": m["vdim"],
              "scale": m["scale"], "sink": True, "stream": "float32"}
    names = {"q": "q", "k": "k", "o": "o", "sink": "sink"}
    children = {}
    if kind == "window":
        params.update(mask=(("kind", "window"), ("size", m["mask"]["size"])), projection_norm_eps=eps, values_from_keys=True)
        names.update({"q_norm": "q.norm", "k_norm": "k.norm"})
        if m.get("rot"):
            children = {"position": PartSpec.make("rotary_blend", {"head_dim": m["dim"], "dims": m["rot"]["dims"], "base": m["rot"]["base"],
                                                                   "scaling": None})}
    else:
        params.update(mask=(("kind", "blocks"), ("size", m["mask"]["size"])), bias=True, head_gate=True)
        names.update({"v": "v", "q_bias": "q.b", "k_bias": "k.b", "v_bias": "v.b", "g": "g"})
    spec = PartSpec.make("normed_attention", params, names, children)
    return MIXERS.get(spec.kind)(spec, {role: tensors[name] for role, name in names.items()}, runtime(dtype))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads,kv_heads,d,dv", [(4, 2, 16, 24), (3, 1, 10, 14), (2, 2, 64, 64), (6, 3, 24, 8), (2, 1, 128, 128), (12, 1, 64, 48),
                                                 (5, 1, 40, 128)])
@pytest.mark.parametrize("size", [33, 16, 1, 64, 130, 1000])
@pytest.mark.parametrize("kind", ["window", "chunks"])
def test_attention_sees_exactly_its_window_or_chunk(dtype, kind, heads, kv_heads, d, dv, size):
    """The part as a prompt, in portions and as decoded rows over scrambled pages full of stale data, against the plain
    function.  The case is sharp: a window or chunk one position longer or shorter, chunks counted from elsewhere, a forgotten
    sink or gate, values taken behind the norm would change marked rows."""
    from tesseract_b200.parts import CacheBinding

    T, page, eps = 330, 16, 1e-5
    if kind == "window":
        dv = d
    tensors, h, m, pairs = attention_case(kind, heads, kv_heads, d, dv, size, T, seed=heads * 100 + d + size)
    weights, marked = as_plain(tensors), [row for row, _ in pairs]

    def plainly(m=m, w=weights, rows=h, store=plain.identity):
        x = rows.double().numpy()
        return plain.shared_kv_attention(m, w, x, eps, store) if kind == "window" else plain.chunk_attention(m, w, x, store)

    want = plainly()

    def changes(other, rows=marked):
        return float(np.abs(other[rows] - want[rows]).max())

    every = slice(None)
    if size < T:
        assert changes(plainly(dict(m, mask={"size": size + 1}))) > 0.03
        assert size == 1 or changes(plainly(dict(m, mask={"size": size - 1}))) > 0.05
    assert changes(plainly(w=dict(weights, sink=weights["sink"] - 50.0)), every) > 0.05, "no row notices the sink"
    assert changes(plainly(w=dict(weights, sink=weights["sink"] * m["scale"])), every) > 0.05 or abs(m["scale"] - 1.0) < 0.3
    if kind == "window":
        assert size == 1 or changes(plainly(dict(m, rot=dict(m["rot"], base=30.0))), every) > 0.05, "no row notices the rotation"
    else:
        assert changes(plainly(w=dict(weights, g=weights["g"] * 0.0)), every) > 0.05, "no row notices the gate"
    noise = float(np.abs(plainly(store=plain.bfloat16) - want).max()) if dtype == torch.bfloat16 else 0.0
    part = attention_part(dtype, kind, h.shape[1], m, tensors, eps)
    need = part.cache_need()
    assert (need.window, need.block) == ((size, None) if kind == "window" else (None, size))
    count = -(-T // page)
    torch.manual_seed(3)
    order = [1 + i for i in torch.randperm(count).tolist()]              # pages taken in scrambled order
    for cut in ("prompt", "decode", "portions", "twos"):
        binding = CacheBinding(group=0, storage=torch.full((count + 1, need.page_shape(page)[0]), 7.0, dtype=dtype, device=dev()),
                               writes=True, page_size=page)              # stale data
        got = [part.forward(h[lo:hi].to(dtype).to(dev()), step_of([(lo, hi - lo, 0)], [[order]], page), binding)
               for lo, hi in portions_of(cut, T)]
        close(torch.cat(got), want, TOL[dtype], cut, noise)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads,kv_heads,d,rot", [(4, 2, 16, 16), (3, 1, 10, 6), (8, 8, 128, 64), (2, 1, 24, 0), (6, 2, 64, 2), (5, 1, 7, 4)])
@pytest.mark.parametrize("from_keys", [True, False])
def test_projections_are_normed_as_a_whole_then_turned(dtype, heads, kv_heads, d, rot, from_keys):
    """The kernel alone: heads of very different sizes share one root mean square; values are stored as projected."""
    from tesseract_b200 import kernels

    g = torch.Generator().manual_seed(d)
    rows, page, eps, first = 21, 8, 1e-5, 37
    vdim = d if from_keys else d + 3
    both = (heads + kv_heads) * d
    loud = torch.cat([torch.logspace(-1, 1, heads).repeat_interleave(d), torch.logspace(1, -1, kv_heads).repeat_interleave(d)])
    proj = torch.randn(rows, both + (0 if from_keys else kv_heads * vdim) + 5, generator=g)
    proj[:, :both] *= loud
    proj = bf16(proj)
    weight = torch.rand(both, generator=g) + 0.5
    inv = torch.tensor([900.0 ** (-2.0 * i / rot) for i in range(rot // 2)]) if rot else None
    x, w = proj.double().numpy(), weight.double().numpy()
    q = (plain.over_rms(x[:, :heads * d], eps) * w[:heads * d]).reshape(rows, heads, d)
    k = (plain.over_rms(x[:, heads * d:both], eps) * w[heads * d:]).reshape(rows, kv_heads, d)
    if rot:
        q, k = plain.rotate_halves(q, rot, 900.0, first), plain.rotate_halves(k, rot, 900.0, first)
    v = x[:, heads * d:both] if from_keys else x[:, both:both + kv_heads * vdim]
    pages = -(-(first + rows) // page)
    order = list(reversed(range(1, pages + 1)))
    cache = torch.zeros(pages + 1, page * kv_heads * (d + vdim), dtype=dtype, device=dev())
    q_out = torch.empty(rows, heads * d, dtype=dtype, device=dev())
    ctx = step_of([(first, rows, 0)], [[order]], page)
    kernels.row_norm_rope_cache(proj.to(dtype).to(dev()), q_out, cache, ctx.positions, ctx.seq_of_row, ctx.groups[0].block_table,
                                None if inv is None else inv.to(dev()), weight.to(dev()), amplitude=1.0, heads=heads, kv_heads=kv_heads,
                                dim=d, vdim=vdim, rot_dims=rot, eps=eps, page_size=page, values_from_keys=from_keys)
    tol = 2e-5 if dtype == torch.float32 else 1e-2
    close(q_out, q.reshape(rows, -1), tol, "q")
    host = cache.cpu().double().numpy()
    for t in range(rows):
        p = first + t
        held = host[order[p // page]]
        keys = held[:kv_heads * page * d].reshape(kv_heads, page, d)[:, p % page]
        values = held[kv_heads * page * d:].reshape(kv_heads, page, vdim)[:, p % page]
        close(keys, k[t], tol, "k")
        close(values, v[t].reshape(kv_heads, vdim), 1e-6, "v")


# ----------------------------------------------------------------------------- whole models


def make_requests(name):
    vocab = TINY_TIBIVIK[name]["vocab"]
    return {f"{name}{i}": random_tokens(vocab, n, seed=500 + i) for i, n in enumerate(LENGTHS[name])}


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    from tesseract_b200.weights.random_init import write_random_model

    made = {}

    def get(name):
        if name not in made:
            made[name] = write_random_model(str(tmp_path_factory.mktemp(f"tibivik_{name}")), TINY_TIBIVIK[name], seed=23)
        return made[name]

    return get


@pytest.fixture(scope="module")
def engines(folders):
    from tesseract_b200.engine import load_model, make_stepper

    models = {}

    def get(name, dtype, capacity_tokens=4096, max_requests=8):
        if (name, dtype) not in models:
            models[(name, dtype)] = load_model(folders(name), dtype=dtype)
        return make_stepper(models[(name, dtype)], capacity_tokens=capacity_tokens, max_requests=max_requests)

    return get


_PLAIN = {}


def plain_rows(folder, requests, dtype):
    """Per request the plain model's logits, and what rounding alone (of what a bfloat16 run stores; of the weights to 32-bit)
    moves in the plain model's logits at the positions of all requests (the largest |difference| of each)."""
    want, moved = {}, []
    config, tensors = plain.load_folder(folder)
    for rid, tokens in requests.items():
        key = (folder, tuple(tokens))
        if key not in _PLAIN:
            _PLAIN[key] = (plain.forward(config, tensors, tokens)[0], {})
        exact, noises = _PLAIN[key]
        if dtype not in noises:
            others = ([plain.forward(config, tensors, tokens, store=plain.bfloat16)[0]] if dtype == "bfloat16"
                      else [plain.forward(config, reweighed(tensors, seed), tokens)[0] for seed in range(3)])
            noises[dtype] = np.max([np.abs(other - exact).max(axis=1) for other in others], axis=0)
        want[rid] = exact
        moved.append(noises[dtype])
    return want, np.concatenate(moved)


def replay_against_plain(stepper, steps, folder, requests, dtype, what):
    """Replay a trace and compare every wanted row with the plain model.  No row may differ by more than ``REL`` of the
    request's largest |logit| or ``NOISE`` (``NOISE_32``) times what rounding alone moves anywhere in the plain model, and of all rows
    at most one in twenty by more than that many times what rounding moves at nine positions of ten."""
    want, moved = plain_rows(folder, requests, dtype)
    got = replay(stepper, steps)
    assert got, f"{what}: nothing was replayed"
    times = NOISE if dtype == "bfloat16" else NOISE_32
    usual, over = float(np.quantile(moved, 0.9)), []
    for (rid, position), row in sorted(got.items(), key=lambda kv: (str(kv[0][0]), kv[0][1])):
        scale = float(np.abs(want[rid]).max())
        limit = max(REL[dtype] * scale, times * float(moved.max()))
        err = float(np.abs(row.astype(np.float64) - want[rid][position]).max())
        assert np.isfinite(row).all() and err <= limit, (f"{what}: first wrong token is request {rid!r} position "
                                                         f"{position}: max |diff| {err:.3e} > {limit:.3e}")
        if err > max(REL[dtype] * scale, times * usual):
            over.append((rid, position))
    assert len(over) <= 1 + len(got) // 20, f"{what}: {len(over)} of {len(got)} rows beyond the usual rounding, the first {over[:3]}"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["a", "b", "c", "d", "e"])
def test_every_layer_matches_plain(engines, folders, name, dtype):
    """The stream (the sum of its copies) after every layer run against the plain model's."""
    from tesseract_b200.engine import StepEntry
    from tesseract_b200.parts.block import HyperConnectedBlock

    config, tensors = plain.load_folder(folders(name))
    tokens = random_tokens(config["vocab"], 37, seed=8)
    _, want = plain.forward(config, tensors, tokens)
    if dtype == "bfloat16":
        _, coarse = plain.forward(config, tensors, tokens, store=plain.bfloat16)
    else:
        _, coarse = plain.forward(config, reweighed(tensors, 1), tokens)
    seen = []
    original = HyperConnectedBlock.forward

    def recording(self, stream, ctx, cache, next_norm=None):
        out = original(self, stream, ctx, cache, next_norm=next_norm)
        assert out.update is None and out.residual.dtype == torch.float32
        seen.append(out.residual.double().cpu().numpy().reshape(len(tokens), config["streams"], -1).sum(axis=1))
        return out

    stepper = engines(name, dtype)
    assert stepper.cache.admit("one")
    HyperConnectedBlock.forward = recording
    try:
        stepper.step([StepEntry("one", tokens, [len(tokens) - 1])])
    finally:
        HyperConnectedBlock.forward = original
        stepper.cache.release("one")
    assert len(seen) == len(want) == len(plain.run_order(config))
    for index, got in enumerate(seen):
        limit = REL[dtype] * float(np.abs(want[index]).max())
        # or what rounding alone moves in the plain model
        limit = max(limit, (NOISE if dtype == "bfloat16" else NOISE_32) * float(np.abs(coarse[index] - want[index]).max()))
        assert float(np.abs(got - want[index]).max()) <= limit, f"layer {index}"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["a", "b", "c", "d", "e"])
@pytest.mark.parametrize("cut", ["whole", "tail", "portions", "twos"])
def test_cuts_match_plain(engines, folders, name, dtype, cut):
    """Whole prompts, prompts with a decoded tail (over which the windows move and the states are carried),
    portions of changing size, and portions of two and three tokens throughout."""
    requests = make_requests(name)
    if cut == "twos":
        steps = trace_portions(requests, sizes=(2, 3, 2, 2))
    elif cut == "tail":
        steps = trace_tail(requests, tail=60)
    else:
        steps = {"whole": trace_whole, "portions": trace_portions}[cut](requests)
    stepper = engines(name, dtype)
    replay_against_plain(stepper, steps, folders(name), requests, dtype, f"{name}/{dtype}/{cut}")
    stepper.cache.check()
    assert stepper.cache.used_pages() == 0


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["a", "b", "c", "d", "e"])
def test_mixed_batches_with_slots_and_pages_used_again(engines, folders, name, dtype):
    requests = make_requests(name)
    requests.update({f"{name}x{i}": random_tokens(TINY_TIBIVIK[name]["vocab"], n, seed=17 + i)
                     for i, n in enumerate([50, 21, 90, 34, 7])})
    steps = trace_mixed(requests, seed=5, live_max=3)
    assert max(len(e) for e, _ in steps) >= 3, "the trace should batch several requests"
    # three state slots for eight or more requests: every slot serves several requests one after the other
    stepper = engines(name, dtype, capacity_tokens=max_live_tokens(steps), max_requests=3)
    replay_against_plain(stepper, steps, folders(name), requests, dtype, f"{name}/{dtype}/mixed")
    assert stepper.cache.pages_reused > 0, "the pool was sized so that pages must be used again"
    stepper.cache.check()
    assert stepper.cache.used_pages() == 0


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["a", "e"])
def test_a_batch_gives_each_request_what_it_gets_alone(engines, name, dtype):
    """Unequal requests side by side against each alone, in portions that cut windows and pages."""
    from tesseract_b200.engine import StepEntry

    requests = make_requests(name)
    sizes = [9, 2, 30, 5]
    alone = replay(engines(name, dtype), trace_portions(requests, sizes=tuple(sizes)))
    together = {}
    stepper = engines(name, dtype)
    at = {rid: 0 for rid in requests}
    for rid in requests:
        assert stepper.cache.admit(rid)
    turn = 0
    while any(at[rid] < len(t) for rid, t in requests.items()):
        batch, meta = [], []
        for rid, tokens in requests.items():
            if at[rid] >= len(tokens):
                continue
            size = sizes[turn % 4]
            if len(tokens) - at[rid] - size == 1:
                size += 1
            part = tokens[at[rid]:at[rid] + size]
            batch.append(StepEntry(rid, part, list(range(len(part)))))
            meta.append((rid, at[rid], len(part)))
            at[rid] += len(part)
        rows = stepper.step(batch).float().cpu().numpy()
        r = 0
        for rid, base, n in meta:
            for place in range(n):
                together[(rid, base + place)] = rows[r]
                r += 1
        turn += 1
    worst = max(float(np.abs(together[key] - alone[key]).max()) for key in alone)
    scale = max(float(np.abs(row).max()) for row in alone.values())
    # the products of a batch take other kernels at other row counts: equal up to rounding, not bit for bit
    assert worst <= REL[dtype] * scale


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["a", "c", "e"])
def test_long_decoding_while_windows_move(engines, folders, name, dtype):
    tokens = random_tokens(TINY_TIBIVIK[name]["vocab"], 180, seed=77)
    requests = {"long": tokens}
    steps = trace_tail(requests, tail=170)          # ten tokens of prompt, then 170 decoded one by one
    stepper = engines(name, dtype, capacity_tokens=192)
    replay_against_plain(stepper, steps, folders(name), requests, dtype, f"{name}/{dtype}/long decode")
    assert stepper.cache.used_pages() == 0


def test_pages_behind_windows_and_of_earlier_chunks_go_back_while_the_request_lives(engines):
    """Model "a": a window of 21 and chunks of 25 tokens (pages of 16): a request of 200 tokens never holds more than a few
    pages a group."""
    from tesseract_b200.engine import StepEntry

    stepper = engines("a", "float32", capacity_tokens=208)
    assert stepper.cache.admit("one")
    tokens = random_tokens(TINY_TIBIVIK["a"]["vocab"], 200, seed=5)
    paged = [index for index, group in enumerate(stepper.cache.groups) if group.pool is not None]
    assert len(paged) == 2
    for at in range(0, 200, 10):
        stepper.step([StepEntry("one", tokens[at:at + 10], [9])])
        for index in paged:
            need, end = stepper.cache.groups[index].need, at + 10
            first = max(0, end - need.window + 1) if need.window else end // need.block * need.block
            assert set(stepper.cache.pages_of("one", index)) == set(range(first // 16, -(-end // 16)))
    stepper.cache.release("one")
    stepper.cache.check()
    assert stepper.cache.used_pages() == 0


def test_a_slot_used_before_leaves_nothing_behind(engines):
    """The same request in a slot that an unrelated long one has just left gives the same logits, bit for bit, its first token
    (which pairs with nothing) among them."""
    from tesseract_b200.engine import StepEntry

    stepper = engines("a", "float32", capacity_tokens=512, max_requests=1)
    tokens, other = random_tokens(131, 40, seed=1), random_tokens(131, 170, seed=2)

    def run():
        assert stepper.cache.admit("r")
        parts = [stepper.step([StepEntry("r", tokens[lo:hi], list(range(hi - lo)))]).cpu() for lo, hi in ((0, 1), (1, 3), (3, 40))]
        stepper.cache.release("r")
        return torch.cat(parts)

    first = run()
    assert stepper.cache.admit("x")
    stepper.step([StepEntry("x", other, [])])
    stepper.cache.release("x")
    assert torch.equal(run(), first)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("graphs", [False, True])
@pytest.mark.parametrize("name", ["a", "b", "e"])
def test_greedy_generation_through_the_scheduler(folders, name, dtype, graphs):
    from tesseract_b200 import LLM, SamplingParams

    config, tensors = plain.load_folder(folders(name))
    prompts = [random_tokens(config["vocab"], n, seed=n) for n in (3, 19, 75, 1)]
    steps = 24
    llm = LLM(folders(name), dtype=dtype, kv_capacity_tokens=1024, max_running=3, prefill_chunk_tokens=32,
              cuda_graphs=graphs)
    outs = llm.generate(prompts, SamplingParams(max_tokens=steps, temperature=0.0, ignore_eos=True))
    for prompt, out in zip(prompts, outs):
        assert len(out.token_ids) == steps and out.finish_reason == "length"
        tokens = list(prompt)
        for k, got in enumerate(out.token_ids):
            logits = plain.forward(config, tensors, tokens)[0][-1]
            best = int(np.argmax(logits))
            margin = float(logits[best] - logits[got])
            limit = GREEDY_MARGIN[dtype] * float(np.abs(logits).max())
            if got != best and margin > limit and dtype == "bfloat16":
                # what rounding to bfloat16 alone does to this position's logits in the plain model bounds what the
                # engine's token may lose
                coarse = plain.forward(config, tensors, tokens, store=plain.bfloat16)[0][-1]
                limit = max(limit, 3.0 * float(np.abs(coarse - logits).max()))
            assert got == best or margin <= limit, f"{name}/{dtype}: token {k} is {got}, plain says {best}"
            tokens.append(got)
    assert llm.stepper.cache.used_pages() == 0
    if graphs:      # decode steps were replayed as graphs, not issued launch by launch
        assert llm.stepper.graphs.safe and llm.stepper.graphs.replays >= steps - 2
    del llm
    torch.cuda.empty_cache()


def test_replay_program_runs_a_tibivik_folder(folders, tmp_path):
    """``bin/trace_run`` picks the model class by ``config.json`` and writes the logits of the wanted places."""
    import json
    import os
    import subprocess
    import sys

    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    config, tensors = plain.load_folder(folders("b"))
    tokens = random_tokens(config["vocab"], 30, seed=9)
    lines = [json.dumps({"step": 0, "entries": [{"id": "a", "tokens": tokens[:20], "want": [0, 19]}], "end": []}),
             json.dumps({"step": 1, "entries": [{"id": "a", "tokens": tokens[20:], "want": [9]}], "end": ["a"]})]
    out = tmp_path / "out"
    done = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", folders("b"), "--dtype",
                           "float32", "--out", str(out), "--max-tokens", "64"], input="\n".join(lines) + "\n",
                          capture_output=True, text=True, timeout=600)
    assert done.returncode == 0, done.stderr[-2000:]
    assert [l for l in done.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1"]
    want = plain.forward(config, tensors, tokens)[0]
    first = np.fromfile(out / "0.f32", dtype="<f4").reshape(2, -1)
    second = np.fromfile(out / "1.f32", dtype="<f4").reshape(1, -1)
    scale = float(np.abs(want).max())
    assert np.abs(first - want[[0, 19]]).max() <= 5e-5 * scale
    assert np.abs(second - want[[29]]).max() <= 5e-5 * scale


def test_command_line_generates_and_prints_the_plan(folders):
    import json
    import os
    import subprocess
    import sys

    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    folder = folders("a")
    common = [sys.executable, os.path.join(root, "bin", "tesseract"), "--model-path", folder, "--kv-capacity-tokens",
              "256", "--max-running", "2", "--dtype", "float32"]
    done = subprocess.run(common + ["--prompt-ids", "5,6,7,8", "--random-prompt", "11", "--max-tokens", "4",
                                    "--temperature", "0", "--ignore-eos", "--json", "--check-weights"],
                          capture_output=True, text=True, timeout=600)
    assert done.returncode == 0, done.stderr[-2000:]
    records = [json.loads(line) for line in done.stdout.strip().splitlines()]
    assert len(records) == 2 and all(len(r["token_ids"]) == 4 and r["finish_reason"] == "length" for r in records)
    config, tensors = plain.load_folder(folder)
    tokens = [5, 6, 7, 8]
    for got in records[0]["token_ids"]:
        logits = plain.forward(config, tensors, tokens)[0][-1]
        best = int(np.argmax(logits))
        assert got == best or float(logits[best] - logits[got]) <= GREEDY_MARGIN["float32"] * float(np.abs(logits).max())
        tokens.append(got)
    shown = subprocess.run(common + ["--print-plan"], capture_output=True, text=True, timeout=600)
    assert shown.returncode == 0, shown.stderr[-2000:]
    assert "kernel plan for Tibivik" in shown.stdout
    for kind in ("parallel_mixers", "state_space"):
        assert f"mixer '{kind}'" in shown.stdout


@pytest.mark.parametrize("seed", [1, 2, 3, 5, 8, 13, 21, 34])
def test_random_configurations_match_plain_in_float32(tmp_path, seed):
    """Configurations drawn at random (layer order, every size and constant), each whole, with a decoded tail, in
    portions and in mixed batches."""
    import random

    from tesseract_b200.engine import load_model, make_stepper
    from tesseract_b200.weights.random_init import write_random_model

    config = random_config(seed)
    folder = write_random_model(str(tmp_path / "model"), config, seed=seed)
    r = random.Random(seed + 1000)
    lengths = [1, r.randint(2, 40), r.randint(41, 140), r.randint(141, 300), r.randint(5, 90)]
    requests = {f"q{i}": random_tokens(config["vocab"], n, seed=seed * 10 + i) for i, n in enumerate(lengths)}
    model = load_model(folder, dtype="float32")
    for name, steps in (("whole", trace_whole(requests)), ("tail", trace_tail(requests, tail=20)),
                        ("portions", trace_portions(requests)), ("mixed", trace_mixed(requests, seed=seed, live_max=4))):
        stepper = make_stepper(model, capacity_tokens=max(1024, max_live_tokens(steps)), max_requests=4)
        replay_against_plain(stepper, steps, folder, requests, "float32", f"seed {seed}/{name}")
        assert stepper.cache.used_pages() == 0


@pytest.mark.parametrize("seed", [1, 2, 3, 5, 8, 13, 21, 34])
def test_random_configurations_match_plain_in_bfloat16(tmp_path, seed):
    """The same configurations in bfloat16 (products of odd sizes, head sizes on and off the tensor-core kernels),
    whole, with a decoded tail and in mixed batches."""
    import random

    from tesseract_b200.engine import load_model, make_stepper
    from tesseract_b200.weights.random_init import write_random_model

    config = random_config(seed)
    folder = write_random_model(str(tmp_path / "model"), config, seed=seed)
    r = random.Random(seed + 2000)
    lengths = [1, r.randint(2, 40), r.randint(41, 140), r.randint(260, 330), r.randint(5, 90)]
    requests = {f"q{i}": random_tokens(config["vocab"], n, seed=seed * 10 + i) for i, n in enumerate(lengths)}
    model = load_model(folder, dtype="bfloat16")
    for name, steps in (("whole", trace_whole(requests)), ("tail", trace_tail(requests, tail=20)),
                        ("mixed", trace_mixed(requests, seed=seed, live_max=4))):
        stepper = make_stepper(model, capacity_tokens=max(1024, max_live_tokens(steps)), max_requests=4)
        replay_against_plain(stepper, steps, folder, requests, "bfloat16", f"seed {seed}/{name}")
        assert stepper.cache.used_pages() == 0
