"""Rirulix on the GPU against the plain implementation (``tests/plain/rirulix.py``).

First every mechanism alone (its kernel or part against the plain function, with inputs made so that a fault shows: one
key that dominates, placed at the window's first position and one before it, among the kept first tokens and right behind
them, at page borders and hundreds of positions back; a recurrence that remembers one token over hundreds of steps), then
whole tiny models with random weights under every way of cutting the work: whole prompts, token-by-token decoding, portions
down to two tokens, mixed batches with slots and pages used again, long decoding while the windows move over decoded
tokens, and greedy generation through the package's own entry point and scheduler.
"""

import numpy as np
import pytest
import torch

from tests.helpers import (GREEDY_MARGIN, compare, max_live_tokens, random_tokens, replay, trace_mixed, trace_portions,
                           trace_tail, trace_whole)
from tests.plain import rirulix as plain
from tests.rirulix_models import LENGTHS, TINY_RIRULIX, random_config

pytestmark = pytest.mark.gpu

REL = {"float32": 5e-5, "bfloat16": 3e-2}
TOL = {torch.float32: 2e-5, torch.bfloat16: 3e-2}
# In bfloat16 a result may also differ by this many times what rounding to bfloat16 alone moves in the plain computation
# (``store=plain.bfloat16``): the package rounds at other places than the plain functions do, so the two are two draws of
# that noise, and in these tiny models single positions amplify it.
NOISE = 5.0


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


def step_context(positions, tables=(), page=16, slot=0):
    """A step of one sequence whose rows stand at ``positions`` (consecutive); ``tables``: one block table per cache group."""
    from tesseract_b200.parts import GroupView, StepContext

    n = len(positions)
    return StepContext(num_rows=n, num_seqs=1, token_ids=i32([0] * n), positions=i32(positions), seq_of_row=i32([0] * n),
                       row_start=i32([0, n]), seq_begin=i32([positions[0]]), state_slots=i32([slot]),
                       groups=[GroupView(torch.tensor([t], dtype=torch.int32, device=dev()) if t is not None else None, page)
                               for t in tables],
                       host_new=[n], host_begin=[positions[0]], host_slots=[slot], max_new=n, max_context=positions[-1] + 1)


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
    edges = list(range(0, T, 37)) + [T]
    return list(zip(edges[:-1], edges[1:]))


# ----------------------------------------------------------------------------- mechanisms alone


@pytest.mark.parametrize("width,groups", [(5, 1), (42, 7), (42, 2), (66, 3), (96, 24), (256, 2), (4096, 8), (4096, 64), (12288, 3)])
@pytest.mark.parametrize("out_dtype", [torch.float32, torch.bfloat16])
def test_norms_over_parts_around_a_sublayer(width, groups, out_dtype):
    """The norm of an update, the addition and the following norm in one kernel, each over its own number of parts; the
    parts differ in size by orders of magnitude, so a statistic of another part would show."""
    from tesseract_b200 import kernels

    g = torch.Generator().manual_seed(width + groups)
    rows, eps = 7, 1e-5
    loud = torch.logspace(-2, 2, groups).repeat_interleave(width // groups)
    residual, update = torch.randn(rows, width, generator=g) * loud, torch.randn(rows, width, generator=g) * loud.flip(0)
    w1, w2 = torch.rand(width, generator=g) + 0.5, torch.rand(width, generator=g) + 0.5
    for post_groups, next_groups in ((groups, groups), (1, groups), (groups, 1)):
        u = plain.grouped_rms_norm(update.double().numpy(), w1.double().numpy(), post_groups, eps)
        stream = residual.double().numpy() + u
        want = plain.grouped_rms_norm(stream, w2.double().numpy(), next_groups, eps)
        on, out = residual.to(dev()), torch.empty(rows, width, dtype=out_dtype, device=dev())
        kernels.norm_add_norm(on, update.to(dev()), (kernels.NORM_RMS, w1.to(dev()), None, post_groups),
                              (kernels.NORM_RMS, w2.to(dev()), None, next_groups), out, None, eps)
        close(on, stream, 2e-6, "stream")
        close(out, want, 2e-6 if out_dtype == torch.float32 else 1e-2, "normed rows")
    # each alone: no update in front, or nothing behind
    on = residual.to(dev())
    out = torch.empty(rows, width, dtype=out_dtype, device=dev())
    kernels.norm_add_norm(on, None, None, (kernels.NORM_RMS, w2.to(dev()), None, groups), out, None, eps)
    close(out, plain.grouped_rms_norm(residual.double().numpy(), w2.double().numpy(), groups, eps),
          2e-6 if out_dtype == torch.float32 else 1e-2, "norm alone")


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width,groups", [(6, 1), (42, 7), (66, 3), (256, 4), (5120, 2)])
def test_learned_positions_in_front_of_the_embedding_norm(dtype, width, groups):
    from tesseract_b200.config.spec import PartSpec
    from tesseract_b200.parts import EMBEDDINGS

    g = torch.Generator().manual_seed(width)
    vocab, places, eps = 23, 50, 1e-6
    tensors = {"embed": bf16(torch.randn(vocab, width, generator=g)), "pos": bf16(torch.randn(places, width, generator=g)),
               "embed.norm": bf16(torch.rand(width, generator=g) + 0.5)}
    spec = PartSpec.make("positioned_embedding", {"vocab_size": vocab, "hidden_size": width, "max_positions": places, "groups": groups,
                                                  "eps": eps}, {"table": "embed", "positions": "pos", "weight": "embed.norm"})
    part = EMBEDDINGS.get(spec.kind)(spec, {role: tensors[name] for role, name in spec.weights.items()}, runtime(dtype))
    tokens, positions = [3, 3, 22, 0, 7], [0, 1, 49, 17, 17]
    got = part.forward(i32(tokens), positions=i32(positions))
    w = as_plain(tensors)
    want = plain.grouped_rms_norm(w["embed"][tokens] + w["pos"][positions], w["embed.norm"], groups, eps)
    assert got.dtype == torch.float32
    close(got, want, 2e-6)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("channels,taps", [(33, 5), (24, 1), (40, 2), (64, 3), (256, 4), (16, 8), (7, 4)])
def test_short_convolution_in_portions_and_batches(dtype, channels, taps):
    """Three requests of other lengths in one batch, cut in portions (one row a request at times), over slots that held
    other requests before."""
    from tesseract_b200 import kernels

    g = torch.Generator().manual_seed(channels * 10 + taps)
    lengths, slots = [57, 1, 90], [2, 0, 3]
    w, bx, bc = torch.randn(taps, channels, generator=g), torch.randn(channels, generator=g), torch.randn(channels, generator=g)
    rows = [torch.randn(n, channels, generator=g).to(dtype) for n in lengths]
    want = [plain.causal_convolution(r.double().numpy() + bx.double().numpy(), w.double().numpy().T, bc.double().numpy()) for r in rows]
    state = torch.full((5, taps - 1, channels), 9.0, device=dev()) if taps > 1 else None
    if state is not None:
        for s in slots:
            state[s].zero_()
    at, got = [0, 0, 0], [[], [], []]
    turn, sizes = 0, [1, 1, 3, 2, 1, 17, 40]
    while any(at[k] < lengths[k] for k in range(3)):
        live = [k for k in range(3) if at[k] < lengths[k] and not (turn % 3 == 2 and k == 0)] or [k for k in range(3) if at[k] < lengths[k]]
        new = [min(sizes[turn % len(sizes)] + (k if turn % 2 else 0), lengths[k] - at[k]) for k in live]
        positions = [at[k] + t for k, n in zip(live, new) for t in range(n)]
        proj = torch.cat([rows[k][at[k]:at[k] + n] for k, n in zip(live, new)]).to(dev())
        out = torch.empty_like(proj)
        kernels.short_conv(proj, bx.to(dev()), w.to(dev()), bc.to(dev()), state, out, i32(positions),
                           i32([j for j, n in enumerate(new) for _ in range(n)]), i32(np.cumsum([0] + new)),
                           i32([at[k] for k in live]), i32([slots[k] for k in live]), num_seqs=len(live), single=max(new) == 1)
        first = 0
        for k, n in zip(live, new):
            got[k].append(out[first:first + n])
            first, at[k] = first + n, at[k] + n
        turn += 1
    for k in range(3):
        close(torch.cat(got[k]), want[k], 2e-6 if dtype == torch.float32 else 1e-2, f"request {k}")
    if state is not None:
        assert bool((state[1] == 9.0).all()) and bool((state[4] == 9.0).all())     # other requests' slots untouched


def rglru_part(dtype, hidden, m, tensors):
    from tesseract_b200.config.spec import PartSpec
    from tesseract_b200.parts import MIXERS

    names = {"y": "y", "y_bias": "y.b", "x": "x", "x_bias": "x.b", "conv": "conv", "conv_bias": "conv.b", "r": "ra", "r_bias": "ra.b",
             "i": "ri", "i_bias": "ri.b", "decay": "lam", "o": "o"}
    spec = PartSpec.make("rglru", {"hidden_size": hidden, "width": m["width"], "blocks": m["blocks"], "conv_taps": m["conv"],
                                   "stream": "float32"}, names)
    return MIXERS.get(spec.kind)(spec, {role: tensors[name] for role, name in names.items()}, runtime(dtype))


def rglru_bindings(part, slots=4, fill=5.0):
    from tesseract_b200.parts import CacheBinding

    needs = part.cache_need()
    made = [CacheBinding(group=0, storage=torch.full((slots,) + tuple(need.shape), fill, dtype=torch.float32, device=dev()))
            for need in (needs if isinstance(needs, tuple) else (needs,))]
    return tuple(made) if len(made) > 1 else made[0]


def all_bindings(bindings):
    return bindings if isinstance(bindings, tuple) else (bindings,)


def rglru_case(hidden, width, blocks, taps, T, seed):
    g = torch.Generator().manual_seed(seed)
    size = width // blocks

    def matrix(*shape):
        return torch.randn(*shape, generator=g) * shape[-1] ** -0.5

    tensors = {"y": matrix(width, hidden), "y.b": torch.randn(width, generator=g) * 0.3, "x": matrix(width, hidden),
               "x.b": torch.randn(width, generator=g) * 0.3, "conv": torch.randn(width, taps, generator=g) * 0.6,
               "conv.b": torch.randn(width, generator=g) * 0.3, "ra": matrix(blocks, size, size) * 2.0,
               "ra.b": torch.randn(blocks, size, generator=g), "ri": matrix(blocks, size, size) * 2.0,
               "ri.b": torch.randn(blocks, size, generator=g), "lam": torch.rand(width, generator=g) * 9.0 - 8.0,
               "o": matrix(hidden, width)}
    return {n: bf16(t) for n, t in tensors.items()}, bf16(torch.randn(T, hidden, generator=g))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("hidden,width,blocks,taps", [(40, 24, 1, 1), (42, 33, 3, 5), (64, 256, 2, 3), (48, 192, 3, 4), (32, 40, 5, 2),
                                                      (32, 64, 1, 4)])
def test_recurrent_unit_in_portions_over_used_slots(dtype, hidden, width, blocks, taps):
    T = 500
    m = {"width": width, "blocks": blocks, "conv": taps}
    tensors, h = rglru_case(hidden, width, blocks, taps, T, seed=width + taps)
    want = plain.rglru(m, as_plain(tensors), h.double().numpy())
    noise = 0.0
    if dtype == torch.bfloat16:
        noise = float(np.abs(plain.rglru(m, as_plain(tensors), h.double().numpy(), store=plain.bfloat16) - want).max())
    part = rglru_part(dtype, hidden, m, tensors)
    bindings = rglru_bindings(part)
    sizes = [1, 1, 2, 3, 64, 65, 1, 130, 7, 2, 31, 1, 1, 100]
    for attempt in range(2):                               # the second request finds the first one's state in the slot
        for b in all_bindings(bindings):
            b.storage[1].zero_()                           # what admitting a request does to its slot
        got, at, k = [], 0, 0
        while at < T:
            n = min(sizes[k % len(sizes)], T - at)
            got.append(part.forward(h[at:at + n].to(dtype).to(dev()), step_context(range(at, at + n), [None, None], slot=1), bindings))
            at, k = at + n, k + 1
        close(torch.cat(got), want, TOL[dtype], f"request {attempt}", noise)
        for b in all_bindings(bindings):                   # other requests' slots untouched
            assert bool((b.storage[0] == 5.0).all()) and bool((b.storage[2:] == 5.0).all())
    for b in all_bindings(bindings):
        b.storage[3].zero_()
    whole = part.forward(h.to(dtype).to(dev()), step_context(range(T), [None, None], slot=3), bindings)
    close(whole, want, TOL[dtype], "whole", noise)
    for b in all_bindings(bindings):
        close(b.storage[3], b.storage[1].double().cpu().numpy(), 2e-5 if dtype == torch.float32 else 2e-2, "state after any cut")


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_recurrent_unit_remembers_one_token_over_hundreds(dtype):
    """A channel whose decay is nearly one: log a = -8 r softplus(lam) of some -1e-4 a step, where sqrt(1 - a^2) taken from a
    rounded a would be off by percents.  One token enters the state; 600 tokens later, decoded one by one, the last row's
    output is that token's share."""
    T, hidden, width = 600, 16, 8
    tensors = {"y": torch.zeros(width, hidden), "y.b": torch.full((width,), 2.0), "x": torch.zeros(width, hidden), "x.b": torch.zeros(width),
               "conv": torch.tensor([[0.0, 1.0]]).repeat(width, 1), "conv.b": torch.zeros(width), "ra": torch.zeros(1, width, width),
               "ra.b": torch.full((1, width), -2.0), "ri": torch.zeros(1, width, width), "ri.b": torch.full((1, width), 3.0),
               "lam": torch.linspace(-10.0, -7.0, width), "o": torch.zeros(hidden, width)}
    tensors["x"][:, :width] = torch.eye(width) * 64.0
    tensors["o"][:width] = torch.eye(width)
    tensors = {n: bf16(t) for n, t in tensors.items()}
    h = torch.zeros(T, hidden)
    h[3, :width] = bf16(torch.linspace(1.0, 4.0, width)).float()
    m = {"width": width, "blocks": 1, "conv": 2}
    want = plain.rglru(m, as_plain(tensors), h.double().numpy())
    assert np.abs(want[T - 1, :width]).min() > 0.2, "the case is not sharp"
    part = rglru_part(dtype, hidden, m, tensors)
    bindings = rglru_bindings(part, fill=0.0)
    got = [part.forward(h[:5].to(dtype).to(dev()), step_context(range(5), [None, None]), bindings)]
    for t in range(5, T):
        got.append(part.forward(h[t:t + 1].to(dtype).to(dev()), step_context([t], [None, None]), bindings))
    close(torch.cat(got), want, 2e-5 if dtype == torch.float32 else 1e-2, "decoded")
    whole = part.forward(h.to(dtype).to(dev()), step_context(range(T), [None, None], slot=2), bindings)
    close(whole, want, 2e-5 if dtype == torch.float32 else 1e-2, "whole")


def window_case(heads, kv_heads, d, dv, size, kept, T, seed):
    """Tensors, input rows and marked (row, key) pairs of a window attention in which queries read one slice of the input and
    keys another, so that a marked row's query points along its key and nowhere else."""
    g = torch.Generator().manual_seed(seed)
    width = 2 * d + 8
    tensors = {"q": torch.zeros(heads * d, width), "k": torch.zeros(kv_heads * d, width),
               "v": torch.randn(kv_heads * dv, width, generator=g) * 0.5, "o": torch.randn(width, heads * dv, generator=g) * 0.2,
               "q.b": torch.randn(heads * d, generator=g) * 0.02, "k.b": torch.randn(kv_heads * d, generator=g) * 0.02,
               "v.b": torch.randn(kv_heads * dv, generator=g) * 0.1, "o.b": torch.randn(width, generator=g) * 0.3,
               "r1": torch.rand(heads, generator=g) * 2.0, "r2": torch.rand(heads, generator=g) * 0.5 + 0.02,
               "vmix": torch.tensor(0.375)}
    tensors["r1"][0] = 0.02
    for head in range(heads):
        tensors["q"][head * d:(head + 1) * d, d:2 * d] = torch.eye(d)
    for head in range(kv_heads):
        tensors["k"][head * d:(head + 1) * d, :d] = torch.eye(d)
    tensors = {n: bf16(t) for n, t in tensors.items()}
    h = torch.randn(T, width, generator=g)
    pairs = []

    def mark(row, key):
        if 0 <= key <= row < T and all(row != r for r, _ in pairs):
            pairs.append((row, key))

    # the last kept tokens and the first that is not, hundreds of positions later and right behind the window
    for row, key in ((T - 2, kept - 1), (T - 3, kept), (T - 4, 0), (size + kept - 1, kept - 1), (size + kept, kept), (T - 5, 1)):
        mark(row, key)
    for row, back in zip([T - 1, 300, 257, 256, 200, 150, 64, 48, size - 1, size], [size - 1, size, size - 1, size, 0, 16, size - 1,
                                                                                       size, size - 1, size]):
        mark(row, row - back)
    for row, key in pairs:
        h[row, d:2 * d] = h[key, :d].clone() * 1.5
    m = {"heads": heads, "kv_heads": kv_heads, "dim": d, "vdim": dv, "mask": {"size": size, "keep_first": kept},
         "scale": 6.0 / d ** 0.5, "v_mix": True}
    return tensors, bf16(h).float(), m, pairs


def window_part(dtype, width, m, tensors, value_mix):
    from tesseract_b200.config.spec import PartSpec
    from tesseract_b200.parts import MIXERS

    names = {"q": "q", "k": "k", "v": "v", "o": "o", "q_bias": "q.b", "k_bias": "k.b", "v_bias": "v.b", "o_bias": "o.b",
             "distance_weight": "r1", "distance_rate": "r2"}
    if value_mix == "mix":
        names["value_mix"] = "vmix"
    spec = PartSpec.make(
        "normed_attention",
        {"hidden_size": width, "num_heads": m["heads"], "num_kv_heads": m["kv_heads"], "key_dim": m["dim"], "value_dim": m["vdim"],
         "scale": m["scale"], "bias": True, "output_bias": True, "distance_bias": True, "value_mix": value_mix, "stream": "float32",
         "mask": (("keep_first", m["mask"]["keep_first"]), ("kind", "window"), ("size", m["mask"]["size"]))}, names)
    return MIXERS.get(spec.kind)(spec, {role: tensors[name] for role, name in names.items()}, runtime(dtype))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads,kv_heads,d,dv", [(4, 2, 16, 24), (3, 1, 6, 10), (2, 2, 64, 128), (6, 3, 12, 8), (2, 1, 128, 64), (12, 1, 64, 48)])
@pytest.mark.parametrize("size,kept", [(33, 4), (16, 16), (5, 17), (1, 1), (40, 1), (80, 40), (64, 0)])
def test_a_window_sees_exactly_its_tokens_and_the_kept_ones(dtype, heads, kv_heads, d, dv, size, kept):
    """The part as a prompt, in portions and as decoded rows over scrambled pages full of stale data, against the plain
    function; its values are mixed with another part's of the same tokens.  The case is sharp: a window one position longer
    or shorter, one kept token more or fewer, a forgotten distance bias or unmixed values would change marked rows."""
    from tesseract_b200.parts import CacheBinding

    T, page = 330, 16
    tensors, h, m, pairs = window_case(heads, kv_heads, d, dv, size, kept, T, seed=heads * 100 + d + size)
    first_tensors, first_h, _, _ = window_case(heads, kv_heads, d, dv, size, kept, T, seed=7)
    weights, first_weights = as_plain(tensors), as_plain(first_tensors)
    first_want, first_values = plain.attention(m, first_weights, first_h.double().numpy())
    want, _ = plain.attention(m, weights, h.double().numpy(), first_values)
    marked = [row for row, _ in pairs]

    def changes(other_m=m, other_w=weights, values=first_values):
        other, _ = plain.attention(other_m, other_w, h.double().numpy(), values)
        return float(np.abs(other[marked] - want[marked]).max())

    noticed = []
    for mask in ({"size": size + 1, "keep_first": kept}, {"size": size - 1, "keep_first": kept}, {"size": size, "keep_first": kept + 1},
                 {"size": size, "keep_first": kept - 1}):
        if mask["size"] > 0 and mask["keep_first"] >= 0:
            noticed.append(changes(dict(m, mask=mask)))
    assert max(noticed) > 0.05 and (d < 12 or min(noticed) > 0.03), f"marked rows do not notice a reach one off: {noticed}"
    assert changes(other_w=dict(weights, r1=weights["r1"] * 0.0)) > 0.02, "no row notices the distance bias"
    assert changes(values=None) > 0.05 and changes(values=np.roll(first_values, 1, axis=0)) > 0.02, "no row notices the mixing"
    noise = first_noise = 0.0
    if dtype == torch.bfloat16:
        coarse_first, coarse_values = plain.attention(m, first_weights, first_h.double().numpy(), store=plain.bfloat16)
        coarse, _ = plain.attention(m, weights, h.double().numpy(), coarse_values, store=plain.bfloat16)
        noise, first_noise = float(np.abs(coarse - want).max()), float(np.abs(coarse_first - first_want).max())
    part = window_part(dtype, h.shape[1], m, tensors, "mix")
    first_part = window_part(dtype, h.shape[1], m, first_tensors, "first")
    need = part.cache_need()
    assert need.window == size and need.keep_first == kept and first_part.cache_need() == need
    count = -(-T // page)
    torch.manual_seed(3)
    order = [1 + i for i in torch.randperm(count).tolist()]              # pages taken in scrambled order
    for cut in ("prompt", "decode", "portions", "twos"):
        bindings = [CacheBinding(group=0, storage=torch.full((count + 1, need.page_shape(page)[0]), 7.0, dtype=dtype, device=dev()),
                                 writes=True, page_size=page) for _ in range(2)]                   # stale data
        got, first_got = [], []
        for lo, hi in portions_of(cut, T):
            ctx = step_context(range(lo, hi), [order], page)
            first_got.append(first_part.forward(first_h[lo:hi].to(dtype).to(dev()), ctx, bindings[0]))
            got.append(part.forward(h[lo:hi].to(dtype).to(dev()), ctx, bindings[1]))
        close(torch.cat(first_got), first_want, TOL[dtype], f"first/{cut}", first_noise)
        close(torch.cat(got), want, TOL[dtype], cut, noise)


def test_mixed_values_need_an_earlier_layer_of_the_same_step():
    from tesseract_b200.parts import CacheBinding

    tensors, h, m, _ = window_case(2, 1, 8, 8, 5, 2, 40, seed=1)
    part = window_part(torch.float32, h.shape[1], m, tensors, "mix")
    binding = CacheBinding(group=0, storage=torch.zeros((4, part.cache_need().page_shape(16)[0]), device=dev()), writes=True, page_size=16)
    with pytest.raises(RuntimeError, match="earlier layer's values"):
        part.forward(h[:4].to(dev()), step_context(range(4), [[1, 2, 3]]), binding)


@pytest.mark.parametrize("experts,top,extra", [(8, 3, 1), (6, 2, 0), (5, 1, 11), (1, 1, 1), (64, 6, 16), (3, 3, 0), (200, 8, 1)])
def test_router_weighs_by_each_score_alone(experts, top, extra):
    from tesseract_b200 import kernels

    g = torch.Generator().manual_seed(experts)
    rows = 37
    logits = torch.randn(rows, experts + extra, generator=g) * 3.0
    logits[:, experts:] = 50.0                               # what lies behind the experts is nobody's
    if experts > 3:
        logits[5, 1] = logits[5, 3] = 9.0                    # equal logits: the lower index first
        logits[6, :experts] = torch.linspace(30.0, 60.0, experts)      # scores that all round to one in 32-bit
    ids = torch.empty(rows, top, dtype=torch.int32, device=dev())
    weights = torch.empty(rows, top, device=dev())
    kernels.choose_sigmoid(logits.to(dev()), experts, ids, weights)
    for t in range(rows):
        chosen, want = plain.route({"experts": experts, "top": top}, logits[t, :experts].double().numpy())
        assert ids[t].tolist() == chosen
        close(weights[t], want, 2e-6)


def experts_part(dtype, width, mlp, tensors):
    from tesseract_b200.config.spec import PartSpec
    from tesseract_b200.parts import FEED_FORWARDS

    names = {"router": "router"}
    for e in range(mlp["router"]["experts"]):
        names.update({f"gate.{e}": f"e{e}.gate", f"up.{e}": f"e{e}.up", f"down.{e}": f"e{e}.down"})
    shared = mlp.get("shared")
    if shared:
        names.update({"shared_gate": "shared.gate", "shared_up": "shared.up", "shared_down": "shared.down", "shared_weight": "shared.sg"})
    spec = PartSpec.make("routed_experts", {"hidden_size": width, "num_experts": mlp["router"]["experts"], "top_k": mlp["router"]["top"],
                                            "expert_size": mlp["expert"]["ff"], "shared_size": shared["ff"] if shared else None,
                                            "scoring": "sigmoid", "weigh": "input", "expert_form": "gated_clamped",
                                            "limit": mlp["expert"]["limit"], "shared_limit": shared["limit"] if shared else 0.0,
                                            "slope": 1.702, "gated_shared": bool(shared), "stream": "float32"}, names)
    return FEED_FORWARDS.get(spec.kind)(spec, {role: tensors[name] for role, name in names.items()}, runtime(dtype))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width,experts,top,ff,limit,shared", [(64, 8, 3, 64, 0.6, (128, 0.9)), (96, 5, 2, 32, 1.5, None),
                                                               (42, 4, 4, 10, 0.4, (6, 2.0)), (128, 16, 1, 192, 1.0, (64, 0.3)),
                                                               (48, 1, 1, 16, 0.8, (24, 0.5))])
@pytest.mark.parametrize("rows", [2, 9, 300])
def test_experts_read_their_rows_times_the_weight(dtype, width, experts, top, ff, limit, shared, rows):
    """The routed feed-forward alone at rows whose router decides clearly; both clamps are reached on either side, and
    weighing the outputs instead of the inputs would show."""
    g = torch.Generator().manual_seed(width + rows)
    mlp = {"router": {"experts": experts, "top": top}, "expert": {"ff": ff, "limit": limit}}
    tensors = {"router": torch.randn(experts, width, generator=g) * (0.7 * width ** -0.5)}
    for e in range(experts):
        tensors.update({f"e{e}.gate": torch.randn(ff, width, generator=g) * (2.0 * width ** -0.5),
                        f"e{e}.up": torch.randn(ff, width, generator=g) * (2.0 * width ** -0.5),
                        f"e{e}.down": torch.randn(width, ff, generator=g) * ff ** -0.5})
    if shared:
        mlp["shared"] = {"ff": shared[0], "limit": shared[1]}
        tensors.update({"shared.gate": torch.randn(shared[0], width, generator=g) * (2.0 * width ** -0.5),
                        "shared.up": torch.randn(shared[0], width, generator=g) * (2.0 * width ** -0.5),
                        "shared.down": torch.randn(width, shared[0], generator=g) * shared[0] ** -0.5,
                        "shared.sg": torch.randn(1, width, generator=g) * (2.0 * width ** -0.5)})
    tensors = {n: bf16(t) for n, t in tensors.items()}
    h = bf16(torch.randn(rows, width, generator=g))
    w = as_plain(tensors)
    gaps = {}
    want = plain.expert_feed_forward(mlp, w, h.double().numpy(), close_calls=gaps)
    other = np.zeros_like(want)                              # the weight on the output instead
    for t in range(rows):
        for e, weight in zip(*plain.route(mlp["router"], h[t].double().numpy() @ w["router"].T)):
            other[t] += weight * plain.clamped_expert(w, f"e{e}.", h[t:t + 1].double().numpy(), limit)[0]
    if shared:
        other += plain.clamped_expert(w, "shared.", h.double().numpy(), shared[1]) * plain.sigmoid(h.double().numpy() @ w["shared.sg"].T)
    assert np.abs(other - want).max() > 0.1
    noise = 0.0
    if dtype == torch.bfloat16:
        noise = float(np.abs(plain.expert_feed_forward(mlp, w, h.double().numpy(), store=plain.bfloat16) - want).max())
    part = experts_part(dtype, width, mlp, tensors)
    got = part.forward(h.to(dtype).to(dev()), step_context(range(rows)))
    clear = [t for t in range(rows) if gaps.get(t, 1.0) > 1e-3]
    assert len(clear) >= rows - 2 and got.dtype == torch.float32
    close(got[clear], want[clear], TOL[dtype] if dtype == torch.float32 else 1e-2, "feed-forward", noise)


# ----------------------------------------------------------------------------- whole models


def make_requests(name):
    vocab = TINY_RIRULIX[name]["vocab"]
    return {f"{name}{i}": random_tokens(vocab, n, seed=500 + i) for i, n in enumerate(LENGTHS[name])}


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    from tesseract_b200.weights.random_init import write_random_model

    made = {}

    def get(name):
        if name not in made:
            made[name] = write_random_model(str(tmp_path_factory.mktemp(f"rirulix_{name}")), TINY_RIRULIX[name], seed=23)
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
# A router whose last chosen logit lies this close to the best one not chosen may decide the other way after a rounding to
# bfloat16: such a position's own logits are not compared in bfloat16 (they are in float32).
CLOSE_CALL = 0.15
CLOSE = {}


def plain_rows(folder, requests, dtype):
    """Per request the plain model's logits and, for bfloat16, the most that rounding to bfloat16 alone changes in the
    plain model's logits of that request (at positions without a close routing call)."""
    want, noise = {}, {}
    config, tensors = plain.load_folder(folder)
    for rid, tokens in requests.items():
        key = (folder, tuple(tokens))
        if key not in _PLAIN:
            gaps = {}
            exact = plain.forward(config, tensors, tokens, close_calls=gaps)[0]
            coarse = plain.forward(config, tensors, tokens, store=plain.bfloat16)[0]
            close_rows = {t for t, gap in gaps.items() if gap < CLOSE_CALL}
            steady = [t for t in range(len(tokens)) if t not in close_rows] or [0]
            _PLAIN[key] = (exact, float(np.abs(coarse - exact)[steady].max()), close_rows)
        want[rid], noise[rid], CLOSE[rid] = _PLAIN[key]
    worst = max(noise.values())           # (one model, one noise: a short request is a small sample of it)
    return want, ({rid: worst for rid in noise} if dtype == "bfloat16" else None)


def replay_against_plain(stepper, steps, folder, requests, dtype, what):
    """Replay a trace and compare every wanted row with the plain model.  In bfloat16 a row may also differ by ``NOISE``
    times what rounding to bfloat16 alone changes in the plain model's logits of its request."""
    want, noise = plain_rows(folder, requests, dtype)
    got = replay(stepper, steps)
    if noise is None:
        return compare(got, want, REL[dtype], what)
    assert got, f"{what}: nothing was replayed"
    for (rid, position), row in sorted(got.items(), key=lambda kv: (str(kv[0][0]), kv[0][1])):
        limit = max(REL[dtype] * float(np.abs(want[rid]).max()), NOISE * noise[rid])
        err = float(np.abs(row.astype(np.float64) - want[rid][position]).max())
        if position in CLOSE[rid]:
            assert np.isfinite(row).all()
            continue
        assert np.isfinite(row).all() and err <= limit, (f"{what}: first wrong token is request {rid!r} position "
                                                         f"{position}: max |diff| {err:.3e} > {limit:.3e}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["a", "b", "c", "d", "e"])
def test_every_layer_matches_plain(engines, folders, name, dtype):
    """The stream after every layer against the plain model's."""
    from tesseract_b200.engine import StepEntry
    from tesseract_b200.parts.block import SandwichBlock

    config, tensors = plain.load_folder(folders(name))
    tokens = random_tokens(config["vocab"], 37, seed=8)
    _, want = plain.forward(config, tensors, tokens)
    _, coarse = plain.forward(config, tensors, tokens, store=plain.bfloat16)
    seen = []
    original = SandwichBlock.forward

    def recording(self, stream, ctx, cache, next_norm=None):
        out = original(self, stream, ctx, cache, next_norm=next_norm)
        assert out.update is None and out.residual.dtype == torch.float32
        seen.append(out.residual.double().cpu().numpy())
        return out

    stepper = engines(name, dtype)
    assert stepper.cache.admit("one")
    SandwichBlock.forward = recording
    try:
        stepper.step([StepEntry("one", tokens, [len(tokens) - 1])])
    finally:
        SandwichBlock.forward = original
        stepper.cache.release("one")
    assert len(seen) == len(want) == len(config["layers"])
    for index, got in enumerate(seen):
        limit = REL[dtype] * float(np.abs(want[index]).max())
        if dtype == "bfloat16":       # or what rounding to bfloat16 alone moves in the plain model, NOISE times
            limit = max(limit, NOISE * float(np.abs(coarse[index] - want[index]).max()))
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
    requests.update({f"{name}x{i}": random_tokens(TINY_RIRULIX[name]["vocab"], n, seed=17 + i)
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
    tokens = random_tokens(TINY_RIRULIX[name]["vocab"], 180, seed=77)
    requests = {"long": tokens}
    steps = trace_tail(requests, tail=170)          # ten tokens of prompt, then 170 decoded one by one
    stepper = engines(name, dtype, capacity_tokens=192)
    replay_against_plain(stepper, steps, folders(name), requests, dtype, f"{name}/{dtype}/long decode")
    assert stepper.cache.used_pages() == 0


def test_pages_behind_the_window_go_back_while_the_request_lives_and_kept_ones_stay(engines):
    """Model "b" has windows of 3, 33 and 16 that keep 7, 1 and 16 tokens (pages of 16): a request of 200 tokens never holds
    more than a few pages a group, its first page among them."""
    from tesseract_b200.engine import StepEntry

    stepper = engines("b", "float32", capacity_tokens=208)
    assert stepper.cache.admit("one")
    tokens = random_tokens(TINY_RIRULIX["b"]["vocab"], 200, seed=5)
    paged = [index for index, group in enumerate(stepper.cache.groups) if group.pool is not None]
    assert len(paged) == 3
    for at in range(0, 200, 10):
        stepper.step([StepEntry("one", tokens[at:at + 10], [9])])
        for index in paged:
            held = stepper.cache.pages_of("one", index)
            window = stepper.cache.groups[index].need.window
            first = max(0, at + 10 - window + 1) // 16
            assert set(held) == {0} | set(range(first, -(-(at + 10) // 16)))
    stepper.cache.release("one")
    stepper.cache.check()
    assert stepper.cache.used_pages() == 0


def test_a_request_may_not_pass_the_position_table(engines, folders):
    from tesseract_b200 import LLM, SamplingParams
    from tesseract_b200.engine import StepEntry, StepError

    places = TINY_RIRULIX["d"]["max_positions"]
    stepper = engines("d", "float32", capacity_tokens=256)
    assert stepper.cache.admit("one")
    tokens = random_tokens(TINY_RIRULIX["d"]["vocab"], places + 1, seed=6)
    stepper.step([StepEntry("one", tokens[:places], [places - 1])])
    with pytest.raises(StepError, match="positions"):
        stepper.step([StepEntry("one", tokens[places:], [0])])
    stepper.cache.release("one")
    llm = LLM(folders("d"), dtype="float32", kv_capacity_tokens=512, max_running=2, prefill_chunk_tokens=32)
    out = llm.generate([tokens[:places - 5]], SamplingParams(max_tokens=5, temperature=0.0, ignore_eos=True))[0]
    assert len(out.token_ids) == 5                         # up to the table's last row, and no further
    del llm
    torch.cuda.empty_cache()


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


def test_replay_program_runs_a_rirulix_folder(folders, tmp_path):
    """``bin/trace_run`` picks the model class by ``config.json`` and writes the logits of the wanted places."""
    import json
    import os
    import subprocess
    import sys

    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    config, tensors = plain.load_folder(folders("c"))
    tokens = random_tokens(config["vocab"], 30, seed=9)
    lines = [json.dumps({"step": 0, "entries": [{"id": "a", "tokens": tokens[:20], "want": [0, 19]}], "end": []}),
             json.dumps({"step": 1, "entries": [{"id": "a", "tokens": tokens[20:], "want": [9]}], "end": ["a"]})]
    out = tmp_path / "out"
    done = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", folders("c"), "--dtype",
                           "float32", "--out", str(out), "--max-tokens", "64"], input="\n".join(lines) + "\n",
                          capture_output=True, text=True, timeout=600)
    assert done.returncode == 0, done.stderr[-2000:]
    assert [l for l in done.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1"]
    want = plain.forward(config, tensors, tokens)[0]
    first = np.fromfile(out / "0.f32", dtype="<f4").reshape(2, -1)
    second = np.fromfile(out / "1.f32", dtype="<f4").reshape(1, -1)
    scale = float(np.abs(want).max())
    assert np.abs(first - want[[0, 19]]).max() <= 2e-5 * scale
    assert np.abs(second - want[[29]]).max() <= 2e-5 * scale


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
    assert "kernel plan for Rirulix" in shown.stdout
    for kind in ("normed_attention", "rglru"):
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
        # (drawn models hold ill-conditioned spots, a head whose output the norm per head divides by almost nothing, say:
        # 32-bit rounding shows there at up to 1e-4 of the largest logit; a lost key or a reach one off moves percents)
        compare(replay(stepper, steps), plain_rows(folder, requests, "float32")[0], 1e-4, f"seed {seed}/{name}")
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
