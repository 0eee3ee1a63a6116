"""Tiny Tibivik configurations for the tests: every size differs between them and between their layers, and the values that make
two mechanisms coincide or vanish (one copy of the stream, one bucket, one group or norm group, kv heads as many as heads, one
convolution tap, a window or a chunk of one or longer than any prompt, a rotation over the whole head or none, equal or zero scales
of the two sides, a layer without a feed-forward, a loop that runs once or covers the last layers) appear in one layer and not in
the next."""


def mamba2(heads, vdim, state, groups, norm_groups, conv):
    return {"type": "mamba2", "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "norm_groups": norm_groups,
                                        "conv": conv}}


def window(heads, kv_heads, dim, size, scale, rot=None):
    out = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "mask": {"size": size}, "scale": scale}
    if rot is not None:
        out["rot"] = {"dims": rot[0], "base": rot[1]}
    return out


def memory(heads, dim, vdim, gate_cap):
    return {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": gate_cap}


def chunks(heads, kv_heads, dim, vdim, size, scale):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": size}, "scale": scale}


def delta(heads, kv_heads, dim, vdim, conv):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}


def parallel(left, right, left_scale, right_scale):
    kind = "parallel" if "gate_cap" in right else "parallel_2"
    return {"type": kind, "mixer": {"left": left, "right": right, "left_scale": left_scale, "right_scale": right_scale}}


def layer(mixer, ff):
    return dict(mixer, mlp=None if ff is None else {"kind": "dense", "ff": ff})


def model(width, vocab, streams, eps, bigram, layers, loop=None):
    out = {"architecture": "Tibivik", "width": width, "vocab": vocab, "streams": streams, "norm": {"eps": eps},
           "embedding": {"bigram": dict(zip(("buckets", "mul_prev", "mul_cur"), bigram))}, "layers": layers}
    if loop is not None:
        out["loop"] = dict(zip(("start", "stop", "times"), loop))
    return out


TINY_TIBIVIK = {
    # all three mixers; two groups, three norm groups; two walks over the middle layers
    "a": model(48, 131, 3, 1e-3, (61, 7, 30), [
        layer(mamba2(6, 12, 20, 2, 3, 3), 72),
        layer(parallel(window(4, 2, 24, 21, 0.3, (12, 900.0)), memory(3, 16, 20, 9.0), 0.7, 1.3), 40),
        layer(parallel(chunks(6, 2, 16, 12, 25, 0.25), delta(6, 3, 12, 20, 3), 1.1, 0.6), None),
        layer(mamba2(4, 16, 36, 4, 1, 2), 56)], (1, 3, 2)),
    # one copy of the stream, one tap, no rotation, kv heads as many as heads, a window of one, a chunk of one; no loop
    "b": model(64, 256, 1, 1e-6, (1, 3, 5), [
        layer(parallel(chunks(3, 3, 8, 32, 1, 0.35), delta(2, 2, 40, 8, 1), 0.5, 0.5), 32),
        layer(parallel(window(2, 2, 16, 1, 0.25), memory(1, 72, 40, 30.0), 1.0, 2.0), None),
        layer(mamba2(1, 64, 8, 1, 4, 1), None),
        layer(parallel(chunks(8, 1, 24, 16, 17, 0.2), delta(4, 1, 8, 48, 5), 1.4, 0.9), 128)]),
    # sizes that are no multiple of four or eight; five copies; four norm groups; a rotation over the whole head; more taps
    "c": model(42, 77, 5, 2e-2, (97, 101, 12345), [
        layer(parallel(window(3, 1, 10, 33, 0.4, (10, 77.0)), memory(2, 7, 9, 4.0), 1.2, 0.8), 30),
        layer(mamba2(6, 6, 13, 3, 4, 5), 42),
        layer(parallel(chunks(5, 5, 6, 10, 13, 0.5), delta(6, 2, 5, 11, 6), 0.9, 1.5), 10)], (0, 2, 3)),
    # windows and chunks longer than any prompt, one side only, states of more than 64 rows, seven copies; the loop covers the end
    "d": model(36, 64, 7, 1e-6, (500, 499, 498), [
        layer(mamba2(2, 20, 100, 1, 2, 4), 20),
        layer(parallel(window(4, 1, 8, 5000, 0.35, (4, 50000.0)), memory(4, 100, 33, 15.0), 1.0, 0.0), 24),
        layer(parallel(chunks(2, 1, 24, 8, 4000, 0.2), delta(2, 1, 136, 12, 2), 0.0, 1.0), None)], (1, 3, 1)),
    # head sizes of the tensor-core attention, two copies, states up to 300 rows, prompts long enough for its tiles
    "e": model(64, 90, 2, 1e-6, (256, 11, 13), [
        layer(parallel(window(4, 2, 64, 100, 0.125, (32, 10000.0)), memory(2, 64, 64, 7.0), 0.8, 1.2), 64),
        layer(mamba2(8, 24, 300, 2, 8, 4), 48),
        layer(parallel(chunks(6, 3, 128, 64, 130, 0.09), delta(4, 2, 200, 32, 4), 1.3, 0.7), 96),
        layer(parallel(window(2, 1, 128, 70, 0.09, (64, 5000.0)), memory(1, 24, 130, 11.0), 0.9, 1.0), None)], (2, 4, 2)),
}

LENGTHS = {"a": [1, 23, 97, 150, 7], "b": [2, 40, 130, 61], "c": [1, 19, 88, 140], "d": [3, 50, 120], "e": [5, 70, 330, 140]}


def random_config(seed: int) -> dict:
    """A Tibivik configuration drawn from ``seed``: two to five layers of the three mixers in any order, some walked several
    times, windows and chunks from 1 to 500 positions.  (Norms over a handful of numbers, or with a tiny eps, amplify whatever
    rounding a recurrence leaves: the sizes here keep a fault larger than that.)"""
    import random

    r = random.Random(seed)
    layers = []
    for _ in range(r.randint(2, 5)):
        kind = r.choice(["mamba2", "parallel", "parallel_2"])
        scales = (r.choice([0.5, 1.0, 1.3]), r.choice([0.7, 1.0, 1.6]))
        size = r.choice([1, 3, 16, 17, 50, 64, 120, 500])
        if kind == "mamba2":
            groups = r.choice([1, 1, 2, 3])
            heads, vdim = groups * r.choice([1, 2, 4]), r.choice([17, 24, 30, 32, 48])
            norm_groups = r.choice([n for n in (1, 1, 2, heads) if heads * vdim % n == 0])
            mixer = mamba2(heads, vdim, r.choice([5, 16, 32, 48, 80, 130]), groups, norm_groups, r.choice([1, 2, 3, 4, 4, 6]))
        elif kind == "parallel":
            kv_heads, dim = r.choice([1, 2, 3]), r.choice([6, 8, 16, 32, 64, 64, 128])
            rot = None if r.random() < 0.2 else (r.choice([n for n in (2, 4, 6, 8, 16, dim) if n <= dim]), r.choice([50.0, 1e4, 3e5]))
            mixer = parallel(window(kv_heads * r.choice([1, 2, 3, 4]), kv_heads, dim, size, r.choice([dim ** -0.5, 0.3]), rot),
                             memory(r.randint(1, 4), r.choice([6, 16, 32, 48, 96]), r.choice([19, 24, 32, 64]), r.choice([3.0, 8.0, 20.0])),
                             *scales)
        else:
            kv_heads, heads = r.choice([1, 2, 3]), r.choice([1, 2, 4])
            mixer = parallel(chunks(kv_heads * r.choice([1, 2, 4]), kv_heads, r.choice([6, 8, 24, 64, 128]), r.choice([4, 10, 48, 64]), size,
                                    r.choice([0.1, 0.3])),
                             delta(heads * r.choice([1, 2, 3]), heads, r.choice([6, 16, 32, 64, 100]), r.choice([21, 24, 32, 64]),
                                   r.choice([1, 2, 3, 4, 4, 5])), *scales)
        layers.append(layer(mixer, r.choice([None, 16, 40, 64, 100])))
    loop = None
    if r.random() < 0.7:
        start = r.randrange(len(layers))
        loop = (start, r.randint(start + 1, len(layers)), r.choice([1, 2, 3]))
    buckets = r.choice([1, 7, 100, 509, 4096])
    return model(r.choice([24, 40, 64, 66, 96, 136, 200]), r.randint(40, 700), r.choice([1, 2, 3, 4, 4, 6, 8, 9]), r.choice([1e-3, 1e-4]),
                 (buckets, r.randint(1, 5000), r.randint(1, 5000)), layers, loop)
