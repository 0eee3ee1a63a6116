"""Tiny Rirulix configurations for the tests: every size differs between them and between their layers, and the values
that make two mechanisms coincide or vanish (one norm group, no kept tokens, more kept tokens than the window holds, a window
of one or longer than any prompt, kv heads as many as heads, one convolution tap, one block of channels, every expert
chosen, one expert, no shared expert, layers that mix no values, a layer without a feed-forward) appear in one layer and not
in the next."""


def attention(heads, kv_heads, dim, vdim, size, keep_first, scale, v_mix):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale,
                                           "mask": {"size": size, "keep_first": keep_first}, "v_mix": v_mix}}


def rglru(width, blocks, conv):
    return {"type": "rglru", "mixer": {"width": width, "blocks": blocks, "conv": conv}}


def moe(experts, top, ff, limit, shared=None):
    out = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff, "limit": limit}}
    if shared is not None:
        out["shared"] = {"ff": shared[0], "limit": shared[1]}
    return out


def layer(mixer, mlp):
    return dict(mixer, mlp=mlp)


def model(width, vocab, groups, eps, max_positions, layers):
    return {"architecture": "Rirulix", "width": width, "vocab": vocab, "norm": {"groups": groups, "eps": eps},
            "max_positions": max_positions, "layers": layers}


TINY_RIRULIX = {
    # three norm groups; a window of 21 keeping 3, then one of 9 keeping none; both mixers
    "a": model(48, 131, 3, 1e-6, 260, [
        layer(attention(4, 2, 12, 20, 21, 3, 0.4, True), moe(6, 2, 16, 0.8, (24, 1.5))),
        layer(rglru(40, 5, 4), moe(4, 1, 20, 2.0, (12, 0.5))),
        layer(attention(2, 1, 16, 40, 9, 0, 0.25, True), None),
        layer(attention(5, 5, 8, 8, 40, 17, 0.5, True), moe(3, 2, 8, 1.0))]),
    # a recurrence first; an attention layer that mixes nothing in front of the first that does; one group; more kept tokens
    # than the window holds; one tap; one block
    "b": model(64, 256, 1, 1e-5, 400, [
        layer(rglru(24, 1, 1), None),
        layer(attention(2, 2, 16, 12, 3, 7, 0.3, False), moe(5, 3, 24, 0.6, (40, 0.7))),
        layer(rglru(96, 3, 2), moe(8, 8, 8, 3.0)),
        layer(attention(6, 3, 8, 16, 33, 1, 0.35, True), moe(2, 1, 64, 1.2, (64, 1.2))),
        layer(attention(4, 1, 24, 48, 16, 16, 0.2, True), moe(7, 2, 16, 0.9, (8, 4.0)))]),
    # widths that are no multiple of four or eight; seven groups; five taps
    "c": model(42, 77, 7, 1e-4, 200, [
        layer(rglru(33, 3, 5), moe(4, 2, 10, 0.5, (6, 0.9))),
        layer(attention(3, 1, 6, 10, 5, 2, 0.5, True), moe(3, 3, 30, 1.1)),
        layer(rglru(22, 11, 3), moe(5, 1, 7, 0.4, (5, 2.5))),
        layer(attention(2, 1, 10, 10, 17, 4, 0.3, True), moe(4, 2, 9, 1.4, (11, 0.3)))]),
    # a window of one that keeps one token; a window longer than any prompt; a single expert; every layer mixes nothing
    "d": model(32, 64, 4, 1e-6, 150, [
        layer(attention(4, 1, 8, 8, 1, 1, 0.35, False), moe(1, 1, 16, 0.7)),
        layer(attention(2, 1, 24, 8, 1000, 5, 0.2, False), moe(1, 1, 12, 5.0, (12, 0.2))),
        layer(rglru(16, 4, 8), moe(6, 1, 8, 1.0, (16, 1.0)))]),
    # head, block and expert sizes of the tensor-core kernels, with prompts long enough for their tiles
    "e": model(64, 90, 2, 1e-6, 700, [
        layer(attention(4, 1, 64, 128, 100, 4, 0.125, True), moe(8, 3, 64, 1.3, (128, 0.8))),
        layer(rglru(256, 2, 3), moe(4, 2, 32, 0.9, (96, 1.1))),
        layer(attention(2, 2, 128, 64, 70, 9, 0.09, True), moe(5, 1, 128, 2.0)),
        layer(rglru(192, 3, 4), None),
        layer(attention(6, 2, 64, 64, 130, 20, 0.125, True), moe(8, 2, 40, 0.7, (48, 0.6)))]),
}

LENGTHS = {"a": [1, 23, 97, 150, 7], "b": [2, 40, 130, 61], "c": [1, 19, 88, 140], "d": [3, 50, 120], "e": [5, 70, 330, 140]}


def random_config(seed: int) -> dict:
    """A Rirulix configuration drawn from ``seed``: two to five layers of the two mixers in any order, with experts or
    without a feed-forward, windows from 1 to 500 positions that keep up to 40."""
    import random

    r = random.Random(seed)
    width = r.choice([24, 40, 64, 66, 96, 136, 200])
    groups = r.choice([g for g in (1, 2, 3, 4, 8, 11) if width % g == 0])
    value_width = r.choice([8, 24, 48, 64, 128])           # what layers that mix values share
    layers = []
    for _ in range(r.randint(2, 5)):
        if r.random() < 0.4:
            blocks = r.choice([1, 2, 3, 4, 8])
            mixer = rglru(blocks * r.choice([3, 8, 16, 20, 64]), blocks, r.choice([1, 2, 3, 4, 4, 6]))
        else:
            v_mix = r.random() < 0.7
            kv_heads = r.choice([1, 2, 4]) if v_mix else r.choice([1, 2, 3])
            vdim = value_width // kv_heads if v_mix else r.choice([4, 10, 16, 48, 64, 128])
            dim = r.choice([6, 8, 12, 16, 24, 32, 64, 64, 128])
            mixer = attention(kv_heads * r.choice([1, 2, 3, 4]), kv_heads, dim, vdim, r.choice([1, 3, 16, 17, 50, 64, 120, 500]),
                              r.choice([0, 1, 2, 5, 16, 19, 40]), r.choice([dim ** -0.5, 0.3, 0.07]), v_mix)
        mlp = None
        if r.random() < 0.8:
            experts = r.randint(1, 9)
            mlp = moe(experts, r.randint(1, min(4, experts)), r.choice([8, 16, 40, 64]), r.choice([0.3, 1.0, 2.5]),
                      r.choice([None, (8, 0.6), (48, 1.5)]))
        layers.append(layer(mixer, mlp))
    return model(width, r.randint(40, 700), groups, r.choice([1e-5, 1e-6]), r.randint(360, 900), layers)
