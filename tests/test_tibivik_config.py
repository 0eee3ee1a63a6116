"""Tibivik without a GPU: reading ``config.json``, the model description, the tensors it expects, the cache manager's handling of
chunks and of the states, and the plain implementation against itself (the recurrences continued from a carried state and
written out by hand, the pair hash, the masks and the mixing of copies at their edges)."""

import copy

import numpy as np
import pytest
import torch

from tesseract_b200.cache.manager import CacheManager
from tesseract_b200.config import ConfigError, load_model_description, resolve_architecture
from tesseract_b200.models.decoder import expected_tensors
from tesseract_b200.parts import PagedKeyValueNeed
from tesseract_b200.weights.loader import WeightError, check_and_load
from tesseract_b200.weights.random_init import random_tensors, write_random_model
from tesseract_b200.weights.safetensors_io import write_safetensors
from tests.plain import tibivik as plain
from tests.tibivik_models import TINY_TIBIVIK, random_config


def test_the_architecture_is_found_by_its_single_name():
    assert resolve_architecture({"architecture": "Tibivik"}).name == "Tibivik"


@pytest.mark.parametrize("name", sorted(TINY_TIBIVIK))
def test_description_and_expected_tensors(tmp_path, name):
    config = TINY_TIBIVIK[name]
    folder = write_random_model(str(tmp_path / name), config, seed=3)
    architecture, typed, spec = load_model_description(folder)
    width, s = config["width"], config["streams"]
    assert architecture.name == "Tibivik" and spec.vocab_size == config["vocab"] and spec.hidden_size == width
    assert [entry.layer for entry in spec.run_order] == plain.run_order(config)
    assert all(entry.cache_of is None and entry.inject is None for entry in spec.run_order)
    assert spec.head.weights["weight"] == spec.embedding.weights["table"] == "embed"
    expected = expected_tensors(spec)
    assert expected["embed"].shape == (config["vocab"], width)
    assert expected["bigram"].shape == (config["embedding"]["bigram"]["buckets"] + 1, width)
    for index, entry in enumerate(config["layers"]):
        prefix, mix, m = f"l{index}.", f"l{index}.mix.", entry["mixer"]
        assert expected[prefix + "hc1.in"].shape == expected[prefix + "hc1.out"].shape == (s,) and expected[prefix + "hc1.mix"].shape == (s, s)
        assert (prefix + "norm2" in expected) == (prefix + "hc2.mix" in expected) == (prefix + "mlp.gate" in expected) == (entry["mlp"] is not None)
        if entry["type"] == "mamba2":
            inner, channels = m["heads"] * m["vdim"], m["heads"] * m["vdim"] + 2 * m["groups"] * m["state"]
            assert expected[mix + "in"].shape == (inner + channels + m["heads"], width)
            assert expected[mix + "conv"].shape == (channels, m["conv"]) and expected[mix + "conv.b"].shape == (channels,)
            assert expected[mix + "norm"].shape == (inner,) and expected[mix + "o"].shape == (width, inner)
            continue
        left, right = m["left"], m["right"]
        assert expected[mix + "left.q"].shape == (left["heads"] * left["dim"], width)
        assert expected[mix + "left.sink"].shape == (left["heads"],)
        assert expected[mix + "right.o"].shape == (width, right["heads"] * right["vdim"])
        if entry["type"] == "parallel":
            assert mix + "left.v" not in expected and mix + "left.q.b" not in expected
            assert expected[mix + "left.k.norm"].shape == (left["kv_heads"] * left["dim"],)
            assert expected[mix + "right.norm"].shape == (right["heads"] * right["vdim"],)
            assert expected[mix + "right.i"].shape == expected[mix + "right.f"].shape == (right["heads"], width)
        else:
            assert expected[mix + "left.v.b"].shape == (left["kv_heads"] * left["vdim"],)
            assert expected[mix + "left.g"].shape == (left["heads"], width)
            assert expected[mix + "right.norm"].shape == (right["vdim"],)
            assert expected[mix + "right.k.conv"].shape == (right["kv_heads"] * right["dim"], right["conv"])
    # the plain model reads the same folder
    tokens = [1, 2, 3, 4, 5, 6, 7]
    logits, streams = plain.forward(*plain.load_folder(folder), tokens)
    assert logits.shape == (7, config["vocab"]) and len(streams) == len(spec.run_order) and np.isfinite(logits).all()


def test_tensors_of_an_absent_feed_forward_are_allowed_and_other_strangers_are_not(tmp_path):
    config = TINY_TIBIVIK["b"]                             # layers 1 and 2 have no feed-forward
    tensors = random_tensors(config, seed=2)
    tensors.update({"l1.norm2": torch.ones(64), "l1.hc2.in": torch.ones(1), "l2.hc2.mix": torch.ones(1, 1), "l2.hc2.out": torch.ones(1)})
    folder = write_random_model(str(tmp_path / "m"), config, seed=2)
    write_safetensors(folder + "/model.safetensors", tensors)
    architecture, typed, spec = load_model_description(folder)
    loaded = check_and_load(folder, expected_tensors(spec), architecture.ignorable_tensors(typed))
    assert "l1.norm2" not in loaded
    tensors["l1.mix.left.v"] = torch.ones(32, 64)          # (its values are its keys)
    write_safetensors(folder + "/model.safetensors", tensors)
    with pytest.raises(WeightError, match="l1.mix.left.v"):
        check_and_load(folder, expected_tensors(spec), architecture.ignorable_tensors(typed))


def changed(path, value):
    def apply(config):
        at = config
        for key in path[:-1]:
            at = at[key]
        if value is KeyError:
            del at[path[-1]]
        else:
            at[path[-1]] = value
    return apply


@pytest.mark.parametrize("change,message", [
    (changed(("layers", 0, "mixer", "groups"), 4), "multiple of groups"),
    (changed(("layers", 0, "mixer", "norm_groups"), 7), "norm_groups must divide"),
    (changed(("layers", 0, "mixer", "conv"), 0), "conv must be positive"),
    (changed(("layers", 1, "mixer", "left", "kv_heads"), 3), "multiple of kv_heads"),
    (changed(("layers", 1, "mixer", "left", "vdim"), 20), "values that are keys"),
    (changed(("layers", 1, "mixer", "left", "rot", "dims"), 7), "even"),
    (changed(("layers", 1, "mixer", "left", "rot", "dims"), 26), "at most the head"),
    (changed(("layers", 1, "mixer", "left", "mask", "size"), 0), "size must be positive"),
    (changed(("layers", 1, "mixer", "right", "gate_cap"), 0.0), "gate_cap must be positive"),
    (changed(("layers", 1, "mixer", "left_scale"), KeyError), "left_scale"),
    (changed(("layers", 2, "mixer", "right", "kv_heads"), 4), "multiple of kv_heads"),
    (changed(("layers", 2, "mixer", "left", "mask"), KeyError), "mask"),
    (changed(("layers", 0, "mlp", "kind"), "moe"), "unknown kind"),
    (changed(("layers", 0, "type"), "mamba"), "unknown type"),
    (changed(("loop", "stop"), 5), "start <= stop"),
    (changed(("loop", "times"), 0), "times >= 1"),
    (changed(("embedding", "bigram", "buckets"), 0), "buckets must be positive"),
    (changed(("streams",), 0), "streams must be positive"),
    (changed(("norm", "eps"), 0.0), "eps must be positive"),
    (changed(("layers",), []), "must not be empty"),
])
def test_bad_configurations_are_refused(change, message):
    config = copy.deepcopy(TINY_TIBIVIK["a"])
    change(config)
    with pytest.raises(ConfigError) as caught:
        resolve_architecture(config).read_config(config)
    assert message in str(caught.value)


@pytest.mark.parametrize("seed", range(1, 25))
def test_random_configurations_describe_and_write(tmp_path, seed):
    config = random_config(seed)
    folder = write_random_model(str(tmp_path / "m"), config, seed=seed)
    _, _, spec = load_model_description(folder)
    assert [entry.layer for entry in spec.run_order] == plain.run_order(config)
    _, tensors = plain.load_folder(folder)
    assert set(tensors) == set(expected_tensors(spec))


# ----------------------------------------------------------------------------- the plain functions


def test_the_plain_pair_rows_hash_the_token_in_front():
    config = {"embedding": {"bigram": {"buckets": 10, "mul_prev": 7, "mul_cur": 3}}}
    assert plain.bigram_rows(config, [4, 5, 5, 0]) == [10, (4 * 7 + 5 * 3) % 10, (5 * 7 + 5 * 3) % 10, (5 * 7) % 10]
    assert plain.bigram_rows(config, [0]) == [10]


def test_the_plain_masks_at_their_edges():
    seen = plain.window_mask(6, 3)
    assert seen[5].tolist() == [False, False, False, True, True, True] and seen[1].tolist() == [True, True] + [False] * 4
    seen = plain.chunk_mask(7, 3)
    assert seen[3].tolist() == [False] * 3 + [True] + [False] * 3 and seen[5, 3:6].all() and seen[5].sum() == 3 and seen[6].sum() == 1


def test_a_sink_takes_its_share_and_is_not_scaled():
    q, k, v = np.full((1, 1, 1), 2.0), np.full((1, 1, 1), 3.0), np.full((1, 1, 1), 5.0)
    out = plain.attend(q, k, v, np.ones((1, 1), bool), 0.5, [1.0])
    assert out[0, 0, 0] == pytest.approx(5.0 * np.exp(3.0) / (np.exp(3.0) + np.exp(1.0)))
    assert np.isfinite(plain.attend(q, k, v, np.ones((1, 1), bool), 0.5, [800.0])).all()


@pytest.mark.parametrize("kind", ["memory", "delta", "space"])
def test_the_plain_recurrences_continue_from_a_carried_state(kind):
    rng = np.random.default_rng(4)
    T, H, d, dv, cut = 40, 3, 5, 4, 17
    q, k, v = rng.normal(size=(T, H, d)), rng.normal(size=(T, H, d)), rng.normal(size=(T, H, dv))
    a, b = rng.normal(size=(T, H)), rng.uniform(0.2, 0.9, size=(T, H))

    def run(part, state=None):
        if kind == "memory":
            return plain.matrix_memory(q[part], k[part], v[part], 3 * a[part], np.log(b[part]), state)
        if kind == "delta":
            return plain.gated_delta(plain.unit(q[part]), plain.unit(k[part]), v[part], plain.sigmoid(a[part]), b[part], state)
        return plain.state_space(v[part], k[part], q[part], b[part], a[0], a[1], state)

    whole, last = run(slice(None))
    first, carried = run(slice(0, cut))
    second, final = run(slice(cut, None), carried)
    assert np.allclose(np.concatenate([first, second]), whole, atol=1e-12)
    for one, other in zip(final if kind == "memory" else [final], last if kind == "memory" else [last]):
        assert np.allclose(one, other, atol=1e-12)


def test_the_plain_recurrences_by_hand_on_two_tokens():
    q, k, v = np.array([[[1.0]], [[2.0]]]), np.array([[[3.0]], [[-1.0]]]), np.array([[[5.0]], [[7.0]]])
    # the running maximum starts at zero: a first input gate below zero does not become it
    out, (S, n, m) = plain.matrix_memory(q, k, v, np.array([[-2.0], [1.0]]), np.array([[-0.5], [-0.25]]))
    m0 = -0.5
    S0, n0 = np.exp(-1.5) * 15.0, np.exp(-1.5) * 3.0
    assert out[0, 0, 0] == pytest.approx(S0 / (max(n0, np.exp(0.5)) + 1e-6))
    keep, write = np.exp(-0.25 + m0 - 1.0), 1.0
    assert S[0, 0, 0] == pytest.approx(keep * S0 - 7.0 * write) and n[0, 0] == pytest.approx(keep * n0 - 1.0) and m[0] == 1.0
    assert out[1, 0, 0] == pytest.approx(2 * S[0, 0, 0] / (max(abs(2 * n[0, 0]), np.exp(-1.0)) + 1e-6))
    out, S = plain.gated_delta(q, k, v, np.array([[0.5], [0.25]]), np.array([[0.9], [0.8]]))
    s0 = 3.0 * 0.5 * 5.0
    s1 = 0.8 * s0 - 0.25 * (7.0 + 0.8 * s0)
    assert out[:, 0, 0].tolist() == pytest.approx([s0, 2.0 * s1]) and S[0, 0, 0] == pytest.approx(s1)
    out, S = plain.state_space(v, k, q, np.array([[0.5], [2.0]]), np.array([0.0]), np.array([10.0]))
    s0 = 0.5 * 15.0
    assert out[:, 0, 0].tolist() == pytest.approx([s0 + 50.0, 2.0 * (np.exp(-2.0) * s0 - 14.0) + 70.0])


def test_copies_are_mixed_from_the_old_ones_and_the_matrix_reads_from_then_to():
    streams = np.array([[[1.0]], [[10.0]]])
    w = {"hc1.in": np.array([2.0, 3.0]), "hc1.out": np.array([1.0, -1.0]), "hc1.mix": np.array([[0.5, 7.0], [0.0, 1.0]])}
    seen = []
    out = plain.connect(streams, w, 1, lambda u: seen.append(u.copy()) or u * 0 + 100.0)
    assert seen[0][0, 0] == 32.0 and out[:, 0, 0].tolist() == [0.5 + 100.0, 7.0 + 10.0 - 100.0]


# ----------------------------------------------------------------------------- the cache manager


def test_pages_of_earlier_chunks_go_back_and_every_walk_has_a_state_of_its_own():
    from tesseract_b200.parts import StateNeed

    chunk = PagedKeyValueNeed(num_kv_heads=2, key_dim=8, value_dim=4, block=40)
    state = StateNeed((3, 4, 8), torch.float32)
    token = StateNeed((1,), torch.int32)
    cache = CacheManager([(chunk, state), (chunk, state), token], [None] * 3, num_pages=64, page_size=16, max_requests=2,
                         dtype=torch.float32, device="cpu", max_step_tokens=10)
    assert [len(g.entries) for g in cache.groups] == [2, 2, 1]       # two walks share a group and have storage of their own
    first, second = cache.bindings[0][1].storage, cache.bindings[1][1].storage
    assert first.data_ptr() != second.data_ptr() and first.shape == (3, 3, 4, 8)
    assert cache.bindings[2].storage.dtype == torch.int32
    first.fill_(5.0)
    cache.bindings[2].storage.fill_(9)
    assert cache.admit("r")
    slot = cache.slot("r")
    assert not first[slot].any() and not cache.bindings[2].storage[slot].any()
    for step in range(20):
        cache.extend("r", 10)
        cache.commit("r", 10)
        length = cache.length("r")
        live = set(range((length // 40) * 40 // 16, -(-length // 16)))
        assert set(cache.pages_of("r", 0)) == live
        cache.check()
    cache.release("r")
    assert cache.used_pages() == 0
