"""Rirulix without a GPU: reading ``config.json``, the model description, the tensors it expects, the cache manager's handling
of a window that keeps the first tokens, and the plain implementation against itself (the recurrence continued from a
carried state, the convolution, the router and the experts at their edges)."""

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
from tests.plain import rirulix as plain
from tests.rirulix_models import TINY_RIRULIX, random_config


def test_the_architecture_is_found_by_its_single_name():
    assert resolve_architecture({"architecture": "Rirulix"}).name == "Rirulix"


@pytest.mark.parametrize("name", sorted(TINY_RIRULIX))
def test_description_and_expected_tensors(tmp_path, name):
    config = TINY_RIRULIX[name]
    folder = write_random_model(str(tmp_path / name), config, seed=3)
    architecture, typed, spec = load_model_description(folder)
    assert architecture.name == "Rirulix" and spec.vocab_size == config["vocab"] and spec.hidden_size == config["width"]
    assert spec.max_positions == config["max_positions"]
    assert len(spec.layers) == len(config["layers"]) == len(spec.run_order)
    expected = expected_tensors(spec)
    width = config["width"]
    assert expected["embed"].shape == expected["head"].shape == (config["vocab"], width)
    assert expected["pos"].shape == (config["max_positions"], width) and expected["embed.norm"].shape == (width,)
    mixing = [i for i, layer in enumerate(config["layers"]) if layer["mixer"].get("v_mix")]
    for index, layer in enumerate(config["layers"]):
        prefix, mix, m = f"l{index}.", f"l{index}.mix.", layer["mixer"]
        assert spec.layers[index].block == "sandwich"
        assert all(norm.params["groups"] == config["norm"]["groups"] for norm in spec.layers[index].norms.values())
        assert (prefix + "norm2" in expected) == (prefix + "norm2b" in expected) == (layer["mlp"] is not None)
        if layer["type"] == "rglru":
            size = m["width"] // m["blocks"]
            assert expected[mix + "conv"].shape == (m["width"], m["conv"]) and expected[mix + "lam"].shape == (m["width"],)
            assert expected[mix + "ra"].shape == expected[mix + "ri"].shape == (m["blocks"], size, size)
            assert expected[mix + "ra.b"].shape == (m["blocks"], size) and expected[mix + "o"].shape == (width, m["width"])
        else:
            assert expected[mix + "q"].shape == (m["heads"] * m["dim"], width) and expected[mix + "o.b"].shape == (width,)
            assert expected[mix + "v"].shape == (m["kv_heads"] * m["vdim"], width)
            assert expected[mix + "r1"].shape == expected[mix + "r2"].shape == (m["heads"],)
            assert (mix + "vmix" in expected) == (index in mixing[1:])
            mask = dict(spec.layers[index].mixer.params["mask"])
            assert mask["size"] == m["mask"]["size"] and mask["keep_first"] == m["mask"]["keep_first"]
        mlp = layer["mlp"]
        if mlp:
            assert expected[prefix + "mlp.router"].shape == (mlp["router"]["experts"], width)
            for e in range(mlp["router"]["experts"]):
                assert expected[f"{prefix}mlp.e{e}.gate"].shape == expected[f"{prefix}mlp.e{e}.up"].shape == (mlp["expert"]["ff"], width)
                assert expected[f"{prefix}mlp.e{e}.down"].shape == (width, mlp["expert"]["ff"])
            assert (prefix + "mlp.shared.sg" in expected) == ("shared" in mlp)
    # the plain model reads the same folder
    tokens = [1, 2, 3, 4, 5, 6, 7]
    logits, streams = plain.forward(*plain.load_folder(folder), tokens)
    assert logits.shape == (7, config["vocab"]) and len(streams) == len(config["layers"]) and np.isfinite(logits).all()


def test_unused_mixing_numbers_are_allowed_and_other_strangers_are_not(tmp_path):
    """A checkpoint may hold the mixing number of a layer that mixes nothing (the first with v_mix, or one without)."""
    config = TINY_RIRULIX["b"]
    tensors = random_tensors(config, seed=2)
    assert "l4.mix.vmix" in tensors and "l3.mix.vmix" not in tensors
    tensors.update({"l1.mix.vmix": torch.tensor(0.5), "l3.mix.vmix": torch.tensor(0.5), "l0.norm2": torch.ones(64)})
    folder = write_random_model(str(tmp_path / "m"), config, seed=2)
    write_safetensors(folder + "/model.safetensors", tensors)
    architecture, typed, spec = load_model_description(folder)
    loaded = check_and_load(folder, expected_tensors(spec), architecture.ignorable_tensors(typed))
    assert "l3.mix.vmix" not in loaded and loaded["l4.mix.vmix"].shape == ()
    tensors["l0.mix.vmix"] = torch.tensor(0.5)             # (layer 0 is a recurrence)
    write_safetensors(folder + "/model.safetensors", tensors)
    with pytest.raises(WeightError, match="l0.mix.vmix"):
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
    (changed(("layers", 0, "mixer", "kv_heads"), 3), "multiple of kv_heads"),
    (changed(("layers", 0, "mixer", "mask", "size"), 0), "size must be positive"),
    (changed(("layers", 0, "mixer", "mask", "keep_first"), -1), "keep_first must not be negative"),
    (changed(("layers", 0, "mixer", "mask"), KeyError), "mask"),
    (changed(("layers", 0, "mixer", "scale"), KeyError), "scale"),
    (changed(("layers", 0, "mixer", "v_mix"), 1), "true or false"),
    (changed(("layers", 2, "mixer", "vdim"), 20), "share one value width"),
    (changed(("layers", 1, "mixer", "blocks"), 3), "multiple of blocks"),
    (changed(("layers", 1, "mixer", "conv"), 0), "conv must be positive"),
    (changed(("layers", 0, "mlp", "router", "top"), 7), "top must be at most experts"),
    (changed(("layers", 0, "mlp", "expert", "limit"), 0.0), "limit must be positive"),
    (changed(("layers", 0, "mlp", "shared", "limit"), KeyError), "limit"),
    (changed(("layers", 0, "mlp", "kind"), "dense"), "unknown kind"),
    (changed(("layers", 0, "type"), "mingru"), "unknown type"),
    (changed(("norm", "eps"), 0.0), "eps must be positive"),
    (changed(("norm", "groups"), 5), "groups must divide"),
    (changed(("max_positions",), 0), "must be positive"),
    (changed(("layers",), []), "layers not empty"),
])
def test_bad_configurations_are_refused(change, message):
    config = copy.deepcopy(TINY_RIRULIX["a"])
    change(config)
    with pytest.raises(ConfigError) as caught:
        resolve_architecture(config).read_config(config)
    assert message in str(caught.value)


@pytest.mark.parametrize("seed", range(1, 25))
def test_random_configurations_describe_and_write(tmp_path, seed):
    config = random_config(seed)
    folder = write_random_model(str(tmp_path / "m"), config, seed=seed)
    _, _, spec = load_model_description(folder)
    assert len(spec.layers) == len(config["layers"])
    loaded_config, tensors = plain.load_folder(folder)
    assert set(tensors) == set(expected_tensors(spec))


def test_the_plain_recurrence_continues_from_a_carried_state():
    rng = np.random.default_rng(4)
    u, r, i = rng.normal(size=(40, 6)), rng.uniform(size=(40, 6)), rng.uniform(size=(40, 6))
    lam = rng.uniform(-6, 1, size=6)
    whole, state = plain.gated_linear_recurrence(u, r, i, lam)
    first, carried = plain.gated_linear_recurrence(u[:17], r[:17], i[:17], lam)
    second, final = plain.gated_linear_recurrence(u[17:], r[17:], i[17:], lam, state=carried)
    assert np.allclose(np.concatenate([first, second]), whole, atol=1e-12) and np.allclose(final, state, atol=1e-12)
    # written out by hand for the first two tokens of one channel
    a = np.exp(-8.0 * r[:2, 0] * np.log1p(np.exp(lam[0])))
    s0 = np.sqrt(1 - a[0] ** 2) * i[0, 0] * u[0, 0]
    assert whole[0, 0] == pytest.approx(s0) and whole[1, 0] == pytest.approx(a[1] * s0 + np.sqrt(1 - a[1] ** 2) * i[1, 0] * u[1, 0])


def test_the_plain_convolution_puts_its_last_tap_on_the_row_itself():
    u = np.arange(1.0, 6.0)[:, None]
    taps, bias = np.array([[100.0, 10.0, 1.0]]), np.array([0.5])
    assert plain.causal_convolution(u, taps, bias)[:, 0].tolist() == [1.5, 12.5, 123.5, 234.5, 345.5]


def test_the_plain_router_and_experts_at_their_edges():
    router = {"experts": 4, "top": 2}
    gaps = []
    chosen, weights = plain.route(router, np.array([0.0, 2.0, -1.0, 1.0]), gaps)
    assert chosen == [1, 3] and np.allclose(weights, plain.sigmoid(np.array([2.0, 1.0]))) and gaps == [1.0]
    chosen, _ = plain.route(router, np.zeros(4))
    assert chosen == [0, 1]                                # equal scores: the lowest indices
    # an expert of one hidden number: the gate is clamped from above only, up from both sides, and one is added
    w = {"e0.gate": np.array([[1.0]]), "e0.up": np.array([[-1.0]]), "e0.down": np.array([[1.0]])}
    for h, limit in ((5.0, 2.0), (-5.0, 2.0), (0.5, 2.0)):
        g, u = min(h, limit), max(min(-h, limit), -limit)
        want = g / (1.0 + np.exp(-1.702 * g)) * (u + 1.0)
        assert plain.clamped_expert(w, "e0.", np.array([[h]]), limit)[0, 0] == pytest.approx(want)


def test_pages_of_kept_tokens_stay_while_the_window_moves_on():
    """A window of 40 that keeps the first 19 positions, pages of 16: the first two pages stay, the others come and go."""
    need = PagedKeyValueNeed(num_kv_heads=2, key_dim=8, value_dim=4, window=40, keep_first=19)
    other = PagedKeyValueNeed(num_kv_heads=2, key_dim=8, value_dim=4, window=40)
    cache = CacheManager([need, other], [None, None], num_pages=64, page_size=16, max_requests=2, dtype=torch.float32,
                         device="cpu", allocate_storage=False, max_step_tokens=10)
    assert len(cache.groups) == 2                          # the two needs differ in what they keep
    assert cache.pages_for(cache.groups[0], 1000) == cache.pages_for(cache.groups[1], 1000) + 2
    assert cache.admit("r", reserve_tokens=1000)
    first_pages = None
    for step in range(100):
        cache.extend("r", 10)
        kept = cache.pages_of("r", 0)
        if first_pages is None:
            first_pages = {0: kept[0]}
        if step == 3:
            first_pages = {0: kept[0], 1: kept[1]}
        assert all(kept[logical] == page for logical, page in first_pages.items())
        assert len(kept) <= cache.pages_for(cache.groups[0], 1000)
        cache.commit("r", 10)
        length = cache.length("r")
        live = set(range(max(0, length - 39) // 16, -(-length // 16)))
        assert set(cache.pages_of("r", 0)) == live | set(range(min(2, -(-length // 16))))
        assert set(cache.pages_of("r", 1)) == live
        table = cache.block_table_rows(0, [cache.slot("r")], 64)[0]
        assert all((table[logical] != 0) == (logical in cache.pages_of("r", 0)) for logical in range(64))
        cache.check()
    cache.release("r")
    cache.check()
    assert cache.used_pages() == 0
