"""Host-side pieces of the Kofipel design: configuration, description, tensor names, loops, sizes that only a tensor's shape
gives, cache needs and slots, pages that hold a window's kept first keys, the plain implementation's pieces against closed
forms."""
import math

import pytest
import torch

from plain import kofipel_plain as plain


def small_config(**changes):
    attention = {"heads": 6, "kv_heads": 2, "dim": 8, "vdim": 8, "scale": 0.3, "softcap": 12.0,
                 "mask": {"size": 9, "keep_first": 5}, "rot": {"base": 500.0, "dims": 4}}
    memory = {"heads": 4, "kv_heads": 2, "dim": 10, "vdim": 6, "conv": 3, "decay_rank": 3, "gate_rank": 5}
    config = {
        "architecture": "Kofipel", "vocab": 97, "width": 48, "norm": {"eps": 1e-5}, "canon": {"taps": 3}, "token_side": {"dim": 7},
        "loop": {"start": 1, "stop": 3, "times": 3},
        "layers": [{"type": "channel_delta", "mixer": memory, "mlp": None},
                   {"type": "attention", "mixer": attention, "mlp": {"kind": "dense", "ff": 56}},
                   {"type": "channel_delta", "mixer": memory, "mlp": {"kind": "dense", "ff": 40}},
                   {"type": "attention", "mixer": attention, "mlp": {"kind": "dense", "ff": 56}}],
    }
    config.update(changes)
    return config


def test_the_description_names_the_tensors_that_the_design_has():
    from llm_serving_engine_b200.config import load_config
    from llm_serving_engine_b200.models import cache_requirements, expected_tensors
    from llm_serving_engine_b200.parts import PagedKV, RequestState

    config = small_config()
    entry, typed, spec = load_config(config)
    assert entry.name == "Kofipel" and not spec.tie_word_embeddings
    expected = {name: tuple(item.shape) for name, item in expected_tensors(spec).items()}
    assert expected == {name: shape for name, (shape, _) in plain.tensor_shapes(config).items()}
    assert "l1.mix.v" not in expected and "l0.canon2" not in expected and "l0.norm2" not in expected
    assert spec.order == (0, 1, 2, 1, 2, 1, 2, 3) and spec.embedding_again == (3, 5)
    assert list(zip(spec.order, [position in spec.embedding_again for position in range(8)])) == plain.layer_runs(config)
    assert spec.shared_tensors == {"side.embed": (97, 28)}
    assert [layer.block.params["token_input"]["params"]["offset"] for layer in spec.layers] == [0, 7, 14, 21]
    attention = spec.layers[1].mixer.params
    assert attention["window"] == 9 and attention["keep_first"] == 5 and attention["values"] == "keys" and attention["unit_sink"]
    needs = cache_requirements(spec)
    window = RequestState((2, 48))
    assert needs[0] == (RequestState((4, 10, 6)), RequestState((2, 64)), window)      # no feed-forward: one window
    assert needs[1] == needs[3] == needs[7] == (PagedKV(2, 8, 9, 0, 5), window, window)


def test_sizes_that_only_tensors_give_are_read_from_the_checkpoint(tmp_path):
    from llm_serving_engine_b200.config import load_config
    from llm_serving_engine_b200.config.model_config import ConfigError

    config = small_config()
    weights = plain.random_weights(config, seed=3)
    for layer in (0, 2):
        config["layers"][layer]["mixer"] = {key: value for key, value in config["layers"][layer]["mixer"].items() if "rank" not in key}
    plain.write_model(tmp_path, config, seed=0, weights=weights)
    _, _, spec = load_config(tmp_path)
    assert spec.layers[2].mixer.params["decay_rank"] == 3 and spec.layers[2].mixer.params["gate_rank"] == 5
    with pytest.raises(ConfigError, match="rank of a1"):
        load_config(config)


def _layer(**mixer):
    base = small_config()["layers"][1]
    return {"layers": [{**base, "mixer": {**base["mixer"], **mixer}}], "loop": {"start": 0, "stop": 0, "times": 1}}


@pytest.mark.parametrize("change,message", [
    ({"layers": [{"type": "other", "mixer": {}}], "loop": None}, "unknown type"),
    ({"layers": [{"type": "channel_delta", "mixer": {"heads": 2}, "mlp": None}], "loop": None}, "lacks"),
    (_layer(vdim=16), "vdim must equal dim"),
    (_layer(kv_heads=4), "multiple of kv_heads"),
    (_layer(rot={"base": 10.0, "dims": 10}), "rot.dims"),
    (_layer(softcap=0.0), "softcap"),
    (_layer(mask={"size": 0}), "mask.size"),
    ({"loop": {"start": 2, "stop": 5, "times": 2}}, "loop"),
    ({"loop": {"start": 1, "stop": 3, "times": 0}}, "loop"),
    ({"norm": {}}, "norm.eps"),
    ({"canon": {}}, "canon.taps"),
    ({"vocab": 0}, "positive"),
])
def test_a_configuration_that_cannot_run_is_refused_with_the_reason(change, message):
    from llm_serving_engine_b200.config import load_config
    from llm_serving_engine_b200.config.model_config import ConfigError

    with pytest.raises(ConfigError, match=message):
        load_config(small_config(**change))


@pytest.mark.parametrize("loop,order,again", [
    (None, (0, 1, 2, 3), ()), ((0, 0, 5), (0, 1, 2, 3), ()), ((1, 3, 1), (0, 1, 2, 3), ()),
    ((0, 4, 2), (0, 1, 2, 3, 0, 1, 2, 3), (4,)), ((3, 4, 3), (0, 1, 2, 3, 3, 3), (4, 5)),
])
def test_the_order_of_a_loop(loop, order, again):
    from llm_serving_engine_b200.config import load_config

    config = small_config(loop=None if loop is None else dict(zip(("start", "stop", "times"), loop)))
    _, _, spec = load_config(config)
    assert spec.order == order and spec.embedding_again == again
    assert plain.layer_runs(config) == [(index, position in again) for position, index in enumerate(order)]


def test_every_pass_of_a_looped_layer_gets_pages_and_states_of_its_own():
    from llm_serving_engine_b200.cache.manager import CacheManager
    from llm_serving_engine_b200.config import CacheConfig, load_config
    from llm_serving_engine_b200.models import cache_requirements

    _, _, spec = load_config(small_config())
    cache = CacheManager(cache_requirements(spec), CacheConfig(block_size=4, num_blocks=6), torch.float32, "cpu", 64,
                         num_state_slots=2)
    views = [cache.layer_view(position) for position in range(8)]
    pages = [views[position].parts[0].keys.data_ptr() for position in (1, 3, 5, 7)]
    assert len(set(pages)) == 4 and views[1].parts[0].keys.shape == (6, 2, 4, 8)
    states = [part.state for view in views for part in view.parts if part.state is not None]
    assert len({state.data_ptr() for state in states}) == len(states) == 4 * 4 - 1 + 4 * 2      # the first layer has one window less
    taken = cache.create("a")
    for state in states:
        state[taken.state_slot].fill_(3.0)
    cache.create("b")
    cache.free("a")
    again = cache.create("c")
    assert again.state_slot == taken.state_slot
    assert all(float(state[again.state_slot].abs().max()) == 0.0 for state in states)


@pytest.mark.parametrize("page,window,keep_first", [(4, 6, 5), (4, 6, 4), (4, 6, 0), (8, 3, 1), (4, 1, 40)])
def test_pages_of_the_kept_first_keys_stay(page, window, keep_first):
    """While a request grows token by token exactly the pages stay that hold a kept key or a key of the next token's window."""
    from llm_serving_engine_b200.cache.manager import CacheManager
    from llm_serving_engine_b200.config import CacheConfig
    from llm_serving_engine_b200.parts import PagedKV

    cache = CacheManager([PagedKV(1, 4, window, 0, keep_first)], CacheConfig(block_size=page, num_blocks=40), torch.float32, "cpu", 512)
    cache.create("a")
    for length in range(1, 61):
        cache.reserve("a", 1)
        cache.release_passed("a")
        table = cache.requests["a"].tables[0]
        for logical, physical in enumerate(table):
            keys = range(logical * page, (logical + 1) * page)
            needed = any(key < keep_first or key >= length - window + 1 for key in keys)
            assert (physical >= 0) == needed, (length, logical)
            assert physical < 0 or cache.groups[0].pool.owner_of(physical) == "a"
    cache.free("a")
    assert cache.groups[0].pool.used_pages == 0


def test_plain_sink_softmax_and_mask():
    scores = torch.tensor([[0.3, -1.0, float("-inf")], [40.0, 41.0, 39.0]], dtype=torch.float64)
    direct = torch.exp(scores) / (1.0 + torch.exp(scores).sum(-1, keepdim=True))
    assert torch.allclose(plain.sink_softmax(scores), direct, rtol=1e-12)
    assert float(plain.sink_softmax(torch.full((1, 5), -50.0, dtype=torch.float64)).sum()) < 1e-20
    seen = plain.visible(7, 2, 3)
    assert [[j for j in range(7) if seen[i, j]] for i in range(7)] == [
        [0], [0, 1], [0, 1, 2], [0, 1, 2, 3], [0, 1, 2, 3, 4], [0, 1, 2, 4, 5], [0, 1, 2, 5, 6]]


def test_plain_delta_memory_writes_differences():
    """A full write of an orthonormal key replaces what it held; an overwritten key leaves the others alone; the read-out sees
    the current token's write; the decays act before it."""
    k = torch.eye(3, dtype=torch.float64)[[0, 1, 0]][:, None]
    v = torch.tensor([[2.0, 3.0], [5.0, 7.0], [11.0, 13.0]], dtype=torch.float64)[:, None]
    ones = torch.ones(3, 1, dtype=torch.float64)
    keep = torch.ones(3, 1, 3, dtype=torch.float64)
    o, state = plain.delta_memory(k, k, v, keep, ones)
    assert torch.allclose(o, v) and torch.allclose(state[0, 0], v[2, 0]) and torch.allclose(state[0, 1], v[1, 0])
    half, _ = plain.delta_memory(k, k, v, keep, 0.5 * ones)
    assert torch.allclose(half[2], 0.5 * 0.5 * v[0] + 0.5 * v[2])
    keep[2] = 0.25
    decayed, state = plain.delta_memory(k, k, v, keep, 0.5 * ones)
    assert torch.allclose(decayed[2], 0.25 * 0.25 * v[0] + 0.5 * v[2]) and torch.allclose(state[0, 1], 0.25 * 0.5 * v[1, 0])


def test_plain_convolution_and_rotation():
    u = torch.tensor([[1.0], [10.0], [100.0]], dtype=torch.float64)
    assert plain.causal_conv(u, torch.tensor([[2.0, 3.0, 5.0]], dtype=torch.float64))[:, 0].tolist() == [5.0, 53.0, 532.0]
    x = torch.zeros(5, 1, 6, dtype=torch.float64)
    x[:, 0, 1] = 1.0        # pair (1, 3) of four rotated values; two values pass
    x[:, 0, 5] = 4.0
    y = plain.rotate_half(x, 100.0, 4)
    angle = 4 * 100.0 ** (-2.0 / 4)
    assert math.isclose(float(y[4, 0, 1]), math.cos(angle)) and math.isclose(float(y[4, 0, 3]), math.sin(angle))
    assert float(y[4, 0, 5]) == 4.0
