"""Host-side pieces of the Daferax design: configuration, description, tensor names, cache needs, pages that a window gives
back, the plain implementation's pieces against closed forms."""
import copy
import math

import pytest
import torch

from plain import daferax_plain as plain


def small_config(**changes):
    attention = {"heads": 6, "kv_heads": 2, "dim": 10, "vdim": 14, "scale": 0.3, "v_mix": True, "rot": {"base": 500.0, "dims": 8}}
    latent = {"heads": 3, "dim": 12, "rot_dim": 6, "vdim": 9, "kv_rank": 20, "scale": 0.25, "mask": {"size": 11},
              "rot": {"base": 500.0, "dims": 6, "scaling": {"factor": 3.0, "original": 50, "fast": 8.0, "slow": 1.0}}}
    mlp = {"kind": "moe", "router": {"experts": 6, "top": 2, "scale": 1.5, "groups": {"count": 3, "keep": 1}},
           "expert": {"ff": 22}, "shared": {"ff": 34}}
    config = {"architecture": "Daferax", "vocab": 97, "width": 48, "norm": {"eps": 1e-5},
              "layers": [{"type": "attention", "mixer": dict(attention, v_mix=False, vdim=5), "mlp": mlp},
                         {"type": "attention", "mixer": attention, "mlp": None},
                         {"type": "latent_attention", "mixer": latent, "mlp": mlp},
                         {"type": "attention", "mixer": attention,
                          "mlp": {**mlp, "shared": None, "router": {"experts": 4, "top": 1}}},
                         {"type": "latent_attention", "mixer": {k: v for k, v in latent.items() if k != "mask"}, "mlp": None}]}
    config = copy.deepcopy(config)
    config.update(changes)
    return config


def test_the_description_names_the_tensors_that_the_design_has():
    from llm_serving_engine_b200.config import load_config
    from llm_serving_engine_b200.models import cache_requirements, expected_tensors
    from llm_serving_engine_b200.parts import PagedKV, PagedLatent

    config = small_config()
    entry, typed, spec = load_config(config)
    assert entry.name == "Daferax" and spec.tie_word_embeddings and typed.first_mixing_layer == 1
    expected = {name: tuple(item.shape) for name, item in expected_tensors(spec).items()}
    assert expected == {name: shape for name, (shape, _) in plain.tensor_shapes(config).items()}
    assert "l0.mix.vmix" not in expected and expected["l1.mix.vmix"] == () and "l1.norm2" not in expected
    assert "l3.mlp.shared.up" not in expected and "head" not in expected
    assert [layer.mixer.params.get("value_mix") for layer in spec.layers] == [None, "first", None, "later", None]
    router = spec.layers[0].feed_forward.params
    assert router["groups"] == {"count": 3, "keep": 1} and router["router_scale"] == 1.5 and not router["shared_gate"]
    assert spec.layers[3].feed_forward.params["groups"] is None and spec.layers[3].feed_forward.params["router_scale"] == 1.0
    needs = cache_requirements(spec)
    assert needs == [PagedKV(2, 10, 0, 5), PagedKV(2, 10, 0, 14), PagedLatent(26, 11), PagedKV(2, 10, 0, 14), PagedLatent(26, 0)]


def test_a_model_folder_is_read_by_its_config(tmp_path):
    from llm_serving_engine_b200.config import load_config
    from llm_serving_engine_b200.models import expected_tensors
    from llm_serving_engine_b200.weights import load_weights

    config = small_config()
    weights = plain.write_model(tmp_path, config, seed=3)
    _, _, spec = load_config(tmp_path)
    loaded = load_weights(tmp_path, expected_tensors(spec), torch.bfloat16, "cpu")
    assert set(loaded) == set(weights)
    assert loaded["l2.mix.uk"].dtype == torch.bfloat16 and loaded["l1.mix.vmix"].dtype == torch.float32
    assert all(torch.equal(loaded[name].float(), weights[name].float()) for name in weights)


def _with_layer(index, path, value):
    config = small_config()
    place = config["layers"][index]
    for key in path[:-1]:
        place = place[key]
    if value is None:
        del place[path[-1]]
    else:
        place[path[-1]] = value
    return config


@pytest.mark.parametrize("config,message", [
    (_with_layer(0, ("type",), "other"), "unknown type"),
    (_with_layer(1, ("mixer", "kv_heads"), 4), "multiple of kv_heads"),
    (_with_layer(1, ("mixer", "rot", "dims"), 12), "rot.dims"),
    (_with_layer(2, ("mixer", "rot", "dims"), 5), "rot.dims"),
    (_with_layer(2, ("mixer", "rot", "scaling", "fast"), None), "rot.scaling"),
    (_with_layer(2, ("mixer", "mask", "size"), 0), "mask.size"),
    (_with_layer(2, ("mixer", "kv_rank"), None), "lacks"),
    (_with_layer(3, ("mixer",), dict(small_config()["layers"][3]["mixer"], vdim=16)), "different shapes"),
    (_with_layer(0, ("mlp", "kind"), "dense"), "must be 'moe'"),
    (_with_layer(0, ("mlp", "router", "top"), 3), "fewer experts"),
    (_with_layer(0, ("mlp", "router", "groups", "count"), 4), "router.groups"),
    (_with_layer(3, ("mlp", "router", "top"), 5), "router.top"),
    (_with_layer(0, ("mlp", "shared", "ff"), 0), "shared.ff"),
    (small_config(norm={}), "norm.eps"),
    (small_config(vocab=0), "positive"),
])
def test_a_configuration_that_cannot_run_is_refused_with_the_reason(config, message):
    from llm_serving_engine_b200.config import load_config
    from llm_serving_engine_b200.config.model_config import ConfigError

    with pytest.raises(ConfigError, match=message):
        load_config(config)


@pytest.mark.parametrize("page,window", [(4, 6), (4, 1), (8, 3), (4, 40), (16, 17)])
def test_pages_of_latent_rows_that_a_window_has_passed_go_back(page, window):
    """While a request grows token by token exactly the pages stay that hold a row of the next token's window; the other
    groups keep theirs."""
    from llm_serving_engine_b200.cache.manager import CacheManager
    from llm_serving_engine_b200.config import CacheConfig
    from llm_serving_engine_b200.parts import PagedKV, PagedLatent

    cache = CacheManager([PagedLatent(6, window), PagedKV(1, 4, 0, 2)], CacheConfig(block_size=page, num_blocks=40), torch.float32, "cpu", 512)
    assert cache.layer_view(0).keys.shape == (40, page, 6) and cache.layer_view(1).values.shape == (40, 1, page, 2)
    cache.create("a")
    for length in range(1, 61):
        cache.reserve("a", 1)
        cache.release_passed("a")
        for logical, physical in enumerate(cache.requests["a"].tables[0]):
            needed = (logical + 1) * page > length - window + 1
            assert (physical >= 0) == needed, (length, logical)
        assert all(physical >= 0 for physical in cache.requests["a"].tables[1])
    cache.free("a")
    assert all(group.pool.used_pages == 0 for group in cache.groups)


def test_plain_rotation_turns_neighbouring_pairs():
    x = torch.zeros(5, 1, 6, dtype=torch.float64)
    x[:, 0, 2] = 1.0        # the second pair's first value; two values pass
    x[:, 0, 5] = 4.0
    y = plain.rotate_pairs(x, {"base": 100.0, "dims": 4}, first=3)
    angle = 7 * 100.0 ** (-2.0 / 4)
    assert math.isclose(float(y[4, 0, 2]), math.cos(angle)) and math.isclose(float(y[4, 0, 3]), math.sin(angle))
    assert float(y[4, 0, 5]) == 4.0 and float(y[4, 0, 0]) == 0.0


def test_plain_stretched_frequencies():
    """Pairs that turn often keep their frequency, pairs that turn rarely are slowed by the factor, cosine and sine grow."""
    rot = {"base": 10000.0, "dims": 32, "scaling": {"factor": 8.0, "original": 4096, "fast": 32.0, "slow": 1.0}}
    stretched, factor = plain.frequencies(rot)
    plainly, one = plain.frequencies({"base": 10000.0, "dims": 32})
    ratios = [a / b for a, b in zip(stretched, plainly)]
    assert one == 1.0 and math.isclose(factor, 0.1 * math.log(8.0) + 1.0)
    assert ratios[0] == 1.0 and math.isclose(ratios[-1], 1.0 / 8.0) and all(a >= b - 1e-12 for a, b in zip(ratios, ratios[1:]))


def test_plain_mask_norm_and_values():
    assert [[j for j in range(5) if plain.visible(5, 2)[i, j]] for i in range(5)] == [[0], [0, 1], [1, 2], [2, 3], [3, 4]]
    assert bool(plain.visible(4).equal(torch.ones(4, 4).tril().bool()))
    x = torch.tensor([[1.0, 3.0]], dtype=torch.float64)
    y = plain.layer_norm(x, torch.tensor([2.0, 5.0]).double(), torch.tensor([0.5, -1.0]).double(), 0.0)
    assert torch.allclose(y, torch.tensor([[-1.5, 4.0]]).double())
    assert torch.allclose(plain.mix_values(x, x + 4.0, torch.tensor(0.25).double()), x + 1.0)


def test_plain_router_takes_the_group_of_the_best_expert():
    z = torch.tensor([[1.0, 0.9, 1.1, -5.0]], dtype=torch.float64)
    scores = torch.softmax(z, dim=-1)
    weights = plain.route(z, 1, {"count": 2, "keep": 1}, 2.0)
    assert torch.allclose(weights, torch.tensor([[0.0, 0.0, 1.0, 0.0]]).double() * scores * 2.0)
    both = plain.route(z, 2, {"count": 2, "keep": 1}, 1.0)           # the second choice is confined to the same group
    assert float(both[0, 0]) == 0.0 and float(both[0, 3]) > 0.0
    assert float(plain.route(z, 2, None, 1.0)[0, 0]) > 0.0
