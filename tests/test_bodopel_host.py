"""Host-side tests of the Bodopel design: its configuration, its description made of parts, the tensors it expects, the state
its blocks keep, and properties of the plain implementation the GPU tests compare with."""
import copy
import math

import pytest
import torch

import plain_bodopel
from bodopel_configs import BA, BB, BC, BD, BE, CONFIGS


def test_the_registry_resolves_the_design():
    from torchinferno_b200.config.registry import registered_architectures, resolve_architecture
    assert "Bodopel" in registered_architectures()
    assert resolve_architecture({"architecture": "Bodopel"}).name == "Bodopel"
    with pytest.raises(ValueError):
        resolve_architecture({"architecture": "Bodopel", "architectures": ["LlamaForCausalLM"]})


def test_config_errors_name_what_is_missing_or_wrong():
    from torchinferno_b200.config.bodopel_config import BodopelConfig
    from torchinferno_b200.config.model_config import ConfigError
    for config, _ in CONFIGS.values():
        BodopelConfig.from_dict(config)
    for path, value in ((("width",), None), (("max_positions",), None), (("max_positions",), 0), (("norm", "eps"), 0.0),
                        (("canon",), None), (("canon", "taps"), 0), (("embedding", "scale"), None), (("embedding", "scale"), "2"),
                        (("loop", "stop"), 5), (("loop", "start"), 3), (("loop", "times"), 0), (("loop", "times"), None),
                        (("layers", 0, "type"), "conv"), (("layers", 0, "mixer", "kv_heads"), 3), (("layers", 0, "mixer", "vdim"), None),
                        (("layers", 0, "mixer", "scale"), 0.0), (("layers", 0, "mixer", "softcap"), None), (("layers", 0, "mixer", "softcap"), -1.0),
                        (("layers", 0, "mixer", "mask"), None), (("layers", 0, "mixer", "mask", "size"), 0),
                        (("layers", 0, "mlp", "kind"), "moe"), (("layers", 0, "mlp", "ff"), None)):
        bad = copy.deepcopy(BA)
        node = bad
        for key in path[:-1]:
            node = node[key]
        if value is None:
            del node[path[-1]]
        else:
            node[path[-1]] = value
        with pytest.raises(ConfigError, match=str(path[-1])):
            BodopelConfig.from_dict(bad)


def test_the_schedule_gives_every_run_of_a_layer_a_cache_and_opens_every_pass():
    from torchinferno_b200.config.bodopel_config import BodopelConfig
    from torchinferno_b200.models.bodopel import build_bodopel
    from torchinferno_b200.models.spec import StageCall

    def order(config):
        spec = build_bodopel(BodopelConfig.from_dict(config))
        return spec, [("pass", c.arg) if isinstance(c, StageCall) else (c.layer, c.cache) for c in spec.schedule]

    spec, steps = order(BA)
    assert steps == [(0, 0), ("pass", 0), (1, 1), (2, 2), ("pass", 1), (1, 3), (2, 4), (3, 5)]
    assert spec.embedding_scale == 6.0 and spec.position_embedding_name == "pos" and spec.max_positions == 400
    assert [plain_bodopel.layer_runs(BA)[i] for i in (1, 2, 3)] == [(1, 0), (2, None), (1, 1)]
    assert order(BB)[1] == [(0, 0), (1, 1), (2, 2)] and not order(BB)[0].stages
    assert order(BC)[1][-3:] == [("pass", 2), (0, 4), (1, 5)] and order(BD)[1][-2:] == [("pass", 1), (2, 3)]
    params = spec.layers[0].block.params["mixer"].params
    assert params["window"] == 20 and params["softcap"] == 2.0 and params["row_norm_eps"] == 1e-5
    free = build_bodopel(BodopelConfig.from_dict(BB)).layers[1].block.params["mixer"].params
    assert free["window"] is None and free["softcap"] is None
    assert spec.layers[1].block.params["feed_forward"] is None and spec.layers[1].block.params["feed_forward_input"] is None


def test_expected_tensors_caches_and_the_blocks_state():
    from torchinferno_b200.weights.random_init import build_model
    model = build_model(BA, dtype=torch.float32, device="cpu")
    names = model.expected_tensors()
    assert names["pos"].shape == (400, 64) and names["loop.step"].shape == (2, 64) and names["head"].shape == (101, 64)
    assert names["l0.mix.q"].shape == (64, 64) and names["l0.mix.q.b"].shape == (64,) and names["l0.mix.q.norm"].shape == (64,)
    assert names["l0.mix.k.norm"].shape == (32,) and names["l0.mix.v.b"].shape == (48,) and "l0.mix.v.norm" not in names
    assert names["l0.mix.talk"].shape == (4, 4) and names["l0.mix.r1"].shape == (4,) and names["l0.mix.g"].shape == (96, 64)
    assert names["l0.canon1"].shape == (64, 3) and names["l0.canon2"].shape == (64, 3) and names["l0.mlp.up"].shape == (40, 64)
    assert "l1.norm2" not in names and "l1.canon2" not in names and "l1.mlp.up" not in names and "l1.canon1" in names
    assert "loop.step" not in build_model(BB, dtype=torch.float32, device="cpu").expected_tensors()
    caches, states = model.cache_requirements(), model.state_requirements()
    assert [(c.window, c.kv_heads, c.head_dim, c.value_width) for c in caches] == [
        (20, 2, 16, 24), (33, 2, 8, 8), (50, 1, 24, 16), (33, 2, 8, 8), (50, 1, 24, 16), (20, 2, 16, 24)]
    # (mixers keep none; a block carries two rows for each of its sublayers; the pass's vector carries nothing)
    assert [None if s is None else s.shape for s in states] == [None] * 8 + [(256,), None, (128,), (256,), None, (128,), (256,), (256,)]
    assert model.capturable()
    assert build_model(BB, dtype=torch.float32, device="cpu").state_requirements() == [None] * 3      # (one tap looks at no earlier row)


def test_the_blocks_state_is_zeroed_for_a_new_request():
    from torchinferno_b200.cache.manager import CacheManager
    from torchinferno_b200.weights.random_init import build_model
    model = build_model(BC, dtype=torch.float32, device="cpu")
    cache = CacheManager(model.cache_requirements(), model.state_requirements(), page_size=4, num_pages=40, max_requests=2,
                         max_request_tokens=100, dtype=torch.float32, device=torch.device("cpu"))
    slot = cache.open("a")
    at = len(model.spec.schedule) + 1
    assert cache.state(at).shape == (2, 2 * 4 * 50)
    cache.state(at)[slot].fill_(3.0)
    cache.close("a")
    assert cache.open("b") == slot and float(cache.state(at)[slot].abs().sum()) == 0.0


def test_a_random_model_folder_holds_exactly_the_expected_tensors(tmp_path):
    from torchinferno_b200.weights.random_init import build_model, write_random_model
    write_random_model(BC, tmp_path, seed=3)
    config, weights = plain_bodopel.read_model_folder(tmp_path)
    assert set(weights) == set(build_model(BC, dtype=torch.float32, device="cpu").expected_tensors())
    assert config["layers"] == BC["layers"]
    assert 0.01 < float(weights["l1.norm1"].abs().max()) < 0.8 and float(weights["l0.mix.r2"].min()) > 0      # (norms around zero)


def test_a_norm_may_store_what_its_gain_exceeds_one_by():
    from torchinferno_b200.parts.base import PartSpec, build_part
    stored = torch.tensor([0.5, -0.25, 0.0])
    for offset, want in ((0.0, stored), (1.0, 1 + stored)):
        norm = build_part("norm", PartSpec("rmsnorm", {"width": 3, "eps": 1e-6, "weight_name": "n", "weight_offset": offset}),
                          dtype=torch.float32, device=torch.device("cpu"))
        norm.bind({"n": stored})
        assert torch.equal(norm.weight, want)


def test_a_block_refuses_an_input_stage_without_its_sublayer():
    from torchinferno_b200.parts.base import PartSpec, build_part
    spec = BA["layers"][0]["mixer"]
    mixer = PartSpec("talking_heads_attention", {"hidden_size": 8, "heads": 2, "kv_heads": 1, "dim": 4, "value_dim": 4, "scale": spec["scale"],
                                                 "max_positions": 10}, prefix="mix.")
    norm = PartSpec("rmsnorm", {"width": 8, "eps": 1e-6, "weight_name": "n"})
    conv = PartSpec("causal_conv", {"width": 8, "taps": 2})
    with pytest.raises(ValueError):
        build_part("block", PartSpec("prenorm", {"mixer": mixer, "mixer_norm": norm, "feed_forward": None, "feed_forward_norm": None,
                                                 "feed_forward_input": conv}), dtype=torch.float32, device=torch.device("cpu"))


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_the_plain_implementation_is_causal(name, tmp_path):
    from bodopel_configs import write_model
    config, seed = CONFIGS[name]
    write_model(config, tmp_path, seed=seed)
    cfg, w = plain_bodopel.read_model_folder(tmp_path)
    tokens = torch.randint(0, cfg["vocab"], (53,)).tolist()
    whole, layers = plain_bodopel.forward(cfg, w, tokens, return_layers=True)
    assert torch.isfinite(whole).all() and whole.abs().max() > 0.5
    assert layers.shape[:2] == (len(plain_bodopel.layer_runs(cfg)), 53)
    assert torch.allclose(plain_bodopel.forward(cfg, w, tokens[:19]), whole[:19], atol=1e-12, rtol=1e-10)


def test_plain_mechanisms_against_closed_forms():
    D = torch.float64
    # the norm's gain is one more than what is stored
    x = torch.tensor([[3.0, 4.0]], dtype=D)
    assert torch.allclose(plain_bodopel.zero_centred_norm(x, torch.tensor([0.0, 1.0], dtype=D), 0.0), x / math.sqrt(12.5) * torch.tensor([1.0, 2.0], dtype=D))
    # the convolution: the last column is the current row's, the row itself is added, nothing before the start
    h = torch.tensor([[1.0], [10.0], [100.0]], dtype=D)
    out = plain_bodopel.input_convolution(h, torch.tensor([[3.0, 2.0]], dtype=D))
    assert out.flatten().tolist() == [1 + 2, 10 + 20 + 3, 100 + 200 + 30]
    assert torch.allclose(plain_bodopel.input_convolution(h, torch.tensor([[0.5]], dtype=D)), 1.5 * h)
    # the cap bends and bounds; none leaves the scores as they are
    s = torch.tensor([0.1, 4.0, -900.0], dtype=D)
    assert torch.allclose(plain_bodopel.capped(s, 2.0), 2 * torch.tanh(s / 2)) and torch.equal(plain_bodopel.capped(s, None), s)
    # the distance takes off r1 ln(1 + r2 n): nothing at distance 0
    loss = plain_bodopel.distance_loss(torch.tensor([2.0, 1.0], dtype=D), torch.tensor([1.0, 0.5], dtype=D), torch.tensor([0, 1, 3]))
    assert torch.allclose(loss, torch.tensor([[0.0, 2 * math.log(2), 2 * math.log(4)], [0.0, math.log(1.5), math.log(2.5)]], dtype=D))
    # a window of two: a query sees itself and the token before it
    weights = plain_bodopel.window_weights(torch.zeros(1, 4, 4, dtype=D), 2)[0]
    assert weights.tolist() == [[1, 0, 0, 0], [0.5, 0.5, 0, 0], [0, 0.5, 0.5, 0], [0, 0, 0.5, 0.5]]
    # the mix is indexed [to, from]
    w = torch.stack([torch.full((1, 1), 1.0, dtype=D), torch.full((1, 1), 10.0, dtype=D)])
    mixed = plain_bodopel.mix_heads(w, torch.tensor([[0.0, 1.0], [2.0, 0.0]], dtype=D))
    assert mixed.flatten().tolist() == [10.0, 2.0]
    # a squared relu between two products
    unit = plain_bodopel.squared_relu_unit(torch.tensor([[2.0, -3.0]], dtype=D), {"p.up": torch.eye(2, dtype=D), "p.down": torch.ones(1, 2, dtype=D)}, "p.")
    assert unit.item() == 4.0
