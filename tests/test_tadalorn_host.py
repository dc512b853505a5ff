"""Host-side tests of the Tadalorn design: its configuration, its description made of parts, the tensors it expects, what its caches
and states hold, and properties of the plain implementation the GPU tests compare with."""
import copy
import math

import pytest
import torch

import plain_tadalorn
from tadalorn_configs import CONFIGS, TA, TB, TC, TD, TE


def test_the_registry_resolves_the_design():
    from torchinferno_b200.config.registry import registered_architectures, resolve_architecture
    assert "Tadalorn" in registered_architectures()
    assert resolve_architecture({"architecture": "Tadalorn"}).name == "Tadalorn"
    with pytest.raises(ValueError):
        resolve_architecture({"architecture": "Tadalorn", "architectures": ["LlamaForCausalLM"]})


def test_config_errors_name_what_is_missing_or_wrong():
    from torchinferno_b200.config.model_config import ConfigError
    from torchinferno_b200.config.tadalorn_config import TadalornConfig
    for config, _ in CONFIGS.values():
        TadalornConfig.from_dict(config)
    drop = object()
    for path, value in ((("width",), drop), (("vocab",), 0), (("norm", "eps"), 0.0), (("residual_mult",), drop), (("residual_mult",), "1"),
                        (("logit_softcap",), drop), (("logit_softcap",), -1.0), (("layers", 0, "type"), "conv"),
                        (("layers", 0, "mixer", "kv_heads"), 3), (("layers", 0, "mixer", "vdim"), 24), (("layers", 0, "mixer", "conv"), 0),
                        (("layers", 0, "mixer", "scale"), drop), (("layers", 0, "mixer", "mask"), drop),
                        (("layers", 0, "mixer", "mask", "size"), 0), (("layers", 0, "mixer", "mask", "keep_first"), drop),
                        (("layers", 0, "mixer", "mask", "keep_first"), -1), (("layers", 0, "mixer", "rot", "dims"), 18),
                        (("layers", 0, "mixer", "rot", "dims"), 5), (("layers", 0, "mixer", "rot", "base"), 0),
                        (("layers", 1, "mixer", "gate_cap"), drop), (("layers", 1, "mixer", "gate_cap"), 0.0),
                        (("layers", 2, "mixer", "kv_rank"), drop), (("layers", 2, "mixer", "rot", "dims"), 4),
                        (("layers", 2, "mlp", "kind"), "sparse"), (("layers", 1, "mlp", "ff"), drop),
                        (("layers", 2, "mlp", "router", "top"), 7), (("layers", 0, "mlp", "expert"), drop),
                        (("layers", 3, "weights_of"), 9), (("layers", 3, "weights_of"), -1), (("layers", 3, "weights_of"), 1),
                        (("layers", 3, "weights_of"), 3)):
        bad = copy.deepcopy(TA)
        node = bad
        for key in path[:-1]:
            node = node[key]
        if value is drop:
            del node[path[-1]]
        else:
            node[path[-1]] = value
        with pytest.raises(ConfigError, match=str(path[-1])):
            TadalornConfig.from_dict(bad)


def test_layers_that_share_tensors_have_caches_and_states_of_their_own():
    from torchinferno_b200.config.tadalorn_config import TadalornConfig
    from torchinferno_b200.models.tadalorn import build_tadalorn
    from torchinferno_b200.weights.random_init import build_model

    def order(config):
        spec = build_tadalorn(TadalornConfig.from_dict(config))
        return [block.prefix for block in spec.layers], [(call.layer, call.cache) for call in spec.schedule]

    assert order(TA) == (["l0.", "l1.", "l2.", "l4."], [(0, 0), (1, None), (2, 1), (0, 2), (3, 3), (1, None)])
    assert order(TC) == (["l0.", "l1."], [(0, None), (1, None), (0, None), (0, None)])
    chained = copy.deepcopy(TC)
    chained["layers"][3]["weights_of"] = 2                   # (a layer that names one which names another)
    assert order(chained) == order(TC) and plain_tadalorn.tensors_of(chained, 3) == 0
    model = build_model(TA, dtype=torch.float32, device="cpu")
    assert [(c.window, c.keep_first, c.kv_heads, c.head_dim, c.value_width) for c in model.cache_requirements()] == [
        (20, 3, 2, 16, 16), (None, 0, 1, 48, 0), (20, 3, 2, 16, 16), (None, 0, 1, 28, 0)]
    memory = -(-(3 * 16 * 24 + 3 * 17) // 4) * 4
    assert [None if s is None else s.shape for s in model.state_requirements()] == [
        (2 * 6 * 16,), (memory,), None, (2 * 6 * 16,), None, (memory,)]
    assert model.capturable()
    # a convolution of one tap carries nothing, heads wider than a tile keep a sum of keys and a maximum per tile
    assert [None if s is None else s.shape for s in build_model(TB, dtype=torch.float32, device="cpu").state_requirements()][:3] == [
        None, (4 * 6,), None]
    assert build_model(TD, dtype=torch.float32, device="cpu").state_requirements()[0].shape == (2 * 40 * 136 + 2 * 2 * 41,)


def test_expected_tensors(tmp_path):
    from torchinferno_b200.weights.random_init import build_model, write_random_model
    names = build_model(TA, dtype=torch.float32, device="cpu").expected_tensors()
    shapes = {n: tuple(s.shape) for n, s in names.items()}
    assert shapes["embed"] == shapes["head"] == (101, 64) and shapes["final.norm"] == (64,)
    assert shapes["l0.mix.q"] == (64, 64) and shapes["l0.mix.k"] == (32, 64) and "l0.mix.v" not in shapes
    assert shapes["l0.mix.q.conv"] == (64, 3) and shapes["l0.mix.k.conv"] == (32, 3) and shapes["l0.mix.q.norm"] == (64,)
    assert shapes["l0.mix.g"] == (64, 64) and shapes["l0.mix.o"] == (64, 64) and "l0.mix.sink" not in shapes
    assert shapes["l0.mlp.router"] == (5, 64) and shapes["l0.mlp.router.b"] == (5,) and shapes["l0.mlp.e4.up"] == (24, 64)
    assert shapes["l0.mlp.shared.down"] == (64, 40) and "l0.mlp.shared.sg" not in shapes and "l2.mlp.shared.up" not in shapes
    assert shapes["l1.mix.i"] == shapes["l1.mix.f"] == (3, 64) and shapes["l1.mix.f.b"] == (3,) and shapes["l1.mix.norm"] == (72,)
    assert shapes["l1.mlp.gate"] == (72, 64) and shapes["l2.mix.sink"] == (2,) and shapes["l2.mix.dkv.norm"] == (40,)
    assert not any(n.startswith(("l3.", "l5.")) for n in shapes) and "l4.norm2" not in shapes and "l4.norm1" in shapes
    write_random_model(TC, tmp_path, seed=3)
    config, weights = plain_tadalorn.read_model_folder(tmp_path)
    assert set(weights) == set(build_model(TC, dtype=torch.float32, device="cpu").expected_tensors())
    assert config["layers"] == TC["layers"]


def test_a_group_with_a_window_keeps_the_pages_of_its_first_tokens():
    from torchinferno_b200.cache.manager import CacheManager
    from torchinferno_b200.parts.base import CacheSpec
    specs = [CacheSpec(1, 4, 5, keep_first=k) for k in (0, 1, 4, 5, 40)] + [CacheSpec(1, 4, None)]
    cache = CacheManager(specs, [None] * 6, page_size=4, num_pages=16, max_requests=2, max_request_tokens=60, dtype=torch.float32, device="cpu")
    assert len(cache.groups) == 6                            # (what is kept tells groups apart)
    cache.open("a")
    for _ in range(6):
        cache.extend("a", 5)
        cache.release_behind_window("a")
        cache.audit()
    # 30 tokens; the next query, at 30, sees 26 .. 29 and the kept ones: pages 6 and 7, and what holds the first 0, 1, 4, 5, 40 tokens
    held = [[i for i, p in enumerate(cache.block_table("a", g)) if p >= 0] for g in range(6)]
    assert held == [[6, 7], [0, 6, 7], [0, 6, 7], [0, 1, 6, 7], list(range(8)), list(range(8))]
    assert cache.free_pages() == [14, 13, 13, 12, 8, 8]
    cache.close("a")
    cache.audit()
    assert cache.free_pages() == [16] * 6


def test_the_states_are_zeroed_for_a_new_request():
    from torchinferno_b200.cache.manager import CacheManager
    from torchinferno_b200.weights.random_init import build_model
    model = build_model(TA, dtype=torch.float32, device="cpu")
    cache = CacheManager(model.cache_requirements(), model.state_requirements(), page_size=4, num_pages=40, max_requests=2,
                         max_request_tokens=100, dtype=torch.float32, device=torch.device("cpu"))
    slot = cache.open("a")
    for call in (0, 1, 3, 5):
        cache.state(call)[slot].fill_(3.0)
    cache.close("a")
    assert cache.open("b") == slot and all(float(cache.state(call)[slot].abs().sum()) == 0.0 for call in (0, 1, 3, 5))


def test_parts_refuse_what_their_kernels_do_not_do():
    from torchinferno_b200.parts.base import PartSpec, build_part
    base = {"hidden_size": 8, "heads": 2, "kv_heads": 1, "dim": 4, "scale": 0.5, "taps": 2, "window": 3, "keep_first": 1,
            "position": PartSpec("rotary", {"head_dim": 4, "theta": 100.0, "rot_dim": 2, "interleaved": True})}
    make = lambda **changes: build_part("mixer", PartSpec("kept_window_attention", {**base, **changes}), dtype=torch.float32,
                                        device=torch.device("cpu"))
    assert make().cache_spec().keep_first == 1 and make(window=None).cache_spec().keep_first == 0
    for bad in ({"heads": 3, "kv_heads": 2}, {"window": 0}, {"taps": 0}, {"sink": "two"}, {"keep_first": -1},
                {"position": PartSpec("rotary", {"head_dim": 4, "theta": 100.0})}):
        with pytest.raises(ValueError):
            make(**bad)
    norm = PartSpec("rmsnorm", {"width": 8, "eps": 1e-6, "weight_name": "n"})
    block = lambda **params: build_part("block", PartSpec("postnorm", {"mixer": PartSpec("kept_window_attention", base), **params}),
                                        dtype=torch.float32, device=torch.device("cpu"))
    block(mixer_norm=norm)
    with pytest.raises(ValueError):
        block(mixer_norm=norm, feed_forward=PartSpec("swiglu", {"hidden_size": 8, "intermediate_size": 8}))
    with pytest.raises(ValueError):
        block(mixer_norm=PartSpec("layernorm", {"width": 8, "eps": 1e-6}))


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_the_plain_implementation_is_causal(name, tmp_path):
    from tadalorn_configs import write_model
    config, seed = CONFIGS[name]
    write_model(config, tmp_path, seed=seed)
    cfg, w = plain_tadalorn.read_model_folder(tmp_path)
    tokens = torch.randint(0, cfg["vocab"], (53,)).tolist()
    whole, layers = plain_tadalorn.forward(cfg, w, tokens, return_layers=True)
    assert torch.isfinite(whole).all() and whole.abs().max() > 0.5
    assert layers.shape[:2] == (len(cfg["layers"]), 53)
    assert torch.allclose(plain_tadalorn.forward(cfg, w, tokens[:19]), whole[:19], atol=1e-12, rtol=1e-10)


def test_plain_mechanisms_against_closed_forms():
    D = torch.float64
    # the convolution: the last column is the current row's, nothing before the start
    u = torch.tensor([[1.0], [10.0], [100.0]], dtype=D)
    assert plain_tadalorn.channel_convolution(u, torch.tensor([[3.0, 2.0]], dtype=D)).flatten().tolist() == [2, 23, 230]
    # a window of two that keeps one token: a query sees itself, the token before it and token 0
    assert plain_tadalorn.seen_keys(4, 2, 1).int().tolist() == [[1, 0, 0, 0], [1, 1, 0, 0], [1, 1, 1, 0], [1, 0, 1, 1]]
    assert plain_tadalorn.seen_keys(3, 1, 0).int().tolist() == [[1, 0, 0], [0, 1, 0], [0, 0, 1]]
    # a sink of 0 adds one to the denominator
    s = torch.tensor([[[math.log(3.0), 0.0], [math.log(3.0), math.log(6.0)]]], dtype=D)
    weights = plain_tadalorn.softmax_with_sink(s, plain_tadalorn.seen_keys(2, None, 0), torch.zeros(1, dtype=D))
    assert torch.allclose(weights, torch.tensor([[[0.75, 0.0], [0.3, 0.6]]], dtype=D))
    # rotary: pair (2i, 2i + 1), a quarter turn
    x = torch.tensor([[1.0, 2.0, 5.0, 6.0, 7.0]], dtype=D)
    turned = plain_tadalorn.rotate_pairs(x, torch.tensor([math.pi / 2]), 4.0, 4)
    c, n = math.cos(math.pi / 4), math.sin(math.pi / 4)
    assert torch.allclose(turned, torch.tensor([[-2.0, 1.0, 5 * c - 6 * n, 6 * c + 5 * n, 7.0]], dtype=D))
    # gelu: x times the normal distribution's cumulative function
    assert torch.allclose(plain_tadalorn.gelu(torch.tensor([0.0, 1.0, -1.0], dtype=D)), torch.tensor([0.0, 0.8413447460685429, -0.15865525393145707], dtype=D))
    # the memory: two tokens by hand; the denominator is at least exp(-m)
    q, k, v = (torch.tensor(t, dtype=D).view(2, 1, -1) for t in ([[1.0, 0.0], [1.0, 2.0]], [[3.0, 1.0], [0.0, 1.0]], [[5.0], [7.0]]))
    li, lf = torch.tensor([[1.0], [-2.0]], dtype=D), torch.tensor([[-0.5], [-1.0]], dtype=D)
    out = plain_tadalorn.matrix_memory(q, k, v, li, lf).flatten()
    # (m: max(-0.5, 1) = 1, then max(0, -2) = 0)
    assert math.isclose(out[0], 15.0 / (max(3.0, math.exp(-1)) + 1e-6))
    top = (3 + 2) * 5 * math.exp(0.0) + math.exp(-2.0) * 2 * 7
    bottom = abs((3 + 2) * math.exp(0.0) + math.exp(-2.0) * 2)
    assert math.isclose(out[1], top / (max(bottom, 1.0) + 1e-6))


def test_plain_routing_reads_the_bias_and_weighs_the_chosen_alone():
    D = torch.float64
    g = torch.Generator().manual_seed(1)
    mlp = {"router": {"experts": 4, "top": 2}, "expert": {"ff": 3}}
    w = {f"e{e}.{n}": torch.randn(s, generator=g, dtype=D) for e in range(4) for n, s in (("up", (3, 5)), ("down", (5, 3)))}
    w["router"], w["router.b"] = torch.zeros(4, 5, dtype=D), torch.tensor([0.0, 2.0, -1.0, 1.0], dtype=D)
    h = torch.randn(2, 5, generator=g, dtype=D)
    gaps = [[], []]
    got = plain_tadalorn.routed_experts(h, w, "", mlp, gaps)
    share = 1 / (1 + math.exp(-1.0))
    want = share * plain_tadalorn.gelu_expert(h, w["e1.up"], w["e1.down"]) + (1 - share) * plain_tadalorn.gelu_expert(h, w["e3.up"], w["e3.down"])
    assert torch.allclose(got, want) and gaps == [[1.0], [1.0]]
