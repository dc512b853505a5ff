"""The Bodopel design on the GPU against the plain implementation (tests/plain_bodopel.py): each mechanism alone, the residual
stream layer run by layer run, whole prompts, token-by-token decoding, portions down to two tokens, mixed batches on a tight
pool with four slots, long decoding, keys far away, at page borders and at the window's edge, slots and pages used again, greedy
generation through the engine's entry point, and the trace program."""
import math
import random

import numpy as np
import pytest
import torch

import plain_bodopel
import replay_util
from bodopel_configs import CONFIGS, attention, layer, model, write_model
from gpu_common import F32_ATOL, F32_RTOL, need_gpu, note_worst

pytestmark = pytest.mark.gpu
CUDA = torch.device("cuda")
# float32: every row within the bounds the Llama tests use.  bfloat16 (rows, keys and values are kept in bfloat16 between
# kernels; the models are narrow, so a row's error is the sum of few roundings and scatters widely): every row within
# BF16_REL of the largest logit of its sequence, and half of the rows within a third of that.
BF16_REL = 0.025
PAGES = {"BA": 16, "BB": 4, "BC": 8, "BD": 8, "BE": 2}


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    return {name: write_model(config, tmp_path_factory.mktemp(name), seed) for name, (config, seed) in CONFIGS.items()}


_plain: dict = {}


def plain(folder, tokens):
    key = (str(folder), tuple(tokens))
    if key not in _plain:
        if str(folder) not in _plain:
            _plain[str(folder)] = plain_bodopel.read_model_folder(folder)
        config, weights = _plain[str(folder)]
        _plain[key] = plain_bodopel.forward(config, weights, tokens).numpy()
    return _plain[key]


def requests_for(config, seed, lengths):
    g = torch.Generator().manual_seed(900 + seed)
    return {f"q{i}": torch.randint(0, config["vocab"], (n,), generator=g).tolist() for i, n in enumerate(lengths)}


def compare(rows, folder, requests, dtype, what):
    assert rows, "nothing was compared"
    shares = []
    for (name, pos), got_list in rows.items():
        ref = plain(folder, requests[name])
        for got in got_list:
            got = np.asarray(got, dtype=np.float64)
            assert np.isfinite(got).all(), f"{name}@{pos}: non-finite logits"
            err = np.abs(got - ref[pos]).max()
            bound = F32_ATOL + F32_RTOL * np.abs(ref[pos]).max() if dtype == "float32" else BF16_REL * np.abs(ref).max()
            assert err <= bound, f"{what}: {name}@{pos} ({dtype}): max error {err:.3e} exceeds {bound:.3e}"
            shares.append(err / bound)
    note_worst(f"bodopel {what} [{dtype}]", max(shares))
    if dtype == "bfloat16":
        assert sorted(shares)[len(shares) // 2] <= 1 / 3


def make_runner(folder, dtype, max_tokens, page_size=16, max_requests=4):
    from torchinferno_b200.engine.factory import load_model, make_runner as make
    return make(load_model(folder, dtype=dtype), page_size=page_size, max_tokens=max_tokens + page_size * max_requests, max_requests=max_requests)


def run_steps(runner, steps):
    from torchinferno_b200.engine.batch import StepEntry
    out = {}
    with torch.inference_mode():
        for step in steps:
            logits = runner.step([StepEntry(e["id"], e["tokens"], e["want"]) for e in step["entries"]])
            if logits.shape[0]:
                out[step["step"]] = logits.cpu().numpy()
            runner.end(step["end"])
            runner.cache.audit()
    return out


# ------------------------------------------------------------ whole models
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_the_residual_stream_after_every_layer_run(name, folders):
    need_gpu()
    from torchinferno_b200.engine.batch import StepEntry
    from torchinferno_b200.parts.block import PreNormBlock
    config, seed = CONFIGS[name]
    tokens = requests_for(config, seed, [75])["q0"]
    cfg, w = plain_bodopel.read_model_folder(folders[name])
    _, want = plain_bodopel.forward(cfg, w, tokens, return_layers=True)
    runner = make_runner(folders[name], "float32", 96)
    seen, original = [], PreNormBlock.forward

    def recording(self, stream, ctx):
        original(self, stream, ctx)
        seen.append(stream.settle().clone())
    PreNormBlock.forward = recording
    try:
        with torch.inference_mode():
            runner.step([StepEntry("a", tokens, [0])])
    finally:
        PreNormBlock.forward = original
    assert len(seen) == want.shape[0]
    for i, got in enumerate(seen):
        err = (got.cpu().double() - want[i]).abs().max()
        assert err <= 2e-5 * want[i].abs().max(), f"run {i}: {err:.3e}"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_whole_tail_portions_and_mixed_batches(name, dtype, folders):
    need_gpu()
    config, seed = CONFIGS[name]
    requests = requests_for(config, seed, [1, 2, 37, 70, 131, 64, 33])
    for kind, (steps, index) in {
            "whole": replay_util.trace_whole(requests), "tail": replay_util.trace_tail_decode(requests, tail=40),
            "portions": replay_util.trace_portions(requests, sizes=(2, 7, 16, 3, 33, 2, 5, 31, 32, 2, 64)),
            "mixed": replay_util.trace_mixed(requests, seed=seed)}.items():
        runner = make_runner(folders[name], dtype, replay_util.peak_tokens(steps), page_size=PAGES[name])
        rows = replay_util.gather(run_steps(runner, steps), index)
        compare(rows, folders[name], requests, dtype, f"{name} {kind}")
        assert not runner.cache.live_requests


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["BA", "BC", "BD", "BE"])
def test_every_token_decoded_alone_from_the_first_and_long_decoding(name, dtype, folders):
    need_gpu()
    config, seed = CONFIGS[name]
    requests = requests_for(config, seed + 5, [190, 9])
    steps, index = replay_util.trace_tail_decode(requests, tail=10 ** 6)       # one token a step from position 0
    runner = make_runner(folders[name], dtype, replay_util.peak_tokens(steps), page_size=4)
    rows = replay_util.gather(run_steps(runner, steps), index)
    assert runner.counters["graph_steps"] > 100                              # the captured decode pass ran them
    assert runner.counters["pages_freed"] > 0                                # windows gave pages back on the way
    compare(rows, folders[name], requests, dtype, f"{name} token by token")


def test_a_batch_of_unequal_requests_gives_each_what_it_gets_alone(folders):
    need_gpu()
    from torchinferno_b200.engine.batch import StepEntry
    config, seed = CONFIGS["BA"]
    reqs = requests_for(config, seed + 9, [150, 3, 69, 1])
    runner = make_runner(folders["BA"], "float32", 4 * 192, page_size=8)
    with torch.inference_mode():
        alone = {}
        for k, toks in reqs.items():
            alone[k] = runner.step([StepEntry(k + "a", toks, list(range(len(toks))))]).cpu()
            runner.end([k + "a"])
        # together: a portion of each, then the rest of each, in another order (slots and pages are used again)
        first = {k: max(1, len(t) // 2) for k, t in reqs.items()}
        got = {k: [] for k in reqs}
        out = runner.step([StepEntry(k, reqs[k][:first[k]], list(range(first[k]))) for k in reqs]).cpu()
        row = 0
        for k in reqs:
            got[k].append(out[row:row + first[k]]); row += first[k]
        rest = [k for k in reversed(list(reqs)) if len(reqs[k]) > first[k]]
        out = runner.step([StepEntry(k, reqs[k][first[k]:], list(range(len(reqs[k]) - first[k]))) for k in rest]).cpu()
        row = 0
        for k in rest:
            n = len(reqs[k]) - first[k]
            got[k].append(out[row:row + n]); row += n
        runner.end(list(reqs))
    for k in reqs:
        assert torch.allclose(torch.cat(got[k]), alone[k], atol=2e-6, rtol=2e-5), k


def test_a_request_cannot_pass_the_last_learned_position(folders):
    need_gpu()
    from torchinferno_b200.engine.batch import StepEntry
    from torchinferno_b200.engine.runner import StepError
    config, seed = CONFIGS["BB"]
    tokens = requests_for(config, 3, [401])["q0"]
    runner = make_runner(folders["BB"], "float32", 448, page_size=16)
    with torch.inference_mode():
        out = runner.step([StepEntry("a", tokens[:400], [399])]).cpu().numpy()
        assert np.abs(out[0] - plain(folders["BB"], tokens[:400])[399]).max() <= 1e-4 * np.abs(out).max()
        with pytest.raises(StepError):
            runner.step([StepEntry("a", tokens[400:], [0])])


# ------------------------------------------------------- mechanisms alone
def _i32(values):
    return torch.tensor(values, dtype=torch.int32, device=CUDA)


def _entries_batch(entries):
    from torchinferno_b200.engine.batch import EntryPlacement, build_batch
    places, row = [], 0
    for rid, slot, start, n in entries:
        places.append(EntryPlacement(rid, slot, row, n, start))
        row += n
    batch, _ = build_batch(places, [[0] * p.q_len for p in places], [[] for _ in places], [], CUDA)
    return batch


def _bind(part, stored, dtype, prefix):
    """Bind weights given in bfloat16-exact values (as a checkpoint would hold them); returns them in float64 by full name."""
    vectors = {ws.name for ws in part.weight_specs() if ws.role == "vector"}
    part.bind({k: (v.float() if dtype == torch.float32 or k in vectors else v.to(torch.bfloat16)).cuda() for k, v in stored.items()})
    return {prefix + k: v.double() for k, v in stored.items()}


def _apply_tables(cache):
    from torchinferno_b200.kernels import ops
    for group, (idx, val) in zip(cache.groups, cache.drain_table_updates()):
        if idx:
            ops.scatter_i32(group.table_device, _i32(idx), _i32(val))


def _context(cache, entries):
    from torchinferno_b200.parts.base import KVBinding, LayerContext
    b = cache.kv_binding(0)
    return LayerContext(batch=_entries_batch(entries), error_word=cache.error_word,
                        kv=KVBinding(b.pool, b.block_table, b.page_size, b.window, True, b.keys, b.values))


def _cache_for(mixer, dtype, page, pages, max_requests, tokens):
    from torchinferno_b200.cache.manager import CacheManager
    cache = CacheManager([mixer.cache_spec()], [None], page_size=page, num_pages=pages, max_requests=max_requests,
                         max_request_tokens=tokens, dtype=dtype, device=CUDA)
    for group in cache.groups:
        group.pool.fill_(float("nan"))       # (what was never written must never be read)
    return cache


def _run_portions(mixer, cache, name, x, portions, release=False):
    outs, at = [], 0
    for n in portions:
        start = cache.extend(name, n)
        _apply_tables(cache)
        outs.append(mixer.forward(x[at:at + n].cuda().contiguous(), _context(cache, [(name, cache.slot(name), start, n)])))
        if release:
            cache.release_behind_window(name)
        at += n
    assert at == x.shape[0] and int(cache.error_word) == 0
    cache.audit()
    return torch.cat(outs).cpu().double()


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("taps,width", [(1, 16), (2, 50), (3, 64), (4, 520), (5, 44), (8, 96), (9, 40), (30, 13), (4, 6)])
def test_the_input_convolution_in_portions_over_its_carried_rows(dtype, taps, width):
    """Portions shorter and longer than what is carried, single tokens with the norm in the same launch, two requests in a
    step, a slot used again, and another slot's rows and the numbers around the state untouched.  The rows grow with
    position, so that a row taken from one place further or nearer shows."""
    need_gpu()
    from torchinferno_b200.kernels import ops
    g = torch.Generator().manual_seed(taps * 100 + width)
    T, pad = 97, 4
    weight = torch.randn(width, taps, generator=g).to(torch.bfloat16)
    gain = (1 + 0.3 * torch.randn(width, generator=g)).to(torch.bfloat16)
    x = torch.randn(T, width, generator=g) * torch.linspace(0.5, 3.0, T)[:, None]
    want = plain_bodopel.input_convolution(plain_bodopel.rms_norm(x.double(), gain.double(), 1e-5), weight.double())
    other = torch.randn(40, width, generator=g)
    want_other = plain_bodopel.input_convolution(plain_bodopel.rms_norm(other.double(), gain.double(), 1e-5), weight.double())
    wt, gn = weight.float().t().contiguous().cuda(), gain.float().cuda()
    floats = (taps - 1) * width
    state = torch.full((3, floats + 2 * pad), 7.0, device=CUDA)
    tol = 2e-5 if dtype == torch.float32 else 0.02

    def step(parts):
        """parts: (slot, rows); returns the outputs in their order."""
        rows = torch.cat([r for _, r in parts])
        lengths = [len(r) for _, r in parts]
        residual = (rows * 0.25).cuda().contiguous()
        delta = (rows - residual.cpu()).to(dtype).cuda()
        residual += rows.cuda() - (residual + delta.float())          # (what the 16-bit delta leaves out)
        out = torch.empty(rows.shape, dtype=dtype, device=CUDA)
        slots = _i32([s for s, _ in parts])
        if max(lengths) == 1:
            ops.norm_conv_step(delta, residual, gn, 1e-5, wt, state, pad, slots, out)
            assert (residual.cpu() - rows).abs().max() <= 1e-5 * rows.abs().max()
        else:
            normed = torch.empty_like(out)
            ops.add_rmsnorm(delta, residual, gn, 1e-5, normed)
            starts = np.cumsum([0] + lengths).tolist()
            ops.input_conv(normed, out, wt, state, pad, _i32(starts), slots, len(parts), max(lengths))
        return out.cpu().double().split(lengths)

    for slot in (1, 2):
        state[slot, pad:pad + floats] = 0
    got, got_other, at, oat = [], [], 0, 0
    for n, k in ((1, 0), (1, 1), (2, 5), (17, 1), (1, 1), (1, 16), (33, 2), (5, 0), (1, 1), (1, 1), (30, 12), (1, 0), (3, 0)):
        parts = [(1, x[at:at + n])] + ([(2, other[oat:oat + k])] if k else [])
        outs = step(parts)
        got.append(outs[0])
        if k:
            got_other.append(outs[1])
        at, oat = at + n, oat + k
    assert at == T and oat == 40
    got, got_other = torch.cat(got), torch.cat(got_other)
    assert ((got - want).abs().max(dim=1).values <= tol * want.abs().max()).all()
    assert (got_other - want_other).abs().max() <= tol * want_other.abs().max()
    # losing what is carried shows at a portion's start, and so does a row too many
    if taps > 1:
        fresh = plain_bodopel.input_convolution(plain_bodopel.rms_norm(x[20:].double(), gain.double(), 1e-5), weight.double())
        assert (fresh[0] - want[20]).abs().max() > 10 * tol * want[20].abs().max()
        carried = state[1, pad:pad + floats].view(taps - 1, width).cpu().double()
        rows = torch.cat([torch.zeros(taps, width, dtype=torch.float64), plain_bodopel.rms_norm(x.double(), gain.double(), 1e-5)])[-(taps - 1):]
        assert (carried - rows).abs().max() <= (1e-5 if dtype == torch.float32 else 0.01) * rows.abs().max()
    assert float((state[0] - 7).abs().max()) == 0.0 and float((state[:, :pad] - 7).abs().max()) == 0.0 \
        and float((state[:, pad + floats:] - 7).abs().max()) == 0.0
    # the slot goes to a new request
    state[1, pad:pad + floats] = 0
    again = torch.cat(step([(1, x[:1])]) + step([(1, x[1:4])]))
    assert (again - want[:4]).abs().max() <= tol * want.abs().max()


def _direct_attention(m, dtype, seed, max_positions=2000):
    """An attention whose input row is [q | k | v | gate] itself: the projections pick their columns (the products are then
    exact in both number formats), so that a test sets queries, keys and values by hand.  Biases, norm weights, the heads'
    matrix, the decay and the output projection are random.  Returns (mixer, weights in float64, the columns' starts)."""
    from torchinferno_b200.parts.base import PartSpec, build_part
    from torchinferno_b200.weights.random_init import random_tensor
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    widths = {"q": H * d, "k": G * d, "v": G * dv, "g": H * dv}
    W = sum(widths.values())
    mixer = build_part("mixer", PartSpec("talking_heads_attention", {
        "hidden_size": W, "heads": H, "kv_heads": G, "dim": d, "value_dim": dv, "scale": m["scale"], "max_positions": max_positions,
        "window": None if m["mask"] is None else m["mask"]["size"], "softcap": m["softcap"], "bias": True, "row_norm_eps": 1e-5,
        "distance_decay": True, "gate": True}), dtype=dtype, device=CUDA)
    stored = {ws.name: random_tensor(ws, seed, dtype=torch.bfloat16) for ws in mixer.weight_specs()}
    starts, at = {}, 0
    for name, width in widths.items():
        pick = torch.zeros(width, W)
        pick[torch.arange(width), at + torch.arange(width)] = 1.0
        stored[name] = pick.to(torch.bfloat16)
        starts[name], at = at, at + width
    return mixer, _bind(mixer, stored, dtype, "mix."), starts


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads,kv_heads,dim,vdim,window,softcap,page", [
    (4, 2, 16, 24, 20, 2.0, 8), (3, 1, 40, 8, 7, 5.0, 4), (2, 2, 64, 64, 33, 50.0, 16), (2, 1, 8, 4, 2, 3.0, 2),
    (1, 1, 12, 6, 1, None, 4), (6, 2, 32, 32, 64, 8.0, 16), (6, 3, 128, 72, 65, 4.0, 8), (5, 5, 16, 16, 63, 10.0, 16), (17, 1, 8, 16, 30, 6.0, 8),
    (16, 1, 16, 16, 9, 6.0, 8), (36, 4, 8, 8, 70, 20.0, 16), (3, 1, 200, 136, 40, 6.0, 8)])
def test_the_attention_alone_at_the_edges_of_windows_and_pages(dtype, heads, kv_heads, dim, vdim, window, softcap, page):
    """A prompt in portions, then single tokens, in a pool whose pages were used before and go back as the window leaves them.
    Some tokens carry values thirty times the usual size: a query that sees such a token one position too long or too short,
    in a prompt or decoded alone, is far off, and so is one that reads a wrong page, leaves the heads unmixed or mixes them
    the other way round, leaves the cap, a bias or a norm's weight out, or takes the distance one off."""
    need_gpu()
    m = attention(heads, kv_heads, dim, vdim, 2.0 / math.sqrt(dim), window, softcap)
    mixer, w, starts = _direct_attention(m, dtype, seed=3)
    w["mix.talk"] = (torch.eye(heads, dtype=torch.float64) + 0.5 * torch.randn(heads, heads, generator=torch.Generator().manual_seed(1),
                                                                               dtype=torch.float64)).to(torch.bfloat16).double()
    _bind(mixer, {k[4:]: v for k, v in w.items()}, dtype, "mix.")
    T = 2 * window + 4 * page + 75
    g = torch.Generator().manual_seed(window * 100 + heads)
    x = torch.randn(T, mixer.hidden_size, generator=g)
    v0, v1 = starts["v"], starts["v"] + kv_heads * vdim
    for p in (3, page - 1, page, page + window, T - window - 2, T - window - 1, T - 2 - window // 2):
        if p >= 0:
            x[p, v0:v1] *= 30
    x = x.to(torch.bfloat16).to(dtype)
    want = plain_bodopel.attention(x.double(), w, "mix.", m, 1e-5)

    def differs(other):
        return float(((other - want).abs().max(dim=1).values / want.abs().max(dim=1).values).max())

    tol = 2e-5 if dtype == torch.float32 else BF16_REL
    run = lambda weights=w, **changes: plain_bodopel.attention(x.double(), weights, "mix.", {**m, **changes}, 1e-5)
    # the test can tell
    assert differs(run(mask={"size": window + 1})) > 0.2
    if window > 1:
        assert differs(run(mask={"size": window - 1})) > 0.2
        assert differs(run(dict(w, **{"mix.r1": 0 * w["mix.r1"]}))) > 0.05
        if softcap is not None and softcap <= 5:
            assert differs(run(softcap=None)) > 0.02
        assert differs(run(dict(w, **{"mix.q.b": 0 * w["mix.q.b"]}))) > 0.05
        assert differs(run(dict(w, **{"mix.k.norm": torch.ones_like(w["mix.k.norm"])}))) > 0.01
    if heads > 1:
        assert differs(run(dict(w, **{"mix.talk": w["mix.talk"].T}))) > 0.1
    cache = _cache_for(mixer, dtype, page, -(-T // page) + 8, 3, T + page)
    cache.open("old"), cache.extend("old", 2 * page + 1), cache.open("warm"), cache.extend("warm", page + 1)
    cache.close("old")                  # its pages go to "r", out of order
    cache.open("r")
    portions = [max(window - 1, 1), 2, page, 1, 1, window // 2 + 3, 2]
    portions += [1] * (T - sum(portions))
    got = _run_portions(mixer, cache, "r", x, portions, release=True)
    scale = want.abs().max(dim=1).values.clamp(min=0.05 * float(want.abs().max()))
    err = (got - want).abs().max(dim=1).values / scale
    assert err.max() <= tol, (int(err.argmax()), float(err.max()))
    note_worst(f"bodopel attention alone [{dtype}]", float(err.max()) / tol)
    # a second request in the slot and pages the first one leaves, whole: nothing of the first shows
    cache.close("r"), cache.close("warm")
    cache.open("s")
    again = _run_portions(mixer, cache, "s", x[:window + 40], [window + 38, 2])
    assert ((again - want[:window + 40]).abs().max(dim=1).values / scale[:window + 40]).max() <= tol


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_a_far_key_just_inside_and_just_outside_the_window_with_two_requests_side_by_side(dtype):
    """700 tokens, a window of 600, pages of 16: the token at position 95 has a value a hundred times the usual size and a key
    along the direction of the last queries, and takes most of their weight among 600 keys; it is in sight up to position
    694 and out of it from 695 on, which decoded tokens pass.  A second, shorter request is in the same steps."""
    need_gpu()
    m = attention(4, 2, 32, 16, 0.6, 600, 30.0)
    mixer, w, starts = _direct_attention(m, dtype, seed=5)
    w["mix.r1"] *= 0.25
    w["mix.q.b"] *= 0
    w["mix.k.b"] *= 0
    w = {k: v.to(torch.bfloat16).double() for k, v in w.items()}
    _bind(mixer, {k[4:]: v for k, v in w.items()}, dtype, "mix.")
    T, far = 700, 95
    g = torch.Generator().manual_seed(11)
    x = torch.randn(T, mixer.hidden_size, generator=g)
    looked = torch.randn(32, generator=g)
    for h in range(4):
        x[-12:, starts["q"] + h * 32:starts["q"] + (h + 1) * 32] = looked + 0.1 * torch.randn(12, 32, generator=g)
    for kh in range(2):
        x[far, starts["k"] + kh * 32:starts["k"] + (kh + 1) * 32] = looked
    x[far, starts["v"]:starts["g"]] *= 100
    x = x.to(torch.bfloat16).to(dtype)
    other = torch.randn(90, mixer.hidden_size, generator=g).to(torch.bfloat16).to(dtype)
    want = plain_bodopel.attention(x.double(), w, "mix.", m, 1e-5)
    want_other = plain_bodopel.attention(other.double(), w, "mix.", m, 1e-5)
    assert want[694].abs().max() > 10 * want[695].abs().max()                  # inside and outside differ by far
    cache = _cache_for(mixer, dtype, 16, 60, 3, 720)
    cache.open("r"), cache.open("o")
    outs, outs_other, at, oat = [], [], 0, 0
    for n, k in ((600, 50), (90, 2), (1, 1), (1, 30), (1, 1), (1, 0), (1, 1), (1, 5), (4, 0)):
        start, ostart = cache.extend("r", n), (cache.extend("o", k) if k else 0)
        _apply_tables(cache)
        entries = [("r", cache.slot("r"), start, n)] + ([("o", cache.slot("o"), ostart, k)] if k else [])
        rows = torch.cat([x[at:at + n]] + ([other[oat:oat + k]] if k else [])).cuda().contiguous()
        out = mixer.forward(rows, _context(cache, entries))
        outs.append(out[:n]), outs_other.append(out[n:])
        at, oat = at + n, oat + k
    assert at == T and int(cache.error_word) == 0
    got, got_other = torch.cat(outs).cpu().double(), torch.cat(outs_other).cpu().double()
    tol = 2e-5 if dtype == torch.float32 else BF16_REL
    rows = (got - want).abs().max(dim=1).values / want.abs().max(dim=1).values.clamp(min=0.01 * float(want.abs().max()))
    assert rows.max() <= tol, (int(rows.argmax()), float(rows.max()))
    assert (got_other - want_other).abs().max() <= tol * want_other.abs().max()


@pytest.mark.parametrize("heads,kv_heads,dim,vdim,window,page", [
    (4, 2, 32, 16, 300, 16), (16, 1, 128, 128, 1 << 30, 16), (3, 3, 8, 72, 64, 4), (8, 4, 96, 96, 65, 8), (24, 12, 64, 40, 129, 32), (40, 8, 16, 16, 1 << 30, 16)])
def test_the_forms_of_the_kernel_against_plain_arithmetic(heads, kv_heads, dim, vdim, window, page):
    """Single tokens at contexts of 1 to 700 keys whose keys are shared out over blocks in tiles of 1, 2, 3 and all, and short
    portions at the same contexts whose scratch holds all tokens, a few, or one range of 64; every form against float64, with
    scores beyond the cap, a heads' matrix that bfloat16 does not hold exactly, a gate, and NaN in all unwritten cache."""
    need_gpu()
    from torchinferno_b200.kernels import ops
    g = torch.Generator().manual_seed(heads * 10 + dim)
    lengths = {"single": [1] * 6, "portions": [40, 1, 65, 2, 130, 129]}
    contexts = [700, 1, 65, 64, 333, 129]
    n = len(contexts)
    per = -(-max(contexts) // page)
    keys = torch.full((n * per + 3, kv_heads, page, dim), float("nan"))
    values = torch.full((n * per + 3, kv_heads, page, vdim), float("nan"))
    table = torch.randperm(n * per + 3, generator=g)[:n * per].view(n, per).to(torch.int32)
    k_all = [torch.randn(c, kv_heads, dim, generator=g).to(torch.bfloat16) for c in contexts]
    v_all = [torch.randn(c, kv_heads, vdim, generator=g).to(torch.bfloat16) for c in contexts]
    for e, c in enumerate(contexts):
        for pos in range(c):
            keys[table[e, pos // page], :, pos % page] = k_all[e][pos].float()
            values[table[e, pos // page], :, pos % page] = v_all[e][pos].float()
    pool = torch.cat([keys.flatten(1), values.flatten(1)], dim=1).to(torch.bfloat16).cuda()
    keys_d = pool[:, :kv_heads * page * dim].unflatten(1, (kv_heads, page, dim))
    values_d = pool[:, kv_heads * page * dim:].unflatten(1, (kv_heads, page, vdim))
    span, cap, scale = 90, 3.0, 1.5 / math.sqrt(dim)
    bias = -torch.rand(heads, span, generator=g).cumsum(dim=1) * 0.1
    talk = torch.eye(heads) + 0.3 * torch.randn(heads, heads, generator=g)
    padded = 16 if heads <= 16 else 32 if heads <= 32 else 64
    wide = torch.zeros(padded, padded)
    wide[:heads, :heads] = talk
    hi = wide.to(torch.bfloat16)
    lo = (wide - hi.float()).to(torch.bfloat16)
    for mode, lens in lengths.items():
        lens = [min(q, c) for q, c in zip(lens, contexts)]
        total = sum(lens)
        q = torch.randn(total, heads, dim, generator=g).to(torch.bfloat16)
        gate = torch.randn(total, heads * vdim + 5, generator=g).to(torch.bfloat16)
        want = torch.zeros(total, heads, vdim, dtype=torch.float64)
        row, positions = 0, []
        for e, c in enumerate(contexts):
            for i in range(c - lens[e], c):
                first = max(0, i - window + 1)
                kk = k_all[e][first:i + 1].double().repeat_interleave(heads // kv_heads, dim=1)
                vv = v_all[e][first:i + 1].double().repeat_interleave(heads // kv_heads, dim=1)
                s = cap * torch.tanh(torch.einsum("hd,jhd->hj", q[row].double(), kk) * scale / cap)
                s = s + bias.double()[:, (i - torch.arange(first, i + 1)).clamp(max=span - 1)]
                mixed = talk.double() @ torch.softmax(s, dim=-1)
                want[row] = torch.einsum("hj,jhd->hd", mixed, vv)
                positions.append(i)
                row += 1
        want = want.flatten(1) * torch.sigmoid(gate[:, 5:].double())
        starts = np.cumsum([0] + lens).tolist()
        cases = [dict(force_simt=True)]
        if mode == "single":
            cases += [dict(tiles_per_part=t) for t in (1, 2, 3, 11)] + [dict(), dict(force_portions=True)]
        else:
            cases += [dict(), dict(scratch_bytes=1), dict(scratch_bytes=heads * 768 * 4 * 100)]
        for case in cases:
            out = torch.full((total, heads * vdim), float("nan"), dtype=torch.bfloat16, device=CUDA)
            error = torch.zeros(1, dtype=torch.int32, device=CUDA)
            ops.talking_heads_attention(
                q.flatten(1).cuda(), out, _i32(starts), _i32([c - k for c, k in zip(contexts, lens)]), _i32(list(range(n))), _i32(positions),
                keys_d, values_d, table.cuda(), n, max(lens), heads, kv_heads, window=window, scale=scale, softcap=cap, bias=bias.cuda(),
                talk=talk.cuda(), talk_hi=hi.cuda(), talk_lo=lo.cuda(), gate=gate.cuda()[:, 5:], max_kv_len=max(contexts), error_word=error, **case)
            got = out.cpu().double()
            assert torch.isfinite(got).all() and int(error) == 0, (mode, case)
            # (inputs and weights are exact here: what is left is the sums' and the output's rounding)
            assert (got - want).abs().max() <= 0.006 * want.abs().max(), (mode, case, float((got - want).abs().max() / want.abs().max()))


def test_norms_over_whole_rows_with_biases_and_the_store():
    """q and k normed over all heads at once (a norm per head gives other rows), biases ahead of it, keys and values in their
    pages and nowhere else, in both number formats, with widths that vector loads take and that they do not."""
    need_gpu()
    from torchinferno_b200.kernels import ops
    g = torch.Generator().manual_seed(3)
    for dtype, heads, kv, d, dv, page in ((torch.float32, 3, 1, 7, 5, 4), (torch.bfloat16, 4, 2, 16, 24, 8), (torch.bfloat16, 5, 5, 6, 10, 4),
                                          (torch.bfloat16, 72, 36, 128, 128, 16), (torch.float32, 8, 4, 300, 40, 16)):
        n = 11
        up = lambda v: -(-v // 8) * 8
        k_off = up(heads * d)
        v_off = up(k_off + kv * d)
        proj = (torch.randn(n, up(v_off + kv * dv), generator=g) * torch.rand(n, 1, generator=g).mul(4)).to(dtype)
        bias = [torch.randn(width, generator=g) for width in (heads * d, kv * d, kv * dv)]
        gain = [1 + 0.2 * torch.randn(width, generator=g) for width in (heads * d, kv * d)]
        pool = torch.full((6, kv * page * (d + dv)), float("nan")).to(dtype).cuda()
        keys, values = pool[:, :kv * page * d].unflatten(1, (kv, page, d)), pool[:, kv * page * d:].unflatten(1, (kv, page, dv))
        table = torch.tensor([[5, 0, 3], [1, 4, 2]], dtype=torch.int32, device=CUDA)
        slots, positions = [0] * 6 + [1] * 5, list(range(2, 8)) + list(range(5))
        q_out, error = torch.empty(n, heads * d, dtype=dtype, device=CUDA), torch.zeros(1, dtype=torch.int32, device=CUDA)
        ops.row_norm_append(proj.cuda(), 0, k_off, v_off, q_out, keys, values, _i32(positions), _i32(slots), table, heads, kv, d, dv, eps=1e-5,
                            q_bias=bias[0].cuda(), k_bias=bias[1].cuda(), v_bias=bias[2].cuda(), q_weight=gain[0].cuda(),
                            k_weight=gain[1].cuda(), error_word=error)
        tol = 1e-5 if dtype == torch.float32 else 0.006
        want_q = plain_bodopel.rms_norm(proj[:, :heads * d].double() + bias[0].double(), gain[0].double(), 1e-5)
        want_k = plain_bodopel.rms_norm(proj[:, k_off:k_off + kv * d].double() + bias[1].double(), gain[1].double(), 1e-5).view(n, kv, d)
        want_v = (proj[:, v_off:v_off + kv * dv].double() + bias[2].double()).view(n, kv, dv)
        assert (q_out.cpu().double() - want_q).abs().max() <= tol * want_q.abs().max() and int(error) == 0
        tb = table.cpu()
        for t in range(n):
            at = int(tb[slots[t], positions[t] // page]), positions[t] % page
            assert (keys[at[0], :, at[1]].cpu().double() - want_k[t]).abs().max() <= tol * want_k.abs().max()
            assert (values[at[0], :, at[1]].cpu().double() - want_v[t]).abs().max() <= tol * want_v.abs().max()
        assert int(torch.isfinite(keys).sum()) == n * kv * d and int(torch.isfinite(values).sum()) == n * kv * dv


def test_scaled_embedding_with_learned_positions_and_the_vector_of_a_pass():
    need_gpu()
    from torchinferno_b200.kernels import ops
    g = torch.Generator().manual_seed(4)
    for dtype, width in ((torch.float32, 50), (torch.bfloat16, 50), (torch.bfloat16, 264)):
        table, pos = torch.randn(9, width, generator=g).to(dtype), torch.randn(7, width, generator=g).to(dtype)
        ids, at = [3, 0, 8, 9, 2], [6, 0, 3, 1, 7]
        out = torch.empty(5, width, device=CUDA)
        ops.embedding(_i32(ids), table.cuda(), out, scale=1.7, positions=_i32(at), position_table=pos.cuda())
        want = table[[3, 0, 8]].double() * 1.7 + pos[[6, 0, 3]].double()
        assert (out[:3].cpu().double() - want).abs().max() <= 1e-6 * want.abs().max()
        assert torch.isnan(out[3:]).all()                     # an id or a position outside its table shows
        ops.embedding(_i32(ids), table.cuda(), out)
        assert torch.equal(out[:3].cpu(), table[[3, 0, 8]].float())
        x, v, delta = torch.randn(5, width, generator=g), torch.randn(width, generator=g), torch.randn(5, width, generator=g).to(dtype)
        got = ops.add_vector(x.cuda(), v.cuda(), delta.cuda()).cpu()
        assert (got - (x + delta.float() + v)).abs().max() <= 1e-5
        assert (ops.add_vector(x.cuda(), v.cuda()).cpu() - (x + v)).abs().max() <= 1e-6


# ------------------------------------------------ entry point and programs
def test_greedy_generation_through_the_engine_and_its_scheduler(folders):
    need_gpu()
    from torchinferno_b200.config.engine_config import EngineConfig
    from torchinferno_b200.engine.engine import InferenceEngine
    from torchinferno_b200.engine.types import GenerateRequest, SamplingConfig
    config, seed = CONFIGS["BA"]
    cfg, w = plain_bodopel.read_model_folder(folders["BA"])
    prompts = list(requests_for(config, seed + 2, [5, 41, 1, 18, 66]).values())
    new = 30                                                # (decoding passes the shortest window)
    for dtype in ("float32", "bfloat16"):
        with InferenceEngine.from_config(EngineConfig(model=str(folders["BA"]), dtype=dtype, page_size=8, max_batch_size=3,
                                                      prefill_chunk_size=16, max_num_batched_tokens=48, kv_cache_tokens=512)) as engine:
            outs = engine.generate_many([GenerateRequest(f"g{i}", prompt_token_ids=p, sampling=SamplingConfig(new))
                                         for i, p in enumerate(prompts)])
        for prompt, out in zip(prompts, outs):
            tokens = list(out.token_ids)
            assert len(tokens) == new
            logits = plain_bodopel.forward(cfg, w, (prompt + tokens)[:-1])
            for i, tok in enumerate(tokens):
                row = logits[len(prompt) + i - 1]
                short = float(row.max() - row[tok])         # by how much the drawn token misses the best
                assert short <= (1e-4 if dtype == "float32" else BF16_REL) * float(logits.abs().max())


def test_the_command_line_generates_from_a_bodopel_folder(folders, capsys):
    need_gpu()
    from torchinferno_b200 import cli
    assert cli.main(["generate", str(folders["BC"]), "--input-ids", "5", "3", "9", "--new-tokens", "4", "--dtype", "float32"]) == 0
    assert capsys.readouterr().out.strip()


def test_the_trace_program_replays_a_bodopel_folder(folders, tmp_path):
    need_gpu()
    config, seed = CONFIGS["BC"]
    requests = requests_for(config, seed + 3, [30, 75, 2])
    steps, index = replay_util.trace_mixed(requests, seed=3)
    results = replay_util.run_trace_program(folders["BC"], "float32", replay_util.peak_tokens(steps), steps, tmp_path / "out")
    compare(replay_util.gather(results, index), folders["BC"], requests, "float32", "BC trace program")


# ------------------------------------------------------- sizes drawn at random
def _random_config(rng):
    """A small Bodopel configuration with sizes drawn from lists that mix multiples of 8, 16, 64 with odd ones."""
    pick = rng.choice
    layers = []
    for _ in range(pick([1, 2, 3, 4])):
        kv_heads, dim = pick([1, 2, 3, 5]), pick([4, 8, 12, 24, 40, 64])
        layers.append(layer(attention(kv_heads * pick([1, 2, 3, 4]), kv_heads, dim, pick([2, 6, 8, 20, 40, 72]), pick([0.1, 0.3]),
                                      pick([1, 2, 9, 31, 32, 64, 65, 300]), pick([None, 1.5, 8.0, 50.0])), pick([None, 8, 24, 36, 70])))
    loop = None
    if rng.random() < 0.7:
        start = rng.randrange(len(layers))
        loop = (start, rng.randint(start + 1, len(layers)), pick([1, 2, 3]))
    return model(pick([50, 97, 128]), pick([24, 40, 72, 96, 136]), pick([1, 2, 3, 4, 6, 9]), layers, loop, scale=pick([1.0, 5.5]),
                 eps=pick([1e-6, 1e-5]), max_positions=pick([80, 128, 1000]))


@pytest.mark.parametrize("draw", range(8))
def test_sizes_drawn_at_random(draw, tmp_path):
    """Whole prompts, portions and token-by-token decoding of models whose every size was drawn at random, in both number
    formats."""
    need_gpu()
    rng = random.Random(7700 + draw)
    config = _random_config(rng)
    write_model(config, tmp_path, seed=draw)
    requests = requests_for(config, 50 + draw, [41, 3, 70])
    for dtype in ("float32", "bfloat16"):
        for kind, (steps, index) in {"whole": replay_util.trace_whole(requests), "tail": replay_util.trace_tail_decode(requests, tail=12),
                                     "portions": replay_util.trace_portions(requests, sizes=(2, 31, 3, 33, 2, 16))}.items():
            runner = make_runner(tmp_path, dtype, replay_util.peak_tokens(steps), page_size=rng.choice([4, 16]))
            rows = replay_util.gather(run_steps(runner, steps), index)
            compare(rows, tmp_path, requests, dtype, f"draw {draw} {kind}")
