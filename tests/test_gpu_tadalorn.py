"""The Tadalorn design on the GPU against the plain implementation (tests/plain_tadalorn.py): each mechanism alone, the residual
stream layer by layer, whole prompts, token-by-token decoding, portions down to two tokens, mixed batches on a tight pool with four
slots, long decoding, keys far away, at page borders, at the window's edge and at the edge of the kept tokens, slots and pages used
again, greedy generation through the engine's entry point, and the trace program."""
import math
import random

import numpy as np
import pytest
import torch

import plain_tadalorn
import replay_util
from gpu_common import F32_ATOL, F32_RTOL, need_gpu, note_worst
from tadalorn_configs import CONFIGS, attention, dense, latent, layer, mlstm, model, moe, write_model

pytestmark = pytest.mark.gpu
CUDA = torch.device("cuda")
# float32: every row within the bounds the Llama tests use, but for a token at which a router's last chosen logit lies within CLOSE
# of the next one (it may choose otherwise after rounding, which is no rounding error).
# bfloat16: a memory whose readout nearly cancels is divided by its own small root mean square, which makes a few rows' rounding
# errors large (the float64 model with every product's operands and results rounded to bfloat16 has its median row at 0.006 to 0.010 of
# the sequence's largest logit, nine in ten below 0.018 and the worst at 0.02 to 0.09).  So: half of the rows within a third of
# BF16_REL, nine in ten within BF16_REL, all within four times that.  With routers half of the rows within half of BF16_REL and no
# bound on the worst: now and then a token is routed differently from the float64 model, and what it then leaves in keys and states
# is read by every later token of its request.
CLOSE = {"float32": 2e-5, "bfloat16": 0.1}
BF16_REL = 0.045
PAGES = {"TA": 16, "TB": 4, "TC": 8, "TD": 8, "TE": 2}


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    return {name: write_model(config, tmp_path_factory.mktemp(name), seed) for name, (config, seed) in CONFIGS.items()}


_plain: dict = {}


def plain(folder, tokens, dtype):
    """(logits [T, vocab], positions that a router's close call makes incomparable, whether there are routers)."""
    key = (str(folder), tuple(tokens))
    if key not in _plain:
        if str(folder) not in _plain:
            _plain[str(folder)] = plain_tadalorn.read_model_folder(folder)
        config, weights = _plain[str(folder)]
        gaps = [[] for _ in tokens]
        _plain[key] = (plain_tadalorn.forward(config, weights, tokens, gaps=gaps).numpy(), gaps)
    logits, gaps = _plain[key]
    return logits, {t for t, g in enumerate(gaps) if min(g, default=1.0) < CLOSE[dtype]}, any(gaps)


def requests_for(config, seed, lengths):
    g = torch.Generator().manual_seed(900 + seed)
    return {f"q{i}": torch.randint(0, config["vocab"], (n,), generator=g).tolist() for i, n in enumerate(lengths)}


def compare(rows, folder, requests, dtype, what):
    shares, routed = [], False
    for (name, pos), got_list in rows.items():
        ref, close, routers = plain(folder, requests[name], dtype)
        routed = routed or routers
        if pos in close:
            continue
        for got in got_list:
            got = np.asarray(got, dtype=np.float64)
            assert np.isfinite(got).all(), f"{name}@{pos}: non-finite logits"
            err = np.abs(got - ref[pos]).max()
            bound = F32_ATOL + F32_RTOL * np.abs(ref[pos]).max() if dtype == "float32" else BF16_REL * np.abs(ref).max()
            if dtype == "float32" or not routers:
                assert err <= (1 if dtype == "float32" else 4) * bound, f"{what}: {name}@{pos} ({dtype}): max error {err:.3e}, bound {bound:.3e}"
            shares.append(err / bound)
    assert len(shares) >= max(1, len(rows) // 3), f"{what}: only {len(shares)} of {len(rows)} rows could be compared"
    shares = sorted(shares)
    if dtype == "bfloat16":
        assert shares[len(shares) // 2] <= (1 / 2 if routed else 1 / 3), f"{what}: the median row is at {shares[len(shares) // 2]:.2f} of the bound"
        ninth = shares[int(0.9 * (len(shares) - 1))]
        assert ninth <= 1.0, f"{what}: nine in ten rows within {ninth:.2f} of the bound"
        return note_worst(f"tadalorn {what}, nine rows in ten [{dtype}]", ninth)
    note_worst(f"tadalorn {what} [{dtype}]", shares[-1])


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
def test_the_residual_stream_after_every_layer(name, folders):
    need_gpu()
    from torchinferno_b200.engine.batch import StepEntry
    from torchinferno_b200.parts.postnorm_block import PostNormBlock
    config, seed = CONFIGS[name]
    tokens = requests_for(config, seed, [75])["q0"]
    cfg, w = plain_tadalorn.read_model_folder(folders[name])
    _, want = plain_tadalorn.forward(cfg, w, tokens, return_layers=True)
    runner = make_runner(folders[name], "float32", 96)
    seen, original = [], PostNormBlock.forward

    def recording(self, stream, ctx):
        original(self, stream, ctx)
        seen.append(stream.settle().clone())
    PostNormBlock.forward = recording
    try:
        with torch.inference_mode():
            runner.step([StepEntry("a", tokens, [0])])
    finally:
        PostNormBlock.forward = original
    assert len(seen) == want.shape[0]
    for i, got in enumerate(seen):
        err = (got.cpu().double() - want[i]).abs().max()
        assert err <= 2e-5 * want[i].abs().max(), f"layer {i}: {err:.3e}"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_whole_tail_portions_and_mixed_batches(name, dtype, folders):
    need_gpu()
    config, seed = CONFIGS[name]
    requests = requests_for(config, seed, [1, 2, 37, 70, 150, 64, 33])
    for kind, (steps, index) in {
            "whole": replay_util.trace_whole(requests), "tail": replay_util.trace_tail_decode(requests, tail=40),
            "portions": replay_util.trace_portions(requests, sizes=(2, 7, 16, 3, 33, 2, 5, 31, 32, 2, 64)),
            "mixed": replay_util.trace_mixed(requests, seed=seed)}.items():
        runner = make_runner(folders[name], dtype, replay_util.peak_tokens(steps), page_size=PAGES[name])
        rows = replay_util.gather(run_steps(runner, steps), index)
        compare(rows, folders[name], requests, dtype, f"{name} {kind}")
        assert not runner.cache.live_requests


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_every_token_decoded_alone_from_the_first_and_long_decoding(name, dtype, folders):
    need_gpu()
    config, seed = CONFIGS[name]
    requests = requests_for(config, seed + 5, [190, 9])
    steps, index = replay_util.trace_tail_decode(requests, tail=10 ** 6)       # one token a step from position 0
    runner = make_runner(folders[name], dtype, replay_util.peak_tokens(steps), page_size=4)
    rows = replay_util.gather(run_steps(runner, steps), index)
    assert runner.counters["graph_steps"] > 100                              # the captured decode pass ran them
    if any(entry["type"] == "attention" and entry["mixer"]["mask"] for entry in config["layers"]):
        assert runner.counters["pages_freed"] > 0                            # windows gave pages back on the way
    compare(rows, folders[name], requests, dtype, f"{name} token by token")


@pytest.mark.parametrize("name", ["TA", "TD", "TE"])
def test_a_batch_of_unequal_requests_gives_each_what_it_gets_alone(name, folders):
    need_gpu()
    from torchinferno_b200.engine.batch import StepEntry
    config, seed = CONFIGS[name]
    reqs = requests_for(config, seed + 9, [150, 3, 69, 1])
    runner = make_runner(folders[name], "float32", 4 * 192, page_size=8)
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
        assert torch.allclose(torch.cat(got[k]), alone[k], atol=1e-5, rtol=5e-5), k


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
    kv = None
    if cache.groups:
        b = cache.kv_binding(0)
        kv = KVBinding(b.pool, b.block_table, b.page_size, b.window, True, b.keys, b.values)
    return LayerContext(batch=_entries_batch(entries), error_word=cache.error_word, kv=kv, state=cache.state(0))


def _cache_for(mixer, dtype, page, pages, max_requests, tokens):
    from torchinferno_b200.cache.manager import CacheManager
    spec = mixer.cache_spec()
    cache = CacheManager([] if spec is None else [spec], [mixer.state_spec()], page_size=page, num_pages=pages, max_requests=max_requests,
                         max_request_tokens=tokens, dtype=dtype, device=CUDA)
    for group in cache.groups:
        group.pool.fill_(float("nan"))       # (what was never written must never be read)
    if cache.state(0) is not None:
        cache.state(0).fill_(float("nan"))   # (zeroed for a new request, and nobody else's is read)
    return cache


def _run_steps(mixer, cache, steps, rows_of):
    """steps: lists of (request, tokens of it); rows_of: its input rows.  Returns every request's outputs in float64."""
    outs, at = {name: [] for name in rows_of}, {name: 0 for name in rows_of}
    for step in steps:
        entries, rows = [], []
        for name, n in step:
            start = cache.extend(name, n)
            entries.append((name, cache.slot(name), start, n))
            rows.append(rows_of[name][at[name]:at[name] + n])
            at[name] += n
        _apply_tables(cache)
        out = mixer.forward(torch.cat(rows).cuda().contiguous(), _context(cache, entries))
        for (name, n), part in zip(step, out.split([n for _, n in step])):
            outs[name].append(part)
            cache.release_behind_window(name)
    assert all(at[name] == len(rows) for name, rows in rows_of.items()) and int(cache.error_word) == 0
    cache.audit()
    return {name: torch.cat(parts).cpu().double() for name, parts in outs.items()}


def _row_error(got, want, floor=0.05):
    """The largest error of a row as a share of its own largest element (a small row counts as ``floor`` of the largest)."""
    scale = want.abs().max(dim=1).values.clamp(min=floor * float(want.abs().max()))
    return (got - want).abs().max(dim=1).values / scale


def _picked_columns(mixer, widths, stored):
    """Projections that pick their columns from an input row laid out as ``widths`` says: the products are then exact in both number
    formats, and a test sets queries, keys and values by hand.  Returns the columns' starts."""
    starts, at, W = {}, 0, sum(widths.values())
    for name, width in widths.items():
        pick = torch.zeros(width, W)
        pick[torch.arange(width), at + torch.arange(width)] = 1.0
        stored[name] = pick.to(torch.bfloat16)
        starts[name], at = at, at + width
    return starts


def _direct_attention(m, dtype, seed):
    from torchinferno_b200.parts.base import PartSpec, build_part
    from torchinferno_b200.weights.random_init import random_tensor
    H, G, d = m["heads"], m["kv_heads"], m["dim"]
    widths = {"q": H * d, "k": G * d, "g": H * d}
    mask = m["mask"]
    mixer = build_part("mixer", PartSpec("kept_window_attention", {
        "hidden_size": sum(widths.values()), "heads": H, "kv_heads": G, "dim": d, "scale": m["scale"], "taps": m["conv"],
        "window": None if mask is None else mask["size"], "keep_first": 0 if mask is None else mask["keep_first"], "row_norm_eps": 1e-5,
        "sink": "one", "gate": True, "position": PartSpec("rotary", {
            "head_dim": d, "theta": m["rot"]["base"], "rot_dim": m["rot"]["dims"], "interleaved": True, "exact": True})}), dtype=dtype, device=CUDA)
    stored = {ws.name: random_tensor(ws, seed, dtype=torch.bfloat16) for ws in mixer.weight_specs()}
    starts = _picked_columns(mixer, widths, stored)
    return mixer, stored, starts


def _attention(x, w, m):
    return plain_tadalorn.window_attention(x.double(), w, "mix.", m, 1e-5, torch.arange(x.shape[0]))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads,kv_heads,dim,taps,window,keep,rot,page", [
    (4, 2, 16, 3, 20, 3, 8, 8), (3, 1, 40, 4, 7, 1, 40, 4), (2, 2, 64, 2, 33, 40, 24, 16), (2, 1, 8, 4, 2, 2, 4, 2), (1, 1, 12, 1, 1, 5, 2, 4),
    (6, 2, 32, 5, 64, 64, 32, 16), (6, 3, 128, 4, 65, 65, 64, 8), (5, 5, 16, 8, 63, 0, 6, 16), (17, 1, 8, 2, 30, 9, 8, 8), (3, 1, 200, 3, 40, 7, 100, 8),
    (2, 2, 24, 4, 130, 130, 8, 16)])
def test_the_window_attention_at_the_edges_of_windows_kept_tokens_and_pages(dtype, heads, kv_heads, dim, taps, window, keep, rot, page):
    """A prompt in portions, then single tokens, in a pool whose pages were used before and go back as the window leaves them.
    Some tokens carry keys (and so values) thirty times the usual size: the norm takes the size off the keys, and a query that sees
    such a token one position too long or too short, in a prompt or decoded alone, is far off; so is one that reads a wrong page or a
    wrong carried row, takes the values behind norm or rotation, or leaves the one in the denominator out."""
    need_gpu()
    m = attention(heads, kv_heads, dim, taps, 1.5 / math.sqrt(dim), window, keep, rot, base=1000.0)
    mixer, stored, starts = _direct_attention(m, dtype, seed=3)
    # (the last taps weigh most, so that a token's own size shows at its own place)
    for name in ("q.conv", "k.conv"):
        stored[name] = torch.cat([0.2 * stored[name][:, :-1].float(), 1 + 0.1 * stored[name][:, -1:].float()], dim=1).to(torch.bfloat16)
    w = _bind(mixer, stored, dtype, "mix.")
    T = 2 * window + keep + 4 * page + 75
    g = torch.Generator().manual_seed(window * 100 + heads)
    x = torch.randn(T, mixer.hidden_size, generator=g)
    for p in {keep - 1, keep, keep + 1, page - 1, page + window, T - window - 2, T - window - 1, T - 2 - window // 2}:
        if p >= 0:
            x[p, starts["k"]:starts["g"]] *= 30
    x = x.to(torch.bfloat16).to(dtype)
    want = _attention(x, w, m)

    def differs(weights=w, **changes):
        other = _attention(x, weights, {**m, **changes})
        return float(_row_error(other, want).max())

    # the test can tell
    size = lambda s, k: {"size": s, "keep_first": k}
    assert differs(mask=size(window + 1, keep)) > 0.2 and differs(mask=size(window, keep + 1)) > 0.2
    if window > 1:
        assert differs(mask=size(window - 1, keep)) > 0.2
        assert differs(rot={"base": 1000.0, "dims": rot - 2}) > 0.02
    if keep:
        assert differs(mask=size(window, keep - 1)) > 0.2
    if taps > 1:
        shifted = dict(w, **{"mix.k.conv": torch.roll(w["mix.k.conv"], 1, dims=1)})
        assert differs(shifted) > 0.2
    tol = 2e-5 if dtype == torch.float32 else 0.02
    cache = _cache_for(mixer, dtype, page, -(-T // page) + 8, 3, T + page)
    cache.open("old"), cache.extend("old", 2 * page + 1), cache.open("warm"), cache.extend("warm", page + 1)
    cache.close("old")                  # its pages go to "r", out of order
    cache.open("r")
    portions = [max(window - 1, 1), 2, page, 1, 1, window // 2 + 3, 2]
    portions += [1] * (T - sum(portions))
    got = _run_steps(mixer, cache, [[("r", n)] for n in portions], {"r": x})["r"]
    err = _row_error(got, want)
    assert err.max() <= tol, (int(err.argmax()), float(err.max()))
    note_worst(f"tadalorn window attention alone [{dtype}]", float(err.max()) / tol)
    # a second request in the slot and pages the first one leaves, beside a third: nothing of the first shows
    cache.close("r"), cache.close("warm")
    cache.open("s"), cache.open("u")
    short = x[window // 2:window // 2 + 21]
    got = _run_steps(mixer, cache, [[("s", window + 5), ("u", 1)], [("u", 2), ("s", 1)], [("s", 2), ("u", 18)], [("s", 1)]],
                     {"s": x[:window + 9], "u": short})
    assert _row_error(got["s"], want[:window + 9]).max() <= tol
    assert _row_error(got["u"], _attention(short, w, m)).max() <= tol


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_a_far_key_in_and_out_of_the_window_and_a_kept_key_that_stays(dtype):
    """700 tokens, a window of 600 that keeps five, pages of 16.  The token at position 95 has a value a hundred times the usual size
    and a key along the direction of the last queries, and takes most of their weight among 600 keys: in sight up to position 694,
    out of it from 695 on, which decoded tokens pass.  With the same token at position 4 it stays in sight, at position 5 it does
    not.  A second, shorter request is in the same steps.  No rotation here, so that the directions meet at any distance."""
    need_gpu()
    m = attention(4, 2, 32, 2, 2.8 / math.sqrt(32), 600, 5, 0)
    mixer, stored, starts = _direct_attention(m, dtype, seed=5)
    for name in ("q", "k"):
        stored[name + ".conv"][:, 0] = 0                    # (the current row alone)
        stored[name + ".conv"][:, 1] = 1
        stored[name + ".norm"][:] = 1
    w = _bind(mixer, stored, dtype, "mix.")
    T = 700
    tol = 2e-5 if dtype == torch.float32 else 0.03
    for far in (95, 4, 5):
        g = torch.Generator().manual_seed(11)
        x = torch.randn(T, mixer.hidden_size, generator=g)
        looked = torch.randn(32, generator=g)
        for h in range(4):
            x[-12:, starts["q"] + h * 32:starts["q"] + (h + 1) * 32] = looked + 0.1 * torch.randn(12, 32, generator=g)
        for kh in range(2):
            x[far, starts["k"] + kh * 32:starts["k"] + (kh + 1) * 32] = 100 * looked
        x = x.to(torch.bfloat16).to(dtype)
        other = torch.randn(90, mixer.hidden_size, generator=g).to(torch.bfloat16).to(dtype)
        want, want_other = _attention(x, w, m), _attention(other, w, m)
        if far == 95:
            assert want[694].abs().max() > 10 * want[695].abs().max()                  # inside and outside differ by far
        else:
            assert (want[699].abs().max() > 10 * want[300].abs().max()) == (far == 4)
        cache = _cache_for(mixer, dtype, 16, 60, 3, 720)
        cache.open("r"), cache.open("o")
        steps = [[("r", n)] + ([("o", k)] if k else []) for n, k in
                 ((600, 50), (90, 2), (1, 1), (1, 30), (1, 1), (1, 0), (1, 1), (1, 5), (4, 0))]
        got = _run_steps(mixer, cache, steps, {"r": x, "o": other})
        assert _row_error(got["r"], want, floor=0.01).max() <= tol, far
        assert _row_error(got["o"], want_other).max() <= tol, far


@pytest.mark.parametrize("heads,kv_heads,dim,vdim,window,keep,page", [
    (4, 2, 32, 16, 300, 5, 16), (16, 1, 128, 128, 200, 130, 16), (3, 3, 8, 72, 64, 64, 4), (8, 4, 96, 96, 65, 1, 8), (24, 12, 64, 40, 129, 700, 32),
    (20, 1, 16, 16, 1, 65, 16)])
def test_the_forms_of_the_attention_kernel_that_keeps_first_tokens(heads, kv_heads, dim, vdim, window, keep, page):
    """Single tokens at contexts of 1 to 700 keys, whose keys are shared out over 1 to 9 blocks, and portions at the same contexts, on
    the tensor cores and on the CUDA cores, against float64; a sink per head, a gate, and NaN in all unwritten cache.  Pages that
    neither the window nor the kept tokens need are gone from the table."""
    need_gpu()
    from torchinferno_b200.kernels import ops
    g = torch.Generator().manual_seed(heads * 10 + dim)
    contexts = [700, 1, 65, 64, 333, 129]
    n = len(contexts)
    per = -(-max(contexts) // page)
    pool_k = torch.full((n * per + 3, kv_heads, page, dim), float("nan"))
    pool_v = torch.full((n * per + 3, kv_heads, page, vdim), float("nan"))
    order = torch.randperm(n * per + 3, generator=g)[:n * per].view(n, per).to(torch.int32)
    k_all = [torch.randn(c, kv_heads, dim, generator=g).to(torch.bfloat16) for c in contexts]
    v_all = [torch.randn(c, kv_heads, vdim, generator=g).to(torch.bfloat16) for c in contexts]
    for e, c in enumerate(contexts):
        for pos in range(c):
            pool_k[order[e, pos // page], :, pos % page] = k_all[e][pos].float()
            pool_v[order[e, pos // page], :, pos % page] = v_all[e][pos].float()
    pool = torch.cat([pool_k.flatten(1), pool_v.flatten(1)], dim=1).to(torch.bfloat16).cuda()
    keys = pool[:, :kv_heads * page * dim].unflatten(1, (kv_heads, page, dim))
    values = pool[:, kv_heads * page * dim:].unflatten(1, (kv_heads, page, vdim))
    scale = 1.5 / math.sqrt(dim)
    sink = torch.randn(heads, generator=g)
    for lens in ([1] * n, [min(q, c) for q, c in zip([40, 1, 65, 2, 130, 129], contexts)]):
        total = sum(lens)
        table = order.clone()
        for e, c in enumerate(contexts):
            for logical in range(per):
                first_seen = max(0, c - lens[e] - window + 1)
                if logical * page >= c or (logical * page >= keep and (logical + 1) * page <= first_seen):
                    table[e, logical] = -1
        q = torch.randn(total, heads, dim, generator=g).to(torch.bfloat16)
        gate = torch.randn(total, heads * vdim + 5, generator=g).to(torch.bfloat16)
        want, row = torch.zeros(total, heads, vdim, dtype=torch.float64), 0
        for e, c in enumerate(contexts):
            for i in range(c - lens[e], c):
                seen = [j for j in range(i + 1) if i - j < window or j < keep]
                kk = k_all[e][seen].double().repeat_interleave(heads // kv_heads, dim=1)
                vv = v_all[e][seen].double().repeat_interleave(heads // kv_heads, dim=1)
                s = torch.exp(torch.einsum("hd,jhd->hj", q[row].double(), kk) * scale)
                want[row] = torch.einsum("hj,jhd->hd", s / (s.sum(dim=1, keepdim=True) + torch.exp(sink.double())[:, None]), vv)
                row += 1
        want = want.flatten(1) * torch.sigmoid(gate[:, 5:].double())
        cases = [dict(force_simt=True), dict()]
        if max(lens) == 1:
            cases += [dict(max_kv_len=700, splits=s) for s in (1, 2, 5, 9)] + [dict(max_kv_len=700)]
        for case in cases:
            out = torch.full((total, heads * vdim), float("nan"), dtype=torch.bfloat16, device=CUDA)
            error = torch.zeros(1, dtype=torch.int32, device=CUDA)
            ops.pooled_window_attention(
                q.flatten(1).cuda(), out, _i32(np.cumsum([0] + lens).tolist()), _i32([c - k for c, k in zip(contexts, lens)]),
                _i32(list(range(n))), keys, values, table.cuda(), None, None, None, n, max(lens), heads, kv_heads, window=window, keep=keep,
                pool=0, scale=scale, sink=sink.cuda(), gate=gate.cuda()[:, 5:], error_word=error, **case)
            got = out.cpu().double()
            assert torch.isfinite(got).all() and int(error) == 0, case
            # (inputs are exact here: what is left is the sums' and the output's rounding)
            assert (got - want).abs().max() <= 0.006 * want.abs().max(), (case, float((got - want).abs().max() / want.abs().max()))


def _direct_memory(m, dtype, seed):
    """A memory whose input row is [q | k | v | g | i | f] itself; the input and forget gates' rows are set by the input too."""
    from torchinferno_b200.parts.base import PartSpec, build_part
    from torchinferno_b200.weights.random_init import random_tensor
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    widths = {"q": H * d, "k": H * d, "v": H * dv, "g": H * dv, "i": H, "f": H}
    mixer = build_part("mixer", PartSpec("matrix_memory", {
        "hidden_size": sum(widths.values()), "heads": H, "dim": d, "value_dim": dv, "gate_cap": m["gate_cap"], "eps": 1e-5}), dtype=dtype, device=CUDA)
    stored = {ws.name: random_tensor(ws, seed, dtype=torch.bfloat16) for ws in mixer.weight_specs()}
    return mixer, stored, _picked_columns(mixer, widths, stored)


def _memory_input(mixer, starts, T, g, steady=False):
    """Random rows.  Gates: long stretches that keep everything (forget gates near 1), now and then a token that forgets nearly all
    or comes in with a gate far above what is there."""
    x = torch.randn(T, mixer.hidden_size, generator=g)
    H = mixer.heads
    x[:, starts["i"]:starts["i"] + H] = torch.randn(T, H, generator=g)
    x[:, starts["f"]:starts["f"] + H] = 5 + torch.randn(T, H, generator=g)
    if not steady:
        x[torch.rand(T, generator=g) < 0.03, starts["f"]:starts["f"] + H] -= 18
        x[torch.rand(T, generator=g) < 0.03, starts["i"]:starts["i"] + H] += 9
        x[torch.rand(T, generator=g) < 0.03, starts["i"]:starts["i"] + H] -= 20
    return x.to(torch.bfloat16)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads,dim,vdim,cap", [(2, 16, 24, 15.0), (3, 7, 9, 4.0), (1, 40, 136, 15.0), (2, 128, 64, 6.0), (1, 8, 300, 15.0),
                                                (2, 64, 128, 15.0), (1, 200, 48, 10.0), (1, 300, 40, 15.0), (5, 24, 8, 1.0)])
def test_the_matrix_memory_in_portions_over_its_state(dtype, heads, dim, vdim, cap):
    """Portions below, at and above a chunk's length and down to two tokens, single tokens between them, two requests in a step, a
    slot used again.  The reference walks the recurrence token by token in float64."""
    need_gpu()
    m = mlstm(heads, dim, vdim, cap)
    mixer, stored, starts = _direct_memory(m, dtype, seed=heads * 7 + dim)
    w = _bind(mixer, stored, dtype, "mix.")
    g = torch.Generator().manual_seed(dim)
    T = 330
    x, other = _memory_input(mixer, starts, T, g).to(dtype), _memory_input(mixer, starts, 90, g).to(dtype)
    mem = lambda rows, weights=w: plain_tadalorn.mlstm(rows.double(), weights, "mix.", m, 1e-5)
    want, want_other = mem(x), mem(other)
    # the test can tell: a state lost between portions, another cap on the gates, forget gates without their bias
    assert _row_error(mem(x[130:]), want[130:]).max() > 0.2
    assert _row_error(plain_tadalorn.mlstm(x.double(), w, "mix.", dict(m, gate_cap=1.2 * cap), 1e-5), want).max() > 0.05
    if cap > 1:
        assert _row_error(mem(x, dict(w, **{"mix.f.b": w["mix.f.b"] - 1})), want).max() > 0.05
    tol = 1e-4 if dtype == torch.float32 else 0.02
    cache = _cache_for(mixer, dtype, 4, 8, 3, 1000)
    cache.open("r"), cache.open("o")
    steps = [[("r", n)] + ([("o", k)] if k else []) for n, k in
             ((63, 1), (1, 1), (2, 64), (65, 2), (1, 0), (1, 1), (9, 9), (128, 1), (8, 5), (17, 1), (3, 2), (30, 1), (1, 1), (1, 1))]
    got = _run_steps(mixer, cache, steps, {"r": x, "o": other})
    # (a readout that nearly cancels is divided by its own small root mean square: nine rows in ten within the bound in bfloat16)
    for name, ref in (("r", want), ("o", want_other)):
        err = _row_error(got[name], ref).sort().values
        assert err[int(0.9 * (len(err) - 1))] <= tol and err[-1] <= (tol if dtype == torch.float32 else 5 * tol), (name, float(err[-1]))
        note_worst(f"tadalorn memory alone [{dtype}]", float(err[int(0.9 * (len(err) - 1))]) / tol)
    cache.close("r")
    cache.open("s")
    again = _run_steps(mixer, cache, [[("s", 70)], [("s", 1)], [("s", 2)]], {"s": x[:73]})["s"]
    assert _row_error(again, want[:73]).sort().values[64] <= tol


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_what_a_memory_keeps_over_two_thousand_tokens_and_what_it_forgets(dtype):
    """A value a hundred times the usual size with the key that the last queries look along, 2,000 tokens back: with forget gates
    near 1 all that time the last outputs point along it; with the gates of four tokens shut in between nothing of it is left.  Portions of 700,
    then single tokens; the running maximum stays at the early token's input gate."""
    need_gpu()
    m = mlstm(2, 32, 16, 15.0)
    mixer, stored, starts = _direct_memory(m, dtype, seed=9)
    for name in ("i.b", "f.b"):
        stored[name][:] = 0
    stored["norm"][:] = 1
    pick = torch.eye(mixer.hidden_size)[:2 * 16]            # (the output row is the heads' rows, padded with zeros)
    stored["o"] = pick.t().contiguous().to(torch.bfloat16)
    w = _bind(mixer, stored, dtype, "mix.")
    g = torch.Generator().manual_seed(2)
    T = 2050
    x = 0.1 * torch.randn(T, mixer.hidden_size, generator=g)
    looked, left = torch.randn(64, generator=g), torch.randn(32, generator=g)
    x[10, starts["k"]:starts["v"]] = looked
    x[10, starts["v"]:starts["g"]] = 100 * left
    x[-20:, starts["q"]:starts["k"]] = looked
    x[:, starts["g"]:starts["i"]] = 20.0                     # (gates open)
    x[:, starts["i"]:starts["f"]] = -6.0
    x[10, starts["i"]:starts["f"]] = 6.0
    x[:, starts["f"]:] = 12.0
    for shut in (None, 1500):
        rows = x.clone()
        if shut is not None:
            rows[shut:shut + 4, starts["f"]:] = -14.0
        rows = rows.to(torch.bfloat16).to(dtype)
        want = plain_tadalorn.mlstm(rows.double(), w, "mix.", m, 1e-5)
        along = torch.cosine_similarity(want[-1, :32].view(2, 16), left.double().view(2, 16), dim=1)
        assert (along > 0.99).all() if shut is None else (along.abs() < 0.9).any()
        cache = _cache_for(mixer, dtype, 4, 8, 1, 3000)
        cache.open("r")
        got = _run_steps(mixer, cache, [[("r", 700)], [("r", 700)], [("r", 630)]] + [[("r", 1)]] * 20, {"r": rows})["r"]
        tol = 1e-4 if dtype == torch.float32 else 0.02
        assert _row_error(got[-60:, :32], want[-60:, :32]).max() <= tol, shut
        # m lies behind every head's sum of keys; it is what it is however the portions were cut
        top = cache.state(0)[cache.slot("r")][2 * 32 * 16:2 * 32 * 16 + 66].view(2, 33)[:, 32].cpu().double()
        gates = plain_tadalorn.memory_gates(rows.double(), w, "mix.", 15.0)
        m_ref = torch.zeros(2, dtype=torch.float64)
        for t in range(T):
            m_ref = torch.maximum(gates[1][t] + m_ref, gates[0][t])
        assert (top - m_ref).abs().max() <= 1e-3


def test_the_two_forms_of_the_memory_kernel_agree():
    """The same bfloat16 rows walked token by token and cut into chunks: outputs and the state left behind."""
    need_gpu()
    from torchinferno_b200.kernels import ops
    for heads, dim, vdim in ((3, 64, 128), (2, 24, 40), (1, 256, 264), (4, 128, 64)):
        g = torch.Generator().manual_seed(dim)
        mixer, stored, starts = _direct_memory(mlstm(heads, dim, vdim, 12.0), torch.bfloat16, seed=dim)
        _bind(mixer, stored, torch.bfloat16, "mix.")
        lens = [1, 200, 64, 3, 65]
        x = _memory_input(mixer, starts, sum(lens), g).cuda()
        batch = _entries_batch([(str(i), i, 5, n) for i, n in enumerate(lens)])
        proj = torch.nn.functional.pad(x[:, :starts["i"]], (0, mixer.in_width - starts["i"])).contiguous()
        floats = ops.matrix_memory_state_floats(heads, dim, vdim)
        start = 0.1 * torch.randn(len(lens), floats, generator=g)
        tiles = -(-vdim // 128)
        norms = start[:, heads * dim * vdim:heads * dim * vdim + heads * tiles * (dim + 1)].view(len(lens), heads, tiles, dim + 1)
        norms[:] = norms[:, :, :1].clone()                   # (every tile holds the same sum of keys and maximum)
        results = []
        for walk in (True, False):
            state, out = start.clone().cuda(), torch.empty(x.shape[0], heads * vdim, dtype=torch.bfloat16, device=CUDA)
            ops.matrix_memory(proj, 0, starts["k"], starts["v"], starts["g"], x, mixer.gate_weight, mixer.gate_bias, 12.0, state, batch.q_start,
                              batch.slots, len(lens), max(lens), mixer.norm_weight, 1e-5, out, heads=heads, dim=dim, vdim=vdim,
                              q_scale=dim ** -0.5, walk=walk)
            results.append((out.float(), state))
        (a, sa), (b, sb) = results
        close = ((a - b).abs() / a.abs().max(dim=1, keepdim=True).values).max(dim=1).values.sort().values
        assert close[int(0.9 * (len(close) - 1))] <= 0.01 and close[-1] <= 0.1, (heads, dim, vdim)
        assert (sa - sb).abs().max() <= 2e-4 * sa.abs().max()


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads,dim,rot,vdim,rank", [(2, 16, 8, 24, 40), (4, 32, 16, 32, 64), (1, 13, 6, 21, 36), (20, 16, 16, 8, 128), (3, 24, 2, 8, 200)])
def test_a_sink_in_the_latent_attention(dtype, heads, dim, rot, vdim, rank):
    """Whole prompts, portions and single tokens (whose contexts are shared out over blocks); sinks from far below the scores to far
    above them, so that a head that counts its sink twice, not at all, scaled, or another head's is far off, also at the first token,
    which has nothing but itself and the sink."""
    need_gpu()
    from torchinferno_b200.parts.base import PartSpec, build_part
    from torchinferno_b200.weights.random_init import random_tensor
    W = 48
    m = latent(heads, dim, rot, vdim, rank, 0.7 / math.sqrt(dim + rot), base=3000.0)
    mixer = build_part("mixer", PartSpec("latent_attention", {
        "hidden_size": W, "heads": heads, "dim": dim, "rot_dim": rot, "value_dim": vdim, "kv_rank": rank, "scale": m["scale"],
        "rot_base": 3000.0, "eps": 1e-5, "sink": True, "gate": True}), dtype=dtype, device=CUDA)
    stored = {ws.name: random_tensor(ws, 4, dtype=torch.bfloat16) for ws in mixer.weight_specs()}
    stored["sink"] = torch.linspace(-3.0, 7.0, heads).to(torch.bfloat16) if heads > 1 else torch.tensor([3.0]).to(torch.bfloat16)
    w = _bind(mixer, stored, dtype, "mix.")
    T = 300
    x = torch.randn(T, W, generator=torch.Generator().manual_seed(rank)).to(torch.bfloat16).to(dtype)
    run = lambda weights: plain_tadalorn.latent_attention(x.double(), weights, "mix.", m, 1e-5, torch.arange(T))
    want = run(w)
    for changed in (w["mix.sink"] - 40, w["mix.sink"] + math.log(2.0), w["mix.sink"] * m["scale"]):
        assert _row_error(run(dict(w, **{"mix.sink": changed})), want).max() > 0.1
    tol = 3e-5 if dtype == torch.float32 else 0.03
    for page, portions in ((16, [T]), (4, [130, 2, 1, 1, 65, 31, 2] + [1] * 68)):
        cache = _cache_for(mixer, dtype, page, -(-T // page) + 4, 2, T + page)
        cache.open("old"), cache.extend("old", 2 * page), cache.open("r"), cache.close("old")
        got = _run_steps(mixer, cache, [[("r", n)] for n in portions], {"r": x})["r"]
        err = _row_error(got, want)
        assert err.max() <= tol, (page, int(err.argmax()), float(err.max()))
        note_worst(f"tadalorn latent attention alone [{dtype}]", float(err.max()) / tol)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("experts,top,ff,shared,width", [(5, 2, 24, 40, 64), (3, 3, 20, None, 45), (16, 1, 96, 128, 80), (7, 4, 33, 17, 44), (1, 1, 8, 8, 16)])
def test_experts_with_gelu_behind_a_router_with_a_bias(dtype, experts, top, ff, shared, width):
    need_gpu()
    from torchinferno_b200.parts.base import PartSpec, build_part
    from torchinferno_b200.weights.random_init import random_tensor
    mlp = moe(experts, top, ff, shared)
    part = build_part("feed_forward", PartSpec("routed_experts", {
        "hidden_size": width, "experts": experts, "top": top, "expert_size": ff, "activation": "gelu", "scores": "softmax", "normalize": True,
        "router_bias": True, "shared_size": shared or 0}), dtype=dtype, device=CUDA)
    stored = {ws.name: random_tensor(ws, 6, dtype=torch.bfloat16) for ws in part.weight_specs()}
    stored["router.b"] = torch.linspace(-1.5, 1.5, experts).to(torch.bfloat16)
    w = _bind(part, stored, dtype, "mlp.")
    for n in (1, 3, 70):
        x = (2 * torch.randn(n, width, generator=torch.Generator().manual_seed(n))).to(torch.bfloat16).to(dtype)
        gaps = [[] for _ in range(n)]
        want = plain_tadalorn.routed_experts(x.double(), w, "mlp.", mlp, gaps)
        clear = torch.tensor([min(gap, default=1.0) > 1e-4 for gap in gaps])
        got = part.forward(x.cuda(), None).cpu().double()
        tol = 2e-5 if dtype == torch.float32 else 0.02
        assert _row_error(got, want)[clear].max() <= tol and clear.sum() >= n // 2
    if 1 < top < experts:      # the bias counts, for the choice and for the weights; the activation is the exact form
        free = plain_tadalorn.routed_experts(x.double(), dict(w, **{"mlp.router.b": 0 * w["mlp.router.b"]}), "mlp.", mlp)
        assert _row_error(free, want).max() > 0.2


def test_gelu_is_the_exact_form():
    need_gpu()
    from torchinferno_b200.kernels import ops
    x = torch.linspace(-6, 6, 1001)
    for dtype in (torch.float32, torch.bfloat16):
        rows = x.to(dtype)
        got = ops.gelu(rows.cuda(), torch.empty(1001, dtype=torch.float32, device=CUDA)).cpu().double()
        want = plain_tadalorn.gelu(rows.double())
        assert (got - want).abs().max() <= 1e-6
        approx = torch.nn.functional.gelu(rows.double(), approximate="tanh")
        assert (approx - want).abs().max() > 1e-4            # (the tanh form would show)


@pytest.mark.parametrize("width", [16, 50, 520, 4096, 9000])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_the_normed_way_back_into_the_residual(dtype, width):
    need_gpu()
    from torchinferno_b200.kernels import ops
    g = torch.Generator().manual_seed(width)
    x, weight = torch.randn(5, width, generator=g), 1 + 0.3 * torch.randn(width, generator=g)
    y = (torch.randn(5, width, generator=g) * torch.tensor([1e-4, 1.0, 30.0, 0.0, 2.0])[:, None]).to(dtype)
    want = x.double() + 0.7 * plain_tadalorn.rms_norm(y.double(), weight.double(), 1e-5)
    residual = x.cuda()
    copy = torch.empty(5, width, dtype=dtype, device=CUDA)
    ops.unit_norm_add(residual, y.cuda(), weight.cuda(), 1e-5, 0.7, copy)
    assert (residual.cpu().double() - want).abs().max() <= 1e-5
    assert torch.equal(copy, residual.to(dtype))
    residual = x.cuda()
    ops.unit_norm_add(residual, y.cuda(), weight.cuda(), 1e-5)
    assert (residual.cpu().double() - (x.double() + plain_tadalorn.rms_norm(y.double(), weight.double(), 1e-5))).abs().max() <= 1e-5


def test_a_norm_in_parts_ahead_of_its_gate():
    need_gpu()
    from torchinferno_b200.kernels import ops
    g = torch.Generator().manual_seed(4)
    y, z, weight = torch.randn(7, 60, generator=g), torch.randn(7, 70, generator=g), torch.randn(60, generator=g)
    out = ops.gated_group_norm(y.cuda(), z.cuda(), 5, weight.cuda(), 1e-5, torch.empty(7, 60, device=CUDA), 3, gate_last=True).cpu().double()
    want = plain_tadalorn.unit_rms(y.double().view(7, 3, 20), 1e-5).reshape(7, 60) * weight.double() * torch.sigmoid(z[:, 5:65].double())
    assert (out - want).abs().max() <= 1e-5


def test_the_state_of_the_convolution_and_what_is_stored():
    """Rows in portions of every length around the carried rows, several requests, odd and even head sizes: the values are the
    convolved keys ahead of norm and rotation, the carried rows are the last projected ones, nothing else is touched."""
    need_gpu()
    from torchinferno_b200.kernels import ops
    for dtype, heads, kv, d, taps, rot, page in ((torch.float32, 3, 1, 7, 4, 4, 4), (torch.bfloat16, 4, 2, 16, 3, 16, 8), (torch.bfloat16, 5, 5, 6, 9, 2, 4),
                                                 (torch.bfloat16, 40, 20, 128, 4, 64, 16), (torch.float32, 2, 2, 300, 2, 300, 16), (torch.bfloat16, 2, 1, 8, 1, 0, 2), (torch.bfloat16, 3, 2, 16, 2, 6, 4)):
        g = torch.Generator().manual_seed(d * taps)
        T, qw, kw, pad = 40, heads * d, kv * d, 4
        k_off = -(-qw // 8) * 8
        u = torch.zeros(T, -(-(k_off + kw) // 8) * 8)
        u[:, :qw], u[:, k_off:k_off + kw] = torch.randn(T, qw, generator=g), torch.randn(T, kw, generator=g)
        u = (u * torch.linspace(0.5, 3.0, T)[:, None]).to(dtype)
        conv = [torch.randn(taps, width, generator=g) for width in (qw, kw)]
        gain = [1 + 0.2 * torch.randn(width, generator=g) for width in (qw, kw)]
        freq = 100.0 ** (-2.0 * torch.arange(rot // 2) / max(rot, 1))
        c = [plain_tadalorn.channel_convolution(part.double(), w.double().t()) for part, w in ((u[:, :qw], conv[0]), (u[:, k_off:k_off + kw], conv[1]))]
        positions = torch.arange(T)
        q_want, k_want = (plain_tadalorn.rotate_pairs(plain_tadalorn.rms_norm(r, w.double(), 1e-5).view(T, -1, d), positions, 100.0, rot) for r, w in zip(c, gain))
        per = -(-T // page)
        pool = torch.full((2 * per, 2 * kv * page * d), float("nan")).to(dtype).cuda()
        keys, values = (part.unflatten(1, (kv, page, d)) for part in pool.chunk(2, dim=1))
        table = torch.randperm(2 * per, generator=g).view(2, per).to(torch.int32).cuda()
        floats = (taps - 1) * (qw + kw)
        state = torch.full((2, floats + 2 * pad), 7.0, device=CUDA)
        state[:, pad:pad + floats] = 0
        at, oat, tol = 0, 0, 2e-5 if dtype == torch.float32 else 0.01
        for n, k in ((1, 2), (1, 1), (2, 0), (3, 1), (9, 7), (1, 1), (13, 2), (10, 3)):
            rows = torch.cat([u[at:at + n], u[oat:oat + k]]).cuda()
            lens = [n] + ([k] if k else [])
            pos = list(range(at, at + n)) + list(range(oat, oat + k))
            q_out, error = torch.empty(n + k, qw, dtype=dtype, device=CUDA), torch.zeros(1, dtype=torch.int32, device=CUDA)
            ops.conv_norm_append(rows, 0, k_off, q_out, keys, values, conv[0].cuda(), conv[1].cuda(), _i32(pos), table,
                                 _i32(np.cumsum([0] + lens).tolist()), _i32([1, 0][:len(lens)]), len(lens), max(lens), heads, kv, d, freq=freq.cuda(),
                                 q_weight=gain[0].cuda(), k_weight=gain[1].cuda(), eps=1e-5, state=state, state_off=pad, error_word=error)
            assert int(error) == 0
            assert (q_out.cpu().double().view(n + k, heads, d) - q_want[pos]).abs().max() <= tol * q_want.abs().max()
            at, oat = at + n, oat + k
        for slot, length in ((1, at), (0, oat)):
            for p in range(length):
                where = int(table[slot, p // page]), p % page
                assert (keys[where[0], :, where[1]].cpu().double() - k_want[p]).abs().max() <= tol * k_want.abs().max()
                assert (values[where[0], :, where[1]].cpu().double() - c[1][p].view(kv, d)).abs().max() <= tol * c[1].abs().max()
            ahead = torch.cat([torch.zeros(taps, qw + kw), torch.cat([u[:length, :qw], u[:length, k_off:k_off + kw]], dim=1).float()])
            carried = ahead[len(ahead) - (taps - 1):]
            assert torch.equal(state[slot, pad:pad + floats].cpu().view(taps - 1, qw + kw), carried)
        assert int(torch.isfinite(keys).sum()) == int(torch.isfinite(values).sum()) == (at + oat) * kv * d
        assert float((state[:, :pad] - 7).abs().max()) == 0.0 and float((state[:, pad + floats:] - 7).abs().max()) == 0.0


# ------------------------------------------------ entry point and programs
def test_greedy_generation_through_the_engine_and_its_scheduler(folders):
    need_gpu()
    from torchinferno_b200.config.engine_config import EngineConfig
    from torchinferno_b200.engine.engine import InferenceEngine
    from torchinferno_b200.engine.types import GenerateRequest, SamplingConfig
    for name in ("TA", "TE"):
        config, seed = CONFIGS[name]
        cfg, w = plain_tadalorn.read_model_folder(folders[name])
        prompts = list(requests_for(config, seed + 2, [5, 41, 1, 18, 66]).values())
        new = 30                                                # (decoding passes the shortest window)
        for dtype in ("float32", "bfloat16"):
            with InferenceEngine.from_config(EngineConfig(model=str(folders[name]), dtype=dtype, page_size=8, max_batch_size=3,
                                                          prefill_chunk_size=16, max_num_batched_tokens=48, kv_cache_tokens=512)) as engine:
                outs = engine.generate_many([GenerateRequest(f"g{i}", prompt_token_ids=p, sampling=SamplingConfig(new))
                                             for i, p in enumerate(prompts)])
            misses = []
            for prompt, out in zip(prompts, outs):
                tokens = list(out.token_ids)
                assert len(tokens) == new
                logits = plain_tadalorn.forward(cfg, w, (prompt + tokens)[:-1])
                rows = logits[len(prompt) - 1:]
                # by how much a drawn token misses the best, as a share of the largest logit
                misses += [float((row.max() - row[tok]) / logits.abs().max()) for row, tok in zip(rows, tokens)]
            misses.sort()
            if dtype == "float32":
                assert misses[-1] <= 1e-4
            else:
                assert misses[int(0.9 * len(misses))] <= BF16_REL


def test_the_command_line_generates_from_a_tadalorn_folder(folders, capsys):
    need_gpu()
    from torchinferno_b200 import cli
    assert cli.main(["generate", str(folders["TC"]), "--input-ids", "5", "3", "9", "--new-tokens", "4", "--dtype", "float32"]) == 0
    assert capsys.readouterr().out.strip()


def test_the_trace_program_replays_a_tadalorn_folder(folders, tmp_path):
    need_gpu()
    config, seed = CONFIGS["TA"]
    requests = requests_for(config, seed + 3, [30, 75, 2])
    steps, index = replay_util.trace_mixed(requests, seed=3)
    results = replay_util.run_trace_program(folders["TA"], "float32", replay_util.peak_tokens(steps), steps, tmp_path / "out")
    compare(replay_util.gather(results, index), folders["TA"], requests, "float32", "TA trace program")


# ------------------------------------------------------- sizes drawn at random
def _random_config(rng):
    """A small Tadalorn configuration with sizes drawn from lists that mix multiples of 8, 16, 64 with odd ones."""
    pick = rng.choice

    def mlp():
        kind = pick(["dense", "moe", None])
        if kind == "dense":
            return dense(pick([8, 24, 36, 70]))
        if kind is None:
            return None
        experts = pick([1, 2, 5, 9, 40])
        return moe(experts, rng.randint(1, min(experts, 4)), pick([7, 16, 24]), pick([None, 8, 30]))

    layers = []
    for _ in range(pick([2, 3, 4, 5])):
        owners = [i for i, entry in enumerate(layers) if "weights_of" not in entry]
        if owners and rng.random() < 0.25:
            source = pick(owners)
            layers.append(dict(layers[source], weights_of=source))
            continue
        kind = pick(["mlstm", "attention", "latent_attention"])
        if kind == "mlstm":
            mixer = mlstm(pick([1, 2, 3, 5]), pick([4, 8, 13, 24, 40, 64]), pick([5, 8, 24, 72, 130]), pick([2.0, 8.0, 15.0]))
        elif kind == "attention":
            kv_heads, dim = pick([1, 2, 3, 5]), pick([4, 8, 12, 24, 40, 64])
            window = pick([None, 1, 2, 9, 31, 32, 64, 65, 300])
            mixer = attention(kv_heads * pick([1, 2, 3, 4]), kv_heads, dim, pick([1, 2, 3, 4, 6, 9]), pick([0.1, 0.4]), window,
                              pick([0, 1, 4, 7, 33, 70]), 2 * rng.randint(1, dim // 2), base=pick([100.0, 10000.0, 1e6]))
        else:
            mixer = latent(pick([1, 2, 3, 6, 18]), pick([4, 8, 13, 32]), pick([2, 6, 8, 16]), pick([5, 8, 24]), pick([12, 36, 64, 128]), pick([0.1, 0.3]))
        layers.append(layer(kind, mixer, mlp()))
    return model(pick([50, 97, 128]), pick([24, 40, 45, 72, 96, 136]), layers, residual_mult=pick([0.25, 0.7, 1.0]), softcap=pick([None, 5.0, 30.0]),
                 eps=pick([1e-6, 1e-5]))


@pytest.mark.parametrize("draw", range(12))
def test_sizes_drawn_at_random(draw, tmp_path):
    """Whole prompts, portions and token-by-token decoding of models whose every size was drawn at random, in both number formats."""
    need_gpu()
    rng = random.Random(8800 + draw)
    config = _random_config(rng)
    write_model(config, tmp_path, seed=draw, decided=True)
    requests = requests_for(config, 50 + draw, [41, 3, 75])
    for dtype in ("float32", "bfloat16"):
        for kind, (steps, index) in {"whole": replay_util.trace_whole(requests), "tail": replay_util.trace_tail_decode(requests, tail=12),
                                     "portions": replay_util.trace_portions(requests, sizes=(2, 31, 3, 33, 2, 16))}.items():
            runner = make_runner(tmp_path, dtype, replay_util.peak_tokens(steps), page_size=rng.choice([4, 16]))
            rows = replay_util.gather(run_steps(runner, steps), index)
            compare(rows, tmp_path, requests, dtype, f"draw {draw} {kind}")
