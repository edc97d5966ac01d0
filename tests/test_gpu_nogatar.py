"""Nogatar on the GPU against the plain implementation: the new kernels alone, the step function under every way of
cutting requests into steps, window edges, batches, pages and slots used again, then generation through the entry
point."""

from __future__ import annotations

import io
import itertools
import json
import random

import numpy as np
import pytest
import torch

import plain_nogatar as plain
from nogatar_cases import (PAGE_TOKENS, all_experts, assert_rows_close, config, leaning_model, leaning_tokens, plain_greedy,
                           plain_logits, random_config, random_weights, relative_error, rounding_spread, tokens_for)

from mini_gpt_inference_b200 import EngineConfig, LLMEngine, NogatarConfig, SamplingParams
from mini_gpt_inference_b200.engine.build import load_model, make_runner
from mini_gpt_inference_b200.engine.runner import StepEntry

pytestmark = pytest.mark.gpu

# Largest |engine - plain| on a row of logits, over the row's own spread.  32-bit: rounding of sums.
# bfloat16: both sides use the same weights; activations are rounded to 8 bits between kernels.  A
# lost key, state, sink, norm or expert shows as 0.3 and more.
TOL = {"float32": 3e-4, "bfloat16": 1e-1}
DTYPES = {"float32": torch.float32, "bfloat16": torch.bfloat16}
CASES = [(w, d) for w in "ABCDE" for d in ("float32", "bfloat16")]
IDS = [f"{w}-{d}" for w, d in CASES]


@pytest.fixture(scope="module")
def ops():
    from mini_gpt_inference_b200.kernels.ops import default_ops

    return default_ops("cuda:0")


def dev(t, dtype=None):
    return t.to(device="cuda:0", dtype=dtype or t.dtype).contiguous()


# ---- the new kernels alone ---------------------------------------------------------------------------------------
@pytest.mark.parametrize("rows,width", [(1, 40), (5, 192), (37, 101), (130, 1024), (3, 5120), (2, 9000)])
def test_layer_norm_behind_a_sublayer(ops, rows, width):
    """The stream plus a factor times the centred norm of a sublayer's output; also of a sum over entries; the copy of
    the new stream in bfloat16; both kinds of norm."""
    gen = torch.Generator().manual_seed(rows + width)
    x, a, b = (torch.randn(rows, width, generator=gen) for _ in range(3))
    a = 20.0 * a + 30.0                                                            # a mean that must be taken off first
    w = 1 + 0.3 * torch.randn(width, generator=gen)
    want = x.double() + 0.7 * plain.layer_norm(a.double(), w.double(), 1e-3)
    xa, ya = dev(x), dev(a)
    rows16 = ops.norm_add(xa, ya, dev(w), 1e-3, center=True, norm_scale=0.7, rows_dtype=torch.bfloat16)
    assert torch.allclose(xa.double().cpu(), want, atol=2e-5)
    assert torch.equal(rows16, xa.to(torch.bfloat16)) and torch.equal(ya.cpu(), a)
    xb = dev(x)
    assert ops.norm_add(xb, ya, dev(w), 1e-3, center=True, norm_scale=0.7, clear=True, rows_dtype=torch.float32) is xb
    assert torch.equal(xb, xa) and not bool(ya.any())
    got = dev(x)
    assert ops.norm_add(got, dev(a), dev(w), 1e-3, center=True, other32=dev(b), scale=1.2, other_scale=-0.5) is None
    assert torch.allclose(got.double().cpu(), x.double() + plain.layer_norm(1.2 * a.double() - 0.5 * b.double(), w.double(), 1e-3), atol=2e-5)
    got = dev(x)
    ops.norm_add(got, dev(a), dev(w), 1e-3, offset=1.0, norm_scale=-2.0)            # a root-mean-square norm, stored around zero
    y = a.double() / torch.sqrt((a.double() ** 2).mean(-1, keepdim=True) + 1e-3)
    assert torch.allclose(got.double().cpu(), x.double() - 2.0 * y * (1 + w.double()), atol=2e-5)
    # the sum over a token's entries, some of them empty
    from mini_gpt_inference_b200.kernels.ops import EntrySum

    top = 3
    terms = torch.randn(rows * top, width, generator=gen)
    slots = torch.randperm(rows * top, generator=gen).view(rows, top).to(torch.int32)
    slots[0, 1] = -1
    total = torch.zeros(rows, width, dtype=torch.float64)
    for r in range(rows):
        for s in slots[r].tolist():
            if s >= 0:
                total[r] += terms[s].double()
    got = dev(x)
    rows16 = ops.norm_add(got, EntrySum(dev(terms), dev(slots)), dev(w), 1e-3, center=True, norm_scale=0.7, rows_dtype=torch.bfloat16)
    assert torch.allclose(got.double().cpu(), x.double() + 0.7 * plain.layer_norm(total, w.double(), 1e-3), atol=2e-5)
    assert torch.equal(rows16, got.to(torch.bfloat16))
    # a padding row (all its entries empty) leaves the stream as it is
    got = dev(x)
    ops.norm_add(got, EntrySum(dev(terms), dev(torch.full((rows, top), -1, dtype=torch.int32))), dev(w), 1e-3, center=True)
    assert torch.equal(got.cpu(), x)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("heads,q_dim,rot,rank,magnitude", [(3, 24, 8, 40, 1.14), (1, 16, 16, 16, 1.0), (5, 10, 6, 20, 0.5),
                                                            (2, 128, 64, 256, 1.28), (2, 7, 2, 11, 1.1)])
def test_latent_rows_with_neighbouring_features_turned(ops, dtype, heads, q_dim, rot, rank, magnitude):
    from mini_gpt_inference_b200.cache.storage import PagedKVView

    t = DTYPES[dtype]
    gen = torch.Generator().manual_seed(heads * rank + rot)
    positions = torch.tensor([0, 3, 1, 900, -1, 3300], dtype=torch.int32)
    slots = torch.tensor([5, 0, 11, 6, -1, 2], dtype=torch.int32)
    n, q_off = positions.numel(), 8
    low_off = q_off + heads * (q_dim + rot)
    proj = torch.randn(n, low_off + rank + rot, generator=gen).to(t)
    gain = 1 + 0.3 * torch.randn(rank, generator=gen)
    freq = [300.0 ** (-2.0 * i / rot) / (1 + i) for i in range(rot // 2)]
    eps, pt = 1e-3, 4
    pages = dev(torch.full((3, 1, pt, rank + rot), float("nan")), t)
    cache = PagedKVView(pages, pages, 0, pt, None, True, values_in_keys=True)
    q = ops.latent_prepare(dev(proj), heads, q_off, q_dim, rot, low_off, rank, dev(gain), eps,
                           dev(torch.tensor(freq, dtype=torch.float64).float()), cache, dev(slots), dev(positions),
                           neighbours=True, magnitude=magnitude).double().cpu().view(n, heads, rank + rot)
    x, live, pos = proj.double(), positions >= 0, positions.clamp(min=0)
    tol = 5e-5 if dtype == "float32" else 2e-2
    # (the plain rotation in 32-bit: angles are 32-bit numbers by design)
    q_rot = plain.rotate_pairs(x[:, q_off:low_off].float().view(n, heads, q_dim + rot)[..., q_dim:], pos, freq, magnitude).double()
    assert torch.allclose(q[live][..., rank:], q_rot[live], atol=tol, rtol=tol)
    latent = plain.unit_rms(x[:, low_off: low_off + rank], eps) * gain.double()
    shared = plain.rotate_pairs(x[:, low_off + rank:].float().view(n, 1, rot), pos, freq, magnitude).double().view(n, rot)
    rows = pages.double().cpu().view(-1, rank + rot)
    for i in range(n):
        if live[i]:
            assert torch.allclose(rows[slots[i]], torch.cat([latent[i], shared[i]]), atol=tol, rtol=tol), f"token {i}"
    written = torch.zeros(3 * pt, dtype=torch.bool)
    written[slots[live].long()] = True
    assert bool(torch.isnan(rows[~written]).all())


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("tokens", [1, 5, 64, 65, 200, 1187])
@pytest.mark.parametrize("experts,top,width,inner,shared", [(5, 2, 64, 40, 40), (4, 1, 96, 48, None), (3, 3, 72, 20, 50),
                                                            (16, 4, 128, 128, 64), (2, 1, 70, 33, 33)])
def test_router_and_experts_without_a_gate(ops, dtype, tokens, experts, top, width, inner, shared):
    """The part on its own against the plain feed-forward, the shared expert among the chosen ones; both ways of handing
    its output on; a padding row."""
    from types import SimpleNamespace

    from mini_gpt_inference_b200.parts.base import FEED_FORWARDS
    from mini_gpt_inference_b200.parts.spec import PartSpec

    t = DTYPES[dtype]
    gen = torch.Generator().manual_seed(experts * 100 + inner)
    part = FEED_FORWARDS.build(PartSpec("routed_experts", {
        "width": width, "n_experts": experts, "top": top, "inner": inner, "shared_inner": shared, "activation": "relu_sq",
        "gated": False}, "mlp"), "")
    w = {}
    for name, spec in part.tensor_specs().items():
        w[name] = (torch.randn(*spec.shape, generator=gen) * spec.shape[-1] ** -0.5).to(torch.bfloat16).float()
    w["mlp.router"] *= 3.0
    part.bind({k: dev(v, torch.float32 if part.tensor_specs()[k].role == "vector" else t) for k, v in w.items()})
    h = torch.randn(tokens, width, generator=gen).to(torch.bfloat16).float()
    raw = {"router": {"experts": experts, "top": top}, **({"shared": {"ff": shared}} if shared else {})}
    # rows whose choice is a close call are left out: rounding may turn it
    z = (h.double() @ w["mlp.router"].double().T).sort(dim=-1, descending=True).values
    clear = torch.ones(tokens, dtype=torch.bool) if top == experts else (z[:, top - 1] - z[:, top]) > 1e-4
    want = plain.routed_experts(h.double(), {k: v.double() for k, v in w.items()}, "mlp.", raw)
    positions = torch.arange(tokens, dtype=torch.int32)
    padded = tokens > 1
    if padded:
        positions[tokens // 2] = -1
        want[tokens // 2] = 0
    ctx = SimpleNamespace(ops=ops, positions=dev(positions), act_dtype=t)
    x = torch.randn(tokens, width, generator=gen)
    res = dev(x)
    assert part.forward(ctx, dev(h, t), res) is None
    tol = 2e-5 if dtype == "float32" else 3e-2
    assert torch.allclose((res.double().cpu() - x.double())[clear], want[clear], atol=tol, rtol=tol)
    out = part.forward(ctx, dev(h, t), None)                                        # the sum left for the norm behind it
    got, gain = dev(x), dev(torch.ones(width))
    ops.norm_add(got, out, gain, 1e-6, center=True)
    base = dev(x)
    ops.norm_add(base, res - dev(x), gain, 1e-6, center=True)
    assert torch.allclose(got.cpu(), base.cpu(), atol=2e-3)
    assert not padded or torch.equal(got[tokens // 2].cpu(), x[tokens // 2])


@pytest.mark.parametrize("dtype,path", [("float32", "general"), ("bfloat16", "general"), ("bfloat16", "tiles"), ("bfloat16", "wide")])
@pytest.mark.parametrize("window,pt", [(1, 8), (40, 8), (64, 16), (129, 4), (200, 16)])
def test_edges_of_the_window_over_latents(ops, dtype, path, window, pt):
    """The last query leans on one key: just inside the window it decides the row, just outside it must not touch it; in
    a whole prompt, in the last of two portions and decoded.  Places at page borders and the first token included."""
    rank = 152 if path == "wide" else 24                                            # rows of 160 and of 32 numbers
    raw, tensors = leaning_model(window, rank)
    loaded = load_model(config=NogatarConfig.from_dict(raw), tensors=tensors, dtype=dtype, device="cuda:0")
    kept = ops.use_mma_attention
    ops.use_mma_attention = path != "general"
    try:
        runner = make_runner(loaded, ops, pt, 420 // pt + 4, 2)
        length = 300
        for back in sorted({window - 1, window, window + 1, window // 2, (length - 1) % pt, length - 1}):
            if back == 0:
                continue                                                            # (the query's own place)
            tokens = leaning_tokens(raw, length, 3, length - 1 - back)
            want, other = (plain_logits(raw, tensors, t, [length - 1]) for t in (tokens, leaning_tokens(raw, length, 3, length - 1 - back, False)))
            moved = float(relative_error(other, want))
            assert moved > 0.3 if back < window else moved == 0.0
            for cut in (0, 150, length - 2, length - 1):
                if cut:
                    runner.step([StepEntry("r", tokens[:cut], [])])
                got = runner.step([StepEntry("r", tokens[cut:], [length - 1 - cut])])
                assert_rows_close(got, want, TOL[dtype], f"{back} back, cut at {cut}")
                runner.finish("r")
    finally:
        ops.use_mma_attention = kept


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("rank", [24, 152, 248])
def test_a_far_key_without_a_window_and_the_sinks(ops, dtype, rank):
    """No window: one key among hundreds, at page borders, decoded from many key ranges; then the sinks: heads whose sinks
    differ, at the first tokens (where the sink is most of the denominator) and later."""
    raw, tensors = leaning_model(None, rank)
    loaded = load_model(config=NogatarConfig.from_dict(raw), tensors=tensors, dtype=dtype, device="cuda:0")
    runner = make_runner(loaded, ops, 16, 100, 2)
    for far in (0, 15, 16, 31, 32, 500):
        tokens = leaning_tokens(raw, 700, 3, far)
        want = plain_logits(raw, tensors, tokens)
        assert float(relative_error(plain_logits(raw, tensors, leaning_tokens(raw, 700, 3, far, False), [699]), want[699:])) > 0.3
        got = runner.step([StepEntry("w", tokens, [699])])
        assert_rows_close(got, want[699:], TOL[dtype], f"whole, key at {far}")
        runner.step([StepEntry("d", tokens[:698], [])])
        outs = [runner.step([StepEntry("d", tokens[t: t + 1], [0])]) for t in (698, 699)]
        assert_rows_close(torch.cat(outs), want[698:], TOL[dtype], f"decoded, key at {far}")
        runner.finish("w"), runner.finish("d")
    tensors["l0.mix.sink"] = torch.tensor([4.0, -80.0])
    loaded = load_model(config=NogatarConfig.from_dict(raw), tensors=tensors, dtype=dtype, device="cuda:0")
    runner = make_runner(loaded, ops, 16, 100, 2)
    tokens = tokens_for(raw, 40, 5)
    want = plain_logits(raw, tensors, tokens)
    without = plain_logits(raw, {**tensors, "l0.mix.sink": torch.tensor([-80.0, -80.0])}, tokens)
    assert float(relative_error(without, want).median()) > 0.3
    assert_rows_close(runner.step([StepEntry("w", tokens, list(range(40)))]), want, TOL[dtype], "sinks, whole")
    outs = [runner.step([StepEntry("d", tokens[t: t + 1], [0])]) for t in range(40)]
    assert_rows_close(torch.cat(outs), want, TOL[dtype], "sinks, decoded")


# ---- the step function ---------------------------------------------------------------------------------------------
def setup(which, dtype, num_pages=64, seed=3, max_requests=4, raw=None, page_tokens=None, sharp=None):
    from mini_gpt_inference_b200.kernels.ops import default_ops

    raw = raw or config(which, every_expert=dtype == "bfloat16")      # (see nogatar_cases.all_experts)
    # (sharp softmaxes in 32-bit, where nothing but the order of sums differs; in bfloat16 they would magnify
    # the rounding of queries and keys)
    sharp = sharp if sharp is not None else (3.0 if dtype == "float32" else 1.0)
    tensors = random_weights(raw, seed, sharp=sharp, as_bfloat16=dtype == "bfloat16", steady=dtype == "bfloat16")
    loaded = load_model(config=NogatarConfig.from_dict(raw), tensors=tensors, dtype=dtype, device="cuda:0")
    runner = make_runner(loaded, default_ops("cuda:0"), page_tokens or PAGE_TOKENS[which], num_pages, max_requests)
    return raw, tensors, runner, (TOL[dtype], 0.03 if dtype == "bfloat16" else 0.0, dtype)


def expect(raw, tensors, tokens, tol):
    """The plain logits of a sequence and the keywords of the comparison with them (see ``rounding_spread``)."""
    kw = {"outliers": tol[1]}
    if tol[2] == "bfloat16":
        kw["slack"] = rounding_spread(raw, tensors, tokens)
    return plain_logits(raw, tensors, tokens), kw


@pytest.mark.parametrize("which,dtype", CASES, ids=IDS)
def test_whole_prompts(which, dtype):
    raw, tensors, runner, tol = setup(which, dtype, num_pages=100)
    pt = PAGE_TOKENS[which]
    for length, seed in [(150, 1), (37, 2), (1, 3), (2, 4), (pt + 1, 5), (pt, 6), (190, 7)]:
        tokens = tokens_for(raw, length, seed)
        got = runner.step([StepEntry("r", tokens, list(range(length)))])
        runner.finish("r")
        assert got.shape == (length, raw["vocab"]) and got.dtype == torch.float32
        want, kw = expect(raw, tensors, tokens, tol)
        assert_rows_close(got, want, tol[0], f"whole prompt of {length}", **kw)
    runner.manager.check()
    assert runner.manager.stats()["allocated_blocks"] == 0


@pytest.mark.parametrize("which,dtype", CASES, ids=IDS)
def test_prefill_then_single_tokens(which, dtype):
    """A short prompt, then a long run of single tokens (replayed from a CUDA graph), and the same sequence token by
    token from the very first token."""
    raw, tensors, runner, tol = setup(which, dtype)
    tokens = tokens_for(raw, 150, 7)
    want, kw = expect(raw, tensors, tokens, tol)
    outs = [runner.step([StepEntry("r", tokens[:9], list(range(9)))])]
    outs += [runner.step([StepEntry("r", tokens[t: t + 1], [0])]) for t in range(9, 150)]
    assert_rows_close(torch.cat(outs), want, tol[0], "prefill then single tokens", **kw)
    assert runner.graph_replays > 100
    one_by_one = torch.cat([runner.step([StepEntry("s", tokens[t: t + 1], [0])]) for t in range(40)])
    assert_rows_close(one_by_one, want[:40], tol[0], "single tokens from the first",
                      **{k: (v[:40] if k == "slack" else v) for k, v in kw.items()})
    if dtype == "float32":
        # in 32-bit the cut into steps changes no bit
        assert torch.equal(one_by_one, torch.cat(outs)[:40])


@pytest.mark.parametrize("which,dtype", CASES, ids=IDS)
def test_portions_of_changing_size(which, dtype):
    raw, tensors, runner, tol = setup(which, dtype)
    tokens = tokens_for(raw, 171, 8)
    want, kw = expect(raw, tensors, tokens, tol)
    sizes = itertools.cycle([13, 7, 2, 5, 2, 1, 3, 16, 2, 9, 70])
    outs, pos = [], 0
    while pos < len(tokens):
        n = min(next(sizes), len(tokens) - pos)
        outs.append(runner.step([StepEntry("r", tokens[pos: pos + n], list(range(n)))]))
        pos += n
    assert_rows_close(torch.cat(outs), want, tol[0], "portions of changing size", **kw)
    if dtype == "float32":
        runner.finish("r")
        assert torch.equal(torch.cat(outs), runner.step([StepEntry("r", tokens, list(range(len(tokens))))]))


@pytest.mark.parametrize("which,dtype", CASES, ids=IDS)
def test_mixed_batches_reuse_pages_and_slots(which, dtype):
    """Up to four live requests, portions of some beside single tokens of others, requests left out of
    steps; pages and state slots are handed out again.  Every cache row and state slot starts as NaN and
    turns NaN again as soon as no request holds it."""
    pt = PAGE_TOKENS[which]
    lengths = [90, 29, 71, 3, 41, 2 * pt, 17, 55, 1]
    pool = sum(sorted(-(-n // pt) for n in lengths)[-4:])
    raw, tensors, runner, tol = setup(which, dtype, num_pages=pool)
    for pages in runner.storage.k + runner.storage.v:
        if pages is not None:
            pages.fill_(float("nan"))
    for state in runner.storage.state.values():
        state.fill_(float("nan") if state.is_floating_point() else -1)
    reqs = {f"q{i}": tokens_for(raw, n, 20 + i) for i, n in enumerate(lengths)}
    want = {rid: expect(raw, tensors, toks, tol) for rid, toks in reqs.items()}
    got = {rid: [] for rid in reqs}
    waiting, live = list(reqs), {}
    sizes = itertools.cycle([5, 1, 2, 11, 1, 1, 7, 3, 1, 2, 1, 1, 40])
    gen = torch.Generator().manual_seed(99)
    while waiting or live:
        while waiting and len(live) < 4:
            live[waiting.pop(0)] = 0
        entries, order = [], []
        for rid in list(live):
            if len(live) > 1 and torch.rand((), generator=gen).item() < 0.25:
                continue
            pos = live[rid]
            n = min(next(sizes), len(reqs[rid]) - pos)
            entries.append(StepEntry(rid, reqs[rid][pos: pos + n], list(range(n))))
            order.append((rid, n))
            live[rid] = pos + n
        if not entries:
            continue
        logits = runner.step(entries)
        row = 0
        for rid, n in order:
            got[rid].append(logits[row: row + n].clone())
            row += n
            if live[rid] == len(reqs[rid]):
                slot = runner.manager.get(rid).state_slot
                runner.finish(rid)
                del live[rid]
                for state in runner.storage.state.values():
                    state[slot] = float("nan") if state.is_floating_point() else -1
        for g, group in enumerate(runner.manager.groups):                 # pages that nobody holds, a window's old ones too
            held = {p for r in runner.manager.requests.values() for p in r.tables[g]}
            free = [p for p in range(group.num_pages) if p not in held]
            runner.storage.k[g][:, free] = float("nan")
    for rid in reqs:
        assert_rows_close(torch.cat(got[rid]), want[rid][0], tol[0], f"request {rid} in mixed batches", **want[rid][1])
    runner.manager.check()
    assert runner.manager.stats()["allocated_blocks"] == 0


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_batch_of_unequal_requests_equals_each_alone(dtype):
    raw, tensors, runner, tol = setup("A", dtype, num_pages=64, max_requests=8)
    prompts = [tokens_for(raw, n, 70 + n) for n in (1, 2, 33, 64, 7)]
    alone = []
    for i, p in enumerate(prompts):
        alone.append(runner.step([StepEntry(f"a{i}", p, list(range(len(p))))]))
        runner.finish(f"a{i}")
    together = runner.step([StepEntry(f"b{i}", p, list(range(len(p)))) for i, p in enumerate(prompts)])
    if dtype == "float32":
        assert torch.equal(together, torch.cat(alone))
    else:
        assert float(relative_error(together, torch.cat(alone).cpu()).max()) < tol[0]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_prompts_and_long_decoding(dtype):
    raw, tensors, runner, tol = setup("B", dtype, num_pages=40)
    tokens = tokens_for(raw, 400, 17)
    want, kw = expect(raw, tensors, tokens, tol)
    outs = [runner.step([StepEntry("r", tokens[:300], list(range(300)))])]
    outs += [runner.step([StepEntry("r", tokens[t: t + 1], [0])]) for t in range(300, 400)]
    assert_rows_close(torch.cat(outs), want, tol[0], "long prompt, long decoding", **kw)


@pytest.mark.parametrize("seed", range(8))
def test_configurations_drawn_at_random(seed):
    rng = random.Random(seed)
    raw = random_config(rng)
    pt = rng.choice([16, 64])
    for dtype in ("float32", "bfloat16"):
        if dtype == "bfloat16":
            raw = all_experts(raw)
        _, tensors, runner, tol = setup(None, dtype, num_pages=600 // pt + 8, seed=seed, raw=raw, page_tokens=pt, sharp=1.0)
        tokens = tokens_for(raw, 200, seed)
        want, kw = expect(raw, tensors, tokens, tol)
        whole = runner.step([StepEntry("w", tokens, list(range(200)))])
        assert_rows_close(whole, want, tol[0], f"seed {seed} {dtype} whole", **kw)
        sizes = itertools.cycle([70, 3, 2, 33, 1, 64])
        outs, pos = [], 0
        while pos < 170:
            n = min(next(sizes), 170 - pos)
            outs.append(runner.step([StepEntry("p", tokens[pos: pos + n], list(range(n)))]))
            pos += n
        outs += [runner.step([StepEntry("p", tokens[t: t + 1], [0])]) for t in range(170, 200)]
        assert_rows_close(torch.cat(outs), want, tol[0], f"seed {seed} {dtype} portions", **kw)
        if dtype == "float32":
            assert torch.equal(torch.cat(outs), whole)


# ---- generation through the entry point, its scheduler and sampler ---------------------------------
@pytest.mark.parametrize("which", "ABC")
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_greedy_generation_through_the_engine(which, dtype):
    raw = config(which, every_expert=dtype == "bfloat16")
    tensors = random_weights(raw, 11, as_bfloat16=dtype == "bfloat16", steady=dtype == "bfloat16")
    loaded = load_model(config=NogatarConfig.from_dict(raw), tensors=tensors, dtype=dtype, device="cuda:0")
    engine = LLMEngine(loaded, EngineConfig(dtype=dtype, block_size=PAGE_TOKENS[which], num_blocks=48,
                                            max_batch_size=3, max_num_batched_tokens=16, max_prefill_chunk=7))
    prompts = [tokens_for(raw, n, 40 + i) for i, n in enumerate([5, 1, 23, 12, 2, 17])]
    outs = engine.generate(prompts, SamplingParams(max_tokens=12, temperature=0.0))
    for prompt, out in zip(prompts, outs):
        assert len(out["token_ids"]) == 12 and out["finish_reason"] == "length"
        seq = prompt + out["token_ids"]
        want = plain_logits(raw, tensors, seq[:-1])
        slack = rounding_spread(raw, tensors, seq[:-1]) if dtype == "bfloat16" else torch.zeros(len(seq))
        for i, token in enumerate(out["token_ids"]):
            row, at = want[len(prompt) - 1 + i], len(prompt) - 1 + i
            assert row.max() - row[token] <= 2 * (TOL[dtype] + 3 * float(slack[at])) * row.std(), (i, token, int(row.argmax()))
        if dtype == "float32":
            assert out["token_ids"] == plain_greedy(raw, tensors, prompt, 12)
    assert engine.stats()["allocated_blocks"] == 0
    engine.runner.manager.check()


def test_preemption_and_recompute_through_the_engine():
    raw = config("C")
    tensors = random_weights(raw, 14)
    loaded = load_model(config=NogatarConfig.from_dict(raw), tensors=tensors, dtype="float32", device="cuda:0")
    engine = LLMEngine(loaded, EngineConfig(dtype="float32", block_size=8, num_blocks=10, max_batch_size=3,
                                            max_num_batched_tokens=16, max_prefill_chunk=7))
    prompts = [tokens_for(raw, n, 60 + i) for i, n in enumerate([20, 25, 18, 9])]
    outs = engine.generate(prompts, SamplingParams(max_tokens=16, temperature=0.0))
    assert engine.scheduler.num_preemptions > 0
    for prompt, out in zip(prompts, outs):
        assert out["token_ids"] == plain_greedy(raw, tensors, prompt, 16)
    assert engine.stats()["allocated_blocks"] == 0
    engine.runner.manager.check()


def test_long_decoding_through_the_engine():
    raw = config("A")
    tensors = random_weights(raw, 12)
    loaded = load_model(config=NogatarConfig.from_dict(raw), tensors=tensors, dtype="float32", device="cuda:0")
    engine = LLMEngine(loaded, EngineConfig(dtype="float32", block_size=8, num_blocks=40, max_batch_size=2))
    prompt = tokens_for(raw, 3, 9)
    out = engine.generate([prompt], SamplingParams(max_tokens=160, temperature=0.0))[0]
    assert out["token_ids"] == plain_greedy(raw, tensors, prompt, 160)


def test_trace_replay(tmp_path):
    """The replay program on a model folder: two requests, portions beside single tokens, a slot and pages
    used again by a third request."""
    from mini_gpt_inference_b200.engine.trace import main
    from mini_gpt_inference_b200.weights.safetensors_io import save_file

    raw = config("A", every_expert=True)
    tensors = random_weights(raw, 13, as_bfloat16=True, steady=True)
    folder = tmp_path / "model"
    folder.mkdir()
    (folder / "config.json").write_text(json.dumps(raw))
    save_file({k: v.to(torch.bfloat16) for k, v in tensors.items()}, folder / "model.safetensors")
    a, b, c = tokens_for(raw, 50, 1), tokens_for(raw, 20, 2), tokens_for(raw, 64, 3)
    steps = [
        {"step": 0, "entries": [{"id": "a", "tokens": a[:30], "want": [0, 29]}], "end": []},
        {"step": 1, "entries": [{"id": "a", "tokens": a[30:31], "want": [0]}, {"id": "b", "tokens": b[:7], "want": []}], "end": []},
        {"step": 2, "entries": [{"id": "b", "tokens": b[7:], "want": [12]}, {"id": "a", "tokens": a[31:], "want": [18]}], "end": ["a", "b"]},
        {"step": 3, "entries": [{"id": "c", "tokens": c[:62], "want": [61]}], "end": []},
        {"step": 4, "entries": [{"id": "c", "tokens": c[62:], "want": [0, 1]}], "end": ["c"]},
    ]
    for dtype in ("float32", "bfloat16"):
        out = tmp_path / dtype
        stdout = io.StringIO()
        code = main(["--model", str(folder), "--dtype", dtype, "--out", str(out), "--max-tokens", "128",
                     "--live-requests", "2"], stdin=io.StringIO("\n".join(json.dumps(s) for s in steps) + "\n"),
                    stdout=stdout)
        assert code == 0 and stdout.getvalue().split() == ["done", "0", "done", "1", "done", "2", "done", "3", "done", "4"]
        la, lb, lc = (plain_logits(raw, tensors, t) for t in (a, b, c))
        sa, sb, sc = (rounding_spread(raw, tensors, t) if dtype == "bfloat16" else torch.zeros(len(t)) for t in (a, b, c))
        want = {0: (la[[0, 29]], sa[[0, 29]]), 1: (la[[30]], sa[[30]]), 2: (torch.stack([lb[19], la[49]]), torch.stack([sb[19], sa[49]])),
                3: (lc[[61]], sc[[61]]), 4: (lc[[62, 63]], sc[[62, 63]])}
        for step, (rows, slack) in want.items():
            got = torch.from_numpy(np.fromfile(out / f"{step}.f32", dtype="<f4").reshape(len(rows), raw["vocab"]))
            assert_rows_close(got, rows, 2 * TOL[dtype], f"{dtype} step {step}", slack=slack)


def test_command_line_writes_and_generates(tmp_path):
    """bin/generate: a random-weights folder from a config.json, then greedy tokens from it that equal the
    plain implementation's on the folder's own tensors."""
    import subprocess
    import sys
    from pathlib import Path

    from mini_gpt_inference_b200.weights import load_file

    root = Path(__file__).resolve().parent.parent
    raw = config("D")
    cfg_path = tmp_path / "config.json"
    cfg_path.write_text(json.dumps(raw))
    folder = tmp_path / "model"
    made = subprocess.run([sys.executable, str(root / "bin" / "generate"), "--random-weights", "3", "--config", str(cfg_path),
                           "--write-model", str(folder), "--weights-dtype", "bfloat16"], capture_output=True, text=True)
    assert made.returncode == 0, made.stderr[-2000:]
    prompt = tokens_for(raw, 9, 5)
    run = subprocess.run([sys.executable, str(root / "bin" / "generate"), "--model", str(folder), "--dtype", "float32",
                          "--prompt-ids", ",".join(map(str, prompt)), "--max-new-tokens", "8", "--temperature", "0"],
                         capture_output=True, text=True)
    assert run.returncode == 0, run.stderr[-2000:]
    out = json.loads(run.stdout.strip().splitlines()[-1])
    assert out["token_ids"] == plain_greedy(raw, load_file(folder / "model.safetensors"), prompt, 8)
