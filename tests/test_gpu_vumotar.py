"""Vumotar on the GPU against the plain implementation: the new kernels alone, single keys at the edges of windows and
among the kept first tokens, the step function under every way of cutting requests into steps, batches, pages and slots
used again, then generation through the entry point."""

from __future__ import annotations

import io
import itertools
import json
import random
from types import SimpleNamespace

import numpy as np
import pytest
import torch

import plain_vumotar as plain
from vumotar_cases import (PAGE_TOKENS, _attention, _latent, _tempered, all_experts, assert_rows_close, config, disliking_model,
                           leaning_model, leaning_tokens, plain_greedy, plain_logits, random_config, random_weights, relative_error,
                           rounding_spread, tokens_for)

from mini_gpt_inference_b200 import EngineConfig, LLMEngine, SamplingParams, VumotarConfig
from mini_gpt_inference_b200.engine.build import load_model, make_runner
from mini_gpt_inference_b200.engine.runner import StepEntry

pytestmark = pytest.mark.gpu

# Largest |engine - plain| on a row of logits, over the row's own spread.  32-bit: rounding of sums.
# bfloat16: both sides use the same weights; activations are rounded to 8 bits between kernels.  A
# lost key, sink, norm or expert shows as 0.3 and more.
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
def test_norm_behind_a_sublayer_and_the_next_one(ops, rows, width):
    """The stream plus the norm of a sublayer's output, and another norm of the new stream, in both types; from one
    buffer (left as zeros or not) and from a sum over entries; widths that the vector form takes and that it does not."""
    from mini_gpt_inference_b200.kernels.ops import EntrySum

    gen = torch.Generator().manual_seed(rows + width)
    x, a = torch.randn(rows, width, generator=gen), 5.0 * torch.randn(rows, width, generator=gen)
    w, w2 = (1 + 0.3 * torch.randn(width, generator=gen) for _ in range(2))
    new = x.double() + plain.rms_norm(a.double(), w.double(), 1e-3)
    want = plain.rms_norm(new, w2.double(), 1e-2)
    for clear in (False, True):
        for t in (torch.float32, torch.bfloat16):
            xa, ya = dev(x), dev(a)
            got = ops.norm_add(xa, ya, dev(w), 1e-3, clear=clear, rows_dtype=t, then=(dev(w2), 1e-2, 0.0))
            assert torch.allclose(xa.double().cpu(), new, atol=2e-5) and got.dtype == t
            tol = 3e-5 if t == torch.float32 else 2e-2
            assert torch.allclose(got.double().cpu(), want, atol=tol, rtol=tol)
            assert not bool(ya.any()) if clear else torch.equal(ya.cpu(), a)
    top = 3
    terms = torch.randn(rows * top, width, generator=gen)
    slots = torch.randperm(rows * top, generator=gen).view(rows, top).to(torch.int32)
    slots[0, 1] = -1
    total = torch.stack([sum((terms[s].double() for s in r if s >= 0), torch.zeros(width, dtype=torch.float64)) for r in slots.tolist()])
    new = x.double() + 0.7 * plain.rms_norm(total, w.double() + 1, 1e-3)
    xa = dev(x)
    got = ops.norm_add(xa, EntrySum(dev(terms), dev(slots)), dev(w), 1e-3, offset=1.0, norm_scale=0.7, rows_dtype=torch.float32,
                       then=(dev(w2), 1e-4, 1.0))
    assert torch.allclose(xa.double().cpu(), new, atol=3e-5)
    assert torch.allclose(got.double().cpu(), plain.rms_norm(new, w2.double() + 1, 1e-4), atol=5e-5, rtol=5e-5)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("q_rank,rank,gap", [(96, 64, 0), (13, 40, 3), (1536, 512, 8), (8, 21, 0), (32, 1024, 0)])
def test_two_latents_of_a_token(ops, dtype, q_rank, rank, gap):
    from mini_gpt_inference_b200.cache.storage import PagedKVView

    t = DTYPES[dtype]
    gen = torch.Generator().manual_seed(q_rank + rank)
    positions = torch.tensor([0, 3, 1, 900, -1, 3300], dtype=torch.int32)
    slots = torch.tensor([5, 0, 11, 6, -1, 2], dtype=torch.int32)
    n, low_off, pt, eps = positions.numel(), q_rank + gap, 4, 1e-3
    proj = torch.randn(n, low_off + rank + 8, generator=gen).to(t)
    q_gain, gain = (1 + 0.3 * torch.randn(k, generator=gen) for k in (q_rank, rank))
    pages = dev(torch.full((3, 1, pt, rank), float("nan")), t)
    cache = PagedKVView(pages, pages, 0, pt, None, True, values_in_keys=True)
    got = ops.latent_pair_prepare(dev(proj), 0, q_rank, dev(q_gain), low_off, rank, dev(gain), eps, cache, dev(slots), dev(positions))
    x, live = proj.double(), positions >= 0
    tol = 3e-5 if dtype == "float32" else 2e-2
    assert torch.allclose(got.double().cpu()[live], plain.rms_norm(x[:, :q_rank], q_gain.double(), eps)[live], atol=tol, rtol=tol)
    rows = pages.double().cpu().view(-1, rank)
    want = plain.rms_norm(x[:, low_off: low_off + rank], gain.double(), eps)
    assert torch.allclose(rows[slots[live].long()], want[live], atol=tol, rtol=tol)
    written = torch.zeros(3 * pt, dtype=torch.bool)
    written[slots[live].long()] = True
    assert bool(torch.isnan(rows[~written]).all())


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("tokens", [1, 7, 16, 17, 40, 300])
@pytest.mark.parametrize("heads,n_in,n_out", [(6, 128, 40), (3, 40, 24), (5, 20, 14), (16, 512, 128)])
def test_heads_matrices_with_one_gate_a_head(ops, dtype, tokens, heads, n_in, n_out):
    t = DTYPES[dtype]
    gen = torch.Generator().manual_seed(tokens + n_in)
    x = torch.randn(tokens, heads * n_in, generator=gen).to(t)
    w = (torch.randn(heads * n_out, n_in, generator=gen) * n_in ** -0.5).to(t)
    rows = torch.randn(tokens, 9 + heads, generator=gen).to(t)                      # (gates at an odd column of wider rows)
    got = ops.head_linear(dev(x), 0, n_in, dev(w), False, heads, n_in, n_out, gate=dev(rows)[:, 9:])
    y = torch.einsum("nhi,hji->nhj", x.double().view(tokens, heads, n_in), w.double().view(heads, n_out, n_in))
    want = (y * torch.sigmoid(rows.double()[:, 9:])[:, :, None]).reshape(tokens, -1)
    tol = 3e-5 if dtype == "float32" else 2e-2
    assert got.shape == want.shape and torch.allclose(got.double().cpu(), want, atol=tol, rtol=tol)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("norm", [False, True])
@pytest.mark.parametrize("coef,every", [(0.25, 128), (-0.4, 1), (1.5, 7), (0.2, 2.5)])
def test_query_temperature(ops, dtype, norm, coef, every):
    """At the steps' edges and far away; keys and values do not change with it."""
    from mini_gpt_inference_b200.cache.storage import PagedKVView

    t = DTYPES[dtype]
    heads, kv, d, dv, pt = 3, 1, 24, 40, 4
    positions = torch.tensor([0, 1, 5, 6, 7, 254, 255, 256, 511, -1, 100000], dtype=torch.int32)
    n = positions.numel()
    slots = torch.arange(n, dtype=torch.int32)
    slots[9] = -1
    gen = torch.Generator().manual_seed(int(every))
    proj = torch.randn(n, heads * d + kv * (d + dv), generator=gen).to(t)
    gains = {"q_gain": 1 + 0.3 * torch.randn(d, generator=gen), "k_gain": 1 + 0.3 * torch.randn(d, generator=gen)} if norm else {}
    k_pages, v_pages = dev(torch.zeros(3, kv, pt, d), t), dev(torch.zeros(3, kv, pt, dv), t)
    rows = dev(proj)
    ops.head_prepare(rows, heads, kv, d, dv, 0, heads * d, heads * d + kv * d, norm, 1e-3, PagedKVView(k_pages, v_pages, 0, pt, None, True),
                     dev(slots), dev(positions), q_temperature=(coef, every), **{k: dev(v) for k, v in gains.items()})
    q, k = proj[:, : heads * d].double().view(n, heads, d), proj[:, heads * d: heads * d + kv * d].double().view(n, kv, d)
    if norm:
        q, k = plain.rms_norm(q, gains["q_gain"].double(), 1e-3), plain.rms_norm(k, gains["k_gain"].double(), 1e-3)
    grown = plain.temperature(100001, coef, every)[positions.clamp(min=0).long()]
    tol, live = (2e-5 if dtype == "float32" else 1e-2), positions >= 0
    got = rows[:, : heads * d].double().cpu().view(n, heads, d)
    assert torch.allclose(got[live], (q * grown[:, None, None])[live], atol=tol, rtol=tol)
    assert torch.equal(rows[~live].cpu(), proj[~live])
    kept = k_pages.double().cpu().permute(0, 2, 1, 3).reshape(-1, kv, d)[: n]
    assert torch.allclose(kept[live], k[live], atol=tol, rtol=tol)
    assert torch.equal(v_pages.cpu().permute(0, 2, 1, 3).reshape(-1, dv)[: n][live], proj[live, heads * d + kv * d:])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("tokens", [1, 5, 64, 65, 200, 1187])
@pytest.mark.parametrize("experts,top,width,inner,shared", [(5, 2, 64, 40, 40), (4, 1, 96, 48, None), (3, 3, 72, 20, 50),
                                                            (16, 4, 128, 128, 64), (2, 1, 70, 33, 33)])
def test_router_and_experts_whose_input_is_weighed(ops, dtype, tokens, experts, top, width, inner, shared):
    """The part on its own against the plain feed-forward, the shared expert among the chosen ones; both ways of handing
    its output on; a padding row."""
    from mini_gpt_inference_b200.parts.base import FEED_FORWARDS
    from mini_gpt_inference_b200.parts.spec import PartSpec

    t = DTYPES[dtype]
    gen = torch.Generator().manual_seed(experts * 100 + inner)
    part = FEED_FORWARDS.build(PartSpec("routed_experts", {
        "width": width, "n_experts": experts, "top": top, "inner": inner, "shared_inner": shared, "shared_gate": False,
        "scoring": "sigmoid", "weigh": "input"}, "mlp"), "")
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
    got, base, gain = dev(x), dev(x), dev(torch.ones(width))
    ops.norm_add(got, out, gain, 1e-6)
    ops.norm_add(base, res - dev(x), gain, 1e-6)
    assert torch.allclose(got.cpu()[clear], base.cpu()[clear], atol=2e-3)
    assert not padded or torch.equal(got[tokens // 2].cpu(), x[tokens // 2])


def test_sigmoid_router_takes_the_lower_number_of_equal_scores(ops):
    """Also where the scores are as large as they get: the logistic function of large logits is 1 for all of them."""
    h = torch.ones(3, 64)
    w = torch.zeros(6, 64)
    w[2:5] = 10.0
    ids, weights, gate = ops.moe_route(dev(h), dev(w), None, dev(torch.tensor([0, 1, -1], dtype=torch.int32)), 2, always=1,
                                       scoring="sigmoid", scale=0.5)
    assert gate is None and ids.cpu().tolist() == [[2, 3, 6]] * 2 + [[-1] * 3]
    assert weights.cpu()[:2].tolist() == [[0.5, 0.5, 1.0]] * 2


@pytest.mark.parametrize("dtype,path", [("float32", "general"), ("bfloat16", "general"), ("bfloat16", "tiles")])
@pytest.mark.parametrize("heads,kv,d,dv", [(4, 2, 32, 24), (6, 1, 96, 64), (3, 3, 128, 128), (20, 1, 64, 80)])
@pytest.mark.parametrize("window,keep", [(20, 4), (64, 64), (1, 1), (100, 65), (30, 200), (129, 7), (None, 0)])
def test_attention_with_kept_first_tokens(ops, dtype, path, heads, kv, d, dv, window, keep):
    """The attention kernels alone against plain attention: two requests of unequal length as whole portions, the ends of
    portions, and single tokens; pages that no query may read are missing from the tables and hold NaN."""
    from mini_gpt_inference_b200.cache.storage import PagedKVView

    t, pt, lengths, scale = DTYPES[dtype], 16, (391, 130), 1.3 * d ** -0.5
    gen = torch.Generator().manual_seed(d + keep)
    size = None if window is None else window
    data = [[(torch.randn(n, c, f, generator=gen)).to(t) for c, f in ((heads, d), (kv, d), (kv, dv))] for n in lengths]
    sinks = torch.randn(heads, generator=gen)
    want = [plain.attend(*(x.double() for x in req), scale, plain.visible(n, size, keep), sinks.double()) for req, n in zip(data, lengths)]
    n_pages = [-(-n // pt) for n in lengths]
    total = sum(n_pages)
    order = torch.randperm(total, generator=gen).tolist()
    kept = ops.use_mma_attention
    ops.use_mma_attention = path == "tiles"
    try:
        for portions in ((391, 130), (1, 1), (70, 2), (1, 65), (33, 1)):
            k_pages = torch.full((total, kv, pt, d), float("nan"), dtype=t)
            v_pages = torch.full((total, kv, pt, dv), float("nan"), dtype=t)
            table = torch.full((2, max(n_pages)), -1, dtype=torch.int32)
            ids = iter(order)
            for r, n in enumerate(lengths):
                lo = 0 if window is None else max(0, n - portions[r] - window + 1)
                for page in range(n_pages[r]):
                    first, last = page * pt, min(n, (page + 1) * pt)
                    if first >= keep and last <= lo:
                        continue                                                    # given back long ago
                    slot = next(ids)
                    table[r, page] = slot
                    k_pages[slot, :, : last - first] = data[r][1][first:last].transpose(0, 1)
                    v_pages[slot, :, : last - first] = data[r][2][first:last].transpose(0, 1)
            cache = PagedKVView(dev(k_pages), dev(v_pages), 0, pt, window, True, keep_first=keep)
            q = torch.cat([data[r][0][lengths[r] - m:].reshape(m, -1) for r, m in enumerate(portions)])
            pos = torch.cat([torch.arange(lengths[r] - m, lengths[r]) for r, m in enumerate(portions)]).to(torch.int32)
            single = portions == (1, 1)
            ctx = SimpleNamespace(block_tables=[dev(table)], token_request=dev(torch.repeat_interleave(torch.arange(2), torch.tensor(portions)).to(torch.int32)),
                                  positions=dev(pos), req_q_start=dev(torch.tensor([0, portions[0]], dtype=torch.int32)),
                                  req_q_len=dev(torch.tensor(portions, dtype=torch.int32)), host_q_len=list(portions), extra={},
                                  decode_only=single, max_ctx_after=max(lengths))
            got = ops.paged_attention_general(dev(q), heads, kv, d, dv, scale, cache, ctx, sinks=dev(sinks)).double().cpu()
            expected = torch.cat([want[r][lengths[r] - m:].reshape(m, -1) for r, m in enumerate(portions)])
            tol = 2e-5 if dtype == "float32" else 2e-2
            assert torch.allclose(got, expected, atol=tol, rtol=tol), (portions, float((got - expected).abs().max()))
    finally:
        ops.use_mma_attention = kept


# ---- single keys ------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype,path", [("float32", "general"), ("bfloat16", "general"), ("bfloat16", "tiles")])
@pytest.mark.parametrize("kind,window,keep,pt", [
    ("attention", 40, 4, 8), ("attention", 64, 16, 16), ("attention", 129, 1, 4), ("attention", 70, 100, 16), ("attention", 1, 3, 8),
    ("attention", None, 0, 16), ("latent", 1, 0, 8), ("latent", 40, 0, 8), ("latent", 64, 0, 16), ("latent", 129, 0, 4),
    ("wide latent", 100, 0, 16), ("latent", None, 0, 16), ("attention_2", None, 0, 16), ("attention_2 64", None, 0, 16)])
def test_single_keys_at_every_edge(ops, dtype, path, kind, window, keep, pt):
    """The last query leans on one key: just inside the window or among the kept first tokens it decides the row, just
    outside it must not touch it; in a whole prompt, in the last of two portions and decoded.  Places at page borders,
    far away and the first token included."""
    layer = {"attention": _attention(4, 2, 32, 24, window, keep, 0.2), "attention_2": _tempered(4, 2, 32, 24, 0.4, 64, 0.2),
             "attention_2 64": _tempered(4, 2, 64, 64, 0.4, 64, 0.125), "latent": _latent(2, 32, 24, 24, 40, window, 0.2),
             "wide latent": _latent(2, 32, 24, 24, 160, window, 0.2)}[kind]
    raw, tensors = leaning_model(layer)
    loaded = load_model(config=VumotarConfig.from_dict(raw), tensors=tensors, dtype=dtype, device="cuda:0")
    mma = ops.use_mma_attention
    ops.use_mma_attention = path != "general"
    try:
        runner = make_runner(loaded, ops, pt, 420 // pt + 4, 2)
        length = 300
        last = length - 1
        places = {0, 1, pt - 1, pt, 63, 64, keep - 1, keep, keep + 1, last - 1, last - last % pt - 1}
        if window is not None:
            places |= {last - window + 1, last - window, last - window - 1, last - window // 2}
        for at in sorted(p for p in places if 0 <= p < last):
            seen = window is None or last - at < window or at < keep
            tokens = leaning_tokens(raw, length, 3, at)
            want, other = (plain_logits(raw, tensors, t, [last]) for t in (tokens, leaning_tokens(raw, length, 3, at, False)))
            moved = float(relative_error(other, want))
            assert moved > 0.3 if seen else moved == 0.0
            for cut in (0, 150, last - 1, last):
                if cut:
                    runner.step([StepEntry("r", tokens[:cut], [])])
                got = runner.step([StepEntry("r", tokens[cut:], [last - cut])])
                assert_rows_close(got, want, TOL[dtype], f"key at {at} of {length}, cut at {cut}")
                runner.finish("r")
    finally:
        ops.use_mma_attention = mma


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("what", ["learned sinks", "term of 1", "temperature"])
def test_sinks_and_temperature_show(ops, dtype, what):
    """What each of them changes is far above the tolerance.  (The norm behind a mixer takes a factor that all heads share
    away: a sink shows where heads differ.)"""
    if what == "learned sinks":
        raw, w = leaning_model(_latent(2, 32, 24, 24, 40, 30, 0.2))
        w["l0.mix.sink"] = torch.tensor([4.0, -80.0])
        without = plain_logits(raw, {**w, "l0.mix.sink": torch.tensor([-80.0, -80.0])}, tokens_for(raw, 60, 5))
    elif what == "term of 1":
        raw, w = disliking_model()
        attend = plain.attend
        plain.attend = lambda q, k, v, scale, seen, extra=None: attend(q, k, v, scale, seen)
        try:
            without = plain_logits(raw, w, tokens_for(raw, 60, 5))
        finally:
            plain.attend = attend
    else:
        raw, _ = leaning_model(_tempered(4, 2, 32, 24, 1.5, 4, 0.2))
        w = random_weights(raw, 6, sharp=2.0, as_bfloat16=True)
        flat = json.loads(json.dumps(raw))
        del flat["layers"][0]["mixer"]["q_temp"]
        without = plain_logits(flat, w, tokens_for(raw, 60, 5))
    tokens = tokens_for(raw, 60, 5)
    want = plain_logits(raw, w, tokens)
    assert float(relative_error(without, want)[10:].median()) > 0.3
    kw = {"slack": rounding_spread(raw, w, tokens)} if dtype == "bfloat16" else {}
    loaded = load_model(config=VumotarConfig.from_dict(raw), tensors=w, dtype=dtype, device="cuda:0")
    runner = make_runner(loaded, ops, 16, 100, 2)
    assert_rows_close(runner.step([StepEntry("w", tokens, list(range(60)))]), want, TOL[dtype], what + ", whole", **kw)
    outs = [runner.step([StepEntry("d", tokens[t: t + 1], [0])]) for t in range(60)]
    assert_rows_close(torch.cat(outs), want, TOL[dtype], what + ", decoded", **kw)


# ---- the step function ---------------------------------------------------------------------------------------------
def setup(which, dtype, num_pages=64, seed=3, max_requests=4, raw=None, page_tokens=None, sharp=None):
    from mini_gpt_inference_b200.kernels.ops import default_ops

    raw = raw or config(which, every_expert=dtype == "bfloat16")      # (see vumotar_cases.all_experts)
    # (sharp softmaxes in 32-bit, where nothing but the order of sums differs; in bfloat16 they would magnify
    # the rounding of queries and keys)
    sharp = sharp if sharp is not None else (3.0 if dtype == "float32" else 1.0)
    tensors = random_weights(raw, seed, sharp=sharp, as_bfloat16=dtype == "bfloat16")
    loaded = load_model(config=VumotarConfig.from_dict(raw), tensors=tensors, dtype=dtype, device="cuda:0")
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
    steps; pages and state slots are handed out again.  Every cache row starts as NaN and turns NaN again as soon as no
    request holds it."""
    pt = PAGE_TOKENS[which]
    lengths = [90, 29, 71, 3, 41, 2 * pt, 17, 55, 1]
    pool = sum(sorted(-(-n // pt) for n in lengths)[-4:])
    raw, tensors, runner, tol = setup(which, dtype, num_pages=pool)
    for pages in runner.storage.k + runner.storage.v:
        if pages is not None:
            pages.fill_(float("nan"))
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
                runner.finish(rid)
                del live[rid]
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
    tensors = random_weights(raw, 11, as_bfloat16=dtype == "bfloat16")
    loaded = load_model(config=VumotarConfig.from_dict(raw), tensors=tensors, dtype=dtype, device="cuda:0")
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
    loaded = load_model(config=VumotarConfig.from_dict(raw), tensors=tensors, dtype="float32", device="cuda:0")
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
    loaded = load_model(config=VumotarConfig.from_dict(raw), tensors=tensors, dtype="float32", device="cuda:0")
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
    tensors = random_weights(raw, 13, as_bfloat16=True)
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
