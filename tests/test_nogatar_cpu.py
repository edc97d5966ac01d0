"""Nogatar without a GPU: the plain implementation's mechanisms against restatements by hand, the configuration and the
loader, and the model through the step function, the cache manager, the scheduler and the entry point with the torch
test double in place of the CUDA kernel set."""

from __future__ import annotations

import itertools
import json
import math

import pytest
import torch

import plain_nogatar as pn
from nogatar_cases import (PAGE_TOKENS, assert_rows_close, config, leaning_model, leaning_tokens, plain_greedy, plain_logits, random_weights,
                           relative_error, tokens_for)
from torch_ops import TorchOps

from mini_gpt_inference_b200 import EngineConfig, LLMEngine, NogatarConfig, SamplingParams
from mini_gpt_inference_b200.cache.spec import FixedStateSpec, PagedKVSpec
from mini_gpt_inference_b200.config import ConfigError, lookup
from mini_gpt_inference_b200.engine.build import load_model, make_runner
from mini_gpt_inference_b200.engine.runner import StepEntry
from mini_gpt_inference_b200.parts import DecoderModel
from mini_gpt_inference_b200.parts.base import FEED_FORWARDS
from mini_gpt_inference_b200.parts.rotary import rotary_frequencies
from mini_gpt_inference_b200.parts.spec import PartSpec
from mini_gpt_inference_b200.weights import WeightsError, check_and_bind, load_file, write_random_model

F64 = torch.float64


def _rand(shapes, seed):
    gen = torch.Generator().manual_seed(seed)
    return {k: torch.randn(*s, generator=gen, dtype=F64) for k, s in shapes.items()}


def _unit(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


# ---- the plain mechanisms against restatements by hand ---------------------------------------------------
def test_matrix_memory_is_a_gated_sum_over_the_past():
    """Without the running maximum: the weight of token j in the read at t is exp(i_j + f_(j+1) + .. + f_t); the
    denominator is the larger of the same sum of q . k and 1 (what exp(-m) is before both are scaled by exp(-m))."""
    T, c, H, d, dv, cap, eps = 8, 9, 2, 4, 3, 3.0, 1e-4
    shapes = {"q": (H * d, c), "k": (H * d, c), "v": (H * dv, c), "g": (H * dv, c), "o": (c, H * dv), "norm": (H * dv,),
              "i": (H, c), "i.b": (H,), "f": (H, c), "f.b": (H,)}
    w = _rand(shapes, 0)
    h = _rand({"h": (T, c)}, 1)["h"]
    got = pn.mlstm_mixer(h, w, "", {"heads": H, "dim": d, "vdim": dv, "gate_cap": cap}, eps)
    q, k, v = (h @ w["q"].T).view(T, H, d) / 2.0, (h @ w["k"].T).view(T, H, d), (h @ w["v"].T).view(T, H, dv)
    i = cap * torch.tanh((h @ w["i"].T + w["i.b"]) / cap)
    z = cap * torch.tanh((h @ w["f"].T + w["f.b"]) / cap)
    f = -torch.log1p(torch.exp(-z))
    o = torch.zeros(T, H, dv, dtype=F64)
    for a in range(H):
        m = 0.0
        for t in range(T):
            m = max(float(f[t, a]) + m, float(i[t, a]))
            num, den = torch.zeros(dv, dtype=F64), 0.0
            for j in range(t + 1):
                share = math.exp(float(i[j, a] + f[j + 1: t + 1, a].sum()))
                num, den = num + share * (q[t, a] @ k[j, a]) * v[j, a], den + share * float(q[t, a] @ k[j, a])
            o[t, a] = num / (max(abs(den), 1.0) + 1e-6 * math.exp(m))
    g = h @ w["g"].T
    want = (_unit(o, eps).reshape(T, -1) * w["norm"] / (1 + torch.exp(-g))) @ w["o"].T
    assert torch.allclose(got, want, atol=1e-9)


def test_stretched_frequencies_by_hand_and_as_the_engine_works_them_out():
    # 8 pairs, base 100: turns over `original` positions fall from pair to pair
    scaling = {"factor": 4.0, "original": 300, "fast": 20.0, "slow": 2.0}
    freq, mag = pn.stretched_frequencies(16, 100.0, scaling)
    assert mag == pytest.approx(0.1 * math.log(4.0) + 1.0)
    plain = [100.0 ** (-i / 8) for i in range(8)]
    turns = [300 * f / (2 * math.pi) for f in plain]
    assert turns[0] > 20 > turns[7] and turns[7] < 2
    fast_pair = 16 * math.log(300 / (2 * math.pi * 20)) / (2 * math.log(100.0))
    slow_pair = 16 * math.log(300 / (2 * math.pi * 2)) / (2 * math.log(100.0))
    lo, hi = math.floor(fast_pair), math.ceil(slow_pair)
    assert 0 < lo < hi < 15
    for i in range(8):
        if i <= lo:
            assert freq[i] == pytest.approx(plain[i])
        elif i >= hi:
            assert freq[i] == pytest.approx(plain[i] / 4)
        else:
            share = (i - lo) / (hi - lo)
            assert freq[i] == pytest.approx(plain[i] * (1 - share) + plain[i] / 4 * share)
    for n, base, s in ((16, 100.0, scaling), (8, 1e6, {"factor": 8.0, "original": 20, "fast": 16.0, "slow": 0.5}),
                       (2, 50.0, {"factor": 3.0, "original": 30, "fast": 4.0, "slow": 1.0}), (12, 1e4, None),
                       (64, 1e4, {"factor": 1.0, "original": 4096, "fast": 32.0, "slow": 1.0})):
        want, got = pn.stretched_frequencies(n, base, s), rotary_frequencies(n, base, s)
        assert got[0] == pytest.approx(want[0], rel=1e-12) and got[1] == pytest.approx(want[1])
    assert rotary_frequencies(12, 1e4)[1] == 1.0


def test_neighbouring_features_turn_together():
    x = torch.tensor([[[1.0, 0.0, 0.0, 2.0]]], dtype=F64)
    got = pn.rotate_pairs(x, torch.tensor([3]), [0.5, 0.1], 1.25)
    want = [1.25 * math.cos(1.5), 1.25 * math.sin(1.5), -1.25 * 2 * math.sin(0.3), 1.25 * 2 * math.cos(0.3)]
    assert torch.allclose(got.flatten(), torch.tensor(want, dtype=F64), atol=1e-12)


def test_attention_over_latents_window_and_sink_by_hand():
    T, c, H, d, r, dv, rank, size, eps = 9, 10, 2, 4, 2, 3, 5, 4, 1e-3
    m = {"heads": H, "dim": d, "rot_dim": r, "vdim": dv, "kv_rank": rank, "scale": 0.3, "mask": {"size": size},
         "rot": {"base": 30.0, "dims": r, "scaling": {"factor": 2.0, "original": 10, "fast": 3.0, "slow": 1.0}}}
    w = _rand({"q": (H * (d + r), c), "dkv": (rank + r, c), "dkv.norm": (rank,), "uk": (H * d, rank), "uv": (H * dv, rank),
               "sink": (H,), "o": (c, H * dv)}, 2)
    h = _rand({"h": (T, c)}, 3)["h"]
    got = pn.latent_attention_mixer(h, w, "", m, eps)
    freq, mag = pn.stretched_frequencies(r, 30.0, m["rot"]["scaling"])
    low = h @ w["dkv"].T
    lat = _unit(low[:, :rank], eps) * w["dkv.norm"]
    rows = []
    for i in range(T):
        heads = []
        for a in range(H):
            q = (h[i] @ w["q"].T).view(H, d + r)[a]
            qr = pn.rotate_pairs(q[None, None, d:], torch.tensor([i]), freq, mag)[0, 0]
            scores, values = [], []
            for j in range(max(0, i - size + 1), i + 1):                   # itself and size - 1 before it
                kr = pn.rotate_pairs(low[None, j: j + 1, rank:], torch.tensor([j]), freq, mag)[0, 0]
                scores.append(0.3 * (q[:d] @ (w["uk"].view(H, d, rank)[a] @ lat[j]) + qr @ kr))
                values.append(w["uv"].view(H, dv, rank)[a] @ lat[j])
            e = torch.exp(torch.stack(scores))
            heads.append((e / (e.sum() + torch.exp(w["sink"][a]))) @ torch.stack(values))
        rows.append(torch.cat(heads) @ w["o"].T)
    assert torch.allclose(got, torch.stack(rows), atol=1e-10)
    # the rotated scores depend on the distance alone
    q, k = _rand({"q": (1, 1, 4), "k": (1, 1, 4)}, 4).values()
    dots = [(pn.rotate_pairs(q, torch.tensor([p]), [0.7, 0.2], 1.0) * pn.rotate_pairs(k, torch.tensor([p - 3]), [0.7, 0.2], 1.0)).sum()
            for p in (3, 10, 400)]
    assert torch.allclose(dots[0], dots[1]) and torch.allclose(dots[0], dots[2])


def test_experts_scores_over_all_divided_by_the_chosen_ones_sum():
    c, f = 6, {"kind": "moe", "expert": {"ff": 5}, "router": {"experts": 4, "top": 2}, "shared": {"ff": 3}}
    w = {"router": (4, c), "shared.up": (3, c), "shared.down": (c, 3), "shared.sg": (1, c)}
    for e in range(4):
        w.update({f"e{e}.up": (5, c), f"e{e}.down": (c, 5)})
    w = _rand(w, 5)
    h = _rand({"h": (3, c)}, 6)["h"]
    got = pn.routed_experts(h, w, "", f)
    for t in range(3):
        z = w["router"] @ h[t]
        s = torch.exp(z) / torch.exp(z).sum()
        chosen = sorted(range(4), key=lambda e: -float(s[e]))[:2]
        want = torch.zeros(c, dtype=F64)
        for e in chosen:
            u = w[f"e{e}.up"] @ h[t]
            want += s[e] / (s[chosen[0]] + s[chosen[1]]) * (w[f"e{e}.down"] @ torch.where(u > 0, u * u, 0 * u))
        u = w["shared.up"] @ h[t]
        want += (w["shared.down"] @ torch.where(u > 0, u * u, 0 * u)) / (1 + torch.exp(-(w["shared.sg"] @ h[t])))
        assert torch.allclose(got[t], want, atol=1e-12)


def test_a_layer_by_hand_norms_behind_the_sublayers_only():
    raw = {"architecture": "Nogatar", "vocab": 11, "width": 8, "norm": {"eps": 1e-3}, "embedding": {"scale": 3.0},
           "residual_mult": 0.4, "layers": [{"type": "mlstm", "mixer": {"heads": 1, "dim": 2, "vdim": 2, "gate_cap": 4.0},
                                             "mlp": {"kind": "moe", "expert": {"ff": 4}, "router": {"experts": 2, "top": 1}}}]}
    w = random_weights(raw, 0, dtype=F64)
    toks = [3, 7, 3]
    logits, after = pn.forward(raw, w, toks, return_layers=True)
    x = 3.0 * w["embed"][torch.tensor(toks)]
    for sub, norm in ((lambda h: pn.mlstm_mixer(h, w, "l0.mix.", raw["layers"][0]["mixer"], 1e-3), "l0.norm1"),
                      (lambda h: pn.routed_experts(h, w, "l0.mlp.", raw["layers"][0]["mlp"]), "l0.norm2")):
        y = sub(x)
        d = y - y.mean(-1, keepdim=True)
        x = x + 0.4 * d / torch.sqrt(d.pow(2).mean(-1, keepdim=True) + 1e-3) * w[norm]
    assert torch.allclose(after[0], x, atol=1e-12)
    d = x - x.mean(-1, keepdim=True)
    assert torch.allclose(logits, (d / torch.sqrt(d.pow(2).mean(-1, keepdim=True) + 1e-3) * w["final.norm"]) @ w["head"].T, atol=1e-12)
    capped = pn.forward({**raw, "logit_softcap": 2.0}, w, toks)
    assert torch.allclose(capped, 2.0 * torch.tanh(logits / 2.0), atol=1e-12) and float(capped.abs().max()) < 2.0


# ---- configuration, registry, names, loader ------------------------------------------------------------------
@pytest.mark.parametrize("which", "ABCDE")
def test_config_round_trip_and_names(which, tmp_path):
    raw = config(which)
    cfg = NogatarConfig.from_dict(raw)
    assert NogatarConfig.from_dict(json.loads(json.dumps(cfg.to_dict()))) == cfg
    assert cfg.to_dict() == {**raw, "layers": [{**layer, "mlp": layer["mlp"]} for layer in raw["layers"]]}
    assert lookup("Nogatar").config_class is NogatarConfig
    model = DecoderModel(lookup(cfg.architecture).describe(cfg))
    tensors = random_weights(raw, 1)
    specs = model.tensor_specs()
    assert {k for k, v in specs.items() if not v.optional} == set(tensors)
    assert sum(v.numel() for v in tensors.values()) == cfg.num_parameters()
    bound = check_and_bind(tensors, specs)
    assert all(specs[k].fits(v.shape) for k, v in bound.items())
    for layer, spec in zip(raw["layers"], model.cache_specs()):
        m = layer["mixer"]
        if layer["type"] == "mlstm":
            assert isinstance(spec, FixedStateSpec) and spec.dtype == "float32"
            assert spec.shape == (m["heads"] * (m["dim"] * (m["vdim"] + 1) + 1),)
        else:                                                    # one row a token, whatever the number of heads
            assert isinstance(spec, PagedKVSpec) and (spec.n_kv_head, spec.head_dim) == (1, m["kv_rank"] + m["rot_dim"])
            assert spec.values_in_keys and spec.window == (m.get("mask") or {}).get("size")
    folder = write_random_model(tmp_path / which, cfg, 3, "bfloat16")
    assert {k for k in load_file(folder / "model.safetensors")} >= set(tensors)
    assert NogatarConfig.from_json(folder) == cfg


def test_config_errors_and_loader_errors():
    raw = config("A")
    for breaker in (lambda r: r.pop("width"), lambda r: r.pop("residual_mult"), lambda r: r.pop("embedding"),
                    lambda r: r["layers"][0].update(type="conv"), lambda r: r["layers"][0]["mixer"].pop("scale"),
                    lambda r: r["layers"][0]["mixer"].update(rot_dim=7),
                    lambda r: r["layers"][0]["mixer"]["rot"].update(dims=6),
                    lambda r: r["layers"][0]["mixer"]["rot"]["scaling"].pop("slow"),
                    lambda r: r["layers"][0]["mixer"]["rot"]["scaling"].update(factor=0),
                    lambda r: r["layers"][0]["mixer"]["mask"].update(size=0),
                    lambda r: r["layers"][1]["mixer"].update(gate_cap=0.0),
                    lambda r: r["layers"][1]["mixer"].pop("vdim"),
                    lambda r: r["layers"][0]["mlp"]["router"].update(top=7),
                    lambda r: r["layers"][0]["mlp"].update(kind="dense"),
                    lambda r: r["layers"][0]["mlp"]["shared"].update(ff=0),
                    lambda r: r.update(logit_softcap=0.0), lambda r: r["norm"].update(eps=0)):
        broken = json.loads(json.dumps(raw))
        breaker(broken)
        with pytest.raises(ConfigError):
            NogatarConfig.from_dict(broken)
    cfg = NogatarConfig.from_dict(raw)
    tensors = random_weights(raw, 2)
    del tensors["l0.mix.sink"]
    tensors["l2.mlp.shared.up"] = tensors["l2.mlp.shared.up"][:8]
    tensors["l1.mix.i.b"] = tensors["l1.mix.i.b"][:1]
    with pytest.raises(WeightsError) as err:
        load_model(config=cfg, tensors=tensors, dtype="float32", device="cpu")
    assert all(name in str(err.value) for name in ("l0.mix.sink", "l2.mlp.shared.up", "l1.mix.i.b"))


def test_a_plain_shared_expert_as_experts_that_every_token_uses():
    """Its hidden features in parts as large as an expert's, the last part filled up with zeros."""
    for shared, parts in ((24, 1), (10, 1), (25, 2), (72, 3)):
        part = FEED_FORWARDS.build(PartSpec("routed_experts", {
            "width": 16, "n_experts": 3, "top": 2, "inner": 24, "shared_inner": shared, "activation": "relu_sq", "gated": False}, "mlp"), "l0.")
        assert part.always == parts
        gen = torch.Generator().manual_seed(shared)
        tensors = {k: torch.randn(*s.shape, generator=gen) for k, s in part.tensor_specs().items()}
        part.bind(tensors)
        assert part.w_in.shape == (3 + parts, 24, 16) and part.w_out.shape == (3 + parts, 16, 24)
        h = torch.randn(16, generator=gen)
        want = tensors["l0.mlp.shared.down"] @ (tensors["l0.mlp.shared.up"] @ h).clamp(min=0) ** 2
        got = sum(part.w_out[e] @ (part.w_in[e] @ h).clamp(min=0) ** 2 for e in range(3, 3 + parts))
        assert torch.allclose(got, want, atol=1e-3, rtol=1e-5)
    for bad in ({"gated": False, "activation": "clamped_swish"}, {"gated": True, "activation": "relu_sq"},
                {"gated": False, "activation": "relu_sq", "scoring": "sigmoid"}):
        with pytest.raises(ValueError):
            FEED_FORWARDS.build(PartSpec("routed_experts", {"width": 16, "n_experts": 3, "top": 2, "inner": 24, **bad}, "mlp"), "l0.")


# ---- the model through the step function on the test double ----------------------------------------------------
def cpu_runner(raw, tensors, page_tokens, num_pages, max_requests=4):
    loaded = load_model(config=NogatarConfig.from_dict(raw), tensors=tensors, dtype="float32", device="cpu")
    return make_runner(loaded, TorchOps(), page_tokens, num_pages, max_requests)


@pytest.mark.parametrize("which", "ABCE")
def test_cuttings_agree_with_plain(which):
    raw = config(which)
    tensors = random_weights(raw, 3, sharp=3.0)
    pt = PAGE_TOKENS[which]
    lengths = {"a": 41, "b": 36, "c": 9, "d": 2 * pt + 1}
    runner = cpu_runner(raw, tensors, pt, sum(-(-n // pt) for n in lengths.values()))
    reqs = {k: tokens_for(raw, n, i) for i, (k, n) in enumerate(lengths.items())}
    want = {k: plain_logits(raw, tensors, v) for k, v in reqs.items()}
    got = {k: [] for k in reqs}
    pos = dict.fromkeys(reqs, 0)
    sizes = itertools.cycle([13, 1, 2, 7, 1, 1, 5, 2])
    while any(pos[k] < len(reqs[k]) for k in reqs):
        entries, order = [], []
        for k in reqs:
            if pos[k] == len(reqs[k]):
                continue
            m = min(next(sizes), len(reqs[k]) - pos[k])
            entries.append(StepEntry(k, reqs[k][pos[k]: pos[k] + m], list(range(m))))
            order.append((k, m))
            pos[k] += m
        out = runner.step(entries)
        row = 0
        for k, m in order:
            got[k].append(out[row: row + m])
            row += m
        runner.manager.check()
    for k in reqs:
        assert_rows_close(torch.cat(got[k]), want[k], 2e-4, f"request {k}")
        runner.finish(k)
    assert runner.manager.stats()["allocated_blocks"] == 0


def test_slots_and_pages_used_again():
    raw = config("A")
    tensors = random_weights(raw, 5)
    runner = cpu_runner(raw, tensors, 8, 6, max_requests=2)
    for n, name in enumerate(["p", "q", "r", "s", "t"]):                # five requests through two slots
        toks = tokens_for(raw, 17 + n, 40 + n)
        want = plain_logits(raw, tensors, toks)
        first = runner.step([StepEntry(name, toks[:9], list(range(9)))])
        rest = [runner.step([StepEntry(name, [t], [0])]) for t in toks[9:]]
        assert_rows_close(torch.cat([first] + rest), want, 2e-4, name)
        if n % 2 == 0:
            runner.finish(name)
        else:                                                           # two live at once, the older one ends later
            other = tokens_for(raw, 5, 90 + n)
            got = runner.step([StepEntry(name + "x", other, [4])])
            assert_rows_close(got, plain_logits(raw, tensors, other, [4]), 2e-4, name + "x")
            runner.finish(name)
            runner.finish(name + "x")
        runner.manager.check()


def test_a_windows_pages_are_given_back_while_the_request_lives():
    raw = {**config("A"), "layers": [config("A")["layers"][2]]}          # a window of 7 over pages of 8
    tensors = random_weights(raw, 6)
    runner = cpu_runner(raw, tensors, 8, 8)
    toks = tokens_for(raw, 60, 1)
    want = plain_logits(raw, tensors, toks)
    outs = [runner.step([StepEntry("r", toks[:20], list(range(20)))])]
    held = []
    for t in range(20, 60):
        outs.append(runner.step([StepEntry("r", toks[t: t + 1], [0])]))
        held.append(runner.manager.stats()["allocated_blocks"])
    assert max(held) <= 2
    assert_rows_close(torch.cat(outs), want, 2e-4, "windowed")


@pytest.mark.parametrize("window", [16, 19])
def test_the_leaning_model_shows_the_windows_edge(window):
    """(What the GPU tests of the edge rest on.)  The key one step inside the window decides the last row, the one just
    outside does not touch it; without the sink the row moves as well."""
    raw, w = leaning_model(window, 24)
    for back, matters in ((window - 1, True), (1, True), (window, False), (50, False)):
        with_key, without = (plain_logits(raw, w, leaning_tokens(raw, 60, 3, 59 - back, answer), [59]) for answer in (True, False))
        moved = float(relative_error(without, with_key))
        assert moved > 0.3 if matters else moved == 0.0, back
    toks = tokens_for(raw, 60, 3)
    # (the norm behind the layer takes a factor that all heads share away: a sink shows where heads differ)
    no_sink, one_sink = ({**w, "l0.mix.sink": torch.tensor([s, -80.0])} for s in (-80.0, 4.0))
    moved = relative_error(plain_logits(raw, no_sink, toks), plain_logits(raw, one_sink, toks))
    assert float(moved[0]) > 0.3 and float(moved.median()) > 0.3


def test_generation_through_the_engine_on_the_double():
    raw = config("A")
    tensors = random_weights(raw, 4)
    loaded = load_model(config=NogatarConfig.from_dict(raw), tensors=tensors, dtype="float32", device="cpu")
    engine = LLMEngine(loaded, EngineConfig(dtype="float32", device="cpu", block_size=8, num_blocks=12, max_batch_size=2,
                                            max_num_batched_tokens=12, max_prefill_chunk=5), ops=TorchOps())
    prompts = [tokens_for(raw, n, 30 + n) for n in (7, 1, 18)]
    outs = engine.generate(prompts, SamplingParams(max_tokens=6, temperature=0.0))
    for prompt, out in zip(prompts, outs):
        assert out["token_ids"] == plain_greedy(raw, tensors, prompt, 6)
    assert engine.stats()["allocated_blocks"] == 0


def test_layers_of_other_arrangements_between_post_norm_layers():
    """The copy of the stream that a post-norm layer leaves for the next one is not used once another kind of layer has
    changed the stream."""
    from mini_gpt_inference_b200.config.registry import MODEL_REGISTRY, ModelFamily
    from mini_gpt_inference_b200.models.nogatar import describe_nogatar
    from mini_gpt_inference_b200.parts.spec import LayerSpec
    from dataclasses import replace

    raw = {**config("E"), "layers": [config("E")["layers"][1]] * 3}
    cfg = NogatarConfig.from_dict(raw)
    spec = describe_nogatar(cfg)
    middle = spec.layers[1]
    mixed = replace(spec, layers=(spec.layers[0], LayerSpec(middle.prefix, middle.parts, "pre_norm_mixer_only"), spec.layers[2]))
    tensors = random_weights(raw, 9)
    toks = tokens_for(raw, 12, 2)
    name = "NogatarWithAPreNormLayer"
    MODEL_REGISTRY[name] = ModelFamily(name, NogatarConfig, lambda _: mixed)
    try:
        loaded = load_model(config=replace(cfg, architecture=name), tensors=tensors, dtype="float32", device="cpu")
        # (the double hands the stream itself on in 32-bit; a cast that copies makes a stale copy visible)
        ops = TorchOps()
        ops.cast = lambda x, dtype: x.to(dtype).clone()
        norm_add = ops.norm_add
        ops.norm_add = lambda *a, **k: (lambda rows: None if rows is None else rows.clone())(norm_add(*a, **k))
        got = make_runner(loaded, ops, 8, 8, 2).step([StepEntry("r", toks, list(range(12)))])
    finally:
        del MODEL_REGISTRY[name]
    w = {k: v.double() for k, v in tensors.items()}
    m, eps, x = raw["layers"][0]["mixer"], 1e-5, raw["embedding"]["scale"] * w["embed"][torch.tensor(toks)]
    for i in range(3):
        p = f"l{i}."
        if i == 1:
            x = x + pn.mlstm_mixer(pn.layer_norm(x, w[p + "norm1"], eps), w, p + "mix.", m, eps)
        else:
            x = x + 0.9 * pn.layer_norm(pn.mlstm_mixer(x, w, p + "mix.", m, eps), w[p + "norm1"], eps)
    want = 12.0 * torch.tanh((pn.layer_norm(x, w["final.norm"], eps) @ w["head"].T) / 12.0)
    assert_rows_close(got, want, 2e-4, "mixed arrangements")
