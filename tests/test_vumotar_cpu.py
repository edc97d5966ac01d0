"""Vumotar without a GPU: the plain implementation's mechanisms against restatements by hand, the configuration and the
loader, and the model through the step function, the cache manager, the scheduler and the entry point with the torch
test double in place of the CUDA kernel set."""

from __future__ import annotations

import itertools
import json
import math

import pytest
import torch

import plain_vumotar as pv
from vumotar_cases import (PAGE_TOKENS, _attention, _latent, _tempered, assert_rows_close, config, leaning_model, leaning_tokens,
                           plain_greedy, plain_logits, random_weights, relative_error, tokens_for)
from torch_ops import TorchOps

from mini_gpt_inference_b200 import EngineConfig, LLMEngine, SamplingParams, VumotarConfig
from mini_gpt_inference_b200.cache.manager import NO_PAGE, CacheManager
from mini_gpt_inference_b200.cache.spec import PagedKVSpec
from mini_gpt_inference_b200.config import ConfigError, lookup
from mini_gpt_inference_b200.engine.build import load_model, make_runner
from mini_gpt_inference_b200.engine.runner import StepEntry
from mini_gpt_inference_b200.parts import DecoderModel
from mini_gpt_inference_b200.parts.base import FEED_FORWARDS, MIXERS
from mini_gpt_inference_b200.parts.spec import PartSpec
from mini_gpt_inference_b200.weights import WeightsError, check_and_bind, load_file, write_random_model

F64 = torch.float64


def _rand(shapes, seed):
    gen = torch.Generator().manual_seed(seed)
    return {k: torch.randn(*s, generator=gen, dtype=F64) for k, s in shapes.items()}


def _unit(x, eps):
    return x / math.sqrt(float((x * x).mean()) + eps)


# ---- the plain mechanisms against restatements by hand ---------------------------------------------------
def test_attention_window_kept_tokens_and_the_term_of_one_by_hand():
    T, c, H, G, d, dv, eps = 11, 10, 4, 2, 6, 3, 1e-3
    for size, keep in ((4, 2), (1, 3), (3, 0), (20, 2)):
        m = {"heads": H, "kv_heads": G, "dim": d, "vdim": dv, "scale": 0.3, "mask": {"size": size, "keep_first": keep}}
        w = _rand({"q": (H * d, c), "k": (G * d, c), "v": (G * dv, c), "q.norm": (d,), "k.norm": (d,), "o": (c, H * dv)}, 2)
        h = _rand({"h": (T, c)}, 3)["h"]
        rows = []
        for i in range(T):
            seen = [j for j in range(i + 1) if j > i - size or j < keep]
            heads = []
            for a in range(H):
                q = _unit((w["q"] @ h[i])[a * d: (a + 1) * d], eps) * w["q.norm"]
                g = a // 2
                e = [math.exp(0.3 * float(q @ (_unit((w["k"] @ h[j])[g * d: (g + 1) * d], eps) * w["k.norm"]))) for j in seen]
                v = [(w["v"] @ h[j])[g * dv: (g + 1) * dv] for j in seen]
                heads.append(sum(x * y for x, y in zip(e, v)) / (1.0 + sum(e)))
            rows.append(w["o"] @ torch.cat(heads))
        assert torch.allclose(pv.attention_mixer(h, w, "", m, eps), torch.stack(rows), atol=1e-10), (size, keep)


def test_tempered_attention_by_hand():
    T, c, H, G, d, dv = 9, 7, 2, 1, 4, 5
    w = _rand({"q": (H * d, c), "k": (G * d, c), "v": (G * dv, c), "o": (c, H * dv)}, 4)
    h = _rand({"h": (T, c)}, 5)["h"]
    for coef, every in ((0.5, 3), (0.2, 1), (-0.3, 100)):
        m = {"heads": H, "kv_heads": G, "dim": d, "vdim": dv, "scale": 0.4, "q_temp": {"coef": coef, "every": every}}
        rows = []
        for i in range(T):
            grown = 1.0 + coef * math.log((i + 1) // every + 1)
            heads = []
            for a in range(H):
                q = grown * (w["q"] @ h[i])[a * d: (a + 1) * d]
                e = [math.exp(0.4 * float(q @ (w["k"] @ h[j]))) for j in range(i + 1)]
                heads.append(sum(x * (w["v"] @ h[j]) for j, x in enumerate(e)) / sum(e))
            rows.append(w["o"] @ torch.cat(heads))
        assert torch.allclose(pv.tempered_attention_mixer(h, w, "", m, 1e-3), torch.stack(rows), atol=1e-10)
    # the first step lies at position every - 1
    assert pv.temperature(6, 1.0, 3).tolist() == pytest.approx([1.0, 1.0, 1 + math.log(2), 1 + math.log(2), 1 + math.log(2), 1 + math.log(3)])


def test_attention_over_latents_by_hand():
    T, c, H, d, dv, qr, kr, size, eps = 9, 10, 2, 4, 3, 6, 5, 4, 1e-3
    m = {"heads": H, "dim": d, "vdim": dv, "q_rank": qr, "kv_rank": kr, "scale": 0.3, "mask": {"size": size}}
    w = _rand({"dq": (qr, c), "dq.norm": (qr,), "uq": (H * d, qr), "dkv": (kr, c), "dkv.norm": (kr,), "uk": (H * d, kr),
               "uv": (H * dv, kr), "sink": (H,), "g": (H, c), "o": (c, H * dv)}, 6)
    h = _rand({"h": (T, c)}, 7)["h"]
    lat = [_unit(w["dkv"] @ h[j], eps) * w["dkv.norm"] for j in range(T)]
    rows = []
    for i in range(T):
        q = w["uq"] @ (_unit(w["dq"] @ h[i], eps) * w["dq.norm"])
        heads = []
        for a in range(H):
            seen = range(max(0, i - size + 1), i + 1)                        # itself and size - 1 before it
            e = [math.exp(0.3 * float(q[a * d: (a + 1) * d] @ (w["uk"] @ lat[j])[a * d: (a + 1) * d])) for j in seen]
            v = [(w["uv"] @ lat[j])[a * dv: (a + 1) * dv] for j in seen]
            o = sum(x * y for x, y in zip(e, v)) / (math.exp(float(w["sink"][a])) + sum(e))
            heads.append(o / (1.0 + math.exp(-float(w["g"][a] @ h[i]))))
        rows.append(w["o"] @ torch.cat(heads))
    assert torch.allclose(pv.latent_attention_mixer(h, w, "", m, eps), torch.stack(rows), atol=1e-10)


def test_experts_read_the_token_times_their_own_score():
    c, f = 6, {"kind": "moe", "expert": {"ff": 5}, "router": {"experts": 4, "top": 2}, "shared": {"ff": 3}}
    w = {"router": (4, c), "shared.gate": (3, c), "shared.up": (3, c), "shared.down": (c, 3)}
    for e in range(4):
        w.update({f"e{e}.gate": (5, c), f"e{e}.up": (5, c), f"e{e}.down": (c, 5)})
    w = _rand(w, 5)
    h = _rand({"h": (3, c)}, 6)["h"]

    def unit(u, p):
        a = w[p + "gate"] @ u
        return w[p + "down"] @ (a * torch.sigmoid(a) * (w[p + "up"] @ u))
    for t, got in enumerate(pv.routed_experts(h, w, "", f)):
        s = [1 / (1 + math.exp(-float(z))) for z in w["router"] @ h[t]]
        chosen = sorted(range(4), key=lambda e: -s[e])[:2]
        want = sum(unit(s[e] * h[t], f"e{e}.") for e in chosen) + unit(h[t], "shared.")
        assert torch.allclose(got, want, atol=1e-12)
        outside = sum(s[e] * unit(h[t], f"e{e}.") for e in chosen) + unit(h[t], "shared.")
        assert not torch.allclose(got, outside, atol=1e-3)                   # the place of the weight matters


def test_layers_loop_and_head_by_hand():
    raw = {"architecture": "Vumotar", "vocab": 11, "width": 8, "norm": {"eps": 1e-3}, "loop": {"start": 1, "stop": 3, "times": 2},
           "layers": [{**_attention(1, 1, 4, 2, 3, 1), "mlp": None},
                      {**_tempered(1, 1, 2, 2, 0.5, 2), "mlp": {"kind": "moe", "expert": {"ff": 4}, "router": {"experts": 2, "top": 1}}},
                      {**_latent(1, 2, 2, 3, 4, 2), "mlp": None}]}
    w = random_weights(raw, 0, dtype=F64)
    toks = [3, 7, 3, 1]
    assert pv.run_order(raw) == [0, 1, 2, 1, 2]
    logits, after = pv.forward(raw, w, toks, return_layers=True)
    x = w["embed"][torch.tensor(toks)]
    run = {0: pv.attention_mixer, 1: pv.tempered_attention_mixer, 2: pv.latent_attention_mixer}
    for n, i in enumerate([0, 1, 2, 1, 2]):
        p = f"l{i}."
        y = run[i](pv.rms_norm(x, w[p + "norm1"], 1e-3), w, p + "mix.", raw["layers"][i]["mixer"], 1e-3)
        x = x + y / torch.sqrt(y.pow(2).mean(-1, keepdim=True) + 1e-3) * w[p + "norm1b"]
        if i == 1:
            y = pv.routed_experts(pv.rms_norm(x, w[p + "norm2"], 1e-3), w, p + "mlp.", raw["layers"][i]["mlp"])
            x = x + y / torch.sqrt(y.pow(2).mean(-1, keepdim=True) + 1e-3) * w[p + "norm2b"]
        assert torch.allclose(after[n], x, atol=1e-12)
    assert torch.allclose(logits, (x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + 1e-3) * w["final.norm"]) @ w["embed"].T, atol=1e-12)


# ---- configuration, registry, names, loader ------------------------------------------------------------------
@pytest.mark.parametrize("which", "ABCDE")
def test_config_round_trip_and_names(which, tmp_path):
    raw = config(which)
    cfg = VumotarConfig.from_dict(raw)
    assert VumotarConfig.from_dict(json.loads(json.dumps(cfg.to_dict()))) == cfg
    assert cfg.to_dict() == raw
    assert cfg.run_order() == pv.run_order(raw)
    assert lookup("Vumotar").config_class is VumotarConfig
    model = DecoderModel(lookup(cfg.architecture).describe(cfg))
    tensors = random_weights(raw, 1)
    specs = model.tensor_specs()
    assert {k for k, v in specs.items() if not v.optional} == set(tensors)
    assert sum(v.numel() for v in tensors.values()) == cfg.num_parameters()
    bound = check_and_bind(tensors, specs)
    assert all(specs[k].fits(v.shape) for k, v in bound.items())
    assert len(model.cache_specs()) == len(cfg.run_order())                  # every run of a layer keeps its own
    for i, spec in zip(cfg.run_order(), model.cache_specs()):
        m, kind = raw["layers"][i]["mixer"], raw["layers"][i]["type"]
        mask = m.get("mask") or {}
        assert isinstance(spec, PagedKVSpec) and spec.window == mask.get("size") and spec.keep_first == mask.get("keep_first", 0)
        if kind == "latent_attention":                                       # one row a token, whatever the number of heads
            assert (spec.n_kv_head, spec.head_dim) == (1, m["kv_rank"]) and spec.values_in_keys
        else:
            assert (spec.n_kv_head, spec.head_dim, spec.value_dim) == (m["kv_heads"], m["dim"], m["vdim"])
    folder = write_random_model(tmp_path / which, cfg, 3, "bfloat16")
    assert {k for k in load_file(folder / "model.safetensors")} >= set(tensors)
    assert VumotarConfig.from_json(folder) == cfg


def test_config_errors_and_loader_errors():
    raw = config("A")
    for breaker in (lambda r: r.pop("width"), lambda r: r.pop("norm"), lambda r: r["norm"].update(eps=0),
                    lambda r: r["layers"][0].update(type="conv"), lambda r: r["layers"][0]["mixer"].pop("scale"),
                    lambda r: r["layers"][0]["mixer"].pop("q_rank"), lambda r: r["layers"][0]["mixer"]["mask"].update(size=0),
                    lambda r: r["layers"][1]["mixer"].update(kv_heads=4), lambda r: r["layers"][1]["mixer"]["mask"].update(keep_first=-1),
                    lambda r: r["layers"][1]["mixer"]["mask"].pop("size"), lambda r: r["layers"][2]["mixer"]["q_temp"].update(every=0),
                    lambda r: r["layers"][2]["mixer"]["q_temp"].pop("coef"),
                    lambda r: r["layers"][0]["mlp"]["router"].update(top=7), lambda r: r["layers"][0]["mlp"].update(kind="dense"),
                    lambda r: r["layers"][0]["mlp"]["shared"].update(ff=0), lambda r: r["loop"].update(stop=9),
                    lambda r: r["loop"].update(times=0)):
        broken = json.loads(json.dumps(raw))
        breaker(broken)
        with pytest.raises(ConfigError):
            VumotarConfig.from_dict(broken)
    tensors = random_weights(raw, 2)
    del tensors["l0.mix.sink"]
    tensors["l2.mlp.shared.up"] = tensors["l2.mlp.shared.up"][:8]
    tensors["l1.mix.q.norm"] = tensors["l1.mix.q.norm"][:1]
    with pytest.raises(WeightsError) as err:
        load_model(config=VumotarConfig.from_dict(raw), tensors=tensors, dtype="float32", device="cpu")
    assert all(name in str(err.value) for name in ("l0.mix.sink", "l2.mlp.shared.up", "l1.mix.q.norm"))


def test_parts_refuse_what_they_do_not_combine():
    base = {"width": 16, "n_head": 2, "head_dim": 8, "eps": 1e-5}
    for bad in ({"keep_first": 2}, {"keep_first": -1, "window": 4}, {"sink": True, "unit_sink": True}, {"query_temperature": (0.1, 0)},
                {"query_temperature": (0.1, 4), "rot_dims": 4, "unit_norm": False}):
        with pytest.raises(ValueError):
            MIXERS.build(PartSpec("gated_unit_attention", {**base, **bad}, "mix"), "l0.")
    latent = {**base, "v_head_dim": 8, "kv_rank": 8, "scale": 1.0}
    for bad in ({"q_rank": 4, "rot_dim": 2}, {"rot_dim": 0, "gate": "token"}, {"rot_dim": 0, "q_rank": 4, "own_latents": False}):
        with pytest.raises(ValueError):
            MIXERS.build(PartSpec("latent_attention", {**latent, **bad}, "mix"), "l0.")
    experts = {"width": 16, "n_experts": 3, "top": 2, "inner": 24}
    for bad in ({"weigh": "both"}, {"weigh": "input", "shared_inner": 8, "shared_gate": True}):
        with pytest.raises(ValueError):
            FEED_FORWARDS.build(PartSpec("routed_experts", {**experts, **bad}, "mlp"), "l0.")


def test_a_gated_shared_expert_as_experts_that_every_token_uses():
    """Its hidden features in parts as large as an expert's, the last part filled up with zeros."""
    for shared, parts in ((24, 1), (10, 1), (25, 2), (72, 3)):
        part = FEED_FORWARDS.build(PartSpec("routed_experts", {
            "width": 16, "n_experts": 3, "top": 2, "inner": 24, "shared_inner": shared, "shared_gate": False, "scoring": "sigmoid",
            "weigh": "input"}, "mlp"), "l0.")
        assert part.always == parts and part.returns_output
        gen = torch.Generator().manual_seed(shared)
        tensors = {k: torch.randn(*s.shape, generator=gen, dtype=F64) for k, s in part.tensor_specs().items()}
        part.bind(tensors)
        assert part.w_in.shape == (3 + parts, 48, 16) and part.w_out.shape == (3 + parts, 16, 24)
        h = torch.randn(1, 16, generator=gen, dtype=F64)

        def unit(e):
            a = part.w_in[e] @ h[0]
            return part.w_out[e] @ (a[:24] * torch.sigmoid(a[:24]) * a[24:])
        assert torch.allclose(sum(unit(e) for e in range(3, 3 + parts)), pv.gated_unit(h, tensors, "l0.mlp.shared.")[0], atol=1e-9)


# ---- pages of kept first tokens ---------------------------------------------------------------------------------
def test_a_window_keeps_the_pages_of_first_tokens():
    specs = [PagedKVSpec(2, 8, window=10, keep_first=5), PagedKVSpec(2, 8, window=10), PagedKVSpec(2, 8)]
    m = CacheManager(specs, page_tokens=4, num_pages=40, max_requests=2, window_slack_tokens=6)
    assert len(m.groups) == 3
    m.admit("a")
    for length in range(1, 60):
        assert m.reserve("a", length)
        m.advance("a", length)
        m.check()
        first = max(0, length - 9) // 4                                     # the page of the first key a later query reads
        for g, kept in ((0, 2), (1, 0), (2, 99)):
            table = m.block_table("a", g)
            for i, page in enumerate(table):
                assert (page == NO_PAGE) == (kept <= i < first and g != 2), (length, g, i)
    assert sum(p != NO_PAGE for p in m.block_table("a", 0)) == sum(p != NO_PAGE for p in m.block_table("a", 1)) + 2
    assert m.groups[0].num_pages == 2 * ((10 + 6 + 3) // 4 + 2 + 2)         # the pool has room for them
    assert m.stats()["internal_fragmentation_slots"] >= 0
    m.release("a")
    assert m.stats()["allocated_blocks"] == 0
    m.check()
    # (a window group of 6 pages: the window and one step's tokens fit, the kept pages as well or not)
    for keep, fits in ((0, True), (8, False)):
        tight = CacheManager([PagedKVSpec(1, 8, window=8, keep_first=keep, num_pages=6)], page_tokens=4, num_pages=40,
                             max_requests=1, window_slack_tokens=4)
        assert tight.can_ever_hold(100) is fits
    for bad in ({"keep_first": 3}, {"window": 4, "keep_first": -1}):
        with pytest.raises(ValueError):
            PagedKVSpec(1, 8, **bad)


# ---- the model through the step function on the test double ----------------------------------------------------
def cpu_runner(raw, tensors, page_tokens, num_pages, max_requests=4):
    loaded = load_model(config=VumotarConfig.from_dict(raw), tensors=tensors, dtype="float32", device="cpu")
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
        assert_rows_close(torch.cat(got[k]), want[k], 5e-4, f"request {k}")
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
        assert_rows_close(torch.cat([first] + rest), want, 5e-4, name)
        if n % 2 == 0:
            runner.finish(name)
        else:                                                           # two live at once, the older one ends later
            other = tokens_for(raw, 5, 90 + n)
            got = runner.step([StepEntry(name + "x", other, [4])])
            assert_rows_close(got, plain_logits(raw, tensors, other, [4]), 5e-4, name + "x")
            runner.finish(name)
            runner.finish(name + "x")
        runner.manager.check()


def test_a_windows_pages_are_given_back_while_the_request_lives():
    raw = {**config("A"), "layers": [config("A")["layers"][1]]}          # a window of 19 and 3 kept tokens over pages of 8
    del raw["loop"]
    tensors = random_weights(raw, 6)
    runner = cpu_runner(raw, tensors, 8, 8)
    toks = tokens_for(raw, 64, 1)
    want = plain_logits(raw, tensors, toks)
    outs = [runner.step([StepEntry("r", toks[:20], list(range(20)))])]
    held = []
    for t in range(20, 64):
        outs.append(runner.step([StepEntry("r", toks[t: t + 1], [0])]))
        held.append(runner.manager.stats()["allocated_blocks"])
    assert max(held) <= 1 + 4
    assert_rows_close(torch.cat(outs), want, 5e-4, "windowed")


LEANING = {"attention": _attention(4, 2, 32, 24, 16, 3, 0.2), "attention_2": _tempered(4, 2, 32, 24, 0.4, 16, 0.2),
           "latent_attention": _latent(2, 32, 24, 24, 40, 16, 0.2)}


@pytest.mark.parametrize("kind", sorted(LEANING))
def test_the_leaning_model_shows_a_single_key(kind):
    """(What the GPU tests of the edges rest on.)  A key that the last query sees decides the row, one just outside its
    sight does not touch it."""
    raw, w = leaning_model(LEANING[kind])
    length = 60
    for at in (0, 2, 3, 4, 20, length - 18, length - 17, length - 16, length - 2):
        back = length - 1 - at
        seen = kind == "attention_2" or back < 16 or (kind == "attention" and at < 3)
        with_key, without = (plain_logits(raw, w, leaning_tokens(raw, length, 3, at, answer), [length - 1]) for answer in (True, False))
        moved = float(relative_error(without, with_key))
        assert moved > 0.3 if seen else moved == 0.0, (at, moved)


def test_generation_through_the_engine_on_the_double():
    raw = config("A")
    tensors = random_weights(raw, 4)
    loaded = load_model(config=VumotarConfig.from_dict(raw), tensors=tensors, dtype="float32", device="cpu")
    engine = LLMEngine(loaded, EngineConfig(dtype="float32", device="cpu", block_size=8, num_blocks=12, max_batch_size=2,
                                            max_num_batched_tokens=12, max_prefill_chunk=5), ops=TorchOps())
    prompts = [tokens_for(raw, n, 30 + n) for n in (7, 1, 18)]
    outs = engine.generate(prompts, SamplingParams(max_tokens=6, temperature=0.0))
    for prompt, out in zip(prompts, outs):
        assert out["token_ids"] == plain_greedy(raw, tensors, prompt, 6)
    assert engine.stats()["allocated_blocks"] == 0
