"""Small Vumotar configurations and random weights for the tests, made here (names and shapes written out from the
design, not taken from the engine's own list), and the plain logits."""

from __future__ import annotations

import math

import torch

import plain_vumotar


def _attention(heads, kv_heads, dim, vdim, window, keep, scale=None):
    mixer = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": dim ** -0.5 if scale is None else scale}
    if window is not None:
        mixer["mask"] = {"size": window, "keep_first": keep}
    return {"type": "attention", "mixer": mixer}


def _tempered(heads, kv_heads, dim, vdim, coef, every, scale=None):
    mixer = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": dim ** -0.5 if scale is None else scale}
    if coef is not None:
        mixer["q_temp"] = {"coef": coef, "every": every}
    return {"type": "attention_2", "mixer": mixer}


def _latent(heads, dim, vdim, q_rank, kv_rank, window, scale=None):
    mixer = {"heads": heads, "dim": dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
             "scale": dim ** -0.5 if scale is None else scale}
    if window is not None:
        mixer["mask"] = {"size": window}
    return {"type": "latent_attention", "mixer": mixer}


def _moe(experts, top, ff, shared):
    out = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared is not None:
        out["shared"] = {"ff": shared}
    return out


def all_experts(raw: dict) -> dict:
    """The same configuration with every router choosing all its experts (each with its own score).  A choice among experts
    is discrete: where two scores are close, the rounding of bfloat16 activations can turn it, and the two sides then
    compute different functions.  Whole models are therefore compared with real choices in 32-bit and with all experts in
    bfloat16; the router alone is compared in both formats."""
    for layer in raw["layers"]:
        if layer.get("mlp") is not None:
            layer["mlp"]["router"]["top"] = layer["mlp"]["router"]["experts"]
    return raw


def config(which: str, every_expert: bool = False) -> dict:
    return all_experts(_config(which)) if every_expert else _config(which)


def _config(which: str) -> dict:
    """A: every mixer, a loop of two passes over the first layers, windows that end inside a page and across pages, shared
    experts as wide as the others, wider and narrower, a layer without a feed-forward.  B: a loop in the middle with layers
    around it, one chosen expert, no shared expert, no kept tokens, as many key heads as query heads.  C: odd sizes
    everywhere, no loop, windows of one token, more kept tokens than the window has, a temperature that grows with every
    token.  D: latents of 160 and 256 numbers, more query heads than a tile has rows, heads of 128, kept tokens over two key
    blocks, a loop of one pass.  E: nothing has a window, queries keep their temperature."""
    if which == "A":
        layers = [
            {**_latent(4, 16, 12, 24, 40, 24), "mlp": _moe(6, 2, 40, 40)},
            {**_attention(6, 2, 24, 16, 19, 3), "mlp": None},
            {**_tempered(4, 2, 16, 24, 0.4, 16), "mlp": _moe(4, 3, 24, 56)},
            {**_attention(3, 3, 16, 40, 40, 9), "mlp": _moe(6, 2, 40, 16)},
        ]
        return {"architecture": "Vumotar", "vocab": 211, "width": 64, "layers": layers, "norm": {"eps": 1e-5},
                "loop": {"start": 0, "stop": 3, "times": 2}}
    if which == "B":
        layers = [
            {**_tempered(3, 3, 40, 48, -0.2, 7), "mlp": _moe(5, 1, 64, None)},
            {**_latent(8, 16, 16, 40, 48, 33), "mlp": _moe(3, 2, 32, None)},
            {**_attention(4, 4, 32, 32, 50, 0), "mlp": None},
            {**_latent(2, 40, 48, 16, 64, None), "mlp": _moe(4, 1, 48, 96)},
        ]
        return {"architecture": "Vumotar", "vocab": 300, "width": 96, "layers": layers, "norm": {"eps": 1e-6},
                "loop": {"start": 1, "stop": 3, "times": 3}}
    if which == "C":
        layers = [
            {**_latent(5, 10, 14, 13, 20, 1, 0.5), "mlp": _moe(3, 3, 20, 9)},
            {**_attention(5, 1, 11, 9, 1, 5, 0.4), "mlp": _moe(2, 2, 12, 30)},
            {**_tempered(2, 1, 7, 13, 0.7, 1, 0.3), "mlp": None},
            {**_attention(7, 7, 10, 34, 4, 6), "mlp": None},
        ]
        return {"architecture": "Vumotar", "vocab": 97, "width": 70, "layers": layers, "norm": {"eps": 1e-4}}
    if which == "D":
        layers = [
            {**_latent(20, 32, 24, 96, 160, 100), "mlp": _moe(4, 2, 128, 128)},
            {**_attention(12, 2, 128, 64, 60, 70), "mlp": _moe(4, 2, 64, 192)},
            {**_latent(4, 128, 128, 64, 256, 50), "mlp": None},
            {**_tempered(2, 2, 64, 64, 0.3, 64), "mlp": _moe(4, 2, 64, 128)},
        ]
        return {"architecture": "Vumotar", "vocab": 384, "width": 128, "layers": layers, "norm": {"eps": 1e-5},
                "loop": {"start": 0, "stop": 4, "times": 1}}
    if which == "E":
        layers = [
            {**_attention(4, 2, 24, 24, None, 0), "mlp": _moe(4, 2, 32, 32)},
            {**_tempered(2, 1, 16, 16, None, 1), "mlp": _moe(4, 1, 32, 64)},
            {**_latent(3, 16, 8, 24, 32, None), "mlp": None},
        ]
        return {"architecture": "Vumotar", "vocab": 64, "width": 40, "layers": layers, "norm": {"eps": 1e-5},
                "loop": {"start": 1, "stop": 2, "times": 2}}
    raise KeyError(which)


def random_config(rng) -> dict:
    """A configuration drawn at random: 2 to 6 layers of the three kinds in any order, some without a feed-forward, with or
    without a loop, sizes and constants that are not the fixed cases'."""
    width = rng.choice([96, 128, 160, 192, 320, 384])
    layers = []
    for _ in range(rng.randint(2, 6)):
        mlp = None
        if rng.random() > 0.2:
            experts = rng.choice([2, 4, 8, 16])
            mlp = _moe(experts, rng.randint(1, min(experts, 4)), rng.choice([32, 48, 64, 128]), rng.choice([None, 32, 64, 80, 128]))
        kind = rng.choice(["attention", "attention_2", "latent_attention"])
        kv = rng.choice([1, 2, 3, 4])
        heads = kv * rng.choice([1, 2, 3, 5])
        dim, vdim = rng.choice([16, 24, 32, 48, 96, 128]), rng.choice([16, 32, 48, 64, 80])
        if kind == "attention":
            layer = _attention(heads, kv, dim, vdim, rng.choice([None, 17, 64, 100, 129]), rng.choice([0, 1, 4, 16, 65]))
        elif kind == "attention_2":
            layer = _tempered(heads, kv, dim, vdim, rng.choice([0.1, 0.5, 1.0]), rng.choice([1, 10, 64, 100]))
        else:
            layer = _latent(rng.randint(1, 12), dim, vdim, rng.choice([32, 48, 128]), rng.choice([32, 64, 96, 160, 192]),
                            rng.choice([None, 17, 64, 100, 129]))
        layers.append({**layer, "mlp": mlp})
    raw = {"architecture": "Vumotar", "vocab": rng.choice([300, 480, 512, 1000]), "width": width, "layers": layers,
           "norm": {"eps": rng.choice([1e-5, 1e-6])}}
    if rng.random() < 0.7:
        start = rng.randint(0, len(layers) - 1)
        raw["loop"] = {"start": start, "stop": rng.randint(start + 1, len(layers)), "times": rng.randint(1, 3)}
    return raw


PAGE_TOKENS = {"A": 8, "B": 16, "C": 4, "D": 16, "E": 8}


def random_weights(raw: dict, seed: int, dtype=torch.float32, sharp: float = 1.0, as_bfloat16: bool = False) -> dict:
    """Weights with unit-variance activations: matrices ``N(0, 1 / inputs)``, norm weights ``1 + N(0, 0.3)``, sinks
    ``1 + N(0, 1)``.  ``sharp`` scales what the queries are made with (a softmax that leans on few keys).
    ``as_bfloat16``: every number is one that bfloat16 holds."""
    gen = torch.Generator().manual_seed(seed)
    c = raw["width"]

    def mat(rows, cols, scale=1.0):
        return torch.randn(rows, cols, generator=gen) * (scale / math.sqrt(cols))

    def vec(n, scale=0.3):
        return torch.randn(n, generator=gen) * scale

    w = {"embed": torch.randn(raw["vocab"], c, generator=gen), "final.norm": 1.0 + vec(c)}
    for i, layer in enumerate(raw["layers"]):
        p, m, h = f"l{i}.", layer["mixer"], layer["mixer"]["heads"]
        x = p + "mix."
        w[p + "norm1"], w[p + "norm1b"] = 1.0 + vec(c), 1.0 + vec(c)
        if layer["type"] == "latent_attention":
            w[x + "dq"], w[x + "dq.norm"] = mat(m["q_rank"], c), 1.0 + vec(m["q_rank"])
            w[x + "uq"] = mat(h * m["dim"], m["q_rank"], sharp)
            w[x + "dkv"], w[x + "dkv.norm"] = mat(m["kv_rank"], c), 1.0 + vec(m["kv_rank"])
            w[x + "uk"], w[x + "uv"] = mat(h * m["dim"], m["kv_rank"]), mat(h * m["vdim"], m["kv_rank"])
            w[x + "sink"], w[x + "g"] = vec(h, 1.0) + 1.0, mat(h, c)
        else:
            g = m["kv_heads"]
            w[x + "q"], w[x + "k"], w[x + "v"] = mat(h * m["dim"], c, sharp), mat(g * m["dim"], c), mat(g * m["vdim"], c)
            if layer["type"] == "attention":
                w[x + "q.norm"], w[x + "k.norm"] = sharp * (1.0 + vec(m["dim"])), 1.0 + vec(m["dim"])
        w[x + "o"] = mat(c, h * m["vdim"])
        f = layer.get("mlp")
        if f is not None:
            w[p + "norm2"], w[p + "norm2b"] = 1.0 + vec(c), 1.0 + vec(c)
            y = p + "mlp."
            w[y + "router"] = mat(f["router"]["experts"], c, 2.0)
            units = [(f"e{e}.", f["expert"]["ff"]) for e in range(f["router"]["experts"])]
            if f.get("shared") is not None:
                units.append(("shared.", f["shared"]["ff"]))
            for name, ff in units:
                w[y + name + "gate"], w[y + name + "up"], w[y + name + "down"] = mat(ff, c), mat(ff, c), mat(c, ff)
    if as_bfloat16:
        w = {k: v.to(torch.bfloat16).float() for k, v in w.items()}
    return {k: v.to(dtype).contiguous() for k, v in w.items()}


def tokens_for(raw: dict, length: int, seed: int) -> list[int]:
    gen = torch.Generator().manual_seed(1000 + seed)
    return torch.randint(0, raw["vocab"], (length,), generator=gen).tolist()


def plain_logits(raw: dict, tensors: dict, tokens, rows=None, dtype=torch.float64) -> torch.Tensor:
    out = plain_vumotar.forward(raw, tensors, tokens, dtype)
    return out if rows is None else out[list(rows)]


def rounding_spread(raw: dict, tensors: dict, tokens, rows=None) -> torch.Tensor:
    """Per row: how far the logits move (over the row's spread) when the activations between matrix products are rounded to
    bfloat16 in the plain implementation and nothing else changes.  A bfloat16 run is held to its tolerance plus three
    times this."""
    exact = plain_vumotar.forward(raw, tensors, tokens)
    moved = plain_vumotar.forward(raw, tensors, tokens, round_inputs=torch.bfloat16)
    err = relative_error(moved, exact)
    return err if rows is None else err[list(rows)]


def plain_greedy(raw: dict, tensors: dict, prompt, new_tokens: int) -> list[int]:
    return plain_vumotar.greedy(raw, tensors, prompt, new_tokens)


ASKS, ANSWERS = 7, 9     # in the leaning model a token ASKS scores far higher against a token ANSWERS than against any other


def leaning_model(layer: dict, seed: int = 5, sinks: float = -2.0, height: float = 14.0) -> tuple[dict, dict]:
    """A model of one layer, ``layer`` (its mixer entry), whose queries lean on one key: every query head of token ASKS points
    along its key head's key of token ANSWERS, so that their score is ``height`` (before any temperature) where other
    scores are of size 1 or less.  Returns the configuration and its weights."""
    raw = {"architecture": "Vumotar", "vocab": 50, "width": 64, "norm": {"eps": 1e-5}, "layers": [{**layer, "mlp": None}]}
    m, eps = layer["mixer"], 1e-5
    w = random_weights(raw, seed, as_bfloat16=True)
    h, d = m["heads"], m["dim"]
    unit = {t: plain_vumotar.rms_norm(w["embed"][t], w["l0.norm1"], eps) for t in (ASKS, ANSWERS)}
    x = "l0.mix."
    if layer["type"] == "latent_attention":
        source = plain_vumotar.rms_norm(w[x + "dq"] @ unit[ASKS], w[x + "dq.norm"], eps)
        c = plain_vumotar.rms_norm(w[x + "dkv"] @ unit[ANSWERS], w[x + "dkv.norm"], eps)
        keys = (w[x + "uk"] @ c).view(h, d)
        name = "uq"
        w[x + "sink"].fill_(sinks)
    else:
        source, g, name = unit[ASKS], m["kv_heads"], "q"
        keys = (w[x + "k"] @ unit[ANSWERS]).view(g, d)
        if layer["type"] == "attention":
            # the norm takes the size of what is projected away: the gains set the height
            keys = plain_vumotar.rms_norm(keys, w[x + "k.norm"], eps)
            keys = keys / w[x + "q.norm"]
        keys = keys.repeat_interleave(h // g, 0)
    if layer["type"] == "attention":
        rows = keys
        reached = ((plain_vumotar.rms_norm(rows, w[x + "q.norm"], eps) * (keys * w[x + "q.norm"])).sum(-1) * m["scale"]).mean()
        w[x + "q.norm"] = (w[x + "q.norm"] * (height / reached)).to(torch.bfloat16).float()
    else:
        rows = height / m["scale"] * keys / (keys * keys).sum(-1, keepdim=True)
    w[x + name] = (rows[:, :, None] * source / (source * source).sum()).reshape(h * d, -1).to(torch.bfloat16).float().contiguous()
    return raw, w


def disliking_model(seed: int = 8) -> tuple[dict, dict]:
    """One layer of ``attention`` with two heads.  The embeddings share a direction; the first head's keys all point one way
    and its queries the other, so that its scores are all far below zero and the term of 1 takes nearly all its weight."""
    raw = {"architecture": "Vumotar", "vocab": 50, "width": 64, "norm": {"eps": 1e-5},
           "layers": [{**_attention(2, 2, 32, 24, 20, 2, 0.2), "mlp": None}]}
    w = random_weights(raw, seed)
    gen = torch.Generator().manual_seed(seed)
    common, way = torch.randn(64, generator=gen), torch.randn(32, generator=gen)
    w["embed"] = 0.5 * w["embed"] + common
    w["l0.norm1"] = torch.ones(64)
    w["l0.mix.k"][:32] = way[:, None] * common / 8
    w["l0.mix.q"][:32] = -way[:, None] * common / 8
    return raw, {k: v.to(torch.bfloat16).float().contiguous() for k, v in w.items()}


def leaning_tokens(raw: dict, length: int, seed: int, at: int, answer: bool = True) -> list[int]:
    """A sequence that ends with ASKS and holds ANSWERS at place ``at`` only (another token there, not ``answer``)."""
    toks = [t if t not in (ASKS, ANSWERS) else 1 for t in tokens_for(raw, length, seed)]
    toks[-1], toks[at] = ASKS, ANSWERS if answer else 11
    return toks


def relative_error(got: torch.Tensor, want: torch.Tensor) -> torch.Tensor:
    """Per row: the largest difference of the logits over the row's own spread."""
    want = want.double()
    return (got.double().cpu() - want).abs().amax(-1) / want.std(-1)


def assert_rows_close(got, want, tol, what: str, places=None, outliers: float = 0.0, slack=None) -> None:
    """``outliers``: the share of rows (at least one, if not zero) that may miss ``tol``, though not five times ``tol``.
    ``slack``: per row, what rounding alone does (``rounding_spread``); three times it is added to ``tol``."""
    err = relative_error(got, want)
    limit = torch.full_like(err, tol) if slack is None else tol + 3.0 * slack
    bad = (~(err <= limit)).nonzero()
    if outliers and 0 < bad.numel() <= max(1, int(outliers * err.numel())):
        bad = (~(err <= 5 * limit)).nonzero()
    if bad.numel():
        i = int(bad[0])
        raise AssertionError(f"{what}: first wrong logits at {places[i] if places is not None else i}: "
                             f"error {float(err[i]):.3e} of the row's spread > {float(limit[i]):.1e}")
