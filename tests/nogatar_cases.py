"""Small Nogatar configurations and random weights for the tests, made here (names and shapes written out from the
design, not taken from the engine's own list), and the plain logits."""

from __future__ import annotations

import math

import torch

import plain_nogatar


def _latent(heads, dim, rot_dim, vdim, rank, window, base=1e4, scaling=(4.0, 64, 32.0, 1.0), scale=None):
    rot = {"base": base, "dims": rot_dim}
    if scaling is not None:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    mixer = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": rank, "rot": rot,
             "scale": 1.0 / math.sqrt(dim + rot_dim) if scale is None else scale}
    if window is not None:
        mixer["mask"] = {"size": window}
    return {"type": "latent_attention", "mixer": mixer}


def _mlstm(heads, dim, vdim, cap):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}}


def _moe(experts, top, ff, shared):
    out = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared is not None:
        out["shared"] = {"ff": shared}
    return out


def all_experts(raw: dict) -> dict:
    """The same configuration with every router choosing all its experts (the weights stay a softmax).  A choice among
    experts is discrete: where two router logits are close, the rounding of bfloat16 activations can turn it, and the
    two sides then compute different functions.  Whole models are therefore compared with real choices in 32-bit and
    with all experts in bfloat16; the router alone is compared in both formats."""
    for layer in raw["layers"]:
        if layer.get("mlp") is not None:
            layer["mlp"]["router"]["top"] = layer["mlp"]["router"]["experts"]
    return raw


def config(which: str, every_expert: bool = False) -> dict:
    return all_experts(_config(which)) if every_expert else _config(which)


def _config(which: str) -> dict:
    """A: every mixer and feed-forward, windows that end inside a page and across pages, a shared expert as wide as the
    others, wider and narrower, a layer without a feed-forward.  B: a layer without a window, more positions than the
    stretched frequencies were made for, one chosen expert, no shared expert, a factor of 1, no cap on the logits.
    C: odd sizes everywhere, a window of one token (only itself and the sink), frequencies as they are, all experts
    chosen.  D: latents of 160 and 256 numbers (wide cache rows), more query heads than a tile has rows, heads of 128.
    E: recurrent layers alone (nothing is kept in pages)."""
    if which == "A":
        layers = [
            {**_latent(4, 16, 8, 12, 40, 24), "mlp": _moe(6, 2, 40, 40)},
            {**_mlstm(3, 16, 24, 9.0), "mlp": None},
            {**_latent(6, 24, 16, 16, 32, 7, 500.0, (2.5, 40, 8.0, 2.0)), "mlp": _moe(4, 3, 24, 56)},
            {**_mlstm(2, 24, 16, 15.0), "mlp": _moe(6, 2, 40, 16)},
        ]
        return {"architecture": "Nogatar", "vocab": 211, "width": 64, "layers": layers, "norm": {"eps": 1e-5},
                "embedding": {"scale": 8.5}, "residual_mult": 0.7, "logit_softcap": 8.0}
    if which == "B":
        layers = [
            {**_latent(3, 40, 24, 48, 64, None, 1e6, (8.0, 20, 16.0, 0.5)), "mlp": _moe(5, 1, 64, None)},
            {**_mlstm(2, 40, 40, 5.0), "mlp": _moe(3, 2, 32, None)},
            {**_latent(8, 16, 16, 16, 48, 33, 1e4, (1.0, 512, 32.0, 1.0)), "mlp": None},
        ]
        return {"architecture": "Nogatar", "vocab": 300, "width": 96, "layers": layers, "norm": {"eps": 1e-6},
                "embedding": {"scale": 1.0}, "residual_mult": 1.0}
    if which == "C":
        layers = [
            {**_latent(5, 10, 6, 14, 20, 19, 100.0, None), "mlp": _moe(3, 3, 20, 9)},
            {**_mlstm(1, 72, 10, 12.0), "mlp": _moe(2, 2, 12, 30)},
            {**_latent(2, 7, 2, 9, 11, 1, 50.0, (3.0, 30, 4.0, 1.0)), "mlp": None},
            {**_mlstm(3, 10, 34, 30.0), "mlp": None},
        ]
        return {"architecture": "Nogatar", "vocab": 97, "width": 70, "layers": layers, "norm": {"eps": 1e-4},
                "embedding": {"scale": 3.0}, "residual_mult": 0.3, "logit_softcap": 30.0}
    if which == "D":
        layers = [
            {**_latent(20, 32, 32, 24, 160, 100), "mlp": _moe(4, 2, 128, 128)},
            {**_latent(4, 128, 64, 128, 256, 50), "mlp": None},
            {**_mlstm(2, 128, 64, 10.0), "mlp": _moe(4, 2, 64, 192)},
        ]
        return {"architecture": "Nogatar", "vocab": 384, "width": 128, "layers": layers, "norm": {"eps": 1e-5},
                "embedding": {"scale": 11.0}, "residual_mult": 0.5, "logit_softcap": 15.0}
    if which == "E":
        layers = [{**_mlstm(2, 16, 24, 6.0), "mlp": _moe(4, 2, 32, 32)}, {**_mlstm(1, 32, 8, 11.0), "mlp": None}]
        return {"architecture": "Nogatar", "vocab": 64, "width": 40, "layers": layers, "norm": {"eps": 1e-5},
                "embedding": {"scale": 6.0}, "residual_mult": 0.9, "logit_softcap": 12.0}
    raise KeyError(which)


def random_config(rng) -> dict:
    """A configuration drawn at random: 2 to 6 layers of both kinds in any order, some without a feed-forward, sizes and
    constants that are not the fixed cases'."""
    width = rng.choice([96, 128, 160, 192, 256, 384])
    layers = []
    for _ in range(rng.randint(2, 6)):
        mlp = None
        if rng.random() > 0.2:
            experts = rng.choice([2, 4, 8, 12])
            mlp = _moe(experts, rng.randint(1, min(experts, 4)), rng.choice([32, 48, 64, 128]), rng.choice([None, 32, 64, 80, 128]))
        if rng.random() < 0.6:
            dim, rot = rng.choice([16, 24, 32, 64]), rng.choice([8, 16, 32])
            scaling = None if rng.random() < 0.2 else (rng.choice([2.0, 4.0, 16.0]), rng.choice([64, 256, 1024]),
                                                       rng.choice([16.0, 32.0]), rng.choice([1.0, 2.0]))
            layer = _latent(rng.randint(1, 12), dim, rot, rng.choice([16, 32, 48, 64]), rng.choice([32, 64, 96, 128, 192]),
                            rng.choice([None, 17, 64, 100, 129, 256]), rng.choice([1e4, 5e5, 1e6]), scaling)
        else:
            layer = _mlstm(rng.randint(1, 6), rng.choice([16, 32, 48, 64]), rng.choice([16, 32, 64, 96]), rng.choice([5.0, 15.0, 30.0]))
        layers.append({**layer, "mlp": mlp})
    raw = {"architecture": "Nogatar", "vocab": rng.choice([300, 480, 512, 1000]), "width": width, "layers": layers,
           "norm": {"eps": rng.choice([1e-5, 1e-6])}, "embedding": {"scale": rng.choice([1.0, 4.0, math.sqrt(width)])},
           "residual_mult": rng.choice([0.25, 0.5, 1.0, 1.3])}
    if rng.random() < 0.7:
        raw["logit_softcap"] = rng.choice([10.0, 20.0, 30.0])
    return raw


PAGE_TOKENS = {"A": 8, "B": 16, "C": 4, "D": 16, "E": 8}


def random_weights(raw: dict, seed: int, dtype=torch.float32, sharp: float = 1.0, as_bfloat16: bool = False,
                   steady: bool = False) -> dict:
    """Weights with unit-variance activations: matrices ``N(0, 1 / inputs)``, norm weights ``1 + N(0, 0.3)``, biases and
    sinks ``N(0, 1)``, the embedding so that a scaled row has numbers of size 1.  ``sharp`` scales the attention's query
    projection (a softmax that leans on few keys).  ``as_bfloat16``: every number is one that bfloat16 holds.
    ``steady``: the matrix memories' query matrices lean towards their key matrices, so that a token's read-out of its own
    key is well away from zero.  (Every head's read-out is divided by its root mean square: where it is one term, as for
    a sequence's first tokens, and that term nearly cancels, the norm magnifies the rounding of bfloat16 queries and keys
    without bound.  Runs in bfloat16 use steady weights; 32-bit runs do not.)"""
    gen = torch.Generator().manual_seed(seed)
    c = raw["width"]

    def mat(rows, cols, scale=1.0):
        return torch.randn(rows, cols, generator=gen) * (scale / math.sqrt(cols))

    def vec(n, scale=0.3):
        return torch.randn(n, generator=gen) * scale

    w = {"embed": torch.randn(raw["vocab"], c, generator=gen) / raw["embedding"]["scale"], "final.norm": 1.0 + vec(c),
         "head": mat(raw["vocab"], c, 2.0)}
    for i, layer in enumerate(raw["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        x = p + "mix."
        h = m["heads"]
        w[p + "norm1"] = 1.0 + vec(c)
        if layer["type"] == "mlstm":
            n, nv = h * m["dim"], h * m["vdim"]
            w[x + "q"], w[x + "k"], w[x + "v"], w[x + "g"], w[x + "o"] = mat(n, c), mat(n, c), mat(nv, c), mat(nv, c), mat(c, nv)
            for gate, shift in (("i", -1.0), ("f", 3.0)):
                w[x + gate], w[x + gate + ".b"] = mat(h, c), vec(h, 1.0) + shift
            w[x + "norm"] = 1.0 + vec(nv)
            if steady:
                w[x + "q"] = w[x + "k"] + 0.5 * w[x + "q"]
        else:
            w[x + "q"] = mat(h * (m["dim"] + m["rot_dim"]), c, sharp)
            w[x + "dkv"], w[x + "dkv.norm"] = mat(m["kv_rank"] + m["rot_dim"], c), 1.0 + vec(m["kv_rank"])
            w[x + "uk"], w[x + "uv"] = mat(h * m["dim"], m["kv_rank"]), mat(h * m["vdim"], m["kv_rank"])
            w[x + "sink"], w[x + "o"] = vec(h, 1.0) + 1.0, mat(c, h * m["vdim"])
        f = layer.get("mlp")
        if f is not None:
            w[p + "norm2"] = 1.0 + vec(c)
            y = p + "mlp."
            w[y + "router"] = mat(f["router"]["experts"], c, 2.0)
            for e in range(f["router"]["experts"]):
                w[f"{y}e{e}.up"], w[f"{y}e{e}.down"] = mat(f["expert"]["ff"], c), mat(c, f["expert"]["ff"])
            if f.get("shared") is not None:
                s = f["shared"]["ff"]
                w[y + "shared.up"], w[y + "shared.down"], w[y + "shared.sg"] = mat(s, c), mat(c, s), mat(1, c)
    if as_bfloat16:
        w = {k: v.to(torch.bfloat16).float() for k, v in w.items()}
    return {k: v.to(dtype).contiguous() for k, v in w.items()}


def tokens_for(raw: dict, length: int, seed: int) -> list[int]:
    gen = torch.Generator().manual_seed(1000 + seed)
    return torch.randint(0, raw["vocab"], (length,), generator=gen).tolist()


def plain_logits(raw: dict, tensors: dict, tokens, rows=None, dtype=torch.float64) -> torch.Tensor:
    out = plain_nogatar.forward(raw, tensors, tokens, dtype)
    return out if rows is None else out[list(rows)]


def rounding_spread(raw: dict, tensors: dict, tokens, rows=None) -> torch.Tensor:
    """Per row: how far the logits move (over the row's spread) when the activations between matrix products are rounded to
    bfloat16 in the plain implementation and nothing else changes.  The design divides heads and sublayer outputs by their
    own spread, so a row where a sum nearly cancels magnifies rounding many times over; a bfloat16 run is held to its
    tolerance plus three times this."""
    exact = plain_nogatar.forward(raw, tensors, tokens)
    moved = plain_nogatar.forward(raw, tensors, tokens, round_inputs=torch.bfloat16)
    err = relative_error(moved, exact)
    return err if rows is None else err[list(rows)]


def plain_greedy(raw: dict, tensors: dict, prompt, new_tokens: int) -> list[int]:
    return plain_nogatar.greedy(raw, tensors, prompt, new_tokens)


ASKS, ANSWERS = 7, 9     # in the leaning model a token ASKS scores far higher against a token ANSWERS than against any other


def leaning_model(window, rank: int, seed: int = 5, sinks: float = -2.0) -> tuple[dict, dict]:
    """One attention layer whose queries lean on one key: every head's query matrix sends the embedding of token ASKS to
    the key direction of token ANSWERS (the head's key matrix times its latent) and nothing of the queries turns.
    Returns the configuration and its weights."""
    raw = {"architecture": "Nogatar", "vocab": 50, "width": 64, "norm": {"eps": 1e-5}, "embedding": {"scale": 4.0},
           "residual_mult": 1.5, "layers": [{**_latent(2, 32, 8, 32, rank, window, scale=0.6), "mlp": None}]}
    w = random_weights(raw, seed, as_bfloat16=True)
    asks, answers = w["embed"][ASKS], w["embed"][ANSWERS]
    q = w["l0.mix.q"].view(2, 40, 64)
    for head in range(2):
        key = w["l0.mix.uk"].view(2, 32, rank)[head] @ (w["l0.mix.dkv"][:rank] @ answers)
        key = 3.0 * key / key.pow(2).mean().sqrt()
        q[head, :32] = (key[:, None] * asks[None, :] / (4.0 * asks.pow(2).sum())).to(torch.bfloat16).float()
        q[head, 32:] = 0.0
    w["l0.mix.sink"].fill_(sinks)
    return raw, w


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
    """``outliers``: the share of rows (at least one, if not zero) that may miss ``tol``, though not five times
    ``tol`` (bfloat16 runs: a unit norm after a read-out that nearly cancels magnifies one token's rounding).
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
