"""A plain, slow Nogatar: one function per mechanism, whole sequences, float64 by default.

It takes the model as a config dict (the keys of ``config.json``) and a dict of tensors by their
checkpoint names, and shares no code with the engine.  Notation: ``x`` is the residual stream
``[T, width]`` of one sequence, ``h`` the input of a mixer or feed-forward, ``t`` a position.

* embedding:   ``s * E[tok_t]`` with ``s = embedding.scale``
* layer norm:  ``n(y) = (y - mean(y)) / sqrt(mean((y - mean(y))^2) + eps) * w`` (no shift)
* a layer:     ``x += r * n1(mixer(x))``, ``x += r * n2(ff(x))`` (if it has a feed-forward), ``r = residual_mult``;
  nothing stands in front of a sublayer
* mlstm:       ``m_t = max(f + m_(t-1), i)``, ``S_t = exp(f + m_(t-1) - m_t) S_(t-1) + exp(i - m_t) k v^T``, ``n_t``
  the same with ``k`` alone, ``o = S_t^T q / (max(|n_t . q|, exp(-m_t)) + 1e-6)``; per head divided by its root mean
  square, times a gain of all heads' size, times ``sigmoid(W_g h)``, projected
* latents:     one row ``[c | r]`` per token, ``c`` RMS-normed, ``r`` rotated; every head's key is ``[W_uk c | r]`` and
  its value ``W_uv c``; interleaved rotation with stretched frequencies; a sliding window; a softmax whose
  denominator holds one learned term more per head
* experts:     softmax over all router logits scores, the ``top`` largest are used, weighed by their scores over the
  scores' sum; an expert is ``W_down max(W_up h, 0)^2``; one more of the same form for every token, times
  ``sigmoid(W_sg h)``
* output:      ``cap * tanh(W n(x) / cap)``
"""

from __future__ import annotations

import math

import torch


# ---- pieces --------------------------------------------------------------------------------------
ROUND = None      # a dtype through which activations between two products are rounded (see ``forward``), or None


def _r(x):
    return x if ROUND is None else x.to(ROUND).to(x.dtype)


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def layer_norm(y, w, eps):
    d = y - y.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w


def stretched_frequencies(n, base, scaling):
    """``n/2`` rotary frequencies (and the factor on cosine and sine).  ``scaling``: factor, original, fast, slow, or
    None.  Pairs that turn more than ``fast`` times over ``original`` positions keep their frequency, pairs that turn
    fewer than ``slow`` times are slowed by ``factor``, a linear ramp over the pair's number between."""
    freq = [base ** (-2.0 * i / n) for i in range(n // 2)]
    if not scaling:
        return freq, 1.0

    def pair_of(turns):
        return n * math.log(scaling["original"] / (2 * math.pi * turns)) / (2 * math.log(base))
    lo = max(math.floor(pair_of(scaling["fast"])), 0)
    hi = min(math.ceil(pair_of(scaling["slow"])), n - 1)
    out = []
    for i, f in enumerate(freq):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / scaling["factor"] * ramp + f * (1 - ramp))
    return out, 0.1 * math.log(scaling["factor"]) + 1.0


def rotate_pairs(x, positions, freq, magnitude):
    """x: [T, heads, n]: feature ``2i`` with ``2i + 1``, angle ``t * freq[i]``."""
    if x.shape[-1] == 0:
        return x
    angle = positions.to(x.dtype)[:, None] * torch.tensor(freq, dtype=x.dtype)[None, :]
    cos, sin = (magnitude * torch.cos(angle))[:, None, :], (magnitude * torch.sin(angle))[:, None, :]
    u, v = x[..., 0::2], x[..., 1::2]
    return torch.stack([u * cos - v * sin, v * cos + u * sin], dim=-1).flatten(-2)


# ---- mixers --------------------------------------------------------------------------------------
def mlstm_mixer(h, w, p, m, eps):
    T = h.shape[0]
    H, d, dv, cap = m["heads"], m["dim"], m["vdim"], m["gate_cap"]
    q = _r(h @ w[p + "q"].T).view(T, H, d) * d ** -0.5
    k = _r(h @ w[p + "k"].T).view(T, H, d)
    v = _r(h @ w[p + "v"].T).view(T, H, dv)
    i = cap * torch.tanh((h @ w[p + "i"].T + w[p + "i.b"]) / cap)
    f = torch.nn.functional.logsigmoid(cap * torch.tanh((h @ w[p + "f"].T + w[p + "f.b"]) / cap))
    S = torch.zeros(H, d, dv, dtype=h.dtype)
    n = torch.zeros(H, d, dtype=h.dtype)
    top = torch.zeros(H, dtype=h.dtype)
    out = []
    for t in range(T):
        new = torch.maximum(f[t] + top, i[t])
        keep, add = torch.exp(f[t] + top - new), torch.exp(i[t] - new)
        S = keep[:, None, None] * S + add[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + add[:, None] * k[t]
        top = new
        den = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-top)) + 1e-6
        out.append(torch.einsum("hde,hd->he", S, q[t]) / den[:, None])
    o = unit_rms(torch.stack(out), eps).reshape(T, H * dv) * w[p + "norm"]
    return _r(o * torch.sigmoid(_r(h @ w[p + "g"].T))) @ w[p + "o"].T


def latent_attention_mixer(h, w, p, m, eps):
    T = h.shape[0]
    H, d, r, dv, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    rot = m.get("rot") or {"base": 1.0}
    pos = torch.arange(T)
    freq, magnitude = stretched_frequencies(r, rot["base"], rot.get("scaling"))
    q = _r(h @ w[p + "q"].T).view(T, H, d + r)
    low = _r(h @ w[p + "dkv"].T)
    c = _r(unit_rms(low[:, :rank], eps) * w[p + "dkv.norm"])
    shared = _r(rotate_pairs(low[:, rank:].view(T, 1, r), pos, freq, magnitude)).expand(T, H, r)
    q = torch.cat([q[..., :d], _r(rotate_pairs(q[..., d:], pos, freq, magnitude))], dim=-1)
    k = torch.cat([(c @ w[p + "uk"].T).view(T, H, d), shared], dim=-1)
    v = (c @ w[p + "uv"].T).view(T, H, dv)
    s = torch.einsum("ihd,jhd->hij", q, k) * m["scale"]
    gap = pos[:, None] - pos[None, :]
    size = (m.get("mask") or {}).get("size")
    seen = (gap >= 0) if size is None else (gap >= 0) & (gap < size)
    s = s.masked_fill(~seen, float("-inf"))
    sink = w[p + "sink"].view(H, 1, 1).expand(H, T, 1)
    weights = torch.softmax(torch.cat([s, sink], dim=-1), dim=-1)[..., :T]      # the sink's weight meets no value
    o = torch.einsum("hij,jhe->ihe", weights, v).reshape(T, H * dv)
    return _r(o) @ w[p + "o"].T


# ---- feed-forward ---------------------------------------------------------------------------------
def squared_relu_unit(h, w, e):
    z = torch.clamp(h @ w[e + "up"].T, min=0.0)
    return _r(z * z) @ w[e + "down"].T


def routed_experts(h, w, p, f):
    top = f["router"]["top"]
    s = torch.softmax(h @ w[p + "router"].T, dim=-1)
    best, ids = torch.topk(s, top, dim=-1)
    weights = best / (best.sum(-1, keepdim=True) + 1e-20)
    out = torch.zeros(h.shape[0], w[p + "e0.down"].shape[0], dtype=h.dtype)
    for t in range(h.shape[0]):
        for j in range(top):
            out[t] += weights[t, j] * squared_relu_unit(h[t], w, f"{p}e{int(ids[t, j])}.")
    if f.get("shared") is not None:
        out = out + torch.sigmoid(h @ w[p + "shared.sg"].T) * squared_relu_unit(h, w, p + "shared.")
    return out


# ---- the model -----------------------------------------------------------------------------------
def forward(cfg, w, tokens, dtype=torch.float64, return_layers=False, round_inputs=None):
    """Logits ``[T, vocab]`` of one sequence (and the stream after every layer).  ``round_inputs``: a dtype through
    which every activation that passes from one matrix product to the next is rounded on its way (the sublayers'
    inputs, projected queries, keys, values and gates, latents, heads, hidden features), as a run that keeps such
    activations in that dtype does: a measure of how far rounding alone moves a row.  Sums, norms, states and scores
    stay as they are."""
    global ROUND
    if round_inputs is not None and ROUND is None:
        ROUND = round_inputs
        try:
            return forward(cfg, w, tokens, dtype, return_layers, round_inputs)
        finally:
            ROUND = None
    w = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in w.items()}
    eps, mult = cfg["norm"]["eps"], cfg["residual_mult"]
    ids = torch.as_tensor(list(tokens), dtype=torch.long)
    x = w["embed"][ids] * cfg["embedding"]["scale"]
    after = []
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        mixer = {"mlstm": mlstm_mixer, "latent_attention": latent_attention_mixer}[layer["type"]]
        x = x + mult * layer_norm(mixer(_r(x), w, p + "mix.", m, eps), w[p + "norm1"], eps)
        if layer.get("mlp") is not None:
            x = x + mult * layer_norm(routed_experts(_r(x), w, p + "mlp.", layer["mlp"]), w[p + "norm2"], eps)
        after.append(x)
    logits = _r(layer_norm(x, w["final.norm"], eps)) @ w["head"].T
    cap = cfg.get("logit_softcap")
    if cap:
        logits = cap * torch.tanh(logits / cap)
    return (logits, after) if return_layers else logits


def greedy(cfg, w, prompt, new_tokens, dtype=torch.float64):
    """The prompt's greedy continuation, every token from a whole pass over the sequence so far."""
    seq, out = list(prompt), []
    for _ in range(new_tokens):
        out.append(int(forward(cfg, w, seq, dtype)[-1].argmax()))
        seq.append(out[-1])
    return out
