"""A plain, slow Vumotar: one function per mechanism, whole sequences, float64 by default.

It takes the model as a config dict (the keys of ``config.json``) and a dict of tensors by their
checkpoint names, and shares no code with the engine.  Notation: ``x`` is the residual stream
``[T, width]`` of one sequence, ``h`` the input of a mixer or feed-forward, ``t`` a position.

* rms norm:    ``n(y) = y / sqrt(mean(y^2) + eps) * w``
* a layer:     ``x += n1b(mixer(n1(x)))``, ``x += n2b(ff(n2(x)))`` (if it has a feed-forward)
* attention:   query and key heads RMS-normed; no positions in the scores; ``t`` sees the last ``size`` positions, its
  own included, and the first ``keep_first`` of the sequence; one more term, 1, in the softmax's denominator
* attention_2: every earlier position is seen; queries grow by ``1 + coef * ln(floor((t + 1) / every) + 1)``
* latents:     queries from a normed latent of their own; keys and values of every head from one normed latent per
  token; a sliding window; one learned term ``exp(sink_h)`` more in the denominator; heads times ``sigmoid`` of one gate
  number each
* experts:     ``sigmoid`` of every router logit scores, the ``top`` largest are used; expert e adds ``E_e(s_e h)``,
  ``E(u) = W_down (silu(W_gate u) * W_up u)``; one more expert of that form for every token, its input as it is
* a loop:      a range of layers runs several times in a row with the same weights
* output:      ``E n(x)`` with the embedding's table
"""

from __future__ import annotations

import math

import torch


# ---- pieces --------------------------------------------------------------------------------------
ROUND = None      # a dtype through which activations between two products are rounded (see ``forward``), or None


def _r(x):
    return x if ROUND is None else x.to(ROUND).to(x.dtype)


def rms_norm(y, w, eps):
    return y / torch.sqrt((y * y).mean(-1, keepdim=True) + eps) * w


def visible(T, size=None, keep_first=0):
    """``[T, T]``: whether query ``i`` sees key ``j``."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    near = torch.ones(T, T, dtype=torch.bool) if size is None else i - j < size
    return (j <= i) & (near | (j < keep_first))


def attend(q, k, v, scale, seen, extra=None):
    """q: [T, H, d], k: [T, G, d], v: [T, G, e].  Query head ``h`` reads key head ``h // (H / G)``.  ``extra``: per head, a
    logarithm of one more term of the denominator (no key, no value), or None."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T * scale).masked_fill(~seen, float("-inf"))
        top = s.amax(-1, keepdim=True)
        if extra is not None:
            top = torch.maximum(top, extra[h])
        e = torch.exp(s - top)
        total = e.sum(-1, keepdim=True)
        if extra is not None:
            total = total + torch.exp(extra[h] - top)
        out[:, h] = (e / total) @ v[:, g]
    return out


def temperature(T, coef, every):
    """The factor on the query at each of the positions ``0 .. T - 1``."""
    return torch.tensor([1.0 + coef * math.log(math.floor((t + 1) / every) + 1) for t in range(T)], dtype=torch.float64)


# ---- mixers --------------------------------------------------------------------------------------
def attention_mixer(h, w, p, m, eps):
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = _r(rms_norm(_r(h @ w[p + "q"].T).view(T, H, d), w[p + "q.norm"], eps))
    k = _r(rms_norm(_r(h @ w[p + "k"].T).view(T, G, d), w[p + "k.norm"], eps))
    v = _r(h @ w[p + "v"].T).view(T, G, dv)
    mask = m.get("mask") or {}
    seen = visible(T, mask.get("size"), mask.get("keep_first", 0))
    o = attend(q, k, v, m["scale"], seen, torch.zeros(H, dtype=h.dtype))          # a term of 1 is exp(0)
    return _r(o.reshape(T, H * dv)) @ w[p + "o"].T


def tempered_attention_mixer(h, w, p, m, eps):
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = _r(h @ w[p + "q"].T).view(T, H, d)
    if m.get("q_temp") is not None:
        q = _r(q * temperature(T, m["q_temp"]["coef"], m["q_temp"]["every"]).to(h.dtype)[:, None, None])
    k = _r(h @ w[p + "k"].T).view(T, G, d)
    v = _r(h @ w[p + "v"].T).view(T, G, dv)
    o = attend(q, k, v, m["scale"], visible(T))
    return _r(o.reshape(T, H * dv)) @ w[p + "o"].T


def latent_attention_mixer(h, w, p, m, eps):
    T = h.shape[0]
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    cq = _r(rms_norm(_r(h @ w[p + "dq"].T), w[p + "dq.norm"], eps))
    q = _r(cq @ w[p + "uq"].T).view(T, H, d)
    c = _r(rms_norm(_r(h @ w[p + "dkv"].T), w[p + "dkv.norm"], eps))
    k = (c @ w[p + "uk"].T).view(T, H, d)
    v = (c @ w[p + "uv"].T).view(T, H, dv)
    seen = visible(T, (m.get("mask") or {}).get("size"))
    o = _r(attend(q, k, v, m["scale"], seen, w[p + "sink"]))
    o = o * torch.sigmoid(_r(h @ w[p + "g"].T))[:, :, None]
    return _r(o.reshape(T, H * dv)) @ w[p + "o"].T


# ---- feed-forward ---------------------------------------------------------------------------------
def gated_unit(u, w, e):
    a = u @ w[e + "gate"].T
    return _r(a / (1.0 + torch.exp(-a)) * (u @ w[e + "up"].T)) @ w[e + "down"].T


def routed_experts(h, w, p, f):
    top = f["router"]["top"]
    s = 1.0 / (1.0 + torch.exp(-(h @ w[p + "router"].T)))
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e in torch.topk(s[t], top).indices.tolist():
            out[t] += gated_unit(s[t, e] * h[t], w, f"{p}e{e}.")
    if f.get("shared") is not None:
        out = out + gated_unit(h, w, p + "shared.")
    return out


# ---- the model -----------------------------------------------------------------------------------
def run_order(cfg):
    """The layers' numbers in the order they run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if loop is None:
        return list(range(n))
    return (list(range(loop["start"])) + list(range(loop["start"], loop["stop"])) * loop["times"]
            + list(range(loop["stop"], n)))


def forward(cfg, w, tokens, dtype=torch.float64, return_layers=False, round_inputs=None):
    """Logits ``[T, vocab]`` of one sequence (and the stream after every layer run).  ``round_inputs``: a dtype through
    which every activation that passes from one matrix product to the next is rounded on its way (the sublayers'
    inputs, projected queries, keys, values and gates, latents, heads, hidden features), as a run that keeps such
    activations in that dtype does: a measure of how far rounding alone moves a row.  Sums, norms and scores stay as
    they are."""
    global ROUND
    if round_inputs is not None and ROUND is None:
        ROUND = round_inputs
        try:
            return forward(cfg, w, tokens, dtype, return_layers, round_inputs)
        finally:
            ROUND = None
    w = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in w.items()}
    eps = cfg["norm"]["eps"]
    ids = torch.as_tensor(list(tokens), dtype=torch.long)
    x = w["embed"][ids]
    mixers = {"attention": attention_mixer, "attention_2": tempered_attention_mixer, "latent_attention": latent_attention_mixer}
    after = []
    for i in run_order(cfg):
        p, layer = f"l{i}.", cfg["layers"][i]
        y = mixers[layer["type"]](_r(rms_norm(x, w[p + "norm1"], eps)), w, p + "mix.", layer["mixer"], eps)
        x = x + rms_norm(y, w[p + "norm1b"], eps)
        if layer.get("mlp") is not None:
            y = routed_experts(_r(rms_norm(x, w[p + "norm2"], eps)), w, p + "mlp.", layer["mlp"])
            x = x + rms_norm(y, w[p + "norm2b"], eps)
        after.append(x)
    logits = _r(rms_norm(x, w["final.norm"], eps)) @ w["embed"].T
    return (logits, after) if return_layers else logits


def greedy(cfg, w, prompt, new_tokens, dtype=torch.float64):
    """The prompt's greedy continuation, every token from a whole pass over the sequence so far."""
    seq, out = list(prompt), []
    for _ in range(new_tokens):
        out.append(int(forward(cfg, w, seq, dtype)[-1].argmax()))
        seq.append(out[-1])
    return out
