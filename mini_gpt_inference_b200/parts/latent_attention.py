"""Causal attention whose keys and values are made from one small latent per token.

``q = W_q h`` gives every head ``head_dim`` features that do not turn and ``rot_dim`` that turn with the
position (rotary; feature ``i`` pairs with ``i + rot_dim / 2``, angle ``position * rot_base ** (-2 i / rot_dim)``;
``rot_pairs="neighbours"`` pairs ``2i`` with ``2i + 1``, ``rot_scaling`` stretches the frequencies, see ``parts.rotary``).
``W_dkv h`` has ``kv_rank + rot_dim`` numbers: the first ``kv_rank``, RMS-normed with a gain, are the latent
``c``; the last ``rot_dim``, turned, are one key part that all heads share.  Head ``a``'s key is
``[W_uk,a c | shared part]``, its value ``W_uv,a c``, its score ``scale * (q_plain . k_plain + q_rot . k_rot)``;
softmax over positions up to the query's own (``window``: the last ``window`` of them, its own included; ``sink``: a
learned number per head whose exponential joins the denominator); the concatenated heads times ``sigmoid(W_g h)`` if
``gate`` (``"head"``: ``W_g h`` has one number per head, which all of the head's features share), then ``W_o``.

With ``q_rank`` the queries come from a latent of their own: ``c_q = W_dq h`` (``q_rank`` numbers, RMS-normed with a gain),
``q = W_uq c_q``; such heads do not turn (``rot_dim`` 0).  One kernel norms both latents of a token.

Only ``[c | shared part]`` is cached, one row per token whatever the number of heads.  Scores are taken
against those rows themselves: a query's plain part is first carried into the latent's space with its head's
key matrix, ``q_abs = W_uk,a^T q_plain`` (so ``q_abs . c = q_plain . (W_uk,a c)``), attention then runs with one
shared key head of ``kv_rank + rot_dim`` features whose first ``kv_rank`` are also the values, and the heads'
weighted latents are carried to value space with ``W_uv,a`` afterwards.  A layer with ``kv_source`` has no
``W_dkv``: it reads the rows that an earlier layer cached (the run order hands it that layer's cache, read-only),
with matrices, queries and everything else of its own.
"""

from __future__ import annotations

import torch

from ..cache.spec import PagedKVSpec
from .base import Mixer, register_mixer
from .rotary import SCALING_KEYS, rotary_frequencies
from .spec import TensorSpec

_DEFAULT_NAMES = {"q": "q", "q_down": "dq", "q_norm": "dq.norm", "q_up": "uq", "down": "dkv", "norm": "dkv.norm", "up_k": "uk", "up_v": "uv", "gate": "g", "sink": "sink", "out": "o"}


@register_mixer("latent_attention")
class LatentAttention(Mixer):
    graph_safe = True      # launches kernels only; nothing is decided on the host per step
    accepts_deferred_norm = True
    returns_output = True

    def __init__(self, prefix: str, width: int, n_head: int, head_dim: int, rot_dim: int, v_head_dim: int, kv_rank: int,
                 scale: float, eps: float, rot_base: float = 10000.0, gate: bool | str = True, own_latents: bool = True,
                 cache_page_tokens: int | None = None, cache_pages: int | None = None, names: dict | None = None,
                 init: str = "normal", rot_pairs: str = "halves", rot_scaling: dict | None = None,
                 window: int | None = None, sink: bool = False, q_rank: int | None = None, position=None) -> None:
        super().__init__(prefix)
        if rot_pairs not in ("halves", "neighbours"):
            raise ValueError(f"rot_pairs {rot_pairs!r}: halves or neighbours")
        if rot_scaling is not None and set(rot_scaling) != set(SCALING_KEYS):
            raise ValueError(f"rot_scaling: {', '.join(SCALING_KEYS)} (got {sorted(rot_scaling)})")
        if window is not None and not own_latents:
            raise ValueError("a layer that reads another layer's rows has that layer's window")
        if rot_dim < 0 or rot_dim % 2:
            raise ValueError(f"rot_dim {rot_dim}: an even number of features")
        if q_rank is not None and (rot_dim or not own_latents):
            raise ValueError("queries from a latent: heads that do not turn, in a layer that caches latents of its own")
        if gate not in (True, False, "head"):
            raise ValueError(f"gate {gate!r}: True, False or 'head'")
        self.width, self.n_head, self.head_dim, self.rot_dim = width, n_head, head_dim, rot_dim
        self.v_head_dim, self.kv_rank = v_head_dim, kv_rank
        self.scale, self.eps, self.rot_base = float(scale), float(eps), float(rot_base)
        self.has_gate, self.own_latents, self.head_gate = bool(gate), bool(own_latents), gate == "head"
        self.q_rank = q_rank
        self.cache_page_tokens, self.cache_pages = cache_page_tokens, cache_pages
        self.names = {**_DEFAULT_NAMES, **(names or {})}
        self._init = init
        self.rot_neighbours, self.rot_scaling = rot_pairs == "neighbours", rot_scaling
        self.window, self.has_sink = window, bool(sink)
        self.q_width = n_head * (head_dim + rot_dim)
        self.low_width = kv_rank + rot_dim if self.own_latents else 0
        self.o_width = n_head * v_head_dim
        first = self.q_width if q_rank is None else q_rank
        self.low_off, self.g_off = first, first + self.low_width
        self.g_width = n_head if self.head_gate else self.o_width
        self.row_dim = kv_rank + rot_dim                 # a cache row, and a query head as the attention sees it
        self.q_up = self.q_gain = None
        self.fused_weight = self.out_weight = self.up_k = self.up_v = self.latent_gain = self.freq = self.sinks = None
        self.rot_magnitude = 1.0

    def _name(self, which: str) -> str:
        return self.prefix + self.names[which]

    def tensor_specs(self):
        init, init_out = self._init, ("residual_proj" if self._init == "normal" else self._init + "_residual")
        specs = {
            self._name("up_k"): TensorSpec((self.n_head * self.head_dim, self.kv_rank), "matrix", "fan_in"),
            self._name("up_v"): TensorSpec((self.o_width, self.kv_rank), "matrix", "fan_in"),
            self._name("out"): TensorSpec((self.width, self.o_width), "matrix", init_out),
        }
        if self.q_rank is None:
            specs[self._name("q")] = TensorSpec((self.q_width, self.width), "matrix", init)
        else:
            specs[self._name("q_down")] = TensorSpec((self.q_rank, self.width), "matrix", init)
            specs[self._name("q_norm")] = TensorSpec((self.q_rank,), "vector", "norm_gain")
            specs[self._name("q_up")] = TensorSpec((self.q_width, self.q_rank), "matrix", "fan_in")
        if self.own_latents:
            specs[self._name("down")] = TensorSpec((self.low_width, self.width), "matrix", init)
            specs[self._name("norm")] = TensorSpec((self.kv_rank,), "vector", "norm_gain")
        if self.has_gate:
            specs[self._name("gate")] = TensorSpec((self.g_width, self.width), "matrix", init)
        if self.has_sink:
            specs[self._name("sink")] = TensorSpec((self.n_head,), "vector", "unit_normal")
        return specs

    def bind(self, tensors) -> None:
        rows = [tensors.get(self._name("q" if self.q_rank is None else "q_down"))]
        if self.own_latents:
            rows.append(tensors.get(self._name("down")))
        if self.has_gate:
            rows.append(tensors.get(self._name("gate")))
        # one matrix for the step's one projection [q | low | g]: a layout made once, when the weights arrive
        self.fused_weight = torch.cat(rows, dim=0).contiguous() if all(r is not None for r in rows) else None
        if self.q_rank is not None and self.fused_weight is not None:
            # one gate number per head: rows of zeros fill the projection up to whole 16-byte groups of outputs
            self.fused_weight = torch.nn.functional.pad(self.fused_weight, (0, 0, 0, -self.fused_weight.shape[0] % 8))
            self.q_gain, self.q_up = tensors.get(self._name("q_norm")), tensors.get(self._name("q_up"))
        self.out_weight = tensors.get(self._name("out"))
        self.up_k, self.up_v = tensors.get(self._name("up_k")), tensors.get(self._name("up_v"))
        self.latent_gain = tensors.get(self._name("norm")) if self.own_latents else None
        self.sinks = tensors.get(self._name("sink")) if self.has_sink else None
        if self.rot_dim and self.out_weight is not None:
            freq, self.rot_magnitude = rotary_frequencies(self.rot_dim, self.rot_base, self.rot_scaling)
            self.freq = torch.tensor(freq, dtype=torch.float64).to(dtype=torch.float32, device=self.out_weight.device)

    def cache_spec(self):
        """One key head of ``kv_rank + rot_dim`` features per token; its first ``kv_rank`` are the values.  (A layer
        that reads another layer's rows is never asked: the run order names that layer's cache entry.)"""
        if not self.own_latents:
            return None
        return PagedKVSpec(1, self.row_dim, self.window, self.cache_page_tokens, self.cache_pages, self.kv_rank,
                           values_in_keys=True)

    def forward(self, ctx, cache, y, residual32):
        ops = ctx.ops
        if cache is None:
            raise RuntimeError(f"{self.prefix}: no cache entry holds the latents this layer reads")
        proj = ops.linear(y, self.fused_weight, None, "none", ctx.act_dtype)
        # queries as the attention sees them: per head [W_uk^T q_plain | turned q_rot]
        plain = proj
        if self.q_rank is None:
            q = ops.latent_prepare(proj, self.n_head, 0, self.head_dim, self.rot_dim, self.low_off, self.kv_rank,
                                   self.latent_gain, self.eps, self.freq, cache if self.own_latents else None,
                                   ctx.slot_mapping[cache.group], ctx.positions, neighbours=self.rot_neighbours,
                                   magnitude=self.rot_magnitude)
        else:
            latent = ops.latent_pair_prepare(proj, 0, self.q_rank, self.q_gain, self.low_off, self.kv_rank,
                                             self.latent_gain, self.eps, cache, ctx.slot_mapping[cache.group], ctx.positions)
            plain, q = ops.linear(latent, self.q_up, None, "none", ctx.act_dtype), None
        q = ops.head_linear(plain, 0, self.head_dim + self.rot_dim, self.up_k, True, self.n_head, self.head_dim, self.kv_rank,
                            out=q, out_off=0, out_head=self.row_dim)
        mixed = ops.paged_attention_general(q, self.n_head, 1, self.row_dim, self.kv_rank, self.scale, cache, ctx,
                                            sinks=self.sinks)
        gate = proj[:, self.g_off: self.g_off + self.g_width] if self.has_gate else None
        heads = ops.head_linear(mixed, 0, self.kv_rank, self.up_v, False, self.n_head, self.kv_rank, self.v_head_dim,
                                gate=gate)
        return self.add_output(ctx, heads, self.out_weight, residual32)
