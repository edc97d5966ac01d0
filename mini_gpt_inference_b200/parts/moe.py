"""Feed-forward of routed experts, with an optional expert that every token uses.

``z = W_router y`` in 32-bit; the ``top`` experts with the largest ``z`` are chosen and weighted
by the softmax over the chosen ``z`` alone.  An expert is a gated unit without biases,
``W_down (silu(W_gate y) * (W_up y))``; the part adds ``sum_k weight_k expert_k(y)`` to the
residual stream.  With ``shared_inner`` an expert of the same form (its own hidden width) runs for
every token and is added too, times ``sigmoid(w_sg . y)``, one number per token, if
``shared_gate``.

Variants, all parameters: ``scoring="sigmoid"`` scores every expert ``s = sigmoid(z)`` on its own and
weighs the chosen ones by ``route_scale * s`` without renormalising; ``correction`` adds a stored
vector to the scores for the choice only; ``groups=(count, keep)`` cuts the experts into ``count``
equal groups of neighbours, scores a group by the sum of its two largest choice scores and lets only
the experts of the best ``keep`` groups be chosen.  ``activation="clamped_swish"`` makes an expert
``W_down (g * sigmoid(1.702 g) * (u + 1))`` with ``g = min(W_gate y, limit)``,
``u = clamp(W_up y, -limit, limit)``; the shared expert has a limit of its own.

``weigh="input"`` puts a chosen expert's weight on what it reads instead of what it gives, ``expert_k(weight_k y)``.  (The
first product is linear, so the kernel multiplies its 32-bit sums, in front of the activation.)

``gated=False`` makes an expert a plain unit, ``W_down act(W_up y)`` (``activation``: ``relu_sq``, ``gelu_tanh`` or
``silu``; no ``gate`` tensors), and the shared expert of the same form.

A shared expert without a gate matrix, or one without a gate number per token, is cut into parts of its hidden features
as large as an expert's (the last one filled up with zero rows): since its output is a sum over hidden features, the
parts are experts that every token uses with the shared gate (or 1) as their weight, and the whole feed-forward is one
grouping and two grouped products, whose sum over a token's experts the norm behind the part can take on its way.

In the checkpoint expert ``e`` has ``e<e>.gate``, ``e<e>.up``, ``e<e>.down`` under the part's
prefix, the router ``router``, the shared expert ``shared.gate``, ``shared.up``, ``shared.down``
and ``shared.sg``.  When bound, the experts' matrices are stacked (``[E, 2F, C]`` with gate rows
first, ``[E, C, F]``), because the kernels walk them by expert number; the router and the shared
gate stay 32-bit.
"""

from __future__ import annotations

import torch

from .base import FeedForward, register_feed_forward
from .spec import TensorSpec


@register_feed_forward("routed_experts")
class RoutedExperts(FeedForward):
    graph_safe = True      # the tokens are grouped by expert on the device; the host decides nothing per step
    accepts_deferred_norm = False      # the router reads the normalised rows themselves
    GATED, PLAIN = ("silu", "clamped_swish"), ("relu_sq", "gelu_tanh", "silu")

    def __init__(self, prefix: str, width: int, n_experts: int, top: int, inner: int,
                 shared_inner: int | None = None, shared_gate: bool = True, scoring: str = "softmax_top",
                 route_scale: float = 1.0, correction: bool = False, groups: tuple | None = None,
                 activation: str = "silu", limit: float = 0.0, shared_limit: float | None = None,
                 init: str = "normal", gated: bool = True, weigh: str = "output") -> None:
        super().__init__(prefix)
        if not 0 < top <= n_experts:
            raise ValueError(f"top {top} must lie in 1..n_experts ({n_experts})")
        if scoring not in ("softmax_top", "sigmoid"):
            raise ValueError(f"scoring {scoring!r}: softmax_top or sigmoid")
        if activation not in (self.GATED if gated else self.PLAIN):
            raise ValueError(f"activation {activation!r}: one of {', '.join(self.GATED if gated else self.PLAIN)}")
        if not gated and (scoring != "softmax_top" or correction or groups is not None or route_scale != 1.0):
            raise ValueError("experts without a gate are chosen by the plain router")
        if groups is not None:
            count, keep = groups
            if n_experts % count or not 0 < keep <= count or keep * (n_experts // count) < top:
                raise ValueError(f"groups {groups!r} do not fit {n_experts} experts with {top} choices")
        if weigh not in ("output", "input"):
            raise ValueError(f"weigh {weigh!r}: output or input")
        if weigh == "input" and shared_inner is not None and shared_gate:
            raise ValueError("a gated shared expert beside experts whose input is weighed is not built")
        self.weigh = weigh
        self.scoring, self.route_scale, self.has_correction = scoring, float(route_scale), bool(correction)
        self.groups = None if groups is None else (int(groups[0]), int(groups[1]))
        self.activation, self.limit = activation, float(limit)
        self.shared_limit = self.limit if shared_limit is None else float(shared_limit)
        self._init = init
        self.correction = None
        self.width, self.n_experts, self.top, self.inner = width, n_experts, top, inner
        self.shared_inner = shared_inner
        self.gated = bool(gated)
        self.shared_gate = bool(shared_gate) and shared_inner is not None
        # the scores of a plain router: what takes experts that every token uses among the chosen ones
        self.plain_router = not self.has_correction and self.groups is None
        # a shared expert as experts that every token uses (see the module's description)
        folded = not gated or (self.plain_router and not self.shared_gate and activation == "silu")
        self.always = -(-shared_inner // inner) if folded and shared_inner is not None else 0
        self.returns_output = folded
        self.router = self.w_in = self.w_out = None
        self.shared_in = self.shared_out = self.shared_gate_weight = None

    def tensor_specs(self):
        p, c, f = self.prefix, self.width, self.inner
        init, init_out = self._init, ("residual_proj" if self._init == "normal" else self._init + "_residual")
        specs = {p + "router": TensorSpec((self.n_experts, c), "vector", init)}
        if self.has_correction:
            specs[p + "correction"] = TensorSpec((self.n_experts,), "vector", "norm_shift")
        for e in range(self.n_experts):
            if self.gated:
                specs[f"{p}e{e}.gate"] = TensorSpec((f, c), "matrix", init)
            specs[f"{p}e{e}.up"] = TensorSpec((f, c), "matrix", init)
            specs[f"{p}e{e}.down"] = TensorSpec((c, f), "matrix", init_out)
        if self.shared_inner is not None:
            s = self.shared_inner
            if self.gated:
                specs[p + "shared.gate"] = TensorSpec((s, c), "matrix", init)
            specs[p + "shared.up"] = TensorSpec((s, c), "matrix", init)
            specs[p + "shared.down"] = TensorSpec((c, s), "matrix", init_out)
            if self.shared_gate:
                specs[p + "shared.sg"] = TensorSpec((1, c), "vector", "normal")
        return specs

    def bind(self, tensors) -> None:
        p = self.prefix
        if tensors.get(p + "router") is None:
            return
        self.router = tensors[p + "router"]
        self.correction = tensors.get(p + "correction") if self.has_correction else None
        if self.shared_gate:
            self.shared_gate_weight = tensors[p + "shared.sg"].reshape(-1).contiguous()
        kinds = ("gate", "up") if self.gated else ("up",)
        ins = [torch.cat([tensors[f"{p}e{e}.{kind}"] for kind in kinds]) for e in range(self.n_experts)]
        downs = [tensors[f"{p}e{e}.down"] for e in range(self.n_experts)]
        for first in range(0, self.always * self.inner, self.inner):
            part = slice(first, first + self.inner)
            down = tensors[p + "shared.down"][:, part]
            fill = self.inner - down.shape[1]
            ins.append(torch.cat([torch.nn.functional.pad(tensors[f"{p}shared.{kind}"][part], (0, 0, 0, fill)) for kind in kinds]))
            downs.append(torch.nn.functional.pad(down, (0, fill)))
        self.w_in, self.w_out = torch.stack(ins).contiguous(), torch.stack(downs).contiguous()
        if self.shared_inner is not None and not self.always:
            self.shared_in = torch.cat([tensors[p + "shared.gate"], tensors[p + "shared.up"]], dim=0).contiguous()
            self.shared_out = tensors[p + "shared.down"]

    def forward(self, ctx, y, residual32):
        ops = ctx.ops
        extra = {} if self.gated else {"gated": False}
        if self.activation != "silu":
            extra.update(activation=self.activation, limit=self.limit)
        if self.weigh == "input":
            extra["weigh_input"] = True
        if self.plain_router:
            ids, weights, gate = ops.moe_route(y, self.router, self.shared_gate_weight, ctx.positions, self.top,
                                               always=self.always, scoring=self.scoring, scale=self.route_scale)
        else:
            ids, weights, gate = ops.moe_route_scored(y, self.router, self.shared_gate_weight, ctx.positions, self.top,
                                                      self.scoring, self.correction, self.groups, self.route_scale)
        if residual32 is None:
            return ops.moe_experts(y, ids, weights, self.w_in, self.w_out, **extra)
        ops.moe_experts_residual(y, ids, weights, self.w_in, self.w_out, residual32, **extra)
        if self.shared_inner is not None and not self.always:
            plain = self.activation == "silu"
            # the shared expert is an ordinary gated unit over all tokens: the projection kernels
            # serve it; its per-token gate rides on the hidden features (W (g h) = g (W h))
            hidden = ops.glu(ops.linear(y, self.shared_in, None, "none", ctx.act_dtype), gate,
                             **({} if plain else {"activation": self.activation, "limit": self.shared_limit}))
            ops.linear_residual(hidden, self.shared_out, None, residual32)
        return None
