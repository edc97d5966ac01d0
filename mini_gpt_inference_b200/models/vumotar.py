"""The Vumotar decoder as data: which part sits in which layer, and in which order layers run.

Token embedding without positions; layers with a norm on both sides of each sublayer; a mixer per layer out of three:
attention with normed query and key heads, a sliding window that keeps the sequence's first tokens in sight and one
more term of 1 in the softmax's denominator; attention over everything earlier whose queries grow with the logarithm
of their position; attention over cached latents whose queries come from a latent of their own, with a sliding window,
a learned sink per head and one gate number per head; routed experts with a sigmoid score each, which scales the
chosen expert's input, and an expert that every token uses, or no feed-forward; a range of layers that runs several
times with the same weights, every pass with a cache of its own; a final norm and a head that shares the embedding's
matrix.  Tensor names: ``embed``, ``l<i>.norm1``, ``l<i>.mix.*``, ``l<i>.norm1b``, ``l<i>.norm2``, ``l<i>.mlp.*``,
``l<i>.norm2b``, ``final.norm``.
"""

from __future__ import annotations

from ..config.registry import register_model
from ..config.vumotar_config import VumotarConfig
from ..parts.spec import LayerCall, LayerSpec, ModelSpec, PartSpec


def _norm(cfg: VumotarConfig, name: str, optional: bool = False) -> PartSpec:
    return PartSpec("rmsnorm", {"width": cfg.width, "eps": cfg.norm_eps, "offset": 0.0, "weight_name": name,
                                "optional": optional}, "", "norm")


def _mixer(cfg: VumotarConfig, m) -> PartSpec:
    if m.kind == "latent_attention":
        return PartSpec("latent_attention", {
            "width": cfg.width, "n_head": m.heads, "head_dim": m.dim, "rot_dim": 0, "v_head_dim": m.vdim,
            "kv_rank": m.kv_rank, "q_rank": m.q_rank, "scale": m.scale, "eps": cfg.norm_eps, "gate": "head",
            "window": m.window, "sink": True, "init": "fan_in"}, "mix")
    params = {"width": cfg.width, "n_head": m.heads, "n_kv_head": m.kv_heads, "head_dim": m.dim, "v_head_dim": m.vdim,
              "scale": m.scale, "eps": cfg.norm_eps, "gate": False, "init": "fan_in"}
    if m.kind == "attention":
        params.update(unit_norm=True, norm_weights=True, window=m.window, keep_first=m.keep_first, unit_sink=True)
    else:
        params.update(unit_norm=False, query_temperature=None if m.temp_coef is None else (m.temp_coef, m.temp_every))
    return PartSpec("gated_unit_attention", params, "mix")


@register_model("Vumotar", "vumotar", config_class=VumotarConfig)
def describe_vumotar(cfg: VumotarConfig) -> ModelSpec:
    layers = []
    for i, layer in enumerate(cfg.layers):
        p, f = f"l{i}.", layer.mlp
        parts = {"norm1": _norm(cfg, p + "norm1"), "mixer": _mixer(cfg, layer.mixer), "norm1b": _norm(cfg, p + "norm1b")}
        # (a checkpoint may still hold the feed-forward's norms of a layer without one)
        parts["norm2"], parts["norm2b"] = _norm(cfg, p + "norm2", f is None), _norm(cfg, p + "norm2b", f is None)
        if f is not None:
            parts["feed_forward"] = PartSpec("routed_experts", {
                "width": cfg.width, "n_experts": f.experts, "top": f.top, "inner": f.ff, "shared_inner": f.shared_ff,
                "shared_gate": False, "scoring": "sigmoid", "weigh": "input", "init": "fan_in"}, "mlp")
        layers.append(LayerSpec(p, parts, "sandwich_norm"))
    # every run of a layer has a cache entry of its own
    order = tuple(LayerCall(i, n) for n, i in enumerate(cfg.run_order()))
    return ModelSpec(
        architecture=cfg.architecture,
        width=cfg.width,
        vocab_size=cfg.vocab,
        embedding=PartSpec("token_embedding", {"vocab_size": cfg.vocab, "width": cfg.width, "tensor_name": "embed",
                                               "init": "fan_in"}, ""),
        position=PartSpec("none", {}, ""),
        layers=tuple(layers),
        layer_order=order,
        final_norm=_norm(cfg, "final.norm"),
        head=PartSpec("tied_head", {"vocab_size": cfg.vocab, "width": cfg.width, "tied_to": "embed",
                                    "stored_again": False}, ""),
        n_caches=len(order))
