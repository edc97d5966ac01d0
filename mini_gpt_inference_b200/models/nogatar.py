"""The Nogatar decoder as data: which part sits in which layer.

A scaled token embedding without positions; layers whose sublayers read the residual stream itself and whose outputs pass
a layer norm (a gain, no shift) and a factor before they join it; a mixer per layer out of two: attention over cached
latents with neighbouring features rotated, stretched frequencies, a sliding window and a sink in the softmax, or an
mLSTM matrix memory; routed experts without a gate (squared ReLU) and a gated expert of the same form for every token,
or no feed-forward; a final layer norm, an untied head and a soft cap on the logits.  Tensor names: ``embed``,
``l<i>.norm1``, ``l<i>.mix.*``, ``l<i>.norm2``, ``l<i>.mlp.*``, ``final.norm``, ``head``.
"""

from __future__ import annotations

from ..config.nogatar_config import NogatarConfig
from ..config.registry import register_model
from ..parts.spec import LayerCall, LayerSpec, ModelSpec, PartSpec


def _norm(cfg: NogatarConfig, name: str, optional: bool = False) -> PartSpec:
    return PartSpec("layernorm", {"width": cfg.width, "eps": cfg.norm_eps, "bias": False, "gain_name": name,
                                  "optional": optional}, "", "norm")


def _mixer(cfg: NogatarConfig, m) -> PartSpec:
    if m.kind == "mlstm":
        return PartSpec("mlstm", {"width": cfg.width, "n_head": m.heads, "head_dim": m.dim, "v_head_dim": m.vdim,
                                  "gate_cap": m.gate_cap, "eps": cfg.norm_eps}, "mix")
    return PartSpec("latent_attention", {
        "width": cfg.width, "n_head": m.heads, "head_dim": m.dim, "rot_dim": m.rot_dim, "v_head_dim": m.vdim,
        "kv_rank": m.kv_rank, "scale": m.scale, "eps": cfg.norm_eps, "rot_base": m.rot_base, "rot_pairs": "neighbours",
        "rot_scaling": None if m.rot_scaling is None else m.rot_scaling.to_dict(), "gate": False, "window": m.window,
        "sink": True, "init": "fan_in"}, "mix")


@register_model("Nogatar", "nogatar", config_class=NogatarConfig)
def describe_nogatar(cfg: NogatarConfig) -> ModelSpec:
    layers = []
    for i, layer in enumerate(cfg.layers):
        p, f = f"l{i}.", layer.mlp
        parts = {"norm1": _norm(cfg, p + "norm1"), "mixer": _mixer(cfg, layer.mixer)}
        # (a checkpoint may still hold the second norm of a layer without a feed-forward)
        parts["norm2"] = _norm(cfg, p + "norm2", optional=f is None)
        if f is not None:
            parts["feed_forward"] = PartSpec("routed_experts", {
                "width": cfg.width, "n_experts": f.experts, "top": f.top, "inner": f.ff, "shared_inner": f.shared_ff,
                "shared_gate": True, "activation": "relu_sq", "gated": False, "init": "fan_in"}, "mlp")
        layers.append(LayerSpec(p, parts, "post_norm", {"residual_scale": cfg.residual_mult}))
    return ModelSpec(
        architecture=cfg.architecture,
        width=cfg.width,
        vocab_size=cfg.vocab,
        embedding=PartSpec("token_embedding", {"vocab_size": cfg.vocab, "width": cfg.width, "scale": cfg.embedding_scale,
                                               "tensor_name": "embed", "init": "fan_in"}, ""),
        position=PartSpec("none", {}, ""),
        layers=tuple(layers),
        layer_order=tuple(LayerCall(i, i) for i in range(len(layers))),
        final_norm=_norm(cfg, "final.norm"),
        head=PartSpec("linear_head", {"vocab_size": cfg.vocab, "width": cfg.width, "tensor_name": "head",
                                      "softcap": cfg.logit_softcap}, ""))
