"""Typed configuration of the Nogatar decoder, read from its ``config.json``.

The file is nested: ``vocab``, ``width``, ``embedding.scale``, ``norm.eps``, ``residual_mult``, ``logit_softcap`` and a list
``layers``; each entry has ``type`` (the mixer's kind: ``latent_attention`` or ``mlstm``), ``mixer`` (its sizes and
constants) and ``mlp`` (routed experts, or null for none).  Every size and constant is read from the file; a missing key
is an error, a key that this engine does not know a warning.
"""

from __future__ import annotations

import json
from dataclasses import dataclass
from pathlib import Path
from typing import Any, Mapping

from .fakilorn_config import _keys, _number, _positive_int
from .model_config import ConfigError

MIXER_TYPES = ("latent_attention", "mlstm")


def _positive(value, what: str) -> float:
    number = _number(value, what)
    if number <= 0:
        raise ConfigError(f"{what} must be positive, got {value!r}")
    return number


@dataclass(frozen=True)
class RotaryScalingConfig:
    """Stretched rotary frequencies (YaRN)."""

    factor: float             # how far slow pairs are slowed
    original: float           # positions over which turns are counted
    fast: float               # pairs of more turns keep their frequency
    slow: float               # pairs of fewer turns are slowed by the whole factor

    @classmethod
    def from_dict(cls, raw, what: str) -> "RotaryScalingConfig":
        _keys(raw, ("factor", "original", "fast", "slow"), (), what)
        return cls(*(_positive(raw[k], f"{what}.{k}") for k in ("factor", "original", "fast", "slow")))

    def to_dict(self) -> dict:
        return {"factor": self.factor, "fast": self.fast, "original": self.original, "slow": self.slow}


@dataclass(frozen=True)
class NogatarMixerConfig:
    """Sizes and constants of one mixer; fields that a kind does not have are None."""

    kind: str
    heads: int
    dim: int                                           # latent attention: the part of a head that does not turn
    vdim: int
    gate_cap: float | None = None                      # mlstm: cap on the logarithms of its gates
    kv_rank: int | None = None                         # latent attention: size of the cached latent
    rot_dim: int | None = None                         # ... of the turning part of queries and of the shared key part
    rot_base: float | None = None
    rot_scaling: RotaryScalingConfig | None = None
    scale: float | None = None                         # factor on the scores
    window: int | None = None                          # a query sees itself and the window - 1 tokens before it

    @classmethod
    def from_dict(cls, kind: str, raw, what: str) -> "NogatarMixerConfig":
        if kind == "mlstm":
            _keys(raw, ("heads", "dim", "vdim", "gate_cap"), (), what)
            return cls(kind, _positive_int(raw["heads"], what + ".heads"), _positive_int(raw["dim"], what + ".dim"),
                       _positive_int(raw["vdim"], what + ".vdim"), gate_cap=_positive(raw["gate_cap"], what + ".gate_cap"))
        _keys(raw, ("heads", "dim", "vdim", "kv_rank", "rot_dim", "rot", "scale"), ("mask",), what)
        rot_dim, rot = raw["rot_dim"], raw["rot"]
        if not isinstance(rot_dim, int) or isinstance(rot_dim, bool) or rot_dim < 0 or rot_dim % 2:
            raise ConfigError(f"{what}.rot_dim must be an even number of features, got {rot_dim!r}")
        _keys(rot, ("base", "dims"), ("scaling",), what + ".rot")
        if rot["dims"] != rot_dim:
            raise ConfigError(f"{what}: the turning part has {rot_dim} features, rot.dims says {rot['dims']!r}")
        base, scaling = _positive(rot["base"], what + ".rot.base"), rot.get("scaling")
        if scaling is not None:
            scaling = RotaryScalingConfig.from_dict(scaling, what + ".rot.scaling")
            if base == 1.0:
                raise ConfigError(f"{what}.rot: frequencies of base 1 cannot be stretched")
        window = None
        if raw.get("mask") is not None:
            _keys(raw["mask"], ("size",), (), what + ".mask")
            window = _positive_int(raw["mask"]["size"], what + ".mask.size")
        return cls(kind, _positive_int(raw["heads"], what + ".heads"), _positive_int(raw["dim"], what + ".dim"),
                   _positive_int(raw["vdim"], what + ".vdim"), kv_rank=_positive_int(raw["kv_rank"], what + ".kv_rank"),
                   rot_dim=rot_dim, rot_base=base, rot_scaling=scaling, scale=_number(raw["scale"], what + ".scale"),
                   window=window)

    def to_dict(self) -> dict:
        out: dict[str, Any] = {"dim": self.dim, "heads": self.heads, "vdim": self.vdim}
        if self.kind == "mlstm":
            out["gate_cap"] = self.gate_cap
            return out
        rot: dict[str, Any] = {"base": self.rot_base, "dims": self.rot_dim}
        if self.rot_scaling is not None:
            rot["scaling"] = self.rot_scaling.to_dict()
        out.update(kv_rank=self.kv_rank, rot=rot, rot_dim=self.rot_dim, scale=self.scale)
        if self.window is not None:
            out["mask"] = {"size": self.window}
        return out


@dataclass(frozen=True)
class NogatarExpertsConfig:
    ff: int                            # hidden width of an expert
    experts: int
    top: int
    shared_ff: int | None = None       # hidden width of the expert that every token uses; None: there is none

    @classmethod
    def from_dict(cls, raw, what: str) -> "NogatarExpertsConfig":
        if not isinstance(raw, Mapping) or raw.get("kind") != "moe":
            raise ConfigError(f"{what} must be an object of kind 'moe', got {raw!r}")
        _keys(raw, ("kind", "expert", "router"), ("shared",), what)
        _keys(raw["expert"], ("ff",), (), what + ".expert")
        _keys(raw["router"], ("experts", "top"), (), what + ".router")
        experts, top = _positive_int(raw["router"]["experts"], what + ".router.experts"), _positive_int(raw["router"]["top"], what + ".router.top")
        if top > experts:
            raise ConfigError(f"{what}: top ({top}) exceeds experts ({experts})")
        shared = raw.get("shared")
        if shared is not None:
            _keys(shared, ("ff",), (), what + ".shared")
            shared = _positive_int(shared["ff"], what + ".shared.ff")
        return cls(_positive_int(raw["expert"]["ff"], what + ".expert.ff"), experts, top, shared)

    def to_dict(self) -> dict:
        out: dict[str, Any] = {"expert": {"ff": self.ff}, "kind": "moe", "router": {"experts": self.experts, "top": self.top}}
        if self.shared_ff is not None:
            out["shared"] = {"ff": self.shared_ff}
        return out


@dataclass(frozen=True)
class NogatarLayerConfig:
    type: str
    mixer: NogatarMixerConfig
    mlp: NogatarExpertsConfig | None

    @classmethod
    def from_dict(cls, raw, what: str) -> "NogatarLayerConfig":
        _keys(raw, ("type", "mixer"), ("mlp",), what)
        if raw["type"] not in MIXER_TYPES:
            raise ConfigError(f"{what}.type {raw['type']!r} is not a mixer of this design ({', '.join(MIXER_TYPES)})")
        mlp = raw.get("mlp")
        return cls(raw["type"], NogatarMixerConfig.from_dict(raw["type"], raw["mixer"], what + ".mixer"),
                   None if mlp is None else NogatarExpertsConfig.from_dict(mlp, what + ".mlp"))

    def to_dict(self) -> dict:
        return {"mixer": self.mixer.to_dict(), "mlp": None if self.mlp is None else self.mlp.to_dict(),
                "type": self.type}


@dataclass(frozen=True)
class NogatarConfig:
    vocab: int
    width: int
    layers: tuple[NogatarLayerConfig, ...]
    norm_eps: float
    embedding_scale: float
    residual_mult: float                   # factor on what a sublayer adds, behind its norm
    logit_softcap: float | None = None     # logits <- cap * tanh(logits / cap); None: as they are
    architecture: str = "Nogatar"

    @property
    def vocab_size(self) -> int:
        return self.vocab

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any], architecture: str | None = None) -> "NogatarConfig":
        _keys(raw, ("vocab", "width", "layers", "norm", "embedding", "residual_mult"),
              ("logit_softcap", "architecture", "architectures", "model_type", "dtype", "torch_dtype"), "config.json")
        _keys(raw["norm"], ("eps",), (), "norm")
        _keys(raw["embedding"], ("scale",), (), "embedding")
        if not isinstance(raw["layers"], (list, tuple)) or not raw["layers"]:
            raise ConfigError("layers must be a list with at least one layer")
        layers = tuple(NogatarLayerConfig.from_dict(layer, f"layers[{i}]") for i, layer in enumerate(raw["layers"]))
        cap = raw.get("logit_softcap")
        return cls(_positive_int(raw["vocab"], "vocab"), _positive_int(raw["width"], "width"), layers,
                   _positive(raw["norm"]["eps"], "norm.eps"), _number(raw["embedding"]["scale"], "embedding.scale"),
                   _number(raw["residual_mult"], "residual_mult"),
                   None if cap is None else _positive(cap, "logit_softcap"), architecture or "Nogatar")

    @classmethod
    def from_json(cls, path: str | Path) -> "NogatarConfig":
        from .model_config import read_config_json

        path = Path(path)
        return cls.from_dict(read_config_json(path / "config.json" if path.is_dir() else path))

    def to_dict(self) -> dict[str, Any]:
        out: dict[str, Any] = {"architecture": self.architecture, "embedding": {"scale": self.embedding_scale},
                               "layers": [layer.to_dict() for layer in self.layers], "norm": {"eps": self.norm_eps},
                               "residual_mult": self.residual_mult, "vocab": self.vocab, "width": self.width}
        if self.logit_softcap is not None:
            out["logit_softcap"] = self.logit_softcap
        return out

    def num_parameters(self) -> int:
        c = self.width
        total = 2 * self.vocab * c + c
        for layer in self.layers:
            m, f = layer.mixer, layer.mlp
            total += c
            if m.kind == "mlstm":
                n, nv = m.heads * m.dim, m.heads * m.vdim
                total += c * (2 * n + 3 * nv + 2 * m.heads) + 2 * m.heads + nv
            else:
                total += (m.heads * (m.dim + m.rot_dim) + m.kv_rank + m.rot_dim + m.heads * m.vdim) * c
                total += m.kv_rank * (1 + m.heads * (m.dim + m.vdim)) + m.heads
            if f is not None:
                total += c + f.experts * (c + 2 * c * f.ff)
                if f.shared_ff is not None:
                    total += c + 2 * c * f.shared_ff
        return total

    def save(self, model_dir: str | Path) -> Path:
        model_dir = Path(model_dir)
        model_dir.mkdir(parents=True, exist_ok=True)
        path = model_dir / "config.json"
        path.write_text(json.dumps(self.to_dict(), indent=1) + "\n")
        return path
