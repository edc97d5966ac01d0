"""Typed configuration of the Vumotar decoder, read from its ``config.json``.

The file is nested: ``vocab``, ``width``, ``norm.eps``, an optional ``loop`` (``start``, ``stop``, ``times``) and a list
``layers``; each entry has ``type`` (the mixer's kind: ``attention``, ``attention_2`` or ``latent_attention``), ``mixer``
(its sizes and constants) and ``mlp`` (routed experts, or null for none).  Every size and constant is read from the
file; a missing key is an error, a key that this engine does not know a warning.
"""

from __future__ import annotations

import json
from dataclasses import dataclass
from pathlib import Path
from typing import Any, Mapping

from .fakilorn_config import _keys, _number, _positive_int
from .model_config import ConfigError

MIXER_TYPES = ("attention", "attention_2", "latent_attention")


def _positive(value, what: str) -> float:
    number = _number(value, what)
    if number <= 0:
        raise ConfigError(f"{what} must be positive, got {value!r}")
    return number


@dataclass(frozen=True)
class VumotarMixerConfig:
    """Sizes and constants of one mixer; fields that a kind does not have are None."""

    kind: str
    heads: int
    dim: int                                  # features of a query or key head
    vdim: int                                 # features of a value head
    scale: float                              # factor on the scores
    kv_heads: int | None = None               # attention, attention_2
    window: int | None = None                 # a query sees itself and the window - 1 tokens before it; None: all
    keep_first: int = 0                       # attention: first tokens of the sequence that stay in sight
    temp_coef: float | None = None            # attention_2: queries grow with the position (None: they do not)
    temp_every: float | None = None
    q_rank: int | None = None                 # latent attention: sizes of the latents behind the queries ...
    kv_rank: int | None = None                # ... and behind keys and values (the one that is cached)

    @classmethod
    def from_dict(cls, kind: str, raw, what: str) -> "VumotarMixerConfig":
        if kind == "latent_attention":
            _keys(raw, ("heads", "dim", "vdim", "kv_rank", "q_rank", "scale"), ("mask",), what)
        else:
            _keys(raw, ("heads", "kv_heads", "dim", "vdim", "scale"), ("mask",) if kind == "attention" else ("q_temp",), what)
        sizes = {k: _positive_int(raw[k], f"{what}.{k}") for k in ("heads", "dim", "vdim")}
        extra: dict[str, Any] = {}
        if kind == "latent_attention":
            extra.update(q_rank=_positive_int(raw["q_rank"], what + ".q_rank"),
                         kv_rank=_positive_int(raw["kv_rank"], what + ".kv_rank"))
        else:
            extra["kv_heads"] = _positive_int(raw["kv_heads"], what + ".kv_heads")
            if sizes["heads"] % extra["kv_heads"]:
                raise ConfigError(f"{what}: heads ({sizes['heads']}) must be a multiple of kv_heads ({extra['kv_heads']})")
        if kind != "attention_2" and raw.get("mask") is not None:
            mask = raw["mask"]
            _keys(mask, ("size",), ("keep_first",) if kind == "attention" else (), what + ".mask")
            extra["window"] = _positive_int(mask["size"], what + ".mask.size")
            keep = mask.get("keep_first", 0) if kind == "attention" else 0
            if not isinstance(keep, int) or isinstance(keep, bool) or keep < 0:
                raise ConfigError(f"{what}.mask.keep_first must be a number of tokens, got {keep!r}")
            extra["keep_first"] = keep
        if kind == "attention_2" and raw.get("q_temp") is not None:
            _keys(raw["q_temp"], ("coef", "every"), (), what + ".q_temp")
            extra.update(temp_coef=_number(raw["q_temp"]["coef"], what + ".q_temp.coef"),
                         temp_every=_positive(raw["q_temp"]["every"], what + ".q_temp.every"))
        return cls(kind, sizes["heads"], sizes["dim"], sizes["vdim"], _number(raw["scale"], what + ".scale"), **extra)

    def to_dict(self) -> dict:
        out: dict[str, Any] = {"dim": self.dim, "heads": self.heads, "scale": self.scale, "vdim": self.vdim}
        if self.kind == "latent_attention":
            out.update(kv_rank=self.kv_rank, q_rank=self.q_rank)
        else:
            out["kv_heads"] = self.kv_heads
        if self.window is not None:
            out["mask"] = {"size": self.window}
            if self.kind == "attention":
                out["mask"]["keep_first"] = self.keep_first
        if self.temp_coef is not None:
            out["q_temp"] = {"coef": self.temp_coef, "every": self.temp_every}
        return out

    def num_parameters(self, width: int) -> int:
        h = self.heads
        if self.kind == "latent_attention":
            return (width * (self.q_rank + self.kv_rank + h + h * self.vdim) + self.q_rank * (1 + h * self.dim)
                    + self.kv_rank * (1 + h * (self.dim + self.vdim)) + h)
        total = width * ((h + self.kv_heads) * self.dim + (h + self.kv_heads) * self.vdim)
        return total + 2 * self.dim if self.kind == "attention" else total


@dataclass(frozen=True)
class VumotarExpertsConfig:
    ff: int                            # hidden width of an expert
    experts: int
    top: int
    shared_ff: int | None = None       # hidden width of the expert that every token uses; None: there is none

    @classmethod
    def from_dict(cls, raw, what: str) -> "VumotarExpertsConfig":
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

    def num_parameters(self, width: int) -> int:
        return self.experts * width * (1 + 3 * self.ff) + 3 * width * (self.shared_ff or 0)


@dataclass(frozen=True)
class VumotarLayerConfig:
    type: str
    mixer: VumotarMixerConfig
    mlp: VumotarExpertsConfig | None

    @classmethod
    def from_dict(cls, raw, what: str) -> "VumotarLayerConfig":
        _keys(raw, ("type", "mixer"), ("mlp",), what)
        if raw["type"] not in MIXER_TYPES:
            raise ConfigError(f"{what}.type {raw['type']!r} is not a mixer of this design ({', '.join(MIXER_TYPES)})")
        mlp = raw.get("mlp")
        return cls(raw["type"], VumotarMixerConfig.from_dict(raw["type"], raw["mixer"], what + ".mixer"),
                   None if mlp is None else VumotarExpertsConfig.from_dict(mlp, what + ".mlp"))

    def to_dict(self) -> dict:
        return {"mixer": self.mixer.to_dict(), "mlp": None if self.mlp is None else self.mlp.to_dict(),
                "type": self.type}


@dataclass(frozen=True)
class VumotarConfig:
    vocab: int
    width: int
    layers: tuple[VumotarLayerConfig, ...]
    norm_eps: float
    loop_start: int = 0                    # layers loop_start .. loop_stop-1 run loop_times times in a row;
    loop_stop: int = 0                     # loop_times 0: the file names no loop
    loop_times: int = 0
    architecture: str = "Vumotar"

    @property
    def vocab_size(self) -> int:
        return self.vocab

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any], architecture: str | None = None) -> "VumotarConfig":
        _keys(raw, ("vocab", "width", "layers", "norm"),
              ("loop", "architecture", "architectures", "model_type", "dtype", "torch_dtype"), "config.json")
        _keys(raw["norm"], ("eps",), (), "norm")
        if not isinstance(raw["layers"], (list, tuple)) or not raw["layers"]:
            raise ConfigError("layers must be a list with at least one layer")
        layers = tuple(VumotarLayerConfig.from_dict(layer, f"layers[{i}]") for i, layer in enumerate(raw["layers"]))
        start = stop = times = 0
        loop = raw.get("loop")
        if loop is not None:
            _keys(loop, ("start", "stop", "times"), (), "loop")
            start, stop = loop["start"], loop["stop"]
            times = _positive_int(loop["times"], "loop.times")
            if not (isinstance(start, int) and isinstance(stop, int) and 0 <= start < stop <= len(layers)):
                raise ConfigError(f"loop: layers {start!r} .. {stop!r} are not a range of the {len(layers)} layers")
        return cls(_positive_int(raw["vocab"], "vocab"), _positive_int(raw["width"], "width"), layers,
                   _positive(raw["norm"]["eps"], "norm.eps"), start, stop, times, architecture or "Vumotar")

    @classmethod
    def from_json(cls, path: str | Path) -> "VumotarConfig":
        from .model_config import read_config_json

        path = Path(path)
        return cls.from_dict(read_config_json(path / "config.json" if path.is_dir() else path))

    def to_dict(self) -> dict[str, Any]:
        out: dict[str, Any] = {"architecture": self.architecture, "layers": [layer.to_dict() for layer in self.layers],
                               "norm": {"eps": self.norm_eps}, "vocab": self.vocab, "width": self.width}
        if self.loop_times:
            out["loop"] = {"start": self.loop_start, "stop": self.loop_stop, "times": self.loop_times}
        return out

    def run_order(self) -> list[int]:
        """The layers' numbers in the order they run."""
        order = list(range(self.loop_start, self.loop_stop)) * self.loop_times
        return [*range(self.loop_start), *order, *range(self.loop_stop, len(self.layers))]

    def num_parameters(self) -> int:
        c = self.width
        total = self.vocab * c + c
        for layer in self.layers:
            total += 2 * c + layer.mixer.num_parameters(c)
            if layer.mlp is not None:
                total += 2 * c + layer.mlp.num_parameters(c)
        return total

    def save(self, model_dir: str | Path) -> Path:
        model_dir = Path(model_dir)
        model_dir.mkdir(parents=True, exist_ok=True)
        path = model_dir / "config.json"
        path.write_text(json.dumps(self.to_dict(), indent=1) + "\n")
        return path
