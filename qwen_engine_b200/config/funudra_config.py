"""Configuration of the Funudra design, from the keys of its ``config.json``.

A Funudra model is a list of layers, each with one of two mixers beside an optional feed-forward (both read the same
stream, each through a norm of its own):

    {"architecture": "Funudra", "vocab": V, "width": W, "norm": {"eps": e},
     "layers": [{"type": "mamba2" | "parallel", "mixer": {...}, "mlp": null | {"kind": "dense", "ff": F},
                 "weights_of": j}, ...]}

``mamba2`` mixer sizes: heads, vdim (channels of a head), state, groups, conv (taps), norm_groups.
``parallel`` mixer: ``left`` (softmax attention: heads, kv_heads, dim, vdim, conv, scale, softcap, rot {base, dims,
scaling {factor}}), ``right`` (matrix memory: heads, dim, vdim, gate_cap), ``left_scale``, ``right_scale``.
``weights_of`` (optional): the layer whose tensors this one uses; its own caches are its own.  Every size and constant is
read from here.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass, field
from typing import Any, ClassVar

from .ganidra_config import _number
from .model_config import ConfigError, ModelConfig, _require_int

_MIXERS = ("mamba2", "parallel")


def _object(where: str, m: Any) -> dict:
    if not isinstance(m, dict):
        raise ConfigError(f"config.json: {where} must be an object")
    return m


def _check_state_space(where: str, m: Any) -> None:
    for key in ("heads", "vdim", "state", "groups", "conv", "norm_groups"):
        _require_int(f"{where}.{key}", _object(where, m).get(key))
    if m["heads"] % m["groups"]:
        raise ConfigError(f"config.json: {where}.heads ({m['heads']}) must be a multiple of groups ({m['groups']})")
    if (m["heads"] * m["vdim"]) % m["norm_groups"]:
        raise ConfigError(f"config.json: {where}: heads * vdim ({m['heads'] * m['vdim']}) must be a multiple of norm_groups ({m['norm_groups']})")


def _check_attention(where: str, m: Any) -> None:
    for key in ("heads", "kv_heads", "dim", "vdim", "conv"):
        _require_int(f"{where}.{key}", _object(where, m).get(key))
    if m["heads"] % m["kv_heads"]:
        raise ConfigError(f"config.json: {where}.heads ({m['heads']}) must be a multiple of kv_heads ({m['kv_heads']})")
    _number(f"{where}.scale", m.get("scale"))
    _number(f"{where}.softcap", m.get("softcap"))
    rot = _object(f"{where}.rot", m.get("rot"))
    _number(f"{where}.rot.base", rot.get("base"))
    dims = _require_int(f"{where}.rot.dims", rot.get("dims"))
    if dims % 2 or dims > m["dim"]:
        raise ConfigError(f"config.json: {where}.rot.dims ({dims}) must be even and at most dim ({m['dim']})")
    if rot.get("scaling") is not None:
        _number(f"{where}.rot.scaling.factor", _object(f"{where}.rot.scaling", rot["scaling"]).get("factor"))


def _check_memory(where: str, m: Any) -> None:
    for key in ("heads", "dim", "vdim"):
        _require_int(f"{where}.{key}", _object(where, m).get(key))
    _number(f"{where}.gate_cap", m.get("gate_cap"))


@dataclass
class FunudraConfig(ModelConfig):
    architecture: ClassVar[str] = "Funudra"

    vocab: int = 0
    width: int = 0
    norm_eps: float = 1e-6
    layers: tuple = ()                  # the config.json entries, checked
    eos_token_ids: tuple = field(default_factory=tuple)

    # what the engine asks of every configuration
    @property
    def vocab_size(self) -> int:
        return self.vocab

    @property
    def hidden_size(self) -> int:
        return self.width

    @classmethod
    def from_dict(cls, raw: dict[str, Any]) -> "FunudraConfig":
        for key in ("vocab", "width", "layers", "norm"):
            if key not in raw:
                raise ConfigError(f"config.json: '{key}' is missing")
        if not isinstance(raw["norm"], dict) or "eps" not in raw["norm"]:
            raise ConfigError("config.json: norm.eps is missing")
        if not isinstance(raw["layers"], list) or not raw["layers"]:
            raise ConfigError("config.json: 'layers' must be a list with at least one layer")
        eos = raw.get("eos_token_id")
        eos_all = tuple(int(t) for t in eos) if isinstance(eos, list) else (() if eos is None else (int(eos),))
        cfg = cls(vocab=_require_int("vocab", raw["vocab"]), width=_require_int("width", raw["width"]),
                  norm_eps=_number("norm.eps", raw["norm"]["eps"]), layers=tuple(copy.deepcopy(raw["layers"])), eos_token_ids=eos_all)
        cfg.validate()
        return cfg

    def to_dict(self) -> dict[str, Any]:
        out: dict[str, Any] = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width,
                               "norm": {"eps": self.norm_eps}, "layers": copy.deepcopy(list(self.layers))}
        if self.eos_token_ids:
            out["eos_token_id"] = list(self.eos_token_ids)
        return out

    def validate(self) -> None:
        for i, layer in enumerate(self.layers):
            where = f"layers[{i}]"
            _object(where, layer)
            kind, m = layer.get("type"), layer.get("mixer")
            if kind not in _MIXERS:
                raise ConfigError(f"config.json: {where}.type {kind!r} is not a mixer of this design; known: {list(_MIXERS)}")
            if kind == "mamba2":
                _check_state_space(f"{where}.mixer", m)
            else:
                _object(f"{where}.mixer", m)
                _check_attention(f"{where}.mixer.left", m.get("left"))
                _check_memory(f"{where}.mixer.right", m.get("right"))
                _number(f"{where}.mixer.left_scale", m.get("left_scale"), positive=False)
                _number(f"{where}.mixer.right_scale", m.get("right_scale"), positive=False)
            mlp = layer.get("mlp")
            if mlp is not None:
                if not isinstance(mlp, dict) or mlp.get("kind") != "dense":
                    raise ConfigError(f"config.json: {where}.mlp must be null or a 'dense' feed-forward, got {mlp!r}")
                _require_int(f"{where}.mlp.ff", mlp.get("ff"))
            src = layer.get("weights_of")
            if src is not None:
                if _require_int(f"{where}.weights_of", src, 0) >= len(self.layers):
                    raise ConfigError(f"config.json: {where}.weights_of ({src}) names no layer")
                other = self.layers[self.owner_of(i)]
                if any(layer.get(key) != other.get(key) for key in ("type", "mixer", "mlp")):
                    raise ConfigError(f"config.json: {where} uses the weights of layer {src} but is not like it")

    def owner_of(self, i: int) -> int:
        """The layer whose tensors layer i uses (itself, or the one ``weights_of`` leads to)."""
        seen = set()
        while self.layers[i].get("weights_of") is not None:
            if i in seen:
                raise ConfigError(f"config.json: layers[{i}].weights_of leads back to itself")
            seen.add(i)
            i = self.layers[i]["weights_of"]
            if not (0 <= i < len(self.layers)):
                raise ConfigError(f"config.json: weights_of ({i}) names no layer")
        return i
