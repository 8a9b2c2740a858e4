"""Configuration of the Zugunex design, from the keys of its ``config.json``.

A Zugunex model is a list of layers whose sublayers read the stream itself and norm what they return; every mixer is
latent attention, every feed-forward absent, dense or a mixture of experts with a shared one:

    {"architecture": "Zugunex", "vocab": V, "width": W, "norm": {"eps": e},
     "layers": [{"type": "latent_attention",
                 "mixer": {"heads", "dim", "rot_dim", "vdim", "kv_rank", "scale", "mask": {"size": w},
                           "rot": {"base", "dims"}, "kv_from": j (absent: the layer has a latent of its own)},
                 "mlp": null | {"kind": "dense", "ff": F}
                      | {"kind": "moe", "expert": {"ff": F}, "router": {"experts": E, "top": k, "scale": s},
                         "shared": {"ff": G}}}, ...]}

A mixer with ``kv_from`` reads layer j's latent and rotated key part out of layer j's cache; the two layers' windows may
differ.  Every size and constant is read from here.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass, field
from typing import Any, ClassVar

from .ganidra_config import _number
from .model_config import ConfigError, ModelConfig, _require_int

_MIXERS = ("latent_attention",)


def _check_mixer(where: str, m: Any) -> None:
    if not isinstance(m, dict):
        raise ConfigError(f"config.json: {where} must be an object")
    for key in ("heads", "dim", "rot_dim", "vdim", "kv_rank"):
        _require_int(f"{where}.{key}", m.get(key))
    _number(f"{where}.scale", m.get("scale"))
    rot = m.get("rot")
    if not isinstance(rot, dict):
        raise ConfigError(f"config.json: {where}.rot must be an object with 'base' and 'dims'")
    _number(f"{where}.rot.base", rot.get("base"))
    dims = _require_int(f"{where}.rot.dims", rot.get("dims"), 2)
    if dims % 2 or dims > m["rot_dim"]:
        raise ConfigError(f"config.json: {where}.rot.dims ({dims}) must be even and at most rot_dim ({m['rot_dim']})")
    mask = m.get("mask")
    if mask is not None:                            # (absent or null: every earlier token is seen)
        if not isinstance(mask, dict):
            raise ConfigError(f"config.json: {where}.mask must be an object with 'size'")
        _require_int(f"{where}.mask.size", mask.get("size"))


def _check_mlp(where: str, mlp: Any) -> None:
    if mlp is None:
        return
    if not isinstance(mlp, dict) or mlp.get("kind") not in ("dense", "moe"):
        raise ConfigError(f"config.json: {where} must be null, a 'dense' or a 'moe' feed-forward, got {mlp!r}")
    if mlp["kind"] == "dense":
        _require_int(f"{where}.ff", mlp.get("ff"))
        return
    expert, router, shared = mlp.get("expert"), mlp.get("router"), mlp.get("shared")
    if not isinstance(expert, dict) or not isinstance(router, dict):
        raise ConfigError(f"config.json: {where} needs 'expert' and 'router' objects")
    _require_int(f"{where}.expert.ff", expert.get("ff"))
    experts = _require_int(f"{where}.router.experts", router.get("experts"))
    top = _require_int(f"{where}.router.top", router.get("top"))
    if top > experts:
        raise ConfigError(f"config.json: {where}.router.top ({top}) exceeds its experts ({experts})")
    _number(f"{where}.router.scale", router.get("scale"), positive=False)
    if shared is not None:
        if not isinstance(shared, dict):
            raise ConfigError(f"config.json: {where}.shared must be an object with 'ff'")
        _require_int(f"{where}.shared.ff", shared.get("ff"))


@dataclass
class ZugunexConfig(ModelConfig):
    architecture: ClassVar[str] = "Zugunex"

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
    def from_dict(cls, raw: dict[str, Any]) -> "ZugunexConfig":
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
            if not isinstance(layer, dict):
                raise ConfigError(f"config.json: {where} must be an object")
            kind = layer.get("type")
            if kind not in _MIXERS:
                raise ConfigError(f"config.json: {where}.type {kind!r} is not a mixer of this design; known: {list(_MIXERS)}")
            m = layer.get("mixer")
            _check_mixer(f"{where}.mixer", m)
            _check_mlp(f"{where}.mlp", layer.get("mlp"))
            j = m.get("kv_from")
            if j is None:
                continue
            if not isinstance(j, int) or isinstance(j, bool) or not (0 <= j < i):
                raise ConfigError(f"config.json: {where}.mixer.kv_from ({j!r}) must name an earlier layer")
            src = self.layers[j]["mixer"]
            if src.get("kv_from") is not None:
                raise ConfigError(f"config.json: {where}.mixer.kv_from names layer {j}, which has no latent of its own")
            for key in ("kv_rank", "rot_dim"):
                if src[key] != m[key]:
                    raise ConfigError(f"config.json: {where}.mixer.{key} ({m[key]}) differs from layer {j}'s ({src[key]}), whose latent it reads")
            if (float(src["rot"]["base"]), src["rot"]["dims"]) != (float(m["rot"]["base"]), m["rot"]["dims"]):
                raise ConfigError(f"config.json: {where}.mixer.rot differs from layer {j}'s, whose rotated key part it reads")
