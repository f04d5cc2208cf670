"""Configuration of the Dugalix design: a list of layers, each a mixer and a feed-forward between norms on either side.

``config.json`` of this design is nested::

    {"architecture": "Dugalix", "vocab": V, "width": D, "residual_mult": m, "norm": {"eps": e},
     "layers": [{"type": "parallel" | "attention", "mixer": {...}, "mlp": {...} | null}, ...]}

Mixer sizes and constants:

``parallel``   ``left_scale, right_scale``; ``left`` (softmax attention): ``heads, kv_heads, dim, vdim, scale``, optional ``rot:
               {"dims", "base", "scaling": {"factor"}}`` and ``mask: {"size", "keep_first"}``; ``right`` (a matrix memory):
               ``heads, dim, vdim, gate_cap``.
``attention``  (sigmoid weights, the values are the keys) ``heads, kv_heads, dim, vdim = dim, scale``, optional ``rot`` and
               ``mask: {"size"}``.

Feed-forward: ``{"kind": "dense", "ff"}`` or ``{"kind": "moe", "expert": {"ff"}, "router": {"experts", "top", "identity",
"groups": {"count", "keep"}}, "shared": {"ff"}}``. Absent keys mean absent mechanisms: no ``rot`` (or ``dims`` 0) no rotation, no
``scaling`` plain frequencies, no ``mask`` every earlier key, no ``keep_first`` a window alone, no ``identity`` no identity
experts, no ``groups`` one group, no ``shared`` no shared expert, ``mlp: null`` no feed-forward. The design has no position
limit and no end-of-sequence token.
"""

from __future__ import annotations

import copy
import math
from dataclasses import dataclass, field
from typing import Any, ClassVar

from .model_config import ConfigError, ModelConfig, _number, _object, _positive, _take

MIXER_TYPES = ("attention", "parallel")


@dataclass(frozen=True)
class DugalixConfig(ModelConfig):
    norm_eps: float = 0.0
    residual_mult: float = 1.0
    layers: tuple[dict[str, Any], ...] = field(default_factory=tuple)

    ARCHITECTURE: ClassVar[str] = "Dugalix"
    MODEL_TYPE: ClassVar[str] = "dugalix"

    @classmethod
    def from_json_dict(cls, raw: dict[str, Any]) -> "DugalixConfig":
        norm = raw.get("norm")
        if not isinstance(norm, dict):
            raise ConfigError("config.json key 'norm' must be an object")
        layers = raw.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("config.json key 'layers' must be a non-empty list")
        config = cls(
            architecture=cls.ARCHITECTURE,
            vocab_size=_take(raw, "vocab", int),
            hidden_size=_take(raw, "width", int),
            num_hidden_layers=len(layers),
            max_position_embeddings=cls.MAX_POSITIONS,
            eos_token_ids=(),
            norm_eps=_take(norm, "eps", float),
            residual_mult=_take(raw, "residual_mult", float, 1.0),
            layers=tuple(copy.deepcopy(layer) for layer in layers),
        )
        config.validate()
        return config

    def validate(self) -> None:
        super().validate()
        if not (math.isfinite(self.norm_eps) and self.norm_eps > 0):
            raise ConfigError(f"norm.eps={self.norm_eps} must be finite and positive")
        if not math.isfinite(self.residual_mult):
            raise ConfigError(f"residual_mult={self.residual_mult} must be finite")
        for index, layer in enumerate(self.layers):
            where = f"layers[{index}]"
            if not isinstance(layer, dict) or layer.get("type") not in MIXER_TYPES:
                raise ConfigError(f"{where}.type must be one of {sorted(MIXER_TYPES)}")
            mixer = _object(layer, "mixer", where)
            where += ".mixer"
            if layer["type"] == "parallel":
                _number(mixer, "left_scale", where), _number(mixer, "right_scale", where)
                self._validate_attention(_object(mixer, "left", where), where + ".left")
                right = _object(mixer, "right", where)
                _positive(right, ("heads", "dim", "vdim"), where + ".right")
                _number(right, "gate_cap", where + ".right", above=0.0)
            else:
                self._validate_attention(mixer, where)
                if mixer["vdim"] != mixer["dim"]:
                    raise ConfigError(f"{where}: the values are the keys, so vdim={mixer['vdim']} must equal dim={mixer['dim']}")
            if layer.get("mlp") is not None:
                self._validate_mlp(layer["mlp"], f"layers[{index}].mlp")

    @staticmethod
    def _validate_attention(mixer: dict, where: str) -> None:
        _positive(mixer, ("heads", "kv_heads", "dim", "vdim"), where)
        _number(mixer, "scale", where)
        if mixer["heads"] % mixer["kv_heads"]:
            raise ConfigError(f"{where}: heads={mixer['heads']} is not a multiple of kv_heads={mixer['kv_heads']}")
        mask = _object(mixer, "mask", where, optional=True)
        if mask is not None:
            _positive(mask, ("size",), where + ".mask")
            if _take(mask, "keep_first", int, 0) < 0:
                raise ConfigError(f"{where}.mask.keep_first cannot be negative")
        rot = _object(mixer, "rot", where, optional=True)
        if rot is not None:
            dims = _take(rot, "dims", int)
            if dims % 2 or not 0 <= dims <= mixer["dim"]:
                raise ConfigError(f"{where}.rot.dims={dims} must be even and at most dim={mixer['dim']}")
            _number(rot, "base", where + ".rot", above=0.0)
            scaling = _object(rot, "scaling", where + ".rot", optional=True)
            if scaling is not None:
                _number(scaling, "factor", where + ".rot.scaling", above=0.0)

    def _validate_mlp(self, mlp: Any, where: str) -> None:
        if not isinstance(mlp, dict) or mlp.get("kind") not in ("dense", "moe"):
            raise ConfigError(f"{where}.kind must be 'dense' or 'moe' (or mlp null)")
        parts = {"mlp": mlp} if mlp["kind"] == "dense" else {"expert": mlp.get("expert"), "shared": mlp.get("shared")}
        for name, part in parts.items():
            if part is None and name == "shared":
                continue
            if not isinstance(part, dict) or not 0 < _take(part, "ff", int) <= self.MAX_INTERMEDIATE:
                raise ConfigError(f"{where}: ff of '{name}' is missing or out of range")
        if mlp["kind"] == "dense":
            return
        router = _object(mlp, "router", where)
        experts, top, identity = _take(router, "experts", int), _take(router, "top", int), _take(router, "identity", int, 0)
        if experts <= 0 or identity < 0 or not 0 < top <= experts + identity:
            raise ConfigError(f"{where}.router: top={top} of {experts} experts and {identity} identity experts")
        groups = _object(router, "groups", where + ".router", optional=True)
        if groups is not None:
            _positive(groups, ("count", "keep"), where + ".router.groups")
            count, keep = groups["count"], groups["keep"]
            if (experts + identity) % count or keep > count or top > keep * ((experts + identity) // count):
                raise ConfigError(f"{where}.router: top={top} out of {keep} of {count} groups of {experts + identity} experts")

    def to_json_dict(self) -> dict[str, Any]:
        return {
            "architecture": self.architecture,
            "vocab": self.vocab_size,
            "width": self.hidden_size,
            "residual_mult": self.residual_mult,
            "norm": {"eps": self.norm_eps},
            "layers": [copy.deepcopy(layer) for layer in self.layers],
        }
