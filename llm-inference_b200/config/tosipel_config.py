"""Configuration of the Tosipel design: a list of layers, each a mixer and a feed-forward whose outputs are normed.

``config.json`` of this design is nested::

    {"architecture": "Tosipel", "vocab": V, "width": D, "embedding": {"scale": s}, "norm": {"eps": e},
     "layers": [{"type": "attention" | "latent_attention" | "delta", "mixer": {...},
                 "mlp": {"kind": "dense", "ff": F} | null, "weights_of": j (optional)}, ...]}

Mixer sizes and constants:

``attention``         ``heads, kv_heads, dim, vdim, scale``, optional ``rot: {"dims", "base"}`` and ``mask: {"size"}``.
``latent_attention``  ``heads, dim, vdim, kv_rank, q_rank, scale``.
``delta``             ``heads, kv_heads, dim, vdim, conv``.

A layer with ``weights_of: j`` runs layer ``j``'s tensors against a cache or state of its own. Absent keys mean absent
mechanisms: no ``embedding.scale`` a factor of one, no ``rot`` (or ``dims`` 0) no rotation, no ``mask`` every earlier key,
``mlp: null`` no feed-forward. The design has no position limit and no end-of-sequence token.
"""

from __future__ import annotations

import copy
import math
from dataclasses import dataclass, field
from typing import Any, ClassVar

from .model_config import ConfigError, ModelConfig, _number, _object, _positive, _take

MIXER_SIZES = {
    "attention": ("heads", "kv_heads", "dim", "vdim"),
    "latent_attention": ("heads", "dim", "vdim", "kv_rank", "q_rank"),
    "delta": ("heads", "kv_heads", "dim", "vdim", "conv"),
}


@dataclass(frozen=True)
class TosipelConfig(ModelConfig):
    norm_eps: float = 0.0
    embedding_scale: float = 1.0
    layers: tuple[dict[str, Any], ...] = field(default_factory=tuple)

    ARCHITECTURE: ClassVar[str] = "Tosipel"
    MODEL_TYPE: ClassVar[str] = "tosipel"

    @classmethod
    def from_json_dict(cls, raw: dict[str, Any]) -> "TosipelConfig":
        layers = raw.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("config.json key 'layers' must be a non-empty list")
        norm = _object(raw, "norm", "config.json")
        embedding = _object(raw, "embedding", "config.json", optional=True) or {}
        config = cls(
            architecture=cls.ARCHITECTURE,
            vocab_size=_take(raw, "vocab", int),
            hidden_size=_take(raw, "width", int),
            num_hidden_layers=len(layers),
            max_position_embeddings=cls.MAX_POSITIONS,
            eos_token_ids=(),
            norm_eps=_take(norm, "eps", float),
            embedding_scale=_take(embedding, "scale", float, 1.0),
            layers=tuple(copy.deepcopy(layer) for layer in layers),
        )
        config.validate()
        return config

    def owner(self, index: int) -> int:
        """The layer whose tensors layer ``index`` runs (itself unless it names another)."""
        seen = set()
        while self.layers[index].get("weights_of") is not None:
            if index in seen:
                raise ConfigError(f"layers[{index}].weights_of runs in a circle")
            seen.add(index)
            index = int(self.layers[index]["weights_of"])
        return index

    def validate(self) -> None:
        super().validate()
        if not (math.isfinite(self.norm_eps) and self.norm_eps > 0):
            raise ConfigError(f"norm.eps={self.norm_eps} must be finite and positive")
        if not math.isfinite(self.embedding_scale):
            raise ConfigError(f"embedding.scale={self.embedding_scale} must be finite")
        for index, layer in enumerate(self.layers):
            where = f"layers[{index}]"
            if not isinstance(layer, dict) or layer.get("type") not in MIXER_SIZES:
                raise ConfigError(f"{where}.type must be one of {sorted(MIXER_SIZES)}")
            mixer = _object(layer, "mixer", where)
            self._validate_mixer(layer["type"], mixer, where + ".mixer")
            mlp = _object(layer, "mlp", where, optional=True)
            if mlp is not None:
                if mlp.get("kind") != "dense":
                    raise ConfigError(f"{where}.mlp.kind must be 'dense' (or mlp null)")
                if not 0 < _take(mlp, "ff", int) <= self.MAX_INTERMEDIATE:
                    raise ConfigError(f"{where}.mlp.ff is out of range")
        for index, layer in enumerate(self.layers):
            other = layer.get("weights_of")
            if other is None:
                continue
            where = f"layers[{index}]"
            if isinstance(other, bool) or not isinstance(other, int) or not 0 <= other < len(self.layers) or other == index:
                raise ConfigError(f"{where}.weights_of must name another layer")
            if any(self.layers[other].get(key) != layer.get(key) for key in ("type", "mixer", "mlp")):
                raise ConfigError(f"{where} runs layer {other}'s tensors, so its type, mixer and mlp must equal that layer's")
        for index in range(len(self.layers)):
            self.owner(index)

    @staticmethod
    def _validate_mixer(kind: str, mixer: dict, where: str) -> None:
        _positive(mixer, MIXER_SIZES[kind], where)
        if kind != "latent_attention" and mixer["heads"] % mixer["kv_heads"]:
            raise ConfigError(f"{where}: heads={mixer['heads']} is not a multiple of kv_heads={mixer['kv_heads']}")
        if kind != "delta":
            _number(mixer, "scale", where)
        if kind != "attention":
            return
        mask = _object(mixer, "mask", where, optional=True)
        if mask is not None:
            _positive(mask, ("size",), where + ".mask")
        rot = _object(mixer, "rot", where, optional=True)
        if rot is not None:
            dims = _take(rot, "dims", int)
            if dims % 2 or not 0 <= dims <= mixer["dim"]:
                raise ConfigError(f"{where}.rot.dims={dims} must be even and at most dim={mixer['dim']}")
            _number(rot, "base", where + ".rot", above=0.0)

    def to_json_dict(self) -> dict[str, Any]:
        return {
            "architecture": self.architecture,
            "vocab": self.vocab_size,
            "width": self.hidden_size,
            "embedding": {"scale": self.embedding_scale},
            "norm": {"eps": self.norm_eps},
            "layers": [copy.deepcopy(layer) for layer in self.layers],
        }
