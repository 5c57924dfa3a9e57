"""``Pifelix``'s own config.json keys as a typed configuration.

config.json names ``architecture`` (a string), ``vocab``, ``width``, ``norm.eps``, ``embedding.scale``,
``residual_mult`` (the factor on every sublayer's normed result) and ``layers``: one entry per layer with ``type``
(which mixer: "attention"), ``mixer`` and ``mlp`` (``{"kind": "moe", "expert": {"ff", "limit"}, "router": {"experts",
"top"}}``, or null for a layer without a feed-forward).

``attention``: ``heads``, ``kv_heads``, ``dim``, ``vdim``, ``scale``, ``conv`` (taps of the projections' convolutions),
``rot`` (``base``, ``dims`` and optionally ``scaling``: ``factor``, ``original``, ``fast``, ``slow``), ``mask.size`` (the
positions of a chunk; without ``mask`` every earlier key is seen) and optionally ``kv_from`` (the earlier layer whose
keys and values the layer reads instead of projecting its own).  Every size and constant the model uses comes from here
or from a tensor's shape.
"""

from __future__ import annotations

import copy
from dataclasses import dataclass, field
from typing import Any

from gllm_b200.config.model_config import DTYPE_NAMES, ConfigError, ModelConfig, as_eos, require

MIXER_KEYS = ("heads", "kv_heads", "dim", "vdim", "scale", "conv")
POSITIVE = ("heads", "kv_heads", "dim", "vdim", "conv")
SCALING_KEYS = ("factor", "original", "fast", "slow")


def _check_mixer(where: str, m: dict) -> None:
    for key in MIXER_KEYS:
        if key not in m:
            raise ConfigError(f"{where}.mixer lacks {key!r}")
        if key in POSITIVE and int(m[key]) <= 0:
            raise ConfigError(f"{where}.mixer.{key} must be positive")
    if int(m["heads"]) % int(m["kv_heads"]):
        raise ConfigError(f"{where}.mixer: heads is not a multiple of kv_heads")
    rot = m.get("rot")
    if rot is not None:
        if "base" not in rot or "dims" not in rot:
            raise ConfigError(f"{where}.mixer.rot needs 'base' and 'dims'")
        dims = int(rot["dims"])
        if dims % 2 or not 0 <= dims <= int(m["dim"]):
            raise ConfigError(f"{where}.mixer.rot.dims must be even and at most dim")
        scaling = rot.get("scaling")
        if scaling is not None:
            for key in SCALING_KEYS:
                if key not in scaling:
                    raise ConfigError(f"{where}.mixer.rot.scaling lacks {key!r}")
                if not float(scaling[key]) > 0:
                    raise ConfigError(f"{where}.mixer.rot.scaling.{key} must be positive")
    mask = m.get("mask")
    if mask is not None and int(require(mask, "size")) <= 0:
        raise ConfigError(f"{where}.mixer.mask.size must be positive")


def _check_mlp(where: str, mlp: dict) -> None:
    if mlp.get("kind") != "moe":
        raise ConfigError(f"{where}.mlp: unknown kind {mlp.get('kind')!r}; known: ['moe']")
    expert, router = require(mlp, "expert"), require(mlp, "router")
    if int(require(expert, "ff")) <= 0:
        raise ConfigError(f"{where}.mlp.expert.ff must be positive")
    if not float(require(expert, "limit")) > 0:
        raise ConfigError(f"{where}.mlp.expert.limit must be positive")
    experts, top = int(require(router, "experts")), int(require(router, "top"))
    if experts <= 0 or not 1 <= top <= experts:
        raise ConfigError(f"{where}.mlp.router: 1 <= top <= experts is needed")


@dataclass(frozen=True)
class PifelixLayer:
    type: str
    mixer: dict[str, Any]
    mlp: dict[str, Any] | None

    @classmethod
    def from_dict(cls, index: int, d: dict) -> "PifelixLayer":
        where = f"layers[{index}]"
        kind = require(d, "type")
        if kind != "attention":
            raise ConfigError(f"{where}: unknown layer type {kind!r}; known: ['attention']")
        mixer = require(d, "mixer")
        _check_mixer(where, mixer)
        mlp = d.get("mlp")
        if mlp is not None:
            _check_mlp(where, mlp)
        return cls(kind, copy.deepcopy(mixer), copy.deepcopy(mlp))

    def to_dict(self) -> dict:
        return {"type": self.type, "mixer": copy.deepcopy(self.mixer), "mlp": copy.deepcopy(self.mlp)}


@dataclass(frozen=True)
class PifelixConfig(ModelConfig):
    """A decoder of attention within chunks over convolved projections and clamped routed experts, every sublayer's
    result being normed before it joins the residual; layers may read an earlier layer's keys and values; the output head
    has a matrix of its own."""

    layers: tuple[PifelixLayer, ...] = field(default_factory=tuple)
    norm_eps: float = 0.0
    embedding_scale: float = 1.0
    residual_mult: float = 1.0

    @classmethod
    def from_dict(cls, d: dict[str, Any]) -> "PifelixConfig":
        arch = d.get("architecture") or (d.get("architectures") or [None])[0]
        raw = require(d, "layers")
        if not isinstance(raw, list) or not raw:
            raise ConfigError("'layers' must be a non-empty list")
        dtype = d.get("torch_dtype", d.get("dtype", "bfloat16"))
        if dtype not in DTYPE_NAMES:
            raise ConfigError(f"unsupported dtype {dtype!r}")
        vocab, width = int(require(d, "vocab")), int(require(d, "width"))
        if vocab <= 0 or width <= 0:
            raise ConfigError("'vocab' and 'width' must be positive")
        layers = tuple(PifelixLayer.from_dict(i, layer) for i, layer in enumerate(raw))
        for i, layer in enumerate(layers):
            source = layer.mixer.get("kv_from")
            if source is None:
                continue
            source = int(source)
            if not 0 <= source < i or layers[source].mixer.get("kv_from") is not None:
                raise ConfigError(f"layers[{i}].mixer.kv_from names {source}, which is not an earlier layer with keys of "
                                  "its own")
            for key in ("kv_heads", "dim", "vdim"):
                if int(layers[source].mixer[key]) != int(layer.mixer[key]):
                    raise ConfigError(f"layers[{i}].mixer.{key} differs from that of the layer whose keys it reads")
        return cls(
            architecture=str(arch), vocab_size=vocab, hidden_size=width, dtype=DTYPE_NAMES[dtype],
            eos_token_ids=as_eos(d.get("eos_token_id")), layers=layers,
            norm_eps=float(require(require(d, "norm"), "eps")),
            embedding_scale=float(require(require(d, "embedding"), "scale")),
            residual_mult=float(require(d, "residual_mult")),
        )

    def to_dict(self) -> dict[str, Any]:
        out: dict[str, Any] = {
            "architecture": self.architecture,
            "embedding": {"scale": self.embedding_scale},
            "layers": [layer.to_dict() for layer in self.layers],
            "norm": {"eps": self.norm_eps},
            "residual_mult": self.residual_mult,
            "torch_dtype": self.dtype,
            "vocab": self.vocab_size,
            "width": self.hidden_size,
        }
        if self.eos_token_ids:
            out["eos_token_id"] = list(self.eos_token_ids)
        return out
