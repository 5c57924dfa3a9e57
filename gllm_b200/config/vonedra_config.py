"""``Vonedra``'s own config.json keys as a typed configuration.

config.json names ``architecture`` (a string), ``vocab``, ``width``, ``norm.eps``, ``embedding.scale``, ``canon.taps``
(taps of the convolution every sublayer's input passes) and ``layers``: one entry per layer with ``type`` (which mixer:
"attention", "latent_attention" or "delta"), ``mixer`` (that mixer's sizes and constants) and ``mlp`` (``{"kind":
"dense", "ff": n}``, or null for a layer without a feed-forward).

``attention``: ``heads``, ``kv_heads``, ``dim``, ``vdim``, ``scale``, ``bias_max`` (the distance from which the last
bias row holds), optionally ``mask`` (``size``, ``keep_first``), ``v_mix`` (the layer's values are mixed with those of
the first layer that has it) and ``bias_rows`` (rows of the bias table: a checkpoint's tensor gives them, only the
random-weights mode needs them named).  ``latent_attention``: ``heads``, ``dim``, ``rot_dim``, ``vdim``, ``q_rank``,
``kv_rank``, ``scale``, ``rot`` (``base``, ``dims``), optionally ``mask.size``.  ``delta``: ``heads``, ``kv_heads``,
``dim``, ``vdim``, ``conv``.  Every size and constant the model uses comes from here or from a tensor's shape.
"""

from __future__ import annotations

import copy
from dataclasses import dataclass, field
from typing import Any

from gllm_b200.config.model_config import DTYPE_NAMES, ConfigError, ModelConfig, as_eos, require

MIXER_KEYS = {
    "attention": ("heads", "kv_heads", "dim", "vdim", "scale", "bias_max"),
    "latent_attention": ("heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank", "scale", "rot"),
    "delta": ("heads", "kv_heads", "dim", "vdim", "conv"),
}
POSITIVE = ("heads", "kv_heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank", "conv")


def _check_mixer(where: str, kind: str, m: dict) -> None:
    for key in MIXER_KEYS[kind]:
        if key not in m:
            raise ConfigError(f"{where}.mixer lacks {key!r}")
        if key in POSITIVE and int(m[key]) <= 0:
            raise ConfigError(f"{where}.mixer.{key} must be positive")
    if "kv_heads" in MIXER_KEYS[kind] and int(m["heads"]) % int(m["kv_heads"]):
        raise ConfigError(f"{where}.mixer: heads is not a multiple of kv_heads")
    mask = m.get("mask")
    if mask is not None:
        if int(require(mask, "size")) <= 0 or int(mask.get("keep_first", 0)) < 0:
            raise ConfigError(f"{where}.mixer.mask needs a positive size and a keep_first that is not negative")
        if kind != "attention" and int(mask.get("keep_first", 0)):
            raise ConfigError(f"{where}.mixer.mask: only 'attention' keeps first tokens")
    if kind == "attention":
        if not float(m["bias_max"]) > 0:
            raise ConfigError(f"{where}.mixer.bias_max must be positive")
        if "bias_rows" in m and not 0 < int(m["bias_rows"]) < 2 * float(m["bias_max"]):
            raise ConfigError(f"{where}.mixer.bias_rows must be positive and less than twice bias_max")
    if kind == "latent_attention":
        rot = m["rot"]
        if "base" not in rot or "dims" not in rot:
            raise ConfigError(f"{where}.mixer.rot needs 'base' and 'dims'")
        if int(rot["dims"]) % 2 or not 0 < int(rot["dims"]) <= int(m["rot_dim"]):
            raise ConfigError(f"{where}.mixer.rot.dims must be even, positive and at most rot_dim")


@dataclass(frozen=True)
class VonedraLayer:
    type: str
    mixer: dict[str, Any]
    mlp: dict[str, Any] | None

    @classmethod
    def from_dict(cls, index: int, d: dict) -> "VonedraLayer":
        where = f"layers[{index}]"
        kind = require(d, "type")
        if kind not in MIXER_KEYS:
            raise ConfigError(f"{where}: unknown layer type {kind!r}; known: {sorted(MIXER_KEYS)}")
        mixer = require(d, "mixer")
        _check_mixer(where, kind, mixer)
        mlp = d.get("mlp")
        if mlp is not None:
            if mlp.get("kind") != "dense":
                raise ConfigError(f"{where}.mlp: unknown kind {mlp.get('kind')!r}; known: ['dense']")
            if int(require(mlp, "ff")) <= 0:
                raise ConfigError(f"{where}.mlp.ff must be positive")
        return cls(kind, copy.deepcopy(mixer), copy.deepcopy(mlp))

    def to_dict(self) -> dict:
        return {"type": self.type, "mixer": copy.deepcopy(self.mixer), "mlp": copy.deepcopy(self.mlp)}


@dataclass(frozen=True)
class VonedraConfig(ModelConfig):
    """A decoder whose layers norm their sublayers' results, read the residual convolved over time and average over the
    depth of the model; the mixer is attention with a bias by distance, latent attention or a gated delta rule."""

    layers: tuple[VonedraLayer, ...] = field(default_factory=tuple)
    norm_eps: float = 0.0
    embedding_scale: float = 1.0
    conv_taps: int = 1

    def value_mixing_layers(self) -> list[int]:
        return [i for i, l in enumerate(self.layers) if l.type == "attention" and l.mixer.get("v_mix")]

    @classmethod
    def from_dict(cls, d: dict[str, Any]) -> "VonedraConfig":
        arch = d.get("architecture") or (d.get("architectures") or [None])[0]
        layers = require(d, "layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("'layers' must be a non-empty list")
        dtype = d.get("torch_dtype", d.get("dtype", "bfloat16"))
        if dtype not in DTYPE_NAMES:
            raise ConfigError(f"unsupported dtype {dtype!r}")
        vocab, width = int(require(d, "vocab")), int(require(d, "width"))
        if vocab <= 0 or width <= 0:
            raise ConfigError("'vocab' and 'width' must be positive")
        taps = int(require(require(d, "canon"), "taps"))
        if not 1 <= taps <= 16:
            raise ConfigError("'canon.taps' must lie between 1 and 16")
        cfg = cls(
            architecture=str(arch), vocab_size=vocab, hidden_size=width, dtype=DTYPE_NAMES[dtype],
            eos_token_ids=as_eos(d.get("eos_token_id")),
            layers=tuple(VonedraLayer.from_dict(i, layer) for i, layer in enumerate(layers)),
            norm_eps=float(require(require(d, "norm"), "eps")),
            embedding_scale=float(require(require(d, "embedding"), "scale")),
            conv_taps=taps,
        )
        mixing = cfg.value_mixing_layers()
        if len({int(cfg.layers[i].mixer["kv_heads"]) * int(cfg.layers[i].mixer["vdim"]) for i in mixing}) > 1:
            raise ConfigError("layers that mix their values with the first one's need values of its size")
        return cfg

    def to_dict(self) -> dict[str, Any]:
        out: dict[str, Any] = {
            "architecture": self.architecture,
            "canon": {"taps": self.conv_taps},
            "embedding": {"scale": self.embedding_scale},
            "layers": [layer.to_dict() for layer in self.layers],
            "norm": {"eps": self.norm_eps},
            "vocab": self.vocab_size,
            "width": self.hidden_size,
            "torch_dtype": self.dtype,
        }
        if self.eos_token_ids:
            out["eos_token_id"] = list(self.eos_token_ids)
        return out
