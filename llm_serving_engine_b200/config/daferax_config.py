"""Typed ``config.json`` of the Daferax design.

Daferax is a decoder whose sublayers read the residual itself and whose outputs are layer-normed before the residual takes
them: x <- x + norm(sublayer(x)).  A layer's token mixer is ``attention`` (heads of q and k RMS-normed one by one and rotated
in neighbouring pairs, plain causal softmax, a gate per head, values mixed with those of the first layer that mixes) or
``latent_attention`` (queries projected directly, keys and values of all heads made from one cached latent, one rotated key
part that the heads share, a sliding window, a gate per output element); its feed-forward is a mixture of silu-gated experts
(softmax scores, the choice confined to the groups with the best expert, weights not renormalised, times a constant) with a
shared expert that every token uses, or absent.  The output head is the embedding table.

Keys: ``architecture`` ("Daferax"), ``vocab``, ``width``, ``norm.eps``, ``layers`` (a list of ``{"type", "mixer", "mlp"}``;
attention mixer: ``heads, kv_heads, dim, vdim, scale, rot {base, dims}, v_mix``; latent_attention mixer: ``heads, dim, rot_dim,
vdim, kv_rank, scale, mask {size}, rot {base, dims, scaling {factor, original, fast, slow}}``; mlp: ``kind`` "moe" with
``router {experts, top, scale, groups {count, keep}}``, ``expert {ff}`` and ``shared {ff}``, or null).
``max_position_embeddings`` is this engine's own optional key (the design has no limit of its own; the cache manager wants
one for its tables).
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any

from .model_config import ConfigError

MIXER_TYPES = ("attention", "latent_attention")
_MIXER_KEYS = {
    "attention": ("heads", "kv_heads", "dim", "vdim", "scale"),
    "latent_attention": ("heads", "dim", "rot_dim", "vdim", "kv_rank", "scale", "rot"),
}


def _check_rotation(where: str, rot: dict, limit: int, what: str) -> None:
    if "base" not in rot or "dims" not in rot:
        raise ConfigError(f"{where}: rot needs base and dims")
    if int(rot["dims"]) % 2 or not 0 <= int(rot["dims"]) <= limit:
        raise ConfigError(f"{where}: rot.dims must be even and at most {what}")
    scaling = rot.get("scaling")
    if scaling and any(key not in scaling for key in ("factor", "original", "fast", "slow")):
        raise ConfigError(f"{where}: rot.scaling needs factor, original, fast and slow")


def _check_mixture(where: str, mlp: dict) -> None:
    if mlp.get("kind", "moe") != "moe":
        raise ConfigError(f"{where}: mlp.kind must be 'moe', got {mlp.get('kind')!r}")
    router = mlp.get("router") or {}
    if "experts" not in router or "top" not in router or int((mlp.get("expert") or {}).get("ff", 0)) <= 0:
        raise ConfigError(f"{where}: the mixture lacks router.experts, router.top or expert.ff")
    experts, top = int(router["experts"]), int(router["top"])
    if not 0 < top <= experts:
        raise ConfigError(f"{where}: router.top must lie in 1 .. experts")
    if mlp.get("shared") and int(mlp["shared"].get("ff", 0)) <= 0:
        raise ConfigError(f"{where}: shared.ff must be positive")
    groups = router.get("groups")
    if groups:
        count, keep = int(groups["count"]), int(groups["keep"])
        if count <= 0 or experts % count or not 0 < keep <= count:
            raise ConfigError(f"{where}: router.groups must divide the experts, keep in 1 .. count")
        if keep * (experts // count) < top:
            raise ConfigError(f"{where}: the kept groups hold fewer experts than router.top")


@dataclass(frozen=True)
class DaferaxConfig:
    vocab: int
    width: int
    layers: tuple
    norm_eps: float
    max_position_embeddings: int = 131_072

    def __post_init__(self) -> None:
        if self.vocab <= 0 or self.width <= 0 or not self.layers:
            raise ConfigError("vocab, width and the number of layers must be positive")
        if not self.norm_eps > 0:
            raise ConfigError("norm.eps must be positive")
        mixed: dict[int, tuple[int, int]] = {}     # layers that mix values: their number of values per token
        for index, layer in enumerate(self.layers):
            kind = layer.get("type")
            if kind not in MIXER_TYPES:
                raise ConfigError(f"layer {index}: unknown type {kind!r}; known: {list(MIXER_TYPES)}")
            mixer, where = layer.get("mixer") or {}, f"layer {index} ({kind})"
            missing = [key for key in _MIXER_KEYS[kind] if key not in mixer]
            if missing:
                raise ConfigError(f"{where}: mixer lacks {missing}")
            if kind == "attention":
                if int(mixer["heads"]) % int(mixer["kv_heads"]):
                    raise ConfigError(f"{where}: heads must be a multiple of kv_heads")
                if mixer.get("rot"):
                    _check_rotation(where, mixer["rot"], int(mixer["dim"]), "dim")
                if mixer.get("v_mix"):
                    mixed[index] = (int(mixer["kv_heads"]), int(mixer["vdim"]))
            else:
                _check_rotation(where, mixer["rot"], int(mixer["rot_dim"]), "rot_dim")
                if mixer.get("mask") and int(mixer["mask"].get("size", 0)) <= 0:
                    raise ConfigError(f"{where}: mask.size must be positive")
            if layer.get("mlp") is not None:
                _check_mixture(where, layer["mlp"])
        if len(set(mixed.values())) > 1:
            raise ConfigError(f"layers {sorted(mixed)} mix values of different shapes")

    @property
    def first_mixing_layer(self) -> int | None:
        """The layer whose values the later mixing layers take in."""
        return next((index for index, layer in enumerate(self.layers)
                     if layer["type"] == "attention" and layer["mixer"].get("v_mix")), None)

    @classmethod
    def from_dict(cls, values: dict[str, Any]) -> "DaferaxConfig":
        missing = [key for key in ("vocab", "width", "layers", "norm") if key not in values]
        if missing:
            raise ConfigError(f"config.json lacks required keys: {missing}")
        if "eps" not in values["norm"]:
            raise ConfigError("config.json lacks norm.eps")
        return cls(vocab=int(values["vocab"]), width=int(values["width"]), layers=tuple(values["layers"]),
                   norm_eps=float(values["norm"]["eps"]),
                   max_position_embeddings=int(values.get("max_position_embeddings", 131_072)))
