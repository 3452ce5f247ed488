"""Typed ``config.json`` of the Kofipel design.

Kofipel is a pre-norm decoder that lists its layers one by one.  What a sublayer reads is h + conv(h): the normed rows and a
short causal convolution of them per channel.  A layer's token mixer is ``attention`` (a window that keeps the sequence's
first tokens, values that are the unrotated keys, biases, a learned factor per head on capped scores, one more unit in the
softmax's denominator) or ``channel_delta`` (a matrix memory that decays per key channel and writes the difference to what it
holds); its feed-forward is dense with a squared relu, or absent; behind it the layer adds a normed projection of a gated
vector that a table holds per token and layer.  A range of layers may run several times with the same tensors, each pass
with caches of its own, the embedding's output added again before every pass but the first.  The output head is a
matrix of its own.

Keys: ``architecture`` ("Kofipel"), ``vocab``, ``width``, ``norm.eps``, ``canon.taps``, ``token_side.dim``, ``loop {start,
stop, times}`` and ``layers`` (a list of ``{"type", "mixer", "mlp"}``; attention mixer: ``heads, kv_heads, dim, vdim, scale,
softcap, mask {size, keep_first}, rot {base, dims}``; channel_delta mixer: ``heads, kv_heads, dim, vdim, conv``; mlp:
``kind`` "dense" with ``ff``, or null).  The ranks of a channel_delta layer's two low-rank maps are the first dimensions of
its ``mix.a1`` and ``mix.g1`` tensors; without a checkpoint they are read from the mixer's ``decay_rank`` and ``gate_rank``.
``max_position_embeddings`` is this engine's own optional key (the design has no limit of its own; the cache manager
wants one for its tables).
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any

from .model_config import ConfigError

_MIXER_KEYS = {
    "attention": ("heads", "kv_heads", "dim", "vdim", "scale"),
    "channel_delta": ("heads", "kv_heads", "dim", "vdim", "conv"),
}
_RANKS = (("decay_rank", "a1"), ("gate_rank", "g1"))


@dataclass(frozen=True)
class KofipelConfig:
    vocab: int
    width: int
    layers: tuple
    norm_eps: float
    taps: int
    side_dim: int
    loop_start: int = 0
    loop_stop: int = 0
    loop_times: int = 1
    max_position_embeddings: int = 131_072

    def __post_init__(self) -> None:
        if self.vocab <= 0 or self.width <= 0 or not self.layers:
            raise ConfigError("vocab, width and the number of layers must be positive")
        if not self.norm_eps > 0:
            raise ConfigError("norm.eps must be positive")
        if self.taps < 1 or self.side_dim < 1:
            raise ConfigError("canon.taps and token_side.dim must be at least 1")
        if not 0 <= self.loop_start <= self.loop_stop <= len(self.layers) or self.loop_times < 1:
            raise ConfigError("loop must name a range of the layers and run it at least once")
        for index, layer in enumerate(self.layers):
            kind = layer.get("type")
            if kind not in _MIXER_KEYS:
                raise ConfigError(f"layer {index}: unknown type {kind!r}; known: {list(_MIXER_KEYS)}")
            mixer = layer.get("mixer") or {}
            missing = [key for key in _MIXER_KEYS[kind] if key not in mixer]
            if missing:
                raise ConfigError(f"layer {index} ({kind}): mixer lacks {missing}")
            if int(mixer["kv_heads"]) < 1 or int(mixer["heads"]) % int(mixer["kv_heads"]):
                raise ConfigError(f"layer {index}: heads must be a multiple of kv_heads")
            if kind == "attention":
                if int(mixer["dim"]) != int(mixer["vdim"]):
                    raise ConfigError(f"layer {index}: the values are the keys, so vdim must equal dim")
                rot = mixer.get("rot")
                if rot and (int(rot["dims"]) % 2 or int(rot["dims"]) > int(mixer["dim"])):
                    raise ConfigError(f"layer {index}: rot.dims must be even and at most dim")
                if "softcap" in mixer and not float(mixer["softcap"]) > 0:
                    raise ConfigError(f"layer {index}: softcap must be positive")
                mask = mixer.get("mask")
                if mask and (int(mask["size"]) < 1 or int(mask.get("keep_first", 0)) < 0):
                    raise ConfigError(f"layer {index}: mask.size must be at least 1, mask.keep_first at least 0")
            else:
                if int(mixer["conv"]) < 1:
                    raise ConfigError(f"layer {index}: conv must be at least 1")
                for key, tensor in _RANKS:
                    if int(mixer.get(key, 0)) <= 0:
                        raise ConfigError(f"layer {index}: the rank of {tensor} is neither in the checkpoint nor in mixer.{key}")
            mlp = layer.get("mlp")
            if mlp is not None and (mlp.get("kind") != "dense" or int(mlp.get("ff", 0)) <= 0):
                raise ConfigError(f"layer {index}: mlp must be null or dense with a positive ff")

    @property
    def order(self) -> tuple[int, ...]:
        looped = tuple(range(self.loop_start, self.loop_stop))
        return tuple(range(self.loop_start)) + looped * self.loop_times + tuple(range(self.loop_stop, len(self.layers)))

    @property
    def embedding_again(self) -> tuple[int, ...]:
        """Positions in ``order`` of the first layer of every pass but the first."""
        length = self.loop_stop - self.loop_start
        return tuple(self.loop_start + turn * length for turn in range(1, self.loop_times)) if length else ()

    @classmethod
    def from_dict(cls, values: dict[str, Any], tensor_shapes: dict | None = None) -> "KofipelConfig":
        missing = [key for key in ("vocab", "width", "layers", "norm", "canon", "token_side") if key not in values]
        if missing:
            raise ConfigError(f"config.json lacks required keys: {missing}")
        for section, key in (("norm", "eps"), ("canon", "taps"), ("token_side", "dim")):
            if key not in values[section]:
                raise ConfigError(f"config.json lacks {section}.{key}")
        layers = []
        for index, layer in enumerate(values["layers"]):
            if layer.get("type") == "channel_delta" and tensor_shapes is not None:      # sizes that only the tensors give
                found = {key: int(tensor_shapes[f"l{index}.mix.{tensor}"][0]) for key, tensor in _RANKS
                         if f"l{index}.mix.{tensor}" in tensor_shapes}
                layer = {**layer, "mixer": {**layer["mixer"], **found}}
            layers.append(layer)
        loop = values.get("loop") or {}
        return cls(vocab=int(values["vocab"]), width=int(values["width"]), layers=tuple(layers),
                   norm_eps=float(values["norm"]["eps"]), taps=int(values["canon"]["taps"]),
                   side_dim=int(values["token_side"]["dim"]), loop_start=int(loop.get("start", 0)),
                   loop_stop=int(loop.get("stop", 0)), loop_times=int(loop.get("times", 1)),
                   max_position_embeddings=int(values.get("max_position_embeddings", 131_072)))
