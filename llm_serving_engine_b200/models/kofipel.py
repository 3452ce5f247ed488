"""The Kofipel design as a ``ModelSpec`` (``config/kofipel_config.py`` describes the design and its keys).

Tensor names: ``embed``, ``side.embed`` [vocab, layers * dim], ``head``, ``final.norm``; for layer i ``l<i>.norm1``,
``l<i>.canon1`` (the convolution of the mixer's input), ``l<i>.norm2`` and ``l<i>.canon2`` (the feed-forward's), ``l<i>.mix.*``
(attention: ``q q.b k k.b temp o o.b``; channel_delta: ``q k v`` each with ``.conv``, ``b A_log norm a1 a2 dt_bias g1 g2 o``),
``l<i>.mlp.{up,down}`` and ``l<i>.side.{gate,proj,norm}``.  Every mechanism is a registered part with its constants as
parameters: ``convolved_residual`` (block), ``rmsnorm``, ``head_norm_rotary_attention`` (without head norms; tied values,
head factors, kept first keys, unit sink), ``channel_delta_memory``, ``squared_relu_mlp``, ``gated_token_lookup``; the loop is
the ``ModelSpec``'s order and ``embedding_again``.
"""
from __future__ import annotations

from ..config.kofipel_config import KofipelConfig
from ..config.model_config import LayerSpec, ModelSpec, PartSpec
from ..config.registry import register_architecture

_SIDE_TABLE = "side.embed"


def _mixer_spec(kind: str, mixer: dict, eps: float) -> PartSpec:
    sizes = {key: int(mixer[key]) for key in ("heads", "kv_heads", "dim", "vdim")}
    if kind == "attention":
        mask = mixer.get("mask") or {}
        return PartSpec("head_norm_rotary_attention", {
            **sizes, "eps": eps, "scale": float(mixer["scale"]), "rot": mixer.get("rot"), "head_norm": False, "bias": True,
            "output_bias": True, "values": "keys", "head_factor": True, "unit_sink": True,
            "softcap": float(mixer.get("softcap", 0.0)), "window": int(mask.get("size", 0)),
            "keep_first": int(mask.get("keep_first", 0))})
    return PartSpec("channel_delta_memory", {**sizes, "eps": eps, "conv": int(mixer["conv"]),
                                             "decay_rank": int(mixer["decay_rank"]), "gate_rank": int(mixer["gate_rank"])})


def build_kofipel_spec(config: KofipelConfig) -> ModelSpec:
    norm = PartSpec("rmsnorm", {"eps": config.norm_eps, "weight_name": ""})
    layers = []
    for index, entry in enumerate(config.layers):
        mlp = entry.get("mlp")
        mixer = _mixer_spec(entry["type"], entry["mixer"], config.norm_eps)
        side = {"kind": "gated_token_lookup", "prefix": "side.",
                "params": {"dim": config.side_dim, "table": _SIDE_TABLE, "offset": index * config.side_dim, "eps": config.norm_eps}}
        block = PartSpec("convolved_residual", {
            "taps": config.taps, "conv_names": {"mixer": "canon1", "feed_forward": "canon2"},
            "mixer": {"kind": mixer.kind, "params": mixer.params}, "token_input": side, "feed_forward": mlp is not None,
            "tensor_prefixes": {"mixer_norm": "norm1", "mixer": "mix.", "feed_forward_norm": "norm2", "feed_forward": "mlp."}})
        layers.append(LayerSpec(
            prefix=f"l{index}.", block=block, mixer=mixer,
            feed_forward=None if mlp is None else PartSpec("squared_relu_mlp", {
                "intermediate_size": int(mlp["ff"]), "tensor_names": {"up": "up", "down": "down"}}),
            mixer_norm=norm, feed_forward_norm=None if mlp is None else norm))
    return ModelSpec(
        architecture="Kofipel", vocab_size=config.vocab, hidden_size=config.width, layers=tuple(layers), order=config.order,
        final_norm=norm, embedding_name="embed", final_norm_prefix="final.norm", lm_head_name="head",
        tie_word_embeddings=False, max_position_embeddings=config.max_position_embeddings,
        embedding_again=config.embedding_again,
        shared_tensors={_SIDE_TABLE: (config.vocab, len(config.layers) * config.side_dim)})


register_architecture("Kofipel", KofipelConfig, build_kofipel_spec, model_types=("kofipel",))
