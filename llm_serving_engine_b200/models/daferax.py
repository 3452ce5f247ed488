"""The Daferax design as a ``ModelSpec`` (``config/daferax_config.py`` describes the design and its keys).

Tensor names: ``embed`` (also the head), ``final.norm``, ``final.norm.b``; for layer i ``l<i>.norm1``, ``l<i>.norm2`` (each with
``.b``), ``l<i>.mix.*`` (attention: ``q k v g o q.norm k.norm vmix``; latent_attention: ``q dkv dkv.norm uk uv g o``) and
``l<i>.mlp.*`` (``router e<j>.{gate,up,down} shared.{gate,up,down}``).  Every mechanism is a registered part with its constants
as parameters: ``normed_branch_residual`` (block), ``layernorm``, ``head_norm_rotary_attention`` (neighbouring pairs, gates,
mixed values), ``latent_attention`` (a window, a gate per element), ``routed_experts`` (softmax scores within groups, a shared
expert without a gate).
"""
from __future__ import annotations

from ..config.daferax_config import DaferaxConfig
from ..config.model_config import LayerSpec, ModelSpec, PartSpec
from ..config.registry import register_architecture


def _mixer_spec(kind: str, mixer: dict, eps: float, is_first: bool) -> PartSpec:
    if kind == "attention":
        return PartSpec("head_norm_rotary_attention", {
            "heads": int(mixer["heads"]), "kv_heads": int(mixer["kv_heads"]), "dim": int(mixer["dim"]),
            "vdim": int(mixer["vdim"]), "scale": float(mixer["scale"]), "eps": eps, "rot": mixer.get("rot"),
            "pairing": "neighbours", "gate": True,
            "value_mix": ("first" if is_first else "later") if mixer.get("v_mix") else None})
    return PartSpec("latent_attention", {
        "heads": int(mixer["heads"]), "dim": int(mixer["dim"]), "rot_dim": int(mixer["rot_dim"]),
        "vdim": int(mixer["vdim"]), "kv_rank": int(mixer["kv_rank"]), "q_rank": 0, "scale": float(mixer["scale"]),
        "rot": dict(mixer["rot"]), "eps": eps, "gate": "elements",
        "window": int((mixer.get("mask") or {}).get("size", 0))})


def _feed_forward_spec(mlp: dict) -> PartSpec:
    router, shared = mlp["router"], mlp.get("shared")
    return PartSpec("routed_experts", {
        "experts": int(router["experts"]), "top": int(router["top"]), "ff": int(mlp["expert"]["ff"]),
        "correction": False, "scores": "softmax", "groups": router.get("groups"), "group_score": "best",
        "router_scale": float(router.get("scale", 1.0)), "activation": "silu",
        "shared": {"ff": int(shared["ff"])} if shared else None, "shared_gate": False})


def build_daferax_spec(config: DaferaxConfig) -> ModelSpec:
    norm = PartSpec("layernorm", {"eps": config.norm_eps, "weight_name": ""})
    block = PartSpec("normed_branch_residual", {
        # the norms' tensors are named without a suffix: the part's prefix is the whole name
        "tensor_prefixes": {"mixer_norm": "norm1", "mixer": "mix.", "feed_forward_norm": "norm2", "feed_forward": "mlp."}})
    layers = []
    for index, entry in enumerate(config.layers):
        mlp = entry.get("mlp")
        layers.append(LayerSpec(
            prefix=f"l{index}.", block=block,
            mixer=_mixer_spec(entry["type"], entry["mixer"], config.norm_eps, index == config.first_mixing_layer),
            feed_forward=None if mlp is None else _feed_forward_spec(mlp),
            mixer_norm=norm, feed_forward_norm=None if mlp is None else norm))
    return ModelSpec(
        architecture="Daferax", vocab_size=config.vocab, hidden_size=config.width, layers=tuple(layers),
        order=tuple(range(len(layers))), final_norm=norm, embedding_name="embed", final_norm_prefix="final.norm",
        lm_head_name="head", tie_word_embeddings=True, max_position_embeddings=config.max_position_embeddings)


register_architecture("Daferax", DaferaxConfig, build_daferax_spec, model_types=("daferax",))
