"""Inputs that a layer takes from the token itself, beside the residual."""
from __future__ import annotations

import torch

from ..kernels import ops
from ..weights.tensor_spec import TensorSpec
from .base import TokenInput, register_token_input
from .linear import linear_partials
from .norm import RMSNorm

_DEFAULT_NAMES = {"gate": "gate", "proj": "proj", "norm": "norm"}


@register_token_input("gated_token_lookup")
class GatedTokenLookup(TokenInput):
    """params: ``dim``, ``table`` (full name of a table [vocab, >= offset + dim] that the layers share, declared in
    ``ModelSpec.shared_tensors``), ``offset`` (the layer's first column in it), ``eps`` (of the norm), ``tensor_names``.

        g = gelu_tanh(W_gate x) * table[token, offset .. offset + dim];      y = W_proj g,
    and y passes an RMS norm (``norm``) before the residual takes it.  x is the residual itself, not normed.  The columns
    of W_proj are padded to whole tiles of the products' inner size."""

    graph_safe = True
    kernel_sources = ("conv_norm",)

    def __init__(self, params, weights, ctx) -> None:
        super().__init__(params, weights, ctx)
        self.dim, self.offset = int(params["dim"]), int(params["offset"])
        names = {**_DEFAULT_NAMES, **params.get("tensor_names", {})}
        self.table = ctx.shared[params["table"]]
        gate, proj = weights[names["gate"]], weights[names["proj"]]
        pad = -self.dim % 16
        self.gate_weight = (torch.cat([gate, gate.new_zeros((pad, gate.shape[1]))]) if pad else gate).contiguous()
        self.proj_weight = (torch.cat([proj, proj.new_zeros((proj.shape[0], pad))], dim=1) if pad else proj).contiguous()
        self.norm = RMSNorm({"eps": params["eps"], "weight_name": names["norm"]}, weights, ctx)

    @classmethod
    def expected_tensors(cls, params, hidden_size):
        dim = int(params["dim"])
        names = {**_DEFAULT_NAMES, **params.get("tensor_names", {})}
        return {names["gate"]: TensorSpec((dim, hidden_size)), names["proj"]: TensorSpec((hidden_size, dim)),
                names["norm"]: TensorSpec((hidden_size,), "norm")}

    def forward(self, x, step):
        z = linear_partials(x, self.gate_weight)
        g = torch.empty((x.shape[0], self.proj_weight.shape[1]), dtype=x.dtype, device=x.device)
        ops.token_gate(z, self.table, self.offset, step.token_ids, g, self.dim)
        return linear_partials(g, self.proj_weight)
