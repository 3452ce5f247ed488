"""A matrix memory that decays per key channel and writes the difference to what it already holds."""
from __future__ import annotations

import torch

from ..kernels import ops
from ..weights.tensor_spec import TensorSpec
from .base import Mixer, RequestState, register_mixer
from .linear import linear_partials, linear_sums

_DEFAULT_NAMES = {"q": "q", "k": "k", "v": "v", "beta": "b", "out": "o", "norm": "norm", "conv_suffix": ".conv", "a_log": "A_log",
                  "dt_bias": "dt_bias", "decay_down": "a1", "decay_up": "a2", "gate_down": "g1", "gate_up": "g2"}


@register_mixer("channel_delta_memory")
class ChannelDeltaMemory(Mixer):
    """params: ``heads``, ``kv_heads`` (q and k come in so many heads, head h uses h // (heads / kv_heads)), ``dim`` (of a
    head's q and k), ``vdim`` (of its value), ``conv`` (taps of the short causal convolution that q, k and v each pass),
    ``decay_rank``, ``gate_rank``, ``eps`` (of the output norm), ``tensor_names``.

    q, k, v = silu(conv(W x)); every head of q and k divided by its length (sqrt(sum of squares + 1e-6)), q also by
    sqrt(dim);  beta = sigmoid(W_b x) per head;  keep = exp(-exp(A_log_h) softplus(W_a2 (W_a1 x) + dt_bias)) per head and
    key channel.  Per head, token by token (S is [dim, vdim]):
        S <- diag(keep) S;     u = beta (v - S^T k);     S <- S + k u^T;     o = S^T q.
    Each head's o is RMS-normed over ``vdim`` with one weight vector for all heads, multiplied by sigmoid(W_g2 (W_g1 x))
    and projected by W_o.  Kept per request, in float32: S [heads, dim, vdim] and the last ``conv`` - 1 projected rows of
    [q | k | v].

    One stacked product gives [q | k | v | beta | W_a1 x | W_g1 x]; one kernel does the convolutions, the activations and
    the unit vectors; a second product over both low-rank inputs (their matrices on the diagonal of one) gives the
    decays' and the gate's pre-activations with float32 results; from there the recurrence is float32."""

    graph_safe = True
    kernel_sources = ("delta_memory", "delta_memory_chunks", "linear_attention",)

    def __init__(self, params, weights, ctx) -> None:
        super().__init__(params, weights, ctx)
        p = params
        self.heads, self.groups, self.dim, self.vdim = int(p["heads"]), int(p["kv_heads"]), int(p["dim"]), int(p["vdim"])
        self.taps, self.eps = int(p["conv"]), float(p["eps"])
        if self.heads % self.groups or self.taps < 1:
            raise ops.KernelError(f"delta memory: {self.heads} heads on {self.groups}, {self.taps} taps")
        names = {**_DEFAULT_NAMES, **p.get("tensor_names", {})}
        stacked = [weights[names[role]] for role in ("q", "k", "v", "beta", "decay_down", "gate_down")]
        pad = -sum(w.shape[0] for w in stacked) % 16     # whole tiles of the few-rows product
        if pad:
            stacked.append(stacked[0].new_zeros((pad, stacked[0].shape[1])))
        self.in_weight = torch.cat(stacked, dim=0).contiguous()
        self.conv_weight = torch.cat([weights[names[role] + names["conv_suffix"]].to(torch.float32)
                                      for role in ("q", "k", "v")], dim=0).contiguous()
        decay_up, gate_up = weights[names["decay_up"]], weights[names["gate_up"]]
        self.rank = decay_up.shape[1] + gate_up.shape[1]
        low = self.rank + -self.rank % 16
        self.up_weight = decay_up.new_zeros((decay_up.shape[0] + gate_up.shape[0], low))
        self.up_weight[:decay_up.shape[0], :decay_up.shape[1]] = decay_up
        self.up_weight[decay_up.shape[0]:, decay_up.shape[1]:self.rank] = gate_up
        self.dt_bias = weights[names["dt_bias"]].to(torch.float32).contiguous()
        self.a_log = weights[names["a_log"]].to(torch.float32).contiguous()
        self.norm_weight = weights[names["norm"]].to(torch.float32).contiguous()
        self.out_weight = weights[names["out"]].contiguous()

    @classmethod
    def expected_tensors(cls, params, hidden_size):
        p = params
        heads, groups, dim, vdim, taps = (int(p[key]) for key in ("heads", "kv_heads", "dim", "vdim", "conv"))
        decay_rank, gate_rank = int(p["decay_rank"]), int(p["gate_rank"])
        names = {**_DEFAULT_NAMES, **p.get("tensor_names", {})}
        out = {}
        for role, rows in (("q", groups * dim), ("k", groups * dim), ("v", heads * vdim)):
            out[names[role]] = TensorSpec((rows, hidden_size))
            out[names[role] + names["conv_suffix"]] = TensorSpec((rows, taps), "filter")
        out.update({
            names["beta"]: TensorSpec((heads, hidden_size)), names["a_log"]: TensorSpec((heads,), "bias"),
            names["norm"]: TensorSpec((vdim,), "norm"), names["decay_down"]: TensorSpec((decay_rank, hidden_size)),
            names["decay_up"]: TensorSpec((heads * dim, decay_rank)), names["dt_bias"]: TensorSpec((heads * dim,), "bias"),
            names["gate_down"]: TensorSpec((gate_rank, hidden_size)), names["gate_up"]: TensorSpec((heads * vdim, gate_rank)),
            names["out"]: TensorSpec((hidden_size, heads * vdim))})
        return out

    @classmethod
    def cache_requirement(cls, params, hidden_size):
        heads, groups, dim, vdim, taps = (int(params[key]) for key in ("heads", "kv_heads", "dim", "vdim", "conv"))
        return (RequestState((heads, dim, vdim), "float32"),
                RequestState((taps - 1, 2 * groups * dim + heads * vdim), "float32"))

    def forward(self, x, step, cache):
        state, window = cache.parts[0].state, cache.parts[1].state
        tokens = x.shape[0]
        proj = linear_partials(x, self.in_weight)
        low = torch.empty((tokens, self.up_weight.shape[1]), dtype=x.dtype, device=x.device)
        q, k, v, beta = ops.delta_prepare(proj, self.conv_weight, window, step, low, self.groups, self.heads, self.dim,
                                          self.vdim, self.rank, self.dim ** -0.5)
        up = linear_sums(low, self.up_weight)        # [decays' pre-activations | gate's]
        read = torch.empty((tokens, self.heads * self.vdim), dtype=torch.float32, device=x.device)
        ops.delta_scan(q, k, v, beta, up, self.dt_bias, self.a_log, state, step.segment_start, step.segment_state_slot, read,
                       self.heads, self.groups, self.dim, self.vdim)
        gated = torch.empty((tokens, self.heads * self.vdim), dtype=x.dtype, device=x.device)
        ops.gated_group_rmsnorm(read, up, self.heads * self.dim, self.norm_weight, self.eps, gated, self.heads,
                                gate_first=False, gate_activation="sigmoid", segment_of_token=step.segment_of_token)
        return linear_partials(gated, self.out_weight)
