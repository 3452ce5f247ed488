"""Plain, slow, whole-sequence implementation of the Kofipel decoder.

The oracle of the Kofipel tests: no cache, no batching, no kernels, one function per mechanism, float64 torch ops on
the CPU.  It shares no code with the engine package: it reads ``config.json`` and the safetensors file by itself and
takes every size and constant from the configuration dictionary.

Notation: T tokens, W the model width, x [T, W].  Linear weights are kept [out, in] and applied as x @ W^T.

The design
* norms before each sublayer and gives it h + conv(h), h the normed rows, conv a short causal convolution per channel;
* has two token mixers: ``attention`` (values are the unrotated keys, biases, a learned factor per head on capped
  scores, a window that keeps the sequence's first tokens, one more unit in the softmax's denominator) and
  ``channel_delta`` (a matrix memory that decays per key channel and writes the difference to what it already holds);
* feeds forward densely with a squared relu;
* after the feed-forward adds a normed projection of a gated vector looked up per token and layer;
* runs a range of layers several times, the embedding output added again before every pass but the first.
"""
from __future__ import annotations

import json
import math
from pathlib import Path

import torch
import torch.nn.functional as F

from .sebudra_plain import read_safetensors, write_safetensors    # the file format's plain reader and writer


# --------------------------------------------------------------------------- small parts
def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps)


def unit(x: torch.Tensor) -> torch.Tensor:
    return x / torch.sqrt(x.pow(2).sum(-1, keepdim=True) + 1e-6)


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def causal_conv(u: torch.Tensor, taps: torch.Tensor) -> torch.Tensor:
    """u [T, C], taps [C, K]: y_t = sum_j taps[:, j] u_(t - K + 1 + j), zeros before the sequence."""
    count, width = u.shape[0], taps.shape[1]
    padded = torch.cat([torch.zeros(width - 1, u.shape[1], dtype=u.dtype), u], dim=0)
    y = torch.zeros_like(u)
    for j in range(width):
        y = y + padded[j:j + count] * taps[:, j]
    return y


def sublayer_input(x, norm_weight, taps, eps) -> torch.Tensor:
    """What a sublayer reads: the normed rows plus their convolution over time."""
    h = rms(x, eps) * norm_weight
    return h + causal_conv(h, taps)


# --------------------------------------------------------------------------- attention
def rotate_half(x: torch.Tensor, base: float, dims: int) -> torch.Tensor:
    """x [T, heads, d]: value i of the first ``dims`` is paired with value i + dims / 2, by the angle
    position * base^(-2i / dims); the rest pass."""
    half = dims // 2
    freq = torch.tensor([base ** (-2.0 * i / dims) for i in range(half)], dtype=torch.float64)
    angle = torch.arange(x.shape[0], dtype=torch.float64)[:, None] * freq[None, :]
    c, s = torch.cos(angle)[:, None, :], torch.sin(angle)[:, None, :]
    a, b, rest = x[..., :half], x[..., half:dims], x[..., dims:]
    return torch.cat([a * c - b * s, b * c + a * s, rest], dim=-1)


def visible(count: int, window: int, keep_first: int) -> torch.Tensor:
    """[T, T] bool: row i sees j <= i that is less than ``window`` back or among the first ``keep_first``."""
    i, j = torch.arange(count)[:, None], torch.arange(count)[None, :]
    return (j <= i) & ((i - j < window) | (j < keep_first))


def sink_softmax(scores: torch.Tensor) -> torch.Tensor:
    """exp(s_j) / (1 + sum exp(s)) over the last axis."""
    top = scores.amax(-1, keepdim=True).clamp(min=0.0)
    e = torch.exp(scores - top)
    return e / (torch.exp(-top) + e.sum(-1, keepdim=True))


def attention(h, w, prefix, m) -> torch.Tensor:
    count = h.shape[0]
    heads, groups, d = int(m["heads"]), int(m["kv_heads"]), int(m["dim"])
    q = (h @ w[prefix + "q"].t() + w[prefix + "q.b"]).view(count, heads, d)
    k = (h @ w[prefix + "k"].t() + w[prefix + "k.b"]).view(count, groups, d)
    v = k
    rot = m["rot"]
    q, k = (rotate_half(t, float(rot["base"]), int(rot["dims"])) for t in (q, k))
    k, v = (t.repeat_interleave(heads // groups, dim=1) for t in (k, v))
    scores = torch.einsum("ihd,jhd->hij", q, k) * float(m["scale"]) * w[prefix + "temp"][:, None, None]
    cap = float(m["softcap"])
    scores = cap * torch.tanh(scores / cap)
    seen = visible(count, int(m["mask"]["size"]), int(m["mask"]["keep_first"]))
    weights = sink_softmax(scores.masked_fill(~seen, float("-inf")))
    o = torch.einsum("hij,jhe->ihe", weights, v).reshape(count, heads * d)
    return o @ w[prefix + "o"].t() + w[prefix + "o.b"]


# --------------------------------------------------------------------------- delta memory
def delta_memory(q, k, v, keep, beta, state=None):
    """q, k, keep [T, H, d], v [T, H, e], beta [T, H]:  S <- diag(keep_t) S;  S <- S + k_t (beta_t (v_t - S^T k_t))^T;
    o_t = S^T q_t.  S [H, d, e] from zero (or ``state``); returns (o, S)."""
    count, heads, d = q.shape
    state = torch.zeros(heads, d, v.shape[2], dtype=q.dtype) if state is None else state
    out = []
    for t in range(count):
        state = keep[t][:, :, None] * state
        u = beta[t][:, None] * (v[t] - torch.einsum("hde,hd->he", state, k[t]))
        state = state + k[t][:, :, None] * u[:, None, :]
        out.append(torch.einsum("hde,hd->he", state, q[t]))
    return torch.stack(out), state


def delta_decays(h, w, prefix, heads: int, d: int) -> torch.Tensor:
    """[T, H, d]: exp(-exp(A_log_h) softplus(low-rank map of h + dt_bias))."""
    z = (h @ w[prefix + "a1"].t()) @ w[prefix + "a2"].t() + w[prefix + "dt_bias"]
    rate = torch.exp(w[prefix + "A_log"])[None, :, None]
    return torch.exp(-rate * F.softplus(z, threshold=1e9).view(h.shape[0], heads, d))


def channel_delta(h, w, prefix, m, eps) -> torch.Tensor:
    count = h.shape[0]
    heads, groups, d, e = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])

    def convolved(name):
        return F.silu(causal_conv(h @ w[prefix + name].t(), w[prefix + name + ".conv"]))

    q = unit(convolved("q").view(count, groups, d)) * d ** -0.5
    k = unit(convolved("k").view(count, groups, d))
    v = convolved("v").view(count, heads, e)
    q, k = (t.repeat_interleave(heads // groups, dim=1) for t in (q, k))
    beta = torch.sigmoid(h @ w[prefix + "b"].t())
    o, _ = delta_memory(q, k, v, delta_decays(h, w, prefix, heads, d), beta)
    o = rms(o, eps) * w[prefix + "norm"]
    gate = torch.sigmoid((h @ w[prefix + "g1"].t()) @ w[prefix + "g2"].t())
    return (o.reshape(count, heads * e) * gate) @ w[prefix + "o"].t()


# --------------------------------------------------------------------------- feed-forward and the token's own input
def feed_forward(h, w, prefix) -> torch.Tensor:
    return F.relu(h @ w[prefix + "up"].t()).pow(2) @ w[prefix + "down"].t()


def token_side(x, e, w, prefix, eps) -> torch.Tensor:
    """What the layer adds after the feed-forward; e [T, dim] is the token's part of the side table for the layer."""
    g = gelu_tanh(x @ w[prefix + "gate"].t()) * e
    return rms(g @ w[prefix + "proj"].t(), eps) * w[prefix + "norm"]


# --------------------------------------------------------------------------- the model
def layer_runs(cfg: dict) -> list[tuple[int, bool]]:
    """(layer, whether the embedding output is added before it) of every layer run in order."""
    count = len(cfg["layers"])
    loop = cfg.get("loop") or {"start": 0, "stop": 0, "times": 1}
    start, stop, times = int(loop["start"]), int(loop["stop"]), int(loop["times"])
    runs = [(i, False) for i in range(start)]
    for turn in range(times):
        runs += [(i, turn > 0 and i == start) for i in range(start, stop)]
    return runs + [(i, False) for i in range(stop, count)]


def forward_layers(cfg: dict, w: dict, tokens: list[int]) -> list[torch.Tensor]:
    """The residual after the embedding and after every layer run: a list of [T, W]."""
    eps = float(cfg["norm"]["eps"])
    ids = torch.tensor(tokens, dtype=torch.long)
    embedded = x = w["embed"][ids]
    dim = int(cfg["token_side"]["dim"])
    side = w["side.embed"][ids]
    seen = [x]
    for index, again in layer_runs(cfg):
        if again:
            x = x + embedded
        layer, p = cfg["layers"][index], f"l{index}."
        h = sublayer_input(x, w[p + "norm1"], w[p + "canon1"], eps)
        if layer["type"] == "attention":
            x = x + attention(h, w, p + "mix.", layer["mixer"])
        elif layer["type"] == "channel_delta":
            x = x + channel_delta(h, w, p + "mix.", layer["mixer"], eps)
        else:
            raise ValueError(f"layer {index}: unknown type {layer['type']!r}")
        if layer.get("mlp") is not None:
            x = x + feed_forward(sublayer_input(x, w[p + "norm2"], w[p + "canon2"], eps), w, p + "mlp.")
        x = x + token_side(x, side[:, index * dim:(index + 1) * dim], w, p + "side.", eps)
        seen.append(x)
    return seen


def logits_of(cfg: dict, w: dict, x: torch.Tensor) -> torch.Tensor:
    return (rms(x, float(cfg["norm"]["eps"])) * w["final.norm"]) @ w["head"].t()


def forward_full(cfg: dict, w: dict, tokens: list[int]) -> torch.Tensor:
    """Logits [T, vocab] at every position of one sequence."""
    return logits_of(cfg, w, forward_layers(cfg, w, tokens)[-1])


# --------------------------------------------------------------------------- files
def load_folder(folder, round_to=None):
    """(config dictionary, weights in float64).  ``round_to``: round the weights to this dtype first."""
    folder = Path(folder)
    cfg = json.loads((folder / "config.json").read_text())
    weights = {}
    for name, tensor in read_safetensors(folder / "model.safetensors").items():
        if tensor.is_floating_point():
            tensor = (tensor.to(round_to) if round_to is not None else tensor).to(torch.float64)
        weights[name] = tensor
    return cfg, weights


def tensor_shapes(cfg: dict) -> dict[str, tuple]:
    """name -> (shape, kind) of every tensor of a model of this configuration; kind says how random values are drawn."""
    width, vocab, taps = int(cfg["width"]), int(cfg["vocab"]), int(cfg["canon"]["taps"])
    dim = int(cfg["token_side"]["dim"])
    out = {"embed": ((vocab, width), "embed"), "side.embed": ((vocab, len(cfg["layers"]) * dim), "embed"),
           "final.norm": ((width,), "norm"), "head": ((vocab, width), "matrix")}
    for index, layer in enumerate(cfg["layers"]):
        p, m = f"l{index}.", layer["mixer"]
        out[p + "norm1"] = ((width,), "norm")
        out[p + "canon1"] = ((width, taps), "filter")
        q = p + "mix."
        heads, groups, d, e = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
        if layer["type"] == "attention":
            for name, rows in (("q", heads * d), ("k", groups * d)):
                out[q + name] = ((rows, width), "matrix")
                out[q + name + ".b"] = ((rows,), "bias")
            out[q + "temp"] = ((heads,), "temp")
            out[q + "o"] = ((width, heads * e), "matrix")
            out[q + "o.b"] = ((width,), "bias")
        else:
            rank_a, rank_g = int(m["decay_rank"]), int(m["gate_rank"])   # only the tensors give these: a model written here names them
            for name, rows in (("q", groups * d), ("k", groups * d), ("v", heads * e)):
                out[q + name] = ((rows, width), "matrix")
                out[q + name + ".conv"] = ((rows, int(m["conv"])), "filter")
            out[q + "b"] = ((heads, width), "matrix")
            out[q + "A_log"] = ((heads,), "rate")
            out[q + "norm"] = ((e,), "norm")
            out[q + "a1"] = ((rank_a, width), "matrix")
            out[q + "a2"] = ((heads * d, rank_a), "matrix")
            out[q + "dt_bias"] = ((heads * d,), "step_bias")
            out[q + "g1"] = ((rank_g, width), "matrix")
            out[q + "g2"] = ((heads * e, rank_g), "matrix")
            out[q + "o"] = ((width, heads * e), "matrix")
        if layer.get("mlp") is not None:
            ff = int(layer["mlp"]["ff"])
            out[p + "norm2"] = ((width,), "norm")
            out[p + "canon2"] = ((width, taps), "filter")
            out[p + "mlp.up"] = ((ff, width), "matrix")
            out[p + "mlp.down"] = ((width, ff), "matrix")
        out[p + "side.gate"] = ((dim, width), "matrix")
        out[p + "side.proj"] = ((width, dim), "matrix")
        out[p + "side.norm"] = ((width,), "side_norm")
    return out


def random_weights(cfg: dict, seed: int) -> dict[str, torch.Tensor]:
    """Random weights, rounded to bfloat16 values: large enough that every mechanism moves the logits."""
    generator = torch.Generator().manual_seed(seed)
    out = {}
    for name, (shape, kind) in tensor_shapes(cfg).items():
        draw = torch.randn(shape, generator=generator)
        uniform = torch.rand(shape, generator=generator) - 0.5
        out[name] = {"matrix": lambda: draw / math.sqrt(shape[-1]), "embed": lambda: draw, "norm": lambda: 1.0 + 0.2 * uniform,
                     "side_norm": lambda: 0.4 + 0.2 * uniform, "bias": lambda: 0.3 * draw, "filter": lambda: 0.4 * draw,
                     "temp": lambda: 1.0 + uniform, "rate": lambda: draw, "step_bias": lambda: draw - 2.0}[kind]().to(torch.bfloat16)
    return out


def write_model(folder, cfg: dict, seed: int, weights: dict | None = None) -> dict[str, torch.Tensor]:
    folder = Path(folder)
    folder.mkdir(parents=True, exist_ok=True)
    weights = weights if weights is not None else random_weights(cfg, seed)
    (folder / "config.json").write_text(json.dumps(cfg, indent=1))
    write_safetensors(folder / "model.safetensors", weights)
    return weights
