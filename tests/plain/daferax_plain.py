"""Plain, slow, whole-sequence implementation of the Daferax decoder.

The oracle of the Daferax tests: no cache, no batching, no kernels, one function per mechanism, float64 torch ops on
the CPU.  It shares no code with the engine package: it reads ``config.json`` and the safetensors file by itself and
takes every size and constant from the configuration dictionary.

Notation: T tokens, W the model width, x [T, W].  Linear weights are kept [out, in] and applied as x @ W^T.

The design
* gives each sublayer the residual itself and adds the layer-normed output: x <- x + norm(sublayer(x));
* has two token mixers: ``attention`` (heads of q and k RMS-normed, rotated in neighbouring pairs, values mixed with those
  of the first such layer, one gate per head) and ``latent_attention`` (keys and values are linear maps of a normed latent,
  one rotated key part for all heads with stretched frequencies, a sliding window, a gate per output element);
* feeds forward through a mixture of silu-gated experts chosen within the best groups by softmax scores, and a shared expert;
* reads the logits off the embedding table.
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


def layer_norm(x: torch.Tensor, w: torch.Tensor, b: torch.Tensor, eps: float) -> torch.Tensor:
    centred = x - x.mean(-1, keepdim=True)
    return centred / torch.sqrt(centred.pow(2).mean(-1, keepdim=True) + eps) * w + b


# --------------------------------------------------------------------------- rotation
def frequencies(rot: dict) -> tuple[list[float], float]:
    """Per pair the angle of one position, and the factor on cosine and sine."""
    dims, base = int(rot["dims"]), float(rot["base"])
    plain = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    s = rot.get("scaling")
    if not s:
        return plain, 1.0
    factor, original = float(s["factor"]), float(s["original"])

    def place(turns: float) -> float:
        return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo, hi = max(math.floor(place(float(s["fast"]))), 0), min(math.ceil(place(float(s["slow"]))), dims - 1)
    out = []
    for i, f in enumerate(plain):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / factor * ramp + f * (1.0 - ramp))
    return out, 0.1 * math.log(factor) + 1.0


def rotate_pairs(x: torch.Tensor, rot: dict, first: int = 0) -> torch.Tensor:
    """x [T, heads, d]: values 2i and 2i + 1 of the first ``dims`` form pair i, turned by position * f_i; the rest pass.
    Row t stands at position first + t."""
    dims = int(rot["dims"])
    freq, factor = frequencies(rot)
    angle = (torch.arange(x.shape[0], dtype=torch.float64) + first)[:, None] * torch.tensor(freq, dtype=torch.float64)[None, :]
    c, s = (torch.cos(angle) * factor)[:, None, :], (torch.sin(angle) * factor)[:, None, :]
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    turned = torch.stack([u * c - v * s, v * c + u * s], dim=-1).reshape(*x.shape[:-1], dims)
    return torch.cat([turned, x[..., dims:]], dim=-1)


# --------------------------------------------------------------------------- attention
def visible(count: int, window: int = 0) -> torch.Tensor:
    """[T, T] bool: row i sees j <= i, with a window only i - j < window."""
    i, j = torch.arange(count)[:, None], torch.arange(count)[None, :]
    return (j <= i) & ((i - j < window) if window > 0 else torch.ones(count, count, dtype=torch.bool))


def softmax_attention(q, k, v, scale: float, window: int = 0) -> torch.Tensor:
    """q, k [T, H, d], v [T, H, e] -> [T, H, e]."""
    scores = torch.einsum("ihd,jhd->hij", q, k) * scale
    weights = torch.softmax(scores.masked_fill(~visible(q.shape[0], window), float("-inf")), dim=-1)
    return torch.einsum("hij,jhe->ihe", weights, v)


def mix_values(v: torch.Tensor, first: torch.Tensor, amount: torch.Tensor) -> torch.Tensor:
    return (1.0 - amount) * v + amount * first


def attention(x, w, prefix, m, eps, first_values):
    """Returns (output [T, W], this layer's values before any mixing [T, G, e])."""
    count = x.shape[0]
    heads, groups, d, e = (int(m[key]) for key in ("heads", "kv_heads", "dim", "vdim"))
    q = rms((x @ w[prefix + "q"].t()).view(count, heads, d), eps) * w[prefix + "q.norm"]
    k = rms((x @ w[prefix + "k"].t()).view(count, groups, d), eps) * w[prefix + "k.norm"]
    own = v = (x @ w[prefix + "v"].t()).view(count, groups, e)
    if m.get("v_mix") and first_values is not None:
        v = mix_values(v, first_values, w[prefix + "vmix"])
    q, k = rotate_pairs(q, m["rot"]), rotate_pairs(k, m["rot"])
    k, v = (t.repeat_interleave(heads // groups, dim=1) for t in (k, v))
    o = softmax_attention(q, k, v, float(m["scale"]))
    o = o * torch.sigmoid(x @ w[prefix + "g"].t())[:, :, None]
    return o.reshape(count, heads * e) @ w[prefix + "o"].t(), own


def latent_attention(x, w, prefix, m, eps) -> torch.Tensor:
    count = x.shape[0]
    heads, d, r, e, rank = (int(m[key]) for key in ("heads", "dim", "rot_dim", "vdim", "kv_rank"))
    q = (x @ w[prefix + "q"].t()).view(count, heads, d + r)
    low = x @ w[prefix + "dkv"].t()
    c = rms(low[:, :rank], eps) * w[prefix + "dkv.norm"]
    shared = rotate_pairs(low[:, None, rank:], m["rot"]).expand(count, heads, r)
    k = torch.cat([(c @ w[prefix + "uk"].t()).view(count, heads, d), shared], dim=-1)
    v = (c @ w[prefix + "uv"].t()).view(count, heads, e)
    q = torch.cat([q[..., :d], rotate_pairs(q[..., d:], m["rot"])], dim=-1)
    o = softmax_attention(q, k, v, float(m["scale"]), int((m.get("mask") or {}).get("size", 0)))
    o = o.reshape(count, heads * e) * torch.sigmoid(x @ w[prefix + "g"].t())
    return o @ w[prefix + "o"].t()


# --------------------------------------------------------------------------- feed-forward
def expert(x, w, prefix) -> torch.Tensor:
    return (F.silu(x @ w[prefix + "gate"].t()) * (x @ w[prefix + "up"].t())) @ w[prefix + "down"].t()


def route(logits: torch.Tensor, top: int, groups: dict | None, scale: float) -> torch.Tensor:
    """logits [T, E] -> dense weights [T, E]: softmax scores, the choice confined to the groups with the largest best score."""
    scores = torch.softmax(logits, dim=-1)
    choice = scores
    if groups:
        count, keep = int(groups["count"]), int(groups["keep"])
        per_group = scores.view(scores.shape[0], count, -1)
        kept = per_group.amax(-1).topk(keep, dim=-1).indices
        allowed = torch.zeros(scores.shape[0], count, dtype=torch.bool).scatter_(1, kept, True)
        choice = per_group.masked_fill(~allowed[:, :, None], -1.0).reshape_as(scores)
    chosen = choice.topk(top, dim=-1).indices
    return torch.zeros_like(scores).scatter_(1, chosen, scores.gather(1, chosen)) * scale


def routing_margin(logits: torch.Tensor, top: int, groups: dict | None) -> torch.Tensor:
    """[T]: how far (in logits) a token's choice of experts is from another one: the smaller of the gaps between the last
    kept group's best expert and the first dropped one's, and between the last chosen expert and the next it could have been."""
    far = torch.full((logits.shape[0],), float("inf"), dtype=logits.dtype)
    allowed = logits
    if groups and int(groups["keep"]) < int(groups["count"]):
        count, keep = int(groups["count"]), int(groups["keep"])
        best = logits.view(logits.shape[0], count, -1)
        order = best.amax(-1).sort(dim=-1, descending=True)
        far = torch.minimum(far, order.values[:, keep - 1] - order.values[:, keep])
        allowed = best.gather(1, order.indices[:, :keep, None].expand(-1, -1, best.shape[2])).flatten(1)
    if top < allowed.shape[1]:
        ranked = allowed.sort(dim=-1, descending=True).values
        far = torch.minimum(far, ranked[:, top - 1] - ranked[:, top])
    return far


def mixture(x, w, prefix, mlp) -> torch.Tensor:
    router = mlp["router"]
    weights = route(x @ w[prefix + "router"].t(), int(router["top"]), router.get("groups"), float(router.get("scale", 1.0)))
    y = expert(x, w, prefix + "shared.") if mlp.get("shared") else torch.zeros_like(x)
    for index in range(int(router["experts"])):
        y = y + weights[:, index:index + 1] * expert(x, w, f"{prefix}e{index}.")
    return y


# --------------------------------------------------------------------------- the model
def forward_layers(cfg: dict, w: dict, tokens: list[int], margins: list | None = None) -> list[torch.Tensor]:
    """The residual after the embedding and after every layer: a list of [T, W].  ``margins``: every mixture adds its tokens'
    routing margins to it."""
    eps = float(cfg["norm"]["eps"])
    x = w["embed"][torch.tensor(tokens, dtype=torch.long)]
    seen, first_values = [x], None
    for index, layer in enumerate(cfg["layers"]):
        p, m = f"l{index}.", layer["mixer"]
        if layer["type"] == "attention":
            y, values = attention(x, w, p + "mix.", m, eps, first_values)
            if m.get("v_mix") and first_values is None:
                first_values = values
        elif layer["type"] == "latent_attention":
            y = latent_attention(x, w, p + "mix.", m, eps)
        else:
            raise ValueError(f"layer {index}: unknown type {layer['type']!r}")
        x = x + layer_norm(y, w[p + "norm1"], w[p + "norm1.b"], eps)
        if layer.get("mlp") is not None:
            if margins is not None:
                router = layer["mlp"]["router"]
                margins.append(routing_margin(x @ w[p + "mlp.router"].t(), int(router["top"]), router.get("groups")))
            x = x + layer_norm(mixture(x, w, p + "mlp.", layer["mlp"]), w[p + "norm2"], w[p + "norm2.b"], eps)
        seen.append(x)
    return seen


def logits_of(cfg: dict, w: dict, x: torch.Tensor) -> torch.Tensor:
    return layer_norm(x, w["final.norm"], w["final.norm.b"], float(cfg["norm"]["eps"])) @ w["embed"].t()


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
    width, vocab = int(cfg["width"]), int(cfg["vocab"])
    out = {"embed": ((vocab, width), "embed"), "final.norm": ((width,), "norm"), "final.norm.b": ((width,), "bias")}
    for index, layer in enumerate(cfg["layers"]):
        p, m = f"l{index}.", layer["mixer"]
        out[p + "norm1"], out[p + "norm1.b"] = ((width,), "norm"), ((width,), "bias")
        q = p + "mix."
        heads, d, e = (int(m[key]) for key in ("heads", "dim", "vdim"))
        if layer["type"] == "attention":
            groups = int(m["kv_heads"])
            for name, rows in (("q", heads * d), ("k", groups * d), ("v", groups * e), ("g", heads)):
                out[q + name] = ((rows, width), "matrix")
            out[q + "q.norm"], out[q + "k.norm"] = ((d,), "head_norm"), ((d,), "head_norm")
            if m.get("v_mix"):
                out[q + "vmix"] = ((), "share")
        else:
            r, rank = int(m["rot_dim"]), int(m["kv_rank"])
            for name, shape in (("q", (heads * (d + r), width)), ("dkv", (rank + r, width)), ("uk", (heads * d, rank)),
                                ("uv", (heads * e, rank)), ("g", (heads * e, width))):
                out[q + name] = (shape, "matrix")
            out[q + "dkv.norm"] = ((rank,), "head_norm")
        out[q + "o"] = ((width, heads * e), "matrix")
        mlp = layer.get("mlp")
        if mlp is not None:
            out[p + "norm2"], out[p + "norm2.b"] = ((width,), "norm"), ((width,), "bias")
            experts = [(f"e{i}.", int(mlp["expert"]["ff"])) for i in range(int(mlp["router"]["experts"]))]
            if mlp.get("shared"):
                experts.append(("shared.", int(mlp["shared"]["ff"])))
            out[p + "mlp.router"] = ((int(mlp["router"]["experts"]), width), "matrix")
            for name, ff in experts:
                out[p + "mlp." + name + "gate"] = ((ff, width), "matrix")
                out[p + "mlp." + name + "up"] = ((ff, width), "matrix")
                out[p + "mlp." + name + "down"] = ((width, ff), "matrix")
    return out


def random_weights(cfg: dict, seed: int) -> dict[str, torch.Tensor]:
    """Random weights, rounded to bfloat16 values: large enough that every mechanism moves the logits, the branches' norms small
    enough that a branch whose output is small (and is blown up by its norm) does not drown the residual in rounding."""
    generator = torch.Generator().manual_seed(seed)
    out = {}
    for name, (shape, kind) in tensor_shapes(cfg).items():
        draw = torch.randn(shape, generator=generator)
        uniform = torch.rand(shape, generator=generator) - 0.5
        out[name] = {"matrix": lambda: draw / math.sqrt(shape[-1]), "embed": lambda: draw, "norm": lambda: 0.4 + 0.3 * uniform,
                     "bias": lambda: 0.1 * draw, "head_norm": lambda: 1.2 + 0.8 * uniform,
                     "share": lambda: 0.5 + 0.6 * uniform}[kind]().to(torch.bfloat16)
    return out


def write_model(folder, cfg: dict, seed: int, weights: dict | None = None) -> dict[str, torch.Tensor]:
    folder = Path(folder)
    folder.mkdir(parents=True, exist_ok=True)
    weights = weights if weights is not None else random_weights(cfg, seed)
    (folder / "config.json").write_text(json.dumps(cfg, indent=1))
    write_safetensors(folder / "model.safetensors", weights)
    return weights
