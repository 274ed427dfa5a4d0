"""A plain, slow Legilix in float64: one function per mechanism, written from the design's equations and
sharing nothing with the package.  Weights come as a dict of torch tensors by checkpoint name; the
configuration is the design's own ``config.json`` dictionary.

The layer: x <- x + mixer(N1(x)); x <- x + ff(N2(x)) (a layer may lack the second half), N being an RMS norm
over equal consecutive groups of the width with one scale per column.  Mixers: ``attention`` (biased
projections, per-head RMS norm of q and k, rotation of halves with YaRN frequencies, the heads' SCORES mixed by
a matrix ahead of the softmax, a window that keeps the first tokens); ``attention_2`` (biased projections, no
rotation, a logarithmic bias on the distance, a window, one sigmoid gate per head).  Feed-forwards: an ungated
GELU one, and a routed one whose weights (sigmoid scores, not renormalised) go on the experts' inputs.
"""

from __future__ import annotations

import math

import torch

F64 = torch.float64


def rms_unit(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def grouped_rms_norm(x: torch.Tensor, w: torch.Tensor, groups: int, eps: float) -> torch.Tensor:
    parts = x.reshape(*x.shape[:-1], groups, x.shape[-1] // groups)
    return rms_unit(parts, eps).reshape(x.shape) * w


def yarn(rot: dict) -> tuple[torch.Tensor, float]:
    """The frequencies of the dims / 2 pairs and the multiplier on cosine and sine."""
    dims, base = int(rot["dims"]), float(rot["base"])
    freqs = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    s = rot.get("scaling")
    if s is None:
        return torch.tensor(freqs, dtype=F64), 1.0

    def place(turns):
        return dims * math.log(float(s["original"]) / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(place(float(s["fast"]))), 0)
    hi = min(math.ceil(place(float(s["slow"]))), dims - 1)
    out = []
    for i, f in enumerate(freqs):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / float(s["factor"]) * r + f * (1.0 - r))
    return torch.tensor(out, dtype=F64), 0.1 * math.log(float(s["factor"])) + 1.0


def rotate_halves(x: torch.Tensor, positions: torch.Tensor, rot: dict) -> torch.Tensor:
    """x [T, heads, dim]: value i < dims / 2 of every head turns together with value i + dims / 2."""
    dims = int(rot["dims"])
    half = dims // 2
    freqs, mult = yarn(rot)
    angle = positions.to(F64).view(-1, 1, 1) * freqs.view(1, 1, half)
    c, s = mult * torch.cos(angle), mult * torch.sin(angle)
    a, b = x[..., :half], x[..., half:dims]
    return torch.cat([a * c - b * s, b * c + a * s, x[..., dims:]], dim=-1)


def window_mask(T: int, size: int, keep_first: int = 0) -> torch.Tensor:
    i = torch.arange(T).view(T, 1)
    j = torch.arange(T).view(1, T)
    return (j <= i) & ((i - j < size) | (j < keep_first))


def softmax_over(scores: torch.Tensor, visible: torch.Tensor) -> torch.Tensor:
    scores = scores.masked_fill(~visible, -math.inf)
    e = torch.exp(scores - scores.max(-1, keepdim=True).values)
    return e / e.sum(-1, keepdim=True)


def raw_scores(q: torch.Tensor, k: torch.Tensor, scale: float) -> torch.Tensor:
    """q [T, H, d], k [T, G, d] -> [H, T, T]: query head h against key head h // (H / G)."""
    per = q.shape[1] // k.shape[1]
    return torch.stack([q[:, h] @ k[:, h // per].T * scale for h in range(q.shape[1])])


def mix_scores(scores: torch.Tensor, talk: torch.Tensor) -> torch.Tensor:
    """Head h's scores become the sum over g of talk[h, g] times head g's."""
    return torch.einsum("hg,gij->hij", talk, scores)


def distance_bias(T: int, r1: torch.Tensor, r2: torch.Tensor) -> torch.Tensor:
    """[H, T, T]: r1_h ln(1 + r2_h (i - j)), zero where j lies behind i (which no mask lets through)."""
    distance = (torch.arange(T).view(T, 1) - torch.arange(T).view(1, T)).clamp(min=0).to(F64)
    return r1.view(-1, 1, 1) * torch.log(1.0 + r2.view(-1, 1, 1) * distance)


def weigh_values(weights: torch.Tensor, v: torch.Tensor) -> torch.Tensor:
    """weights [H, T, T], v [T, G, dv] -> [T, H, dv], head h on the values of head h // (H / G)."""
    per = weights.shape[0] // v.shape[1]
    return torch.stack([weights[h] @ v[:, h // per] for h in range(weights.shape[0])], dim=1)


def projections(h: torch.Tensor, w: dict, prefix: str, m: dict):
    T = h.shape[0]
    out = []
    for name, heads, width in (("q", m["heads"], m["dim"]), ("k", m["kv_heads"], m["dim"]), ("v", m["kv_heads"], m["vdim"])):
        out.append((h @ w[f"{prefix}.{name}"].T + w[f"{prefix}.{name}.b"]).view(T, heads, width))
    return out


def talking_attention(h: torch.Tensor, w: dict, prefix: str, m: dict, eps: float) -> torch.Tensor:
    T = h.shape[0]
    q, k, v = projections(h, w, prefix, m)
    q, k = rms_unit(q, eps) * w[f"{prefix}.q.norm"], rms_unit(k, eps) * w[f"{prefix}.k.norm"]
    positions = torch.arange(T)
    q, k = rotate_halves(q, positions, m["rot"]), rotate_halves(k, positions, m["rot"])
    scores = mix_scores(raw_scores(q, k, float(m["scale"])), w[f"{prefix}.talk"])
    weights = softmax_over(scores, window_mask(T, int(m["mask"]["size"]), int(m["mask"].get("keep_first") or 0)))
    return weigh_values(weights, v).reshape(T, -1) @ w[f"{prefix}.o"].T


def distance_attention(h: torch.Tensor, w: dict, prefix: str, m: dict, eps: float) -> torch.Tensor:
    T = h.shape[0]
    q, k, v = projections(h, w, prefix, m)
    scores = raw_scores(q, k, float(m["scale"])) - distance_bias(T, w[f"{prefix}.r1"], w[f"{prefix}.r2"])
    weights = softmax_over(scores, window_mask(T, int(m["mask"]["size"])))
    gate = torch.sigmoid(h @ w[f"{prefix}.g"].T)
    return (weigh_values(weights, v) * gate.unsqueeze(-1)).reshape(T, -1) @ w[f"{prefix}.o"].T


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(x: torch.Tensor) -> torch.Tensor:
    return x * torch.sigmoid(x)


def dense_feed_forward(h: torch.Tensor, w: dict, prefix: str) -> torch.Tensor:
    return gelu_tanh(h @ w[f"{prefix}.up"].T) @ w[f"{prefix}.down"].T


def route(h: torch.Tensor, w: dict, prefix: str, top: int):
    """(ids [T, top], weights [T, top], margin [T]): the ``top`` largest sigmoid scores as they are, and how
    far the last taken logit lies above the first one left out."""
    z = h @ w[f"{prefix}.router"].T
    ordered, ids = torch.sort(z, dim=-1, descending=True, stable=True)
    margin = ordered[:, top - 1] - ordered[:, top] if z.shape[1] > top else torch.full((h.shape[0],), math.inf, dtype=F64)
    return ids[:, :top], torch.sigmoid(ordered[:, :top]), margin


def routed_feed_forward(h: torch.Tensor, w: dict, prefix: str, mlp: dict, margins: list | None = None) -> torch.Tensor:
    """out[t] = sum over the taken experts of expert(s x_t), the score s on the INPUT of a gated SiLU expert."""
    ids, weights, margin = route(h, w, prefix, int(mlp["router"]["top"]))
    if margins is not None:
        margins.append(margin)
    out = torch.zeros_like(h)
    for e in range(int(mlp["router"]["experts"])):
        token, place = (ids == e).nonzero(as_tuple=True)
        if token.numel() == 0:
            continue
        x = h[token] * weights[token, place].unsqueeze(-1)
        y = silu(x @ w[f"{prefix}.e{e}.gate"].T) * (x @ w[f"{prefix}.e{e}.up"].T)
        out.index_add_(0, token, y @ w[f"{prefix}.e{e}.down"].T)
    return out


MIXERS = {"attention": talking_attention, "attention_2": distance_attention}


def feed_forward(h: torch.Tensor, w: dict, prefix: str, mlp: dict, margins: list | None = None) -> torch.Tensor:
    if mlp["kind"] == "dense":
        return dense_feed_forward(h, w, prefix)
    return routed_feed_forward(h, w, prefix, mlp, margins)


def forward(config: dict, weights: dict, tokens: list[int], layers_out: list | None = None,
            margins: list | None = None) -> torch.Tensor:
    """Logits [T, vocab] of one sequence.  ``layers_out`` collects the stream after every layer, ``margins``
    every routed layer's per-token margin of its choice."""
    w = {name: t.to(F64) for name, t in weights.items()}
    eps, groups = float(config["norm"]["eps"]), int(config["norm"]["groups"])
    x = w["embed"][torch.tensor(tokens, dtype=torch.long)] * float(config["embedding"]["scale"])
    for index, layer in enumerate(config["layers"]):
        prefix = f"l{index}"
        x = x + MIXERS[layer["type"]](grouped_rms_norm(x, w[f"{prefix}.norm1"], groups, eps), w, f"{prefix}.mix",
                                      layer["mixer"], eps)
        if layer.get("mlp") is not None:
            x = x + feed_forward(grouped_rms_norm(x, w[f"{prefix}.norm2"], groups, eps), w, f"{prefix}.mlp", layer["mlp"],
                                 margins)
        if layers_out is not None:
            layers_out.append(x.clone())
    return grouped_rms_norm(x, w["final.norm"], groups, eps) @ w["embed"].T * float(config["logit_scale"])
