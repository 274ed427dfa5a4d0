"""A plain, slow Tedulorn in float64: one function per mechanism, written from the design's equations and
sharing nothing with the package.  Weights come as a dict of torch tensors by checkpoint name; the
configuration is the design's own ``config.json`` dictionary.

The layer: x <- x + mixer(N1(x)); x <- x + ff(N2(x)) (a layer may lack the second half); x <- x + N3(P (gelu(G x) * e))
with e the layer's part of the token's row in a second table.  N are RMS norms with a scale.  Mixers: ``retention``
(a state per head with a fixed decay, rotated queries and keys, unit RMS per head, a SiLU gate per value) and
``attention`` (RMS norm of q and k per head, rotation of halves, a window that keeps the first tokens, a softmax with
one added to its denominator, values mixed with the first such layer's, one sigmoid gate per head).  Feed-forwards:
an ungated one with a squared ReLU, and a routed one of bounded experts, limited to groups, with a shared expert.
"""

from __future__ import annotations

import math

import torch

F64 = torch.float64


def rms_unit(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    return rms_unit(x, eps) * w


def frequencies(rot: dict) -> torch.Tensor:
    dims = int(rot["dims"])
    return torch.tensor([float(rot["base"]) ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=F64)


def rotate_halves(x: torch.Tensor, positions: torch.Tensor, rot: dict) -> torch.Tensor:
    """x [T, heads, dim]: value i < dims / 2 of every head turns together with value i + dims / 2."""
    dims = int(rot["dims"])
    half = dims // 2
    angle = positions.to(F64).view(-1, 1, 1) * frequencies(rot).view(1, 1, half)
    c, s = torch.cos(angle), torch.sin(angle)
    a, b = x[..., :half], x[..., half:dims]
    return torch.cat([a * c - b * s, b * c + a * s, x[..., dims:]], dim=-1)


def silu(x: torch.Tensor) -> torch.Tensor:
    return x * torch.sigmoid(x)


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


# ------------------------------------------------------------------------------------------- retention
def decayed_states(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, decay: torch.Tensor) -> torch.Tensor:
    """S_t = decay_h S_(t-1) + k_t v_t^T, o_t = S_t^T q_t, token by token; q, k [T, H, d], v [T, H, dv] -> [T, H, dv]."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[2], dtype=F64)
    out = []
    for t in range(T):
        S = decay.view(H, 1, 1) * S + k[t].unsqueeze(-1) * v[t].unsqueeze(1)
        out.append(torch.einsum("hdv,hd->hv", S, q[t]))
    return torch.stack(out)


def retention(h: torch.Tensor, w: dict, prefix: str, m: dict, eps: float) -> torch.Tensor:
    T, H, d, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q, k = ((h @ w[f"{prefix}.{n}"].T).view(T, H, d) for n in ("q", "k"))
    v = (h @ w[f"{prefix}.v"].T).view(T, H, dv)
    positions = torch.arange(T)
    q, k = rotate_halves(q, positions, m["rot"]), rotate_halves(k, positions, m["rot"]) * d ** -0.5
    o = rms_unit(decayed_states(q, k, v, torch.tensor([float(a) for a in m["decay"]], dtype=F64)), eps).reshape(T, -1)
    return (o * silu(h @ w[f"{prefix}.g"].T)) @ w[f"{prefix}.o"].T


# ------------------------------------------------------------------------------------------- attention
def window_mask(T: int, size: int, keep_first: int = 0) -> torch.Tensor:
    i = torch.arange(T).view(T, 1)
    j = torch.arange(T).view(1, T)
    return (j <= i) & ((i - j < size) | (j < keep_first))


def softmax_plus_one(scores: torch.Tensor, visible: torch.Tensor) -> torch.Tensor:
    """exp(s_j) / (1 + sum exp(s_j)): the weights of a row add up to less than one."""
    scores = scores.masked_fill(~visible, -math.inf)
    top = scores.max(-1, keepdim=True).values.clamp(min=0.0)
    e = torch.exp(scores - top)
    return e / (torch.exp(-top) + e.sum(-1, keepdim=True))


def raw_scores(q: torch.Tensor, k: torch.Tensor, scale: float) -> torch.Tensor:
    """q [T, H, d], k [T, G, d] -> [H, T, T]: query head h against key head h // (H / G)."""
    per = q.shape[1] // k.shape[1]
    return torch.stack([q[:, h] @ k[:, h // per].T * scale for h in range(q.shape[1])])


def weigh_values(weights: torch.Tensor, v: torch.Tensor) -> torch.Tensor:
    """weights [H, T, T], v [T, G, dv] -> [T, H, dv], head h on the values of head h // (H / G)."""
    per = weights.shape[0] // v.shape[1]
    return torch.stack([weights[h] @ v[:, h // per] for h in range(weights.shape[0])], dim=1)


def mix_values(v: torch.Tensor, first: torch.Tensor | None, share: torch.Tensor) -> torch.Tensor:
    return v if first is None else (1.0 - share) * v + share * first


def attention(h: torch.Tensor, w: dict, prefix: str, m: dict, eps: float, shared: dict) -> torch.Tensor:
    """``shared``: what layers of one pass hand on (the first mixing layer's values)."""
    T, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k = (h @ w[f"{prefix}.q"].T).view(T, H, d), (h @ w[f"{prefix}.k"].T).view(T, G, d)
    v = (h @ w[f"{prefix}.v"].T).view(T, G, dv)
    q, k = rms_norm(q, w[f"{prefix}.q.norm"], eps), rms_norm(k, w[f"{prefix}.k.norm"], eps)
    positions = torch.arange(T)
    q, k = rotate_halves(q, positions, m["rot"]), rotate_halves(k, positions, m["rot"])
    if m.get("v_mix"):
        first = shared.get("values")
        if first is None:
            shared["values"] = v
        v = mix_values(v, first, w[f"{prefix}.vmix"])
    visible = window_mask(T, int(m["mask"]["size"]), int(m["mask"].get("keep_first") or 0))
    out = weigh_values(softmax_plus_one(raw_scores(q, k, float(m["scale"])), visible), v)
    return (out * torch.sigmoid(h @ w[f"{prefix}.g"].T).unsqueeze(-1)).reshape(T, -1) @ w[f"{prefix}.o"].T


# ---------------------------------------------------------------------------------------- feed-forward
def dense_feed_forward(h: torch.Tensor, w: dict, prefix: str) -> torch.Tensor:
    return torch.relu(h @ w[f"{prefix}.up"].T) ** 2 @ w[f"{prefix}.down"].T


def bounded_expert(h: torch.Tensor, w: dict, prefix: str, limit: float) -> torch.Tensor:
    g = (h @ w[f"{prefix}.gate"].T).clamp(max=limit)
    u = (h @ w[f"{prefix}.up"].T).clamp(-limit, limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ w[f"{prefix}.down"].T


def route(z: torch.Tensor, correction: torch.Tensor, router: dict):
    """(ids [T, top], weights [T, top], margin [T]): how far the nearest decision (between groups or between
    experts) is from going the other way, in units of the choice score."""
    T, E = z.shape
    top, count, keep = int(router["top"]), int(router["groups"]["count"]), int(router["groups"]["keep"])
    s = torch.softmax(z, dim=-1)
    choice = s + correction
    marks = choice.view(T, count, E // count).max(-1).values
    ranked, order = torch.sort(marks, dim=-1, descending=True, stable=True)
    margin = ranked[:, keep - 1] - ranked[:, keep] if keep < count else torch.full((T,), math.inf, dtype=F64)
    open_groups = torch.zeros(T, count, dtype=torch.bool).scatter_(1, order[:, :keep], True)
    allowed = choice.masked_fill(~open_groups.repeat_interleave(E // count, dim=1), -math.inf)
    values, ids = torch.sort(allowed, dim=-1, descending=True, stable=True)
    if top < E:
        margin = torch.minimum(margin, values[:, top - 1] - values[:, top])
    ids = ids[:, :top]
    weights = s.gather(1, ids)
    return ids, weights / (weights.sum(-1, keepdim=True) + 1e-20), margin


def routed_feed_forward(h: torch.Tensor, w: dict, prefix: str, mlp: dict, margins: list | None = None) -> torch.Tensor:
    ids, weights, margin = route(h @ w[f"{prefix}.router"].T, w[f"{prefix}.correction"], mlp["router"])
    if margins is not None:
        margins.append(margin)
    out = bounded_expert(h, w, f"{prefix}.shared", float(mlp["shared"]["limit"]))
    for e in range(int(mlp["router"]["experts"])):
        token, place = (ids == e).nonzero(as_tuple=True)
        if token.numel():
            y = bounded_expert(h[token], w, f"{prefix}.e{e}", float(mlp["expert"]["limit"]))
            out.index_add_(0, token, y * weights[token, place].unsqueeze(-1))
    return out


def feed_forward(h: torch.Tensor, w: dict, prefix: str, mlp: dict, margins: list | None = None) -> torch.Tensor:
    if mlp["kind"] == "dense":
        return dense_feed_forward(h, w, prefix)
    return routed_feed_forward(h, w, prefix, mlp, margins)


# ------------------------------------------------------------------------------------ per-layer token input
def token_side(x: torch.Tensor, e: torch.Tensor, w: dict, prefix: str, eps: float) -> torch.Tensor:
    """What the layer's part e of the tokens' second rows adds to the stream x."""
    y = (gelu_tanh(x @ w[f"{prefix}.gate"].T) * e) @ w[f"{prefix}.proj"].T
    return rms_norm(y, w[f"{prefix}.norm"], eps)


def forward(config: dict, weights: dict, tokens: list[int], layers_out: list | None = None,
            margins: list | None = None) -> torch.Tensor:
    """Logits [T, vocab] of one sequence.  ``layers_out`` collects the stream after every layer, ``margins``
    every routed layer's per-token margin of its choice."""
    w = {name: t.to(F64) for name, t in weights.items()}
    eps = float(config["norm"]["eps"])
    dim = int(config["token_side"]["dim"]) if config.get("token_side") else 0
    ids = torch.tensor(tokens, dtype=torch.long)
    x = w["embed"][ids] * float(config["embedding"]["scale"])
    shared: dict = {}
    for index, layer in enumerate(config["layers"]):
        prefix, m = f"l{index}", layer["mixer"]
        h = rms_norm(x, w[f"{prefix}.norm1"], eps)
        if layer["type"] == "retention":
            x = x + retention(h, w, f"{prefix}.mix", m, eps)
        else:
            x = x + attention(h, w, f"{prefix}.mix", m, eps, shared)
        if layer.get("mlp") is not None:
            x = x + feed_forward(rms_norm(x, w[f"{prefix}.norm2"], eps), w, f"{prefix}.mlp", layer["mlp"], margins)
        if dim:
            x = x + token_side(x, w["side.embed"][ids, index * dim:(index + 1) * dim], w, f"{prefix}.side", eps)
        if layers_out is not None:
            layers_out.append(x.clone())
    return rms_norm(x, w["final.norm"], eps) @ w["head"].T
