"""Small Tedulorn configurations and weights for the tests: sizes that differ from one another in every way the
design allows (head counts and ratios, key and value sizes unlike each other and no multiples of 16, rotation on part
of a head and on all of it, decays from forgetting at once to keeping everything, windows smaller and larger than a
page and of one token, kept first tokens from none to more than a window, layers that mix values and layers between
them that do not, routers with one group and several, that take one expert or all, experts and shared experts of
different bounds, layers without a feed-forward, models without a second table)."""

from __future__ import annotations

import copy
import json
from pathlib import Path

import torch


def rot(base, dims):
    return {"base": base, "dims": dims}


def retention(heads, dim, vdim, rotation, decay, mlp):
    return {"type": "retention", "mlp": mlp, "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "rot": rotation, "decay": decay}}


def attention(heads, kv_heads, dim, vdim, size, keep_first, rotation, scale, v_mix, mlp):
    return {"type": "attention", "mlp": mlp,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "rot": rotation,
                      "mask": {"size": size, "keep_first": keep_first}, "v_mix": v_mix}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, count, keep, ff, limit, shared_ff, shared_limit):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "shared": {"ff": shared_ff, "limit": shared_limit},
            "router": {"experts": experts, "top": top, "groups": {"count": count, "keep": keep}}}


def model(vocab, width, eps, side_dim, layers, embedding_scale=1.0):
    out = {"architecture": "Tedulorn", "vocab": vocab, "width": width, "norm": {"eps": eps},
           "embedding": {"scale": embedding_scale}, "layers": layers}
    if side_dim:
        out["token_side"] = {"dim": side_dim}
    return out


CONFIGS = {
    # A: groups of heads of two and three, values wider and narrower than keys, a mixing layer first and last with one
    # that does not mix between them, more kept tokens than the window, a layer without a feed-forward
    "A": model(97, 60, 1e-5, 12, [
        retention(3, 20, 12, rot(300.0, 8), [0.5, 0.97, 0.999], dense(100)),
        attention(4, 2, 24, 40, 19, 5, rot(300.0, 16), 0.25, True, moe(6, 2, 3, 2, 40, 1.2, 24, 2.0)),
        attention(5, 5, 16, 24, 33, 0, rot(10000.0, 16), 0.3, False, None),
        attention(6, 2, 20, 40, 9, 30, rot(1000.0, 6), 0.2, True, dense(72)),
        retention(1, 33, 50, rot(50.0, 32), [0.9], moe(8, 3, 4, 2, 27, 0.8, 40, 0.6))], embedding_scale=3.0),
    # B: key and value widths that the tensor-core kernels share, pages of 32, more kept tokens than a page holds, a
    # window of one token, one group, a decay of one and of nearly nothing, odd sizes of a layer's part of the table
    "B": model(131, 96, 1e-6, 7, [
        attention(4, 4, 32, 32, 36, 35, rot(10000.0, 32), 0.18, False, moe(7, 3, 1, 1, 48, 3.0, 64, 1.0)),
        retention(2, 64, 72, rot(500000.0, 64), [1.0, 0.05], dense(72)),
        attention(9, 3, 64, 64, 40, 0, rot(20.0, 10), 0.1, True, None),
        attention(6, 3, 32, 64, 1, 4, rot(100.0, 32), 0.3, True, moe(4, 1, 2, 1, 13, 0.5, 27, 0.7)),
        attention(3, 3, 16, 64, 50, 1, rot(100.0, 2), 0.35, True, dense(30))]),
    # C: heads of 128 (tcgen05, the split-context kernel, the kept window on mma.sync), heads that only the general
    # kernel takes (33), groups of 17, wide retention heads, many groups
    "C": model(64, 128, 1e-6, 32, [
        attention(4, 2, 128, 128, 70, 0, rot(50000.0, 64), 0.09, True, dense(64)),
        retention(2, 128, 136, rot(10000.0, 128), [0.98, 0.9995], moe(16, 4, 8, 5, 16, 1.0, 16, 1.5)),
        attention(16, 2, 128, 128, 45, 17, rot(500000.0, 32), 0.09, True, moe(12, 4, 4, 2, 24, 1.5, 48, 2.5)),
        attention(33, 3, 12, 8, 21, 4, rot(50.0, 12), 0.3, False, None),
        attention(34, 2, 64, 128, 90, 9, rot(50.0, 64), 0.125, True, dense(40)),
        retention(1, 250, 24, rot(2000.0, 16), [0.96], dense(48))], embedding_scale=0.5),
}
PAGE_SIZE = {"A": 16, "B": 32, "C": 16}


def without_choice(config: dict) -> dict:
    """The same model with routers that take every expert: the weights stay each token's own, and no rounding of
    a layer's input can change which experts run."""
    out = copy.deepcopy(config)
    for layer in out["layers"]:
        if layer.get("mlp") is not None and layer["mlp"]["kind"] == "moe":
            router = layer["mlp"]["router"]
            router["top"], router["groups"]["keep"] = router["experts"], router["groups"]["count"]
    return out


def first_mixing_layer(config: dict) -> int | None:
    return next((i for i, layer in enumerate(config["layers"]) if layer["mixer"].get("v_mix")), None)


def make_weights(config: dict, seed: int) -> dict[str, torch.Tensor]:
    """Float32 tensors by name, from distributions that keep every mechanism alive: scales around one, gates on
    both sides of one half, shares of the first values well between nothing and all, corrections large enough to move
    the choice and to make choice scores negative, expert products that reach their bounds."""
    g = torch.Generator().manual_seed(seed)
    width, layers = config["width"], config["layers"]
    side = config["token_side"]["dim"] if config.get("token_side") else 0

    def normal(*shape, std=1.0, mean=0.0):
        return torch.randn(*shape, generator=g) * std + mean

    def linear(out, inp, gain=1.0):
        return normal(out, inp, std=gain * inp ** -0.5)

    def expert(prefix, ff):
        return {f"{prefix}.gate": linear(ff, width, 1.5), f"{prefix}.up": linear(ff, width, 1.5), f"{prefix}.down": linear(width, ff)}

    W = {"embed": normal(config["vocab"], width), "final.norm": normal(width, std=0.2, mean=1.0),
         "head": linear(config["vocab"], width, 2.0)}
    if side:
        W["side.embed"] = normal(config["vocab"], side * len(layers))
    for index, layer in enumerate(layers):
        L, m = f"l{index}", layer["mixer"]
        H, d, dv = m["heads"], m["dim"], m["vdim"]
        G = m.get("kv_heads", H)
        W[f"{L}.norm1"] = normal(width, std=0.2, mean=1.0)
        W.update({f"{L}.mix.q": linear(H * d, width, 1.5), f"{L}.mix.k": linear(G * d, width, 1.5),
                  f"{L}.mix.v": linear(G * dv, width, 1.5), f"{L}.mix.o": linear(width, H * dv)})
        if layer["type"] == "retention":
            W[f"{L}.mix.g"] = linear(H * dv, width, 1.5)
            # A head's read-out is divided by its own size.  Where a token's query meets every key at a right angle that
            # blows roundings up without end, so a token's own key leans towards its query.
            W[f"{L}.mix.k"] = 0.8 * W[f"{L}.mix.q"] + 0.6 * W[f"{L}.mix.k"]
        else:
            W.update({f"{L}.mix.q.norm": normal(d, std=0.3, mean=1.0), f"{L}.mix.k.norm": normal(d, std=0.3, mean=1.0),
                      f"{L}.mix.g": linear(H, width, 1.5)})
            if m.get("v_mix"):
                W[f"{L}.mix.vmix"] = torch.rand((), generator=g) * 0.6 + 0.2
        if side:
            W.update({f"{L}.side.gate": linear(side, width, 1.5), f"{L}.side.proj": linear(width, side),
                      f"{L}.side.norm": normal(width, std=0.2, mean=0.7)})
        mlp = layer.get("mlp")
        if mlp is None:
            continue
        W[f"{L}.norm2"] = normal(width, std=0.2, mean=1.0)
        if mlp["kind"] == "dense":
            W.update({f"{L}.mlp.up": linear(mlp["ff"], width, 1.2), f"{L}.mlp.down": linear(width, mlp["ff"])})
            continue
        experts = mlp["router"]["experts"]
        W[f"{L}.mlp.router"] = linear(experts, width, 2.0)
        W[f"{L}.mlp.correction"] = normal(experts, std=0.3)
        for e in range(experts):
            W.update(expert(f"{L}.mlp.e{e}", mlp["expert"]["ff"]))
        W.update(expert(f"{L}.mlp.shared", mlp["shared"]["ff"]))
    return W


def write_model(folder: Path, config: dict, seed: int, dtype: torch.dtype) -> Path:
    """config.json and model.safetensors in ``dtype``.  The plain implementation reads the stored (rounded) values
    back, so both sides start from the same numbers."""
    from zephyr_b200.weights.safetensors_io import save_safetensors

    folder.mkdir(parents=True, exist_ok=True)
    (folder / "config.json").write_text(json.dumps(config, indent=1))
    save_safetensors(folder / "model.safetensors",
                     {name: t.to(dtype).contiguous() for name, t in make_weights(config, seed).items()})
    return folder


def read_model(folder: Path) -> tuple[dict, dict[str, torch.Tensor]]:
    from zephyr_b200.weights import Checkpoint

    store = Checkpoint(folder)
    return json.loads((Path(folder) / "config.json").read_text()), {name: store.read(name) for name in store.names()}
