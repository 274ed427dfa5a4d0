"""Small Legilix configurations and weights for the tests: sizes that differ from one another in every way the
design allows (head counts and ratios, key and value sizes unlike each other and no multiples of 16, rotation on
part of a head and on all of it, with and without YaRN, windows smaller and larger than a page and of one token,
kept first tokens from none to more than a window, norms in one group and in several, multipliers of one and
others, routers that take one expert or all, layers without a feed-forward)."""

from __future__ import annotations

import copy
import json
from pathlib import Path

import torch


def yarn(factor, original, fast, slow):
    return {"factor": factor, "original": original, "fast": fast, "slow": slow}


def rot(base, dims, scaling=None):
    return {"base": base, "dims": dims, "scaling": scaling}


def talking(heads, kv_heads, dim, vdim, size, keep_first, rotation, scale, mlp):
    return {"type": "attention", "mlp": mlp,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "rot": rotation,
                      "mask": {"size": size, "keep_first": keep_first}}}


def distant(heads, kv_heads, dim, vdim, size, scale, mlp):
    return {"type": "attention_2", "mlp": mlp,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "mask": {"size": size}}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def model(vocab, width, groups, eps, layers, embedding_scale=1.0, logit_scale=1.0):
    return {"architecture": "Legilix", "vocab": vocab, "width": width, "norm": {"eps": eps, "groups": groups},
            "embedding": {"scale": embedding_scale}, "logit_scale": logit_scale, "layers": layers}


CONFIGS = {
    # A: groups of heads of two and three, values wider and narrower than keys, kept tokens fewer than a page,
    # a window shorter than a page, a router that takes two, a layer without a feed-forward
    "A": model(97, 60, 3, 1e-5, [
        talking(4, 2, 24, 40, 19, 5, rot(300.0, 16, yarn(8.0, 64, 16.0, 1.0)), 0.25, moe(6, 2, 40)),
        distant(6, 3, 20, 12, 9, 0.3, dense(100)),
        talking(6, 2, 20, 12, 23, 30, rot(10000.0, 20), 0.2, None),
        distant(2, 1, 16, 32, 33, 0.4, moe(5, 1, 24))], embedding_scale=3.0, logit_scale=0.7),
    # B: a norm in one group, multipliers of one, as many key/value heads as heads, widths that the tensor-core
    # kernels share, more kept tokens than a page holds, no kept tokens, a window of one token, pages of 32
    "B": model(131, 96, 1, 1e-6, [
        distant(4, 4, 32, 32, 36, 0.18, moe(7, 3, 48)),
        talking(5, 5, 16, 24, 50, 35, rot(1000.0, 6), 0.35, dense(72)),
        talking(3, 1, 64, 64, 12, 0, rot(20.0, 64, yarn(2.0, 16, 4.0, 0.5)), 0.1, moe(3, 2, 27)),
        distant(9, 3, 8, 20, 1, 0.3, None)]),
    # C: heads of 128 (distance bias on tcgen05 and on the split-context kernel), 16 heads on 2 and on 8, 32 heads,
    # heads that the mixing kernel does not take (33), groups of 17
    "C": model(64, 128, 4, 1e-6, [
        distant(4, 2, 128, 128, 70, 0.09, dense(64)),
        talking(16, 8, 128, 128, 45, 17, rot(500000.0, 32, yarn(16.0, 512, 32.0, 1.0)), 0.09, moe(4, 2, 16)),
        talking(32, 2, 16, 16, 100, 3, rot(100.0, 2), 0.2, None),
        talking(33, 3, 12, 8, 21, 4, rot(50.0, 12), 0.3, moe(11, 4, 24)),
        distant(17, 1, 64, 64, 90, 0.125, dense(40))], embedding_scale=0.5, logit_scale=2.0),
}
PAGE_SIZE = {"A": 16, "B": 32, "C": 16}


def without_choice(config: dict) -> dict:
    """The same model with routers that take every expert: the weights stay each token's own, and no rounding of
    a layer's input can change which experts run."""
    out = copy.deepcopy(config)
    for layer in out["layers"]:
        if layer.get("mlp") is not None and layer["mlp"]["kind"] == "moe":
            layer["mlp"]["router"]["top"] = layer["mlp"]["router"]["experts"]
    return out


def make_weights(config: dict, seed: int) -> dict[str, torch.Tensor]:
    """Float32 tensors by name, from distributions that keep every mechanism alive: scales around one, gates on
    both sides of one half, a mixing matrix with entries of both signs beside its diagonal, distance biases from
    weak to strong, router logits spread wide enough that they are told apart."""
    g = torch.Generator().manual_seed(seed)
    width = config["width"]

    def normal(*shape, std=1.0, mean=0.0):
        return torch.randn(*shape, generator=g) * std + mean

    def linear(out, inp, gain=1.0):
        return normal(out, inp, std=gain * inp ** -0.5)

    W = {"embed": normal(config["vocab"], width), "final.norm": normal(width, std=0.2, mean=1.0)}
    for index, layer in enumerate(config["layers"]):
        L, m = f"l{index}", layer["mixer"]
        H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        W[f"{L}.norm1"] = normal(width, std=0.2, mean=1.0)
        W.update({f"{L}.mix.q": linear(H * d, width, 1.5), f"{L}.mix.k": linear(G * d, width, 1.5),
                  f"{L}.mix.v": linear(G * dv, width, 1.5), f"{L}.mix.o": linear(width, H * dv),
                  f"{L}.mix.q.b": normal(H * d, std=0.4), f"{L}.mix.k.b": normal(G * d, std=0.4),
                  f"{L}.mix.v.b": normal(G * dv, std=0.4)})
        if layer["type"] == "attention":
            W.update({f"{L}.mix.q.norm": normal(d, std=0.3, mean=1.0), f"{L}.mix.k.norm": normal(d, std=0.3, mean=1.0),
                      f"{L}.mix.talk": torch.eye(H) * 0.8 + normal(H, H, std=0.3 if H <= 8 else 0.1)})
        else:
            W.update({f"{L}.mix.r1": torch.rand(H, generator=g) * 1.8 + 0.05, f"{L}.mix.r2": torch.rand(H, generator=g) * 0.6 + 0.02,
                      f"{L}.mix.g": linear(H, width, 1.5)})
        mlp = layer.get("mlp")
        if mlp is None:
            continue
        W[f"{L}.norm2"] = normal(width, std=0.2, mean=1.0)
        if mlp["kind"] == "dense":
            W.update({f"{L}.mlp.up": linear(mlp["ff"], width, 1.5), f"{L}.mlp.down": linear(width, mlp["ff"])})
            continue
        ff, experts = mlp["expert"]["ff"], mlp["router"]["experts"]
        W[f"{L}.mlp.router"] = linear(experts, width, 2.0)
        for e in range(experts):
            W.update({f"{L}.mlp.e{e}.gate": linear(ff, width, 1.5), f"{L}.mlp.e{e}.up": linear(ff, width, 1.5),
                      f"{L}.mlp.e{e}.down": linear(width, ff)})
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
