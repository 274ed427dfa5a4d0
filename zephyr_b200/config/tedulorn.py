"""Typed configuration of Tedulorn, a pre-norm decoder that mixes retention layers with windowed attention layers
which hand their values on, and whose layers each add a gated part of the token's row in a second table.

config.json names the design under ``architecture`` and lists its layers under ``layers``; each entry gives
``type`` (which mixer), ``mixer`` (its sizes and constants) and ``mlp`` (the feed-forward, or null for a layer
without one).  Model-wide keys: ``vocab``, ``width``, ``norm.eps``, ``embedding.scale`` (a multiplier on the embedding,
default 1) and ``token_side.dim`` (the width of a layer's part of the second table's rows; without ``token_side`` there
is no second table).

Mixer types:

  * ``retention``: ``heads``, ``dim``, ``vdim``, ``rot`` = {``base``, ``dims``}, ``decay`` (one number per head).  Linear
    attention with a fixed decay per head, rotated queries and keys, unit RMS per head, a SiLU gate per value.
  * ``attention``: ``heads``, ``kv_heads``, ``dim``, ``vdim``, ``scale``, ``rot``, ``mask`` = {``size``, ``keep_first``}
    (null: causal), ``v_mix``.  RMS norm of q and k per head with one scale vector shared by the heads, rotation of
    halves on the first ``rot.dims`` values of a head, a window of ``size`` tokens that keeps the first ``keep_first``,
    one added to the softmax's denominator, one sigmoid gate per head; with ``v_mix`` the values are mixed with those
    of the first such layer.

Feed-forwards (``mlp.kind``): ``dense`` (``ff``; down(max(up(x), 0)^2)) and ``moe``: ``router`` = {``experts``, ``top``,
``groups`` = {``count``, ``keep``}}, ``expert`` = {``ff``, ``limit``} and ``shared`` = {``ff``, ``limit``} (an expert that
runs for every token).  Scores are a softmax over all experts; a learned correction moves the choice only; a group's
mark is its largest corrected score; the taken experts' scores are divided by their sum.  Experts are bounded:
g = min(gate, limit), u = clamp(up, -limit, limit), g sigmoid(1.702 g) (u + 1).

Every layer is x <- x + mixer(N1(x)), x <- x + ff(N2(x)), x <- x + N3(P (gelu(G x) * e)) on a float32 residual stream
(the ``prenorm_residual`` block with a ``token_gate`` side part), N RMS norms with a scale.  The head is a table of its
own.  Tensor names: ``embed``, ``side.embed``, ``l<i>.norm1|norm2``, ``l<i>.mix.q|k|v|g|o``, and for attention
``l<i>.mix.q.norm|k.norm|vmix``; ``l<i>.mlp.up|down`` or ``l<i>.mlp.router|correction`` and ``l<i>.mlp.e<j>|shared`` each
with ``.gate|up|down``; ``l<i>.side.gate|proj|norm``; ``final.norm``, ``head``.
"""

from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Any, Mapping

from .errors import ConfigError
from .legelix import MAX_POSITIONS, _int, _number, _table
from .spec import (FeedForwardSpec, InputSpec, LayerSpec, MixerSpec, ModelSpec, NormSpec, OutputSpec, PositionSpec, SideSpec)

EXPERT_ALPHA = 1.702        # of the experts' gate and the shift of their up values: the design fixes both
EXPERT_UP_SHIFT = 1.0
VALUE_GROUP = "values"      # the name under which attention layers of one step hand their first values on


@dataclass
class TedulornConfig:
    vocab: int
    width: int
    layers: tuple[Mapping[str, Any], ...]
    norm_eps: float
    embedding_scale: float
    side_dim: int           # 0: no second table

    architecture = "Tedulorn"
    model_type = "tedulorn"

    # ------------------------------------------------------------------ reading
    @classmethod
    def from_dict(cls, config: Mapping[str, Any], where: str = "config.json") -> "TedulornConfig":
        if not isinstance(config, Mapping):
            raise ConfigError(f"{where}: the configuration must be a JSON object")
        if config.get("architecture", cls.architecture) != cls.architecture:
            raise ConfigError(f"{where}: not a {cls.architecture} configuration")
        layers = config.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError(f"{where}: 'layers' must be a non-empty list")
        embedding_scale = 1.0
        if config.get("embedding") is not None and _table(config, "embedding", where).get("scale") is not None:
            embedding_scale = _number(config["embedding"], "scale", where)
        side_dim = _int(_table(config, "token_side", where), "dim", where) if config.get("token_side") is not None else 0
        result = cls(vocab=_int(config, "vocab", where), width=_int(config, "width", where), layers=tuple(copy.deepcopy(layers)),
                     norm_eps=_number(_table(config, "norm", where), "eps", where), embedding_scale=embedding_scale,
                     side_dim=side_dim)
        result.validate(where)
        return result

    def validate(self, where: str = "config") -> None:
        if not self.norm_eps > 0.0:
            raise ConfigError(f"{where}: norm.eps must be positive")
        value_sizes = None
        for index, layer in enumerate(self.layers):
            at = f"{where}: layers[{index}]"
            if not isinstance(layer, Mapping):
                raise ConfigError(f"{at} must be a JSON object")
            kind, mixer = layer.get("type"), _table(layer, "mixer", at)
            if kind not in ("retention", "attention"):
                raise ConfigError(f"{at}: unknown layer type {kind!r}; known: retention, attention")
            for key in ("heads", "dim", "vdim"):
                _int(mixer, key, at)
            self._validate_rotation(mixer, at)
            if kind == "retention":
                decay = mixer.get("decay")
                if not isinstance(decay, list) or len(decay) != mixer["heads"]:
                    raise ConfigError(f"{at}: 'decay' must list one number per head")
                for h in range(len(decay)):
                    _number(dict(enumerate(decay)), h, f"{at}: decay")
            else:
                if mixer["heads"] % _int(mixer, "kv_heads", at) != 0:
                    raise ConfigError(f"{at}: heads must be a multiple of kv_heads")
                _number(mixer, "scale", at)
                if mixer.get("mask") is not None:
                    mask = _table(mixer, "mask", at)
                    _int(mask, "size", at)
                    keep = mask.get("keep_first")
                    if keep is not None and (isinstance(keep, bool) or not isinstance(keep, int) or keep < 0):
                        raise ConfigError(f"{at}: mask.keep_first must be a non-negative integer")
                if mixer.get("v_mix"):
                    sizes = (mixer["kv_heads"], mixer["vdim"])
                    if value_sizes not in (None, sizes):
                        raise ConfigError(f"{at}: layers that mix values must agree on kv_heads and vdim")
                    value_sizes = sizes
            self._validate_feed_forward(layer.get("mlp"), at)

    @staticmethod
    def _validate_rotation(mixer: Mapping[str, Any], at: str) -> None:
        rot = _table(mixer, "rot", at)
        if not _number(rot, "base", at) > 1.0:
            raise ConfigError(f"{at}: rot.base must be greater than one")
        if _int(rot, "dims", at) % 2 != 0 or rot["dims"] > mixer["dim"]:
            raise ConfigError(f"{at}: rot.dims must be even and no more than dim")

    @staticmethod
    def _validate_feed_forward(mlp: Any, at: str) -> None:
        if mlp is None:
            return
        if not isinstance(mlp, Mapping) or mlp.get("kind") not in ("dense", "moe"):
            raise ConfigError(f"{at}: 'mlp' must be null, a dense or a moe feed-forward")
        if mlp["kind"] == "dense":
            _int(mlp, "ff", at)
            return
        for key in ("expert", "shared"):
            if key == "shared" and mlp.get(key) is None:
                continue
            expert = _table(mlp, key, at)
            _int(expert, "ff", at)
            if not _number(expert, "limit", at) > 0.0:
                raise ConfigError(f"{at}: {key}.limit must be positive")
        router = _table(mlp, "router", at)
        experts, top = _int(router, "experts", at), _int(router, "top", at)
        if top > experts:
            raise ConfigError(f"{at}: router.top exceeds the number of experts")
        if router.get("groups") is not None:
            groups = _table(router, "groups", at)
            count, keep = _int(groups, "count", at), _int(groups, "keep", at)
            if experts % count != 0 or keep > count or keep * (experts // count) < top:
                raise ConfigError(f"{at}: router.groups must divide the experts evenly, and the kept groups must hold 'top' of them")

    # ------------------------------------------------------------------ writing
    def to_dict(self) -> dict[str, Any]:
        out = {"architecture": self.architecture, "embedding": {"scale": self.embedding_scale},
               "layers": copy.deepcopy(list(self.layers)), "norm": {"eps": self.norm_eps}, "vocab": self.vocab, "width": self.width}
        if self.side_dim:
            out["token_side"] = {"dim": self.side_dim}
        return out

    # --------------------------------------------------------------- model spec
    def _norm(self, name: str) -> NormSpec:
        return NormSpec("rmsnorm", self.width, self.norm_eps, name)

    @staticmethod
    def _position(m: Mapping[str, Any]) -> PositionSpec:
        return PositionSpec("rope_halves", head_dim=m["dim"], max_positions=MAX_POSITIONS,
                            params={"base": float(m["rot"]["base"]), "dims": m["rot"]["dims"]})

    def _retention(self, prefix: str, m: Mapping[str, Any]) -> MixerSpec:
        return MixerSpec("retention", {
            "hidden_size": self.width, "heads": m["heads"], "key_dim": m["dim"], "value_dim": m["vdim"],
            "decay": tuple(float(a) for a in m["decay"]), "norm_eps": self.norm_eps,
            **{name: f"{prefix}.{name}" for name in ("q", "k", "v", "g", "o")}}, self._position(m))

    def _attention(self, prefix: str, m: Mapping[str, Any], first_values: bool) -> MixerSpec:
        mask = m.get("mask") or {}
        params = {
            "hidden_size": self.width, "num_heads": m["heads"], "num_kv_heads": m["kv_heads"], "head_dim": m["dim"],
            "value_dim": m["vdim"], "window": mask.get("size") or 0, "keep_first": int(mask.get("keep_first") or 0),
            "scale": float(m["scale"]), "qk_norm_eps": self.norm_eps, "zero_sinks": True,
            "q_proj": f"{prefix}.q", "k_proj": f"{prefix}.k", "v_proj": f"{prefix}.v", "o_proj": f"{prefix}.o",
            "q_norm": f"{prefix}.q.norm", "k_norm": f"{prefix}.k.norm", "head_gate": f"{prefix}.g"}
        if m.get("v_mix"):
            params["value_mix"] = {"group": VALUE_GROUP, "share": None if first_values else f"{prefix}.vmix"}
        return MixerSpec("attention", params, self._position(m))

    def _expert(self, prefix: str, expert: Mapping[str, Any]) -> dict[str, Any]:
        return {"hidden_size": self.width, "intermediate_size": expert["ff"], "activation": "clamped_swish",
                "limit": float(expert["limit"]), "alpha": EXPERT_ALPHA, "up_shift": EXPERT_UP_SHIFT,
                "gate_proj": f"{prefix}.gate", "up_proj": f"{prefix}.up", "down_proj": f"{prefix}.down"}

    def _feed_forward(self, prefix: str, mlp: Mapping[str, Any]) -> FeedForwardSpec:
        if mlp["kind"] == "dense":
            return FeedForwardSpec("ungated", {
                "hidden_size": self.width, "intermediate_size": mlp["ff"], "activation": "relu_squared",
                "up_proj": f"{prefix}.up", "down_proj": f"{prefix}.down"})
        router = mlp["router"]
        params = {key: value for key, value in self._expert(prefix, mlp["expert"]).items() if not key.endswith("_proj")}
        params.update(
            experts=router["experts"], top=router["top"], scores="softmax", normalize=True, router=f"{prefix}.router",
            correction=f"{prefix}.correction",
            expert_names=tuple((f"{prefix}.e{j}.gate", f"{prefix}.e{j}.up", f"{prefix}.e{j}.down") for j in range(router["experts"])))
        if router.get("groups") is not None:
            params["groups"] = {"count": router["groups"]["count"], "keep": router["groups"]["keep"], "top": 1}
        if mlp.get("shared") is not None:
            params["shared"] = self._expert(f"{prefix}.shared", mlp["shared"])
        return FeedForwardSpec("routed", params)

    def _side(self, prefix: str, index: int) -> SideSpec | None:
        if not self.side_dim:
            return None
        return SideSpec("token_gate", {
            "hidden_size": self.width, "vocab_size": self.vocab, "dim": self.side_dim, "offset": index * self.side_dim,
            "row": len(self.layers) * self.side_dim, "table": "side.embed", "gate": f"{prefix}.gate", "proj": f"{prefix}.proj",
            "norm": self._norm(f"{prefix}.norm")})

    def to_model_spec(self) -> ModelSpec:
        from ..parts.model import run_order_for

        layers, unread = [], []
        first_values = True
        for index, layer in enumerate(self.layers):
            prefix, m = f"l{index}", layer["mixer"]
            if layer["type"] == "retention":
                mixer = self._retention(f"{prefix}.mix", m)
            else:
                mixer = self._attention(f"{prefix}.mix", m, first_values)
                if first_values or not m.get("v_mix"):
                    unread.append(f"{prefix}.mix.vmix")      # the first mixing layer has one that nothing reads
                first_values = first_values and not m.get("v_mix")
            norms = {"mixer": self._norm(f"{prefix}.norm1")}
            feed_forward = None
            if layer.get("mlp") is not None:
                feed_forward = self._feed_forward(f"{prefix}.mlp", layer["mlp"])
                norms["feed_forward"] = self._norm(f"{prefix}.norm2")
            else:
                unread.append(f"{prefix}.norm2")
            layers.append(LayerSpec("prenorm_residual", mixer, feed_forward, norms, side=self._side(f"{prefix}.side", index)))
        spec = ModelSpec(
            architecture=self.architecture, vocab_size=self.vocab, hidden_size=self.width, max_seq_len=MAX_POSITIONS,
            input=InputSpec("embedding", {"weight": "embed", "vocab_size": self.vocab, "hidden_size": self.width,
                                          "float32_stream": True, "scale": self.embedding_scale, "rounded_copy": False}),
            layers=tuple(layers), run_order=run_order_for(layers),
            output=OutputSpec("norm_head", {"norm": self._norm("final.norm"), "weight": "head", "vocab_size": self.vocab,
                                            "hidden_size": self.width}),
            ignorable_weights=tuple(unread))
        spec.validate()
        return spec
