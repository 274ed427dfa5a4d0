"""Typed configuration of Legilix, a pre-norm decoder with norms in groups whose layers mix the heads' scores
ahead of the softmax or take a logarithmic bias on the distance.

config.json names the design under ``architecture`` and lists its layers under ``layers``; each entry gives
``type`` (which mixer), ``mixer`` (its sizes and constants) and ``mlp`` (the feed-forward, or null for a layer
without one).  Model-wide keys: ``vocab``, ``width``, ``norm`` = {``eps``, ``groups``}, ``embedding.scale`` (a
multiplier on the embedding, default 1) and ``logit_scale`` (a multiplier on the logits, default 1).

Mixer types, both with ``heads``, ``kv_heads``, ``dim``, ``vdim``, ``scale`` and biases on q, k and v:

  * ``attention``: ``rot`` = {``base``, ``dims``, ``scaling`` = null or {``factor``, ``original``, ``fast``, ``slow``}
    (YaRN)}, ``mask`` = {``size``, ``keep_first``}.  RMS norm of q and k per head with one scale vector shared by
    the heads, rotation of halves on the first ``dims`` values of a head, the heads' scores mixed by a matrix
    ahead of the softmax, a window of ``size`` tokens that keeps the first ``keep_first``.
  * ``attention_2``: ``mask`` = {``size``}.  No norm, no rotation; r1_h ln(1 + r2_h d) is taken off head h's score of the
    key d positions back; a window of ``size`` tokens; one sigmoid gate per head on its output.

Feed-forwards (``mlp.kind``): ``dense`` (``ff``; down(gelu(up(x))), gelu in its tanh form) and ``moe`` (``expert.ff``;
``router.experts`` gated SiLU experts of which a token takes the ``router.top`` with the largest sigmoid scores; the
score, not renormalised, goes on the expert's input).

Every layer is x <- x + mixer(N1(x)), x <- x + ff(N2(x)) on a float32 residual stream (the ``prenorm_residual``
block), N an RMS norm over ``norm.groups`` equal parts of the width.  The head is the embedding table without its
multiplier.  Tensor names: ``embed``, ``l<i>.norm1|norm2``, ``l<i>.mix.q|k|v`` each with ``.b``, ``l<i>.mix.o`` and
``q.norm|k.norm|talk`` or ``r1|r2|g``, ``l<i>.mlp.up|down`` or ``l<i>.mlp.router|e<j>.gate|up|down``, ``final.norm``.
"""

from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Any, Mapping

from .errors import ConfigError
from .legelix import MAX_POSITIONS, _int, _number, _table
from .spec import FeedForwardSpec, InputSpec, LayerSpec, MixerSpec, ModelSpec, NormSpec, OutputSpec, PositionSpec


@dataclass
class LegilixConfig:
    vocab: int
    width: int
    layers: tuple[Mapping[str, Any], ...]
    norm_eps: float
    norm_groups: int
    embedding_scale: float
    logit_scale: float

    architecture = "Legilix"
    model_type = "legilix"

    # ------------------------------------------------------------------ reading
    @classmethod
    def from_dict(cls, config: Mapping[str, Any], where: str = "config.json") -> "LegilixConfig":
        if not isinstance(config, Mapping):
            raise ConfigError(f"{where}: the configuration must be a JSON object")
        if config.get("architecture", cls.architecture) != cls.architecture:
            raise ConfigError(f"{where}: not a {cls.architecture} configuration")
        layers = config.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError(f"{where}: 'layers' must be a non-empty list")
        norm = _table(config, "norm", where)
        embedding_scale = 1.0
        if config.get("embedding") is not None and _table(config, "embedding", where).get("scale") is not None:
            embedding_scale = _number(config["embedding"], "scale", where)
        result = cls(vocab=_int(config, "vocab", where), width=_int(config, "width", where),
                     layers=tuple(copy.deepcopy(layers)), norm_eps=_number(norm, "eps", where),
                     norm_groups=_int(norm, "groups", where) if norm.get("groups") is not None else 1,
                     embedding_scale=embedding_scale,
                     logit_scale=_number(config, "logit_scale", where) if config.get("logit_scale") is not None else 1.0)
        result.validate(where)
        return result

    def validate(self, where: str = "config") -> None:
        if not self.norm_eps > 0.0:
            raise ConfigError(f"{where}: norm.eps must be positive")
        if self.width % self.norm_groups != 0:
            raise ConfigError(f"{where}: norm.groups must divide the width evenly")
        for index, layer in enumerate(self.layers):
            at = f"{where}: layers[{index}]"
            if not isinstance(layer, Mapping):
                raise ConfigError(f"{at} must be a JSON object")
            kind, mixer = layer.get("type"), _table(layer, "mixer", at)
            if kind not in ("attention", "attention_2"):
                raise ConfigError(f"{at}: unknown layer type {kind!r}; known: attention, attention_2")
            for key in ("heads", "kv_heads", "dim", "vdim"):
                _int(mixer, key, at)
            if mixer["heads"] % mixer["kv_heads"] != 0:
                raise ConfigError(f"{at}: heads must be a multiple of kv_heads")
            _number(mixer, "scale", at)
            mask = _table(mixer, "mask", at)
            _int(mask, "size", at)
            if kind == "attention":
                keep = mask.get("keep_first")
                if keep is not None and (isinstance(keep, bool) or not isinstance(keep, int) or keep < 0):
                    raise ConfigError(f"{at}: mask.keep_first must be a non-negative integer")
                self._validate_rotation(mixer, at)
            self._validate_feed_forward(layer.get("mlp"), at)

    @staticmethod
    def _validate_rotation(mixer: Mapping[str, Any], at: str) -> None:
        rot = _table(mixer, "rot", at)
        if not _number(rot, "base", at) > 1.0:
            raise ConfigError(f"{at}: rot.base must be greater than one")
        if _int(rot, "dims", at) % 2 != 0 or rot["dims"] > mixer["dim"]:
            raise ConfigError(f"{at}: rot.dims must be even and no more than dim")
        if rot.get("scaling") is not None:
            scaling = _table(rot, "scaling", at)
            for key in ("factor", "original", "fast", "slow"):
                if not _number(scaling, key, at) > 0.0:
                    raise ConfigError(f"{at}: rot.scaling.{key} must be positive")

    @staticmethod
    def _validate_feed_forward(mlp: Any, at: str) -> None:
        if mlp is None:
            return
        if not isinstance(mlp, Mapping) or mlp.get("kind") not in ("dense", "moe"):
            raise ConfigError(f"{at}: 'mlp' must be null, a dense or a moe feed-forward")
        if mlp["kind"] == "dense":
            _int(mlp, "ff", at)
            return
        _int(_table(mlp, "expert", at), "ff", at)
        router = _table(mlp, "router", at)
        if _int(router, "top", at) > _int(router, "experts", at):
            raise ConfigError(f"{at}: router.top exceeds the number of experts")

    # ------------------------------------------------------------------ writing
    def to_dict(self) -> dict[str, Any]:
        return {"architecture": self.architecture, "embedding": {"scale": self.embedding_scale},
                "layers": copy.deepcopy(list(self.layers)), "logit_scale": self.logit_scale,
                "norm": {"eps": self.norm_eps, "groups": self.norm_groups}, "vocab": self.vocab, "width": self.width}

    # --------------------------------------------------------------- model spec
    def _mixer(self, prefix: str, kind: str, m: Mapping[str, Any]) -> MixerSpec:
        mask = m["mask"]
        params = {
            "hidden_size": self.width, "num_heads": m["heads"], "num_kv_heads": m["kv_heads"], "head_dim": m["dim"],
            "value_dim": m["vdim"], "window": mask["size"], "scale": float(m["scale"]),
            "q_proj": f"{prefix}.q", "k_proj": f"{prefix}.k", "v_proj": f"{prefix}.v", "o_proj": f"{prefix}.o",
            "q_bias": f"{prefix}.q.b", "k_bias": f"{prefix}.k.b", "v_bias": f"{prefix}.v.b"}
        if kind == "attention_2":
            params.update(distance_bias=(f"{prefix}.r1", f"{prefix}.r2"), head_gate=f"{prefix}.g")
            return MixerSpec("attention", params)
        rot = m["rot"]
        position = PositionSpec("rope_halves", head_dim=m["dim"], max_positions=MAX_POSITIONS, params={
            "base": float(rot["base"]), "dims": rot["dims"],
            "scaling": dict(rot["scaling"]) if rot.get("scaling") is not None else None})
        params.update(qk_norm_eps=self.norm_eps, q_norm=f"{prefix}.q.norm", k_norm=f"{prefix}.k.norm",
                      keep_first=int(mask.get("keep_first") or 0), score_mix=f"{prefix}.talk")
        return MixerSpec("attention", params, position)

    def _feed_forward(self, prefix: str, mlp: Mapping[str, Any]) -> FeedForwardSpec:
        if mlp["kind"] == "dense":
            return FeedForwardSpec("ungated", {
                "hidden_size": self.width, "intermediate_size": mlp["ff"], "activation": "gelu_tanh",
                "up_proj": f"{prefix}.up", "down_proj": f"{prefix}.down"})
        router = mlp["router"]
        return FeedForwardSpec("routed", {
            "hidden_size": self.width, "intermediate_size": mlp["expert"]["ff"], "activation": "silu",
            "experts": router["experts"], "top": router["top"], "scores": "sigmoid", "weigh": "inputs",
            "router": f"{prefix}.router",
            "expert_names": tuple((f"{prefix}.e{j}.gate", f"{prefix}.e{j}.up", f"{prefix}.e{j}.down")
                                  for j in range(router["experts"]))})

    def _norm(self, name: str) -> NormSpec:
        return NormSpec("rmsnorm", self.width, self.norm_eps, name, groups=self.norm_groups)

    def to_model_spec(self) -> ModelSpec:
        from ..parts.model import run_order_for

        layers = []
        for index, layer in enumerate(self.layers):
            prefix = f"l{index}"
            norms = {"mixer": self._norm(f"{prefix}.norm1")}
            feed_forward = None
            if layer.get("mlp") is not None:
                feed_forward = self._feed_forward(f"{prefix}.mlp", layer["mlp"])
                norms["feed_forward"] = self._norm(f"{prefix}.norm2")
            layers.append(LayerSpec("prenorm_residual", self._mixer(f"{prefix}.mix", layer["type"], layer["mixer"]),
                                    feed_forward, norms))
        spec = ModelSpec(
            architecture=self.architecture, vocab_size=self.vocab, hidden_size=self.width, max_seq_len=MAX_POSITIONS,
            input=InputSpec("embedding", {"weight": "embed", "vocab_size": self.vocab, "hidden_size": self.width,
                                          "float32_stream": True, "scale": self.embedding_scale, "rounded_copy": False}),
            layers=tuple(layers), run_order=run_order_for(layers),
            output=OutputSpec("norm_head", {"norm": self._norm("final.norm"), "weight": "embed", "vocab_size": self.vocab,
                                            "hidden_size": self.width, "logit_scale": self.logit_scale}))
        spec.validate()
        return spec
