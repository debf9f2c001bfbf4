"""Tesozen: a decoder whose layers each name their own mixer, with layer norms before and after every sublayer.

``config.json`` holds ``vocab``, ``width``, ``norm.eps``, ``embedding.scale`` (a factor on the embedding's rows) and a list
``layers``; every entry gives ``type`` (which mixer), ``mixer`` (its sizes and constants) and ``mlp`` (its feed-forward, or
null for none).  Three mixers:

- ``attention``: differential grouped-query attention without positions.  Every query and key head has two sub-heads of
  ``dim`` elements, each RMS-normed with a gain; the two maps over one value of ``vdim`` elements are subtracted with a
  weight made from four vectors of the layer and ``diff``, normed per head and multiplied by 1 - ``diff`` and by the sigmoid
  of one logit per head.  ``scale`` on the scores; a query sees the earlier keys of its own chunk of ``mask.size`` positions.
- ``mlstm``: a matrix memory with exponential gates (capped by ``gate_cap``), a running maximum and a normalizer.
- ``latent_attention``: attention over a cached latent of ``kv_rank`` elements without positions, every earlier key visible;
  the heads' outputs times the sigmoid of a gate per element.

The feed-forward is down(relu(up(.))^2) (``kind`` "dense", ``ff``), or a mixture of silu-gated experts (``kind`` "moe":
``router.experts``, ``router.top``, ``router.groups`` = {``count``, ``keep``}, ``router.scale``; ``expert.ff``; an optional
``shared`` = {``ff``} expert for every token): sigmoid scores, a stored correction that the choice alone sees, the choice
limited to the best groups, the chosen scores' shares of their sum times ``router.scale`` as weights.  Norms are layer norms
with a gain and a bias.  The head is the embedding table.  Layer i's tensors start with ``l<i>.``: ``norm1``, ``mix.*``,
``norm1b``, ``norm2``, ``mlp.*``, ``norm2b``.
"""

from __future__ import annotations

import copy
from typing import Any, Mapping

from .registry import register_architecture
from .spec import ConfigError, LayerRun, LayerSpec, ModelSpec, PartSpec

MIXERS = ("attention", "mlstm", "latent_attention")
DEFAULT_MAX_POSITIONS = 32768


def _positive(where: str, raw, *keys: str) -> None:
    if not isinstance(raw, Mapping):
        raise ConfigError(f"{where} is missing")
    for k in keys:
        if k not in raw:
            raise ConfigError(f"{where} lacks {k!r}")
        if not (isinstance(raw[k], int) and not isinstance(raw[k], bool) and raw[k] > 0):
            raise ConfigError(f"{where}: {k} must be a positive integer, got {raw[k]!r}")


def _number(where: str, raw, *keys: str) -> None:
    if not isinstance(raw, Mapping):
        raise ConfigError(f"{where} is missing")
    for k in keys:
        if not isinstance(raw.get(k), (int, float)) or isinstance(raw.get(k), bool):
            raise ConfigError(f"{where}: {k} must be a number, got {raw.get(k)!r}")


def _above_zero(where: str, raw, *keys: str) -> None:
    _number(where, raw, *keys)
    for k in keys:
        if not float(raw[k]) > 0:
            raise ConfigError(f"{where}: {k} must be above zero, got {raw[k]!r}")


@register_architecture("Tesozen")
class TesozenConfig:
    def __init__(self, raw: Mapping[str, Any]):
        self.raw = copy.deepcopy(dict(raw))
        self.validate()

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any]) -> "TesozenConfig":
        return cls(raw)

    def to_dict(self) -> dict[str, Any]:
        return copy.deepcopy(self.raw)

    # -- reading ------------------------------------------------------------
    @property
    def width(self) -> int:
        return int(self.raw["width"])

    @property
    def vocab(self) -> int:
        return int(self.raw["vocab"])

    @property
    def eps(self) -> float:
        return float(self.raw["norm"]["eps"])

    @property
    def layers(self) -> list[dict]:
        return self.raw["layers"]

    def validate(self) -> None:
        r = self.raw
        _positive("config.json", r, "vocab", "width")
        _above_zero("norm", r.get("norm"), "eps")
        _number("embedding", r.get("embedding"), "scale")
        if not isinstance(r.get("layers"), list) or not r["layers"]:
            raise ConfigError("config.json: layers must be a list with at least one layer")
        for i, layer in enumerate(r["layers"]):
            where = f"layers[{i}]"
            kind = layer.get("type") if isinstance(layer, Mapping) else None
            if kind not in MIXERS:
                raise ConfigError(f"{where}: type {kind!r} is not one of {MIXERS}")
            m = layer.get("mixer")
            _positive(where + ".mixer", m, "heads", "dim", "vdim")
            if kind == "mlstm":
                _above_zero(where + ".mixer", m, "gate_cap")
            elif kind == "attention":
                _positive(where + ".mixer", m, "kv_heads")
                _number(where + ".mixer", m, "scale", "diff")
                if m["heads"] % m["kv_heads"]:
                    raise ConfigError(f"{where}: heads must be a multiple of kv_heads")
                if m.get("mask") is not None:
                    _positive(where + ".mixer.mask", m["mask"], "size")
            else:
                _positive(where + ".mixer", m, "kv_rank")
                _number(where + ".mixer", m, "scale")
            self._validate_feed_forward(where + ".mlp", layer.get("mlp"))

    @staticmethod
    def _validate_feed_forward(where: str, f) -> None:
        if f is None:
            return
        kind = f.get("kind", "dense") if isinstance(f, Mapping) else None
        if kind == "dense":
            _positive(where, f, "ff")
            return
        if kind != "moe":
            raise ConfigError(f"{where}: feed-forward kind {kind!r} is not one of dense, moe")
        router = f.get("router")
        _positive(where + ".router", router, "experts", "top")
        _above_zero(where + ".router", router, "scale")
        _positive(where + ".expert", f.get("expert"), "ff")
        if f.get("shared") is not None:
            _positive(where + ".shared", f["shared"], "ff")
        if router["top"] > router["experts"]:
            raise ConfigError(f"{where}: top must not exceed experts")
        groups = router.get("groups")
        if groups is not None:
            _positive(where + ".router.groups", groups, "count", "keep")
            if router["experts"] % groups["count"] or groups["keep"] > groups["count"]:
                raise ConfigError(f"{where}: groups.count must divide experts, and groups.keep not exceed it")
            if groups["keep"] * (router["experts"] // groups["count"]) < router["top"]:
                raise ConfigError(f"{where}: the groups that are kept hold fewer than top experts")

    # -- the model as data --------------------------------------------------
    def _mixer(self, layer: Mapping[str, Any]) -> PartSpec:
        m, eps = layer["mixer"], self.eps
        heads = {"hidden_size": self.width, "num_heads": int(m["heads"])}
        if layer["type"] == "mlstm":
            return PartSpec("mlstm", {**heads, "key_dim": int(m["dim"]), "value_dim": int(m["vdim"]),
                                      "gate_cap": float(m["gate_cap"]), "norm_eps": eps})
        if layer["type"] == "latent_attention":
            return PartSpec("latent_attention", {**heads, "head_dim": int(m["dim"]), "rot_dim": 0, "value_dim": int(m["vdim"]),
                                                 "kv_rank": int(m["kv_rank"]), "scale": float(m["scale"]), "norm_eps": eps,
                                                 "gate": True})
        return PartSpec("gqa_attention", {
            **heads, "num_kv_heads": int(m["kv_heads"]), "head_dim": int(m["dim"]), "value_dim": int(m["vdim"]),
            "scale": float(m["scale"]), "chunk": int((m.get("mask") or {}).get("size", 0)), "qk_norm_eps": eps,
            "difference": {"diff": float(m["diff"])}, "head_gate": True,
            "names": {"q": "q", "k": "k", "v": "v", "o": "o", "q_norm": "q.norm", "k_norm": "k.norm", "gate": "g"}})

    def _feed_forward(self, f) -> PartSpec:
        if f is None:
            return PartSpec("none")
        if f.get("kind", "dense") == "dense":
            return PartSpec("plain_unit", {"hidden_size": self.width, "intermediate_size": int(f["ff"]), "activation": "relu2"})
        router, shared = f["router"], f.get("shared")
        return PartSpec("routed_experts", {
            "hidden_size": self.width, "expert_size": int(f["expert"]["ff"]), "experts": int(router["experts"]),
            "top": int(router["top"]), "score": "sigmoid", "activation": "swiglu", "scale": "output", "correction": True,
            "renormalize": float(router["scale"]), "groups": router.get("groups"),
            "shared": {"ff": int(shared["ff"])} if shared else None})

    def model_spec(self) -> ModelSpec:
        width, vocab = self.width, self.vocab
        norm = PartSpec("layernorm", {"width": width, "eps": self.eps, "tensor": "", "bias": "b"})
        block = PartSpec("sandwich_norm", {"names": {
            "mixer_norm": "norm1", "mixer": "mix", "feed_forward_norm": "norm2", "feed_forward": "mlp",
            "mixer_post_norm": "norm1b", "feed_forward_post_norm": "norm2b"}})
        layers, optional = [], []
        for i, layer in enumerate(self.layers):
            feed_forward = self._feed_forward(layer.get("mlp"))
            if feed_forward.kind == "none":
                optional += [f"l{i}.{name}{b}" for name in ("norm2", "norm2b") for b in ("", ".b")]
            layers.append(LayerSpec(prefix=f"l{i}", block=block, mixer=self._mixer(layer), feed_forward=feed_forward,
                                    mixer_norm=norm, feed_forward_norm=norm, position=PartSpec("none"),
                                    extra={"mixer_post_norm": norm, "feed_forward_post_norm": norm}))
        return ModelSpec(
            architecture="Tesozen", hidden_size=width, vocab_size=vocab,
            max_positions=int(self.raw.get("max_positions", DEFAULT_MAX_POSITIONS)),
            embedding=PartSpec("pair_embedding", {"vocab_size": vocab, "width": width, "tensor": "",
                                                  "scale": float(self.raw["embedding"]["scale"])}),
            final_norm=norm, head=PartSpec("linear_head", {"vocab_size": vocab, "width": width, "tied": True}),
            layers=tuple(layers), schedule=tuple(LayerRun(layer=i, cache=i) for i in range(len(layers))),
            names={"embedding": "embed", "final_norm": "final.norm", "head": "head"}, optional_tensors=tuple(optional))
