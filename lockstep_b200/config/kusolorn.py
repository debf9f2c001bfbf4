"""Kusolorn: a decoder whose layers each name their own mixer, with a row of the token's own for every layer.

``config.json`` holds ``vocab``, ``width``, ``norm.eps``, an optional ``token_side`` = {``dim``} and a list ``layers``;
every entry gives ``type`` (which mixer), ``mixer`` (its sizes and constants) and ``mlp`` (its feed-forward, or null for
none).  Three mixers:

- ``attention``: grouped-query attention; rotation of neighbouring pairs of the first ``rot.dims`` elements of a head
  (base ``rot.base``, frequencies stretched by ``rot.scaling``), q and k divided by their root mean square per head,
  ``scale`` on the scores, scores capped (``softcap``), a sliding window of ``mask.size`` positions beside which the first
  ``mask.keep_first`` positions stay visible, a value size ``vdim`` of its own.  In layers with ``v_mix`` the values are
  mixed with those of the first such layer.
- ``mlstm``: a matrix memory with exponential gates (capped by ``gate_cap``), a running maximum and a normalizer.
- ``delta``: the gated delta rule with one decay per head, short causal convolutions (``conv`` taps) on q, k, v, and a
  gated per-head RMSNorm of the read-out.

The feed-forward is down(gelu(up(.))) (``kind`` "dense", ``ff``), or a mixture of experts (``kind`` "moe":
``router.experts``, ``router.top``, the weights a softmax over the chosen logits; ``expert.ff``, ``expert.limit``: gated
units with clamped inputs).  After it a layer adds its token input: rms(proj(gelu(gate(x)) e)) with e the layer's
``token_side.dim`` elements of the token's row in ``side.embed``.  Norms are RMS norms with a gain.  Layer i's tensors
start with ``l<i>.``: ``norm1``, ``mix.*``, ``norm2``, ``mlp.*``, ``side.*``.
"""

from __future__ import annotations

import copy
from typing import Any, Mapping

from .registry import register_architecture
from .spec import ConfigError, LayerRun, LayerSpec, ModelSpec, PartSpec

MIXERS = ("attention", "mlstm", "delta")
DEFAULT_MAX_POSITIONS = 32768
UNIT_EPS = 1e-6            # under the root when a delta mixer's q and k are made unit vectors
EXPERT_ALPHA = 1.702       # the slope in an expert's g sigmoid(alpha g)


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


@register_architecture("Kusolorn")
class KusolornConfig:
    def __init__(self, raw: Mapping[str, Any]):
        self.raw = copy.deepcopy(dict(raw))
        self.validate()

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any]) -> "KusolornConfig":
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

    @property
    def side_dim(self) -> int:
        return int((self.raw.get("token_side") or {}).get("dim", 0))

    def mixing_layers(self) -> list[int]:
        """The layers that mix values, the one they all mix in first."""
        return [i for i, layer in enumerate(self.layers) if layer["type"] == "attention" and layer["mixer"].get("v_mix")]

    def validate(self) -> None:
        r = self.raw
        _positive("config.json", r, "vocab", "width")
        _above_zero("norm", r.get("norm"), "eps")
        if r.get("token_side") is not None:
            _positive("token_side", r["token_side"], "dim")
        if not isinstance(r.get("layers"), list) or not r["layers"]:
            raise ConfigError("config.json: layers must be a list with at least one layer")
        for i, layer in enumerate(r["layers"]):
            where = f"layers[{i}]"
            kind = layer.get("type") if isinstance(layer, Mapping) else None
            if kind not in MIXERS:
                raise ConfigError(f"{where}: type {kind!r} is not one of {MIXERS}")
            m = layer.get("mixer")
            _positive(where + ".mixer", m, "heads", "dim", "vdim")
            if kind == "attention":
                self._validate_attention(where + ".mixer", m)
            elif kind == "mlstm":
                _above_zero(where + ".mixer", m, "gate_cap")
            else:
                _positive(where + ".mixer", m, "kv_heads", "conv")
                if m["heads"] % m["kv_heads"]:
                    raise ConfigError(f"{where}: heads must be a multiple of kv_heads")
            self._validate_feed_forward(where + ".mlp", layer.get("mlp"))
        mixing = self.mixing_layers()
        for i in mixing[1:]:
            first, m = self.layers[mixing[0]]["mixer"], self.layers[i]["mixer"]
            if first["kv_heads"] * first["vdim"] != m["kv_heads"] * m["vdim"]:
                raise ConfigError(f"layers[{i}]: its values do not have the sizes of layer {mixing[0]}'s, which it mixes in")

    @staticmethod
    def _validate_attention(where: str, m: Mapping[str, Any]) -> None:
        _positive(where, m, "kv_heads")
        _number(where, m, "scale")
        if m["heads"] % m["kv_heads"]:
            raise ConfigError(f"{where}: heads must be a multiple of kv_heads")
        if m.get("softcap") is not None:
            _above_zero(where, m, "softcap")
        rot = m.get("rot")
        if rot is not None:
            _positive(where + ".rot", rot, "dims")
            _above_zero(where + ".rot", rot, "base")
            if rot["dims"] % 2 or rot["dims"] > m["dim"]:
                raise ConfigError(f"{where}.rot: dims must be even and at most dim")
            if rot.get("scaling") is not None:
                _above_zero(where + ".rot.scaling", rot["scaling"], "factor", "low", "high", "original")
                if not float(rot["scaling"]["high"]) > float(rot["scaling"]["low"]):
                    raise ConfigError(f"{where}.rot.scaling: high must be above low")
        mask = m.get("mask")
        if mask is not None:
            _positive(where + ".mask", mask, "size")
            keep = mask.get("keep_first", 0)
            if not isinstance(keep, int) or isinstance(keep, bool) or keep < 0:
                raise ConfigError(f"{where}.mask: keep_first must be an integer that is not negative, got {keep!r}")

    @staticmethod
    def _validate_feed_forward(where: str, f) -> None:
        if f is None:
            return
        kind = f.get("kind", "dense") if isinstance(f, Mapping) else None
        if kind == "dense":
            _positive(where, f, "ff")
        elif kind == "moe":
            _positive(where + ".router", f.get("router"), "experts", "top")
            _positive(where + ".expert", f.get("expert"), "ff")
            _above_zero(where + ".expert", f.get("expert"), "limit")
            if f["router"]["top"] > f["router"]["experts"]:
                raise ConfigError(f"{where}: top must not exceed experts")
        else:
            raise ConfigError(f"{where}: feed-forward kind {kind!r} is not one of dense, moe")

    # -- the model as data --------------------------------------------------
    def _mixer(self, i: int) -> tuple[PartSpec, PartSpec]:
        layer, width, eps = self.layers[i], self.width, self.eps
        m = layer["mixer"]
        heads = {"hidden_size": width, "num_heads": int(m["heads"])}
        if layer["type"] == "mlstm":
            return PartSpec("mlstm", {**heads, "key_dim": int(m["dim"]), "value_dim": int(m["vdim"]),
                                      "gate_cap": float(m["gate_cap"]), "norm_eps": eps}), PartSpec("none")
        if layer["type"] == "delta":
            return PartSpec("gated_delta", {**heads, "num_kv_heads": int(m["kv_heads"]), "key_dim": int(m["dim"]),
                                            "value_dim": int(m["vdim"]), "conv_taps": int(m["conv"]), "norm_eps": eps,
                                            "unit_eps": UNIT_EPS, "decay": "head", "gate": "silu"}), PartSpec("none")
        position = PartSpec("none")
        rot = m.get("rot")
        if rot is not None:
            scaling = rot.get("scaling")
            position = PartSpec("scaled_rotary", {
                "dim": int(rot["dims"]), "theta": float(rot["base"]), "interleaved": True,
                "scaling": {"kind": "wavelength", **scaling} if scaling else None})
        mask, mixing = m.get("mask") or {}, self.mixing_layers()
        return PartSpec("gqa_attention", {
            **heads, "num_kv_heads": int(m["kv_heads"]), "head_dim": int(m["dim"]), "value_dim": int(m["vdim"]),
            "scale": float(m["scale"]), "softcap": float(m.get("softcap") or 0.0), "window": int(mask.get("size", 0)),
            "keep_first": int(mask.get("keep_first", 0)), "qk_norm_eps": eps, "qk_norm_gain": False,
            "value_mix": None if i not in mixing else "first" if i == mixing[0] else "later",
            "names": {"q": "q", "k": "k", "v": "v", "o": "o", "v_mix": "vmix"}}), position

    def _feed_forward(self, f) -> PartSpec:
        if f is None:
            return PartSpec("none")
        if f.get("kind", "dense") == "dense":
            return PartSpec("plain_unit", {"hidden_size": self.width, "intermediate_size": int(f["ff"])})
        return PartSpec("routed_experts", {
            "hidden_size": self.width, "expert_size": int(f["expert"]["ff"]), "experts": int(f["router"]["experts"]),
            "top": int(f["router"]["top"]), "score": "softmax_chosen", "activation": "clamped_glu", "scale": "output",
            "limit": float(f["expert"]["limit"]), "alpha": EXPERT_ALPHA})

    def model_spec(self) -> ModelSpec:
        width, vocab, side = self.width, self.vocab, self.side_dim
        norm = PartSpec("rmsnorm", {"width": width, "eps": self.eps, "tensor": ""})
        mixing = self.mixing_layers()
        # the first layer that mixes values may store a number of its own, which nothing reads
        layers, optional = [], [f"l{i}.mix.vmix" for i in mixing[:1]]
        for i, layer in enumerate(self.layers):
            mixer, position = self._mixer(i)
            feed_forward = self._feed_forward(layer.get("mlp"))
            if feed_forward.kind == "none":
                optional.append(f"l{i}.norm2")
            extra = {}
            if side:
                extra["side"] = PartSpec("token_input", {"hidden_size": width, "dim": side, "at": i * side,
                                                         "table": "token_side", "norm_eps": self.eps})
            block = PartSpec("pre_norm", {"names": {"mixer_norm": "norm1", "mixer": "mix", "feed_forward_norm": "norm2",
                                                    "feed_forward": "mlp", "side": "side"}})
            layers.append(LayerSpec(prefix=f"l{i}", block=block, mixer=mixer, feed_forward=feed_forward, mixer_norm=norm,
                                    feed_forward_norm=norm, position=position, extra=extra))
        shared = {}
        if side:
            shared["token_side"] = PartSpec("token_table", {"vocab_size": vocab, "columns": side * len(layers), "tensor": "embed"})
        return ModelSpec(
            architecture="Kusolorn", hidden_size=width, vocab_size=vocab,
            max_positions=int(self.raw.get("max_positions", DEFAULT_MAX_POSITIONS)),
            embedding=PartSpec("token_embedding", {"vocab_size": vocab, "width": width, "tensor": ""}),
            final_norm=norm,
            head=PartSpec("linear_head", {"vocab_size": vocab, "width": width, "tensor": ""}),
            layers=tuple(layers), schedule=tuple(LayerRun(layer=i, cache=i) for i in range(len(layers))),
            names={"embedding": "embed", "final_norm": "final.norm", "head": "head", "token_side": "side"},
            optional_tensors=tuple(optional), shared=shared)
