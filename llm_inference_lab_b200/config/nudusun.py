"""Nudusun: a post-norm decoder on a 32-bit residual stream that mixes a gated delta rule and differential attention
with a sliding window, with routed experts and a token's own side vector in every layer.

config.json keys: ``vocab``, ``width``, ``max_positions`` (rows of the learned position table), ``embedding.scale``,
``norm.eps``, ``postln_alpha`` (what multiplies the stream before a sublayer's result joins it), ``token_side.dim``
(a layer's part of a token's side vector; absent: no such input) and ``layers``, a list whose entries give ``type``
(the mixer), ``mixer`` (its sizes and constants) and ``mlp`` (or null for a layer without a feed-forward):

``delta``
    the gated delta rule (``heads``, ``kv_heads``, ``dim``, ``vdim``, ``conv`` taps of the short convolutions).
``attention``
    differential attention (``heads``, ``kv_heads``, ``dim``, ``vdim``, ``scale``, ``diff``), q and k normed per head
    and map, no rotation; ``softcap`` on the scores (absent: none); a window of ``mask.size`` keys (``mask`` absent:
    every earlier key).

``mlp.kind`` is ``moe``: ``router.experts`` experts of ``expert.ff`` rows with gates capped at ``expert.limit`` and
``router.identity`` identity experts, of which a token uses ``router.top``; softmax scores over all of them, a
correction for the choice, ``router.groups`` (``count``, ``keep``), weights times ``router.scale``; ``shared`` (``ff``,
``limit``; absent: none) runs for every token.

Each layer is x <- norm1(alpha x + mixer(x)), x <- norm2(alpha x + ff(x)), then x <- x + norm(side(x)).  Tensor names:
``embed``, ``pos``, ``side.embed``, ``l<i>.norm1|norm2``, ``l<i>.mix.*``, ``l<i>.mlp.*``, ``l<i>.side.*``,
``final.norm``, ``head``.
"""
from __future__ import annotations

import dataclasses
from typing import Any

from .base import ConfigError, ModelConfig, finite_positive, optional, positive, required
from ..parts.spec import LayerCall, LayerSpec, ModelBlueprint, PartSpec

MIXER_TYPES = ("delta", "attention")
# Added under the root where q and k of the delta rule become unit vectors: fixed by the design.
UNIT_EPS = 1e-6


def _need(obj: Any, key: str, where: str, kind=(int, float)):
    if not isinstance(obj, dict) or key not in obj:
        raise ConfigError(f"config.json of Nudusun lacks {where}.{key}")
    value = obj[key]
    if isinstance(value, bool) or not isinstance(value, kind):
        raise ConfigError(f"config key {where}.{key} has the wrong type: {value!r}")
    return value


def _positive_int(obj, key, where) -> int:
    value = _need(obj, key, where, (int,))
    if value <= 0:
        raise ConfigError(f"config key {where}.{key} must be positive, got {value!r}")
    return int(value)


def _check_expert(expert, where) -> None:
    _positive_int(expert, "ff", where)
    finite_positive(where + ".limit", _need(expert, "limit", where))


def _check_mlp(mlp, where) -> None:
    if not isinstance(mlp, dict) or mlp.get("kind") != "moe":
        raise ConfigError(f"{where}.kind must be 'moe' (or mlp null)")
    router = _need(mlp, "router", where, (dict,))
    at = where + ".router"
    experts, top = _positive_int(router, "experts", at), _positive_int(router, "top", at)
    finite_positive(at + ".scale", _need(router, "scale", at))
    if router.get("identity") is not None and _need(router, "identity", at, (int,)) < 0:
        raise ConfigError(f"{at}.identity must not be negative")
    outputs = experts + int(router.get("identity") or 0)
    open_ = outputs
    if router.get("groups") is not None:
        count, keep = (_positive_int(router["groups"], k, at + ".groups") for k in ("count", "keep"))
        if outputs % count or keep > count:
            raise ConfigError(f"{at}.groups: count must divide the {outputs} experts and keep must not exceed count")
        open_ = keep * (outputs // count)
    if top > open_:
        raise ConfigError(f"{at}.top must not exceed the {open_} experts that can be chosen")
    _check_expert(_need(mlp, "expert", where, (dict,)), where + ".expert")
    if mlp.get("shared") is not None:
        _check_expert(_need(mlp, "shared", where, (dict,)), where + ".shared")


@dataclasses.dataclass
class NudusunConfig(ModelConfig):
    architecture = "Nudusun"

    vocab: int = required(int, positive)
    width: int = required(int, positive)
    max_positions: int = required(int, positive, doc="rows of the learned position table")
    layers: Any = required("any")
    norm: Any = required("any")
    embedding: Any = required("any")
    postln_alpha: float = required(float, finite_positive)
    token_side: Any = optional("any", None)

    def validate(self) -> None:
        finite_positive("norm.eps", _need(self.norm, "eps", "norm"))
        finite_positive("embedding.scale", _need(self.embedding, "scale", "embedding"))
        if self.token_side is not None:
            _positive_int(self.token_side, "dim", "token_side")
        if not isinstance(self.layers, list) or not self.layers:
            raise ConfigError("'layers' must be a non-empty list")
        for i, layer in enumerate(self.layers):
            where = f"layers[{i}]"
            if not isinstance(layer, dict) or layer.get("type") not in MIXER_TYPES:
                raise ConfigError(f"{where}.type must be one of {MIXER_TYPES}, got "
                                  f"{layer.get('type') if isinstance(layer, dict) else layer!r}")
            m = layer.get("mixer")
            if not isinstance(m, dict):
                raise ConfigError(f"config.json of Nudusun lacks {where}.mixer")
            for key in ("heads", "kv_heads", "dim", "vdim"):
                _positive_int(m, key, where + ".mixer")
            if m["heads"] % m["kv_heads"]:
                raise ConfigError(f"{where}.mixer.heads must be a multiple of {where}.mixer.kv_heads")
            if layer["type"] == "delta":
                _positive_int(m, "conv", where + ".mixer")
            else:
                finite_positive(where + ".mixer.scale", _need(m, "scale", where + ".mixer"))
                _need(m, "diff", where + ".mixer")
                if m.get("softcap") is not None:
                    finite_positive(where + ".mixer.softcap", _need(m, "softcap", where + ".mixer"))
                if m.get("mask") is not None:
                    _positive_int(_need(m, "mask", where + ".mixer", (dict,)), "size", where + ".mixer.mask")
            if layer.get("mlp") is not None:
                _check_mlp(layer["mlp"], where + ".mlp")

    def to_dict(self) -> dict[str, Any]:
        out = {"architecture": self.architecture}
        out.update({k: v for k, v in dataclasses.asdict(self).items() if v is not None})
        return out


def _mixer(layer, width, eps, prefix) -> PartSpec:
    m = layer["mixer"]
    sizes = {"hidden": width, **{k: int(m[k]) for k in ("heads", "kv_heads", "dim", "vdim")}, "eps": eps}
    if layer["type"] == "delta":
        return PartSpec("gated_delta", {**sizes, "taps": int(m["conv"]), "unit_eps": UNIT_EPS}, prefix=prefix)
    return PartSpec("differential_attention", {
        **sizes, "scale": float(m["scale"]), "softcap": float(m.get("softcap") or 0.0), "diff": float(m["diff"]),
        "window": int(m["mask"]["size"]) if m.get("mask") else 0}, prefix=prefix)


def _feed_forward(mlp, width, prefix) -> PartSpec:
    router, shared, groups = mlp["router"], mlp.get("shared"), mlp["router"].get("groups")
    return PartSpec("routed_experts", {
        "hidden": width, "experts": router["experts"], "top": router["top"], "identity": int(router.get("identity") or 0),
        "expert_ff": mlp["expert"]["ff"], "limit": float(mlp["expert"]["limit"]), "renorm": False, "correction": True,
        "router_scale": float(router["scale"]), "groups": (groups["count"], groups["keep"]) if groups else None,
        "shared_ff": shared["ff"] if shared else 0, "shared_limit": float(shared["limit"]) if shared else 0.0},
        prefix=prefix)


def nudusun_blueprint(cfg: NudusunConfig) -> ModelBlueprint:
    """The design's layers as data: every size and constant comes from `cfg`; what the design fixes (the norms' form,
    the experts' gates, scores that are not renormalised, the correction of the choice) is set here as parameters of
    the parts."""
    eps, width = float(cfg.norm["eps"]), cfg.width
    side_dim = int(cfg.token_side["dim"]) if cfg.token_side is not None else 0
    layers = []
    for i, layer in enumerate(cfg.layers):
        p, mlp = f"l{i}.", layer.get("mlp")
        side = None
        if side_dim:
            side = PartSpec("token_gate", {"hidden": width, "dim": side_dim, "at": i * side_dim, "vocab": cfg.vocab,
                                           "table": "side.embed", "table_width": side_dim * len(cfg.layers)},
                            prefix=p + "side.")
        names = ("norm1",) + (("norm2",) if mlp is not None else ()) + (("side.norm",) if side is not None else ())
        norms = tuple(PartSpec("rmsnorm_stream", {"hidden": width, "eps": eps, "offset": 0.0, "name": n}, prefix=p)
                      for n in names)
        block = PartSpec("postnorm_stream", {"hidden": width, "alpha": float(cfg.postln_alpha), "side": side}, prefix=p)
        layers.append(LayerSpec("postnorm_stream", _mixer(layer, width, eps, p + "mix."),
                                _feed_forward(mlp, width, p + "mlp.") if mlp is not None else None, norms, hidden=width,
                                block_spec=block))
    return ModelBlueprint(
        hidden=width, vocab=cfg.vocab,
        embedding=PartSpec("token_position_embedding", {"vocab": cfg.vocab, "hidden": width, "table": "embed",
                                                        "positions": "pos", "max_positions": cfg.max_positions,
                                                        "scale": float(cfg.embedding["scale"])}),
        layers=tuple(layers), order=tuple(LayerCall(layer=i, cache=i) for i in range(len(layers))),
        final_norm=PartSpec("rmsnorm_stream", {"hidden": width, "eps": eps, "offset": 0.0, "name": "norm"},
                            prefix="final."),
        head=PartSpec("linear_head", {"vocab": cfg.vocab, "hidden": width, "tied_to": None, "name": "head"}),
        max_positions=cfg.max_positions, eos_token_ids=(), stream_f32=True)
