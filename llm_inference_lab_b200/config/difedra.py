"""Difedra: a pre-norm decoder on a 32-bit residual stream: windowed attention with norms over the whole query and key
projections, a learned sink and values mixed with an early layer's, before dense or routed feed-forwards.

config.json keys: ``vocab``, ``width``, ``norm.eps`` and ``layers``, a list whose entries give ``type``
(``attention``), ``mixer`` (its sizes and constants) and ``mlp`` (or null for a layer without a feed-forward):

``attention``
    grouped-query softmax attention (``heads``, ``kv_heads``, ``dim``, ``vdim``, ``scale``), no biases; q and k RMS-normed
    over their whole projections (``q.norm``, ``k.norm``); then rotary positions on the first ``rot.dims`` entries of
    a head, entry i paired with entry i + dims / 2 (``rot.base``; ``rot.scaling``: ``factor``, ``low``, ``high``,
    ``original``, frequencies scaled by their wavelength; absent: none); a window of ``mask.size`` keys (``mask``
    absent: every earlier key); a learned term per head in the softmax's denominator (``sink``).  ``v_mix`` true: the
    first such layer leaves its values, later ones mix them into their own with a learned number (``vmix``).

``mlp.kind`` is ``dense`` (``ff``; W_down (gelu(W_gate h) * (W_up h)), the tanh form) or ``moe``: ``router.experts``
experts of ``expert.ff`` rows with SiLU gates, of which a token uses ``router.top``; sigmoid scores, not renormalised,
that multiply the experts' inputs.  The head is the embedding table.  Tensor names: ``embed``, ``l<i>.norm1|norm2``,
``l<i>.mix.*``, ``l<i>.mlp.*``, ``final.norm``.
"""
from __future__ import annotations

import dataclasses
from typing import Any

from .base import ConfigError, ModelConfig, finite_positive, optional, positive, required
from ..parts.spec import LayerCall, LayerSpec, ModelBlueprint, PartSpec

SCALING_KEYS = ("factor", "low", "high", "original")


def _need(obj: Any, key: str, where: str, kind=(int, float)):
    if not isinstance(obj, dict) or key not in obj:
        raise ConfigError(f"config.json of Difedra lacks {where}.{key}")
    value = obj[key]
    if isinstance(value, bool) or not isinstance(value, kind):
        raise ConfigError(f"config key {where}.{key} has the wrong type: {value!r}")
    return value


def _positive_int(obj, key, where) -> int:
    value = _need(obj, key, where, (int,))
    if value <= 0:
        raise ConfigError(f"config key {where}.{key} must be positive, got {value!r}")
    return int(value)


def _check_rot(m, where) -> None:
    rot = _need(m, "rot", where, (dict,))
    where += ".rot"
    finite_positive(where + ".base", _need(rot, "base", where))
    dims = _need(rot, "dims", where, (int,))
    if dims < 0 or dims % 2 or dims > m["dim"]:
        raise ConfigError(f"{where}.dims must be even and at most the mixer's dim, got {dims!r}")
    if rot.get("scaling") is not None:
        for key in SCALING_KEYS:
            finite_positive(f"{where}.scaling.{key}", _need(rot["scaling"], key, where + ".scaling"))
        if rot["scaling"]["low"] > rot["scaling"]["high"]:
            raise ConfigError(f"{where}.scaling.low must not exceed {where}.scaling.high")


def _check_mlp(mlp, where) -> None:
    if not isinstance(mlp, dict) or mlp.get("kind") not in ("dense", "moe"):
        raise ConfigError(f"{where}.kind must be 'dense' or 'moe' (or mlp null)")
    if mlp["kind"] == "dense":
        _positive_int(mlp, "ff", where)
        return
    router = _need(mlp, "router", where, (dict,))
    experts, top = _positive_int(router, "experts", where + ".router"), _positive_int(router, "top", where + ".router")
    if top > experts:
        raise ConfigError(f"{where}.router.top must not exceed {where}.router.experts")
    _positive_int(_need(mlp, "expert", where, (dict,)), "ff", where + ".expert")


@dataclasses.dataclass
class DifedraConfig(ModelConfig):
    architecture = "Difedra"

    vocab: int = required(int, positive)
    width: int = required(int, positive)
    layers: Any = required("any")
    norm: Any = required("any")
    max_positions: int = optional(int, 1 << 17, positive, doc="longest sequence the engine plans for")

    def validate(self) -> None:
        finite_positive("norm.eps", _need(self.norm, "eps", "norm"))
        if not isinstance(self.layers, list) or not self.layers:
            raise ConfigError("'layers' must be a non-empty list")
        values = None      # the width of the values that layers mix
        for i, layer in enumerate(self.layers):
            where = f"layers[{i}]"
            if not isinstance(layer, dict) or layer.get("type") != "attention":
                raise ConfigError(f"{where}.type must be 'attention', got "
                                  f"{layer.get('type') if isinstance(layer, dict) else layer!r}")
            m = layer.get("mixer")
            if not isinstance(m, dict):
                raise ConfigError(f"config.json of Difedra lacks {where}.mixer")
            for key in ("heads", "kv_heads", "dim", "vdim"):
                _positive_int(m, key, where + ".mixer")
            if m["heads"] % m["kv_heads"]:
                raise ConfigError(f"{where}.mixer.heads must be a multiple of {where}.mixer.kv_heads")
            finite_positive(where + ".mixer.scale", _need(m, "scale", where + ".mixer"))
            if m.get("rot") is not None:
                _check_rot(m, where + ".mixer")
            if m.get("mask") is not None:
                _positive_int(_need(m, "mask", where + ".mixer", (dict,)), "size", where + ".mixer.mask")
            if not isinstance(m.get("v_mix", False), (bool, type(None))):
                raise ConfigError(f"{where}.mixer.v_mix must be true or false, got {m['v_mix']!r}")
            if m.get("v_mix"):
                width = m["kv_heads"] * m["vdim"]
                if values is not None and width != values:
                    raise ConfigError(f"{where}.mixer mixes values of {width} numbers, the first such layer leaves {values}")
                values = width
            if layer.get("mlp") is not None:
                _check_mlp(layer["mlp"], where + ".mlp")

    def to_dict(self) -> dict[str, Any]:
        out = {"architecture": self.architecture}
        out.update(dataclasses.asdict(self))
        return out


def difedra_blueprint(cfg: DifedraConfig) -> ModelBlueprint:
    """The design's layers as data: every size and constant comes from `cfg`; what the design fixes (the norms over
    whole projections, the pairing of the rotation, the learned sink, the activations, scores that multiply the
    experts' inputs) is set here as parameters of the parts."""
    eps, width = float(cfg.norm["eps"]), cfg.width
    layers, mixed = [], False
    for i, layer in enumerate(cfg.layers):
        p, m = f"l{i}.", layer["mixer"]
        rot, mask, mlp = m.get("rot"), m.get("mask"), layer.get("mlp")
        scaling = rot.get("scaling") if rot else None
        v_mix = None
        if m.get("v_mix"):
            v_mix, mixed = "mix" if mixed else "first", True
        mixer = PartSpec("pair_rope_attention", {
            "hidden": width, "heads": m["heads"], "kv_heads": m["kv_heads"], "dim": m["dim"], "vdim": m["vdim"],
            "scale": float(m["scale"]), "window": int(mask["size"]) if mask else 0, "keep_first": 0, "bias": False,
            "sink_learned": True, "proj_norm": True, "eps": eps, "rot_layout": "halves",
            "rot_base": float(rot["base"]) if rot else 1.0, "rot_dims": int(rot["dims"]) if rot else 0,
            "rot_bands": tuple(float(scaling[k]) for k in SCALING_KEYS) if scaling else None, "v_mix": v_mix},
            prefix=p + "mix.")
        ffn = None
        if mlp is not None and mlp["kind"] == "dense":
            ffn = PartSpec("gated_mlp", {"hidden": width, "intermediate": mlp["ff"], "act": "gelu_tanh", "out_f32": True,
                                         "names": {"gate": "gate", "up": "up", "down": "down"}}, prefix=p + "mlp.")
        elif mlp is not None:
            ffn = PartSpec("routed_experts", {
                "hidden": width, "experts": mlp["router"]["experts"], "top": mlp["router"]["top"],
                "expert_ff": mlp["expert"]["ff"], "score": "sigmoid", "renorm": False, "scale_input": True},
                prefix=p + "mlp.")
        names = ("norm1", "norm2") if mlp is not None else ("norm1",)
        norms = tuple(PartSpec("rmsnorm_hyper", {"hidden": width, "eps": eps, "name": n}, prefix=p) for n in names)
        block = PartSpec("hyper_stream", {"hidden": width, "streams": 0, "ffn": mlp is not None}, prefix=p)
        layers.append(LayerSpec("hyper_stream", mixer, ffn, norms, hidden=width, block_spec=block))
    return ModelBlueprint(
        hidden=width, vocab=cfg.vocab,
        embedding=PartSpec("token_embedding_stream", {"vocab": cfg.vocab, "hidden": width, "table": "embed"}),
        layers=tuple(layers), order=tuple(LayerCall(layer=i, cache=i, write=True) for i in range(len(layers))),
        final_norm=PartSpec("rmsnorm_hyper", {"hidden": width, "eps": eps, "name": "norm"}, prefix="final."),
        head=PartSpec("linear_head", {"vocab": cfg.vocab, "hidden": width, "tied_to": "embed"}),
        max_positions=cfg.max_positions, eos_token_ids=(), stream_f32=True)
