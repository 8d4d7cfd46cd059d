"""Difedra on the CPU: configuration, registry, blueprint, tensor names, random-weights mode, the rotation's
frequencies, and properties of the plain mechanisms the GPU tests hold the engine against."""
import copy
import json
import math
import os

import numpy as np
import pytest

import plain_difedra as pd
from difedra_helpers import SMALL, SPREAD, attention, config, dense, moe, random_config, rot
from helpers import make_model_folder


def _resolve(cfg):
    from llm_inference_lab_b200.registry import resolve
    arch = resolve(cfg)
    return arch, arch.config_class.from_dict(cfg)


def test_registry_and_round_trip(tmp_path):
    cfg, _ = SMALL["A"]
    arch, typed = _resolve(cfg)
    assert arch.name == "Difedra" and typed.width == 72
    typed.save(str(tmp_path))
    with open(os.path.join(str(tmp_path), "config.json")) as fh:
        again = json.load(fh)
    assert again["architecture"] == "Difedra" and again["layers"] == cfg["layers"]
    assert _resolve(again)[1].to_dict() == typed.to_dict()


def test_windows_caches_and_mixed_values():
    from llm_inference_lab_b200.models.builder import cache_plan
    from llm_inference_lab_b200.parts.spec import PagedKV
    cfg, _ = SMALL["A"]
    arch, typed = _resolve(cfg)
    bp = arch.blueprint(typed)
    plan = cache_plan(bp)
    assert plan.group_windows == (20, 9, 33, 0)      # layers of one window share a block table; 0: all keys
    assert all(isinstance(n, PagedKV) for n in plan.needs)
    assert [n.n_kv_heads for n in plan.needs] == [2, 3, 1, 2] and [n.head_dim for n in plan.needs] == [32, 32, 48, 32]
    # the first layer that mixes leaves its values; layers that do not mix stay out of it
    assert [layer.mixer["v_mix"] for layer in bp.layers] == [None, "first", "mix", "mix"]
    assert [layer.mixer["rot_bands"] for layer in bp.layers][:3] == [(4.0, 1.0, 3.0, 60.0), (2.5, 0.5, 8.0, 200.0), None]
    assert bp.layers[3].mixer["rot_dims"] == 0 and bp.layers[2].ffn is None and bp.stream_f32
    assert bp.layers[1].ffn["score"] == "sigmoid" and bp.layers[1].ffn["scale_input"] and not bp.layers[1].ffn["renorm"]
    one_window, _ = SMALL["B"]
    same = copy.deepcopy(one_window)
    for layer in same["layers"]:
        layer["mixer"]["mask"]["size"] = 12
    arch, typed = _resolve(same)
    assert cache_plan(arch.blueprint(typed)).group_windows == (12,)


def test_tensor_names_and_shapes():
    from llm_inference_lab_b200.models.builder import expected_tensors
    arch, typed = _resolve(SMALL["A"][0])
    got = {t.name: tuple(t.shape) for t in expected_tensors(arch.blueprint(typed))}
    W = 72
    want = {"embed": (101, W), "final.norm": (W,), "l0.norm1": (W,), "l0.norm2": (W,), "l2.norm1": (W,),
            "l0.mix.q": (64, W), "l0.mix.k": (32, W), "l0.mix.v": (48, W), "l0.mix.o": (W, 96),
            "l0.mix.q.norm": (64,), "l0.mix.k.norm": (32,), "l0.mix.sink": (4,),
            "l1.mix.q.norm": (144,), "l1.mix.k.norm": (72,), "l1.mix.vmix": (), "l2.mix.vmix": (), "l2.mix.v": (48, W),
            "l2.mix.o": (W, 240), "l3.mix.vmix": (), "l0.mlp.gate": (56, W), "l0.mlp.up": (56, W), "l0.mlp.down": (W, 56),
            "l1.mlp.router": (5, W), "l1.mlp.e4.gate": (24, W), "l1.mlp.e0.down": (W, 24), "l3.mlp.e2.up": (16, W)}
    for name, shape in want.items():
        assert got.get(name) == shape, (name, got.get(name), shape)
    for absent in ("l0.mix.vmix", "l2.norm2", "l2.mlp.gate", "head", "l1.mlp.e5.gate", "l1.mlp.gate", "l0.mix.q.b"):
        assert absent not in got, absent


@pytest.mark.parametrize("path,value,needle", [
    (("vocab",), None, "vocab"), (("norm",), {}, "norm.eps"), (("layers",), [], "layers"),
    (("layers", 0, "type"), "mamba", "type"), (("layers", 0, "mixer", "heads"), 5, "kv_heads"),
    (("layers", 0, "mixer", "vdim"), 0, "vdim"), (("layers", 0, "mixer", "scale"), -1.0, "scale"),
    (("layers", 0, "mixer", "mask"), {"size": 0}, "size"), (("layers", 1, "mixer", "rot", "dims"), 7, "rot.dims"),
    (("layers", 1, "mixer", "rot", "dims"), 26, "rot.dims"), (("layers", 0, "mixer", "rot", "scaling", "low"), 9.0, "low"),
    (("layers", 0, "mixer", "rot", "scaling", "original"), None, "original"),
    (("layers", 2, "mixer", "v_mix"), 1, "v_mix"), (("layers", 2, "mixer", "vdim"), 24, "values"),
    (("layers", 1, "mlp", "router", "top"), 9, "top"), (("layers", 1, "mlp", "expert"), {}, "ff"),
    (("layers", 0, "mlp", "kind"), "conv", "kind"),
])
def test_configurations_that_are_refused(path, value, needle):
    from llm_inference_lab_b200.config.base import ConfigError
    cfg = copy.deepcopy(SMALL["A"][0])
    at = cfg
    for key in path[:-1]:
        at = at[key]
    if value is None:
        del at[path[-1]]
    else:
        at[path[-1]] = value
    with pytest.raises(ConfigError) as err:
        _resolve(cfg)
    assert needle in str(err.value)


def test_random_configurations_are_accepted():
    from llm_inference_lab_b200.models.builder import cache_plan, expected_tensors
    rng = np.random.default_rng(0)
    for _ in range(40):
        cfg, _ = random_config(rng)
        arch, typed = _resolve(cfg)
        bp = arch.blueprint(typed)
        assert expected_tensors(bp) and cache_plan(bp).needs


def test_random_weights_mode_is_read_by_the_plain_model(tmp_path):
    cfg, opt = SMALL["B"]
    folder = make_model_folder(str(tmp_path / "m"), cfg, opt["seed"], "float32", std=0.08, scales=SPREAD)
    pcfg, w = pd.read_folder(folder)
    assert w["l1.mix.vmix"].shape == () and 0.0 <= float(w["l1.mix.vmix"]) <= 1.0
    logits = pd.forward(pcfg, w, [3, 1, 4, 1, 5, 9, 2, 6])
    assert logits.shape == (8, cfg["vocab"]) and np.isfinite(logits).all()


@pytest.mark.parametrize("base,dims,bands", [(10000.0, 64, None), (500.0, 8, (4.0, 1.0, 3.0, 60)), (500000.0, 128, (8.0, 1.0, 4.0, 4096)),
                                             (30.0, 2, (2.0, 0.7, 0.7, 5)), (77.0, 0, None), (1000.0, 96, (32.0, 0.5, 9.0, 150))])
def test_frequencies_follow_the_plain_rule(base, dims, bands):
    from llm_inference_lab_b200.parts.rope import rope_frequencies
    got = rope_frequencies(base, dims, bands=bands)
    scaling = dict(zip(("factor", "low", "high", "original"), bands)) if bands else None
    want = pd.frequencies(base, dims, scaling)
    assert got.dtype == np.float32 and got.shape == want.shape and np.allclose(got, want, rtol=1e-6)
    assert np.allclose(rope_frequencies(base, dims, divide=3.0), pd.frequencies(base, dims) / 3.0, rtol=1e-6)
    if bands and dims > 8:       # all three bands are met, and the blend lies between its ends
        plain = pd.frequencies(base, dims)
        wave = 2 * math.pi / plain
        assert (wave < bands[3] / bands[2]).any() and (wave > bands[3] / bands[1]).any()
        mid = (wave > bands[3] / bands[2]) & (wave < bands[3] / bands[1])
        assert mid.any() and np.all(got[mid] < plain[mid]) and np.all(got[mid] > plain[mid] / bands[0] * (1 - 1e-6))


# ---------------------------------------------------------------------------------------------
# properties of the plain mechanisms
# ---------------------------------------------------------------------------------------------
def test_rotation_keeps_lengths_and_reads_differences():
    rng = np.random.default_rng(0)
    freq = pd.frequencies(100.0, 6)
    a, b = rng.standard_normal((1, 1, 8)), rng.standard_normal((1, 1, 8))
    at = lambda v, p: pd.rotate_halves(v, [p], freq)[0, 0]  # noqa: E731
    assert np.allclose(at(a, 5)[6:], a[0, 0, 6:])                                # the rest of the head passes
    assert np.isclose(np.sum(at(a, 9) ** 2), np.sum(a ** 2))
    assert np.isclose(at(a, 12) @ at(b, 7), at(a, 105) @ at(b, 100))             # scores depend on the distance alone
    # entry i turns with entry i + 3
    unit = np.zeros((1, 1, 8))
    unit[..., 0] = 1.0
    turned = at(unit, 1)
    assert np.isclose(turned[0], math.cos(1.0)) and np.isclose(turned[3], math.sin(1.0)) and turned[1] == 0.0


def test_window_sink_and_mixed_values():
    seen = pd.in_window(6, 3)
    assert seen.sum(1).tolist() == [1, 2, 3, 3, 3, 3] and seen[5].tolist() == [False, False, False, True, True, True]
    assert pd.in_window(4, None).sum() == 10 and np.array_equal(pd.in_window(5, 1), np.eye(5, dtype=bool))
    rng = np.random.default_rng(1)
    s = rng.standard_normal((2, 6, 6))
    assert np.allclose(pd.sink_softmax(s, seen[None], [-np.inf, -np.inf]).sum(-1), 1.0)
    one = pd.sink_softmax(s, seen[None], np.zeros(2))
    assert np.allclose(one.sum(-1), 1.0 - 1.0 / (1.0 + np.where(seen, np.exp(s), 0).sum(-1)))
    assert pd.sink_softmax(s, seen[None], [50.0, 50.0]).max() < 1e-18
    v, first = rng.standard_normal((3, 4)), rng.standard_normal((3, 4))
    assert np.allclose(pd.mixed_values(v, first, 0.0), v) and np.allclose(pd.mixed_values(v, first, 1.0), first)


def test_scores_multiply_the_experts_inputs():
    """With one expert the result is expert(s h): not s expert(h), since the expert is no linear map."""
    rng = np.random.default_rng(2)
    W, F = 6, 10
    w = {"m.e0.gate": rng.standard_normal((F, W)), "m.e0.up": rng.standard_normal((F, W)),
         "m.e0.down": rng.standard_normal((W, F)), "m.router": rng.standard_normal((1, W))}
    h = rng.standard_normal((4, W))
    s = pd.sigmoid(h @ w["m.router"].T)
    got = pd.routed_experts(h, w, "m.", moe(1, 1, F))
    assert np.allclose(got, pd.gated_mlp(s * h, w, "m.e0.", pd.silu))
    assert np.abs(got - s * pd.gated_mlp(h, w, "m.e0.", pd.silu)).max() > 0.01


def test_prefix_does_not_depend_on_what_follows(tmp_path):
    cfg, opt = SMALL["A"]
    folder = make_model_folder(str(tmp_path / "m"), cfg, opt["seed"], "float32", std=0.08, scales=SPREAD)
    pcfg, w = pd.read_folder(folder)
    ids = [int(t) for t in np.random.default_rng(2).integers(0, cfg["vocab"], size=40)]
    whole = pd.forward(pcfg, w, ids)
    assert np.allclose(pd.forward(pcfg, w, ids[:25]), whole[:25], atol=1e-9)
    # a stack of two windows reaches two windows back and no further
    two = config([attention(2, 1, 8, 8, window=4, turn=rot(10.0, 8), mlp=dense(16)), attention(2, 1, 8, 8, window=3)],
                 vocab=31, width=16)
    folder = make_model_folder(str(tmp_path / "two"), two, 3, "float32", std=0.08)
    pcfg, w = pd.read_folder(folder)
    ids = [int(t) for t in np.random.default_rng(3).integers(0, 31, size=12)]
    base = pd.forward(pcfg, w, ids)
    for p in range(12):
        other = list(ids)
        other[p] = (ids[p] + 1) % 31
        moved = np.abs(pd.forward(pcfg, w, other) - base).max(1) > 1e-9
        assert moved.nonzero()[0].tolist() == list(range(p, min(12, p + 6)))
