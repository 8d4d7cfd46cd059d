"""Nudusun on the CPU: configuration, registry, blueprint, tensor names, random-weights mode, and properties of the
plain mechanisms the GPU tests hold the engine against."""
import copy
import json
import os

import numpy as np
import pytest

import plain_nudusun as pn
from helpers import make_model_folder
from nudusun_helpers import SMALL, SPREAD, attention, config, delta, moe, random_config


def _resolve(cfg):
    from llm_inference_lab_b200.registry import resolve
    arch = resolve(cfg)
    return arch, arch.config_class.from_dict(cfg)


def test_registry_and_round_trip(tmp_path):
    cfg, _ = SMALL["A"]
    arch, typed = _resolve(cfg)
    assert arch.name == "Nudusun" and typed.width == 72 and typed.postln_alpha == 1.5
    typed.save(str(tmp_path))
    with open(os.path.join(str(tmp_path), "config.json")) as fh:
        again = json.load(fh)
    assert again["architecture"] == "Nudusun" and again["layers"] == cfg["layers"]
    assert _resolve(again)[1].to_dict() == typed.to_dict()


def test_blueprint_caches_and_groups():
    from llm_inference_lab_b200.models.builder import cache_plan, kernel_libraries
    from llm_inference_lab_b200.parts.spec import CacheParts, FixedState, PagedKV
    import torch
    arch, typed = _resolve(SMALL["A"][0])
    bp = arch.blueprint(typed)
    plan = cache_plan(bp)
    assert plan.group_windows == (20, 9) and bp.stream_f32 and bp.max_positions == 512
    # the delta rule keeps its state and the convolutions' inputs, attention pages of two keys a head beside one value
    assert plan.needs[0] == CacheParts((FixedState((4, 16, 24)), FixedState((2, 2 * 2 * 16 + 4 * 24))))
    assert plan.needs[1] == PagedKV(3, 32, 20) and plan.needs[2] == PagedKV(1, 48, 9)
    assert bp.layers[0].ffn["groups"] == (3, 2) and bp.layers[0].ffn["identity"] == 3 and not bp.layers[0].ffn["renorm"]
    assert bp.layers[1].ffn["groups"] is None and bp.layers[1].ffn["shared_ff"] == 0 and bp.layers[2].ffn is None
    assert [s.block_spec["side"]["at"] for s in bp.layers] == [0, 10, 20, 30]
    assert ("gated_delta", {}) in kernel_libraries(bp, torch.bfloat16)
    # two keys of 80 do not fit the tensor-core kernels' head: each map is a head of its own
    arch, typed = _resolve(SMALL["D"][0])
    needs = cache_plan(arch.blueprint(typed)).needs
    assert needs[0] == PagedKV(1, 128, 150) and needs[2] == PagedKV(4, 80, 97)
    # no window, no side vector
    arch, typed = _resolve(SMALL["B"][0])
    assert cache_plan(arch.blueprint(typed)).group_windows == (0, 4)
    arch, typed = _resolve(SMALL["C"][0])
    assert all(s.block_spec["side"] is None for s in arch.blueprint(typed).layers)


def test_tensor_names_and_shapes():
    from llm_inference_lab_b200.models.builder import expected_tensors
    arch, typed = _resolve(SMALL["A"][0])
    got = {t.name: tuple(t.shape) for t in expected_tensors(arch.blueprint(typed))}
    W = 72
    want = {"embed": (101, W), "pos": (512, W), "side.embed": (101, 40), "final.norm": (W,), "head": (101, W),
            "l0.mix.q": (32, W), "l0.mix.k": (32, W), "l0.mix.v": (96, W), "l0.mix.q.conv": (32, 3), "l0.mix.k.conv": (32, 3),
            "l0.mix.v.conv": (96, 3), "l0.mix.b": (4, W), "l0.mix.a": (4, W), "l0.mix.A_log": (4,), "l0.mix.dt_bias": (4,),
            "l0.mix.g": (96, W), "l0.mix.norm": (24,), "l0.mix.o": (W, 96),
            "l1.mix.q": (96, W), "l1.mix.k": (48, W), "l1.mix.v": (72, W), "l1.mix.q.norm": (8,), "l1.mix.k.norm": (8,),
            "l1.mix.lq1": (8,), "l1.mix.lk1": (8,), "l1.mix.lq2": (8,), "l1.mix.lk2": (8,), "l1.mix.o": (W, 144),
            "l0.mlp.router": (9, W), "l0.mlp.correction": (9,), "l1.mlp.router": (6, W), "l0.mlp.shared.gate": (40, W),
            "l0.mlp.shared.down": (W, 40), "l0.mlp.e5.up": (24, W), "l3.mlp.e7.down": (W, 16),
            "l2.side.gate": (10, W), "l2.side.proj": (W, 10), "l2.side.norm": (W,), "l0.norm1": (W,), "l0.norm2": (W,)}
    for name, shape in want.items():
        assert got.pop(name) == shape, name
    for name in ("l0.mlp.e6.gate", "l1.mlp.shared.gate", "l2.norm2", "l2.mlp.router"):
        assert name not in got, name


@pytest.mark.parametrize("change", [
    lambda c: c.pop("postln_alpha"), lambda c: c.update(postln_alpha=0.0), lambda c: c["embedding"].pop("scale"),
    lambda c: c.pop("max_positions"), lambda c: c["token_side"].update(dim=0), lambda c: c["norm"].update(eps=-1.0),
    lambda c: c["layers"][0].update(type="mamba"), lambda c: c["layers"][0]["mixer"].pop("conv"),
    lambda c: c["layers"][0]["mixer"].update(heads=5), lambda c: c["layers"][1]["mixer"].pop("diff"),
    lambda c: c["layers"][1]["mixer"].update(softcap=0.0), lambda c: c["layers"][1]["mixer"].update(mask={"size": 0}),
    lambda c: c["layers"][1]["mixer"].pop("scale"), lambda c: c["layers"][0]["mlp"].update(kind="dense"),
    lambda c: c["layers"][0]["mlp"]["expert"].pop("limit"), lambda c: c["layers"][0]["mlp"]["router"].pop("scale"),
    lambda c: c["layers"][0]["mlp"]["router"].update(identity=-1),
    lambda c: c["layers"][0]["mlp"]["router"].update(groups={"count": 4, "keep": 2}),
    lambda c: c["layers"][0]["mlp"]["router"].update(groups={"count": 3, "keep": 4}),
    lambda c: c["layers"][0]["mlp"]["router"].update(top=7), lambda c: c["layers"][0]["mlp"]["shared"].pop("limit"),
    lambda c: c.update(layers=[])])
def test_configurations_that_are_refused(change):
    from llm_inference_lab_b200.config.base import ConfigError
    cfg = copy.deepcopy(SMALL["A"][0])
    change(cfg)
    with pytest.raises(ConfigError):
        _resolve(cfg)


def test_random_weights_fit_the_model(tmp_path):
    from llm_inference_lab_b200.models.builder import expected_tensors
    cfg, opt = SMALL["B"]
    folder = make_model_folder(str(tmp_path / "m"), cfg, opt["seed"], "bfloat16", std=0.08, scales=SPREAD)
    pcfg, w = pn.read_folder(folder)
    arch, typed = _resolve(pcfg)
    assert set(w) == {t.name for t in expected_tensors(arch.blueprint(typed))}
    logits = pn.forward(pcfg, w, [3, 1, 4, 1, 5])
    assert logits.shape == (5, 89) and np.isfinite(logits).all()


def test_random_configurations_are_accepted():
    for trial in range(60):
        cfg, _ = random_config(np.random.default_rng(trial))
        arch, typed = _resolve(cfg)
        arch.blueprint(typed)


# ---- properties of the plain mechanisms ---------------------------------------------------------
def test_delta_rule_writes_what_it_reads_back():
    """With full rate and no decay, the state returns a value at its key; a second write at the same key replaces it."""
    rng = np.random.default_rng(0)
    k = pn.unit(rng.standard_normal((1, 6))).repeat(2, axis=0)
    v = rng.standard_normal((2, 5))
    o, S = pn.gated_delta_rule(k, k, v, np.ones(2), np.ones(2))
    assert np.abs(o - v).max() < 1e-5 and np.abs(S.T @ k[0] - v[1]).max() < 1e-5
    o, _ = pn.gated_delta_rule(k[:1], k[:1], v[:1], np.array([0.5]), np.array([1.0]), state=np.ones((6, 5)))
    assert np.abs(o - v[:1]).max() < 1e-5      # the decayed state's share at the key is removed as well


def test_convolution_starts_from_zeros():
    u = np.arange(1.0, 6.0)[:, None]
    w = np.array([[100.0, 10.0, 1.0]])
    assert list(pn.causal_conv(u, w)[:, 0]) == [1.0, 12.0, 123.0, 234.0, 345.0]


def test_choice_in_groups_with_negative_scores():
    """Experts outside the kept groups stay out although every choice score is negative; the correction decides the
    choice and not the weights."""
    s = np.full(6, 1 / 6)
    corr = np.array([-0.5, -0.9, -0.6, -0.55, -0.7, -0.8])
    assert pn.choose(s, corr, 2, 3, 1)[0] == [0, 1]
    assert pn.choose(s, corr, 3, 3, 2)[0] == [0, 3, 2]
    assert pn.choose(s, corr, 2, 1, 1)[0] == [0, 3]
    assert abs(pn.choose(s, corr, 2, 3, 1)[1] - 0.05) < 1e-9      # the groups' best, -0.5 against -0.55


def test_identity_experts_give_the_input_back():
    rng = np.random.default_rng(1)
    mlp = moe(1, 1, 4, identity=1, scale=2.0)
    w = {"router": np.zeros((2, 3)), "correction": np.array([-1.0, 1.0])}
    h = rng.standard_normal((4, 3))
    assert np.allclose(pn.routed_experts(h, w, "", mlp), 2.0 * 0.5 * h)


def test_window_and_difference():
    assert pn.in_window(4, 2).astype(int).tolist() == [[1, 0, 0, 0], [1, 1, 0, 0], [0, 1, 1, 0], [0, 0, 1, 1]]
    a = np.array([[3.0, 4.0]])
    out = pn.two_map_difference(a, 0 * a, 0.7, 0.0, 0.2)
    assert np.allclose(out, 0.8 * a / np.sqrt(12.5))
    p = {"lq1": np.array([1.0, 0.0]), "lk1": np.array([1.0, 5.0]), "lq2": np.zeros(2), "lk2": np.ones(2)}
    assert abs(pn.map_weight(p, "", 0.3) - (np.e - 1.0 + 0.3)) < 1e-12


def test_a_layer_reads_its_part_of_the_side_vector(tmp_path):
    """Changing one layer's part of a token's side vector changes nothing before that layer."""
    cfg = config([delta(2, 1, 4, 6), attention(1, 1, 4, 8, window=3), delta(1, 1, 4, 4)], vocab=31, width=20, side=3)
    folder = make_model_folder(str(tmp_path / "m"), cfg, 3, "float32", std=0.2, scales=SPREAD)
    pcfg, w = pn.read_folder(folder)
    a, b = [], []
    pn.forward(pcfg, w, [5, 6, 7], layers_out=a)
    w["side.embed"] = w["side.embed"].copy()
    w["side.embed"][:, 3:6] += 1.0
    pn.forward(pcfg, w, [5, 6, 7], layers_out=b)
    assert np.array_equal(a[0], b[0]) and np.abs(a[1] - b[1]).max() > 1e-3
