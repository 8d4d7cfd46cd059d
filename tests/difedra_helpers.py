"""Small Difedra configurations for the tests.  Every size differs from one configuration to the next; none
has the sizes of a published model."""
from __future__ import annotations

import numpy as np


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}


def rot(base, dims, scaling=None):
    """scaling: (factor, low, high, original) or None."""
    out = {"base": base, "dims": dims}
    if scaling is not None:
        out["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return out


def attention(heads, kv_heads, dim, vdim, window=None, turn=None, scale=1.0, v_mix=False, mlp=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": float(scale), "v_mix": v_mix}
    if window is not None:
        m["mask"] = {"size": window}
    if turn is not None:
        m["rot"] = turn
    return {"type": "attention", "mixer": m, "mlp": mlp}


def config(layers, vocab=97, width=48, eps=1e-5):
    return {"architecture": "Difedra", "vocab": vocab, "width": width, "layers": layers, "norm": {"eps": eps}}


# A: windows of several sizes and none, a first layer that mixes no values, mixed values under two ways of cutting
# them into heads, a rotation of part of a head in all three bands, a layer without a feed-forward
SMALL_A = config([attention(4, 2, 16, 24, window=20, turn=rot(500.0, 8, (4.0, 1.0, 3.0, 60)), scale=0.35, mlp=dense(56)),
                  attention(6, 3, 24, 16, window=9, turn=rot(90.0, 24, (2.5, 0.5, 8.0, 200)), scale=0.3, v_mix=True,
                            mlp=moe(5, 2, 24)),
                  attention(5, 1, 8, 48, window=33, turn=rot(2000.0, 8), scale=0.5, v_mix=True),
                  attention(4, 2, 32, 24, scale=0.25, v_mix=True, mlp=moe(3, 3, 16))],
                 vocab=101, width=72)
# B: routed experts in the first layer, one expert of one, as many key/value heads as query heads, a window of one
# page, values from the first layer on
SMALL_B = config([attention(3, 3, 40, 8, window=4, turn=rot(10000.0, 40), scale=0.2, v_mix=True, mlp=moe(1, 1, 40)),
                  attention(3, 3, 8, 8, window=64, turn=rot(300.0, 4, (8.0, 1.0, 4.0, 2048)), scale=0.6, v_mix=True,
                            mlp=dense(24)),
                  attention(2, 1, 16, 32, window=11, turn=rot(700.0, 16), scale=0.4, mlp=moe(7, 4, 8))],
                 vocab=89, width=56, eps=1e-6)
# C: a width that is no multiple of 8 (the products leave the tensor cores), one head everywhere, a window of the
# token itself alone, a rotation of one pair, nothing mixed but by one layer
SMALL_C = config([attention(1, 1, 20, 12, window=1, turn=rot(50.0, 2), scale=0.3, mlp=dense(34)),
                  attention(1, 1, 12, 20, window=30, turn=rot(1000.0, 12, (3.0, 2.0, 2.0, 40)), scale=0.4, v_mix=True,
                            mlp=moe(4, 1, 10))],
                 vocab=67, width=50, eps=3e-6)
# D: heads of 64 entries over one key/value head with long windows, many experts of which one is used
SMALL_D = config([attention(10, 1, 64, 48, window=150, turn=rot(100000.0, 32, (16.0, 1.0, 4.0, 512)), scale=0.11, v_mix=True,
                            mlp=moe(12, 1, 40)),
                  attention(4, 1, 64, 48, window=97, turn=rot(100000.0, 64), scale=0.15, v_mix=True, mlp=dense(120)),
                  attention(2, 1, 128, 48, window=260, turn=rot(4000.0, 96, (2.0, 1.0, 5.0, 300)), scale=0.09, v_mix=True,
                            mlp=moe(16, 5, 32))],
                 vocab=113, width=64)
SMALL = {"A": (SMALL_A, dict(seed=31, page_size=16)), "B": (SMALL_B, dict(seed=32, page_size=4)),
         "C": (SMALL_C, dict(seed=33, page_size=32)), "D": (SMALL_D, dict(seed=34, page_size=16))}

# Random N(0, std) weights give sinks near zero and a router without preferences: both are scaled up.
SPREAD = {".router": 6.0, ".sink": 20.0}


def sequences(rng, vocab, lengths):
    return {f"s{i}": [int(t) for t in rng.integers(0, vocab, size=n)] for i, n in enumerate(lengths)}


def plain_logits(folder, seqs):
    import plain_difedra as pd
    cfg, w = pd.read_folder(folder)
    return {name: np.asarray(pd.forward(cfg, w, ids), dtype=np.float64) for name, ids in seqs.items()}


def close_calls(folder, seqs, margin):
    """The (name, position) at which some router's choice hangs on less than `margin` between two logits."""
    import plain_difedra as pd
    cfg, w = pd.read_folder(folder)
    out = set()
    for name, ids in seqs.items():
        margins = []
        pd.forward(cfg, w, ids, margins=margins)
        if margins:
            out |= {(name, int(p)) for p in np.nonzero(np.min(margins, axis=0) < margin)[0]}
    return out


def random_config(rng):
    """A random Difedra configuration and page size: one to five layers, sizes that are multiples of 8 or only of 2,
    any number of heads and groups, windows of one token to longer than the sequences or none, rotations of none
    to all of a head with and without bands, any layers mixing values, dense, routed or no feed-forward."""
    def size(lo, hi):
        return int(rng.choice([8, 8, 16, 2])) * int(rng.integers(lo, hi))

    def ff():
        kind = rng.choice(["none", "dense", "moe", "moe"])
        if kind == "dense":
            return dense(size(2, 20))
        if kind == "moe":
            experts = int(rng.integers(1, 10))
            return moe(experts, int(rng.integers(1, experts + 1)), size(1, 8))
        return None

    mixed = None       # (groups, values) of the layers that mix
    layers = []
    for _ in range(int(rng.integers(1, 6))):
        G, vdim = int(rng.choice([1, 1, 2, 3])), min(size(1, 12), 160)
        v_mix = bool(rng.random() < 0.7)
        if v_mix:
            if mixed is None:
                mixed = G * vdim
            else:
                G = int(rng.choice([g for g in (1, 2, 3, 4, 6) if mixed % g == 0]))
                vdim = mixed // G
                if vdim > 160:
                    v_mix = False
                    vdim = 16
        dim = min(size(1, 12), 160)
        turn = None
        if rng.random() < 0.85:
            low = float(rng.uniform(0.5, 2.0))
            scaling = (float(rng.choice([2.0, 8.0])), low, low + float(rng.uniform(0.0, 4.0)), int(rng.choice([30, 150, 2048])))
            turn = rot(float(rng.choice([30.0, 10000.0, 500000.0])), 2 * int(rng.integers(0, dim // 2 + 1)),
                       scaling if rng.random() < 0.6 else None)
        layers.append(attention(G * int(rng.choice([1, 2, 4, 5, 8])), G, dim, vdim,
                                window=None if rng.random() < 0.15 else int(rng.choice([1, 2, 7, 16, 33, 64, 65, 129, 400])),
                                turn=turn, scale=float(rng.uniform(0.5, 2.0)) * dim ** -0.5, v_mix=v_mix, mlp=ff()))
    cfg = config(layers, vocab=int(rng.integers(30, 400)), width=size(3, 16), eps=float(rng.choice([1e-6, 1e-5])))
    return cfg, int(rng.choice([16, 16, 4, 8, 32, 64]))
