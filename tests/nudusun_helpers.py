"""Small Nudusun configurations for the tests.  Every size differs from one configuration to the next; none
has the sizes of a published model."""
from __future__ import annotations

import numpy as np


def moe(experts, top, ff, identity=0, groups=None, limit=1.2, scale=1.3, shared=None):
    """groups: (count, keep) or None; shared: (ff, limit) or None."""
    router = {"experts": experts, "top": top, "scale": scale, "identity": identity}
    if groups is not None:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    out = {"kind": "moe", "router": router, "expert": {"ff": ff, "limit": limit}}
    if shared is not None:
        out["shared"] = {"ff": shared[0], "limit": shared[1]}
    return out


def delta(heads, kv_heads, dim, vdim, conv=4, mlp=None):
    return {"type": "delta", "mlp": mlp,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def attention(heads, kv_heads, dim, vdim, window=None, softcap=None, diff=0.3, scale=1.0, mlp=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": float(scale), "diff": diff}
    if window is not None:
        m["mask"] = {"size": window}
    if softcap is not None:
        m["softcap"] = softcap
    return {"type": "attention", "mixer": m, "mlp": mlp}


def config(layers, vocab=97, width=48, eps=1e-5, alpha=1.5, side=6, scale=8.0, positions=512):
    out = {"architecture": "Nudusun", "vocab": vocab, "width": width, "layers": layers, "norm": {"eps": eps},
           "embedding": {"scale": scale}, "postln_alpha": alpha, "max_positions": positions}
    if side:
        out["token_side"] = {"dim": side}
    return out


# A: both mixers twice, values wider and narrower than keys, a window of one page and a bit, groups of experts with
# identities that make up a group and a part of one, a layer without a feed-forward
SMALL_A = config([delta(4, 2, 16, 24, conv=3, mlp=moe(6, 2, 24, identity=3, groups=(3, 2), shared=(40, 0.9))),
                  attention(6, 3, 8, 24, window=20, softcap=4.0, scale=0.9, diff=0.35, mlp=moe(5, 3, 16, identity=1)),
                  attention(2, 1, 24, 16, window=9, softcap=25.0, scale=0.4, diff=0.6),
                  delta(5, 1, 24, 8, conv=5, mlp=moe(8, 3, 16, groups=(4, 3), limit=0.7, shared=(24, 2.0)))],
                 vocab=101, width=72, side=10)
# B: one convolution tap (no kept inputs), as many key as query heads, no cap, no window, one expert of one, a side
# vector of one number
SMALL_B = config([attention(3, 3, 16, 8, softcap=None, scale=0.5, diff=0.1, mlp=moe(1, 1, 40)),
                  delta(3, 3, 40, 16, conv=1, mlp=moe(3, 2, 24, identity=5, groups=(2, 1), scale=2.1)),
                  attention(2, 1, 16, 32, window=4, softcap=8.0, scale=0.7, diff=0.45, mlp=moe(7, 4, 8, shared=(16, 1.5)))],
                 vocab=89, width=56, eps=1e-6, alpha=3.0, side=1, scale=20.0)
# C: a width that is no multiple of 8 (the products leave the tensor cores), one head everywhere, a window of the token
# itself alone, no side vector
SMALL_C = config([delta(1, 1, 20, 12, conv=2, mlp=moe(4, 1, 10, identity=1)),
                  attention(1, 1, 12, 20, window=1, softcap=3.0, scale=0.3, diff=0.2, mlp=moe(4, 2, 10, groups=(2, 1))),
                  attention(1, 1, 6, 10, window=30, scale=0.8, diff=0.5)],
                 vocab=67, width=50, eps=3e-6, alpha=1.0, side=0)
# D: keys of 64 (two of them fill the widest head of the tensor-core kernels) over one key/value head with long windows,
# keys of 80 whose maps are heads of their own, a delta rule with wide heads, many experts
SMALL_D = config([attention(5, 1, 64, 48, window=150, softcap=12.0, scale=0.3, diff=0.4, mlp=moe(12, 2, 40, identity=4, groups=(4, 2))),
                  delta(4, 2, 96, 40, conv=4, mlp=moe(6, 2, 48, shared=(120, 1.1))),
                  attention(4, 2, 80, 24, window=97, softcap=30.0, scale=0.2, diff=0.7, mlp=moe(16, 5, 32)),
                  attention(4, 1, 24, 64, window=260, softcap=6.0, scale=0.5, diff=0.25)],
                 vocab=113, width=64, side=16, scale=5.0, positions=700)
SMALL = {"A": (SMALL_A, dict(seed=41, page_size=16)), "B": (SMALL_B, dict(seed=42, page_size=4)),
         "C": (SMALL_C, dict(seed=43, page_size=32)), "D": (SMALL_D, dict(seed=44, page_size=16))}

# Random N(0, std) weights give decays that are all alike, a map weight that is `diff` alone, a router without
# preferences and corrections that hardly matter: all are scaled up.
SPREAD = {".router": 6.0, ".correction": 3.0, ".A_log": 25.0, ".lq": 5.0, ".lk": 5.0, ".conv": 6.0}


def sequences(rng, vocab, lengths):
    return {f"s{i}": [int(t) for t in rng.integers(0, vocab, size=n)] for i, n in enumerate(lengths)}


def plain_logits(folder, seqs, margin=None):
    """The plain model's logits; with `margin` also the (name, position) at which some router's choice hangs on less
    than that between two choice scores."""
    import plain_nudusun as pn
    cfg, w = pn.read_folder(folder)
    out, close = {}, set()
    for name, ids in seqs.items():
        margins = []
        out[name] = np.asarray(pn.forward(cfg, w, ids, margins=margins), dtype=np.float64)
        if margin is not None and margins:
            close |= {(name, int(p)) for p in np.nonzero(np.min(margins, axis=0) < margin)[0]}
    return out if margin is None else (out, close)


def random_config(rng):
    """A random Nudusun configuration and page size: one to five layers of either mixer, sizes that are multiples of 8
    or only of 2, any number of heads and groups, one to six convolution taps, windows of one token to longer than the
    sequences or none, with and without a cap, any number of experts, identities and groups of them, layers without a
    feed-forward, with and without a side vector."""
    def size(lo, hi, odd=False):
        return int(rng.choice([8, 8, 16, 2] + ([1] if odd else []))) * int(rng.integers(lo, hi))

    def ff():
        if rng.random() < 0.2:
            return None
        count = int(rng.choice([1, 1, 2, 3, 4]))
        per = int(rng.integers(1, 5))
        outputs = count * per
        identity = int(rng.integers(0, outputs))
        keep = int(rng.integers(1, count + 1))
        return moe(outputs - identity, int(rng.integers(1, keep * per + 1)), size(1, 8), identity=identity,
                   groups=(count, keep) if count > 1 or rng.random() < 0.3 else None, limit=float(rng.uniform(0.4, 3.0)),
                   scale=float(rng.uniform(0.5, 2.5)), shared=(size(1, 8), float(rng.uniform(0.4, 3.0))) if rng.random() < 0.5 else None)

    layers = []
    for _ in range(int(rng.integers(1, 6))):
        G = int(rng.choice([1, 1, 2, 3]))
        H = G * int(rng.choice([1, 2, 3, 5]))
        if rng.random() < 0.5:
            layers.append(delta(H, G, min(size(1, 12, True), 160), min(size(1, 12, True), 160), conv=int(rng.integers(1, 7)), mlp=ff()))
        else:
            dim = min(size(1, 12), 160)
            layers.append(attention(H, G, dim, min(size(1, 12), 160),
                                    window=None if rng.random() < 0.15 else int(rng.choice([1, 2, 7, 16, 33, 64, 65, 129, 400])),
                                    softcap=float(rng.uniform(2.0, 40.0)) if rng.random() < 0.8 else None,
                                    diff=float(rng.uniform(0.0, 0.9)), scale=float(rng.uniform(0.5, 4.0)) * dim ** -0.5, mlp=ff()))
    cfg = config(layers, vocab=int(rng.integers(30, 400)), width=size(3, 16), eps=float(rng.choice([1e-6, 1e-5])),
                 alpha=float(rng.uniform(0.8, 4.0)), side=int(rng.choice([0, 1, 8, 10, 24])), scale=float(rng.uniform(1.0, 30.0)))
    return cfg, int(rng.choice([16, 16, 4, 8, 32, 64]))
