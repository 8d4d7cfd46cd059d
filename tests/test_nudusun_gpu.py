"""Nudusun on the GPU against the plain implementation (tests/plain_nudusun.py): each mechanism
alone, then whole models under every way of cutting a trace, then generation through the scheduler."""
import os

import numpy as np
import pytest

import plain_nudusun as pn
from helpers import (error_stats, make_model_folder, run_trace_inprocess, run_trace_program, tokens_needed,
                     trace_mixed, trace_portions, trace_tail_decode, trace_whole)
from nudusun_helpers import SMALL, SPREAD, attention, config, delta, moe, plain_logits, random_config, sequences
from ritizen_helpers import make_ctx

pytestmark = pytest.mark.gpu

F32_MAX = 2e-4      # largest error over the largest logit, 32-bit engine against the 64-bit plain model
BF16_MAX, BF16_RMS = 0.10, 0.04
CLOSE = 0.01        # between two choice scores (softmax scores with a correction)


def _torch():
    import torch
    return torch


def _t(a, dtype=None):
    torch = _torch()
    t = torch.from_numpy(np.ascontiguousarray(a, dtype=np.float32)).cuda()
    return t if dtype is None else t.to(dtype)


def _np(t):
    return t.double().cpu().numpy()


def _summed(t):
    a = _np(t)
    return a.sum(0) if a.ndim == 3 else a


def _dtypes():
    torch = _torch()
    return (torch.float32, torch.bfloat16)


# ---------------------------------------------------------------------------------------------
# the gated delta rule
# ---------------------------------------------------------------------------------------------
def _dots(q, k, q_start):
    """The products of every row's q and k [T, G, D] with the keys of its block of four packed rows, as far as they are
    the request's own: [T, G, 8]."""
    T, G, _ = q.shape
    out = np.zeros((T, G, 8))
    for r in range(len(q_start) - 1):
        for t in range(q_start[r], q_start[r + 1]):
            for j in range(max(t // 4 * 4, q_start[r]), t + 1):
                out[t, :, j % 4] = (q[t] * k[j]).sum(-1)
                if j < t:
                    out[t, :, 4 + j % 4] = (k[t] * k[j]).sum(-1)
    return out


def _records(q, k, q_start):
    """The rows' records [G, T, floats]: k in four shares with four zeros behind each, q likewise, the products."""
    from llm_inference_lab_b200.kernels import ops
    T, G, D = q.shape
    floats, share = ops.delta_record(D)
    assert floats == 8 * (share + 4) + 8 and 4 * share >= D
    out = np.zeros((G, T, floats))
    for e in range(D):
        at = e // share * (share + 4) + e % share
        out[:, :, at], out[:, :, 4 * (share + 4) + at] = k[:, :, e].T, q[:, :, e].T
    out[:, :, -8:] = _dots(q, k, q_start).transpose(1, 0, 2)
    return out


def _walk(q, k, v, decay, rate, state, lens, slots, **more):
    """`ops.delta_walk` over rows of q, k [T, G, D], v [T, H, V]: [T, H, V]."""
    from llm_inference_lab_b200.kernels import ops
    (T, G, D), (_, H, V) = q.shape, v.shape
    ctx, _ = make_ctx(lens, [0] * len(lens), slots, page_size=64)
    rec = _records(q, k, np.concatenate([[0], np.cumsum(lens)]))
    return _np(ops.delta_walk(_t(rec), _t(v.reshape(T, -1)), _t(decay.T), _t(rate.T), state, ctx, H, G, D, V, **more)).reshape(T, H, V)


@pytest.mark.parametrize("H,G,D,V", [(4, 2, 16, 24), (3, 3, 5, 7), (2, 1, 64, 64), (6, 2, 100, 33), (2, 2, 128, 40), (3, 1, 250, 16),
                                     (1, 1, 1, 1), (2, 1, 48, 130), (1, 1, 12, 8)])
def test_delta_rule_walk(H, G, D, V):
    """The recurrence from random states over portions of unequal length that start anywhere in a block of four rows, a
    request of padding between them; then the same rows one at a time; the states left behind; every shape of launch.
    Decays from almost nothing to almost one."""
    from llm_inference_lab_b200.kernels import ops
    rng = np.random.default_rng(D + V)
    lens, slots = [37, 1, 4, 2, 16, 65], [3, 0, -1, 5, 1, 6]
    T = sum(lens)
    q, k = rng.standard_normal((T, G, D)), pn.unit(rng.standard_normal((T, G, D)))
    v = rng.standard_normal((T, H, V))
    decay, rate = rng.random((T, H)) ** rng.choice([0.05, 1.0, 9.0], (T, H)), rng.random((T, H))
    start = rng.standard_normal((8, H, D, V))
    want, want_state = np.zeros((T, H, V)), start.copy()
    at = 0
    for n, slot in zip(lens, slots):
        for h in range(H):
            if slot >= 0:
                rows, g = slice(at, at + n), h // (H // G)
                want[rows, h], want_state[slot, h] = pn.gated_delta_rule(q[rows, g], k[rows, g], v[rows, h], decay[rows, h],
                                                                         rate[rows, h], start[slot, h])
        at += n
    real = np.concatenate([np.full(n, slot >= 0) for n, slot in zip(lens, slots)])
    tol = 3e-5 * max(1.0, np.abs(want).max())
    state_tol = 3e-5 * max(1.0, np.abs(want_state).max())
    state = _t(start)
    got = _walk(q, k, v, decay, rate, state, lens, slots, write=False)
    assert np.array_equal(_np(state), _np(_t(start)))       # a call that only reads leaves the state alone
    assert np.abs(got[real] - want[real]).max() < tol
    for shape in (None, (8, 1), (16, 1), (16, 2), (24, 1), (32, 1), (32, 2), (64, 2)):
        if D > 128 and shape is not None and shape[1] == 2:
            continue
        state = _t(start)
        assert np.abs(_walk(q, k, v, decay, rate, state, lens, slots, shape=shape)[real] - want[real]).max() < tol, shape
        assert np.abs(_np(state) - want_state).max() < state_tol, shape
    state, at = _t(start), 0
    for n, slot in zip(lens, slots):
        for t in range(at, at + n if slot >= 0 else at):
            r = slice(t, t + 1)
            assert np.abs(_walk(q[r], k[r], v[r], decay[r], rate[r], state, [1], [slot])[0] - want[t]).max() < tol
        at += n
    assert np.abs(_np(state) - want_state).max() < state_tol
    ops.take_device_errors()


def test_delta_rule_replaces_a_far_write():
    """A value written at a key stays readable hundreds of tokens later while other keys are written and nothing decays,
    and is gone after a write at the same key: prompt, portions of two and of seven, single tokens; also where the two
    writes fall into one block."""
    from llm_inference_lab_b200.kernels import ops
    D, V, T = 32, 8, 308
    for first, second in ((3, 250), (100, 103), (101, 102), (103, 104)):
        rng = np.random.default_rng(first)
        basis = np.eye(D)
        k = basis[rng.integers(1, D, size=T)]
        v = rng.standard_normal((T, V))
        k[first] = k[second] = basis[0]
        q = np.tile(basis[0], (T, 1))
        one = np.ones((T, 1))
        want, _ = pn.gated_delta_rule(q, k, v, one[:, 0], one[:, 0])
        assert np.allclose(want[first:second], v[first]) and np.allclose(want[second:], v[second])
        for sizes in ((T,), (2,) * (T // 2), (7,) * (T // 7), (1,) * T):
            state, at, outs = _t(np.zeros((1, 1, D, V))), 0, []
            for n in sizes:
                r = slice(at, at + n)
                outs.append(_walk(q[r, None], k[r, None], v[r, None], one[r], one[r], state, [n], [0])[:, 0])
                at += n
            assert np.abs(np.concatenate(outs) - want).max() < 1e-5
    ops.take_device_errors()


@pytest.mark.parametrize("H,G,D,V,taps", [(4, 2, 16, 24, 4), (3, 1, 5, 7, 1), (2, 2, 130, 9, 7), (5, 5, 1, 3, 2), (2, 1, 256, 40, 3)])
def test_delta_preparation(H, G, D, V, taps):
    """Convolutions across steps (portions shorter than the taps among them), unit vectors, rates and decays, the
    products with the keys of a row's block; a row of padding gives zeros; the kept inputs, renewed by the walk, and
    every other slot's left alone."""
    torch = _torch()
    from llm_inference_lab_b200.kernels import ops
    rng = np.random.default_rng(D)
    gd, hv = G * D, H * V
    ch, T = 2 * gd + hv, 30
    b_at, a_at = ch + 5, ch + 5 + H
    for dtype in _dtypes():
        w = _t(rng.standard_normal((ch, taps)), dtype)
        a_log, bias = _t(1.5 * rng.standard_normal(H), dtype), _t(rng.standard_normal(H), dtype)
        u = [rng.standard_normal((T, a_at + H)) * np.where(np.arange(a_at + H) >= a_at, 8.0, 1.0) for _ in range(2)]
        want = []
        for x in u:
            y = pn.silu(pn.causal_conv(x[:, :ch], _np(w)))
            qn, kn = pn.unit(y[:, :gd].reshape(T, G, D)) * 0.3, pn.unit(y[:, gd: 2 * gd].reshape(T, G, D))
            want.append((qn, kn, y[:, 2 * gd:],
                         np.exp(-np.exp(_np(a_log)) * pn.softplus(x[:, a_at: a_at + H] + _np(bias))),
                         pn.sigmoid(x[:, b_at: b_at + H])))
        kept = torch.zeros((4, max(taps - 1, 0), ch), device="cuda")
        state = torch.zeros((4, H, D, V), device="cuda")
        at = [0, 0]
        for n0, n1 in ((3, 1), (1, 2), (2, 9), (11, 1), (1, 5), (12, 12)):
            lens = [n0, 2, n1]
            ctx, _ = make_ctx(lens, [at[0], 0, at[1]], [2, -1, 0], page_size=64)
            proj = _t(np.concatenate([u[0][at[0]: at[0] + n0], 9.0 * np.ones((2, a_at + H)), u[1][at[1]: at[1] + n1]]))
            got = ops.delta_prepare(proj, b_at, a_at, taps, H, G, D, V, w, a_log, bias, kept, ctx, 0.3, 1e-6)
            q, k, v, decay, rate = (np.concatenate([want[0][i][at[0]: at[0] + n0], np.zeros_like(want[0][i][:2]),
                                                    want[1][i][at[1]: at[1] + n1]]) for i in range(5))
            rec = _records(q, k, [0, n0, n0 + 2, n0 + 2 + n1])
            for name, g, w_ in (("records", got[0], rec), ("v", got[1], v), ("decay", got[2], decay.T), ("rate", got[3], rate.T)):
                g = _np(g)
                if name == "records":
                    g[..., -1] = 0.0      # unused
                assert np.abs(g - w_).max() < 2e-5, name
            ops.delta_walk(*got, state, ctx, H, G, D, V, proj=proj, kept=kept, write=False)      # reads only
            ops.delta_walk(*got, state, ctx, H, G, D, V, proj=proj, kept=kept)
            at = [at[0] + n0, at[1] + n1]
            for slot, x, n in ((2, u[0], at[0]), (0, u[1], at[1])):
                last = np.concatenate([np.zeros((taps, ch)), _np(_t(x[:n, :ch]))])[len(x[:n]) + 1:] if taps > 1 else np.zeros((0, ch))
                assert np.array_equal(_np(kept[slot]), last)
        assert not kept[1].any() and not kept[3].any()
    ops.take_device_errors()


def test_norm_and_gate_per_head():
    """Each head over its own root mean square, a weight all heads share, SiLU of the gate; rows of padding are zeros."""
    torch = _torch()
    from llm_inference_lab_b200.kernels import ops
    rng = np.random.default_rng(1)
    for H, V in ((3, 10), (2, 130), (7, 1)):
        ctx, _ = make_ctx([4, 1, 2], [0, 0, 0], [0, -1, 2], page_size=64)
        o, g = rng.standard_normal((7, H, V)) * np.array([1e-3, 1.0, 50.0])[rng.integers(0, 3, (7, H, 1))], rng.standard_normal((7, H * V))
        o[4] = np.nan
        for dtype in _dtypes():
            w = _t(1 + 0.3 * rng.standard_normal(V), dtype)
            wide = _t(np.concatenate([g, g], axis=1))
            got = _np(ops.head_norm_gate(_t(o.reshape(7, -1)), wide[:, H * V:], w, ctx, H, V, 1e-5))
            want = pn.rms_norm(o, _np(w), 1e-5).reshape(7, -1) * pn.silu(g)
            keep = [0, 1, 2, 3, 5, 6]
            assert np.abs(got[keep] - want[keep]).max() < (1e-5 if dtype == torch.float32 else 0.05) and not got[4].any()


def _weights(mixer, width, rng):
    """Random weights of one mixer under the prefix `m.`."""
    m = mixer["mixer"]
    H, G, D, V = (m[k] for k in ("heads", "kv_heads", "dim", "vdim"))
    r = lambda *s: rng.standard_normal(s)  # noqa: E731
    if mixer["type"] == "delta":
        K = m["conv"]
        w = {"q": r(G * D, width), "k": r(G * D, width), "v": r(H * V, width), "g": r(H * V, width), "b": r(H, width),
             "a": r(H, width), "o": r(width, H * V)}
        w = {n: t / np.sqrt(t.shape[1]) for n, t in w.items()}
        w.update({"q.conv": r(G * D, K), "k.conv": r(G * D, K), "v.conv": r(H * V, K), "A_log": 2.0 * r(H), "dt_bias": r(H),
                  "norm": 1 + 0.3 * r(V)})
    else:
        w = {"q": r(2 * H * D, width), "k": r(2 * G * D, width), "v": r(G * V, width), "o": r(width, H * V)}
        w = {n: t / np.sqrt(t.shape[1]) for n, t in w.items()}
        w.update({"q.norm": 1 + 0.3 * r(D), "k.norm": 1 + 0.3 * r(D)})
        w.update({n: 0.7 * r(D) / np.sqrt(D) for n in ("lq1", "lk1", "lq2", "lk2")})
    return {"m." + n: t for n, t in w.items()}


def _mixer(mixer, w, dtype, eps):
    from llm_inference_lab_b200.config.nudusun import _mixer as spec_of
    from llm_inference_lab_b200.parts.base import lookup
    torch = _torch()
    spec = spec_of(mixer, w["m.o"].shape[0], eps, "m.")
    cls = lookup("mixer", spec.kind)
    assert {t.name: tuple(t.shape) for t in cls.tensors(spec)} == {n: t.shape for n, t in w.items()}
    return cls(spec, {n: _t(t, dtype) for n, t in w.items()}, dtype, torch.device("cuda:0"))


@pytest.mark.parametrize("mixer", [delta(4, 2, 16, 24, conv=3), delta(3, 1, 10, 6, conv=1), delta(2, 2, 72, 20, conv=6),
                                   delta(6, 1, 8, 40)])
def test_delta_mixer_under_every_cut(mixer):
    """The whole mixer in a prompt, in portions and token by token, on a slot that held another sequence before."""
    torch = _torch()
    from llm_inference_lab_b200.kernels import ops
    from llm_inference_lab_b200.parts.base import CacheView
    m = mixer["mixer"]
    rng = np.random.default_rng(m["dim"])
    width, T, eps = 40, 37, 1e-5
    raw = _weights(mixer, width, rng)
    for dtype in _dtypes():
        part = _mixer(mixer, raw, dtype, eps)
        w = {n: _np(_t(t, dtype)) for n, t in raw.items()}
        h = _t(rng.standard_normal((T, width)), dtype)
        want = pn.delta_mixer(_np(h), w, "m.", m, eps)
        tol = (5e-5 if dtype == torch.float32 else 0.05) * max(1.0, np.abs(want).max())
        states = [torch.zeros((3,) + s.shape, device="cuda") for s in part.cache_need(part.spec).parts]
        view = CacheView(need=None, parts=[CacheView(need=None, state=s) for s in states])
        for sizes in ((T,), (2, 9, 1, 16, 3, 6), (1,) * T):
            for s in states:
                s.zero_()
            at, outs = 0, []
            for n in sizes:
                ctx, _ = make_ctx([n], [at], [1], page_size=64, dtype=dtype)
                outs.append(_summed(part.forward(h[at: at + n], ctx, view)))
                at += n
            assert np.abs(np.concatenate(outs) - want).max() < tol, (dtype, sizes[:3])
            assert not states[0][0].any() and not states[0][2].any()
    ops.take_device_errors()


# ---------------------------------------------------------------------------------------------
# differential attention
# ---------------------------------------------------------------------------------------------
@pytest.mark.parametrize("H,G,D,V,packed", [(4, 2, 16, 40, True), (3, 3, 12, 8, True), (6, 2, 80, 24, False), (5, 1, 64, 130, True),
                                            (2, 2, 7, 10, True), (4, 1, 72, 96, False)])
def test_norm_per_head_and_map_in_the_store(H, G, D, V, packed):
    """q and k normed per head and map, two keys side by side in a head with the queries at their map's place and zeros
    around them (packed), or every map a head of its own beside the same values; from whole and from partial products;
    a row of padding stores nothing."""
    torch = _torch()
    from llm_inference_lab_b200.kernels import ops
    rng = np.random.default_rng(D)
    page, pages, eps = 4, 64, 1e-3
    ctx, _ = make_ctx([5, 1, 7], [3, 130, 0], [0, 1, 2], page_size=page, num_pages=pages, shuffle=rng.permutation(pages))
    T, head = 13, ops.padded_head(2 * D if packed else D, V)
    n_kv = G if packed else 2 * G
    for dtype in _dtypes():
        tol = 1e-5 if dtype == torch.float32 else 0.03
        wq, wk = _t(1 + 0.3 * rng.standard_normal(D), dtype), _t(1 + 0.3 * rng.standard_normal(D), dtype)
        for splits in (1, 3):
            proj = _t(rng.standard_normal((splits, T, 2 * (H + G) * D + G * V)))
            ck = torch.full((pages, n_kv, page, head), float("nan"), dtype=dtype, device="cuda")
            cv = torch.full_like(ck, float("nan"))
            slots = ctx.groups[0].row_slot.clone()
            slots[2] = -1
            q = ops.head_prep_store(proj if splits > 1 else proj[0], None, ctx.row_pos, None, 0, slots, ck, cv, 2 * H, n_kv, D, V,
                                    head, 2 * H * D, 2 * (H + G) * D, dtype, norm_eps=eps, q_norm_w=wq, k_norm_w=wk,
                                    maps=2 if packed else 1, v_rep=1 if packed else 2)
            full = _np(proj).sum(0)
            fq = pn.rms_norm(full[:, : 2 * H * D].reshape(T, H, 2, D), _np(wq), eps)
            fk = pn.rms_norm(full[:, 2 * H * D: 2 * (H + G) * D].reshape(T, G, 2, D), _np(wk), eps)
            fv = full[:, 2 * (H + G) * D:].reshape(T, G, V)
            got_q = _np(q).reshape(T, H, 2, head)
            for j in range(2):
                lo = j * D if packed else 0
                assert np.abs(got_q[:, :, j, lo: lo + D] - fq[:, :, j]).max() < tol
                assert not got_q[:, :, j, :lo].any() and not got_q[:, :, j, lo + D:].any()
            for t in range(T):
                s = int(slots[t])
                if s < 0:
                    continue
                rk, rv = _np(ck[s // page, :, s % page]), _np(cv[s // page, :, s % page])
                if packed:
                    assert np.abs(rk[:, : 2 * D] - fk[t].reshape(G, -1)).max() < tol and not rk[:, 2 * D:].any()
                    assert np.abs(rv[:, :V] - fv[t]).max() < tol
                else:
                    assert np.abs(rk[:, :D] - fk[t].reshape(2 * G, D)).max() < tol and not rk[:, D:].any()
                    assert np.abs(rv[:, :V] - np.repeat(fv[t], 2, axis=0)).max() < tol
                assert not rv[:, V:].any()
            s = int(ctx.groups[0].row_slot[2])
            assert torch.isnan(ck[s // page, :, s % page]).all() and torch.isnan(cv[s // page, :, s % page]).all()
    ops.take_device_errors()


def _fill_pages(ck, cv, table, r, k, v, page):
    """Keys and values k, v [L, G, D] of request r into its pages."""
    L = k.shape[0]
    for b in range(-(-L // page)):
        n = min(page, L - b * page)
        ck[table[r, b], :, :n] = k[b * page: b * page + n].transpose(0, 1)
        cv[table[r, b], :, :n] = v[b * page: b * page + n].transpose(0, 1)


def _capped_attention(q, k, v, pos_q, scale, window, cap):
    """q [n, H, D] at positions pos_q over keys k, v [L, G, D] at positions 0 .. L - 1."""
    n, H, _ = q.shape
    L, G = k.shape[:2]
    i, j = np.asarray(pos_q)[:, None], np.arange(L)[None, :]
    seen = (j <= i) & (i - j < (window or L + 1))
    s = pn.capped(np.stack([q[:, h] @ k[:, h // (H // G)].T for h in range(H)]) * scale, cap)
    p = pn.softmax(s, seen[None])
    return np.stack([p[h] @ v[:, h // (H // G)] for h in range(H)], axis=1)


@pytest.mark.parametrize("D,H,G,page,window,cap", [(16, 4, 2, 4, 9, 2.0), (48, 16, 1, 16, 33, 5.0), (64, 9, 1, 8, 141, 3.0),
                                                   (64, 4, 2, 16, 0, 0.7), (128, 3, 1, 32, 250, 30.0), (144, 2, 1, 16, 20, 4.0)])
def test_window_and_cap_in_every_attention_kernel(D, H, G, page, window, cap):
    """Random keys with scores well beyond the cap: long and short portions beside single tokens, near the start and
    far from it, on shuffled pages, in both storage types (prefill on tcgen05 and mma.sync, decode with split keys, the
    plain kernel); without the cap the results are far away."""
    torch = _torch()
    from llm_inference_lab_b200.kernels import ops
    rng = np.random.default_rng(D + window)
    q_lens, pos0 = [150, 1, 2, 1, 30, 1], [200, 700, 127, 3, 0, 0]
    pages = sum(-(-(n + p) // page) for n, p in zip(q_lens, pos0)) + 3
    ctx, table = make_ctx(q_lens, pos0, list(range(len(q_lens))), page_size=page, num_pages=pages,
                          shuffle=rng.permutation(pages))
    scale = 4.0 * D ** -0.5
    for dtype in _dtypes():
        ck = torch.zeros((pages, G, page, D), dtype=dtype, device="cuda")
        cv = torch.zeros_like(ck)
        keys, vals = [], []
        for r, (n, p0) in enumerate(zip(q_lens, pos0)):
            k, v = (_t(rng.standard_normal((p0 + n, G, D)), dtype) for _ in range(2))
            keys.append(_np(k)), vals.append(_np(v))
            _fill_pages(ck, cv, table, r, k, v, page)
        q = _t(rng.standard_normal((sum(q_lens), H * D)), dtype)
        wide = ops.attention(q, ck, cv, ctx, ctx.groups[0], H, G, D, window, scale, softcap=cap, out_f32=True)
        rounded = ops.attention(q, ck, cv, ctx, ctx.groups[0], H, G, D, window, scale, softcap=cap)
        assert wide.dtype == torch.float32 and rounded.dtype == dtype and torch.equal(wide.to(dtype), rounded)
        got = _np(wide)
        at = far = 0
        for r, (n, p0) in enumerate(zip(q_lens, pos0)):
            rows = _np(q[at: at + n]).reshape(n, H, D)
            want = _capped_attention(rows, keys[r], vals[r], range(p0, p0 + n), scale, window, cap)
            err = np.abs(got[at: at + n].reshape(n, H, D) - want).max()
            assert err < (1e-5 if dtype == torch.float32 else 0.03), (r, err)
            far = max(far, np.abs(want - _capped_attention(rows, keys[r], vals[r], range(p0, p0 + n), scale, window, None)).max())
            at += n
        assert far > (0.3 if cap < 10 else 0.03)
    ops.take_device_errors()


@pytest.mark.parametrize("n", [1, 2, 6, 140])
@pytest.mark.parametrize("D,page,window", [(64, 16, 150), (128, 32, 260), (32, 8, 65), (64, 8, 8)])
def test_window_edges_show_under_a_cap(n, D, page, window):
    """One key made to stand out up to the cap: the last row's output is its value while the key is the window's last
    place, and no part of it one place further; at page and tile borders; as the first token; for single tokens, short
    portions and portions of more than one tile of rows."""
    torch = _torch()
    from llm_inference_lab_b200.kernels import ops
    H, G, L, cap = 2, 1, 600, 25.0
    for dtype in _dtypes():
        for target in (L - 1, L - window, L - window - 1, L - window + 1, L - 17, L - page, L - 64, 128, 0):
            seen = 0 <= L - 1 - target < window
            rng = np.random.default_rng(target)
            pages = -(-L // page) + 3
            ctx, table = make_ctx([n], [L - n], [0], page_size=page, num_pages=pages, shuffle=rng.permutation(pages))
            k = 0.05 * rng.standard_normal((L, G, D))
            v = rng.standard_normal((L, G, D))
            k[target, 0, 3] = 90.0
            q = np.zeros((n, H, D))
            q[:, :, 3] = 1.0
            ck = torch.zeros((pages, G, page, D), dtype=dtype, device="cuda")
            cv = torch.zeros_like(ck)
            _fill_pages(ck, cv, table, 0, _t(k, dtype), _t(v, dtype), page)
            got = _np(ops.attention(_t(q.reshape(n, -1), dtype), ck, cv, ctx, ctx.groups[0], H, G, D, window, 1.0,
                                    softcap=cap))[-1].reshape(H, D)
            v_t = _np(_t(v[target, 0], dtype))
            if seen:
                assert np.abs(got - v_t).max() < 0.02, target
            else:
                want = _capped_attention(q[-1:], _np(_t(k, dtype)), _np(_t(v, dtype)), [L - 1], 1.0, window, cap)[0]
                assert np.abs(got - want).max() < 0.02 and np.abs(got - v_t).max() > 0.1, target
    ops.take_device_errors()


def test_cap_on_tiny_and_huge_scores():
    """The cap neither loses small scores nor overflows on scores thousands of times as large as it is."""
    torch = _torch()
    from llm_inference_lab_b200.kernels import ops
    D, L, page = 64, 96, 16
    rng = np.random.default_rng(2)
    for n in (1, 3, 90):
        ctx, table = make_ctx([n], [L - n], [0], page_size=page, num_pages=8)
        for size in (1e-3, 1.0, 3e4):
            for dtype in _dtypes():
                k, v, q = (_t(rng.standard_normal(s), dtype) for s in ((L, 1, D), (L, 1, D), (n, D)))
                ck = torch.zeros((8, 1, page, D), dtype=dtype, device="cuda")
                cv = torch.zeros_like(ck)
                _fill_pages(ck, cv, table, 0, k, v, page)
                got = _np(ops.attention(q, ck, cv, ctx, ctx.groups[0], 1, 1, D, 0, size, softcap=4.0))
                want = _capped_attention(_np(q).reshape(n, 1, D), _np(k), _np(v), range(L - n, L), size, 0, 4.0)[:, 0]
                assert np.isfinite(got).all() and np.abs(got - want).max() < (2e-5 if dtype == torch.float32 else 0.02)
    ops.take_device_errors()


@pytest.mark.parametrize("H,V,head,group", [(4, 24, 32, 0), (6, 16, 48, 3), (3, 130, 144, 1), (5, 1, 16, 5)])
def test_difference_of_two_maps(H, V, head, group):
    torch = _torch()
    from llm_inference_lab_b200.kernels import ops
    rng = np.random.default_rng(H)
    a = rng.standard_normal((9, H, 2, head))
    order = a.reshape(9, -1) if not group else a.reshape(9, H // group, group, 2, head).transpose(0, 1, 3, 2, 4).reshape(9, -1)
    for dtype in _dtypes():
        got = _np(ops.map_difference(_t(order, dtype), H, V, head, 0.8, 1e-3, 0.55, group=group)).reshape(9, H, V)
        x = _np(_t(a, dtype))[..., :V]
        want = pn.two_map_difference(x[:, :, 0], x[:, :, 1], 0.8, 1e-3, 0.45)
        assert np.abs(got - want).max() < (1e-5 if dtype == torch.float32 else 0.02)
        # two maps that differ by less than their rounding to bfloat16, a weight near one: 32-bit maps keep the difference
        close = np.repeat(a[:, :, :1], 2, axis=2) * np.array([1.0, 1.001])[:, None]
        flat = close.reshape(9, -1) if not group else close.reshape(9, H // group, group, 2, head).transpose(0, 1, 3, 2, 4).reshape(9, -1)
        out = ops.map_difference(_t(flat), H, V, head, 1.0, 1e-12, 0.55, group=group, dtype=dtype)
        x = _np(_t(close))[..., :V]
        want = pn.two_map_difference(x[:, :, 0], x[:, :, 1], 1.0, 1e-12, 0.45)
        assert out.dtype == dtype and np.abs(_np(out).reshape(9, H, V) - want).max() < (1e-2 if V > 1 else 2.0)


@pytest.mark.parametrize("mixer", [attention(4, 2, 16, 24, window=9, softcap=3.0, diff=0.4, scale=0.7),
                                   attention(6, 2, 72, 40, window=20, softcap=8.0, diff=0.2, scale=0.3),
                                   attention(3, 1, 20, 48, diff=0.6, scale=0.5), attention(2, 2, 10, 6, window=1, softcap=2.0)])
def test_attention_mixer_under_every_cut(mixer):
    """The whole mixer, its maps side by side or apart, in a prompt, in portions and token by token on shuffled pages."""
    torch = _torch()
    from llm_inference_lab_b200.kernels import ops
    from llm_inference_lab_b200.parts.base import CacheView
    m = mixer["mixer"]
    rng = np.random.default_rng(m["dim"])
    width, T, eps, page = 40, 37, 1e-5, 8
    raw = _weights(mixer, width, rng)
    for dtype in _dtypes():
        part = _mixer(mixer, raw, dtype, eps)
        assert part.packed == (m["dim"] < 72)
        w = {n: _np(_t(t, dtype)) for n, t in raw.items()}
        h = _t(rng.standard_normal((T, width)), dtype)
        want = pn.attention(_np(h), w, "m.", m, eps)
        # the first rows see few keys: their two maps are alike and the difference is small next to its rounding
        tol = (1e-4 if dtype == torch.float32 else 0.1) * max(1.0, np.abs(want).max())
        need = part.cache_need(part.spec)
        for sizes in ((T,), (2, 9, 1, 16, 3, 6), (1,) * T):
            k = torch.zeros((8, need.n_kv_heads, page, need.head_dim), dtype=dtype, device="cuda")
            view = CacheView(need=None, group=0, k=k, v=torch.zeros_like(k))
            at, outs = 0, []
            for n in sizes:
                ctx, _ = make_ctx([n], [at], [0], page_size=page, num_pages=8, shuffle=[3, 1, 7, 0, 5, 2, 6, 4], dtype=dtype)
                outs.append(_summed(part.forward(h[at: at + n], ctx, view)))
                at += n
            assert np.abs(np.concatenate(outs) - want).max() < tol, (dtype, sizes[:3])
    ops.take_device_errors()


# ---------------------------------------------------------------------------------------------
# experts, the stream, the token's side vector
# ---------------------------------------------------------------------------------------------
@pytest.mark.parametrize("E,top,groups,keep", [(12, 3, 4, 2), (6, 6, 1, 1), (10, 2, 5, 1), (40, 5, 8, 3), (7, 3, 1, 1), (9, 3, 3, 1),
                                               (70, 4, 35, 33)])
def test_corrected_choice_in_groups(E, top, groups, keep):
    """The choice by score plus correction among the experts of the best groups, most choice scores negative; the
    weights are the scores alone, times the scale."""
    from llm_inference_lab_b200.kernels import ops
    rng = np.random.default_rng(E + top)
    T = 33
    z = 2.0 * rng.standard_normal((T, E))
    corr = -0.5 + 0.4 * rng.standard_normal(E)
    s = np.exp(_np(_t(z)))
    s /= s.sum(1, keepdims=True)
    for score, values in (("softmax", s), ("sigmoid", pn.sigmoid(z))):
        chosen, weight, gate = ops.moe_route(_t(z), E, top, renorm=False, score=score, correction=_t(corr), groups=groups,
                                             keep=keep, scale=1.7)
        assert gate is None
        for t in range(T):
            want, margin = pn.choose(values[t], corr, top, groups, keep)
            if margin > 1e-6:
                assert list(chosen[t].cpu().numpy()) == want, t
                assert np.abs(_np(weight)[t] - 1.7 * values[t, want]).max() < 1e-6
    chosen, weight, _ = ops.moe_route(_t(z), E, top, groups=groups, keep=keep, scale=3.0)      # no correction, renormalised
    for t in range(T):
        want, margin = pn.choose(s[t], np.zeros(E), top, groups, keep)
        if margin > 1e-6:
            assert list(chosen[t].cpu().numpy()) == want and abs(_np(weight)[t].sum() - 3.0) < 1e-5
    with pytest.raises(ops.KernelError):
        ops.moe_route(_t(z), E, E, groups=groups, keep=keep) if keep < groups else ops.moe_route(_t(z), E, top, groups=E + 1)
    ops.take_device_errors()


def test_choice_edges():
    """Equal choice scores go to the smaller index, of groups and of experts; a correction alone can decide; a row of
    padding without numbers names existing experts of as many groups as are kept."""
    torch = _torch()
    from llm_inference_lab_b200.kernels import ops
    z = np.zeros((4, 6))
    z[1] = np.nan
    z[2, 4] = 50.0
    z[3] = [np.inf, np.nan, -np.inf, 0.0, 1.0, 2.0]
    chosen, weight, _ = ops.moe_route(_t(z), 6, 2, renorm=False, correction=torch.zeros(6, device="cuda"), groups=3, keep=2)
    ch = chosen.cpu().numpy()
    assert list(ch[0]) == [0, 1] and list(ch[2])[0] == 4
    for row in ch:
        assert len(set(row)) == 2 and all(0 <= e < 6 for e in row)
    assert bool(torch.isfinite(weight).all()) and abs(float(weight[0, 0]) - 1 / 6) < 1e-6
    corr = torch.tensor([0.0, 0.0, 0.0, 9.0, 0.0, 0.0], device="cuda")
    chosen, weight, _ = ops.moe_route(_t(z[:1]), 6, 2, renorm=False, correction=corr, groups=3, keep=1)
    assert chosen.cpu().numpy().tolist() == [[3, 2]] and abs(float(weight[0, 0]) - 1 / 6) < 1e-6
    ops.take_device_errors()


@pytest.mark.parametrize("T,width,kernel", [(3, 24, "auto"), (9, 50, "auto"), (60, 72, "auto"), (40, 64, "tc"), (70, 41, "tiles")])
def test_routed_layer_with_identities(T, width, kernel):
    """The whole layer, its sum alone and its sum inside the norm of the stream: identity experts among the chosen (a
    token of identities only among the rows), a shared expert with a limit of its own, in all three grouped products.
    In the stream the identities give the 32-bit rows, not their rounding."""
    torch = _torch()
    from llm_inference_lab_b200.config.nudusun import _feed_forward
    from llm_inference_lab_b200.kernels import ops
    from llm_inference_lab_b200.parts.base import lookup
    rng = np.random.default_rng(T)
    for dtype in _dtypes():
        if kernel == "tc" and dtype == torch.float32:
            continue
        for mlp in (moe(4, 3, 16, identity=4, groups=(4, 3), limit=0.8, scale=2.2, shared=(24, 1.1)), moe(2, 2, 8, identity=1, scale=0.7)):
            outs = mlp["router"]["experts"] + mlp["router"]["identity"]
            shapes = {"router": (outs, width), "correction": (outs,)}
            for e in range(mlp["router"]["experts"]):
                F = mlp["expert"]["ff"]
                shapes.update({f"e{e}.gate": (F, width), f"e{e}.up": (F, width), f"e{e}.down": (width, F)})
            if mlp.get("shared"):
                S = mlp["shared"]["ff"]
                shapes.update({"shared.gate": (S, width), "shared.up": (S, width), "shared.down": (width, S)})
            raw = {n: rng.standard_normal(s) * (0.2 if n == "correction" else 2.0 / np.sqrt(s[-1])) for n, s in shapes.items()}
            if outs == 8:      # a token that is sent to identities alone
                raw["correction"][4:7] += 0.3
            spec = _feed_forward(mlp, width, "f.")
            ffn = lookup("feed_forward", spec.kind)(spec, {"f." + n: _t(a, dtype) for n, a in raw.items()}, dtype, torch.device("cuda:0"))
            w = {n: _np(_t(a, dtype)) for n, a in raw.items()}
            x32 = _t(rng.standard_normal((T, width)))
            h = x32.to(dtype)
            margins = []
            want = pn.routed_experts(_np(h), w, "", mlp, margins)
            sure = margins[0] > (1e-5 if dtype == torch.float32 else 1e-4)
            old, ops.GROUPED_KERNEL = ops.GROUPED_KERNEL, kernel
            try:
                got = _np(ffn.forward(h, None))
                stream = x32.clone()
                nw = _t(1 + 0.2 * rng.standard_normal(width), dtype)
                copy = ffn.forward_post_norm(stream, h, None, nw, 1.4, 1e-5, dtype != torch.float32)
            finally:
                ops.GROUPED_KERNEL = old
            tol = (1e-4 if dtype == torch.float32 else 0.03) * max(1.0, np.abs(want).max())
            assert sure.sum() > 0.8 * T and np.abs(got - want)[sure].max() < tol
            # with the stream's own rows where the identities are: the difference to the rounded rows is their share
            share = np.zeros((T, 1))
            for t in range(T):
                z = _np(h)[t] @ w["router"].T
                s = np.exp(z - z.max()) / np.exp(z - z.max()).sum()
                g = mlp["router"].get("groups") or {"count": 1, "keep": 1}
                for e in pn.choose(s, w["correction"], mlp["router"]["top"], g["count"], g["keep"])[0]:
                    share[t] += mlp["router"]["scale"] * s[e] * (e >= mlp["router"]["experts"])
            assert share.max() > 0.05
            y = pn.rms_norm(1.4 * _np(x32) + want + share * (_np(x32) - _np(h)), _np(nw), 1e-5)
            assert np.abs(_np(stream) - y)[sure].max() < (5e-5 if dtype == torch.float32 else 0.03)
            assert copy is None or torch.equal(copy, stream.to(dtype))
    ops.take_device_errors()


def test_sum_under_the_norm_and_the_token_gate():
    """x <- norm(alpha x + product) with the 32-bit x whatever the storage type, for whole and for partial products and
    rows of any width; the gate by a part of the token's row of a side table."""
    torch = _torch()
    from llm_inference_lab_b200.kernels import ops
    rng = np.random.default_rng(4)
    for tokens, W in ((9, 50), (3, 72), (100, 1040), (70, 33)):
        for dtype in _dtypes():
            x, a = _t(100.0 * rng.standard_normal((tokens, W))), _t(0.01 * rng.standard_normal((3, tokens, W)))
            w = _t(1 + 0.2 * rng.standard_normal(W), dtype)
            for part in (a, a[1]):
                stream = x.clone()
                copy = ops.stream_post_norm(stream, part, w, 2.5, 1e-6, copy=True)
                want = pn.rms_norm(2.5 * _np(x) + _summed(part), _np(w), 1e-6)
                assert np.abs(_np(stream) - want).max() < 2e-5 and torch.equal(copy, stream.to(dtype))
            assert ops.stream_post_norm(stream, a, w, 0.5, 1e-6) is None
            n, at = W // 3, 2
            table = _t(rng.standard_normal((11, W)), dtype)
            ids = torch.tensor(rng.integers(0, 11, size=tokens), dtype=torch.int32, device="cuda")
            p = _t(rng.standard_normal((3, tokens, n)))
            for part in (p, p[0].contiguous()):
                want = pn.gelu_tanh(_summed(part)) * _np(table)[ids.cpu().numpy(), at: at + n]
                assert np.abs(_np(ops.token_gate(part, table, ids, at)) - want).max() < (1e-5 if dtype == torch.float32 else 0.05)


def test_scaled_embedding_with_positions():
    """The table's row is scaled, the position's is not, and the stream is 32-bit."""
    torch = _torch()
    from llm_inference_lab_b200.parts.base import lookup
    from llm_inference_lab_b200.parts.spec import PartSpec
    rng = np.random.default_rng(6)
    for dtype in _dtypes():
        w = {"e": _t(rng.standard_normal((7, 10)), dtype), "p": _t(rng.standard_normal((30, 10)), dtype)}
        part = lookup("embedding", "token_position_embedding")(
            PartSpec("token_position_embedding", {"vocab": 7, "hidden": 10, "table": "e", "positions": "p", "max_positions": 30,
                                                  "scale": 6.5}), dict(w), dtype, torch.device("cuda:0"))
        ids, pos = np.array([3, 0, 6]), np.array([29, 0, 11])
        got = part.forward(*(torch.tensor(a, dtype=torch.int32, device="cuda") for a in (ids, pos)))
        assert got.dtype == torch.float32
        assert np.abs(_np(got) - (6.5 * _np(w["e"])[ids] + _np(w["p"])[pos])).max() < 1e-5


# ---------------------------------------------------------------------------------------------
# whole models under every cut
# ---------------------------------------------------------------------------------------------
def _engine(folder, dtype, opt, steps, **kw):
    from llm_inference_lab_b200.engine import Engine
    page = opt["page_size"]
    unit = max(64, page)
    pool = tokens_needed(steps, unit)
    return Engine(folder, dtype, max_tokens=pool, page_size=page, max_requests=4, max_batch_tokens=max(pool, 64),
                  max_seq_len=pool, **kw)


def _check(got, want, dtype, label, close=()):
    """32-bit: every position within F32_MAX.  bfloat16: without the positions of `close` (a routed layer may pick
    another expert where two choice scores are a rounding apart) the rms error within BF16_RMS and all but one position
    in a hundred within BF16_MAX (another expert's result moves later positions a little)."""
    if dtype == "bfloat16":
        got = {key: row for key, row in got.items() if key not in close}
    worst, rms, where = error_stats(got, want)
    if dtype == "float32":
        assert worst < F32_MAX, (label, worst, where)
        return
    peak = max(float(np.abs(v).max()) for v in want.values())
    over = [key for key, row in got.items() if np.abs(row - want[key[0]][key[1]]).max() > BF16_MAX * peak]
    assert rms < BF16_RMS and len(over) <= max(1, len(got) // 100), (label, worst, rms, over[:5])


ONE_LAYER = {
    "attention": config([attention(4, 2, 16, 40, window=7, softcap=3.0, diff=0.3, scale=0.6)], vocab=53, width=32),
    "attention+moe": config([attention(3, 1, 24, 8, window=16, softcap=6.0, diff=0.5, scale=0.5,
                                       mlp=moe(5, 2, 16, identity=1, groups=(3, 2), shared=(24, 1.0)))], vocab=53, width=40),
    "delta": config([delta(4, 2, 8, 16, conv=4)], vocab=53, width=32, side=4),
    "delta+moe": config([delta(6, 3, 24, 8, conv=2, mlp=moe(3, 2, 8, identity=3))], vocab=53, width=48, side=0),
    "heads beyond the tensor cores": config([attention(2, 1, 100, 140, window=12, softcap=9.0, diff=0.2, scale=0.2),
                                             delta(2, 1, 140, 24, conv=3)], vocab=53, width=24),
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(ONE_LAYER))
def test_one_layer_models(tmp_path, name, dtype):
    rng = np.random.default_rng(3)
    cfg = ONE_LAYER[name]
    folder = make_model_folder(str(tmp_path / "m"), cfg, 21, dtype, std=0.08, scales=SPREAD)
    seqs = sequences(rng, cfg["vocab"], [45, 1, 30])
    want, close = plain_logits(folder, seqs, CLOSE)
    for label, steps in (("whole", trace_whole(seqs)), ("tail", trace_tail_decode(seqs, tail=25)),
                         ("portions", trace_portions(seqs))):
        eng = _engine(folder, dtype, dict(page_size=8), steps)
        _check(run_trace_inprocess(eng, steps), want, dtype, (name, label), close)
        assert eng.cache.live_requests == 0


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(SMALL))
def test_models_under_every_cut(tmp_path, name, dtype):
    """Whole prompts; the tail decoded token by token, past every window; portions of 2 to 11 tokens; up to four live
    requests with portions beside single tokens, in a pool so small that pages and state slots are used again."""
    cfg, opt = SMALL[name]
    rng = np.random.default_rng(opt["seed"])
    folder = make_model_folder(str(tmp_path / "m"), cfg, opt["seed"], dtype, std=0.08, scales=SPREAD)
    seqs = sequences(rng, cfg["vocab"], [150, 3, 61, 90, 1, 77, 40])
    want, close = plain_logits(folder, seqs, CLOSE)
    assert len(close) < 0.5 * sum(len(v) for v in seqs.values())
    traces = {"whole": trace_whole(seqs), "tail": trace_tail_decode(seqs, tail=70), "portions": trace_portions(seqs),
              "mixed": trace_mixed(seqs, np.random.default_rng(1), max_live=4)}
    for label, steps in traces.items():
        eng = _engine(folder, dtype, opt, steps)
        got = run_trace_inprocess(eng, steps)
        assert len(got) == sum(len(v) for v in seqs.values())
        _check(got, want, dtype, (name, label), close)
        assert eng.cache.live_requests == 0 and all(f == eng.num_pages for f in eng.free_pages())


def test_long_portions_and_long_decoding(tmp_path):
    """Portions of more than a hundred tokens beside single tokens, and a tail of 150 decoded tokens, with windows of
    up to 260 tokens and a delta rule over the whole sequence."""
    cfg, opt = SMALL["D"]
    folder = make_model_folder(str(tmp_path / "m"), cfg, opt["seed"], "bfloat16", std=0.08, scales=SPREAD)
    seqs = sequences(np.random.default_rng(9), cfg["vocab"], [400, 130, 260])
    want, close = plain_logits(folder, seqs, CLOSE)
    for label, steps in (("whole", trace_whole(seqs)), ("tail", trace_tail_decode(seqs, tail=150)),
                         ("mixed", trace_mixed(seqs, np.random.default_rng(2), max_live=3, max_portion=140))):
        eng = _engine(folder, "bfloat16", opt, steps)
        _check(run_trace_inprocess(eng, steps), want, "bfloat16", label, close)


@pytest.mark.parametrize("trial", range(int(os.environ.get("LAB_RANDOM_NUDUSUN", "6"))))
def test_random_configurations_and_traces(tmp_path, trial):
    """Random configurations (`random_config`) under mixed batches with pages and slots used again, in 32-bit.
    `LAB_RANDOM_NUDUSUN=N` runs N."""
    rng = np.random.default_rng(6000 + trial)
    cfg, page = random_config(rng)
    seqs = sequences(rng, cfg["vocab"], [int(n) for n in rng.integers(1, 150, size=6)])
    steps = trace_mixed(seqs, np.random.default_rng(trial), max_live=4, max_portion=int(rng.choice([9, 40, 140])))
    folder = make_model_folder(str(tmp_path / "m"), cfg, trial, "float32", std=0.08, scales=SPREAD)
    want, close = plain_logits(folder, seqs, 2e-6)
    eng = _engine(folder, "float32", dict(page_size=page), steps)
    got = {key: row for key, row in run_trace_inprocess(eng, steps).items() if key not in close}
    worst, rms, where = error_stats(got, want)
    assert worst < F32_MAX, (trial, cfg, worst, where)
    assert eng.cache.live_requests == 0


def test_cuts_agree_in_32_bit(tmp_path):
    """In 32-bit the logits of a position do not depend on how a prompt was cut or on what else is in the batch,
    beyond the rounding of sums taken in another order (the experts' products of few and of many pairs)."""
    cfg, opt = SMALL["A"]
    folder = make_model_folder(str(tmp_path / "m"), cfg, 5, "float32", std=0.08, scales=SPREAD)
    seqs = sequences(np.random.default_rng(2), cfg["vocab"], [70, 33, 9])
    results = []
    for steps in (trace_whole(seqs), trace_portions(seqs), trace_mixed(seqs, np.random.default_rng(3), max_live=3)):
        results.append(run_trace_inprocess(_engine(folder, "float32", opt, steps), steps))
    peak = max(float(np.abs(row).max()) for row in results[0].values())
    for other in results[1:]:
        for key, row in results[0].items():
            assert np.abs(row - other[key]).max() <= 5e-5 * max(1.0, peak), key


def test_trace_program_and_a_failed_step(tmp_path):
    """bin/trace_run on a Nudusun folder; and a step that fails leaves pages, states and kept inputs as they were."""
    from llm_inference_lab_b200.engine import Entry
    cfg, opt = SMALL["A"]
    folder = make_model_folder(str(tmp_path / "m"), cfg, 8, "float32", std=0.08, scales=SPREAD)
    seqs = sequences(np.random.default_rng(4), cfg["vocab"], [50, 20, 35, 8, 41])
    want = plain_logits(folder, seqs)
    steps = trace_mixed(seqs, np.random.default_rng(6), max_live=4)
    out = str(tmp_path / "out")
    os.makedirs(out)
    got = run_trace_program(folder, "float32", steps, out, tokens_needed(steps, 64))
    _check(got, want, "float32", "program")
    ids = seqs["s0"]
    eng = _engine(folder, "float32", opt, trace_whole(seqs))
    assert len(eng.views) == 4 and len(eng.state_tensors) == 4      # a state and the kept inputs of each delta layer
    eng.step([Entry(0, ids[:20], [])])
    free = eng.free_pages()
    head = eng.model.head
    try:
        old = head.forward
        head.forward = lambda *a, **k: (_ for _ in ()).throw(RuntimeError("injected"))   # fails after the layers ran
        with pytest.raises(RuntimeError):
            eng.step([Entry(0, ids[20:30], [9])])
    finally:
        head.forward = old
    assert eng.free_pages() == free
    logits = eng.step([Entry(0, ids[20:], [len(ids) - 21])]).cpu().numpy()
    assert np.abs(logits[0] - want["s0"][-1]).max() < F32_MAX * max(1.0, np.abs(want["s0"]).max())


# ---------------------------------------------------------------------------------------------
# generation through the scheduler
# ---------------------------------------------------------------------------------------------
def _greedy(cfg, w, prompt, n_new):
    tokens = list(prompt)
    for _ in range(n_new):
        tokens.append(int(np.argmax(pn.forward(cfg, w, tokens)[-1])))
    return tokens[len(prompt):]


@pytest.mark.parametrize("name", ["A", "C"])
def test_greedy_generation_through_the_scheduler(tmp_path, name):
    """More requests than slots, prompts cut under a small token budget: greedy tokens in 32-bit equal
    the plain model's."""
    from llm_inference_lab_b200.engine.llm import LLM
    from llm_inference_lab_b200.kernels import ops
    from llm_inference_lab_b200.sampling import SamplingConfig
    cfg, opt = SMALL[name]
    folder = make_model_folder(str(tmp_path / "m"), cfg, 17, "float32", std=0.08, scales=SPREAD)
    pcfg, w = pn.read_folder(folder)
    rng = np.random.default_rng(7)
    prompts = [[int(t) for t in rng.integers(0, cfg["vocab"], size=n)] for n in (5, 40, 1, 23, 12, 31)]
    llm = LLM(folder, "float32", page_size=opt["page_size"], kv_tokens=512, max_requests=3, max_batch_tokens=24,
              max_seq_len=128, device="cuda:0")
    results = llm.generate(prompts, SamplingConfig(max_new_tokens=12, ignore_eos=True))
    ops.take_device_errors()
    for prompt, res in zip(prompts, results):
        assert res.finish_reason == "length"
        assert res.tokens == _greedy(pcfg, w, prompt, 12)
    assert llm.engine.cache.live_requests == 0


@pytest.mark.parametrize("name,dtype", [("A", "float32"), ("B", "float32"), ("A", "bfloat16")])
def test_decode_steps_from_cuda_graphs(tmp_path, name, dtype):
    """Decode steps replayed from CUDA graphs, states, kept inputs and the tokens' side vectors inside them: batches
    padded with requests of length zero, a batch that shrinks as requests finish.  32-bit: the plain model's tokens;
    bfloat16: the tokens of the same engine stepping eagerly."""
    from llm_inference_lab_b200.engine.llm import LLM
    from llm_inference_lab_b200.kernels import ops
    from llm_inference_lab_b200.sampling import SamplingConfig
    cfg, opt = SMALL[name]
    folder = make_model_folder(str(tmp_path / "m"), cfg, 23, dtype, std=0.08, scales=SPREAD)
    rng = np.random.default_rng(5)
    prompts = [[int(t) for t in rng.integers(0, cfg["vocab"], size=n)] for n in (7, 30, 2, 19, 11)]
    sampling = [SamplingConfig(max_new_tokens=n, ignore_eos=True) for n in (20, 5, 14, 9, 17)]

    def run(graph):
        llm = LLM(folder, dtype, page_size=opt["page_size"], kv_tokens=1024, max_requests=8, max_batch_tokens=64,
                  max_seq_len=128, device="cuda:0", cuda_graph=graph)
        assert llm.cuda_graph == graph
        out = [r.tokens for r in llm.generate(prompts, sampling)]
        ops.take_device_errors()
        assert llm.engine.cache.live_requests == 0
        if graph:
            assert llm.graphs.replays >= 10 and llm.graphs.captures >= 3
        return out

    got = run(True)
    if dtype == "float32":
        pcfg, w = pn.read_folder(folder)
        assert got == [_greedy(pcfg, w, p, s.max_new_tokens) for p, s in zip(prompts, sampling)]
    else:
        assert got == run(False)


def test_command_line_generates(tmp_path):
    import json
    import subprocess
    import sys
    cfg, opt = SMALL["C"]
    folder = make_model_folder(str(tmp_path / "m"), cfg, 19, "float32", std=0.08, scales=SPREAD)
    pcfg, w = pn.read_folder(folder)
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    proc = subprocess.run([sys.executable, "-m", "llm_inference_lab_b200.cli", "--model-dir", folder, "--dtype", "f32",
                           "--prompt-ids", "3,14,15,9,2,6", "--max-new-tokens", "6", "--kv-tokens", "256"],
                          cwd=root, capture_output=True, text=True, timeout=600)
    assert proc.returncode == 0, proc.stderr[-2000:]
    line = json.loads(proc.stdout.strip().splitlines()[-1])
    assert line["generated_ids"] == _greedy(pcfg, w, [3, 14, 15, 9, 2, 6], 6)
