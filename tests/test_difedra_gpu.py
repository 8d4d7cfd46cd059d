"""Difedra on the GPU against the plain implementation (tests/plain_difedra.py): each mechanism
alone, then whole models under every way of cutting a trace, then generation through the scheduler."""
import os

import numpy as np
import pytest

import plain_difedra as pd
from difedra_helpers import (SMALL, SPREAD, attention, close_calls, config, dense, moe, plain_logits, random_config, rot, sequences)
from helpers import (error_stats, make_model_folder, run_trace_inprocess, run_trace_program, tokens_needed,
                     trace_mixed, trace_portions, trace_tail_decode, trace_whole)
from ritizen_helpers import make_ctx

pytestmark = pytest.mark.gpu

F32_MAX = 2e-4      # largest error over the largest logit, 32-bit engine against the 64-bit plain model
BF16_MAX, BF16_RMS = 0.10, 0.04


def _torch():
    import torch
    return torch


def _t(a, dtype=None):
    torch = _torch()
    t = torch.from_numpy(np.ascontiguousarray(a, dtype=np.float32)).cuda()
    return t if dtype is None else t.to(dtype)


def _np(t):
    return t.double().cpu().numpy()


def _dtypes():
    torch = _torch()
    return (torch.float32, torch.bfloat16)


# ---------------------------------------------------------------------------------------------
# mechanisms alone
# ---------------------------------------------------------------------------------------------
def _rotate(v, positions, freq, pairs):
    """The plain rotation; neighbours by reordering the entries around it."""
    if not pairs:
        return pd.rotate_halves(v, positions, freq)
    n = 2 * len(freq)
    order = np.concatenate([np.arange(0, n, 2), np.arange(1, n, 2)])
    out = np.array(v, copy=True)
    out[..., order] = pd.rotate_halves(v[..., order], positions, freq)
    return out


@pytest.mark.parametrize("H,G,D,V,dims,pairs,norm", [
    (4, 2, 16, 24, 8, False, True), (3, 3, 40, 8, 40, False, True), (1, 1, 12, 20, 2, False, True),
    (5, 1, 24, 24, 24, True, True), (2, 2, 32, 16, 16, False, False), (6, 3, 10, 130, 0, False, True),
    (8, 1, 128, 64, 96, False, True), (3, 1, 16, 8, 2, True, True), (14, 2, 96, 64, 96, True, True), (2, 2, 8, 12, 4, False, True)])
def test_whole_projection_norms_rotation_and_mixed_values(H, G, D, V, dims, pairs, norm):
    """q and k normed over all heads at once and then rotated (halves, or neighbours), the values left for later
    layers and mixed with those an earlier layer left, everything stored in the rows' slots with zeros beyond a
    head's own size; from whole and from partial products, with and without norms; a row of padding stores nothing."""
    torch = _torch()
    from llm_inference_lab_b200.kernels import ops
    rng = np.random.default_rng(D + V)
    page, pages, eps, lam = 4, 64, 1e-4, 0.3
    q_lens, pos0 = [5, 1, 7], [3, 130, 0]
    ctx, _ = make_ctx(q_lens, pos0, [0, 1, 2], page_size=page, num_pages=pages, shuffle=rng.permutation(pages))
    T, head = sum(q_lens), ops.padded_head(D, V)
    freq = pd.frequencies(300.0, dims, {"factor": 4.0, "low": 1.0, "high": 3.0, "original": 60})
    inv = _t(freq)
    pos = ctx.row_pos.cpu().numpy()
    width = H * D + G * (D + V)
    for dtype in _dtypes():
        tol = 4e-5 if dtype == torch.float32 else 0.04      # an angle of 130 radians, rounded, is 8e-6 off
        wq, wk = (_t(1 + 0.3 * rng.standard_normal(n * D), dtype) if norm else None for n in (H, G))
        for splits in (1, 3):
            proj = _t(rng.standard_normal((splits, T, width)))
            first = _t(rng.standard_normal((T, G * V)))
            keep = torch.full((T, G * V), float("nan"), device="cuda")
            ck = torch.full((pages, G, page, head), float("nan"), dtype=dtype, device="cuda")
            cv = torch.full_like(ck, float("nan"))
            slots = ctx.groups[0].row_slot.clone()
            slots[2] = -1
            q = ops.qk_norm_store(proj if splits > 1 else proj[0], None, wq, wk, slots, ck, cv, H, G, D, V, head, eps,
                                  dtype=dtype, positions=ctx.row_pos, inv_freq=inv, rot_dims=dims, rot_pairs=pairs,
                                  v_keep=keep, v_first=first, v_mix=lam)
            full = _np(proj).sum(0)
            fq, fk, fv = full[:, : H * D], full[:, H * D: (H + G) * D], full[:, (H + G) * D:]
            if norm:
                fq, fk = pd.rms_norm(fq, _np(wq), eps), pd.rms_norm(fk, _np(wk), eps)
            want_q = _rotate(fq.reshape(T, H, D), pos, freq, pairs)
            want_k = _rotate(fk.reshape(T, G, D), pos, freq, pairs)
            want_v = pd.mixed_values(fv, _np(first), lam).reshape(T, G, V)
            assert q.dtype == dtype and np.abs(_np(keep) - fv).max() < 1e-5      # the values before any mixing
            got_q = _np(q).reshape(T, H, head)
            assert np.abs(got_q[:, :, :D] - want_q).max() < tol and not got_q[:, :, D:].any()
            for t in range(T):
                s = int(slots[t])
                if s < 0:
                    continue
                rk, rv = _np(ck[s // page, :, s % page]), _np(cv[s // page, :, s % page])
                assert np.abs(rk[:, :D] - want_k[t]).max() < tol and np.abs(rv[:, :V] - want_v[t]).max() < tol
                assert not rk[:, D:].any() and not rv[:, V:].any()
            s = int(ctx.groups[0].row_slot[2])
            assert torch.isnan(ck[s // page, :, s % page]).all() and torch.isnan(cv[s // page, :, s % page]).all()
    ops.take_device_errors()


def _mixer(m, weights, dtype, v_mix=None, eps=1e-5, **more):
    torch = _torch()
    from llm_inference_lab_b200.parts.spec import PartSpec
    from llm_inference_lab_b200.parts.window_attention import PairRopeAttention
    turn = m.get("rot") or {"base": 1.0, "dims": 0}
    sc = turn.get("scaling")
    spec = PartSpec("pair_rope_attention", {
        "hidden": weights["m.o"].shape[0], **{k: m[k] for k in ("heads", "kv_heads", "dim", "vdim", "scale")},
        "window": m["mask"]["size"] if m.get("mask") else 0, "sink_learned": True, "proj_norm": True, "eps": eps,
        "rot_layout": "halves", "rot_base": turn["base"], "rot_dims": turn["dims"],
        "rot_bands": tuple(sc[k] for k in ("factor", "low", "high", "original")) if sc else None, "v_mix": v_mix, **more},
        prefix="m.")
    return PairRopeAttention(spec, {k: _t(v, dtype) for k, v in weights.items()}, dtype, torch.device("cuda:0"))


def _mixer_weights(m, width, rng):
    H, G, D, V = (m[k] for k in ("heads", "kv_heads", "dim", "vdim"))
    w = {"m." + n: rng.standard_normal(s) / np.sqrt(s[1]) for n, s in
         {"q": (H * D, width), "k": (G * D, width), "v": (G * V, width), "o": (width, H * V)}.items()}
    w["m.q.norm"], w["m.k.norm"] = 1 + 0.3 * rng.standard_normal(H * D), 1 + 0.3 * rng.standard_normal(G * D)
    w["m.sink"], w["m.vmix"] = 2.0 * rng.standard_normal(H), np.array(0.6)
    return w


@pytest.mark.parametrize("first,second", [
    (attention(4, 2, 16, 24, window=9, turn=rot(500.0, 8), scale=0.4)["mixer"],
     attention(6, 3, 24, 16, window=20, turn=rot(90.0, 24, (2.5, 0.5, 8.0, 200)), scale=0.3)["mixer"]),
    (attention(2, 1, 136, 8, window=5, turn=rot(40.0, 60), scale=0.1)["mixer"],
     attention(3, 1, 6, 8, scale=0.5)["mixer"])])
def test_two_mixers_share_values_within_a_step(first, second):
    """Two attention mixers one after the other: the second mixes the first one's values of the same tokens into its
    own, in a prompt, in portions and token by token; a mixer that wants values nobody left raises."""
    torch = _torch()
    from llm_inference_lab_b200.kernels import ops
    from llm_inference_lab_b200.parts.base import CacheView
    rng = np.random.default_rng(first["dim"])
    width, T, page, eps = 40, 37, 8, 1e-5
    wa, wb = _mixer_weights(first, width, rng), _mixer_weights(second, width, rng)
    for dtype in _dtypes():
        a, b = _mixer(first, wa, dtype, "first"), _mixer(second, wb, dtype, "mix")
        ra, rb = ({k: _np(_t(v, dtype)) for k, v in w.items()} for w in (wa, wb))
        h = _t(rng.standard_normal((T, width)), dtype)
        want_a, kept = pd.attention(_np(h), ra, "m.", {**first, "v_mix": True}, eps, None)
        want_b, _ = pd.attention(_np(h), rb, "m.", {**second, "v_mix": True}, eps, kept)
        tol = (3e-5 if dtype == torch.float32 else 0.05) * max(1.0, np.abs(want_a).max(), np.abs(want_b).max())
        for sizes in ((T,), (2, 9, 1, 16, 3, 6), (1,) * T):
            views = []
            for m in (a, b):
                k = torch.zeros((8, m.n_kv, page, m.head), dtype=dtype, device="cuda")
                views.append(CacheView(need=None, group=0, k=k, v=torch.zeros_like(k)))
            at, outs = 0, ([], [])
            for n in sizes:
                ctx, _ = make_ctx([n], [at], [0], page_size=page, num_pages=8, shuffle=[3, 1, 7, 0, 5, 2, 6, 4], dtype=dtype)
                for mixer, view, out in zip((a, b), views, outs):
                    y = _np(mixer.forward(h[at: at + n], ctx, view))
                    out.append(y.sum(0) if y.ndim == 3 else y)
                at += n
            for got, want in zip(outs, (want_a, want_b)):
                assert np.abs(np.concatenate(got) - want).max() < tol, (dtype, sizes[:3])
        ctx, _ = make_ctx([2], [0], [0], page_size=page, num_pages=8, dtype=dtype)
        with pytest.raises(ValueError):
            b.forward(h[:2], ctx, views[1])
    with pytest.raises(ValueError):
        _mixer(first, wa, torch.float32, "first", head_norm="unit")
    ops.take_device_errors()


def test_rotation_of_halves_without_norms():
    """The layout alone, beside plain projections: an attention whose q and k are not normed."""
    torch = _torch()
    from llm_inference_lab_b200.parts.base import CacheView
    rng = np.random.default_rng(8)
    m = attention(3, 1, 16, 16, window=6, turn=rot(50.0, 12), scale=0.3)["mixer"]
    w = _mixer_weights(m, 24, rng)
    mixer = _mixer(m, w, torch.float32, proj_norm=False)
    T = 20
    h = rng.standard_normal((T, 24))
    q, k, v = ((h @ w["m." + n].T).reshape(T, -1, 16) for n in ("q", "k", "v"))
    freq = pd.frequencies(50.0, 12)
    q, k = pd.rotate_halves(q, range(T), freq), pd.rotate_halves(k, range(T), freq)
    s = np.stack([q[:, i] @ k[:, 0].T for i in range(3)]) * 0.3
    p = pd.sink_softmax(s, pd.in_window(T, 6)[None], w["m.sink"])
    want = np.stack([p[i] @ v[:, 0] for i in range(3)], axis=1).reshape(T, -1) @ w["m.o"].T
    ctx, _ = make_ctx([T], [0], [0], page_size=16, num_pages=2)
    kc = torch.zeros((2, 1, 16, 16), device="cuda")
    got = _np(mixer.forward(_t(h), ctx, CacheView(need=None, group=0, k=kc, v=torch.zeros_like(kc))))
    assert np.abs(got - want).max() < 2e-5 * max(1.0, np.abs(want).max())


def _fill_pages(ck, cv, table, r, k, v, page):
    """Keys and values k, v [L, G, D] of request r into its pages."""
    L = k.shape[0]
    for b in range(-(-L // page)):
        n = min(page, L - b * page)
        ck[table[r, b], :, :n] = k[b * page: b * page + n].transpose(0, 1)
        cv[table[r, b], :, :n] = v[b * page: b * page + n].transpose(0, 1)


def _plain_scores_attention(q, k, v, pos_q, scale, window, sink):
    """q [n, H, D] at positions pos_q over keys k, v [L, G, D] at positions 0 .. L - 1."""
    n, H, _ = q.shape
    L, G = k.shape[:2]
    i, j = np.asarray(pos_q)[:, None], np.arange(L)[None, :]
    seen = (j <= i) & (i - j < (window or L + 1))
    s = np.stack([q[:, h] @ k[:, h // (H // G)].T for h in range(H)]) * scale
    p = pd.sink_softmax(s, seen[None], sink)
    return np.stack([p[h] @ v[:, h // (H // G)] for h in range(H)], axis=1)


@pytest.mark.parametrize("D,H,G,page,window", [(16, 4, 2, 4, 9), (48, 16, 1, 16, 33), (64, 9, 1, 8, 141), (64, 4, 2, 16, 16),
                                               (128, 3, 1, 32, 250), (144, 2, 1, 16, 20)])
def test_window_with_a_learned_sink_in_every_attention_kernel(D, H, G, page, window):
    """Random keys under a window with a learned term per head: long and short portions beside single tokens, near
    the start and far from it, on shuffled pages, in both storage types (prefill on tcgen05 and mma.sync, decode with
    split keys, the plain kernel)."""
    torch = _torch()
    from llm_inference_lab_b200.kernels import ops
    rng = np.random.default_rng(D + window)
    q_lens, pos0 = [150, 1, 2, 1, 30, 1], [200, 700, 127, 3, 0, 0]
    pages = sum(-(-(n + p) // page) for n, p in zip(q_lens, pos0)) + 3
    ctx, table = make_ctx(q_lens, pos0, list(range(len(q_lens))), page_size=page, num_pages=pages,
                          shuffle=rng.permutation(pages))
    sink = 2.0 * rng.standard_normal(H)
    scale = 1.5 * D ** -0.5
    for dtype in _dtypes():
        ck = torch.zeros((pages, G, page, D), dtype=dtype, device="cuda")
        cv = torch.zeros_like(ck)
        keys, vals = [], []
        for r, (n, p0) in enumerate(zip(q_lens, pos0)):
            k, v = (_t(rng.standard_normal((p0 + n, G, D)), dtype) for _ in range(2))
            keys.append(_np(k)), vals.append(_np(v))
            _fill_pages(ck, cv, table, r, k, v, page)
        q = _t(rng.standard_normal((sum(q_lens), H * D)), dtype)
        got = _np(ops.attention(q, ck, cv, ctx, ctx.groups[0], H, G, D, window, scale, sink=_t(sink)))
        at = 0
        for r, (n, p0) in enumerate(zip(q_lens, pos0)):
            want = _plain_scores_attention(_np(q[at: at + n]).reshape(n, H, D), keys[r], vals[r], range(p0, p0 + n), scale,
                                           window, sink)
            err = np.abs(got[at: at + n].reshape(n, H, D) - want).max()
            assert err < (1e-5 if dtype == torch.float32 else 0.03), (r, err)
            at += n
    ops.take_device_errors()


@pytest.mark.parametrize("n", [1, 2, 6, 140])
@pytest.mark.parametrize("D,page,window", [(64, 16, 150), (128, 32, 260), (32, 8, 65), (64, 8, 8)])
def test_window_edges_show_with_a_learned_sink(n, D, page, window):
    """One key made to stand out: the last row's output is its value (less the sink's share) while the key is the
    window's last place, and no part of it one place further; at page and tile borders; as the first token; for
    single tokens, short portions and portions of more than one tile of rows.  A head whose sink is as large as
    that score halves the output."""
    torch = _torch()
    from llm_inference_lab_b200.kernels import ops
    H, G, L = 2, 1, 600
    sink = np.array([-3.0, 40.0])
    for dtype in _dtypes():
        for target in (L - 1, L - window, L - window - 1, L - window + 1, L - 17, L - page, L - 64, 128, 0):
            seen = 0 <= L - 1 - target < window
            rng = np.random.default_rng(target)
            pages = -(-L // page) + 3
            ctx, table = make_ctx([n], [L - n], [0], page_size=page, num_pages=pages, shuffle=rng.permutation(pages))
            k = 0.05 * rng.standard_normal((L, G, D))
            v = rng.standard_normal((L, G, D))
            k[target, 0, 3] = 40.0
            q = np.zeros((n, H, D))
            q[:, :, 3] = 1.0
            ck = torch.zeros((pages, G, page, D), dtype=dtype, device="cuda")
            cv = torch.zeros_like(ck)
            _fill_pages(ck, cv, table, 0, _t(k, dtype), _t(v, dtype), page)
            got = _np(ops.attention(_t(q.reshape(n, -1), dtype), ck, cv, ctx, ctx.groups[0], H, G, D, window, 1.0,
                                    sink=_t(sink)))[-1].reshape(H, D)
            v_t = _np(_t(v[target, 0], dtype))
            if seen:
                assert np.abs(got[0] - v_t).max() < 0.02 and np.abs(got[1] - 0.5 * v_t).max() < 0.02, target
            else:
                want = _plain_scores_attention(q[-1:], _np(_t(k, dtype)), _np(_t(v, dtype)), [L - 1], 1.0, window, sink)[0]
                assert np.abs(got - want).max() < 0.02 and np.abs(got[0] - v_t).max() > 0.1, target
                assert np.abs(got[1]).max() < 1e-6           # a sink far above every seen score takes all the weight
    ops.take_device_errors()


@pytest.mark.parametrize("tokens,n_out,k", [(3, 200, 64), (70, 96, 328), (300, 520, 128), (4100, 512, 264), (9, 50, 36)])
def test_gelu_gate_in_the_products_epilogue(tokens, n_out, k):
    """gelu(gate) * up, the tanh form, as the epilogue of the gated product: both orientations of the tensor-core
    kernel, the kernel on pairs of SMs, and the plain kernel; gates far on both sides of zero stay finite."""
    torch = _torch()
    from llm_inference_lab_b200.kernels import ops
    rng = np.random.default_rng(tokens)
    for dtype in _dtypes():
        x, w = _t(rng.standard_normal((tokens, k)), dtype), _t(2.0 * rng.standard_normal((2 * n_out, k)) / np.sqrt(k), dtype)
        w[0] *= 200.0                             # the first column's gates lie hundreds away from zero
        size = np.where(np.arange(n_out) == 0, 200.0, 1.0)
        got = ops.linear_gated(x, w, act="gelu_tanh")
        g, u = _np(x) @ _np(w)[:n_out].T, _np(x) @ _np(w)[n_out:].T
        ref = pd.gelu_tanh(g) * u
        assert got.dtype == dtype
        tol = 2e-5 if dtype == torch.float32 else 0.01
        assert (np.abs(_np(got) - ref) / (size + np.abs(ref))).max() < tol
        silu = pd.silu(g) * u
        assert (np.abs(_np(ops.linear_gated(x, w)) - silu) / (size + np.abs(silu))).max() < tol
    with pytest.raises(ops.KernelError):
        ops.linear_gated(x, w, act="relu")
    with pytest.raises(ops.KernelError):
        ops.linear_gated(x, w, limit=1.0, act="gelu_tanh")
    ops.take_device_errors()


@pytest.mark.parametrize("E,top,T,K,F,kernel", [(5, 2, 3, 24, 10, "auto"), (7, 7, 33, 40, 16, "auto"), (3, 1, 300, 72, 40, "auto"),
                                                (6, 2, 40, 72, 40, "tc"), (4, 2, 50, 41, 19, "tiles"), (1, 1, 9, 16, 8, "auto"),
                                                (40, 3, 7, 24, 8, "auto")])
def test_sigmoid_scores_on_the_experts_inputs(E, top, T, K, F, kernel):
    """The router's sigmoid scores as they are, multiplying the inputs of the experts, in all three grouped products
    (few rows, tiles, tensor cores); each product also gated by GELU."""
    torch = _torch()
    from llm_inference_lab_b200.kernels import ops
    rng = np.random.default_rng(E * T)
    for dtype in _dtypes():
        if kernel == "tc" and dtype == torch.float32:
            continue
        logits = _t(2.0 * rng.standard_normal((T, E)))
        chosen, weight, gate = ops.moe_route(logits, E, top, renorm=False, score="sigmoid")
        s = pd.sigmoid(_np(logits))
        ch = chosen.cpu().numpy()
        for t in range(T):
            order = sorted(range(E), key=lambda e: (-s[t, e], e))[:top]
            assert list(ch[t]) == order and np.abs(_np(weight)[t] - s[t, order]).max() < 1e-6
        assert gate is None
        x = _t(rng.standard_normal((T, K)), dtype)
        w_gu = _t(2.0 * rng.standard_normal((E, 2 * F, K)) / np.sqrt(K), dtype)
        w_down = _t(rng.standard_normal((E, K, F)) / np.sqrt(F), dtype)
        for act, fn in (("silu", pd.silu), ("gelu_tanh", pd.gelu_tanh)):
            old, ops.GROUPED_KERNEL = ops.GROUPED_KERNEL, kernel
            try:
                lay = ops.moe_layout(chosen, E, dtype, K, F)
                y = ops.moe_experts_down(ops.moe_experts_up(x, w_gu, lay, top, act=act, in_scale=weight), w_down, lay)
            finally:
                ops.GROUPED_KERNEL = old
            out = _np(ops.moe_combine(y, lay.pos_of, None, None, None, top=top))
            ref, wrong = np.zeros((T, K)), np.zeros((T, K))
            for t in range(T):
                for j in range(top):
                    m, sc = _np(w_gu[ch[t, j]]), _np(weight)[t, j]
                    run = lambda h: _np(_t(fn(h @ m[:F].T) * (h @ m[F:].T), dtype)) @ _np(w_down[ch[t, j]]).T  # noqa: E731
                    ref[t] += run(sc * _np(x[t]))
                    wrong[t] += sc * run(_np(x[t]))
            tol = (1e-4 if dtype == torch.float32 else 0.03) * max(1.0, np.abs(ref).max())
            assert np.abs(out - ref).max() < tol and np.abs(ref - wrong).max() > 2 * tol
    ops.take_device_errors()


def test_the_choice_compares_logits():
    """Logits whose sigmoids are equal in 32-bit are still told apart, equal logits go to the smaller index, and a row
    of padding that holds no numbers names existing experts."""
    torch = _torch()
    from llm_inference_lab_b200.kernels import ops
    z = np.array([[30.0, 40.0, 35.0, -1.0], [2.0, 2.0, 5.0, 2.0], [np.nan, np.inf, -np.inf, np.nan], [-200.0, -150.0, -190.0, -300.0]])
    chosen, weight, _ = ops.moe_route(_t(z), 4, 2, renorm=False, score="sigmoid")
    ch = chosen.cpu().numpy()
    assert list(ch[0]) == [1, 2] and list(ch[1]) == [2, 0] and list(ch[3]) == [1, 2]
    assert len(set(ch[2])) == 2 and all(0 <= e < 4 for e in ch[2]) and bool(torch.isfinite(weight).all())
    assert np.allclose(_np(weight)[1], pd.sigmoid(np.array([5.0, 2.0])), atol=1e-6) and float(weight[3].max()) < 1e-30
    ops.take_device_errors()


def test_prenorm_residual_without_streams():
    """The plain pre-norm residual of the streams' block: the sum is 32-bit whatever the storage type, and the norm
    that opens the next sublayer reads the new sum."""
    torch = _torch()
    from llm_inference_lab_b200.kernels import ops
    rng = np.random.default_rng(4)
    T, W = 9, 50
    one = torch.ones((1,), device="cuda")
    for dtype in _dtypes():
        x = _t(rng.standard_normal((T, 1, W)) * 100.0)
        y, w = _t(rng.standard_normal((3, T, W)) * 0.01), _t(1 + 0.2 * rng.standard_normal(W), dtype)
        before = _np(x)[:, 0]
        h = ops.hyper_write(x, y, one.view(1, 1), one, one, w, 1e-6)
        want = before + _np(y).sum(0)
        assert np.abs(_np(x)[:, 0] - want).max() < 2e-5
        assert np.abs(_np(h) - pd.rms_norm(want, _np(w), 1e-6)).max() < (1e-5 if dtype == torch.float32 else 0.02)


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


CLOSE = 0.15      # between two router logits whose spread over the experts is about 4


def _check(got, want, dtype, label, close=()):
    """32-bit: every position within F32_MAX.  bfloat16: without the positions of `close` (a routed layer may pick
    another expert where two logits are a rounding apart) the rms error within BF16_RMS and all but one position in a
    hundred within BF16_MAX (another expert's result moves later positions a little)."""
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
    "attention": config([attention(4, 2, 16, 24, window=7, turn=rot(100.0, 8), scale=0.3)], vocab=53, width=32),
    "attention+dense": config([attention(3, 1, 24, 8, window=16, turn=rot(3000.0, 24, (4.0, 1.0, 2.0, 80)), scale=0.25,
                                         v_mix=True, mlp=dense(56))], vocab=53, width=40),
    "attention+moe": config([attention(8, 1, 32, 16, scale=0.2, mlp=moe(6, 2, 16))], vocab=53, width=48),
    "heads beyond the tensor cores": config([attention(2, 1, 144, 40, window=12, turn=rot(900.0, 64), scale=0.08, v_mix=True),
                                             attention(2, 2, 8, 20, window=20, turn=rot(40.0, 2), scale=0.5, v_mix=True,
                                                       mlp=moe(2, 1, 8))], vocab=53, width=24),
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(ONE_LAYER))
def test_one_layer_models(tmp_path, name, dtype):
    rng = np.random.default_rng(3)
    cfg = ONE_LAYER[name]
    folder = make_model_folder(str(tmp_path / "m"), cfg, 21, dtype, std=0.08, scales=SPREAD)
    seqs = sequences(rng, cfg["vocab"], [45, 1, 30])
    want, close = plain_logits(folder, seqs), close_calls(folder, seqs, CLOSE)
    for label, steps in (("whole", trace_whole(seqs)), ("tail", trace_tail_decode(seqs, tail=25)),
                         ("portions", trace_portions(seqs))):
        eng = _engine(folder, dtype, dict(page_size=8), steps)
        _check(run_trace_inprocess(eng, steps), want, dtype, (name, label), close)
        assert eng.cache.live_requests == 0


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(SMALL))
def test_models_under_every_cut(tmp_path, name, dtype):
    """Whole prompts; the tail decoded token by token, past every window; portions of 2 to 11 tokens; up to four live
    requests with portions beside single tokens, in a pool so small that pages are used again."""
    cfg, opt = SMALL[name]
    rng = np.random.default_rng(opt["seed"])
    folder = make_model_folder(str(tmp_path / "m"), cfg, opt["seed"], dtype, std=0.08, scales=SPREAD)
    seqs = sequences(rng, cfg["vocab"], [150, 3, 61, 90, 1, 77, 40])
    want, close = plain_logits(folder, seqs), close_calls(folder, seqs, CLOSE)
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
    """Portions of more than a hundred tokens beside single tokens, and a tail of 150 decoded tokens, at heads of
    64 and 128 entries over one key/value head with windows of up to 260 tokens."""
    cfg, opt = SMALL["D"]
    folder = make_model_folder(str(tmp_path / "m"), cfg, opt["seed"], "bfloat16", std=0.08, scales=SPREAD)
    seqs = sequences(np.random.default_rng(9), cfg["vocab"], [400, 130, 260])
    want, close = plain_logits(folder, seqs), close_calls(folder, seqs, CLOSE)
    for label, steps in (("whole", trace_whole(seqs)), ("tail", trace_tail_decode(seqs, tail=150)),
                         ("mixed", trace_mixed(seqs, np.random.default_rng(2), max_live=3, max_portion=140))):
        eng = _engine(folder, "bfloat16", opt, steps)
        _check(run_trace_inprocess(eng, steps), want, "bfloat16", label, close)


@pytest.mark.parametrize("trial", range(int(os.environ.get("LAB_RANDOM_DIFEDRA", "6"))))
def test_random_configurations_and_traces(tmp_path, trial):
    """Random configurations (sizes that are no multiples of 8 or 16, any heads, windows of 1 token to none, rotations
    with and without bands, layers that mix values under any cut into heads, 1 to 9 experts, page sizes 4 to 64)
    under mixed batches with pages used again, in 32-bit.  `LAB_RANDOM_DIFEDRA=N` runs N."""
    rng = np.random.default_rng(4000 + trial)
    cfg, page = random_config(rng)
    seqs = sequences(rng, cfg["vocab"], [int(n) for n in rng.integers(1, 150, size=6)])
    steps = trace_mixed(seqs, np.random.default_rng(trial), max_live=4, max_portion=int(rng.choice([9, 40, 140])))
    folder = make_model_folder(str(tmp_path / "m"), cfg, trial, "float32", std=0.08, scales=SPREAD)
    want = plain_logits(folder, seqs)
    eng = _engine(folder, "float32", dict(page_size=page), steps)
    got = run_trace_inprocess(eng, steps)
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
    for other in results[1:]:
        for key, row in results[0].items():
            assert np.abs(row - other[key]).max() <= 1e-5, key


def test_trace_program_and_a_failed_step(tmp_path):
    """bin/trace_run on a Difedra folder; and a step that fails leaves the pages as they were."""
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
    assert len(eng.views) == 4 and len(eng.state_tensors) == 0      # pages only: nothing else outlives a step
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
        tokens.append(int(np.argmax(pd.forward(cfg, w, tokens)[-1])))
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
    pcfg, w = pd.read_folder(folder)
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
    """Decode steps replayed from CUDA graphs, the values of the first mixing layer inside them: batches padded with
    requests of length zero, a batch that shrinks as requests finish.  32-bit: the plain model's tokens;
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
        pcfg, w = pd.read_folder(folder)
        assert got == [_greedy(pcfg, w, p, s.max_new_tokens) for p, s in zip(prompts, sampling)]
    else:
        assert got == run(False)


def test_command_line_generates(tmp_path):
    import json
    import subprocess
    import sys
    cfg, opt = SMALL["C"]
    folder = make_model_folder(str(tmp_path / "m"), cfg, 19, "float32", std=0.08, scales=SPREAD)
    pcfg, w = pd.read_folder(folder)
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    proc = subprocess.run([sys.executable, "-m", "llm_inference_lab_b200.cli", "--model-dir", folder, "--dtype", "f32",
                           "--prompt-ids", "3,14,15,9,2,6", "--max-new-tokens", "6", "--kv-tokens", "256"],
                          cwd=root, capture_output=True, text=True, timeout=600)
    assert proc.returncode == 0, proc.stderr[-2000:]
    line = json.loads(proc.stdout.strip().splitlines()[-1])
    assert line["generated_ids"] == _greedy(pcfg, w, [3, 14, 15, 9, 2, 6], 6)
