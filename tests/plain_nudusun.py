"""A plain, slow NumPy implementation of the Nudusun design: whole sequences, no cache, one
function per mechanism, 64-bit floats.  It shares no code with the engine; the tests hold the
engine against it.

Notation: x[t] is the residual row of token t (positions count from 0), h a sublayer's input,
W_name the matrix stored [out, in] and applied as W h.  A model folder's config.json gives every
size and constant.
"""
from __future__ import annotations

import json
import math
import os
import struct

import numpy as np


# ---------------------------------------------------------------------------------------------
# reading a model folder (safetensors: 8-byte length, JSON header, data)
# ---------------------------------------------------------------------------------------------
def read_folder(folder):
    with open(os.path.join(folder, "config.json")) as fh:
        cfg = json.load(fh)
    with open(os.path.join(folder, "model.safetensors"), "rb") as fh:
        (n,) = struct.unpack("<Q", fh.read(8))
        header = json.loads(fh.read(n))
        data = fh.read()
    w = {}
    for name, info in header.items():
        if name == "__metadata__":
            continue
        lo, hi = info["data_offsets"]
        raw = data[lo:hi]
        if info["dtype"] == "BF16":
            a = (np.frombuffer(raw, dtype="<u2").astype(np.uint32) << 16).view(np.float32).astype(np.float64)
        elif info["dtype"] == "F32":
            a = np.frombuffer(raw, dtype="<f4").astype(np.float64)
        elif info["dtype"] == "I32":
            a = np.frombuffer(raw, dtype="<i4").astype(np.int64)
        else:
            raise ValueError(info["dtype"])
        w[name] = a.reshape(info["shape"])
    return cfg, w


# ---------------------------------------------------------------------------------------------
# small pieces
# ---------------------------------------------------------------------------------------------
def sigmoid(z):
    z = np.asarray(z, dtype=np.float64)
    return np.where(z >= 0, 1.0 / (1.0 + np.exp(-np.abs(z))), np.exp(-np.abs(z)) / (1.0 + np.exp(-np.abs(z))))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def rms_norm(x, w, eps):
    """x over its root mean square along the last axis (eps inside the root), times w."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * w


def unit(x):
    """x over its length along the last axis (1e-6 inside the root)."""
    return x / np.sqrt(np.sum(x * x, axis=-1, keepdims=True) + 1e-6)


def causal_conv(u, w):
    """y[t, c] = sum_j w[c, j] u[t - (taps - 1) + j, c], zeros before the first token."""
    taps = w.shape[1]
    padded = np.concatenate([np.zeros((taps - 1, u.shape[1])), u])
    return sum(padded[j: j + u.shape[0]] * w[:, j] for j in range(taps))


def gated_delta_rule(q, k, v, decay, beta, state=None):
    """Token by token for one head: S <- decay S; S <- S + k (beta (v - S^T k))^T; o = S^T q.  q, k [T, D], v [T, V];
    returns (o [T, V], the last S [D, V])."""
    S = np.zeros((q.shape[1], v.shape[1])) if state is None else np.array(state, dtype=np.float64)
    out = np.zeros_like(v)
    for t in range(q.shape[0]):
        S = decay[t] * S
        S = S + np.outer(k[t], beta[t] * (v[t] - S.T @ k[t]))
        out[t] = S.T @ q[t]
    return out, S


def in_window(n, size):
    """[queries, keys]: which keys a query sees: its own and the size - 1 before it (size None: all before it)."""
    i, j = np.arange(n)[:, None], np.arange(n)[None, :]
    seen = j <= i
    return seen if size is None else seen & (i - j < size)


def capped(scores, cap):
    return scores if not cap else cap * np.tanh(scores / cap)


def softmax(scores, seen):
    s = np.where(seen, scores, -np.inf)
    e = np.exp(s - s.max(axis=-1, keepdims=True))
    return e / e.sum(axis=-1, keepdims=True)


def two_map_difference(a1, a2, lam, eps, diff):
    """(a1 - lam a2) over its root mean square along the last axis, times 1 - diff."""
    return rms_norm(a1 - lam * a2, 1.0, eps) * (1.0 - diff)


def map_weight(w, p, diff):
    """The second map's weight: exp(lq1 . lk1) - exp(lq2 . lk2) + diff."""
    return math.exp(w[p + "lq1"] @ w[p + "lk1"]) - math.exp(w[p + "lq2"] @ w[p + "lk2"]) + diff


# ---------------------------------------------------------------------------------------------
# mixers
# ---------------------------------------------------------------------------------------------
def delta_mixer(h, w, p, m, eps):
    T = h.shape[0]
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(causal_conv(h @ w[p + n].T, w[p + n + ".conv"])) for n in ("q", "k", "v"))
    q, k, v = unit(q.reshape(T, G, D)) * D ** -0.5, unit(k.reshape(T, G, D)), v.reshape(T, H, V)
    beta = sigmoid(h @ w[p + "b"].T)
    decay = np.exp(-np.exp(w[p + "A_log"]) * softplus(h @ w[p + "a"].T + w[p + "dt_bias"]))
    gate = silu((h @ w[p + "g"].T).reshape(T, H, V))
    o = np.stack([gated_delta_rule(q[:, i // (H // G)], k[:, i // (H // G)], v[:, i], decay[:, i], beta[:, i])[0]
                  for i in range(H)], axis=1)
    o = rms_norm(o, w[p + "norm"], eps) * gate
    return o.reshape(T, H * V) @ w[p + "o"].T


def attention(h, w, p, m, eps):
    T = h.shape[0]
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms_norm((h @ w[p + "q"].T).reshape(T, H, 2, D), w[p + "q.norm"], eps)
    k = rms_norm((h @ w[p + "k"].T).reshape(T, G, 2, D), w[p + "k.norm"], eps)
    v = (h @ w[p + "v"].T).reshape(T, G, V)
    seen = in_window(T, m["mask"]["size"] if m.get("mask") else None)
    lam, per = map_weight(w, p, m["diff"]), H // G
    heads = []
    for i in range(H):
        a = [softmax(capped(q[:, i, j] @ k[:, i // per, j].T * m["scale"], m.get("softcap")), seen) @ v[:, i // per]
             for j in range(2)]
        heads.append(two_map_difference(a[0], a[1], lam, eps, m["diff"]))
    return np.stack(heads, axis=1).reshape(T, H * V) @ w[p + "o"].T


# ---------------------------------------------------------------------------------------------
# feed-forward
# ---------------------------------------------------------------------------------------------
def capped_expert(h, w, p, limit):
    g = np.minimum(h @ w[p + "gate"].T, limit)
    u = np.clip(h @ w[p + "up"].T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ w[p + "down"].T


def choose(s, correction, top, groups, keep):
    """Indices of the chosen experts of one token, best first: the largest s + correction among the experts of the
    `keep` groups whose largest one is largest (ties: the smaller index).  Also the smallest margin by which the
    choice was made."""
    c = s + correction
    size = len(c) // groups
    best = [c[g * size: (g + 1) * size].max() for g in range(groups)]
    order = sorted(range(groups), key=lambda g: (-best[g], g))
    margin = best[order[keep - 1]] - best[order[keep]] if keep < groups else np.inf
    open_ = [e for g in order[:keep] for e in range(g * size, (g + 1) * size)]
    ranked = sorted(open_, key=lambda e: (-c[e], e))
    if top < len(ranked):
        margin = min(margin, c[ranked[top - 1]] - c[ranked[top]])
    return ranked[:top], margin


def routed_experts(h, w, p, mlp, margins=None):
    """`margins` (a list) receives, per token, the smallest difference of two choice scores that decided something."""
    r = mlp["router"]
    E, ident = r["experts"], r.get("identity", 0)
    groups = r.get("groups") or {"count": 1, "keep": 1}
    z = h @ w[p + "router"].T
    s = np.exp(z - z.max(axis=1, keepdims=True))
    s = s / s.sum(axis=1, keepdims=True)
    assert s.shape[1] == E + ident
    out, margin = np.zeros_like(h), np.zeros(len(h))
    for t in range(h.shape[0]):
        chosen, margin[t] = choose(s[t], w[p + "correction"], r["top"], groups["count"], groups["keep"])
        for e in chosen:
            y = h[t] if e >= E else capped_expert(h[t:t + 1], w, f"{p}e{e}.", mlp["expert"]["limit"])[0]
            out[t] += r["scale"] * s[t, e] * y
    if margins is not None:
        margins.append(margin)
    if mlp.get("shared") is not None:
        out = out + capped_expert(h, w, p + "shared.", mlp["shared"]["limit"])
    return out


# ---------------------------------------------------------------------------------------------
# the model
# ---------------------------------------------------------------------------------------------
def embedding(cfg, w, tokens):
    return w["embed"][np.asarray(tokens)] * cfg["embedding"]["scale"] + w["pos"][: len(tokens)]


def token_input(x, w, p, tokens, layer, dim, eps):
    """What layer `layer` adds to the stream from its own part of the token's side vector."""
    e = w["side.embed"][np.asarray(tokens)][:, layer * dim: (layer + 1) * dim]
    y = (gelu_tanh(x @ w[p + "side.gate"].T) * e) @ w[p + "side.proj"].T
    return rms_norm(y, w[p + "side.norm"], eps)


def forward(cfg, w, tokens, layers_out=None, margins=None):
    """Logits [tokens, vocab] of one sequence; `layers_out` (a list) receives the residual after every layer,
    `margins` the routers' margins of every routed layer."""
    eps, alpha = cfg["norm"]["eps"], cfg["postln_alpha"]
    x = embedding(cfg, w, tokens)
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        mixer = delta_mixer if layer["type"] == "delta" else attention
        x = rms_norm(alpha * x + mixer(x, w, p + "mix.", layer["mixer"], eps), w[p + "norm1"], eps)
        if layer.get("mlp") is not None:
            x = rms_norm(alpha * x + routed_experts(x, w, p + "mlp.", layer["mlp"], margins), w[p + "norm2"], eps)
        if cfg.get("token_side") is not None:
            x = x + token_input(x, w, p, tokens, i, cfg["token_side"]["dim"], eps)
        if layers_out is not None:
            layers_out.append(x)
    return rms_norm(x, w["final.norm"], eps) @ w["head"].T
