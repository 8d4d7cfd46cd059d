"""A plain, slow NumPy implementation of the Difedra design: whole sequences, no cache, one
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


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def rms_norm(x, w, eps):
    """x over its root mean square along the last axis (eps inside the root), times w."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * w


def frequencies(base, dims, scaling=None):
    """f_i = base^(-2i / dims), i < dims / 2.  With `scaling`: a frequency whose wavelength is longer than
    original / low is divided by factor, one shorter than original / high stays, and between the two the
    results are blended linearly in original / wavelength."""
    out = []
    for i in range(dims // 2):
        f = float(base) ** (-2.0 * i / dims)
        if scaling is not None:
            wave = 2.0 * math.pi / f
            if wave > scaling["original"] / scaling["low"]:
                f = f / scaling["factor"]
            elif wave >= scaling["original"] / scaling["high"]:
                s = (scaling["original"] / wave - scaling["low"]) / (scaling["high"] - scaling["low"])
                f = (1.0 - s) * f / scaling["factor"] + s * f
        out.append(f)
    return np.asarray(out, dtype=np.float64)


def rotate_halves(v, positions, freq):
    """Entries i and i + n of the last axis of v [tokens, heads, d], n = len(freq), turn by position * freq[i];
    entries from 2n on stay."""
    out = np.array(v, dtype=np.float64, copy=True)
    n = len(freq)
    for i in range(n):
        angle = np.asarray(positions, dtype=np.float64) * freq[i]
        cs, sn = np.cos(angle)[:, None], np.sin(angle)[:, None]
        a, b = v[..., i], v[..., i + n]
        out[..., i] = a * cs - b * sn
        out[..., i + n] = b * cs + a * sn
    return out


def in_window(n, size):
    """[queries, keys]: which keys a query sees: its own and the size - 1 before it (size None: all before it)."""
    i, j = np.arange(n)[:, None], np.arange(n)[None, :]
    seen = j <= i
    return seen if size is None else seen & (i - j < size)


def sink_softmax(scores, seen, sink):
    """Softmax over the seen keys of scores [heads, queries, keys]; the denominator also holds exp(sink[head])."""
    s = np.where(seen, scores, -np.inf)
    sink = np.asarray(sink, dtype=np.float64).reshape(-1, 1, 1)
    top = np.maximum(s.max(axis=-1, keepdims=True), sink)
    e = np.exp(s - top)
    return e / (e.sum(axis=-1, keepdims=True) + np.exp(sink - top))


def mixed_values(v, first, lam):
    """(1 - lam) v + lam first."""
    return (1.0 - lam) * v + lam * first


# ---------------------------------------------------------------------------------------------
# mixer and feed-forward
# ---------------------------------------------------------------------------------------------
def attention(h, w, p, m, eps, v_first):
    """The mixer's result and the values to hand on: this layer's own where it is the first that mixes, else
    `v_first` as it came."""
    T = h.shape[0]
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    pos = np.arange(T)
    q = rms_norm(h @ w[p + "q"].T, w[p + "q.norm"], eps).reshape(T, H, D)
    k = rms_norm(h @ w[p + "k"].T, w[p + "k.norm"], eps).reshape(T, G, D)
    v = h @ w[p + "v"].T
    rot = m.get("rot")
    if rot is not None:
        freq = frequencies(rot["base"], rot["dims"], rot.get("scaling"))
        q, k = rotate_halves(q, pos, freq), rotate_halves(k, pos, freq)
    if m.get("v_mix"):
        if v_first is None:
            v_first = v
        else:
            v = mixed_values(v, v_first, float(np.reshape(w[p + "vmix"], -1)[0]))
    v = v.reshape(T, G, V)
    per = H // G
    s = np.stack([q[:, i] @ k[:, i // per].T for i in range(H)]) * m["scale"]
    seen = in_window(T, m["mask"]["size"] if m.get("mask") else None)
    a = sink_softmax(s, seen[None], w[p + "sink"])
    out = np.stack([a[i] @ v[:, i // per] for i in range(H)], axis=1)
    return out.reshape(T, H * V) @ w[p + "o"].T, v_first


def gated_mlp(h, w, p, act):
    return (act(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def routed_experts(h, w, p, mlp, margins=None):
    """Sigmoid scores; the chosen scores as they are multiply the experts' inputs.  `margins` (a list) receives, per
    token, how far the last chosen expert's logit lies above the first one left out."""
    E, top = mlp["router"]["experts"], mlp["router"]["top"]
    z = h @ w[p + "router"].T
    s = sigmoid(z)
    if margins is not None:
        z = -np.sort(-z, axis=1)
        margins.append(z[:, top - 1] - z[:, top] if top < E else np.full(len(z), np.inf))
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        for e in sorted(range(E), key=lambda e: (-s[t, e], e))[:top]:
            out[t] += gated_mlp(s[t, e] * h[t:t + 1], w, f"{p}e{e}.", silu)[0]
    return out


# ---------------------------------------------------------------------------------------------
# the model
# ---------------------------------------------------------------------------------------------
def forward(cfg, w, tokens, layers_out=None, margins=None):
    """Logits [tokens, vocab] of one sequence; `layers_out` (a list) receives the residual after every layer,
    `margins` the routers' margins of every routed layer."""
    eps = cfg["norm"]["eps"]
    x = w["embed"][np.asarray(tokens)]
    v_first = None
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        a, v_first = attention(rms_norm(x, w[p + "norm1"], eps), w, p + "mix.", layer["mixer"], eps, v_first)
        x = x + a
        mlp = layer.get("mlp")
        if mlp is not None:
            h = rms_norm(x, w[p + "norm2"], eps)
            x = x + (gated_mlp(h, w, p + "mlp.", gelu_tanh) if mlp["kind"] == "dense"
                     else routed_experts(h, w, p + "mlp.", mlp, margins))
        if layers_out is not None:
            layers_out.append(x)
    return rms_norm(x, w["final.norm"], eps) @ w["embed"].T
