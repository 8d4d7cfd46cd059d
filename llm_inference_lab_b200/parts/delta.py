"""Recurrent mixers by the delta rule: the generalized rule with decays per channel, and the gated rule with one decay
per head."""
from __future__ import annotations

import math

import torch

from ..kernels import ops
from .base import CacheView, Mixer, StepContext, register_part
from .spec import CacheParts, FixedState, PartSpec, TensorSpec


class GeneralDelta(Mixer):
    """Per head a state matrix S [key channel, value channel] in 32-bit, carried token by token:

        S_t = diag(w_t) S_{t-1} - (a_t * u_t) (u_t^T S_{t-1}) + k_t v_t^T,      o_t = S_t^T r_t

    r, k, v = W_r h, W_k h, W_v h (heads x dim each); decay w = exp(-rate * sigmoid(W_w2 tanh(W_w1 h) + w0))
    per head and key channel through a low-rank pair; removal rate a = sigmoid(W_a h + b_a); u the key
    divided by sqrt(sum k^2 + 1e-6).  Each head's o is divided by its root mean square, the heads side by
    side are multiplied by a plain weight and by sigmoid(W_g h), and W_o closes.  `decay_rate` is a
    parameter (exp(-1/2) where a design fixes it so).

    The six matrices that read h are concatenated at load time: one product.  Everything that enters the
    recurrence besides the products themselves is formed in 32-bit inside the recurrence kernel
    (`csrc/kernels/delta_rule.cu`), which serves prompts' portions and single decoded tokens alike."""
    decode_graph_safe = True


    NAMES = ("r", "k", "v", "g", "a")

    @classmethod
    def tensors(cls, spec: PartSpec):
        h, hd, p = spec["hidden"], spec["heads"] * spec["dim"], spec.prefix
        rank = int(spec.get("decay_rank") or -1)      # -1: the checkpoint's tensors say
        out = [TensorSpec(p + n, (hd, h)) for n in cls.NAMES]
        out += [TensorSpec(p + "a.b", (hd,), init="bias"), TensorSpec(p + "w1", (rank, h)),
                TensorSpec(p + "w2", (hd, rank)), TensorSpec(p + "w0", (hd,), init="bias"),
                TensorSpec(p + "norm", (hd,), init="norm"), TensorSpec(p + "o", (h, hd))]
        return out

    @classmethod
    def cache_need(cls, spec: PartSpec):
        return FixedState((spec["heads"], spec["dim"], spec["dim"]))

    @classmethod
    def libraries(cls, spec, dtype):
        return [("delta_rule", {"LAB_HEAD_DIM": int(spec["dim"])})]

    def __init__(self, spec, weights, dtype, device):
        super().__init__(spec, weights, dtype, device)
        self.heads, self.dim = int(spec["heads"]), int(spec["dim"])
        if not ops.delta_rule_supported(self.dim):
            raise ValueError(f"general_delta: head size {self.dim} is outside what the recurrence kernel takes")
        self.hd = self.heads * self.dim
        w = lambda n: self._weight(weights, n)  # noqa: E731
        self.w_in = torch.cat([w(n) for n in self.NAMES] + [w("w1")], dim=0).contiguous()
        self.w_up = w("w2").contiguous()
        self.decay_bias, self.rate_bias, self.norm_weight = w("w0"), w("a.b"), w("norm")
        self.w_o = w("o").contiguous()
        self.eps = float(spec["eps"])
        self.decay_rate = float(spec.get("decay_rate", math.exp(-0.5)))

    def forward(self, x: torch.Tensor, ctx: StepContext, cache: CacheView) -> torch.Tensor:
        proj = ops.linear(x, self.w_in, None, out_f32=True)
        middle = ops.tanh_cast(proj[:, 5 * self.hd:], self.dtype, self.dim)
        decay_pre = ops.linear(middle, self.w_up, None, out_f32=True)
        o = ops.delta_rule(proj, decay_pre, self.decay_bias, self.rate_bias, self.norm_weight, cache.state, ctx,
                           self.heads, self.dim, self.eps, self.decay_rate, write=cache.write)
        return ops.linear(o, self.w_o, None, out_f32=True, allow_partial=True)


register_part("mixer", "general_delta", GeneralDelta)


class GatedDelta(Mixer):
    """The gated delta rule with short convolutions.  q = W_q h, k = W_k h (`kv_heads` x `dim`), v = W_v h (`heads` x
    `vdim`); head h reads the q and k of group h // (heads / kv_heads).  Every channel of q, k and v passes a causal
    convolution over its last `taps` inputs (tensors `q.conv`, `k.conv`, `v.conv` [channels, taps], the last column on
    the current token, no bias, zeros before the sequence) and SiLU.  q and k become unit vectors per head, x /
    sqrt(sum x^2 + `unit_eps`), q times dim^(-1/2).  Per head, with the rate beta = sigmoid(W_b h) and the decay
    g = exp(-exp(A_log) softplus(W_a h + dt_bias)):

        S <- g S;   S <- S + k (beta (v - S^T k))^T;   o = S^T q

    Each head's o over its root mean square (`eps`), times a weight of `vdim` entries all heads share, times
    silu(W_g h); W_o closes.  Per request the mixer keeps S (32-bit) and the convolutions' last taps - 1 inputs: two
    fixed-size states (`CacheParts`).

    The matrices that read h are one product, taken in 32-bit; one kernel convolves, forms the unit vectors, rates
    and decays, one walks the state in blocks of four tokens and renews the kept inputs, one norms and gates
    (`csrc/kernels/gated_delta.cu`).  All of it is 32-bit up to the rounding before W_o."""
    decode_graph_safe = True
    CONVOLVED = ("q", "k", "v")

    @classmethod
    def _sizes(cls, spec):
        return spec["kv_heads"] * spec["dim"], spec["heads"] * spec["vdim"]

    @classmethod
    def tensors(cls, spec: PartSpec):
        h, H, p = spec["hidden"], spec["heads"], spec.prefix
        gd, hv = cls._sizes(spec)
        out = []
        for n, rows in zip(cls.CONVOLVED, (gd, gd, hv)):
            out += [TensorSpec(p + n, (rows, h)), TensorSpec(p + n + ".conv", (rows, spec["taps"]))]
        out += [TensorSpec(p + "g", (hv, h)), TensorSpec(p + "b", (H, h)), TensorSpec(p + "a", (H, h)),
                TensorSpec(p + "A_log", (H,), init="bias"), TensorSpec(p + "dt_bias", (H,), init="bias"),
                TensorSpec(p + "norm", (spec["vdim"],), init="norm"), TensorSpec(p + "o", (h, hv))]
        return out

    @classmethod
    def cache_need(cls, spec: PartSpec):
        gd, hv = cls._sizes(spec)
        return CacheParts((FixedState((spec["heads"], spec["dim"], spec["vdim"])),
                           FixedState((max(spec["taps"] - 1, 0), 2 * gd + hv))))

    @classmethod
    def libraries(cls, spec, dtype):
        return [("gated_delta", {})]

    def __init__(self, spec, weights, dtype, device):
        super().__init__(spec, weights, dtype, device)
        self.heads, self.groups, self.dim, self.vdim, self.taps = (
            int(spec[k]) for k in ("heads", "kv_heads", "dim", "vdim", "taps"))
        if self.heads % self.groups:
            raise ValueError("gated_delta: heads must be a multiple of kv_heads")
        if not ops.gated_delta_supported(self.dim):
            raise ValueError(f"gated_delta: {self.dim} key channels are outside what the recurrence kernel takes")
        self.eps, self.unit_eps = float(spec["eps"]), float(spec.get("unit_eps", 1e-6))
        w = lambda n: self._weight(weights, n)  # noqa: E731
        self.gd, self.hv = self._sizes(spec)
        self.w_in = torch.cat([w(n) for n in ("q", "k", "v", "g", "b", "a")], dim=0).contiguous()
        self.gate_at = 2 * self.gd + self.hv
        self.rate_at = self.gate_at + self.hv
        self.decay_at = self.rate_at + self.heads
        self.conv_w = torch.cat([w(n + ".conv") for n in self.CONVOLVED], dim=0).contiguous()
        self.a_log, self.dt_bias, self.norm_weight = w("A_log"), w("dt_bias"), w("norm")
        self.w_o = w("o").contiguous()

    def forward(self, x: torch.Tensor, ctx: StepContext, cache: CacheView) -> torch.Tensor:
        proj = ops.linear(x, self.w_in, None, out_f32=True)
        state, kept = cache.part(0), cache.part(1)
        operands = ops.delta_prepare(
            proj, self.rate_at, self.decay_at, self.taps, self.heads, self.groups, self.dim, self.vdim, self.conv_w,
            self.a_log, self.dt_bias, kept.state, ctx, self.dim ** -0.5, self.unit_eps)
        o = ops.delta_walk(*operands, state.state, ctx, self.heads, self.groups, self.dim, self.vdim, write=cache.write,
                           proj=proj, kept=kept.state)
        y = ops.head_norm_gate(o, proj[:, self.gate_at: self.gate_at + self.hv], self.norm_weight, ctx, self.heads,
                               self.vdim, self.eps)
        return ops.linear(y, self.w_o, None, out_f32=True, allow_partial=True)


register_part("mixer", "gated_delta", GatedDelta)
