"""Differential attention: two score maps over the same values, the second subtracted from the first."""
from __future__ import annotations

import math

import torch

from ..kernels import ops
from .base import CacheView, Mixer, StepContext, register_part
from .spec import PagedKV, PartSpec, TensorSpec


class DifferentialAttention(Mixer):
    """q = W_q h (`heads` x 2 maps x `dim`, head by head), k = W_k h (`kv_heads` x 2 x `dim`), v = W_v h (`kv_heads` x
    `vdim`), no biases, no rotation; query head h reads key/value head h // (heads / kv_heads).  Every q and k vector
    of a head and map is RMS-normed over `dim` with a weight all heads and maps share (tensors `q.norm`, `k.norm`).
    A map's scores are q . k * `scale`, with `softcap` c > 0 then c * tanh(score / c); a query sees the last `window`
    keys, itself included (0: every earlier one); softmax per map.  With the maps' outputs a1 and a2 and the learned
    number lambda = exp(lq1 . lk1) - exp(lq2 . lk2) + `diff` (tensors of `dim` entries, one lambda for the layer),
    o = a1 - lambda a2 over its root mean square within the head (no weight), times 1 - `diff`.  W_o closes.

    The maps run as heads of the attention kernels over one cache.  Packed form: a key/value head holds the two keys
    side by side and the values once, and a query lies at its map's half with zeros in the other, so that its product
    with the whole key meets that half alone; where values are twice as wide as keys nothing is padded.  Split form,
    for heads whose two keys together are too wide for the tensor-core kernels: every map is a key/value head of its
    own, with the values stored twice; the queries are then ordered by group, map and head within the group (the
    rows of W_q are reordered at load time).  One kernel norms, rounds and stores; one combines the maps, whose outputs
    leave the attention kernels in 32-bit: the difference of two alike maps is small next to their own rounding."""
    decode_graph_safe = True

    @classmethod
    def _layout(cls, spec: PartSpec) -> tuple[bool, int]:
        """(packed, cached width of a head)."""
        packed = ops.padded_head(2 * spec["dim"], spec["vdim"])
        if packed <= 128:
            return True, packed
        return False, ops.padded_head(spec["dim"], spec["vdim"])

    @classmethod
    def tensors(cls, spec: PartSpec):
        h, H, G, D, V, p = spec["hidden"], spec["heads"], spec["kv_heads"], spec["dim"], spec["vdim"], spec.prefix
        return [TensorSpec(p + "q", (2 * H * D, h)), TensorSpec(p + "k", (2 * G * D, h)), TensorSpec(p + "v", (G * V, h)),
                TensorSpec(p + "q.norm", (D,), init="norm"), TensorSpec(p + "k.norm", (D,), init="norm"),
                *(TensorSpec(p + n, (D,), init="bias") for n in ("lq1", "lk1", "lq2", "lk2")),
                TensorSpec(p + "o", (h, H * V))]

    @classmethod
    def cache_need(cls, spec: PartSpec):
        packed, head = cls._layout(spec)
        return PagedKV(spec["kv_heads"] * (1 if packed else 2), head, int(spec.get("window") or 0))

    @classmethod
    def libraries(cls, spec, dtype):
        out = [("rope_pairs", {}), ("norm_attention", {})]
        _, head = cls._layout(spec)
        if dtype == torch.bfloat16 and ops.attention_tc_supported(head):
            out.append(("attention_tc", {"LAB_HEAD_DIM": head}))
            if head in (64, 128):
                out.append(("attention_tc05", {"LAB_HEAD_DIM": head}))
        else:
            out.append(("attention_plain", {}))
        return out

    def __init__(self, spec, weights, dtype, device):
        super().__init__(spec, weights, dtype, device)
        self.heads, self.groups, self.dim, self.vdim = (int(spec[k]) for k in ("heads", "kv_heads", "dim", "vdim"))
        if self.heads % self.groups:
            raise ValueError("differential_attention: heads must be a multiple of kv_heads")
        self.packed, self.head = self._layout(spec)
        if self.head > 256:
            raise ValueError(f"differential_attention: heads of {max(self.dim, self.vdim)} entries exceed the kernels' 256")
        self.per = self.heads // self.groups
        self.scale, self.softcap, self.eps = float(spec["scale"]), float(spec.get("softcap") or 0.0), float(spec["eps"])
        self.window, self.diff = int(spec.get("window") or 0), float(spec["diff"])
        w = lambda n: self._weight(weights, n)  # noqa: E731
        wq = w("q")
        if not self.packed:
            wq = wq.view(self.groups, self.per, 2, self.dim, -1).transpose(1, 2).reshape(wq.shape)
        self.w_in = torch.cat([wq, w("k"), w("v")], dim=0).contiguous()
        self.k_at = 2 * self.heads * self.dim
        self.v_at = self.k_at + 2 * self.groups * self.dim
        self.norm_q, self.norm_k = w("q.norm"), w("k.norm")
        f32 = lambda n: weights[spec.prefix + n].to(torch.float32)  # noqa: E731
        self.lam = (math.exp(float((f32("lq1") * f32("lk1")).sum())) - math.exp(float((f32("lq2") * f32("lk2")).sum()))
                    + self.diff)
        self.w_o = w("o").contiguous()

    def forward(self, x: torch.Tensor, ctx: StepContext, cache: CacheView) -> torch.Tensor:
        group = ctx.groups[cache.group]
        proj = ops.linear(x, self.w_in, None, out_f32=True, allow_partial=True)
        n_kv = self.groups * (1 if self.packed else 2)
        q = ops.head_prep_store(proj, None, ctx.row_pos, None, 0, group.row_slot if cache.write else None, cache.k,
                                cache.v, 2 * self.heads, n_kv, self.dim, self.vdim, self.head, self.k_at, self.v_at,
                                self.dtype, norm_eps=self.eps, q_norm_w=self.norm_q, k_norm_w=self.norm_k,
                                maps=2 if self.packed else 1, v_rep=1 if self.packed else 2)
        attn = ops.attention(q, cache.k, cache.v, ctx, group, 2 * self.heads, n_kv, self.head, self.window, self.scale,
                             softcap=self.softcap, out_f32=True)
        y = ops.map_difference(attn, self.heads, self.vdim, self.head, self.lam, self.eps, 1.0 - self.diff,
                               group=0 if self.packed else self.per, dtype=self.dtype)
        return ops.linear(y, self.w_o, None, out_f32=True, allow_partial=True)


register_part("mixer", "differential_attention", DifferentialAttention)
