"""A feed-forward gated by the token's own vector."""
from __future__ import annotations

from ..kernels import ops
from .base import FeedForward, register_part
from .spec import PartSpec, TensorSpec


class TokenGate(FeedForward):
    """y = W_proj (gelu(W_gate h) * e), the tanh form, with e the part [at, at + dim) of the token's row of a side
    table [vocab, table_width] that the layers of a model share (tensors `table`; `<prefix>gate` [dim, hidden],
    `<prefix>proj` [hidden, dim]).  The result is 32-bit, whole or as split-K partial products."""

    @classmethod
    def tensors(cls, spec: PartSpec):
        h, d, p = spec["hidden"], spec["dim"], spec.prefix
        return [TensorSpec(spec["table"], (spec["vocab"], spec["table_width"]), init="table"),
                TensorSpec(p + "gate", (d, h)), TensorSpec(p + "proj", (h, d))]

    @classmethod
    def libraries(cls, spec, dtype):
        return [("stream32", {})]

    def __init__(self, spec, weights, dtype, device):
        super().__init__(spec, weights, dtype, device)
        t = weights[spec["table"]]
        self.table = (t if t.dtype == dtype else t.to(dtype)).contiguous()
        weights[spec["table"]] = self.table        # the other layers share this storage
        self.at, self.dim = int(spec["at"]), int(spec["dim"])
        self.w_gate, self.w_proj = self._weight(weights, "gate").contiguous(), self._weight(weights, "proj").contiguous()

    def forward(self, x, ctx):
        p = ops.linear(x, self.w_gate, None, out_f32=True, allow_partial=True)
        return ops.linear(ops.token_gate(p, self.table, ctx.token_ids, self.at), self.w_proj, None, out_f32=True,
                          allow_partial=True)


register_part("feed_forward", "token_gate", TokenGate)
