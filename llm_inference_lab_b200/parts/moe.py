"""A routed feed-forward: a mixture of small gated experts, with an optional shared expert."""
from __future__ import annotations

import torch

from ..kernels import ops
from .base import FeedForward, register_part
from .spec import PartSpec, TensorSpec


class RoutedExperts(FeedForward):
    """`experts` gated feed-forwards W_down (silu(W_gate h) * (W_up h)) of `expert_ff` rows, without biases, of
    which every token uses `top`: router logits z = W_router h in 32-bit, scores softmax(z) over all experts,
    the `top` largest chosen (ties: the smaller index), weighted by their scores over the sum of the chosen
    scores (+ 1e-20).  `score` "sigmoid": scores sigmoid(z), one expert's apart from the others'.  `scale_input` True:
    a weight multiplies its expert's input instead of its output, the result is the sum of expert(w * h).  `shared_ff` > 0: one more expert of that many rows runs for every token and is added,
    with `shared_gate` multiplied by sigmoid(W_sg h), one number per token.  `renorm` False: the weights are the
    chosen scores as they are.  `limit` > 0 (and `shared_limit` for the shared expert): the experts are of the
    capped form W_down (g' * sigmoid(1.702 g') * (u' + 1)) with g' = min(W_gate h, limit) and u' = clamp(W_up h,
    -limit, limit).

    `correction` True: a learned number per expert (tensor `correction`) joins the scores for the choice, not for the
    weights.  `groups` (count, keep): the experts form `count` equal groups of neighbours and only those of the `keep`
    groups whose largest choice score is largest can be chosen.  `identity` > 0: the router has that many more
    outputs, identity experts without matrices whose result is h itself.  `router_scale` multiplies the weights.

    The router's matrix and the gate's row are one product; one kernel picks, one lays the (token, expert)
    pairs out in rows grouped by expert, two grouped products run the experts, and one kernel forms the weighted
    sum, in the order of each token's choice, with the shared expert's share.  Steps of many pairs in bfloat16
    run the grouped products on the tensor cores over rows gathered into the layout; else the ordinary units
    gather while they load.  The result is 32-bit.  `forward_post_norm` leaves the weighted sum in a 32-bit stream
    that is normed as a whole, in one pass."""

    NAMES = {"router": "router", "expert": "e{}.", "gate": "gate", "up": "up", "down": "down", "shared": "shared.",
             "shared_gate": "shared.sg", "correction": "correction"}

    @classmethod
    def names(cls, spec: PartSpec) -> dict:
        return {**cls.NAMES, **(spec.get("names") or {})}

    @classmethod
    def tensors(cls, spec: PartSpec):
        h, E, F, p, n = spec["hidden"], spec["experts"], spec["expert_ff"], spec.prefix, cls.names(spec)
        outputs = E + int(spec.get("identity") or 0)
        out = [TensorSpec(p + n["router"], (outputs, h))]
        if spec.get("correction"):
            out.append(TensorSpec(p + n["correction"], (outputs,), init="bias"))
        for e in range(E):
            q = p + n["expert"].format(e)
            out += [TensorSpec(q + n["gate"], (F, h)), TensorSpec(q + n["up"], (F, h)), TensorSpec(q + n["down"], (h, F))]
        S = int(spec.get("shared_ff") or 0)
        if S:
            q = p + n["shared"]
            out += [TensorSpec(q + n["gate"], (S, h)), TensorSpec(q + n["up"], (S, h)), TensorSpec(q + n["down"], (h, S))]
            if spec.get("shared_gate"):
                out.append(TensorSpec(p + n["shared_gate"], (1, h)))
        return out

    @classmethod
    def libraries(cls, spec, dtype):
        return [("moe", {})]       # the products' libraries belong to every model

    def __init__(self, spec, weights, dtype, device):
        super().__init__(spec, weights, dtype, device)
        self.experts, self.top, self.ff = int(spec["experts"]), int(spec["top"]), int(spec["expert_ff"])
        self.identity = int(spec.get("identity") or 0)
        self.outputs = self.experts + self.identity
        self.groups, self.keep = (int(g) for g in (spec.get("groups") or (1, 1)))
        self.router_scale = float(spec.get("router_scale", 1.0))
        if not 0 < self.top <= self.outputs:
            raise ValueError("routed_experts: top must lie in 1..experts")
        if self.outputs % self.groups or not 1 <= self.keep <= self.groups or \
                self.top > self.keep * (self.outputs // self.groups):
            raise ValueError("routed_experts: groups must divide the experts, and the kept ones hold at least top experts")
        n = self.names(spec)
        w = lambda name: self._weight(weights, name)  # noqa: E731
        self.shared_ff = int(spec.get("shared_ff") or 0)
        self.gated_share = bool(self.shared_ff and spec.get("shared_gate"))
        self.renorm = bool(spec.get("renorm", True))
        self.score = spec.get("score", "softmax")
        if self.score not in ops.MOE_SCORES:
            raise ValueError(f"routed_experts: score {self.score!r} is not one of {tuple(ops.MOE_SCORES)}")
        self.scale_input = bool(spec.get("scale_input"))
        self.limit, self.shared_limit = float(spec.get("limit") or 0.0), float(spec.get("shared_limit") or 0.0)
        rows = [w(n["router"])] + ([w(n["shared_gate"]).reshape(1, -1)] if self.gated_share else [])
        self.w_router = torch.cat(rows, dim=0).contiguous()
        self.correction = None
        if spec.get("correction"):
            self.correction = weights[spec.prefix + n["correction"]].to(device=device, dtype=torch.float32).contiguous()
        if self.scale_input and self.identity:
            raise ValueError("routed_experts: identity experts go with weights on the experts' outputs")
        names = [n["expert"].format(e) for e in range(self.experts)]
        self.w_gate_up = torch.stack([torch.cat([w(q + n["gate"]), w(q + n["up"])], dim=0) for q in names]).contiguous()
        self.w_down = torch.stack([w(q + n["down"]) for q in names]).contiguous()
        if self.shared_ff:
            q = n["shared"]
            self.w_shared_gate_up = torch.cat([w(q + n["gate"]), w(q + n["up"])], dim=0).contiguous()
            self.w_shared_down = w(q + n["down"]).contiguous()

    def _experts(self, x):
        """The choice and the chosen experts' results: (chosen, weights, shared gate, layout, results by layout row)."""
        E, top = self.experts, self.top
        logits = ops.linear(x, self.w_router, None, out_f32=True)
        chosen, weight, gate = ops.moe_route(logits, self.outputs, top, gate_col=self.outputs if self.gated_share else -1,
                                             renorm=self.renorm, score=self.score, correction=self.correction,
                                             groups=self.groups, keep=self.keep, scale=self.router_scale)
        lay = ops.moe_layout(chosen, E, x.dtype, x.shape[1], self.ff)
        act = ops.moe_experts_up(x, self.w_gate_up, lay, top, limit=self.limit,
                                 in_scale=weight if self.scale_input else None)
        return chosen, None if self.scale_input else weight, gate, lay, ops.moe_experts_down(act, self.w_down, lay)

    def _shared(self, x, allow_partial=False):
        if not self.shared_ff:
            return None
        return ops.linear(ops.linear_gated(x, self.w_shared_gate_up, limit=self.shared_limit), self.w_shared_down,
                          None, out_f32=True, allow_partial=allow_partial)

    def forward(self, x, ctx):
        chosen, weight, gate, lay, y = self._experts(x)
        more = {"chosen": chosen, "identity_from": self.experts, "h": x} if self.identity else {}
        return ops.moe_combine(y, lay.pos_of, weight, self._shared(x), gate, top=self.top, **more)

    def forward_post_norm(self, stream, x, ctx, weight, alpha, eps, copy):
        """stream <- rmsnorm(alpha * stream + the layer's result on x) * weight, x the stream's rows rounded; identity
        experts give the stream's own 32-bit rows.  Returns the new rows rounded with `copy`."""
        chosen, w, gate, lay, y = self._experts(x)
        return ops.moe_combine_norm(stream, y, lay.pos_of, w, chosen, self.experts, self._shared(x, allow_partial=True),
                                    gate, weight, alpha, eps, copy=copy)


register_part("feed_forward", "routed_experts", RoutedExperts)
