"""A routed mixture of feed-forward experts, gated or plain, with an optional shared expert.

    z = W_r h  (float)           s = softmax(z) over all experts
    the ``top`` experts with the largest s are chosen; their weights are their s (divided by their sum only with
    ``renormalise``)
    out = sum over the chosen e of s_e * down_e(act(gate_e h) * (up_e h))
          + sigmoid(w_sg . h) * down_s(act(gate_s h) * (up_s h))          the shared expert, for every token

``scores`` "sigmoid": s = sigmoid(z).  ``groups`` (count, keep): the experts form ``count`` equal groups of neighbours; the
choice is among the ``keep`` groups with the largest sums of their two largest scores.  ``scale`` multiplies the weights.
``correction_name``: experts and groups are chosen by s + a learned number per expert, the weights stay the bare s.
``group_score`` "max": a group counts by its largest choice score.  ``identity``: that many router outputs behind the
experts' stand for the identity, out += weight * h; groups and softmax run over all router outputs.
``gated`` False: the experts are down_e(act(up_e h)).  With ``limit`` the experts are clamped gated units instead: g = min(gate_e h, limit), u = clamp(up_e h, -limit, limit),
down_e(g * sigmoid(alpha * g) * (u + shift)).

On the device the step's (token, choice) items are grouped by expert (``ops.moe_sort``), two grouped products run
over the groups (gate|up with the activation in the epilogue, then down), and one kernel forms the weighted sums and
adds the gated shared expert, in float.  Nothing comes back to the host, so steps are recorded like any others.
"""
from __future__ import annotations

from typing import Any, Dict, List, Optional, Sequence

import torch

from .. import ops
from ..weights.spec import MATRIX, VECTOR, ParamSpec
from .base import FEED_FORWARDS, Delta, FeedForward, Part


# steps of more tokens take the router logits from a product (few tokens: product and choice are one kernel)
ROUTE_PRODUCT_MIN_ROWS = 16


@FEED_FORWARDS.register("routed_experts")
class RoutedExperts(FeedForward):
    """expert_names: per expert {"gate", "up", "down"} tensor names (no "gate" with ``gated`` False); router_name: [experts, hidden] (kept in float);
    shared: a feed-forward part for every token or None, with shared_gate_name ([1, hidden] or [hidden], float) the
    weight of its sigmoid gate (None: the shared expert is added as it is)."""

    def __init__(self, hidden: int, inner: int, num_experts: int, top: int, activation: str,
                 expert_names: List[Dict[str, str]], router_name: str, shared: Optional[FeedForward] = None,
                 shared_gate_name: Optional[str] = None, renormalise: bool = False, limit: Optional[float] = None,
                 alpha: float = 1.0, shift: float = 0.0, scores: str = "softmax", groups: Optional[Sequence[int]] = None,
                 scale: float = 1.0, gated: bool = True, correction_name: Optional[str] = None, group_score: str = "top2",
                 identity: int = 0):
        self.limit, self.alpha, self.shift = (float(limit) if limit else None), float(alpha), float(shift)
        if activation not in ops.ACT_CODES:
            raise ValueError(f"activation '{activation}' is not supported ({', '.join(ops.ACT_CODES)})")
        outputs = num_experts + int(identity)          # what the router chooses from
        if len(expert_names) != num_experts or identity < 0 or not 1 <= top <= outputs:
            raise ValueError("a mixture needs names for every expert and 1 <= top <= router outputs")
        self.hidden, self.inner, self.n_experts, self.top, self.activation = hidden, inner, num_experts, top, activation
        self.expert_names, self.router_name = expert_names, router_name
        self.shared, self.shared_gate_name, self.renormalise = shared, shared_gate_name, renormalise
        if limit and not gated:
            raise ValueError("the clamped unit is a gated one")
        if groups and (outputs % groups[0] or not 1 <= groups[1] <= groups[0]):
            raise ValueError("expert groups: the number of router outputs must be a multiple of 'count', and 1 <= keep <= count")
        if groups and groups[1] * (outputs // groups[0]) < top:
            raise ValueError("the kept expert groups hold fewer experts than a token chooses")
        self.rule = dict(renorm=renormalise, scores=scores, groups=tuple(groups) if groups else None, scale=float(scale),
                         group_score=group_score)
        self.n_outputs, self.n_identity, self.correction_name = outputs, int(identity), correction_name
        self.gated = bool(gated)
        self.w_router = self.w_gu = self.w_down = self.w_sg = self.w_router_low = None

    def children(self) -> List[Part]:
        return [self.shared] if self.shared is not None else []

    def param_specs(self) -> List[ParamSpec]:
        specs = [ParamSpec(self.router_name, (self.n_outputs, self.hidden), VECTOR)]
        if self.correction_name:
            specs.append(ParamSpec(self.correction_name, (self.n_outputs,), VECTOR))
        for n in self.expert_names:
            specs += [ParamSpec(n["gate"], (self.inner, self.hidden), MATRIX)] if self.gated else []
            specs += [ParamSpec(n["up"], (self.inner, self.hidden), MATRIX),
                      ParamSpec(n["down"], (self.hidden, self.inner), MATRIX)]
        if self.shared is not None and self.shared_gate_name:
            specs.append(ParamSpec(self.shared_gate_name, (1, self.hidden), VECTOR))
        return specs

    def bind(self, tensors: Dict[str, torch.Tensor]) -> None:
        self.w_router = tensors[self.router_name]
        if self.correction_name:
            self.rule["correction"] = tensors[self.correction_name].to(torch.float32).contiguous()
        # [experts, 2 * inner, hidden]: an expert's gate rows, then its up rows (up rows alone without a gate);
        # [experts, hidden, inner]
        self.w_gu = torch.stack([torch.cat([tensors.pop(n["gate"]), tensors.pop(n["up"])], dim=0) if self.gated
                                 else tensors.pop(n["up"]) for n in self.expert_names]).contiguous()
        if self.w_gu.dtype == torch.bfloat16:
            # bfloat16 factors with float sums give the float router logits exactly: where the stored weights are
            # bfloat16 numbers, steps of many tokens take their logits from a matrix product
            self.w_router_low = ops.lossless_bf16(self.w_router)
        self.w_down = torch.stack([tensors.pop(n["down"]) for n in self.expert_names]).contiguous()
        if self.shared is not None and self.shared_gate_name:
            self.w_sg = tensors[self.shared_gate_name].reshape(-1).contiguous()

    def _experts(self, h: torch.Tensor, ctx: Any):
        """The chosen experts' results: (ExpertSum without the shared expert, the shared expert's gate or None)."""
        if self.w_router_low is not None and self.w_sg is None and h.shape[0] > ROUTE_PRODUCT_MIN_ROWS:
            z = ops.linear(h, self.w_router_low, out_dtype=torch.float32)
            experts, weights = ops.moe_choose(z, self.n_outputs, self.top, ctx.positions, **self.rule)
            gate = None
        else:
            experts, weights, gate = ops.moe_route(h, self.w_router, self.top, ctx.positions, self.w_sg, **self.rule)
        order = ops.moe_sort(experts, self.n_experts)
        if self.limit is not None:
            # gate | up of every item as the product leaves them, then the clamped unit over the rows
            u = ops.gated_clamped_act(ops.gemm_experts(h, self.w_gu, order, gather=True), None, self.limit, self.alpha,
                                      self.shift)
        else:
            u = ops.gemm_experts(h, self.w_gu, order, gather=True, gated=self.gated, act=self.activation)
        y = ops.gemm_experts(u, self.w_down, order, gather=False)
        some = dict(experts=experts, n_real=self.n_experts, identity=h) if self.n_identity else {}
        return ops.ExpertSum(y, order, weights, **some), gate

    def forward_unsummed(self, h: torch.Tensor, ctx: Any) -> Optional[Any]:
        """The experts' results as an ``ops.ExpertSum`` for a block whose next kernel forms the sum (None: this mixture
        has more to add, or more choices than that kernel takes; ``forward`` then)."""
        if self.shared is not None or self.top > ops.scaled_sum_norms_max_top():
            return None
        return self._experts(h, ctx)[0]

    def forward(self, h: torch.Tensor, ctx: Any) -> Delta:
        done, gate = self._experts(h, ctx)
        shared = None
        if self.shared is not None:
            s = self.shared.forward(h, ctx)
            assert s.bias is None and s.parts is None
            shared = s.value
        return Delta(ops.moe_combine(done.y, done.order, done.weights, shared, gate, out_dtype=torch.float32,
                                     identity=done.identity, experts=done.experts, n_real=done.n_real))

    def param_bytes(self) -> int:
        """What a step reads at most: every expert's matrices (a step of few tokens reads only the chosen ones)."""
        return (self.w_gu.numel() + self.w_down.numel()) * self.w_gu.element_size() + self.w_router.numel() * 4
