"""Mixture of experts as a feed-forward part: a router picks ``top_k`` of ``num_experts`` small gated
feed-forwards per token; an optional shared expert runs for every token.

    z = router x                      (32-bit logits; the router matrix is kept in 32-bit)
    s = sigmoid(z)  or  softmax(z)    (``score``; ``router_bias``: z has a bias ``[experts]``, 32-bit)
             or ``score="softmax_chosen"``: s = z, and the weights are the softmax over the chosen logits alone
    chosen = the top_k largest s; weights = their s, divided by their sum if ``renormalize``
             ``choice_correction``: the choice goes by ``s + c`` with a tensor ``c [experts]``, the weights stay
             the chosen experts' ``s``; ``group_count`` / ``group_keep``: the experts form ``group_count`` equal
             groups of neighbours, a group's score is its largest choice score, and only experts of the
             ``group_keep`` best groups can be chosen; ``weight_scale`` multiplies the weights
    y = sum over chosen e of  expert_e(w_e * x)        (``weight_on="input"``)
                         or   w_e * expert_e(x)        (``weight_on="output"``)
    y += sigmoid(g . x) * shared(x)   (``shared`` given; ``shared_gate`` False: plain sum)

    expert(a) = down(silu(gate a) * (up a)), no biases; or with ``join = (alpha, limit, shift)``
                down(g * sigmoid(alpha g) * (u + shift)), g = min(gate a, limit), u = clamp(up a, -limit, limit);
                or with ``activation="squared_relu"``  down(max(up a, 0)^2)  (no gate)

``identity_experts``: that many experts without tensors stand behind the others in the router (whose rows, bias and
correction then count both kinds); their output is their input ``a`` itself.  They take no part in the products: the
kernel that sums a token's experts adds the token's own row for them.

The experts' matrices are stacked ``[E, 2F, K]`` (gate rows, then up rows) and ``[E, K, F]``; the
(token, expert) pairs are grouped by expert on the device and the two products run as grouped
products over that order, so the launches depend on the batch's shape only.  The shared expert is any
registered feed-forward part.
"""
from __future__ import annotations

import torch

from .. import kernels as K
from ..config.model_spec import PartSpec
from .base import FEED_FORWARDS, FeedForward, WeightSlot


class RoutedExperts(FeedForward):
    DEFAULT_TENSOR_NAMES = {
        "router": "router", "router_bias": "router.b", "shared_gate": "shared_gate", "correction": "correction",
        # expert tensors: formatted with the expert's index
        "gate": "experts.{index}.gate_proj.weight", "up": "experts.{index}.up_proj.weight",
        "down": "experts.{index}.down_proj.weight",
    }

    def __init__(self, *, hidden_size: int, num_experts: int, top_k: int, expert_size: int, name: str,
                 score: str = "sigmoid", renormalize: bool = False, weight_on: str = "input",
                 shared: PartSpec | None = None, shared_gate: bool = False, weight_scale: float = 1.0,
                 choice_correction: bool = False, group_count: int = 1, group_keep: int = 1,
                 router_bias: bool = False, join: tuple | None = None, activation: str | None = None,
                 identity_experts: int = 0,
                 tensor_names: dict | None = None, dtype: torch.dtype, device: torch.device) -> None:
        self.hidden_size, self.num_experts = int(hidden_size), int(num_experts)
        self.top_k, self.expert_size = int(top_k), int(expert_size)
        self.identity_experts = int(identity_experts)
        if self.num_experts <= 0 or self.identity_experts < 0:
            raise ValueError(f"a mixture has experts, got {num_experts} and {identity_experts} identity experts")
        self.routed = self.num_experts + self.identity_experts         # what the router chooses among
        if not 0 < self.top_k <= self.routed:
            raise ValueError(f"top_k {top_k} must lie in [1, {self.routed}] (num_experts + identity_experts)")
        if score not in ("sigmoid", "softmax", "softmax_chosen"):
            raise ValueError(f"unknown router score {score!r}")
        if weight_on not in ("input", "output"):
            raise ValueError(f"weight_on must be 'input' or 'output', got {weight_on!r}")
        self.score, self.renormalize, self.weight_on = score, bool(renormalize), weight_on
        self.weight_scale, self.group_count, self.group_keep = float(weight_scale), int(group_count), int(group_keep)
        if (self.group_count <= 0 or self.routed % self.group_count or not 0 < self.group_keep <= self.group_count
                or self.group_keep * (self.routed // self.group_count) < self.top_k):
            raise ValueError(f"{group_keep} of {group_count} equal groups of {self.routed} experts must hold top_k {top_k}")
        if join is not None and (len(join) != 3 or not join[1] > 0):
            raise ValueError(f"join is (alpha, limit, shift) with a positive limit, got {join!r}")
        self.join = None if join is None else tuple(float(v) for v in join)
        if activation not in (None, "squared_relu") or (activation and join is not None):
            raise ValueError(f"an expert's activation is None (gated units) or 'squared_relu' (no gate), got {activation!r}")
        self.activation = activation
        self.name = name
        self.tensor_names = dict(self.DEFAULT_TENSOR_NAMES)
        self.tensor_names.update(tensor_names or {})
        experts, ff, hidden = self.num_experts, self.expert_size, self.hidden_size
        self.router_weight = torch.empty(self.routed, hidden, dtype=torch.float32, device=device)
        self.correction = torch.empty(self.routed, dtype=torch.float32, device=device) if choice_correction else None
        self.router_bias = torch.empty(self.routed, dtype=torch.float32, device=device) if router_bias else None
        # gate rows, then up rows; without a gate the up rows alone
        self.gate_up_weight = torch.empty(experts, (1 if self.activation else 2) * ff, hidden, dtype=dtype, device=device)
        self.down_weight = torch.empty(experts, hidden, ff, dtype=dtype, device=device)
        self.shared = None if shared is None else FEED_FORWARDS.build(shared, dtype=dtype, device=device)
        if shared_gate and self.shared is None:
            raise ValueError("a shared gate needs a shared expert")
        self.shared_gate_weight = (torch.empty(1, hidden, dtype=torch.float32, device=device)
                                   if shared_gate else None)

    @property
    def graph_safe(self) -> bool:
        return self.shared is None or self.shared.graph_safe

    def _tensor(self, key: str, index: int | None = None) -> str:
        return f"{self.name}.{self.tensor_names[key].format(index=index)}"

    def weight_slots(self) -> list[WeightSlot]:
        ff = self.expert_size
        slots = [WeightSlot(self._tensor("router"), self.router_weight)]
        if self.router_bias is not None:
            slots.append(WeightSlot(self._tensor("router_bias"), self.router_bias, init="zeros"))
        if self.correction is not None:
            slots.append(WeightSlot(self._tensor("correction"), self.correction, init="zeros"))
        for e in range(self.num_experts):
            if self.activation is None:
                slots.append(WeightSlot(self._tensor("gate", e), self.gate_up_weight[e, :ff]))
            slots += [
                WeightSlot(self._tensor("up", e), self.gate_up_weight[e, -ff:]),
                WeightSlot(self._tensor("down", e), self.down_weight[e]),
            ]
        if self.shared is not None:
            slots += self.shared.weight_slots()
        if self.shared_gate_weight is not None:
            slots.append(WeightSlot(self._tensor("shared_gate"), self.shared_gate_weight))
        return slots

    def ignorable_tensor_names(self) -> list[str]:
        return [] if self.shared is None else self.shared.ignorable_tensor_names()

    def finalize_weights(self) -> None:
        if self.shared is not None:
            self.shared.finalize_weights()

    def prepare(self, x: torch.Tensor, ctx):
        """The router and the grouping of the pairs by expert, ahead of ``forward``: a block that has other
        work to launch in between (its mixer) calls this first, so that what the host must know of the
        grouping has arrived by the time ``forward`` asks for it."""
        routed = K.moe_route(x, self.router_weight, self.top_k, score=self.score,
                             renormalize=self.renormalize, gate_rows=self.shared_gate_weight,
                             correction=self.correction, group_count=self.group_count, group_keep=self.group_keep,
                             weight_scale=self.weight_scale, bias=self.router_bias)
        grouping = None
        if K.moe_path(x, x.shape[0] * self.top_k, self.expert_size) == "library":
            grouping = K.moe_group(routed[0], self.num_experts, for_library=True, identity=self.identity_experts)
        return routed, grouping

    def _expert_rows(self, x: torch.Tensor, ctx, prepared):
        (ids, weights, gates), grouping = prepared if prepared is not None else self.prepare(x, ctx)
        return gates, K.moe_experts(x, ids, weights, self.gate_up_weight, self.down_weight,
                                    weight_on_input=self.weight_on == "input", grouping=grouping, join=self.join,
                                    activation=self.activation, identity=self.identity_experts)

    def forward_rows(self, x: torch.Tensor, ctx):
        """The chosen experts' rows, for a block whose next norm weights and sums them into the stream (None: a
        shared expert wants a sum of its own)."""
        return None if self.shared is not None else self._expert_rows(x, ctx, None)[1]

    def forward(self, x: torch.Tensor, ctx, prepared=None) -> torch.Tensor:
        gates, pairs = self._expert_rows(x, ctx, prepared)
        shared = None if self.shared is None else self.shared.forward(x, ctx)
        return K.moe_combine(pairs, x.shape[0], self.top_k, shared, gates)


FEED_FORWARDS.register("routed_experts", RoutedExperts)

__all__ = ["RoutedExperts"]
