"""Routed experts: every token runs through the ``top`` of ``experts`` small SwiGLU feed-forwards.

Router logits ``z = W_router h`` in float32; scores ``s = softmax(z)`` over all experts; the
experts with the largest ``s + correction`` are chosen (``correction`` is a stored vector that only
steers the choice); the mixing weights are the chosen experts' ``s`` themselves, renormalised to
sum 1 only if ``renormalize`` says so.  The result is the weighted sum of
``W_down (silu(W_gate h) * (W_up h))`` over the chosen experts, added up in float32 in the order
the experts were chosen.

The experts' matrices are stacked into three tensors at load time ([E, F, H], [E, F, H], [E, H, F];
for bfloat16 with sizes the tensor-core kernels take, gate and up as one [E, 2F, H] with their rows
interleaved in blocks of 16);
Two options: ``router_bias`` adds a stored vector to the logits, and ``score="chosen_softmax"`` chooses the
experts with the largest logits and weights them by the softmax over the chosen logits alone.

``score="sigmoid"`` makes the scores sigmoids of the logits.  ``groups`` = (count, keep): the experts form ``count``
equal groups of neighbours, a group's score is the sum of its two largest choice scores (score + correction), and only
experts of the ``keep`` best groups can be chosen.  ``norm_floor`` is added to the sum that ``renormalize`` divides by.  ``defer_sum``: the weighted sum over the chosen
experts is left to whoever reads the stream next (``WeightedTerms``; for norms that take it).

``activation`` (limit, slope, shift) makes the experts ``W_down (g * sigmoid(slope * g) * (u + shift))`` with ``g =
min(W_gate h, limit)`` and ``u = clamp(W_up h, -limit, limit)`` (None: SiLU(gate) * up).  ``weight_inputs``: a weight
multiplies its expert's INPUT, not its output: the result is the plain sum of ``expert(weight * h)``; since gate and up
are linear the kernels scale their results.  ``shared``: a feed-forward part that every token runs through and whose
result is added (with ``defer_sum``, as one more term).

The kernels group the (token, expert) pairs by expert on the device and never tell the host how
many tokens an expert got, so a step is one fixed sequence of launches.
"""

from __future__ import annotations

from ..config.spec import PartSpec
from ..lazy import WeightedTerms
from .base import FeedForward, TensorSpec, build_part, register_part


class RoutedExperts(FeedForward):
    def __init__(self, hidden_size: int, intermediate_size: int, num_experts: int, top: int,
                 correction: bool = True, renormalize: bool = False,
                 names: dict[str, str] | None = None, router_bias: bool = False, score: str = "softmax",
                 groups: tuple[int, int] = (1, 1), norm_floor: float = 0.0, defer_sum: bool = False,
                 activation: tuple[float, float, float] | None = None, weight_inputs: bool = False,
                 shared: PartSpec | None = None) -> None:
        if not 1 <= top <= num_experts:
            raise ValueError("top must lie in 1..num_experts")
        self.hidden_size = int(hidden_size)
        self.intermediate_size = int(intermediate_size)
        self.num_experts = int(num_experts)
        self.top = int(top)
        self.correction = bool(correction)
        self.renormalize = bool(renormalize)
        self.router_bias = bool(router_bias)
        if score not in ("softmax", "chosen_softmax", "sigmoid"):
            raise ValueError(f"routed experts: score {score!r} is not built (known: softmax, chosen_softmax, sigmoid)")
        count, keep = (int(number) for number in groups)
        if count < 1 or num_experts % count or not 1 <= keep <= count or top > num_experts // count * keep:
            raise ValueError(f"routed experts: {keep} of {count} groups of {num_experts} experts cannot give {top} choices")
        if count > 1 and score == "chosen_softmax":
            raise ValueError("routed experts: groups are built for a choice among scores, not among logits")
        self.groups = (count, keep)
        self.norm_floor = float(norm_floor)
        self.defer_sum = bool(defer_sum)
        self.activation = tuple(float(number) for number in activation) if activation is not None else None
        self.weight_inputs = bool(weight_inputs)
        self.shared = build_part("feed_forward", shared) if shared is not None else None
        self.shared_prefix = shared.prefix if shared is not None else ""
        if self.shared is not None and not self.defer_sum:
            raise ValueError("routed experts: a shared expert's result joins a sum that is deferred")
        if score == "chosen_softmax" and correction:
            raise ValueError("routed experts: a correction steers a choice among softmax scores, not among logits")
        self.score = score
        self.names = dict(router="router", correction="correction", expert="e{}.", gate="gate", up="up", down="down",
                          router_bias="router.b")
        self.names.update(names or {})

    def _expert(self, index: int, which: str) -> str:
        return self.names["expert"].format(index) + self.names[which]

    def tensor_specs(self) -> dict[str, TensorSpec]:
        specs = {self.names["router"]: TensorSpec((self.num_experts, self.hidden_size), role="vector")}
        if self.correction:
            specs[self.names["correction"]] = TensorSpec((self.num_experts,), role="vector")
        if self.router_bias:
            specs[self.names["router_bias"]] = TensorSpec((self.num_experts,), role="vector")
        for e in range(self.num_experts):
            specs[self._expert(e, "gate")] = TensorSpec((self.intermediate_size, self.hidden_size))
            specs[self._expert(e, "up")] = TensorSpec((self.intermediate_size, self.hidden_size))
            specs[self._expert(e, "down")] = TensorSpec((self.hidden_size, self.intermediate_size))
        if self.shared is not None:
            specs.update({self.shared_prefix + name: spec for name, spec in self.shared.tensor_specs().items()})
        return specs

    def subparts(self):
        return (self.shared,) if self.shared is not None else ()

    def bind(self, tensors, runtime) -> None:
        import torch

        self.runtime = runtime
        self.router = tensors[self.names["router"]].contiguous()
        self.bias = tensors[self.names["correction"]].contiguous() if self.correction else None
        self.logit_bias = tensors[self.names["router_bias"]].contiguous() if self.router_bias else None
        stack = lambda which: runtime.ops.prepare_weight(  # noqa: E731
            torch.stack([tensors[self._expert(e, which)] for e in range(self.num_experts)]))
        self.w_gate, self.w_up, self.w_down = stack("gate"), stack("up"), stack("down")
        if runtime.ops.moe_interleaves(self.hidden_size, self.intermediate_size):
            # one tensor for gate and up, rows interleaved in blocks of 16: the tensor-core kernels
            # finish SiLU(gate) * up in their epilogue
            self.w_gate, self.w_up = runtime.ops.interleave_gate_up(self.w_gate, self.w_up), None
        if self.shared is not None:
            self.shared.bind({name: tensors[self.shared_prefix + name] for name in self.shared.tensor_specs()}, runtime)

    def forward(self, x, ctx):
        import torch

        rt = self.runtime
        update = None
        if not self.defer_sum:
            update = rt.workspace.get("feed_forward.update32", x.shape[0], self.hidden_size, torch.float32)
        result = rt.ops.routed_experts(x, self.router, self.bias, self.w_gate, self.w_up, self.w_down,
                                       self.top, self.renormalize, update, rt.workspace, router_bias=self.logit_bias,
                                       chosen_softmax=self.score == "chosen_softmax",
                                       sigmoid=self.score == "sigmoid", groups=self.groups, norm_floor=self.norm_floor,
                                       defer=self.defer_sum, activation=self.activation, weight_inputs=self.weight_inputs)
        if self.shared is None:
            return result
        return WeightedTerms(result.terms, result.weights, result.count, extra=self.shared.forward(x, ctx))


register_part("feed_forward", "routed_experts", RoutedExperts, replace=True)
