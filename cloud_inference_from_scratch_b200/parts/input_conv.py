"""A mixer whose input first passes a causal convolution over time, added to itself.

What the inner mixer reads, h (the layer's normalised rows), becomes ``h + conv(h)`` with a filter per channel,
``conv(h)_t = sum_j w[:, j] * h_(t - taps + 1 + j)``: the last tap is the current token's and rows before a request's
first token are zero.  h of the last ``taps - 1`` tokens is part of every request's state, float32, whatever the inner
mixer keeps; it lies behind the inner mixer's own state in the request's slot.

The norm in front does not run on its own: this part takes it not yet begun (``PendingNorm``) and its kernels go from
the residual add through norm and convolution to the rounded rows.  Tensor name (after the part's prefix): ``weight``
([width, taps]) or what ``name`` says; the inner mixer's tensors lie under its own prefix.
"""

from __future__ import annotations

import math

from ..config.spec import PartSpec
from ..lazy import PendingNorm
from .base import Mixer, StateSpec, TensorSpec, build_part, register_part


class InputState(Mixer):
    """A mixer around an inner one that changes what the inner mixer reads with the help of earlier tokens' rows, which
    it keeps as per-request state of ``kept_floats`` float32 numbers behind the inner mixer's own in the request's slot.
    Where the inner mixer keeps its pages is the inner mixer's business."""

    def __init__(self, inner: PartSpec, kept_floats: int) -> None:
        self.inner = build_part("mixer", inner)
        self.inner_prefix = inner.prefix
        kept = self.inner.state_spec()
        if kept is not None and not getattr(self.inner, "takes_state_views", False):
            raise ValueError(f"{type(self).__name__}: mixer {inner.kind!r} does not take its state as a view of a wider slot")
        if kept is not None and kept.dtype != "float32":
            raise ValueError(f"{type(self).__name__}: the inner state must be float32")
        # rounded up to whole 16-byte pieces, so that both parts of a slot are aligned
        self.inner_floats = -(-math.prod(kept.shape) // 4) * 4 if kept is not None else 0
        self.kept_floats = int(kept_floats)
        self.state_in_graphs = kept is None or self.inner.state_in_graphs
        self.kernels_through_ops = self.inner.kernels_through_ops

    def subparts(self):
        return (self.inner,)

    def cache_spec(self):
        return self.inner.cache_spec()

    def state_spec(self):
        floats = self.inner_floats + -(-self.kept_floats // 4) * 4
        return StateSpec((floats,), "float32") if floats else None

    def own_tensor_specs(self) -> dict[str, TensorSpec]:
        raise NotImplementedError

    def tensor_specs(self) -> dict[str, TensorSpec]:
        specs = {self.inner_prefix + name: spec for name, spec in self.inner.tensor_specs().items()}
        specs.update(self.own_tensor_specs())
        return specs

    def bind(self, tensors, runtime) -> None:
        self.runtime = runtime
        self.inner.bind({name: tensors[self.inner_prefix + name] for name in self.inner.tensor_specs()}, runtime)

    def kept(self, binding):
        """The view of every slot's part that this wrapper keeps (None: nothing)."""
        return binding.state[:, self.inner_floats:] if self.kept_floats else None

    def run_inner(self, x, ctx, binding):
        from dataclasses import replace

        inner = binding.state[:, : self.inner_floats] if self.inner_floats else None
        return self.inner.forward(x, ctx, replace(binding, state=inner))


class InputConvolution(InputState):
    takes_pending_norm = True

    def __init__(self, hidden_size: int, taps: int, inner: PartSpec, name: str = "weight") -> None:
        if taps < 1:
            raise ValueError("the input convolution needs at least one tap")
        self.hidden_size = int(hidden_size)
        self.taps = int(taps)
        self.name = str(name)
        super().__init__(inner, (self.taps - 1) * self.hidden_size)

    def own_tensor_specs(self) -> dict[str, TensorSpec]:
        return {self.name: TensorSpec((self.hidden_size, self.taps), role="vector")}

    def bind(self, tensors, runtime) -> None:
        longest = runtime.ops.require_grouped()
        if self.taps > longest:
            raise ValueError(f"the input convolution takes up to {longest} taps, got {self.taps}")
        super().bind(tensors, runtime)
        self.weight = tensors[self.name].float().contiguous()

    def forward(self, x, ctx, binding):
        if not isinstance(x, PendingNorm):
            raise TypeError("the input convolution begins with the norm in front of it; use a norm that can be handed on")
        rt = self.runtime
        out = rt.workspace.get("norm.out", x.shape[0], self.hidden_size, rt.dtype)
        rt.ops.group_norm_conv(x.residual, x.update, x.gain, x.eps, x.groups, self.weight, self.kept(binding), out, ctx)
        return self.run_inner(out, ctx, binding)


register_part("mixer", "input_conv", InputConvolution, replace=True)
