"""A mixer whose input is first moved towards the token before it, element by element.

What the inner mixer reads, h (the layer's rows of the stream), becomes ``h_t + (h_(t - 1) - h_t) * share`` with a stored
share per element; before a request's first token there are zeros.  h of the last token, as it was before the move, is
part of every request's state, float32, whatever the inner mixer keeps.

The stream comes with the update that still has to join it (``PendingStream``): one kernel goes from that update to the
rounded, moved rows.  Tensor name (after the part's prefix): ``weight`` ([width]) or what ``name`` says; the inner
mixer's tensors lie under its own prefix.
"""

from __future__ import annotations

from ..config.spec import PartSpec
from ..lazy import PendingStream
from .base import TensorSpec, register_part
from .input_conv import InputState


class TokenShift(InputState):
    takes_pending_stream = True

    def __init__(self, hidden_size: int, inner: PartSpec, name: str = "weight") -> None:
        self.hidden_size = int(hidden_size)
        self.name = str(name)
        super().__init__(inner, self.hidden_size)

    def own_tensor_specs(self) -> dict[str, TensorSpec]:
        return {self.name: TensorSpec((self.hidden_size,), role="vector")}

    def bind(self, tensors, runtime) -> None:
        widest = runtime.ops.require_stream_step()
        if self.hidden_size > widest:
            raise ValueError(f"the token shift takes rows of up to {widest} elements, got {self.hidden_size}")
        super().bind(tensors, runtime)
        self.share = tensors[self.name].float().contiguous()

    def forward(self, x, ctx, binding):
        if not isinstance(x, PendingStream):
            raise TypeError("the token shift reads the stream with its pending update; use a block that hands it on")
        rt = self.runtime
        out = rt.workspace.get("norm.out", x.shape[0], self.hidden_size, rt.dtype)
        rt.ops.advance(x.residual, x.update, out, shift=(self.share, self.kept(binding)), ctx=ctx)
        return self.run_inner(out, ctx, binding)


register_part("mixer", "token_shift", TokenShift, replace=True)
