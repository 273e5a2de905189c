"""A side input of the tokens themselves, read by every layer after its sublayers.

A table that all layers share holds a row of ``layers * dim`` numbers per token id; layer ``i`` reads the part
``e = row[i * dim : (i + 1) * dim]`` of each token.  With the residual stream x (not normalised),

    g = gelu_tanh(W_gate x) * e;    y = W_proj g;    x <- x + gain * y / rms(y)

with the root mean square over the whole row, whatever norm the model uses elsewhere.  The rows that enter the two
products are of the compute dtype, their results float32; activation, norm and sum are float32.  The last line is left
to the norm that reads the stream next (``NormedUpdate``).

Tensor names (after the part's prefix): ``gate`` [dim, width], ``proj`` [width, dim], ``norm`` [width]; ``table`` is the
full name of the shared table.
"""

from __future__ import annotations

from ..lazy import NormedUpdate
from .base import FeedForward, TensorSpec, register_part


class TokenSide(FeedForward):
    kernels_through_ops = True

    def __init__(self, hidden_size: int, dim: int, index: int, layers: int, vocab_size: int, eps: float, table: str) -> None:
        if not 0 <= index < layers:
            raise ValueError(f"token side: layer {index} of {layers}")
        self.hidden_size = int(hidden_size)
        self.dim = int(dim)
        self.index = int(index)
        self.layers = int(layers)
        self.vocab_size = int(vocab_size)
        self.eps = float(eps)
        self.table_name = str(table)

    def tensor_specs(self) -> dict[str, TensorSpec]:
        return {"gate": TensorSpec((self.dim, self.hidden_size)), "proj": TensorSpec((self.hidden_size, self.dim)),
                "norm": TensorSpec((self.hidden_size,), init="gain", role="vector")}

    def shared_tensor_specs(self) -> dict[str, TensorSpec]:
        return {self.table_name: TensorSpec((self.vocab_size, self.layers * self.dim))}

    def bind(self, tensors, runtime) -> None:
        self.runtime = runtime
        runtime.ops.require_grouped()
        self.w_gate = runtime.ops.prepare_weight(tensors["gate"])
        self.w_proj = runtime.ops.prepare_weight(tensors["proj"])
        self.gain = tensors["norm"].contiguous()

    def bind_shared(self, tensors) -> None:
        self.table = tensors[self.table_name]

    def forward_stream(self, residual, update, ctx):
        """``residual`` is the float32 stream [T, H], ``update`` what still has to join it (it does here)."""
        import torch

        rt = self.runtime
        ops = rt.ops
        tokens = residual.shape[0]
        rows = rt.workspace.get("norm.out", tokens, self.hidden_size, rt.dtype)
        ops.group_norm(residual, update, None, 0.0, 1, rows)
        gate = rt.workspace.get("side.gate", tokens, self.dim, torch.float32)
        ops.linear(rows, self.w_gate, None, gate)
        gated = rt.workspace.get("side.gated", tokens, self.dim, rt.dtype)
        ops.side_gate(gate, ctx.token_ids, self.table, self.index * self.dim, gated)
        result = rt.workspace.get("side.update32", tokens, self.hidden_size, torch.float32)
        return NormedUpdate(ops.linear(gated, self.w_proj, None, result), self.gain, self.eps)


register_part("feed_forward", "token_side", TokenSide, replace=True)
