"""Hyper-connections: a sublayer reads a weighted sum of several residual streams and writes
every stream back as a mix of the old streams plus its own result.

For one sublayer with result ``y`` and tensors ``in`` [S], ``out`` [S], ``mix`` [S, S] (indexed
[from, to]):  ``u = sum_s in[s] * x_s`` is what the sublayer's norm reads, and afterwards, all
streams at once from the old ones, ``x_t <- sum_s mix[s, t] * x_s + out[t] * y``.  The write is not
done here: it travels as a ``StreamUpdate`` to whoever reads the streams next, whose kernel applies
it in float32 together with its own read and norm.
"""

from __future__ import annotations

from ..lazy import DepthUpdate, StreamUpdate
from .base import Connection, TensorSpec, register_part


class HyperConnection(Connection):
    def __init__(self, streams: int) -> None:
        if streams < 1:
            raise ValueError("a hyper-connection needs at least one stream")
        self.streams = int(streams)

    def tensor_specs(self) -> dict[str, TensorSpec]:
        s = self.streams
        return {
            "in": TensorSpec((s,), init="gain", role="vector"),
            "out": TensorSpec((s,), init="gain", role="vector"),
            "mix": TensorSpec((s, s), init="eye", role="vector"),
        }

    def bind(self, tensors, runtime) -> None:
        self.runtime = runtime
        self.w_in = tensors["in"].contiguous()
        self.w_out = tensors["out"].contiguous()
        self.w_mix = tensors["mix"].contiguous()

    def read_weights(self):
        return self.w_in

    def pending(self, y):
        return StreamUpdate(y, self.w_mix, self.w_out)


register_part("connection", "hyper", HyperConnection, replace=True)


class DepthAverage(Connection):
    """What goes on from layer ``index`` is a weighted sum of everything there has been so far: with X_0 the stream as it
    entered the first layer and X_(i + 1) layer i's own result, ``x <- sum_(j <= index + 1) share[j] * X_j``.  Every
    token's states lie side by side in one float32 buffer of the step ([T, states * H], ``states`` = layers + 1); the
    sum itself travels as a ``DepthUpdate`` to whoever reads the stream next.  ``name``: the tensor's name after the
    part's prefix."""

    def __init__(self, hidden_size: int, index: int, states: int, name: str = "weight") -> None:
        if not 0 <= index < states - 1:
            raise ValueError(f"depth average: layer {index} with {states} states")
        self.hidden_size = int(hidden_size)
        self.index = int(index)
        self.states = int(states)
        self.name = str(name)

    def tensor_specs(self) -> dict[str, TensorSpec]:
        return {self.name: TensorSpec((self.index + 2,), init="mean", role="vector")}

    def bind(self, tensors, runtime) -> None:
        self.runtime = runtime
        self.share = tensors[self.name].contiguous()

    def history(self, tokens: int):
        import torch

        return self.runtime.workspace.get("depth.history", tokens, self.states * self.hidden_size, torch.float32)

    def entering(self, update, history):
        """What is pending as the layer begins: before the first one, the stream itself becomes state 0."""
        return DepthUpdate(update, None, history, 0, None) if self.index == 0 else update

    def midway(self, update, history):
        """The layer's state after its first of two sublayers: kept where its result will be."""
        return DepthUpdate(update, None, history, self.index + 1, None)

    def leaving(self, update, history, continues: bool):
        """The layer's result (``continues``: its state so far is the one that ``midway`` kept) and the average."""
        place = self.index + 1
        base = history[:, place * self.hidden_size:(place + 1) * self.hidden_size] if continues else None
        return DepthUpdate(update, base, history, place, self.share)


register_part("connection", "depth_average", DepthAverage, replace=True)
