"""Values that travel between parts instead of tensors.

A part hands the next one a tensor, or one of these: a product whose last additions are left to
its consumer (``Partials``), a product that has already added itself into the residual stream
(``Accumulated``), rows of a norm that its consumer finishes (``NormedInput``).  ``ResidualSink`` is
how a block tells a projection where the residual stream is; ``GateUpWeight`` is a stacked weight
with its layout.  A part that knows none of this gets tensors (``Ops.resolve``, ``materialize``);
the kernels behind ``Ops`` produce and consume them.
"""

from __future__ import annotations

from typing import Any


class Partials:
    """A projection whose last additions are left to the kernel that consumes it.

    ``splits`` > 0: ``data`` holds float32 partial sums [splits, rows, width] of a matrix product
    that was cut along K.  ``splits`` == 0: ``data`` is the product itself [rows, width] in the
    compute dtype.  In both cases ``bias`` (or None) is still to be added.  The consumers
    (residual-add + RMSNorm, rotary + cache write) add everything up in float32, parts in
    ascending split order."""

    def __init__(self, data: Any, splits: int, rows: int, width: int, bias: Any) -> None:
        self.data, self.splits, self.rows, self.width, self.bias = data, splits, rows, width, bias
        self.stride = rows * width      # elements from one partial sum to the next

    @property
    def shape(self) -> tuple[int, int]:
        return (self.rows, self.width)

    @classmethod
    def of_terms(cls, first: Any, second: Any) -> "Partials":
        """Two float32 results [rows, width] of equal shape, each contiguous in a buffer of its own,
        as two terms still to be added: the term at the lower address is the base and the distance
        between the buffers (in elements) is the stride from one term to the next."""
        import torch

        if (first.dtype != torch.float32 or second.dtype != torch.float32 or first.shape != second.shape
                or not first.is_contiguous() or not second.is_contiguous()):
            raise ValueError("of_terms wants two contiguous float32 tensors of one shape")
        low, high = (first, second) if first.data_ptr() < second.data_ptr() else (second, first)
        distance = (high.data_ptr() - low.data_ptr()) // 4
        rows, width = first.shape
        if distance < rows * width:
            raise ValueError("of_terms: the two results overlap")
        terms = cls(low, 2, rows, width, None)
        terms.stride = distance
        terms.terms = (first, second)     # keeps both buffers named for whoever wants to look at them
        return terms


class ResidualSink:
    """The float32 residual stream [T, H] as a target: a projection handed this (``Ops.linear(...,
    residual=sink)``) may add its result into ``tensor`` itself.  ``gain`` is the gain vector of the
    norm that will read the stream next, when that norm can take its input pre-scaled (else None);
    whoever arranges the layers sets it before each projection."""

    def __init__(self, tensor: Any) -> None:
        self.tensor = tensor
        self.gain: Any = None
        self.following_gain: Any = None   # for the last projection of the current layer
        # Whoever arranges the layers may set this when it knows that the kernel after such a
        # projection touches, before its own dependency wait, only what no kernel of the same step
        # writes: the projection then lets that kernel start beside the kernel before itself.
        self.early_trigger = False


class Accumulated:
    """A projection that its own kernel has already added into the float32 residual stream.

    ``sq`` holds, for every token row, the sums of squares of the new residual row per block of 32
    columns ([rows, tiles] float32): a norm that follows needs no pass over the row to know its
    mean square.  ``scaled`` (or None) is bfloat16(new row * ``gain``) for the norm whose gain
    vector ``gain`` is.  A consumer that only wants the sum treats this as "nothing left to add"."""

    def __init__(self, residual: Any, sq: Any, tiles: int, scaled: Any = None, gain: Any = None) -> None:
        self.residual, self.sq, self.tiles, self.scaled, self.gain = residual, sq, tiles, scaled, gain

    @property
    def shape(self) -> tuple[int, ...]:
        return tuple(self.residual.shape)


class NormedInput:
    """RMSNorm of the residual rows, not yet divided by the root mean square: ``accumulated.scaled``
    holds bfloat16(row * gain) and the matrix product that takes this (``Ops.linear``,
    ``Ops.gate_up``) multiplies its result rows by rstd, which it forms from ``accumulated.sq``.
    ``materialize()`` runs the ordinary norm kernel and returns a plain tensor for anyone else."""

    def __init__(self, accumulated: Accumulated, eps: float, materialize: Any) -> None:
        self.accumulated, self.eps, self.materialize = accumulated, eps, materialize

    @property
    def shape(self) -> tuple[int, ...]:
        return tuple(self.accumulated.scaled.shape)


class NormedUpdate:
    """A result ``y`` [T, H] that joins the residual stream RMS-normalised: ``x <- x + gain * y / rms(y)``, the root mean
    square over the whole row with ``eps`` inside; ``centred``: layer-normalised, ``gain * (y - mean(y)) / sqrt(mean((y -
    mean(y))^2) + eps)``.  Whoever reads the stream next applies it in its own kernel, in float32."""

    def __init__(self, y: Any, gain: Any, eps: float, centred: bool = False) -> None:
        self.y, self.gain, self.eps, self.centred = y, gain, float(eps), bool(centred)

    @property
    def shape(self) -> tuple[int, ...]:
        return tuple(self.y.shape)


class WeightedTerms:
    """A weighted sum that has not been taken yet: row t is ``sum_j weights[t, j] * terms[t, j]``, with ``terms`` float32
    [T, count * H] (the ``count`` terms of a row side by side) and ``weights`` float32 [T, count] (None: all ones; then
    ``count`` is given), plus ``extra[t]`` (float32 [T, H], or ``Partials``) if there is one.  Whoever reads the stream next takes it in its
    own kernel, in float32, in ascending order."""

    def __init__(self, terms: Any, weights: Any, count: int = 0, extra: Any = None) -> None:
        self.terms, self.weights, self.count = terms, weights, int(count or weights.shape[1])
        self.extra = extra

    @property
    def shape(self) -> tuple[int, ...]:
        return (int(self.terms.shape[0]), int(self.terms.shape[1]) // self.count)


class PendingNorm:
    """A norm that has not run yet, with what it needs: the stream, the update that still has to join it, gain, eps and
    the number of parts.  Whoever takes this instead of a tensor (``takes_pending_norm``) runs the norm as the first
    step of its own kernel."""

    def __init__(self, residual: Any, update: Any, gain: Any, eps: float, groups: int) -> None:
        self.residual, self.update, self.gain, self.eps, self.groups = residual, update, gain, float(eps), int(groups)

    @property
    def shape(self) -> tuple[int, ...]:
        return tuple(self.residual.shape)


class PendingStream:
    """The stream as a sublayer reads it where no norm stands in front, with the update that still has to join it.
    Whoever takes this instead of a tensor (``takes_pending_stream``) lets it join in its own first kernel."""

    def __init__(self, residual: Any, update: Any) -> None:
        self.residual, self.update = residual, update

    @property
    def shape(self) -> tuple[int, ...]:
        return tuple(self.residual.shape)


class DepthUpdate:
    """A layer's last update together with what the layer's result means for the stream.  With ``row = base + update``
    (``base`` None: the stream itself) the row is kept as state ``place`` of ``history`` [T, states * H] (None: it is
    not kept), and the stream becomes ``sum_(j < place) share[j] * history_j + share[place] * row``, or the row itself
    if ``share`` is None."""

    def __init__(self, update: Any, base: Any, history: Any, place: int, share: Any) -> None:
        self.update, self.base, self.history, self.place, self.share = update, base, history, int(place), share


class StreamUpdate:
    """A sublayer's result ``y`` [T, H] that has not been written to the residual streams yet: every
    stream t becomes ``sum_s mix[s, t] * stream_s + out[t] * y``.  ``mix`` None is the identity and
    ``out`` None all ones, which with one stream is the plain residual add.  Whoever reads the
    streams next (a norm) applies it first, in the same kernel."""

    def __init__(self, y: Any, mix: Any = None, out: Any = None) -> None:
        self.y, self.mix, self.out = y, mix, out

    @property
    def shape(self) -> tuple[int, ...]:
        return tuple(self.y.shape)


class GateUpWeight:
    """Stacked gate and up matrices [2I, H].  ``block`` == I: all gate rows, then all up rows.
    ``block`` < I: rows interleaved in blocks (``block`` gate rows, the matching ``block`` up
    rows, ...), which lets one CTA of the streaming kernel finish SiLU(gate) * up by itself."""

    def __init__(self, weight: Any, inter: int, block: int) -> None:
        self.weight, self.inter, self.block = weight, inter, block
