"""Mamba-2: a state-space recurrence with one decay per head and token, behind a short convolution.

For input ``h`` one product gives ``[z | x | B | C | r]``: gate and values (heads x vdim each), B and C (groups x state
each), a rate per head.  x, B and C together pass a causal convolution over time per channel (``taps`` taps and a bias;
the last tap is the current token's, zeros before a request's first token) and SiLU.  Per head, with
``dt = softplus(r + dt_bias)``,

    S <- exp(-exp(A_log) dt) S + dt B x^T        S: [state, vdim]
    y  = S^T C + D x

where the heads of a group (neighbours) share B and C.  The heads of y side by side are multiplied by ``silu(z)``, divided
in ``norm_groups`` equal parts by each part's own root mean square, multiplied by a gain vector and projected by
``W_o``.

The product's results are float32 and are not rounded before the recurrence; convolution, rates, decays, state and norm
are float32.  A step of single tokens walks the recurrence token by token; prompt portions run in chunks (the same
sums in another order).  A request's state is the heads' matrices and the convolution's last ``taps - 1`` inputs,
float32, in its slot; the mixer holds no pages.

Tensor names (after the part's prefix): ``in``, ``conv``, ``conv.b``, ``dt_bias``, ``A_log``, ``D``, ``norm``, ``o``.
"""

from __future__ import annotations

from .base import Mixer, StateSpec, TensorSpec, register_part

NAMES = ("in", "conv", "conv.b", "dt_bias", "A_log", "D", "norm", "o")


class Mamba2(Mixer):
    state_in_graphs = True       # the kernels read the step's numbers on the device and honour request_active
    kernels_through_ops = True
    takes_state_views = True     # slots may be wider than this mixer's own state

    def __init__(self, hidden_size: int, num_heads: int, value_dim: int, state_dim: int, num_groups: int, taps: int,
                 norm_groups: int, eps: float, names: dict[str, str] | None = None) -> None:
        self.hidden_size = int(hidden_size)
        self.num_heads = int(num_heads)
        self.value_dim = int(value_dim)
        self.state_dim = int(state_dim)
        self.num_groups = int(num_groups)
        self.taps = int(taps)
        self.norm_groups = int(norm_groups)
        self.eps = float(eps)
        self.inner = self.num_heads * self.value_dim
        if self.num_heads % self.num_groups:
            raise ValueError("mamba2: the number of heads must be a multiple of the number of groups")
        if self.inner % self.norm_groups:
            raise ValueError("mamba2: the heads side by side must divide into the norm's groups")
        if self.taps < 1:
            raise ValueError("mamba2: the short convolution needs at least one tap")
        self.channels = self.inner + 2 * self.num_groups * self.state_dim     # what passes the convolution
        self.matrix_floats = self.num_heads * self.state_dim * self.value_dim
        self.names = {key: key for key in NAMES}
        self.names.update(names or {})

    @property
    def plan_key(self):
        return ("ssd.chunks",)

    def plan(self, host, cache):
        """Chunk work lists for a step with prompt portions (one list serves every such layer)."""
        return self.runtime.ops.plan_ssd(host)

    def state_spec(self) -> StateSpec:
        # the heads' matrices, then the convolution's history [taps - 1, channels]
        return StateSpec((self.matrix_floats + (self.taps - 1) * self.channels,), "float32")

    def tensor_specs(self) -> dict[str, TensorSpec]:
        n = self.names
        return {
            n["in"]: TensorSpec((self.inner + self.channels + self.num_heads, self.hidden_size)),
            n["conv"]: TensorSpec((self.channels, self.taps), role="vector"),
            n["conv.b"]: TensorSpec((self.channels,), role="vector"),
            n["dt_bias"]: TensorSpec((self.num_heads,), role="vector"),
            n["A_log"]: TensorSpec((self.num_heads,), role="vector"),
            n["D"]: TensorSpec((self.num_heads,), init="gain", role="vector"),
            n["norm"]: TensorSpec((self.inner,), init="gain", role="vector"),
            n["o"]: TensorSpec((self.hidden_size, self.inner)),
        }

    def bind(self, tensors, runtime) -> None:
        self.runtime = runtime
        ops, n = runtime.ops, self.names
        largest = ops.require_ssd()
        if self.state_dim > largest:
            raise ValueError(f"the state-space kernels take states of up to {largest}, got {self.state_dim}")
        longest = ops.require_recurrent()[1]
        if self.taps > longest:
            raise ValueError(f"the short convolution takes up to {longest} taps, got {self.taps}")
        ops.require_grouped()
        self.w_in = ops.prepare_weight(tensors[n["in"]])
        self.w_out = ops.prepare_weight(tensors[n["o"]])
        self.w_conv = tensors[n["conv"]].float().contiguous()
        self.b_conv, self.dt_bias, self.a_log, self.skip, self.gain = (
            tensors[n[key]].contiguous() for key in ("conv.b", "dt_bias", "A_log", "D", "norm"))

    def forward(self, x, ctx, binding):
        import torch

        rt = self.runtime
        ops = rt.ops
        tokens, f32 = x.shape[0], torch.float32
        inner, channels, heads = self.inner, self.channels, self.num_heads
        proj = rt.workspace.get("mamba2.proj", tokens, self.w_in.shape[0], f32)
        ops.linear(x, self.w_in, None, proj)
        conv = rt.workspace.get("mamba2.conv", tokens, channels, f32)
        ops.short_conv(proj[:, inner:], self.w_conv, binding.state[:, self.matrix_floats:], conv, ctx, bias=self.b_conv)
        mixed = rt.workspace.get("mamba2.y", tokens, inner, f32)
        ops.ssd(conv, (0, inner, inner + self.num_groups * self.state_dim), proj[:, inner + channels:], self.a_log,
                self.dt_bias, self.skip, mixed, binding.state, ctx, heads, self.num_groups, self.state_dim, self.value_dim,
                plan=getattr(ctx, "extras", {}).get(self.plan_key) or None)
        gated = rt.workspace.get("mamba2.gated", tokens, inner, rt.dtype)
        ops.gated_group_norm(mixed, proj, self.gain, self.eps, self.norm_groups, gated)
        update = rt.workspace.get("mixer.update32", tokens, self.hidden_size, f32)
        return ops.linear(gated, self.w_out, None, update)


register_part("mixer", "mamba2", Mamba2, replace=True)
