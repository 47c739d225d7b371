"""State-space mixer with one scalar decay per head and token (Mamba-2): a recurrence whose state is one
[state][vdim] matrix per head and request.

Per token, with h the mixer's input, one projection gives z | x | B | C | dt (inner, inner, groups x state, groups x
state, heads numbers, inner = heads x vdim).  x, B and C pass a short causal convolution over time per channel with
a bias, and silu.  Per head (head j reads group j // (heads/groups) of B and C), with dt = softplus(dt + dt_bias),

    S <- exp(-exp(A_log) dt) S + dt B x^T;     y = S^T C + D x

and the output is W_o of  weight * unit(y * silu(z)),  the root mean square taken over each of ``norm_groups`` equal
runs of the inner channels on its own.  S and the convolution's last inputs live in the request's state slot (fp32,
zero at admission), so a sequence may be cut into steps anywhere.  The projection leaves its product in fp32; in
bfloat16 mode the convolved rows are rounded, everything else that enters the recurrence is computed in 32-bit.
"""
from __future__ import annotations

import torch

from ..kernels import mixing, ops
from ..kernels import state_space as kernels
from ..weights.loader import TensorDecl
from .base import FixedState, Mixer, Precision, register_mixer


@register_mixer("state_space")
class StateSpace(Mixer):
    """params: hidden_size, num_heads, vdim, state, groups (1), taps, norm_groups (1), eps (of the output's norm).
    tensors: in [2 inner + 2 groups state + heads][H]; conv [inner + 2 groups state][taps], conv_bias; dt_bias,
    a_log, skip [heads]; norm [inner]; o [H][inner]."""
    graph_safe = True

    def __init__(self, spec):
        super().__init__(spec)
        p = self.params
        self.hidden = int(p["hidden_size"])
        self.n_heads = int(p["num_heads"])
        self.vdim = int(p["vdim"])
        self.state = int(p["state"])
        self.groups = int(p.get("groups", 1))
        self.taps_len = int(p["taps"])
        self.norm_groups = int(p.get("norm_groups", 1))
        self.eps = float(p["eps"])
        if min(self.n_heads, self.vdim, self.state, self.groups, self.norm_groups) <= 0:
            raise ValueError("state space: heads, vdim, state, groups and norm_groups must be positive")
        if self.n_heads % self.groups:
            raise ValueError(f"state space: {self.n_heads} heads do not share {self.groups} groups evenly")
        if self.inner % self.norm_groups:
            raise ValueError(f"state space: {self.inner} channels are not {self.norm_groups} equal norm groups")
        if self.taps_len < 1:
            raise ValueError("the short convolution needs at least one tap")
        self.w_in = self.w_o = self.taps = self.conv_bias = self.dt_bias = self.a_log = self.skip = self.norm = None

    @property
    def inner(self) -> int:
        return self.n_heads * self.vdim

    @property
    def channels(self) -> int:
        """Channels that pass the convolution: x | B | C."""
        return self.inner + 2 * self.groups * self.state

    @property
    def _rows(self) -> int:
        return self.inner + self.channels + self.n_heads

    def declare(self):
        n, H = self.names, self.hidden
        return {n["in"]: TensorDecl((self._rows, H)), n["conv"]: TensorDecl((self.channels, self.taps_len), "taps"),
                n["conv_bias"]: TensorDecl((self.channels,), "bias"), n["dt_bias"]: TensorDecl((self.n_heads,), "bias"),
                n["a_log"]: TensorDecl((self.n_heads,), "bias"), n["skip"]: TensorDecl((self.n_heads,), "norm"),
                n["norm"]: TensorDecl((self.inner,), "norm"), n["o"]: TensorDecl((H, self.inner))}

    def bind(self, get, precision: Precision, device):
        n = self.names
        rows = get(n["in"])
        pad = -self._rows % 8                       # (a row count the products' tiles like)
        if pad:
            rows = torch.cat([rows, rows.new_zeros((pad, rows.shape[1]))], dim=0)
        self.w_in = precision.matrix(rows, device)
        self.w_o = precision.matrix(get(n["o"]), device)
        self.taps = precision.vector(get(n["conv"]), device)
        for name, tensor in (("conv_bias", "conv_bias"), ("dt_bias", "dt_bias"), ("a_log", "a_log"), ("skip", "skip"),
                             ("norm", "norm")):
            setattr(self, name, precision.vector(get(n[tensor]), device))

    def weight_bytes(self):
        return (self.w_in.numel() * self.w_in.element_size() + self.w_o.numel() * self.w_o.element_size()
                + (self.taps.numel() + self.norm.numel()) * 4)

    def flops_per_token(self):
        # the products, and per head two passes over the [state][vdim] state (decay and write, read-out)
        return 2.0 * (self.w_in.numel() + self.w_o.numel()) + 4.0 * self.n_heads * self.state * self.vdim

    @property
    def _matrix_entries(self) -> int:
        # (the convolution's rows behind the matrices start on a 16-byte border)
        return -(-self.n_heads * self.state * self.vdim // 4) * 4

    def state_spec(self):
        size = self._matrix_entries + (self.taps_len - 1) * self.channels
        return FixedState((-(-size // 4) * 4,))

    def forward(self, ctx, h, cache):
        act = ctx.precision.act_dtype
        p = ops.linear(h, self.w_in, torch.float32)
        rolling = None
        if self.taps_len > 1:
            rows = (self.taps_len - 1) * self.channels
            at = self._matrix_entries
            rolling = cache.state[:, at:at + rows].unflatten(1, (self.taps_len - 1, self.channels))
        u = mixing.causal_conv(p, self.taps, rolling, ctx.batch, col0=self.inner, bias=self.conv_bias, silu=True,
                               out_dtype=act)
        y = kernels.state_space(u, p, self.inner + self.channels, self.dt_bias, self.a_log, self.skip, cache.state,
                                ctx.batch, self.n_heads, self.groups, self.state, self.vdim)
        z = kernels.gate_group_norm(y, p, 0, self.norm, self.norm_groups, self.eps, act)
        return ops.linear(z, self.w_o, torch.float32)
