"""minGRU mixer: a gated average over time with one number of state per channel, whose gates read only the
current token.

Per token, with h the mixer's input:  z = sigmoid(W_z h + b_z), u = W_x h + b_x; the candidate is u + 1/2 where
u >= 0 and sigmoid(u) below; channel by channel

    S <- (1 - z) S + z candidate

and the output is ``W_o (S * silu(W_g h))``.  S lives in the request's state slot (fp32, zero at admission), so
a sequence may be cut into steps anywhere.  One fused projection z|x|gate leaves its product in fp32; biases,
gates, candidate and recurrence are computed in 32-bit in both precisions.
"""
from __future__ import annotations

import torch

from ..kernels import mixing, ops
from ..weights.loader import TensorDecl
from .base import FixedState, Mixer, Precision, register_mixer


@register_mixer("mingru")
class MinGRU(Mixer):
    """params: hidden_size, width.  tensors: z, x, g [width][H]; z_b, x_b [width]; o [H][width]."""
    graph_safe = True
    takes_deferred_norm = True
    adds_residual = True

    def __init__(self, spec):
        super().__init__(spec)
        self.hidden = int(self.params["hidden_size"])
        self.width = int(self.params["width"])
        if self.width <= 0:
            raise ValueError("minGRU: width must be positive")
        self.out_width = -(-self.width // 8) * 8           # (what the output product's tiles take)
        self.w_in = self.w_o = self.z_bias = self.x_bias = None

    def declare(self):
        n, H, W = self.names, self.hidden, self.width
        return {n["z"]: TensorDecl((W, H)), n["x"]: TensorDecl((W, H)), n["g"]: TensorDecl((W, H)),
                n["z_b"]: TensorDecl((W,), "bias"), n["x_b"]: TensorDecl((W,), "bias"), n["o"]: TensorDecl((H, W))}

    def bind(self, get, precision: Precision, device):
        n = self.names
        mats = [get(n[name]) for name in ("z", "x", "g")]
        if len({m.dtype for m in mats}) > 1:
            mats = [m.to(torch.float32) for m in mats]
        # one projection: the rows of the three matrices, one after the other
        self.w_in = precision.matrix(torch.cat(mats, dim=0), device)
        w_o = get(n["o"])
        if self.out_width != self.width:
            wide = w_o.new_zeros((w_o.shape[0], self.out_width))
            wide[:, :self.width] = w_o
            w_o = wide
        self.w_o = precision.matrix(w_o, device)
        self.z_bias = precision.vector(get(n["z_b"]), device)
        self.x_bias = precision.vector(get(n["x_b"]), device)

    def weight_bytes(self):
        return (self.w_in.numel() * self.w_in.element_size() + self.w_o.numel() * self.w_o.element_size()
                + 8 * self.width)

    def flops_per_token(self):
        return 2.0 * (self.w_in.numel() + self.w_o.numel())

    def state_spec(self):
        return FixedState((-(-self.width // 4) * 4,))       # (slots start on 16-byte borders)

    def forward(self, ctx, h, cache, residual=None):
        p = ops.linear(h, self.w_in, torch.float32)
        y = mixing.gated_average(p, 0, self.width, 2 * self.width, self.z_bias, self.x_bias, cache.state, ctx.batch,
                                 self.width, ctx.precision.act_dtype, self.out_width)
        return ops.linear_into_residual(y, self.w_o, residual)
