"""Two mixers side by side on one input.  How their outputs become one is a parameter:

* ``combine`` "normed": half the sum, each output brought to unit root mean square over the model width and
  multiplied by a weight of its own first, ``y = 0.5 (w_left * unit(left(h)) + w_right * unit(right(h)))``;
* ``combine`` "scaled": ``y = left_scale * left(h) + right_scale * right(h)`` with two constants.

The two may be of any registered kinds; between them they keep at most one set of pages and one
fixed-size state (an attention beside a recurrence), which the cache manager serves through the layer's
one ``LayerCache``.  A scaled sum of two mixers that ``joins`` runs as one input product for both (their
matrices' rows below one another) and one output product over both halves' rows side by side: the constants
are applied to the rows, in fp32, before they are rounded, and the sum is the product's own.
"""
from __future__ import annotations

import torch

from ..kernels import mixing, ops
from ..weights.loader import TensorDecl
from .base import FixedState, Mixer, PagedKV, Precision, build_mixer, register_mixer


@register_mixer("mixer_pair")
class MixerPair(Mixer):
    """params: hidden_size, left, right (``PartSpec`` of a mixer each), combine ("normed", the default, with
    eps; or "scaled" with left_scale and right_scale).  tensors: left_out, right_out [H] ("normed" only: the
    weights of the two output norms)."""

    def __init__(self, spec):
        super().__init__(spec)
        self.hidden = int(self.params["hidden_size"])
        self.combine = str(self.params.get("combine", "normed"))
        if self.combine not in ("normed", "scaled"):
            raise ValueError(f"a mixer pair combines by 'normed' or 'scaled', not by {self.combine!r}")
        self.eps = float(self.params["eps"]) if self.combine == "normed" else 0.0
        self.scales = ((float(self.params["left_scale"]), float(self.params["right_scale"]))
                       if self.combine == "scaled" else None)
        self.left = build_mixer(self.params["left"])
        self.right = build_mixer(self.params["right"])
        self.graph_safe = bool(self.left.graph_safe and self.right.graph_safe)
        self.joined = self.combine == "scaled" and self.left.joins and self.right.joins
        self.takes_deferred_norm = self.adds_residual = self.joined
        specs = self.state_spec()
        specs = specs if isinstance(specs, tuple) else (() if specs is None else (specs,))
        for kind in (PagedKV, FixedState):
            if sum(isinstance(s, kind) for s in specs) > 1:
                raise ValueError("the two halves of a mixer pair may keep one set of pages and one fixed state "
                                 f"between them, not two {kind.__name__}")
        self.w_left = self.w_right = self.w_in = self.w_o = None

    def _halves(self):
        return (self.left, self.right)

    def declare(self):
        out = {}
        if self.combine == "normed":
            out = {self.names["left_out"]: TensorDecl((self.hidden,), "norm"),
                   self.names["right_out"]: TensorDecl((self.hidden,), "norm")}
        for half in self._halves():
            out.update(half.declare())
        return out

    def bind(self, get, precision: Precision, device):
        if self.joined:
            inputs, outputs = zip(*(half.bind_joined(get, precision, device) for half in self._halves()))
            if len({m.dtype for m in inputs + outputs}) > 1:
                inputs, outputs = ([m.to(torch.float32) for m in side] for side in (inputs, outputs))
            # the left half's projections and heads first; output rows padded to what the products' tiles take
            self._right_in = inputs[0].shape[0]
            self._right_out = outputs[0].shape[1]
            used = self._right_out + outputs[1].shape[1]
            self._row = -(-used // 8) * 8
            wide = outputs[0].new_zeros((self.hidden, self._row))
            wide[:, :self._right_out] = outputs[0]
            wide[:, self._right_out:used] = outputs[1]
            self._padded = self._row != used
            self.w_in = precision.matrix(torch.cat(list(inputs), dim=0), device)
            self.w_o = precision.matrix(wide, device)
            return
        for half in self._halves():
            half.bind(get, precision, device)
        if self.combine == "normed":
            self.w_left = precision.vector(get(self.names["left_out"]), device)
            self.w_right = precision.vector(get(self.names["right_out"]), device)

    def _own_bytes(self):
        if self.joined:
            return self.w_in.numel() * self.w_in.element_size() + self.w_o.numel() * self.w_o.element_size()
        return 8 * self.hidden if self.combine == "normed" else 0

    def weight_bytes(self):
        return sum(half.weight_bytes() for half in self._halves()) + self._own_bytes()

    def active_weight_bytes(self, n_tokens):
        return sum(half.active_weight_bytes(n_tokens) for half in self._halves()) + self._own_bytes()

    def flops_per_token(self):
        own = 2.0 * (self.w_in.numel() + self.w_o.numel()) if self.joined else 0.0
        return own + sum(half.flops_per_token() for half in self._halves())

    def context_flops(self, n_tokens):
        return sum(half.context_flops(n_tokens) for half in self._halves())

    def state_spec(self):
        specs = []
        for half in self._halves():
            spec = half.state_spec()
            if spec is not None:
                specs.extend(spec if isinstance(spec, tuple) else (spec,))
        if not specs:
            return None
        return specs[0] if len(specs) == 1 else tuple(specs)

    def prepare(self, max_positions, device):
        for half in self._halves():
            half.prepare(max_positions, device)

    def forward(self, ctx, h, cache, residual=None):
        if self.joined:
            act = ctx.precision.act_dtype
            p = ops.linear(h, self.w_in, torch.float32)
            rows = (torch.zeros if self._padded else torch.empty)((p.shape[0], self._row), dtype=act, device=p.device)
            self.left.forward_joined(ctx, p, 0, cache, rows, 0, self.scales[0])
            self.right.forward_joined(ctx, p, self._right_in, cache, rows, self._right_out, self.scales[1])
            return ops.linear_into_residual(rows, self.w_o, residual)
        a = self.left.forward(ctx, h, cache)
        b = self.right.forward(ctx, h, cache)
        if self.combine == "normed":
            return mixing.pair_norm_mean(a, self.w_left, b, self.w_right, self.eps)
        ops.add_(ops.scale_(a, self.scales[0]), ops.scale_(b, self.scales[1]))
        return a
