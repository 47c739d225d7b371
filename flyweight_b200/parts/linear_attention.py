"""Linear attention with a fixed decay per head: a recurrence whose state is one [dim][vdim] matrix per head
and request, in two forms that differ around it.

Per token, with h the mixer's input:  q = W_q h, k = W_k h (heads x dim), v = W_v h (heads x vdim), all three
through silu when ``activation`` says so, k times ``k_scale``; per head

    S <- decay_h S + k v^T;     o = S^T q

Lightning attention (``norm`` "all", ``gate`` "sigmoid"): ``W_o( w * o / rms(o) * sigmoid(W_g h) )`` with the
root mean square over all heads of a token together and a weight per channel.  Retention (``norm`` "head",
``gate`` "silu"): every head's o is brought to unit root mean square without a weight, then ``W_o( o *
silu(W_g h) )``.  S lives in the request's state slot (fp32, zero at admission), so a sequence may be cut
into steps anywhere.  One fused projection q|k|v|gate leaves its product in fp32; the activations, the
recurrence, the norm and the gate are computed in 32-bit in both precisions.
"""
from __future__ import annotations

import torch

from ..kernels import mixing, ops, recurrent
from ..weights.loader import TensorDecl
from .base import FixedState, Mixer, Precision, register_mixer


@register_mixer("decayed_linear_attention")
class DecayedLinearAttention(Mixer):
    """params: hidden_size, num_heads, dim, vdim, decay (one number per head), eps (of the output's norm), and
    optionally activation ("silu", the default, or None), k_scale (1), norm ("all" | "head"), gate ("sigmoid" with
    norm "all", "silu" with norm "head").
    tensors: q, k [heads dim][H]; v, g [heads vdim][H]; norm [heads vdim] (norm "all" only); o [H][heads vdim]."""
    graph_safe = True
    RUNS_FROM = 16      # the longest portion of a step from which the tensor-core form takes the step

    def __init__(self, spec):
        super().__init__(spec)
        p = self.params
        self.hidden = int(p["hidden_size"])
        self.n_heads = int(p["num_heads"])
        self.dim = int(p["dim"])
        self.vdim = int(p["vdim"])
        self.eps = float(p["eps"])
        self.decay_values = [float(x) for x in p["decay"]]
        self.activation = p.get("activation", "silu")
        self.k_scale = float(p.get("k_scale", 1.0))
        self.norm_over = str(p.get("norm", "all"))
        gate = p.get("gate", "sigmoid" if self.norm_over == "all" else "silu")
        if min(self.n_heads, self.dim, self.vdim) <= 0:
            raise ValueError("linear attention: heads, dim and vdim must be positive")
        if len(self.decay_values) != self.n_heads:
            raise ValueError(f"linear attention: {len(self.decay_values)} decays for {self.n_heads} heads")
        if self.activation not in ("silu", None):
            raise ValueError(f"linear attention: unknown activation {self.activation!r}; known: silu, None")
        if (self.norm_over, gate) not in (("all", "sigmoid"), ("head", "silu")):
            raise ValueError(f"linear attention: a norm over {self.norm_over!r} with the gate {gate!r} has no form; "
                             "known: all with sigmoid, head with silu")
        self.joins = self.norm_over == "head"
        self.w_in = self.w_o = self.norm = self.decay = None

    @property
    def _qk(self) -> int:
        return self.n_heads * self.dim

    @property
    def _v(self) -> int:
        return self.n_heads * self.vdim

    @property
    def out_width(self) -> int:
        """Columns this mixer fills of a joined output row."""
        return self._v

    def declare(self):
        n, H = self.names, self.hidden
        out = {n["q"]: TensorDecl((self._qk, H)), n["k"]: TensorDecl((self._qk, H)),
               n["v"]: TensorDecl((self._v, H)), n["g"]: TensorDecl((self._v, H))}
        if self.norm_over == "all":
            out[n["norm"]] = TensorDecl((self._v,), "norm")
        out[n["o"]] = TensorDecl((H, self._v))
        return out

    def bind(self, get, precision: Precision, device):
        rows, w_o = self.bind_joined(get, precision, device)
        self.w_in = precision.matrix(rows, device)
        self.w_o = precision.matrix(w_o, device)

    def bind_joined(self, get, precision: Precision, device):
        n = self.names
        mats = [get(n[name]) for name in ("q", "k", "v", "g")]
        if len({m.dtype for m in mats}) > 1:
            mats = [m.to(torch.float32) for m in mats]
        if self.norm_over == "all":
            self.norm = precision.vector(get(n["norm"]), device)
        self.decay = torch.tensor(self.decay_values, dtype=torch.float32, device=device)
        # one projection: the rows of the four matrices, one after the other
        return torch.cat(mats, dim=0), get(n["o"])

    def weight_bytes(self):
        if self.w_in is None:                     # (the matrices belong to the mixer that joined this one)
            return 0
        return self.w_in.numel() * self.w_in.element_size() + self.w_o.numel() * self.w_o.element_size()

    def flops_per_token(self):
        # the products, and per head two passes over the [dim][vdim] state (decay and write, read-out)
        products = 0 if self.w_in is None else 2.0 * (self.w_in.numel() + self.w_o.numel())
        return products + 4.0 * self.n_heads * self.dim * self.vdim

    def state_spec(self):
        # (slots start on 16-byte borders)
        return FixedState((-(-self.n_heads * self.dim * self.vdim // 4) * 4,))

    def _recurrence(self, ctx, p, col0, cache):
        # portions of prompts in bfloat16 walk 64 tokens at a time on tensor cores (q, k, v rounded to bfloat16,
        # the state and the sums in fp32); single tokens, short portions and 32-bit runs go token by token
        runs = (ctx.precision.act_dtype == torch.bfloat16 and self.dim <= 256
                and getattr(ctx.batch, "max_segment", 1) >= self.RUNS_FROM)
        return (mixing.decay_runs if runs else mixing.decay_scan)(
            p, col0, col0 + self._qk, col0 + 2 * self._qk, self.decay, cache.state, ctx.batch, self.n_heads, self.dim,
            self.vdim, act_silu=self.activation == "silu", k_scale=self.k_scale)

    def forward_joined(self, ctx, p, col0, cache, rows, out_col, scale):
        """Everything between the two products: ``p`` holds this mixer's projections (fp32) from column ``col0``
        on, its columns of ``rows`` from ``out_col`` on receive the normed and gated heads times ``scale``."""
        o = self._recurrence(ctx, p, col0, cache)
        gate_at = col0 + 2 * self._qk + self._v
        recurrent.gated_head_norm(o.view(-1, self.n_heads, self.vdim), p[:, gate_at:gate_at + self._v], None, self.eps,
                                  rows.dtype, out=rows, col0=out_col, scale=scale)

    def forward(self, ctx, h, cache):
        p = ops.linear(h, self.w_in, torch.float32)
        if self.norm_over == "head":
            z = torch.empty((p.shape[0], self._v), dtype=ctx.precision.act_dtype, device=p.device)
            self.forward_joined(ctx, p, 0, cache, z, 0, 1.0)
        else:
            o = self._recurrence(ctx, p, 0, cache)
            gate_at = 2 * self._qk + self._v
            z = mixing.gated_rmsnorm(o, p[:, gate_at:gate_at + self._v], self.norm, self.eps, ctx.precision.act_dtype)
        return ops.linear(z, self.w_o, torch.float32)
