"""Python faces of ``csrc/state_space.cu``: the state-space recurrence with a scalar decay per head and token, and
the gate with the norm over runs of channels that follows it."""
from __future__ import annotations

import torch

from . import lib
from .lib import KernelError, c_float, c_longlong, check_tensor, is_bf16, ptr, stream
from .ops import _i32

SM_COUNT = 148
MAX_RUN_STATE = 256        # state rows up to which the tensor-core form takes a recurrence
RUNS_FROM = 16             # the longest portion of a step from which it is used
PIECES = (128, 256, 512, 1024)


def piece_tokens(tokens: int, heads: int) -> int:
    """Tokens of a segment that one block of the tensor-core form walks: the longest piece that still makes two blocks
    an SM out of the step's tokens (a segment of several pieces costs a second pass over its tokens, for their sums)."""
    for piece in reversed(PIECES):
        if -(-tokens // piece) * heads >= 2 * SM_COUNT:
            return piece
    return PIECES[0]


def _state_stride(state: torch.Tensor, size: int) -> int:
    if (not state.is_cuda or state.dtype != torch.float32 or state.dim() != 2 or state.shape[1] < size
            or state.stride(1) != 1):
        raise KernelError(f"the recurrent state must be CUDA fp32 [slots][>= {size}], got {tuple(state.shape)}")
    return state.stride(0) if state.shape[0] > 1 else state.shape[1]


def state_space(u: torch.Tensor, p: torch.Tensor, raw_col: int, dt_bias: torch.Tensor, a_log: torch.Tensor,
                skip: torch.Tensor, state: torch.Tensor, batch, heads: int, groups: int, n: int, e: int,
                runs=None) -> torch.Tensor:
    """``S <- exp(-exp(a_log) dt) S + dt b x^T; y = S^T c + skip x`` with ``dt = softplus(raw + dt_bias)`` over the
    step's ragged segments.  ``u``: [T][x (heads e) | b (groups n) | c (groups n)], fp32 or bf16; raw is ``heads``
    columns of ``p`` (fp32) from ``raw_col`` on; ``state``: fp32 [slots][>= heads n e], read at the head of every
    segment and advanced.  Returns y, fp32 [T][heads e].  Portions of prompts in bfloat16 go 64 tokens at a time
    on tensor cores; single tokens at the step's head, short portions and 32-bit runs token by token (``runs``:
    None chooses, True or False pins one form for every segment)."""
    check_tensor("recurrence input", u)
    check_tensor("projection", p, torch.float32)
    T, width = u.shape
    if width < heads * e + 2 * groups * n or raw_col + heads > p.shape[1] or p.shape[0] != T:
        raise KernelError("the recurrence's rows are shorter than the columns asked for")
    for name, t in (("step bias", dt_bias), ("decay", a_log), ("skip", skip)):
        check_tensor(name, t, torch.float32, (heads,))
    size = heads * n * e
    stride = _state_stride(state, size)
    S = batch.n_segments
    _i32("seg_start", batch.seg_start, S + 1)
    _i32("seg_slot", batch.seg_slot, S)
    y = torch.empty((T, heads * e), dtype=torch.float32, device=u.device)
    raw = p.data_ptr() + raw_col * 4
    if runs is None:
        runs = u.dtype == torch.bfloat16 and n <= MAX_RUN_STATE and batch.max_segment >= RUNS_FROM
        singles = batch.leading_singles if runs else S
    else:
        singles = 0 if runs else S
    if singles > 0:
        lib.call("fwb_state_scan", ptr(u), is_bf16(u), c_longlong(width), raw, c_longlong(p.shape[1]), ptr(dt_bias),
                 ptr(a_log), ptr(skip), ptr(state), c_longlong(stride), ptr(batch.seg_start), ptr(batch.seg_slot),
                 ptr(y), 0, singles, heads, groups, n, e, stream())
    if singles < S:
        check_tensor("recurrence input", u, torch.bfloat16)
        piece = piece_tokens(T, heads)
        piece_seg, piece_tok0, pieces = batch.attention_tiles(piece, singles)
        chained = batch.max_segment > piece
        scratch = torch.empty((pieces, size), dtype=torch.float32, device=u.device) if chained else None
        logs = torch.empty((pieces, heads), dtype=torch.float32, device=u.device) if chained else None
        lib.call("fwb_state_runs", ptr(u), c_longlong(width), raw, c_longlong(p.shape[1]), ptr(dt_bias), ptr(a_log),
                 ptr(skip), ptr(state), c_longlong(stride), ptr(batch.seg_start), ptr(batch.seg_slot), ptr(piece_seg),
                 ptr(piece_tok0), piece, 1 if chained else 0, ptr(scratch), ptr(logs), ptr(y), pieces, heads, groups,
                 n, e, stream(), launches=3 if chained else 1)
    return y


def gate_group_norm(y: torch.Tensor, p: torch.Tensor, z_col: int, weight: torch.Tensor, groups: int, eps: float,
                    out_dtype: torch.dtype) -> torch.Tensor:
    """``weight * unit(y * silu(z))``, the root mean square over each of ``groups`` equal runs of a row's channels on
    its own; z is columns of ``p`` (fp32) from ``z_col`` on.  y: fp32 [T][width]."""
    check_tensor("recurrence output", y, torch.float32)
    check_tensor("projection", p, torch.float32)
    T, width = y.shape
    check_tensor("norm weight", weight, torch.float32, (width,))
    if z_col + width > p.shape[1] or p.shape[0] != T or groups <= 0 or width % groups:
        raise KernelError("the gate's columns or the norm's groups do not fit the rows")
    out = torch.empty((T, width), dtype=out_dtype, device=y.device)
    lib.call("fwb_gate_group_norm", ptr(y), p.data_ptr() + z_col * 4, c_longlong(p.shape[1]), ptr(weight),
             c_float(eps), ptr(out), is_bf16(out), T, width, int(groups), stream())
    return out
