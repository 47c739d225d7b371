"""Python faces of the mixture-of-experts kernels (``csrc/moe.cu``): router, sorting of the
(token, expert) pairs, the experts' products over the sorted rows, the weighted sum."""
from __future__ import annotations

from typing import Optional

import torch

from . import lib
from .lib import KernelError, c_float, c_longlong, check_tensor, is_bf16, ptr, stream
from .ops import GATE_ACTIVATIONS, OUTPUT_ACTIVATIONS


SIMT_TILE_ROWS = 64          # rows of a tile of fwb_moe_gemm
_use_tensor_cores = True


def set_tensor_cores(flag: bool) -> None:
    """Tests switch the grouped tcgen05 product off to compare it with the fp32-FMA kernel."""
    global _use_tensor_cores
    _use_tensor_cores = bool(flag)


TENSOR_CORE_ROUTER_FROM = 256      # tokens of a step from which a bfloat16 router is a matrix product
ROUTER_SCORES = {"softmax": 0, "sigmoid": 1, "softmax_chosen": 2}


def route(h: torch.Tensor, router: torch.Tensor, correction: Optional[torch.Tensor], n_groups: int, keep: int, top: int,
          scores: str = "softmax", router16: Optional[torch.Tensor] = None, gate: bool = False):
    """ids int32 [T][top] and weights fp32 [T][top]: ``scores`` "softmax" over all router outputs or the
    "sigmoid" of each; the choice on score (+ correction), or (
    "softmax_chosen") on the outputs themselves (+ correction) with the softmax over the chosen alone; inside the ``keep`` best of ``n_groups`` runs of
    neighbours; the weights are the chosen outputs' plain scores.  ``router16``: the same router in bfloat16, when
    that loses nothing: bfloat16 rows of a prompt then take the tensor-core product (products of bfloat16 numbers
    are exact in fp32, and so is what they are summed in) and a kernel that only chooses.  ``gate``: the router's
    matrix has one row more; a third tensor, fp32 [T], is returned with the sigmoid of that row's product."""
    check_tensor("router input", h)
    T, W = h.shape
    rows = router.shape[0]
    N = rows - (1 if gate else 0)
    check_tensor("router", router, torch.float32, (rows, W))
    if correction is not None:
        check_tensor("router correction", correction, torch.float32, (N,))
    if scores not in ROUTER_SCORES:
        raise KernelError(f"unknown router scores {scores!r}; known: " + ", ".join(ROUTER_SCORES))
    ids = torch.empty((T, top), dtype=torch.int32, device=h.device)
    weights = torch.empty((T, top), dtype=torch.float32, device=h.device)
    gates = torch.empty(T, dtype=torch.float32, device=h.device) if gate else None
    out = (ids, weights, gates) if gate else (ids, weights)
    if router16 is not None and T >= TENSOR_CORE_ROUTER_FROM and h.dtype == torch.bfloat16:
        from . import tensorcore
        if tensorcore.accepts(h, router16, torch.float32):
            # one tile of features: token tiles and slices of K make the CTAs
            tile = 64 if T <= 2048 else 128
            splits = 4 if -(-T // tile) <= 37 and W >= 1024 else (2 if -(-T // tile) <= 74 and W >= 512 else 1)
            logits = tensorcore.gemm(h, router16, torch.float32, splits=splits, tile_tokens=tile)
            lib.call("fwb_moe_choose", ptr(logits), ptr(correction), ptr(ids), ptr(weights), T, N, int(n_groups), int(keep),
                     int(top), ROUTER_SCORES[scores], c_longlong(logits.shape[1]), ptr(gates), stream())
            return out
    lib.call("fwb_moe_route", ptr(h), is_bf16(h), ptr(router), ptr(correction), ptr(ids), ptr(weights), T, W, N,
             int(n_groups), int(keep), int(top), ROUTER_SCORES[scores], ptr(gates), stream())
    return out


def route_table(token_ids: torch.Tensor, table: torch.Tensor, top: int):
    """ids int32 [T][top] and weights fp32 [T][top] of a router that is a table: row ``token_ids[t]`` of
    ``table`` (int32 [vocab][top]) names the token's experts, each with weight 1 / top."""
    check_tensor("token ids", token_ids, torch.int32)
    check_tensor("expert table", table, torch.int32)
    if table.dim() != 2 or table.shape[1] != top:
        raise KernelError(f"the expert table must be [vocab][{top}], got {tuple(table.shape)}")
    T = token_ids.numel()
    ids = torch.empty((T, top), dtype=torch.int32, device=table.device)
    weights = torch.empty((T, top), dtype=torch.float32, device=table.device)
    lib.call("fwb_moe_route_table", ptr(token_ids), ptr(table), table.shape[0], int(top), T, ptr(ids), ptr(weights),
             stream())
    return ids, weights


def experts_forward(h: torch.Tensor, ids: torch.Tensor, weights: torch.Tensor, w_gate_up: torch.Tensor,
                    w_down: torch.Tensor, activation: str = "silu", add_normed_into=None, limit: float = 0.0,
                    weights_on: str = "output", gated: bool = True, plus=None):
    """``sum_slot weights * expert(h)`` as fp32 [T][W].  ``w_gate_up``: [E][2F][W] (gate rows, then up
    rows), ``w_down``: [E][W][F], both in the dtype of ``h``.  Router outputs from E on are identity
    experts: they pass ``h`` itself on.  ``gated`` False: experts without a gate, ``down(act(up h))`` with ``activation``
    one of ``OUTPUT_ACTIVATIONS``; ``w_gate_up`` is then [E][F][W].  ``add_normed_into`` = (x, norm weight, eps): the sum is not
    returned but normed and added, ``x += weight * sum / sqrt(mean(sum^2) + eps)`` in fp32, by the kernel
    that makes it (returns None); a fourth entry, fp32 [T][W], is added to every token's sum first (the output of an
    expert that every token shares), times its entry of a fifth, fp32 [T], when there is one.  ``plus`` = (fp32 [T][W], fp32 [T] or None): the same two for a sum that is returned.
    ``weights_on`` "input": a pair's weight multiplies what the expert reads,
    ``sum_slot expert(weights * h)``, and the experts' rows are added as they are."""
    check_tensor("expert input", h)
    T, W = h.shape
    top = ids.shape[1]
    E, F2, _ = w_gate_up.shape
    F = F2 // 2 if gated else F2
    check_tensor("expert gate|up", w_gate_up, h.dtype, (E, 2 * F if gated else F, W))
    check_tensor("expert down", w_down, h.dtype, (E, W, F))
    check_tensor("expert ids", ids, torch.int32, (T, top))
    check_tensor("expert weights", weights, torch.float32, (T, top))
    act = (GATE_ACTIVATIONS if gated else OUTPUT_ACTIVATIONS)[activation]
    A = T * top
    bf16 = is_bf16(h)
    # bfloat16 rows whose lengths the tensor maps take run the grouped tcgen05 product, on token tiles
    # as wide as an expert's share of the step's rows; everything else the fp32-FMA kernel (tiles of 64)
    tensor_cores = bool(bf16 and _use_tensor_cores and E > 0 and W % 8 == 0 and F % 8 == 0)
    tile_rows = SIMT_TILE_ROWS
    if tensor_cores:
        share = -(-A // E)
        tile_rows = 16 if share <= 16 else (32 if share <= 32 else (64 if share <= 64 else 128))
    max_tiles = A // tile_rows + E + 1
    dev = h.device
    meta = torch.empty(E + 1 + 2 * A + 1 + 2 * max_tiles, dtype=torch.int32, device=dev)
    offsets, row_token = meta[:E + 1], meta[E + 1:E + 1 + A]
    pair_row, tiles = meta[E + 1 + A:E + 1 + 2 * A], meta[E + 1 + 2 * A:]
    if weights_on not in ("output", "input"):
        raise KernelError(f"expert weights go on the output or on the input, not on {weights_on!r}")
    weighted_in = 1 if weights_on == "input" else 0
    row_weight = torch.empty(A, dtype=torch.float32, device=dev) if weighted_in else None
    lib.call("fwb_moe_sort", ptr(ids), A, top, E, tile_rows, ptr(offsets), ptr(row_token), ptr(pair_row), ptr(tiles),
             ptr(weights) if weighted_in else None, ptr(row_weight), stream())
    a = torch.empty((A, F), dtype=h.dtype, device=dev)
    y = torch.empty((A, W), dtype=torch.float32, device=dev)
    if tensor_cores:
        from .tensorcore import EPI_F32, _gated_epilogue, _output_epilogue
        rows = torch.empty((A, W), dtype=h.dtype, device=dev)
        lib.call("fwb_moe_gather_rows", ptr(h), ptr(row_token), ptr(offsets), E, ptr(rows), A, W, ptr(row_weight),
                 stream())
        lib.call("fwb_gemm_tcgen05_grouped", ptr(rows), ptr(w_gate_up), ptr(a), ptr(offsets), ptr(tiles), max_tiles,
                 tile_rows, A, F, W, E, F2, F, _gated_epilogue(activation) if gated else _output_epilogue(activation),
                 F if gated else 0, c_float(limit), stream(), tag=f"experts {'gate|up' if gated else 'up'} {F}x{W}")
        lib.call("fwb_gemm_tcgen05_grouped", ptr(a), ptr(w_down), ptr(y), ptr(offsets), ptr(tiles), max_tiles,
                 tile_rows, A, W, F, E, W, W, EPI_F32, 0, c_float(0.0), stream(), tag=f"experts down {W}x{F}")
    elif E > 0:                                 # (a router may have identity experts only)
        lib.call("fwb_moe_gemm", ptr(h), ptr(w_gate_up), bf16, ptr(a), ptr(offsets), ptr(row_token), ptr(tiles),
                 max_tiles, F, W, 1 if gated else 2, act, c_float(limit), ptr(row_weight), stream())
        lib.call("fwb_moe_gemm", ptr(a), ptr(w_down), bf16, ptr(y), ptr(offsets), ptr(row_token), ptr(tiles),
                 max_tiles, W, F, 0, 0, c_float(0.0), None, stream())
    if add_normed_into is not None:
        x, norm_weight, eps = add_normed_into[:3]
        extra, extra_gate = (tuple(add_normed_into[3:]) + (None, None))[:2]
        check_tensor("residual", x, torch.float32, (T, W))
        check_tensor("norm weight", norm_weight, torch.float32, (W,))
        if extra is not None:
            check_tensor("shared output", extra, torch.float32, (T, W))
        if extra_gate is not None:
            check_tensor("shared gate", extra_gate, torch.float32, (T,))
        lib.call("fwb_moe_combine_norm_add", ptr(y), ptr(h), bf16, ptr(pair_row), ptr(ids), ptr(weights), ptr(x),
                 ptr(norm_weight), c_float(eps), T, W, top, E, ptr(extra), ptr(extra_gate), weighted_in, stream())
        return None
    out = torch.empty((T, W), dtype=torch.float32, device=dev)
    lib.call("fwb_moe_combine", ptr(y), ptr(h), bf16, ptr(pair_row), ptr(ids), ptr(weights), ptr(out), T, W, top,
             E, ptr(plus[0]) if plus else None, ptr(plus[1]) if plus else None, weighted_in, stream())
    return out
