"""Python faces of the CUDA kernels: argument checks, output allocation, launch.

Each function is one kernel (or one dispatch between kernels of the same operation).
Shapes are checked here on the host before anything is launched.
"""
from __future__ import annotations

from typing import Optional

import torch

from . import lib
from .lib import KernelError, c_float, c_longlong, check_tensor, is_bf16, ptr, stream


def _i32(name: str, tensor: torch.Tensor, count: Optional[int] = None) -> None:
    check_tensor(name, tensor, torch.int32)
    if count is not None and tensor.numel() < count:
        raise KernelError(f"{name} holds {tensor.numel()} entries, {count} are needed")


# ------------------------------------------------------------------ embedding
def embed(table: torch.Tensor, ids: torch.Tensor, bad_flag: Optional[torch.Tensor] = None,
          scale: float = 1.0) -> torch.Tensor:
    """Rows ``ids`` of ``table`` ([V][H], fp32 or bf16) widened to fp32 and multiplied by
    ``scale``: [T][H]."""
    check_tensor("embedding table", table)
    _i32("token ids", ids)
    T, (V, H) = ids.numel(), table.shape
    out = torch.empty((T, H), dtype=torch.float32, device=table.device)
    lib.call("fwb_embed", ptr(table), is_bf16(table), ptr(ids), ptr(out), T, H, V, ptr(bad_flag),
             c_float(scale), stream())
    return out


def patch_tokens_(token_ids: torch.Tensor, dst: torch.Tensor, source: torch.Tensor, src: torch.Tensor) -> None:
    """``token_ids[dst[i]] = source[src[i]]`` on the device (all int32): ids that the step before
    sampled and the host has not read yet go straight into this step's batch."""
    for name, tensor in (("token ids", token_ids), ("patch places", dst), ("patch source", source),
                         ("patch rows", src)):
        _i32(name, tensor)
    if dst.numel() != src.numel():
        raise KernelError("one source row per patched place is needed")
    lib.call("fwb_patch_tokens", ptr(token_ids), ptr(dst), ptr(source), ptr(src), dst.numel(), stream())


# ------------------------------------------------------------------ norms
def rmsnorm(x: torch.Tensor, weight: torch.Tensor, eps: float, out_dtype: torch.dtype,
            delta: Optional[torch.Tensor] = None, rows: Optional[torch.Tensor] = None
            ) -> torch.Tensor:
    """``(x * rsqrt(mean(x^2) + eps)) * weight`` per row of the fp32 residual ``x``.

    With ``delta`` the residual sum ``x += delta`` happens first, in place and in fp32.
    With ``rows`` (int32 indices) only those rows are normalised, into a compact output.
    """
    check_tensor("residual", x, torch.float32)
    H = x.shape[-1]
    check_tensor("norm weight", weight, torch.float32, (H,))
    if delta is not None:
        check_tensor("delta", delta, torch.float32, x.shape)
    if rows is not None:
        _i32("row indices", rows)
        R = rows.numel()
    else:
        R = x.numel() // H
    out = torch.empty((R, H), dtype=out_dtype, device=x.device)
    lib.call("fwb_rmsnorm", ptr(x), ptr(delta), ptr(weight), ptr(out), is_bf16(out), ptr(rows), R, H,
             c_float(eps), stream())
    return out


def rmsnorm_add_(x: torch.Tensor, y: torch.Tensor, weight: torch.Tensor, eps: float,
                 next_weight: Optional[torch.Tensor] = None, next_eps: float = 0.0,
                 next_dtype: Optional[torch.dtype] = None) -> Optional[torch.Tensor]:
    """``x += weight * y / sqrt(mean(y^2) + eps)`` per row, in place and in fp32: a norm on a
    sublayer's output with the residual sum behind it.  With ``next_weight`` the same pass also
    returns ``next_weight * x / sqrt(mean(x^2) + next_eps)`` of the new rows in ``next_dtype``: the norm
    in front of the next sublayer."""
    check_tensor("residual", x, torch.float32)
    check_tensor("sublayer output", y, torch.float32, x.shape)
    H = x.shape[-1]
    check_tensor("norm weight", weight, torch.float32, (H,))
    out = None
    if next_weight is not None:
        check_tensor("next norm weight", next_weight, torch.float32, (H,))
        out = torch.empty(x.shape, dtype=next_dtype or torch.float32, device=x.device)
    lib.call("fwb_rmsnorm_add", ptr(x), ptr(y), ptr(weight), c_float(eps), ptr(next_weight), c_float(next_eps),
             ptr(out), is_bf16(out) if out is not None else 0, x.numel() // H, H, stream())
    return out


def add_(x: torch.Tensor, delta: torch.Tensor) -> None:
    check_tensor("residual", x, torch.float32)
    check_tensor("delta", delta, torch.float32, x.shape)
    lib.call("fwb_add", ptr(x), ptr(delta), c_longlong(x.numel()), stream())


def softcap_(logits: torch.Tensor, cap: float) -> torch.Tensor:
    """``cap * tanh(logits / cap)`` in place on fp32."""
    check_tensor("logits", logits, torch.float32)
    if not cap > 0:
        raise KernelError("a soft-cap must be positive")
    lib.call("fwb_softcap", ptr(logits), c_longlong(logits.numel()), c_float(cap), stream())
    return logits


def scale_(x: torch.Tensor, factor: float) -> torch.Tensor:
    """``x *= factor`` in place on fp32."""
    check_tensor("scaled tensor", x, torch.float32)
    lib.call("fwb_scale", ptr(x), c_longlong(x.numel()), c_float(factor), stream())
    return x


def cast(x: torch.Tensor, dtype: torch.dtype) -> torch.Tensor:
    if x.dtype == dtype:
        return x
    check_tensor("cast input", x)
    out = torch.empty(x.shape, dtype=dtype, device=x.device)
    lib.call("fwb_cast", ptr(x), is_bf16(x), ptr(out), is_bf16(out), c_longlong(x.numel()), stream())
    return out


# ------------------------------------------------------------------ matrix products
def gemm_simt(x: torch.Tensor, w: torch.Tensor, out_dtype: torch.dtype,
              addend: Optional[torch.Tensor] = None, out: Optional[torch.Tensor] = None
              ) -> torch.Tensor:
    """``x @ w.T`` with fp32 FMA accumulation (no tensor cores).  x: [M][K], w: [N][K]."""
    check_tensor("gemm input", x)
    check_tensor("gemm weight", w)
    M, K = x.shape
    N, K2 = w.shape
    if K != K2:
        raise KernelError(f"gemm: input has {K} columns, weight has {K2}")
    if out is None:
        out = torch.empty((M, N), dtype=out_dtype, device=x.device)
    else:
        check_tensor("gemm output", out, out_dtype, (M, N))
    if addend is not None:
        check_tensor("gemm addend", addend, torch.float32, (M, N))
    lib.call("fwb_gemm_simt", ptr(x), is_bf16(x), ptr(w), is_bf16(w), ptr(out), is_bf16(out),
             ptr(addend), M, N, K, K, N, stream())
    return out


def linear(x, w: torch.Tensor, out_dtype: torch.dtype,
           addend: Optional[torch.Tensor] = None) -> torch.Tensor:
    """The matrix product the model uses: picks the kernel for the dtypes and sizes.

    float32 weights always take the SIMT kernel (true 32-bit).  bfloat16 weights take
    the tensor-core kernel when it accepts the shape, else the SIMT kernel.  ``x`` may be a
    norm not yet applied (``parts.base.DeferredNorm``): an RMS norm in front of a decode-sized
    bfloat16 product runs inside that product's kernel, otherwise its own kernel runs first.
    """
    from . import tensorcore
    if not isinstance(x, torch.Tensor):                       # a DeferredNorm
        if (addend is None and x.kind == "rmsnorm"
                and tensorcore.normed_accepts(x.n_rows, x.x.shape[-1], w, 1, w.shape[0])):
            return tensorcore.gemm_normed(x.x, x.weight, x.eps, w, out_dtype, rows=x.rows, n_rows=x.n_rows)
        x = x.materialize(torch.float32 if w.dtype == torch.float32 else torch.bfloat16)
    if w.dtype == torch.float32:
        if x.dtype != torch.float32:
            x = cast(x, torch.float32)
        return gemm_simt(x, w, out_dtype, addend)
    if x.dtype != torch.bfloat16:
        x = cast(x, torch.bfloat16)
    if tensorcore.accepts(x, w, out_dtype, addend):
        return tensorcore.gemm(x, w, out_dtype, addend)
    return gemm_simt(x, w, out_dtype, addend)


def linear_act(x: torch.Tensor, w: torch.Tensor, activation: str, out_dtype: torch.dtype) -> torch.Tensor:
    """``act(x @ w.T)``, the activation (one of ``OUTPUT_ACTIVATIONS``) on the product's fp32 sums: in the tensor-core
    product's epilogue when the output is bfloat16, else as a pass of its own."""
    from . import mixing, tensorcore
    if w.dtype == torch.bfloat16 and out_dtype == torch.bfloat16:
        x = cast(x, torch.bfloat16)
        if tensorcore.accepts(x, w, out_dtype):
            return tensorcore.gemm(x, w, out_dtype, activation=activation)
    return mixing.unary_act(linear(x, w, torch.float32), activation, out_dtype)


def linear_into_residual(x: torch.Tensor, w: torch.Tensor, residual: Optional[torch.Tensor]):
    """``residual += x @ w.T`` in the product's epilogue when the tensor-core kernel has that
    form for the shape (returns None); otherwise the fp32 product, for the caller to hand on."""
    from . import tensorcore
    if (residual is not None and w.dtype == torch.bfloat16 and x.dtype == torch.bfloat16
            and tensorcore.adds_in_place(x, w, residual)):
        tensorcore.gemm(x, w, torch.float32, addend=residual, out=residual)
        return None
    return linear(x, w, torch.float32)


def silu_mul(gate_up: torch.Tensor, out_dtype: torch.dtype) -> torch.Tensor:
    """``silu(gate) * up`` for ``gate_up`` = [T][gate(F) | up(F)]."""
    check_tensor("gate|up", gate_up)
    T, F2 = gate_up.shape
    if F2 % 2:
        raise KernelError("gate|up needs an even number of columns")
    out = torch.empty((T, F2 // 2), dtype=out_dtype, device=gate_up.device)
    lib.call("fwb_silu_mul", ptr(gate_up), is_bf16(gate_up), ptr(out), is_bf16(out), T, F2 // 2,
             stream())
    return out


# what a gated feed-forward makes of gate g and up u: silu(g) u, gelu(g) u (tanh form), or the clamped swish
# min(g, L) sigmoid(1.702 min(g, L)) (clamp(u, -L, L) + 1) with a limit L, or max(g, 0) u
GATE_ACTIVATIONS = {"silu": 0, "gelu_tanh": 1, "swish_clamped": 2, "relu": 3}
# what a product without a gate may do to a bfloat16 output on its way out (in fp32, ahead of the rounding)
OUTPUT_ACTIVATIONS = {None: 0, "relu_squared": 1}


def gate_act_mul(gate_up: torch.Tensor, out_dtype: torch.dtype, activation: str = "silu",
                 limit: float = 0.0) -> torch.Tensor:
    """``act(gate) * up`` for ``gate_up`` = [T][gate(F) | up(F)]; ``activation``: "silu", "gelu_tanh"
    (0.5 g (1 + tanh(sqrt(2/pi) (g + 0.044715 g^3)))), "swish_clamped" with its ``limit``, or "relu"."""
    check_tensor("gate|up", gate_up)
    T, F2 = gate_up.shape
    if F2 % 2:
        raise KernelError("gate|up needs an even number of columns")
    try:
        act = GATE_ACTIVATIONS[activation]
    except KeyError:
        raise KernelError(f"unknown gate activation {activation!r}; known: " + ", ".join(GATE_ACTIVATIONS)) from None
    out = torch.empty((T, F2 // 2), dtype=out_dtype, device=gate_up.device)
    lib.call("fwb_gate_act_mul", ptr(gate_up), is_bf16(gate_up), ptr(out), is_bf16(out), T, F2 // 2, act,
             lib.c_float(limit), stream())
    return out


# ------------------------------------------------------------------ gated short convolution
def shortconv(p: torch.Tensor, taps: torch.Tensor, bias: Optional[torch.Tensor],
              state: torch.Tensor, seg_start: torch.Tensor, seg_slot: torch.Tensor,
              tok_seg: torch.Tensor, n_segments: int, out_dtype: torch.dtype) -> torch.Tensor:
    """p: [T][B|C|x]; taps: [H][L] fp32; state: [slots][H][L-1] fp32 (read and advanced)."""
    check_tensor("conv input", p)
    T, H3 = p.shape
    H = H3 // 3
    if H * 3 != H3:
        raise KernelError("conv input needs 3*H columns")
    L = taps.shape[1]
    check_tensor("conv taps", taps, torch.float32, (H, L))
    if bias is not None:
        check_tensor("conv bias", bias, torch.float32, (H,))
    if not state.is_cuda or state.dtype != torch.float32 or tuple(state.shape[1:]) != (H, L - 1):
        raise KernelError(f"conv state must be CUDA fp32 [slots][{H}][{L - 1}], got {tuple(state.shape)}")
    if state.stride(2) != 1 or state.stride(1) != L - 1 or (state.shape[0] > 1 and state.stride(0) < H * (L - 1)):
        raise KernelError("a slot of the conv state must be contiguous")
    slot_stride = state.stride(0) if state.shape[0] > 1 else H * (L - 1)
    _i32("seg_start", seg_start, n_segments + 1)
    _i32("seg_slot", seg_slot, n_segments)
    _i32("tok_seg", tok_seg, T)
    out = torch.empty((T, H), dtype=out_dtype, device=p.device)
    lib.call("fwb_shortconv", ptr(p), is_bf16(p), ptr(taps), ptr(bias), ptr(state), ptr(seg_start),
             ptr(seg_slot), ptr(tok_seg), ptr(out), is_bf16(out), T, n_segments, H, L,
             c_longlong(slot_stride), stream())
    return out


# ------------------------------------------------------------------ attention
ROPE_PAIRINGS = {"half_split": 0, "interleaved": 1}


def qk_norm_rope(qkv: torch.Tensor, q_norm: Optional[torch.Tensor], k_norm: Optional[torch.Tensor],
                 table: torch.Tensor, positions: torch.Tensor, tok_seg: torch.Tensor,
                 block_table: Optional[torch.Tensor], k_pool: Optional[torch.Tensor],
                 v_pool: Optional[torch.Tensor], n_heads: int, n_kv_in: int, head_dim: int,
                 rotary_dim: int, eps: float, q_dtype: torch.dtype, pairing: str = "half_split",
                 unit_rms_after: bool = False, norm_dim: int = 0, bias: Optional[torch.Tensor] = None,
                 temp: Optional[torch.Tensor] = None, value_table: Optional[torch.Tensor] = None,
                 value_rotary: int = 0) -> torch.Tensor:
    """Per-head RMSNorm + RoPE of q and k, k/v written to their pages; returns q [T][nh*hd].

    ``unit_rms_after``: instead of the weighted norm in front of the rotation, every head of q and k
    is brought to unit root mean square *behind* it, without a weight (``q_norm``/``k_norm`` are not
    read).  ``norm_dim``: over how many channels the mean of squares is taken (0: all ``head_dim``; fewer
    when the last channels of every head are zero padding).

    ``n_kv_in`` is the number of KV heads present in ``qkv`` (0: queries only).
    ``table`` is [max_pos][rotary_dim/2][2] fp32 (cos, sin); pair i turns by entry i.
    ``pairing``: which two channels pair i is made of -- "half_split" (i, i + rotary_dim/2) or
    "interleaved" (2i, 2i + 1).

    ``qkv`` may be the first columns of a wider buffer.  ``bias``: fp32 [columns of q|k|v], added to the
    projection first; ``temp``: fp32 [n_heads], multiplies the finished query of its head;
    ``value_rotary`` > 0: the first that many channels of every value head turn by their own position as
    well, by ``value_table`` ([max_pos][value_rotary/2][2]) with the same pairing, before they are stored."""
    try:
        pairing_code = ROPE_PAIRINGS[pairing]
    except KeyError:
        raise KernelError(f"unknown rotary pairing {pairing!r}; known: " + ", ".join(ROPE_PAIRINGS)) from None
    width = (n_heads + 2 * n_kv_in) * head_dim
    if not qkv.is_cuda or qkv.dim() != 2 or qkv.stride(1) != 1:
        raise KernelError("qkv must be a CUDA matrix with contiguous rows")
    T = qkv.shape[0]
    if qkv.shape[1] != width:
        raise KernelError(f"qkv has {qkv.shape[1]} columns, expected {width}")
    if bias is not None:
        check_tensor("q|k|v bias", bias, torch.float32, (width,))
    if temp is not None:
        check_tensor("head factors", temp, torch.float32, (n_heads,))
    if value_rotary:
        check_tensor("value table", value_table, torch.float32)
        if value_rotary % 2 or value_rotary > head_dim or tuple(value_table.shape[1:]) != (value_rotary // 2, 2):
            raise KernelError("value table must be [positions][value_rotary/2][2]")
    check_tensor("rope table", table, torch.float32)
    if table.dim() != 3 or table.shape[1] != max(1, rotary_dim // 2) or table.shape[2] != 2:
        raise KernelError("rope table must be [positions][rotary_dim/2][2]")
    use_norm = 2 if unit_rms_after else (1 if q_norm is not None else 0)
    if use_norm == 1:
        check_tensor("q norm weight", q_norm, torch.float32, (head_dim,))
        if n_kv_in:
            check_tensor("k norm weight", k_norm, torch.float32, (head_dim,))
    if not 0 <= norm_dim <= head_dim:
        raise KernelError(f"the norm of a head of {head_dim} channels cannot go over {norm_dim}")
    _i32("positions", positions, T)
    _i32("tok_seg", tok_seg, T)
    max_pages = page_size = 0
    cache_bf16 = is_bf16(qkv) if n_kv_in == 0 else 0
    if n_kv_in:
        _i32("block table", block_table)
        check_tensor("k pool", k_pool)
        check_tensor("v pool", v_pool, k_pool.dtype, k_pool.shape)
        if k_pool.dim() != 4 or k_pool.shape[1] != n_kv_in or k_pool.shape[3] != head_dim:
            raise KernelError("cache pools must be [pages][kv_heads][page_size][head_dim]")
        max_pages, page_size = block_table.shape[1], k_pool.shape[2]
        cache_bf16 = is_bf16(k_pool)
    q_out = torch.empty((T, n_heads * head_dim), dtype=q_dtype, device=qkv.device)
    if n_kv_in == 0:
        cache_bf16 = is_bf16(q_out)
    lib.call("fwb_qk_norm_rope_ordered", ptr(qkv), is_bf16(qkv), ptr(q_norm if use_norm == 1 else None),
             ptr(k_norm if use_norm == 1 else None), ptr(table),
             ptr(positions), ptr(tok_seg), ptr(block_table), max_pages, page_size, ptr(q_out),
             is_bf16(q_out), ptr(k_pool), ptr(v_pool), cache_bf16, T, n_heads, n_kv_in, head_dim,
             rotary_dim, c_float(eps), use_norm, pairing_code, int(norm_dim), c_longlong(qkv.stride(0) if T > 1 else width),
             ptr(bias), ptr(temp), ptr(value_table) if value_rotary else None, int(value_rotary), stream())
    return q_out


def attention_simt(q: torch.Tensor, k_pool: torch.Tensor, v_pool: torch.Tensor,
                   positions: torch.Tensor, tok_seg: torch.Tensor, block_table: torch.Tensor,
                   n_heads: int, window: int, scale: float, out_dtype: torch.dtype,
                   sink: Optional[torch.Tensor] = None, softcap: float = 0.0, keep_first: int = 0) -> torch.Tensor:
    """Causal GQA over the paged cache, SIMT fp32 arithmetic.  q: [T][nh*hd].  ``sink``: fp32 [nh], a
    score per head that joins every softmax denominator (not scaled, not capped, without a value);
    ``softcap`` > 0: scores become ``softcap * tanh(score / softcap)`` behind the scale; ``keep_first`` > 0
    (with a sliding window): the sequence's first that many positions stay visible."""
    check_tensor("q", q)
    check_tensor("k pool", k_pool)
    check_tensor("v pool", v_pool, k_pool.dtype, k_pool.shape)
    T = q.shape[0]
    _, n_kv, page_size, head_dim = k_pool.shape
    if q.shape[1] != n_heads * head_dim:
        raise KernelError(f"q has {q.shape[1]} columns, expected {n_heads * head_dim}")
    _i32("positions", positions, T)
    _i32("tok_seg", tok_seg, T)
    _i32("block table", block_table)
    if sink is not None:
        check_tensor("sink", sink, torch.float32, (n_heads,))
    if softcap < 0:
        raise KernelError("a soft-cap must not be negative")
    out = torch.empty((T, n_heads * head_dim), dtype=out_dtype, device=q.device)
    lib.call("fwb_attention_simt_sink", ptr(q), is_bf16(q), ptr(k_pool), ptr(v_pool), is_bf16(k_pool),
             ptr(positions), ptr(tok_seg), ptr(block_table), block_table.shape[1], page_size,
             ptr(out), is_bf16(out), T, n_heads, n_kv, head_dim, window, c_float(scale), ptr(sink),
             c_float(softcap), int(keep_first), stream())
    return out


def attention_mma_shape_ok(n_heads: int, n_kv: int, head_dim: int, page_size: int) -> bool:
    """Shapes the tensor-core attention kernels take (the SIMT kernel takes the rest)."""
    return (n_heads % n_kv == 0 and n_heads // n_kv <= 16 and 16 <= head_dim <= 128
            and head_dim % 16 == 0 and page_size == 64)


def _sink_and_groups(sink, groups, n_heads: int, n_kv: int):
    """Checks of the two optional arguments of the attention kernels: ``sink`` (fp32 [n_heads]: a score
    per head that joins every softmax denominator, not scaled, without a value) and ``groups`` (query
    heads come in this many groups, each reading pool head ``group * n_kv // groups``: more groups
    than pool heads when many query heads share one cached row)."""
    if sink is not None:
        check_tensor("sink", sink, torch.float32, (n_heads,))
    groups = n_kv if groups is None else int(groups)
    if groups < n_kv or groups % n_kv or n_heads % groups:
        raise KernelError(f"{n_heads} query heads in {groups} groups over {n_kv} pool heads")
    return groups


def attention_prefill_mma(q, k_pool, v_pool, positions, seg_start, tile_seg, tile_tok0, n_tiles,
                          tokens_per_tile, block_table, n_heads, window, scale, out=None,
                          sink=None, groups=None, softcap: float = 0.0, keep_first: int = 0) -> torch.Tensor:
    """Causal GQA of prompt portions (any mix of segments) on tensor cores; all bf16.  Only the
    rows of the given tiles are written (``out``: a tensor like q that other rows already live in).
    ``v_pool`` may be ``k_pool`` itself; ``sink``, ``groups``: see ``_sink_and_groups``; ``softcap`` > 0:
    scores become ``softcap * tanh(score / softcap)`` behind the scale."""
    check_tensor("q", q, torch.bfloat16)
    check_tensor("k pool", k_pool, torch.bfloat16)
    check_tensor("v pool", v_pool, torch.bfloat16, k_pool.shape)
    T = q.shape[0]
    _, n_kv, page_size, head_dim = k_pool.shape
    if q.shape[1] != n_heads * head_dim:
        raise KernelError(f"q has {q.shape[1]} columns, expected {n_heads * head_dim}")
    _i32("positions", positions, T)
    _i32("seg_start", seg_start)
    _i32("tile_seg", tile_seg, n_tiles)
    _i32("tile_tok0", tile_tok0, n_tiles)
    _i32("block table", block_table)
    if out is None:
        out = torch.empty_like(q)
    else:
        check_tensor("attention output", out, torch.bfloat16, q.shape)
    groups = _sink_and_groups(sink, groups, n_heads, n_kv)
    lib.call("fwb_attention_prefill_mma_capped", ptr(q), ptr(k_pool), ptr(v_pool), ptr(positions),
             ptr(seg_start), ptr(tile_seg), ptr(tile_tok0), ptr(block_table), block_table.shape[1],
             page_size, ptr(out), n_tiles, n_heads, groups, head_dim, tokens_per_tile, window,
             c_float(scale), ptr(sink), n_kv, c_float(softcap), int(keep_first), stream())
    return out


def attention_tcgen05_shape_ok(n_heads: int, n_kv: int, head_dim: int, page_size: int) -> bool:
    """Shapes the tcgen05 prompt kernel takes: head sizes 64 and 128, up to 128 rows per KV head."""
    return (head_dim in (64, 128) and page_size == 64 and n_kv > 0 and n_heads % n_kv == 0
            and n_heads // n_kv <= 128)


def attention_prefill_tcgen05(q, k_pool, v_pool, positions, seg_start, tile_seg, tile_tok0, n_tiles,
                              tokens_per_tile, block_table, n_heads, window, scale, out=None,
                              sink=None, softcap: float = 0.0, keep_first: int = 0) -> torch.Tensor:
    """The same operation on tcgen05 tensor cores: 128 query rows per CTA, S and PV in tensor
    memory (head sizes 64 and 128); all bf16."""
    check_tensor("q", q, torch.bfloat16)
    check_tensor("k pool", k_pool, torch.bfloat16)
    check_tensor("v pool", v_pool, torch.bfloat16, k_pool.shape)
    T = q.shape[0]
    num_pages, n_kv, page_size, head_dim = k_pool.shape
    if q.shape[1] != n_heads * head_dim:
        raise KernelError(f"q has {q.shape[1]} columns, expected {n_heads * head_dim}")
    _i32("positions", positions, T)
    _i32("seg_start", seg_start)
    _i32("tile_seg", tile_seg, n_tiles)
    _i32("tile_tok0", tile_tok0, n_tiles)
    _i32("block table", block_table)
    if out is None:
        out = torch.empty_like(q)
    else:
        check_tensor("attention output", out, torch.bfloat16, q.shape)
    _sink_and_groups(sink, None, n_heads, n_kv)
    lib.call("fwb_attention_prefill_tcgen05_capped", ptr(q), ptr(k_pool), ptr(v_pool), ptr(positions),
             ptr(seg_start), ptr(tile_seg), ptr(tile_tok0), ptr(block_table), block_table.shape[1],
             page_size, num_pages, ptr(out), n_tiles, n_heads, n_kv, head_dim, tokens_per_tile, window,
             c_float(scale), ptr(sink), c_float(softcap), int(keep_first), stream())
    return out


def attention_decode_fused(qkv, q_norm, k_norm, table, rotary_dim: int, eps: float, pairing: str, n_kv_in: int,
                           k_pool, v_pool, positions, tok_seg, block_table, n_heads: int, window: int,
                           scale: float, splits: int, tiles_per_split: int, merge_in_cluster: bool = False
                           ) -> torch.Tensor:
    """``qk_norm_rope`` and ``attention_decode_mma`` of a step of single tokens in one kernel: every
    CTA of the attention norms and turns the queries of its KV head's group itself, and the slice that
    holds a token's own position its key (and copies its value) into the pages.  ``qkv`` is the fused
    projection [T][(n_heads + 2 n_kv_in) head_dim] in bfloat16; the other arguments are those of the two
    functions.  The same bits as the two kernels (one device function does the arithmetic of both)."""
    pairing_code = ROPE_PAIRINGS[pairing]
    check_tensor("qkv", qkv, torch.bfloat16)
    check_tensor("k pool", k_pool, torch.bfloat16)
    check_tensor("v pool", v_pool, torch.bfloat16, k_pool.shape)
    check_tensor("rope table", table, torch.float32)
    T = qkv.shape[0]
    num_pages, n_kv, page_size, head_dim = k_pool.shape
    if qkv.shape[1] != (n_heads + 2 * n_kv_in) * head_dim:
        raise KernelError(f"qkv has {qkv.shape[1]} columns, expected {(n_heads + 2 * n_kv_in) * head_dim}")
    if table.dim() != 3 or table.shape[1] != max(1, rotary_dim // 2) or table.shape[2] != 2:
        raise KernelError("rope table must be [positions][rotary_dim/2][2]")
    use_norm = 1 if q_norm is not None else 0
    if use_norm:
        check_tensor("q norm weight", q_norm, torch.float32, (head_dim,))
        if n_kv_in:
            check_tensor("k norm weight", k_norm, torch.float32, (head_dim,))
    _i32("positions", positions, T)
    _i32("tok_seg", tok_seg, T)
    _i32("block table", block_table)
    out = torch.empty((T, n_heads * head_dim), dtype=torch.bfloat16, device=qkv.device)
    part_o = part_ml = None
    in_cluster = merge_in_cluster and 1 < splits <= 8
    if splits > 1 and not in_cluster:
        group = n_heads // n_kv
        part_o = torch.empty((T, n_kv, splits, group, head_dim), dtype=torch.float32, device=qkv.device)
        part_ml = torch.empty((T, n_kv, splits, group, 2), dtype=torch.float32, device=qkv.device)
    lib.call("fwb_attention_decode_fused", ptr(qkv), n_kv_in, ptr(q_norm), ptr(k_norm), ptr(table), rotary_dim,
             c_float(eps), use_norm, pairing_code, ptr(k_pool), ptr(v_pool), ptr(positions), ptr(tok_seg),
             ptr(block_table), block_table.shape[1], page_size, num_pages, ptr(out), ptr(part_o), ptr(part_ml),
             T, n_heads, n_kv, head_dim, splits, tiles_per_split, window, c_float(scale),
             1 if in_cluster else 0, stream(), launches=2 if (splits > 1 and not in_cluster) else 1)
    return out


def set_decode_attention_tma(on: bool, stages: int = 0) -> None:
    """Test switch: whether the decode attention kernel takes its key and value tiles by TMA at head
    sizes 64 and 128 (the default) or by cp.async, as at the other head sizes; and the depth of the TMA
    way's ring (2 to 8; 0: the launcher's choice).  The same bits."""
    lib.call("fwb_attention_decode_set_tma", 1 if on else 0, int(stages))


def attention_decode_mma(q, k_pool, v_pool, positions, tok_seg, block_table, n_heads, window, scale,
                         splits: int, tiles_per_split: int, merge_in_cluster: bool = False,
                         out=None, n_tokens=None, sink=None, groups=None, softcap: float = 0.0,
                         keep_first: int = 0) -> torch.Tensor:
    """Causal GQA of single decode tokens on tensor cores, the context cut into ``splits``
    slices of ``tiles_per_split`` 64-key tiles that run as separate CTAs and are merged: inside
    the kernel (``merge_in_cluster``, up to 8 slices as a thread-block cluster) or through scratch
    and a second kernel.  ``n_tokens``: only the first that many rows of q are decode tokens (the
    head of a mixed step); the other rows of ``out`` are left alone."""
    check_tensor("q", q, torch.bfloat16)
    check_tensor("k pool", k_pool, torch.bfloat16)
    check_tensor("v pool", v_pool, torch.bfloat16, k_pool.shape)
    T = q.shape[0] if n_tokens is None else int(n_tokens)
    if not 0 < T <= q.shape[0]:
        raise KernelError(f"{T} decode tokens of {q.shape[0]} rows")
    _, n_kv, page_size, head_dim = k_pool.shape
    if q.shape[1] != n_heads * head_dim:
        raise KernelError(f"q has {q.shape[1]} columns, expected {n_heads * head_dim}")
    _i32("positions", positions, T)
    _i32("tok_seg", tok_seg, T)
    _i32("block table", block_table)
    if out is None:
        out = torch.empty_like(q)
    else:
        check_tensor("attention output", out, torch.bfloat16, q.shape)
    part_o = part_ml = None
    in_cluster = merge_in_cluster and 1 < splits <= 8
    groups = _sink_and_groups(sink, groups, n_heads, n_kv)
    if splits > 1 and not in_cluster:
        group = n_heads // groups
        part_o = torch.empty((T, groups, splits, group, head_dim), dtype=torch.float32, device=q.device)
        part_ml = torch.empty((T, groups, splits, group, 2), dtype=torch.float32, device=q.device)
    lib.call("fwb_attention_decode_mma_capped", ptr(q), ptr(k_pool), ptr(v_pool), ptr(positions),
             ptr(tok_seg), ptr(block_table), block_table.shape[1], page_size, k_pool.shape[0], ptr(out), ptr(part_o),
             ptr(part_ml), T, n_heads, groups, head_dim, splits, tiles_per_split, window,
             c_float(scale), 1 if in_cluster else 0, ptr(sink), n_kv, c_float(softcap), int(keep_first), stream(),
             launches=2 if (splits > 1 and not in_cluster) else 1)
    return out
