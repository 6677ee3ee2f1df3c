"""Tensor-level wrappers over the C ABI: validate, pass raw pointers, launch on torch's current stream.

PyTorch is used for device memory and streams only; all arithmetic of the cache path runs in the
CUDA kernels of libtrimkv_b200.so.
"""
from __future__ import annotations

from typing import Optional

import torch

from . import _lib
from ._lib import TKV_BF16, TKV_F16, TKV_F32, check, lib

_DTYPE = {torch.bfloat16: TKV_BF16, torch.float16: TKV_F16, torch.float32: TKV_F32}


def dtype_code(dt: torch.dtype) -> int:
    try:
        return _DTYPE[dt]
    except KeyError:
        raise TypeError(f"unsupported dtype {dt}") from None


def _stream(t: torch.Tensor) -> int:
    if not t.is_cuda:
        raise _lib.TrimKVNativeError("trimkv_b200 runs on CUDA tensors only (no CPU path)")
    return torch.cuda.current_stream(t.device).cuda_stream


def _ptr(t: Optional[torch.Tensor]) -> Optional[int]:
    return None if t is None else t.data_ptr()


# Kernels launched through this module since import (the benchmark reports the delta of a timed region).
launch_count = 0


def _count(n: int) -> None:
    global launch_count
    launch_count += n


def new_status(device) -> torch.Tensor:
    return torch.zeros(1, dtype=torch.int32, device=device)


def read_status(status: torch.Tensor) -> int:
    """Synchronises the current stream and returns (then clears) the device status word."""
    return lib().tkv_read_status(status.data_ptr(), _stream(status))


def append(k_cache, v_cache, beta_cache, pos_cache, seg_len, cu_seqlens,
           k_new, v_new, beta_new, pos_new, cap: int, status=None) -> None:
    """In-place append of ``k_new/v_new [B,H,S,D]``, ``beta_new [B,H,S]``, ``pos_new`` int64 ``[S]`` or ``[B,H,S]``."""
    b, h, s, d = k_new.shape
    if v_new.shape != k_new.shape or v_new.stride() != k_new.stride():
        v_new = v_new.contiguous(); k_new = k_new.contiguous()
    if k_new.stride(3) != 1:
        k_new = k_new.contiguous(); v_new = v_new.contiguous()
    if pos_new.dtype != torch.int64:
        pos_new = pos_new.to(torch.int64)
    if pos_new.dim() == 1:
        ps = (0, 0, pos_new.stride(0))
    else:
        pos_new = pos_new.expand(b, h, s)
        ps = pos_new.stride()
    if beta_new.shape != (b, h, s):
        raise ValueError(f"retention weights {tuple(beta_new.shape)} do not match keys {tuple(k_new.shape)}")
    rc = lib().tkv_append(
        k_cache.data_ptr(), v_cache.data_ptr(), beta_cache.data_ptr(), pos_cache.data_ptr(),
        seg_len.data_ptr(), _ptr(cu_seqlens),
        k_new.data_ptr(), v_new.data_ptr(), k_new.stride(0), k_new.stride(1), k_new.stride(2),
        beta_new.data_ptr(), dtype_code(beta_new.dtype), beta_new.stride(0), beta_new.stride(1), beta_new.stride(2),
        pos_new.data_ptr(), ps[0], ps[1], ps[2],
        b, h, s, d, cap, dtype_code(k_cache.dtype), _ptr(status), _stream(k_cache))
    check(rc, "tkv_append")
    _count(1 if s <= 8 else 2)


def evict(k_cache, v_cache, beta_cache, pos_cache, seg_len, cu_seqlens, group: int, nseg: int, cap: int,
          q_idx: int, memory_size: int, trigger_len: int, max_len: int, kept_idx_out=None, status=None) -> None:
    d = k_cache.shape[-1]
    rc = lib().tkv_evict(
        k_cache.data_ptr(), v_cache.data_ptr(), beta_cache.data_ptr(), pos_cache.data_ptr(),
        seg_len.data_ptr(), _ptr(cu_seqlens), group, nseg, cap, d, dtype_code(k_cache.dtype), q_idx,
        memory_size, trigger_len, max_len, _ptr(kept_idx_out), _ptr(status), _stream(k_cache))
    check(rc, "tkv_evict")
    _count(1 if cu_seqlens is None else 2)


def evict_select(beta, pos, seg_len, n_uniform: int, nseg: int, q_idx: int, memory_size: int,
                 trigger_len: int, max_len: int, kept_idx, kept_cnt, status=None) -> None:
    """beta f32 ``[nseg, n]`` (row stride taken from the tensor); pos i32 ``[nseg, n]`` or ``[n]`` (shared)."""
    if beta.dtype != torch.float32 or pos.dtype != torch.int32:
        raise TypeError("evict_select wants f32 log beta and i32 positions")
    pos_stride = 0 if pos.dim() == 1 else pos.stride(0)
    rc = lib().tkv_evict_select(
        beta.data_ptr(), beta.stride(0), pos.data_ptr(), pos_stride, _ptr(seg_len), n_uniform, nseg, q_idx,
        memory_size, trigger_len, max_len, kept_idx.data_ptr(), kept_cnt.data_ptr(), _ptr(status), _stream(beta))
    check(rc, "tkv_evict_select")
    _count(1)


def compact(k_dst, v_dst, beta_dst, pos_dst, cap: int, k_src, v_src, beta_src, pos_src, kept_idx, kept_cnt,
            seg_len, cu_seqlens, group: int, status=None) -> None:
    """Gather rows of dense ``k_src/v_src [B,H,n,D]`` listed in ``kept_idx [B*H, M]`` into a strided cache."""
    b, h, n, d = k_src.shape
    if v_src.stride() != k_src.stride() or k_src.stride(3) != 1:
        k_src = k_src.contiguous(); v_src = v_src.contiguous()
    pos_stride = 0 if pos_src.dim() == 1 else pos_src.stride(0)
    rc = lib().tkv_compact(
        k_dst.data_ptr(), v_dst.data_ptr(), beta_dst.data_ptr(), pos_dst.data_ptr(), cap,
        k_src.data_ptr(), v_src.data_ptr(), k_src.stride(0), k_src.stride(1), k_src.stride(2),
        beta_src.data_ptr(), beta_src.stride(0), pos_src.data_ptr(), pos_stride,
        _ptr(kept_idx), 0 if kept_idx is None else kept_idx.stride(0), _ptr(kept_cnt),
        seg_len.data_ptr(), _ptr(cu_seqlens), group, b, h, n, d, dtype_code(k_dst.dtype),
        _ptr(status), _stream(k_dst))
    check(rc, "tkv_compact")
    _count(1 if cu_seqlens is None else 2)


def rebuild_cu_seqlens(seg_len, cu_seqlens, nseg: int, group: int) -> None:
    check(lib().tkv_rebuild_cu_seqlens(seg_len.data_ptr(), cu_seqlens.data_ptr(), nseg, group, _stream(seg_len)),
          "tkv_rebuild_cu_seqlens")


def decode_attn_workspace_bytes(batch: int, hq: int, hkv: int, head_dim: int, max_len: int) -> int:
    return int(lib().tkv_decode_attn_workspace_bytes(batch, hq, hkv, head_dim, max_len))


def decode_attn_workspace_bytes_ragged(batch: int, hq: int, hkv: int, head_dim: int, max_len: int,
                                       total_len_bound: int) -> int:
    return int(lib().tkv_decode_attn_ragged_workspace_bytes(batch, hq, hkv, head_dim, max_len, total_len_bound))


def decode_attn(q, k_cache, v_cache, seg_len, seg_start, cap: int, out, workspace, hkv: int, scale: float,
                max_len: int, status=None, total_len_bound=None, packed_rows=None) -> None:
    """q ``[B,Hq,D]`` (any batch/head strides), out ``[B,Hq,D]`` contiguous, workspace uint8.
    ``total_len_bound``: host-known bound on ``seg_len.sum()`` for ragged lengths (sizes the grid by tokens instead of
    by ``max_len``); the workspace must then have ``decode_attn_workspace_bytes_ragged`` bytes.
    With ``seg_start`` (packed ``[sum n, D]`` K/V) the C entry point takes the packed row count in place of ``cap``:
    ``packed_rows`` (default: the K tensor's first dimension; 0 = not stated, which selects the CUDA-core kernel)."""
    b, hq, d = q.shape
    if q.stride(2) != 1:
        q = q.contiguous()
    if seg_start is not None:
        cap = int(packed_rows) if packed_rows is not None else (k_cache.shape[0] if k_cache.dim() == 2 else 0)
    if total_len_bound is not None:
        rc = lib().tkv_decode_attn_ragged(
            q.data_ptr(), q.stride(0), q.stride(1), k_cache.data_ptr(), v_cache.data_ptr(),
            seg_len.data_ptr(), _ptr(seg_start), cap, out.data_ptr(), workspace.data_ptr(), workspace.numel(),
            b, hq, hkv, d, dtype_code(k_cache.dtype), float(scale), max_len, int(total_len_bound), _ptr(status), _stream(q))
        check(rc, "tkv_decode_attn_ragged")
        _count(3)
        return
    rc = lib().tkv_decode_attn(
        q.data_ptr(), q.stride(0), q.stride(1), k_cache.data_ptr(), v_cache.data_ptr(),
        seg_len.data_ptr(), _ptr(seg_start), cap, out.data_ptr(), workspace.data_ptr(), workspace.numel(),
        b, hq, hkv, d, dtype_code(k_cache.dtype), float(scale), max_len, _ptr(status), _stream(q))
    check(rc, "tkv_decode_attn")
    _count(2)


def decode_attn_multi(q, k_cache, v_cache, seg_len, cap: int, out, hkv: int, scale: float, max_len: int,
                      workspace=None, status=None):
    """q ``[B,Q,Hq,D]`` (any batch/token/head strides) against caches that already hold the Q new tokens; out
    ``[B,Q,Hq,D]`` contiguous; bottom-right aligned causal mask per segment."""
    b, ql, hq, d = q.shape
    if q.stride(3) != 1:
        q = q.contiguous()
    if workspace is None:
        workspace = torch.empty(lib().tkv_decode_attn_multi_workspace_bytes(b, hq, hkv, d, max_len, ql), dtype=torch.uint8,
                                device=q.device)
    rc = lib().tkv_decode_attn_multi(
        q.data_ptr(), q.stride(0), q.stride(1), q.stride(2), k_cache.data_ptr(), v_cache.data_ptr(), seg_len.data_ptr(), cap,
        out.data_ptr(), workspace.data_ptr(), workspace.numel(), b, hq, hkv, d, dtype_code(k_cache.dtype), float(scale),
        max_len, ql, _ptr(status), _stream(q))
    check(rc, "tkv_decode_attn_multi")
    _count(2)


def prefill_attn(q, k_cache, v_cache, seg_len, cap: int, out, hkv: int, scale: float, max_len: int, status=None):
    """q ``[B,Q,Hq,D]`` (any batch/token/head strides) against capacity-strided caches that already hold the Q new
    tokens (``seg_len`` None: every segment holds ``max_len`` tokens, e.g. a dense prompt with ``cap`` = S); out
    ``[B,Q,Hq,D]`` contiguous; bottom-right aligned causal mask per segment.  Query-resident kernel, no workspace."""
    b, ql, hq, d = q.shape
    if q.stride(3) != 1:
        q = q.contiguous()
    rc = lib().tkv_prefill_attn(
        q.data_ptr(), q.stride(0), q.stride(1), q.stride(2), k_cache.data_ptr(), v_cache.data_ptr(), _ptr(seg_len), cap,
        out.data_ptr(), b, hq, hkv, d, dtype_code(k_cache.dtype), float(scale), max_len, ql, _ptr(status), _stream(q))
    check(rc, "tkv_prefill_attn")
    _count(1)


def decode_attn_push(q, k_cache, v_cache, seg_len, cap: int, out, workspace, hkv: int, scale: float, max_len: int,
                     peer_out, peer_flags, world: int, rank: int, row_stride: int, col_offset: int, sync_state,
                     status=None) -> None:
    """:func:`decode_attn` whose merge step stores into every rank's gathered buffer and raises this rank's flag on
    the peers.  ``peer_out`` / ``peer_flags``: ``ctypes`` arrays of ``world`` device pointers."""
    b, hq, d = q.shape
    if q.stride(2) != 1:
        q = q.contiguous()
    rc = lib().tkv_decode_attn_push(
        q.data_ptr(), q.stride(0), q.stride(1), k_cache.data_ptr(), v_cache.data_ptr(),
        seg_len.data_ptr(), None, cap, out.data_ptr(), workspace.data_ptr(), workspace.numel(),
        b, hq, hkv, d, dtype_code(k_cache.dtype), float(scale), max_len,
        peer_out, peer_flags, world, rank, row_stride, col_offset, sync_state.data_ptr(), _ptr(status), _stream(q))
    check(rc, "tkv_decode_attn_push")
    _count(2)


def enable_peer_access(peer_device: int) -> None:
    check(lib().tkv_enable_peer_access(int(peer_device)), "tkv_enable_peer_access")


def ipc_export(t: torch.Tensor):
    """``(handle bytes, offset)`` under which other rank processes of this box can map ``t``'s allocation."""
    import ctypes
    handle, off = ctypes.create_string_buffer(64), ctypes.c_int64(0)
    check(lib().tkv_ipc_export(t.data_ptr(), handle, ctypes.byref(off)), "tkv_ipc_export")
    return handle.raw, int(off.value)


_ipc_bases = {}   # (device, handle) -> [base address, users]: an allocation is mapped once per process and device


def ipc_import(handle: bytes) -> int:
    """Maps an exported allocation with the current device; returns its base address in this process.  A handle that
    is already mapped is not opened again (one mapping per handle and process); ``ipc_release`` undoes one import."""
    import ctypes
    key = (torch.cuda.current_device(), handle)
    if key not in _ipc_bases:
        base = ctypes.c_void_p(0)
        check(lib().tkv_ipc_import(ctypes.create_string_buffer(handle, 64), ctypes.byref(base)), "tkv_ipc_import")
        _ipc_bases[key] = [int(base.value), 0]
    _ipc_bases[key][1] += 1
    return _ipc_bases[key][0]


def ipc_release(handle: bytes) -> None:
    """Drops one user of an imported allocation; the mapping is closed when the last one is gone."""
    import ctypes
    key = (torch.cuda.current_device(), handle)
    entry = _ipc_bases.get(key)
    if entry is None:
        return
    entry[1] -= 1
    if entry[1] <= 0:
        del _ipc_bases[key]
        check(lib().tkv_ipc_close(ctypes.c_void_p(entry[0])), "tkv_ipc_close")


def peer_wait(flags, sync_state, world: int, rank: int, status=None, max_polls: int = 0) -> None:
    """Holds the stream until every peer has raised its flag for this rank's next exchange.  Bounded: after
    ``max_polls`` polls (default about four seconds) the status word reports a timeout and the stream carries on."""
    rc = lib().tkv_peer_wait(flags.data_ptr(), sync_state.data_ptr(), world, rank, max_polls, _ptr(status), _stream(flags))
    check(rc, "tkv_peer_wait")
    _count(1)


def decode_prep(qkvg, q_norm_w, k_norm_w, eps: float, cos, sin, gate_w2, gate_bias, pos, q_out,
                k_cache, v_cache, beta_cache, pos_cache, seg_len, cu_seqlens, cap: int, hq: int, hkv: int,
                status=None, in_splits: int = 0, in_bias=None) -> None:
    """Fused q/k-norm + RoPE + retention-gate tail + append for one new token per request (head_dim 128).
    ``q_norm_w`` / ``k_norm_w`` are both None for families without a per-head norm (Llama, Phi-3).
    ``qkvg`` is ``[B, cols]`` in the model dtype, or (``in_splits`` > 0) the fp32 ``[splits, B, cols]`` of skinny_gemm."""
    b, cols = qkvg.shape[-2], qkvg.shape[-1]
    rc = lib().tkv_decode_prep(
        qkvg.data_ptr(), cols if in_splits else qkvg.stride(0), _ptr(q_norm_w), _ptr(k_norm_w), float(eps),
        cos.data_ptr(), sin.data_ptr(), gate_w2.data_ptr(), gate_bias.data_ptr(), gate_w2.shape[1],
        pos.data_ptr(), q_out.data_ptr(), k_cache.data_ptr(), v_cache.data_ptr(), beta_cache.data_ptr(),
        pos_cache.data_ptr(), seg_len.data_ptr(), _ptr(cu_seqlens), cap, b, hq, hkv, 128,
        dtype_code(q_out.dtype), in_splits, _ptr(in_bias), _ptr(status), _stream(qkvg))
    check(rc, "tkv_decode_prep")
    _count(1)


def add_rmsnorm(residual, delta, weight, out, eps: float, in_splits: int = 0, in_bias=None) -> None:
    rows, cols = residual.shape
    rc = lib().tkv_add_rmsnorm(residual.data_ptr(), _ptr(delta), weight.data_ptr(), out.data_ptr(), rows, cols,
                               float(eps), dtype_code(residual.dtype), in_splits, _ptr(in_bias), _stream(residual))
    check(rc, "tkv_add_rmsnorm")
    _count(1)


def silu_mul(gate_up, out, in_splits: int = 0, in_bias=None) -> None:
    rows, two_inter = gate_up.shape[-2], gate_up.shape[-1]
    rc = lib().tkv_silu_mul(gate_up.data_ptr(), out.data_ptr(), rows, two_inter // 2, dtype_code(out.dtype),
                            in_splits, _ptr(in_bias), _stream(gate_up))
    check(rc, "tkv_silu_mul")
    _count(1)


def skinny_gemm_splits(m: int, n: int, k: int) -> int:
    """Number of fp32 partial sums tkv_skinny_gemm produces for this shape; 0 = shape not supported."""
    return int(lib().tkv_skinny_gemm_splits(m, n, k))


def skinny_gemm(x, w, partial, status=None) -> int:
    """``partial [splits, M, N]`` fp32 with ``sum(partial, 0) == x [M, K] @ w [N, K].T``; returns ``splits``."""
    m, k = x.shape
    n = w.shape[0]
    if not (x.is_contiguous() and w.is_contiguous() and partial.is_contiguous() and partial.dtype == torch.float32):
        raise ValueError("skinny_gemm wants contiguous x, w and an fp32 contiguous partial buffer")
    rc = lib().tkv_skinny_gemm(x.data_ptr(), w.data_ptr(), partial.data_ptr(), m, n, k, dtype_code(x.dtype),
                               _ptr(status), _stream(x))
    check(rc, "tkv_skinny_gemm")
    _count(1)
    return skinny_gemm_splits(m, n, k)


def skinny_gemm_swiglu(gate_up, w, partial, status=None) -> int:
    """:func:`skinny_gemm` over ``x = SiLU(gate_up[:, :K]) * gate_up[:, K:]`` computed inside the kernel
    (``gate_up [M, 2K]``, ``w [N, K]``): the MLP's activation and down projection in one launch."""
    m, two_k = gate_up.shape
    n, k = w.shape
    if two_k != 2 * k:
        raise ValueError(f"gate_up has {two_k} columns, the weight wants 2 x {k}")
    if not (gate_up.is_contiguous() and w.is_contiguous() and partial.is_contiguous() and partial.dtype == torch.float32):
        raise ValueError("skinny_gemm_swiglu wants contiguous gate_up, w and an fp32 contiguous partial buffer")
    rc = lib().tkv_skinny_gemm_swiglu(gate_up.data_ptr(), w.data_ptr(), partial.data_ptr(), m, n, k,
                                      dtype_code(gate_up.dtype), _ptr(status), _stream(gate_up))
    check(rc, "tkv_skinny_gemm_swiglu")
    _count(1)
    return skinny_gemm_splits(m, n, k)


def evict_ex(k_cache, v_cache, beta_cache, pos_cache, seg_len, cu_seqlens, group: int, nseg: int, cap: int,
             q_idx: int, max_len: int, keep_cnt, protect_last: int = 0, memory_size: int = 1, trigger_len: int = 0,
             kept_idx_out=None, kept_stride: int = 0, status=None, knorm: bool = False, score_dtype: int = 0,
             scores=None) -> None:
    """In-place eviction with a keep count per segment (``keep_cnt`` int32 ``[nseg]``) and/or a protected tail.
    ``score_dtype``: 0 fp32, 1 bf16, 2 f16 (the dtype the retention score is computed in)."""
    d = k_cache.shape[-1]
    rc = lib().tkv_evict_ex(
        k_cache.data_ptr(), v_cache.data_ptr(), beta_cache.data_ptr(), pos_cache.data_ptr(),
        seg_len.data_ptr(), _ptr(cu_seqlens), group, nseg, cap, d, dtype_code(k_cache.dtype), q_idx,
        memory_size, trigger_len, max_len, _ptr(keep_cnt), protect_last, kept_stride,
        (1 if knorm else 0) | (score_dtype << 8), _ptr(scores), _ptr(kept_idx_out),
        _ptr(status), _stream(k_cache))
    check(rc, "tkv_evict_ex")
    _count(1 if cu_seqlens is None else 2)


def evict_multi_workspace(nseg: int, memory_size: int, ctas_per_segment: int, device) -> torch.Tensor:
    """Scratch for :func:`evict_multi` (contents irrelevant between calls; one stream at a time)."""
    nbytes = lib().tkv_evict_multi_workspace_bytes(nseg, memory_size, ctas_per_segment)
    return torch.empty(max(nbytes, 4) // 4, dtype=torch.int32, device=device)


def evict_multi(k_cache, v_cache, beta_cache, pos_cache, seg_len, cu_seqlens, group: int, nseg: int, cap: int,
                q_idx: int, memory_size: int, trigger_len: int, max_len: int, ctas_per_segment: int, workspace,
                protect_last: int = 0, knorm: bool = False, kept_idx_out=None, status=None) -> None:
    """:func:`evict` with ``ctas_per_segment`` CTAs sharing each evicting segment (identical result)."""
    d = k_cache.shape[-1]
    rc = lib().tkv_evict_multi(
        k_cache.data_ptr(), v_cache.data_ptr(), beta_cache.data_ptr(), pos_cache.data_ptr(),
        seg_len.data_ptr(), _ptr(cu_seqlens), group, nseg, cap, d, dtype_code(k_cache.dtype), q_idx,
        memory_size, trigger_len, max_len, protect_last, 1 if knorm else 0, ctas_per_segment,
        _ptr(workspace), 0 if workspace is None else workspace.numel() * workspace.element_size(),
        _ptr(kept_idx_out), _ptr(status), _stream(k_cache))
    check(rc, "tkv_evict_multi")
    n = 1 if ctas_per_segment <= 1 else 2
    _count(n if cu_seqlens is None else n + 1)


def flat_scores(k_cache, beta_cache, pos_cache, seg_len, nseg: int, cap: int, q_idx: int, max_len: int, scores_out,
                knorm: bool = True, score_dtype: int = 0) -> None:
    """Scores of every live row (fp32 array of ``nseg*cap``) for the strategies that read K ("knorm_alpha" on the
    flat caches: the norm is clamped at 1e-12 as the reference does there)."""
    rc = lib().tkv_flat_scores(k_cache.data_ptr(), beta_cache.data_ptr(), pos_cache.data_ptr(), seg_len.data_ptr(),
                               nseg, cap, k_cache.shape[-1], dtype_code(k_cache.dtype), q_idx,
                               (2 if knorm else 0) | (score_dtype << 8), max_len, scores_out.data_ptr(),
                               _stream(k_cache))
    check(rc, "tkv_flat_scores")
    _count(1)


def group_budget(beta_cache, pos_cache, seg_len, cap: int, groups: int, inner: int, n_outer: int, outer_stride: int,
                 q_idx: int, k_total: int, keep_cnt, threshold=None, floor_mode: int = 0, floor_cnt: int = 0,
                 status=None, score_dtype: int = 0, scores=None) -> None:
    """Per-segment keep counts when ``k_total`` rows (or all rows scoring >= ``threshold``) are kept per group."""
    rc = lib().tkv_group_budget(
        beta_cache.data_ptr(), pos_cache.data_ptr(), seg_len.data_ptr(), cap, groups, inner, n_outer, outer_stride,
        q_idx, k_total, 0 if threshold is None else 1, 0.0 if threshold is None else float(threshold),
        floor_mode, floor_cnt, score_dtype, _ptr(scores), keep_cnt.data_ptr(), _ptr(status), _stream(beta_cache))
    check(rc, "tkv_group_budget")
    _count(1)


def update_flatten_view(cache: torch.Tensor, state: torch.Tensor, headlens: torch.Tensor,
                        cu_headlens: torch.Tensor) -> torch.Tensor:
    """Functional packed append with the contract of the reference's ``update_flatten_view_triton``
    (src/trimkv/triton/db_cache_utils.py:86-186): ``cache [origin_len, D]`` + ``state [1, H, S, D]`` ->
    ``out [origin_len + H*S, D]``; same argument checks, no host synchronisation."""
    assert cache.is_cuda and state.is_cuda, "Tensors must be on CUDA device"
    assert headlens.is_cuda and cu_headlens.is_cuda, "Index tensors must be on CUDA"
    assert headlens.dtype == torch.int32, "headlens must be int32"
    assert cu_headlens.dtype == torch.int32, "cu_headlens must be int32"
    assert cache.dtype == state.dtype, "cache/state dtypes must match"
    assert cache.is_contiguous(), "cache must be contiguous [origin_len, D]"
    assert headlens.is_contiguous() and cu_headlens.is_contiguous(), "index tensors must be contiguous"
    assert state.ndim == 4, "state must be [B, H, state_len, D]"
    b, h, s, d_state = state.shape
    assert b == 1, "This kernel currently assumes B == 1"
    origin_len, d = cache.shape
    assert d == d_state, "cache and state last dim (D) must match"
    assert headlens.shape[0] == h, "headlens must be length H"
    assert cu_headlens.numel() == h + 1, "cu_headlens must be length H+1"
    assert state.is_contiguous(), "state must be contiguous [B, H, state_len, D]"
    out = torch.empty((origin_len + h * s, d), dtype=cache.dtype, device=cache.device)
    rc = lib().tkv_flat_append_packed(cache.data_ptr(), state.data_ptr(), cu_headlens.data_ptr(), out.data_ptr(),
                                      h, s, origin_len, d * cache.element_size(), _stream(cache))
    check(rc, "tkv_flat_append_packed")
    _count(1)
    return out


update_flatten_view_triton = update_flatten_view  # the reference's name for the same operation


# --------------------------------------------------------------------------------------------------------------------
# Decoders with recurrent layers, windowed attention and experts.  ``batch`` is a ``state_cache.StepBatch``: packed
# tokens, ``cu`` (None in a one-token step), ``slots`` and ``pos0`` of the step's requests.

def batch_begin(lens, slots, cu, pos0) -> None:
    check(lib().tkv_batch_begin(lens.data_ptr(), slots.data_ptr(), _ptr(cu), pos0.data_ptr(), slots.shape[0], _stream(lens)),
          "tkv_batch_begin")
    _count(1)


def embed_stream(ids, table, stream, copy, status=None, scale: float = 1.0) -> None:
    check(lib().tkv_embed_stream(ids.data_ptr(), table.data_ptr(), table.shape[0], stream.data_ptr(), _ptr(copy), stream.shape[0],
                                 stream.shape[1], float(scale), dtype_code(table.dtype), _ptr(status), _stream(ids)), "tkv_embed_stream")
    _count(1)


def postnorm_add(stream, y, weight, copy, eps: float, mult: float, weight_offset: float) -> None:
    """``stream += mult * RMSNorm(y) * (weight_offset + weight)`` (fp32, in place); ``copy`` (or None): the sum in y's type."""
    check(lib().tkv_postnorm_add(stream.data_ptr(), y.data_ptr(), weight.data_ptr(), _ptr(copy), stream.shape[0], stream.shape[1],
                                 float(eps), float(mult), float(weight_offset), dtype_code(y.dtype), _stream(stream)),
          "tkv_postnorm_add")
    _count(1)


def gated_sum_norm(stream, y, weight, copy, groups: int, eps: float, alpha: float, gate=None, gate_bias=None, place=None,
                   choice_weight=None) -> None:
    """``stream = GroupRMSNorm(alpha * stream + sigmoid(gate + gate_bias) * y) * weight`` (fp32, in place); ``copy`` (or None):
    the result in y's type.  ``place`` / ``choice_weight`` ``[rows, top]``: y holds expert rows to be gathered and added up
    (place -1: the stream itself)."""
    check(lib().tkv_gated_sum_norm(stream.data_ptr(), y.data_ptr(), _ptr(place), _ptr(choice_weight), 0 if place is None else place.shape[1],
                                   _ptr(gate), 0 if gate is None else gate.stride(0), _ptr(gate_bias), weight.data_ptr(), _ptr(copy),
                                   stream.shape[0], stream.shape[1], groups, float(eps), float(alpha), dtype_code(y.dtype),
                                   _stream(stream)), "tkv_gated_sum_norm")
    _count(1)


def stream_norm(stream, rows, weight, out, eps: float, weight_offset: float, groups: int = 1) -> None:
    """RMS norm of the stream's rows (``rows`` int32, or None: all) into ``out``, in ``groups`` equal parts."""
    check(lib().tkv_stream_norm(stream.data_ptr(), _ptr(rows), weight.data_ptr(), out.data_ptr(), out.shape[0], out.shape[1], groups,
                                float(eps), float(weight_offset), dtype_code(out.dtype), _stream(stream)), "tkv_stream_norm")
    _count(1)


def gated_norm(y, z, weight, out, groups: int, eps: float, gate_first: bool = False) -> None:
    """Group RMS norm with a SiLU gate before (times ``weight``) or after it; ``z`` may be None (no gate) or a column slice of a
    wider array; a ``weight`` of one group's length serves all groups."""
    shared = weight is not None and weight.numel() * groups == out.shape[1] and groups > 1
    check(lib().tkv_gated_norm(y.data_ptr(), y.stride(0), _ptr(z), 0 if z is None else z.stride(0), _ptr(weight), int(shared),
                               out.data_ptr(), out.shape[0], groups, out.shape[1] // groups, float(eps), int(gate_first),
                               dtype_code(out.dtype), _stream(y)), "tkv_gated_norm")
    _count(1)


def swiglu(u, out) -> None:
    """``out = SiLU(u[:, :ff]) * u[:, ff:2 ff]``, ``ff`` the width of ``out``; u may have further columns."""
    check(lib().tkv_swiglu(u.data_ptr(), u.stride(0), out.data_ptr(), out.shape[0], out.shape[1], dtype_code(out.dtype), _stream(u)),
          "tkv_swiglu")
    _count(1)


def gelu_tanh(u) -> None:
    check(lib().tkv_gelu_tanh(u.data_ptr(), u.numel(), dtype_code(u.dtype), _stream(u)), "tkv_gelu_tanh")
    _count(1)


def rotate_qk(proj, out, batch, heads: int, dim: int, rot_dims: int, freq, k_scale: float) -> None:
    check(lib().tkv_rotate_qk(proj.data_ptr(), proj.stride(0), out.data_ptr(), _ptr(batch.cu), batch.pos0.data_ptr(), batch.size,
                              batch.tokens, heads, dim, rot_dims, freq.data_ptr(), float(k_scale), dtype_code(proj.dtype),
                              _stream(proj)), "tkv_rotate_qk")
    _count(1)


def conv_silu(x, ring, weight, bias, out, batch) -> None:
    """``x`` [tokens, channels] is a column slice of the projection; ``ring`` [slots, taps, channels]."""
    check(lib().tkv_conv_silu(x.data_ptr(), x.stride(0), ring.data_ptr(), weight.data_ptr(), bias.data_ptr(), out.data_ptr(),
                              batch.cu.data_ptr(), batch.slots.data_ptr(), batch.pos0.data_ptr(), batch.size, batch.max_tokens,
                              x.shape[1], weight.shape[1], dtype_code(x.dtype), _stream(x)), "tkv_conv_silu")
    _count(2)


def ssd_steps(dt_in, dt_bias, a_log, dt, log_decay) -> None:
    check(lib().tkv_ssd_steps(dt_in.data_ptr(), dt_in.stride(0), dt_bias.data_ptr(), a_log.data_ptr(), dt.data_ptr(),
                              log_decay.data_ptr(), dt.shape[0], dt.shape[1], dtype_code(dt_in.dtype), _stream(dt)), "tkv_ssd_steps")
    _count(1)


def retention_step(proj, state, batch, decay, freq, out, dim: int, rot_dims: int, k_scale: float, eps: float) -> None:
    heads, vdim = state.shape[1], state.shape[3]
    check(lib().tkv_retention_step(proj.data_ptr(), proj.stride(0), state.data_ptr(), batch.slots.data_ptr(), batch.pos0.data_ptr(),
                                   decay.data_ptr(), freq.data_ptr(), out.data_ptr(), batch.size, heads, dim, vdim, rot_dims,
                                   float(k_scale), float(eps), dtype_code(proj.dtype), _stream(proj)), "tkv_retention_step")
    _count(1)


def ssd_step(proj, ring, state, batch, conv_w, conv_b, dt_bias, a_log, skip, out, groups: int) -> None:
    heads, n, vdim = state.shape[1:]
    check(lib().tkv_ssd_step(proj.data_ptr(), proj.stride(0), ring.data_ptr(), state.data_ptr(), batch.slots.data_ptr(),
                             batch.pos0.data_ptr(), conv_w.data_ptr(), conv_b.data_ptr(), dt_bias.data_ptr(), a_log.data_ptr(),
                             skip.data_ptr(), out.data_ptr(), batch.size, heads, groups, n, vdim, conv_w.shape[1],
                             dtype_code(proj.dtype), _stream(proj)), "tkv_ssd_step")
    _count(1)


def linrec(q, k, v, state, batch, out, groups: int, log_decay=None, head_decay=None, head_log_decay=None, v_scale=None,
           skip=None, force_scan: bool = False) -> None:
    """Scalar-decay linear recurrence over the packed tokens of ``batch`` (see tkv_linrec_scan in the header): the chunked
    tensor-core kernel where it covers the shape, the token-by-token scan otherwise.  ``state`` [slots, heads, n, p]."""
    heads, n, p = state.shape[1:]
    dt = dtype_code(out.dtype)
    es = out.element_size()
    need = lib().tkv_linrec_chunk_workspace_bytes(batch.size, batch.max_tokens, batch.tokens, heads, n, p, dt)
    rows_ok = all((t.stride(0) * es) % 16 == 0 and t.data_ptr() % 16 == 0 for t in (q, k, v, out))
    if need >= 0 and rows_ok and batch.cu is not None and not force_scan and batch.size * heads <= 65535:
        ws = torch.empty(need, dtype=torch.uint8, device=out.device) if need else None
        check(lib().tkv_linrec_chunk(q.data_ptr(), q.stride(0), k.data_ptr(), k.stride(0), v.data_ptr(), v.stride(0),
                                     _ptr(log_decay), _ptr(head_log_decay), _ptr(v_scale), _ptr(skip), out.data_ptr(),
                                     state.data_ptr(), batch.slots.data_ptr(), batch.cu.data_ptr(), batch.pos0.data_ptr(), _ptr(ws),
                                     need, batch.size, batch.max_tokens, batch.tokens, heads, groups, n, p, dt, _ptr(batch.status),
                                     _stream(out)), "tkv_linrec_chunk")
        _count(3 if need else 1)
        return
    check(lib().tkv_linrec_scan(q.data_ptr(), q.stride(0), k.data_ptr(), k.stride(0), v.data_ptr(), v.stride(0), _ptr(log_decay),
                                _ptr(head_decay), _ptr(v_scale), _ptr(skip), out.data_ptr(), state.data_ptr(),
                                batch.slots.data_ptr(), _ptr(batch.cu), batch.pos0.data_ptr(), batch.size, heads, groups, n, p, dt,
                                _stream(out)), "tkv_linrec_scan")
    _count(1)


def diff_attention(proj, gate, q_norm, k_norm, k_ring, v_ring, batch, lam, diff: float, scale: float, eps: float, out,
                   heads: int, dim: int, vdim: int, window: int) -> None:
    """Differential attention of a step (see tkv_diff_prep in the header).  ``k_ring`` [slots, kv_heads, rows, 2, dp],
    ``v_ring`` [slots, kv_heads, rows, pp]; ``proj`` holds q | k | v per token, ``gate`` [tokens, heads]; ``out``
    [tokens, heads * vdim]."""
    _, kv_heads, rows, _, dp = k_ring.shape
    pp = v_ring.shape[3]
    dev, dt, T = proj.device, dtype_code(proj.dtype), batch.tokens
    q = torch.empty(T, heads, 2, dp, dtype=proj.dtype, device=dev)
    k_lin = v_lin = kv_start = None
    hist = kv_rows = 0
    if batch.cu is not None:
        kv_start, kv_rows, hist = batch.window_plan(window)
        k_lin = torch.empty(kv_rows, kv_heads, 2, dp, dtype=proj.dtype, device=dev)
        v_lin = torch.empty(kv_rows, kv_heads, pp, dtype=proj.dtype, device=dev)
    check(lib().tkv_diff_prep(proj.data_ptr(), proj.stride(0), q_norm.data_ptr(), k_norm.data_ptr(), float(eps), q.data_ptr(),
                              k_ring.data_ptr(), v_ring.data_ptr(), rows, _ptr(k_lin), _ptr(v_lin), _ptr(kv_start), _ptr(batch.cu),
                              batch.slots.data_ptr(), batch.pos0.data_ptr(), batch.size, T, hist, heads, kv_heads, dim, vdim, dp, pp,
                              window, dt, _stream(proj)), "tkv_diff_prep")
    if batch.cu is not None:
        check(lib().tkv_diff_prefill(q.data_ptr(), k_lin.data_ptr(), v_lin.data_ptr(), kv_start.data_ptr(), kv_rows,
                                     batch.cu.data_ptr(), batch.pos0.data_ptr(), lam.data_ptr(), float(diff), float(scale), float(eps),
                                     gate.data_ptr(), gate.stride(0), out.data_ptr(), batch.size, T, batch.max_tokens, heads, kv_heads,
                                     dim, vdim, dp, pp, window, dt, _ptr(batch.status), _stream(proj)), "tkv_diff_prefill")
        _count(3 if hist else 2)
        return
    need = lib().tkv_diff_decode_workspace_bytes(batch.size, heads, kv_heads, rows, dp, pp, dt)
    ws = torch.empty(need, dtype=torch.uint8, device=dev) if need else None
    check(lib().tkv_diff_decode(q.data_ptr(), k_ring.data_ptr(), v_ring.data_ptr(), rows, batch.slots.data_ptr(),
                                batch.pos0.data_ptr(), lam.data_ptr(), float(diff), float(scale), float(eps), gate.data_ptr(),
                                gate.stride(0), out.data_ptr(), _ptr(ws), need, batch.size, heads, kv_heads, dim, vdim, dp, pp, dt,
                                _stream(proj)), "tkv_diff_decode")
    _count(3 if need else 2)


# ---- channel-decay recurrence
def chanrec_step(q, f, v, f_bias, lower, norm, state, batch, out, eps: float) -> None:
    """One token per request; ``q``, ``f``, ``v`` are column slices of one projection, ``out`` is normed per head."""
    _, heads, n, p = state.shape
    check(lib().tkv_chanrec_step(q.data_ptr(), f.data_ptr(), v.data_ptr(), q.stride(0), f_bias.data_ptr(), lower.data_ptr(), norm.data_ptr(),
                                 float(eps), out.data_ptr(), state.data_ptr(), batch.slots.data_ptr(), batch.pos0.data_ptr(), batch.size,
                                 heads, n, p, dtype_code(out.dtype), _stream(out)), "tkv_chanrec_step")
    _count(1)


def chanrec(q, f, v, f_bias, lower, state, batch, out, force_scan: bool = False) -> None:
    """The recurrence over the packed tokens of ``batch`` (see tkv_chanrec_scan in the header): the chunked tensor-core kernel
    where it covers the shape, the token-by-token scan otherwise."""
    _, heads, n, p = state.shape
    dt = dtype_code(out.dtype)
    need = lib().tkv_chanrec_chunk_workspace_bytes(batch.size, batch.max_tokens, heads, n, p, dt)
    rows_ok = q.stride(0) % 8 == 0 and all(t.data_ptr() % 16 == 0 for t in (q, f, v, out))
    if need >= 0 and rows_ok and batch.cu is not None and not force_scan and batch.size * heads <= 65535:
        ws = torch.empty(need, dtype=torch.uint8, device=out.device) if need else None
        check(lib().tkv_chanrec_chunk(q.data_ptr(), f.data_ptr(), v.data_ptr(), q.stride(0), f_bias.data_ptr(), lower.data_ptr(),
                                      out.data_ptr(), state.data_ptr(), batch.slots.data_ptr(), batch.cu.data_ptr(), batch.pos0.data_ptr(),
                                      _ptr(ws), need, batch.size, batch.max_tokens, heads, n, p, dt, _ptr(batch.status), _stream(out)), "tkv_chanrec_chunk")
        _count(3 if need else 1)
        return
    check(lib().tkv_chanrec_scan(q.data_ptr(), f.data_ptr(), v.data_ptr(), q.stride(0), f_bias.data_ptr(), lower.data_ptr(), out.data_ptr(),
                                 state.data_ptr(), batch.slots.data_ptr(), _ptr(batch.cu), batch.pos0.data_ptr(), batch.size, heads, n, p,
                                 dtype_code(out.dtype), _stream(out)), "tkv_chanrec_scan")
    _count(1)


# ---- latent attention
def rotate_pairs(x, batch, heads: int, head_len: int, offset: int, rot_dims: int, freq) -> None:
    """Rotary positions (pairs of neighbours) in place on a part of every head; ``x`` [tokens, >= heads * head_len]."""
    check(lib().tkv_rotate_pairs(x.data_ptr(), x.stride(0), _ptr(batch.cu), batch.pos0.data_ptr(), batch.size, batch.tokens, heads,
                                 head_len, offset, rot_dims, freq.data_ptr(), dtype_code(x.dtype), _stream(x)), "tkv_rotate_pairs")
    _count(1)


def latent_prep(u, q_norm, kv_norm, eps: float, rot_dim: int, rot_dims: int, freq, ring, batch, window: int):
    """Query latent ``[tokens, q_rank]`` and (steps of several tokens) the linear buffer ``[rows, lw]`` of a step; stores the
    latents of its tokens in ``ring`` [slots, rows, lw]."""
    q_rank, kv_rank = q_norm.shape[0], kv_norm.shape[0]
    cq = torch.empty(batch.tokens, q_rank, dtype=u.dtype, device=u.device)
    lin = kv_start = None
    hist = 0
    if batch.cu is not None:
        kv_start, rows, hist = batch.window_plan(window)
        lin = torch.empty(rows, ring.shape[2], dtype=u.dtype, device=u.device)
    check(lib().tkv_latent_prep(u.data_ptr(), u.stride(0), q_norm.data_ptr(), kv_norm.data_ptr(), float(eps), q_rank, kv_rank, rot_dim,
                                rot_dims, freq.data_ptr(), cq.data_ptr(), ring.data_ptr(), ring.shape[1], _ptr(lin), _ptr(kv_start),
                                _ptr(batch.cu), batch.slots.data_ptr(), batch.pos0.data_ptr(), batch.size, batch.tokens, hist, window,
                                dtype_code(u.dtype), _stream(u)), "tkv_latent_prep")
    _count(2 if hist else 1)
    return cq, lin


def latent_prefill(q, kv, lin, batch, scale: float, out, heads: int, dim: int, rot_dim: int, vdim: int, kv_rank: int, window: int) -> None:
    """``q`` [tokens, heads * (dim + rot_dim)] rotated, ``kv`` [rows, >= heads * (dim + vdim)] keys and values of ``lin``'s rows."""
    kv_start, rows, _ = batch.window_plan(window)
    check(lib().tkv_latent_prefill(q.data_ptr(), q.stride(0), kv.data_ptr(), kv.stride(0), lin.data_ptr(), kv_start.data_ptr(), rows,
                                   batch.cu.data_ptr(), batch.pos0.data_ptr(), float(scale), out.data_ptr(), batch.size, batch.tokens,
                                   batch.max_tokens, heads, dim, rot_dim, vdim, kv_rank, window, dtype_code(q.dtype), _ptr(batch.status),
                                   _stream(q)), "tkv_latent_prefill")
    _count(1)


def latent_decode(q_abs, q, rot_dim: int, freq, ring, batch, scale: float, out, rot_dims: int) -> None:
    """One token per request: ``q_abs`` [B, heads, kv_rank], ``q`` [B, heads, dim + rot_dim] whose last part is not yet rotated
    (it is rotated in place where the form for every size runs), ``out`` [B, heads, kv_rank]; ``q_abs`` and ``out`` with any
    token and head strides."""
    bsz, heads, rank = q_abs.shape
    dt, q_rot = dtype_code(q_abs.dtype), q[:, :, q.shape[2] - rot_dim:]
    need = lib().tkv_latent_decode_workspace_bytes(bsz, heads, rank, rot_dim, ring.shape[1], dt)
    if need < 0 and rot_dims:
        rotate_pairs(q.view(bsz, -1), batch, heads, q.shape[2], q.shape[2] - rot_dim, rot_dims, freq)
    ws = torch.empty(need, dtype=torch.uint8, device=out.device) if need > 0 else None
    check(lib().tkv_latent_decode(q_abs.data_ptr(), q_abs.stride(0), q_abs.stride(1), q_rot.data_ptr(), q_rot.stride(0), q_rot.stride(1),
                                  freq.data_ptr(), ring.data_ptr(), ring.shape[1], batch.slots.data_ptr(), batch.pos0.data_ptr(),
                                  float(scale), out.data_ptr(), out.stride(0), out.stride(1), _ptr(ws), max(need, 0), bsz, heads, rank,
                                  rot_dim, rot_dims, dt, _stream(out)), "tkv_latent_decode")
    _count(2 if need > 0 else 1)


# ---- mixture of experts
def moe_route(logits, correction, identity: int, top: int, groups: int, keep: int, scale: float):
    """``(place [T, top], weight [T, top], src [T * top], offsets)`` of fp32 router logits (see tkv_moe_route in the header)."""
    T, E = logits.shape
    dev = logits.device
    ints = torch.empty(3 * T * top + E - identity + 1, dtype=torch.int32, device=dev)
    place, choice, src, offsets = ints[:T * top].view(T, top), ints[T * top:2 * T * top], ints[2 * T * top:3 * T * top], ints[3 * T * top:]
    weight = torch.empty(T, top, dtype=torch.float32, device=dev)
    counts = torch.zeros(E, dtype=torch.int32, device=dev) if T > 128 else None
    check(lib().tkv_moe_route(logits.data_ptr(), logits.stride(0), correction.data_ptr(), T, E, identity, top, groups, keep, float(scale),
                              weight.data_ptr(), choice.data_ptr(), place.data_ptr(), src.data_ptr(), _ptr(counts), offsets.data_ptr(),
                              _stream(logits)), "tkv_moe_route")
    _count(2 if T > 128 else 1)
    return place, weight, src, offsets


def moe_gemm(a, w, offsets, out, src=None, act: str = "none", status=None) -> None:
    """Grouped product: ``out[r] = act(a[src[r] or r] @ w[e].T)`` for the rows r of expert e; ``w`` [experts, n, k]."""
    check(lib().tkv_moe_gemm(a.data_ptr(), a.stride(0), a.shape[0], _ptr(src), w.data_ptr(), offsets.data_ptr(), out.data_ptr(), out.shape[0],
                             w.shape[0], w.shape[1], w.shape[2], {"none": 0, "gelu": 1}[act], dtype_code(a.dtype), _ptr(status),
                             _stream(a)), "tkv_moe_gemm")
    _count(1)
