"""Queries, keys and values on their way to attention whose scores are mixed across heads
(csrc/mixed_heads.cu)."""

from __future__ import annotations

import torch

from atomserve_b200.ops.library import KernelLibraryError, check, dtype_code, lib, ptr, require_cuda, stream
from atomserve_b200.ops.linear import PartialSums


def mixed_heads_prepare(proj: torch.Tensor | PartialSums, heads: int, kv_heads: int, dim: int, vdim: int, head_dim: int,
                        positions: torch.Tensor, talk: torch.Tensor, *, bias: torch.Tensor | None = None,
                        q_gain: torch.Tensor | None = None, k_gain: torch.Tensor | None = None, eps: float = 0.0,
                        inv_freq: torch.Tensor | None = None, rotary_dim: int = 0, interleaved: bool = True,
                        v_first: torch.Tensor | None = None, lam: float = 0.0, keep_values: bool = False,
                        slots: torch.Tensor | None = None, k_cache: torch.Tensor | None = None,
                        v_cache: torch.Tensor | None = None) -> tuple[torch.Tensor, torch.Tensor | None]:  # fmt: skip
    """proj [T, >= heads * dim + kv_heads * (dim + vdim)]: per row queries, keys and values (or such
    a product's partial sums); `bias` (float32) is added. q and k are RMS-normed over all their heads
    at once where gains are given, and their first `rotary_dim` entries turned (neighbouring pairs, or
    pairs (i, i + rotary_dim / 2)). Returns queries [T, heads, kv_heads, head_dim] whose part c of head
    h is sum over the heads g of kv head c of talk[h, g] q_g (float32, rounded once, zeros behind
    `dim`), and with `keep_values` the values [T, kv_heads * vdim]. Keys go to their pages, and values,
    mixed (1 - lam) v + lam v_first where `v_first` is given."""
    partial = isinstance(proj, PartialSums)
    T = proj.tokens if partial else proj.shape[0]
    device, dtype = (proj.workspace.device, torch.bfloat16) if partial else (proj.device, proj.dtype)
    require_cuda(None if partial else proj, positions, talk, bias, q_gain, k_gain, inv_freq, v_first, slots, k_cache, v_cache)
    if not partial and (proj.dim() != 2 or proj.stride(1) != 1):
        raise KernelLibraryError("mixed_heads_prepare: proj must be [tokens, columns] with unit column stride")
    if positions.dtype != torch.int32 or positions.shape[0] < T:
        raise KernelLibraryError("mixed_heads_prepare: positions must be int32, one per token")
    columns = heads * dim + (kv_heads * (dim + vdim) if k_cache is not None else 0)
    for t, name, shape in ((talk, "talk", (heads, heads)), (q_gain, "q_gain", (heads * dim,)), (k_gain, "k_gain", (kv_heads * dim,))):
        if t is not None and (t.dtype != torch.float32 or tuple(t.shape) != shape or not t.is_contiguous()):
            raise KernelLibraryError(f"mixed_heads_prepare: {name} must be contiguous float32 {list(shape)}")
    if bias is not None and (bias.dtype != torch.float32 or bias.numel() < columns or not bias.is_contiguous()):
        raise KernelLibraryError("mixed_heads_prepare: bias must be contiguous float32, one per column")
    if inv_freq is not None and (inv_freq.dtype != torch.float32 or inv_freq.shape[0] * 2 < rotary_dim):
        raise KernelLibraryError("mixed_heads_prepare: inv_freq must be float32 [rotary_dim / 2]")
    bs = 0
    if k_cache is not None:
        if slots is None or v_cache is None or k_cache.shape != v_cache.shape or k_cache.dtype != dtype or v_cache.dtype != dtype:
            raise KernelLibraryError("mixed_heads_prepare: pages of keys and values of the projection's dtype, with slots")
        if k_cache.shape[1] != kv_heads or k_cache.shape[3] != head_dim or not k_cache.is_contiguous() or not v_cache.is_contiguous():
            raise KernelLibraryError(f"mixed_heads_prepare: pages must be [blocks, {kv_heads}, page, {head_dim}]")
        bs = k_cache.shape[2]
    elif v_first is not None or keep_values:
        raise KernelLibraryError("mixed_heads_prepare: without pages only queries are made")
    if v_first is not None and (v_first.dtype != dtype or v_first.shape != (T, kv_heads * vdim) or not v_first.is_contiguous()):
        raise KernelLibraryError(f"mixed_heads_prepare: v_first must be contiguous [{T}, {kv_heads * vdim}] in the compute dtype")
    q = torch.empty(T, heads, kv_heads, head_dim, device=device, dtype=dtype)
    values = torch.empty(T, kv_heads * vdim, device=device, dtype=dtype) if keep_values else None
    layout = proj.layout() if partial else (0, 0, 0, 0, 0)
    check(lib().asb_mixed_heads_prepare(None if partial else ptr(proj), ptr(proj.workspace) if partial else None, *layout, ptr(bias),
                                        ptr(q_gain), ptr(k_gain), ptr(talk), ptr(v_first), ptr(values), ptr(q), ptr(k_cache), ptr(v_cache),
                                        ptr(positions), ptr(slots), ptr(inv_freq), T, 0 if partial else proj.stride(0), heads, kv_heads,
                                        dim, vdim, head_dim, rotary_dim, int(interleaved), bs, float(eps), float(lam), dtype_code(q),
                                        stream()))  # fmt: skip
    return q, values
