"""Queries, keys and values on their way to the paged attention kernels: of heads that hold several
score maps, with the maps' outputs joined afterwards (csrc/qk_prepare.cu), and of heads normed all at
once (csrc/projection_prepare.cu)."""

from __future__ import annotations

import torch

from atomserve_b200.ops.library import KernelLibraryError, check, dtype_code, lib, ptr, require_cuda, stream


def qk_prepare_store(proj: torch.Tensor, heads: int, kv_heads: int, maps: int, dim: int, vdim: int, head_dim: int,
                     positions: torch.Tensor, *, inv_freq: torch.Tensor | None = None, rotary_dim: int = 0,
                     temperature: tuple[float, int] | None = None, slots: torch.Tensor | None = None,
                     k_cache: torch.Tensor | None = None, v_cache: torch.Tensor | None = None) -> torch.Tensor:  # fmt: skip
    """proj [T, >= (heads + kv_heads) * maps * dim + kv_heads * vdim]: per row the queries
    [heads][maps][dim], keys [kv_heads][maps][dim] and values [kv_heads][vdim]. Every map of q and
    k has its first `rotary_dim` entries turned (pairs (i, i + rotary_dim / 2), angle position *
    inv_freq[i]); q is multiplied by 1 + coef ln(floor((position + 1) / every) + 1) for
    `temperature=(coef, every)`. Returns queries [T, heads * maps, head_dim] in which map j of head
    h is head h * maps + j with its entries at offset j * dim among zeros; keys go to their page
    as [kv_heads, head_dim] (a head's maps side by side, zeros behind) and values likewise, where
    `slots`, `k_cache` and `v_cache` are given (without them only queries are read)."""
    require_cuda(proj, positions, inv_freq, slots, k_cache, v_cache)
    if proj.dim() != 2 or proj.stride(1) != 1:
        raise KernelLibraryError("qk_prepare_store: proj must be [tokens, columns] with unit column stride")
    T = proj.shape[0]
    if positions.dtype != torch.int32 or positions.shape[0] < T:
        raise KernelLibraryError("qk_prepare_store: positions must be int32, one per token")
    if inv_freq is not None and (inv_freq.dtype != torch.float32 or inv_freq.shape[0] * 2 < rotary_dim):
        raise KernelLibraryError("qk_prepare_store: inv_freq must be float32 [rotary_dim / 2]")
    bs = 0
    if k_cache is not None:
        if slots is None or v_cache is None or k_cache.shape != v_cache.shape or k_cache.dtype != proj.dtype or v_cache.dtype != proj.dtype:
            raise KernelLibraryError("qk_prepare_store: pages of keys and values of the projection's dtype, with slots")
        if k_cache.shape[1] != kv_heads or k_cache.shape[3] != head_dim or not k_cache.is_contiguous() or not v_cache.is_contiguous():
            raise KernelLibraryError(f"qk_prepare_store: pages must be [blocks, {kv_heads}, page, {head_dim}]")
        bs = k_cache.shape[2]
    q = torch.empty(T, heads * maps, head_dim, device=proj.device, dtype=proj.dtype)
    coef, every = temperature if temperature is not None else (0.0, 0)
    check(lib().asb_qk_prepare_store(ptr(proj), ptr(q), ptr(k_cache), ptr(v_cache), ptr(positions), ptr(slots),
                                     ptr(inv_freq), T, proj.stride(0), heads, kv_heads, maps, dim, vdim, head_dim,
                                     rotary_dim, bs, float(coef), int(every), dtype_code(proj), stream()))  # fmt: skip
    return q


def projection_norm_rope_store(proj: torch.Tensor, q_off: int, heads: int, kv_heads: int, dim: int, vdim: int, head_dim: int,
                               positions: torch.Tensor, q_gain: torch.Tensor, k_gain: torch.Tensor, eps: float, *,
                               inv_freq: torch.Tensor | None = None, rotary_dim: int = 0, interleaved: bool = False,
                               slots: torch.Tensor | None = None, k_cache: torch.Tensor | None = None,
                               v_cache: torch.Tensor | None = None) -> torch.Tensor:  # fmt: skip
    """proj [T, columns] holds, from column q_off on, queries [heads][dim], keys [kv_heads][dim] and values
    [kv_heads][vdim] of every token. Queries and keys are RMS-normed over all their heads at once, times
    their gains, and the first `rotary_dim` entries of each head turned (pairs (i, i + rotary_dim / 2), or
    neighbours, by position * inv_freq[i]). Returns queries [T, heads, head_dim]; keys and values go to
    their pages [blocks, kv_heads, page, head_dim] where `slots` says, zeros behind `dim` and `vdim`
    (without pages only queries are read)."""
    require_cuda(proj, positions, q_gain, k_gain, inv_freq, slots, k_cache, v_cache)
    if proj.dim() != 2 or proj.stride(1) != 1:
        raise KernelLibraryError("projection_norm_rope_store: proj must be [tokens, columns] with unit column stride")
    T = proj.shape[0]
    if positions.dtype != torch.int32 or positions.shape[0] < T:
        raise KernelLibraryError("projection_norm_rope_store: positions must be int32, one per token")
    for t, n, name in ((q_gain, heads * dim, "q_gain"), (k_gain, kv_heads * dim, "k_gain")):
        if t.dtype != torch.float32 or t.shape != (n,) or not t.is_contiguous():
            raise KernelLibraryError(f"projection_norm_rope_store: {name} must be contiguous float32 [{n}]")
    if rotary_dim and (inv_freq is None or inv_freq.dtype != torch.float32 or inv_freq.shape[0] * 2 < rotary_dim):
        raise KernelLibraryError("projection_norm_rope_store: inv_freq must be float32 [rotary_dim / 2]")
    bs = 0
    if k_cache is not None:
        if slots is None or v_cache is None or k_cache.shape != v_cache.shape or k_cache.dtype != proj.dtype or v_cache.dtype != proj.dtype:
            raise KernelLibraryError("projection_norm_rope_store: pages of keys and values of the projection's dtype, with slots")
        if k_cache.shape[1] != kv_heads or k_cache.shape[3] != head_dim or not k_cache.is_contiguous() or not v_cache.is_contiguous():
            raise KernelLibraryError(f"projection_norm_rope_store: pages must be [blocks, {kv_heads}, page, {head_dim}]")
        bs = k_cache.shape[2]
    q = torch.empty(T, heads, head_dim, device=proj.device, dtype=proj.dtype)
    check(lib().asb_projection_norm_rope_store(ptr(proj), proj.stride(0), q_off, ptr(q), ptr(k_cache), ptr(v_cache), ptr(q_gain),
                                               ptr(k_gain), ptr(positions), ptr(slots), ptr(inv_freq), T, heads, kv_heads, dim, vdim,
                                               head_dim, rotary_dim, int(interleaved), bs, float(eps), dtype_code(proj), stream()))  # fmt: skip
    return q


def differential_combine(a: torch.Tensor, vdim: int, lam: float, post: float, eps: float) -> torch.Tensor:
    """a [T, 2 H, hd], the outputs of map 1 and map 2 of head h at 2h and 2h + 1: returns
    [T, H * vdim] with o = a1 - lam * a2 over the first vdim entries, o / sqrt(mean(o^2) + eps) * post."""
    require_cuda(a)
    T, heads2, hd = a.shape
    if heads2 % 2 or not a.is_contiguous():
        raise KernelLibraryError("differential_combine: a must be contiguous [tokens, 2 heads, head_dim]")
    out = torch.empty(T, heads2 // 2 * vdim, device=a.device, dtype=a.dtype)
    check(lib().asb_differential_combine(ptr(out), ptr(a), T * (heads2 // 2), hd, vdim, float(lam), float(post), float(eps),
                                         dtype_code(a), stream()))  # fmt: skip
    return out
