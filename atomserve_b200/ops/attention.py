"""Paged grouped-query attention over cache pages for a flat batch of requests."""

from __future__ import annotations

import ctypes
import functools
import os

import torch

from atomserve_b200.ops.library import KernelLibraryError, check, dtype_code, lib, ptr, require_cuda, stream

KEY_TILE = 32
TARGET_BLOCKS = 296  # two blocks for each of the 148 SMs before the key range is split
SHORT_ROWS = 8  # requests with at most this many new tokens run row by row in the decode kernel
MIXED_SCRATCH_BYTES = 128 << 20  # most that a mixed step's partial results may take (see _paged_attention_mma)


# Which kernel serves prompt portions in bfloat16 with head size 128: "tcgen05" (scores and output
# in tensor memory; the default where its shape rules hold) or "mma" (the mma.sync kernel).
PREFILL_KERNEL = os.environ.get("ATOMSERVE_B200_PREFILL_ATTENTION", "tcgen05")


# In a step that holds prompt portions and single tokens, the two attention kernels touch disjoint
# rows and neither fills the device (a portion of a few hundred tokens is one block per SM or
# fewer; a few dozen single tokens are short chains of key tiles), so the single tokens' kernels
# run on a second stream beside the portions' kernel. "0" keeps them on one stream.
MIXED_OVERLAP = os.environ.get("ATOMSERVE_B200_MIXED_OVERLAP", "1") != "0"
_SIDE: dict[torch.device, tuple] = {}  # device -> (second stream, fork event, join event)


def _side_stream(device: torch.device):
    if device not in _SIDE:
        with torch.cuda.device(device):
            _SIDE[device] = (torch.cuda.Stream(), torch.cuda.Event(), torch.cuda.Event())
    return _SIDE[device]


def attention_tile_shape(group: int) -> tuple[int, int]:
    """(tokens per query tile, query heads per block) for `group` query heads per kv head."""
    qt, gc = ctypes.c_int(), ctypes.c_int()
    lib().asb_attention_tile_shape(group, ctypes.byref(qt), ctypes.byref(gc))
    return qt.value, gc.value


def plan_partitions(num_tokens: int, num_requests: int, num_kv_heads: int, group: int,
                    max_context: int, window: int) -> tuple[int, int]:  # fmt: skip
    """(partition size, partitions): split the keys only when the batch alone cannot fill the GPU.

    Partitions are aligned to absolute key positions, so the choice never changes which keys a
    row sees, only how its sum is grouped."""
    qt, gc = attention_tile_shape(group)
    blocks = (-(-num_tokens // qt) + num_requests) * num_kv_heads * -(-group // gc)
    span = max_context if window <= 0 else min(max_context, window + qt - 1)
    if blocks >= TARGET_BLOCKS or span <= 256:
        return 1 << 30, 1
    want = -(-TARGET_BLOCKS // blocks)
    size = max(256, -(-(-(-span // want)) // 256) * 256)
    if window <= 0:
        parts = (max_context - 1) // size + 1
    else:
        parts = min((max_context - 1) // size + 1, -(-span // size) + 1)
    return (size, parts) if parts > 1 else (1 << 30, 1)


@functools.lru_cache(maxsize=4096)
def plan_decode_partitions(rows: int, num_kv_heads: int, group: int, max_context: int, window: int,
                           head_dim: int = 128) -> tuple[int, int]:  # fmt: skip
    """(partition size, partitions) for the tensor-core decode kernel, one block per (row, kv
    head, partition). The device holds a fixed number of its blocks at once, so the blocks run in
    waves; the choice minimises waves x (64-key tiles per block + 3 tiles' worth of start-up) plus
    half a tile per partition for the merge, which is what a sweep over batch 4-128 and context
    1k-8k fitted: small batches want one nearly full wave, large ones two to five, and a count
    that spills a few blocks into one more wave is the worst. Never below one tile of 64 keys a
    block (which only short contexts at small batches choose: batch 1 at 512 keys runs 8.2 us with
    four partitions of 128 against 10.3 us with two of 256)."""
    blocks = rows * num_kv_heads * -(-group // 16)
    span = max_context if window <= 0 else min(max_context, window)
    resident = lib().asb_decode_attention_resident_blocks(head_dim) or 3 * 148
    best = None
    for want in range(1, max(1, span // 64) + 1):
        size = max(64, -(-(-(-span // want)) // 64) * 64)
        if window <= 0:
            parts = (max_context - 1) // size + 1
        else:
            parts = min((max_context - 1) // size + 1, -(-span // size) + 1)
        waves = -(-blocks * parts // resident)
        cost = waves * (size // 64 + 3) + 0.5 * parts
        if best is None or cost < best[0]:
            best = (cost, size, parts)
        if want > 64:
            break
    _, size, parts = best
    return (size, parts) if parts > 1 else (1 << 30, 1)


def paged_attention(
    q: torch.Tensor,
    k_cache: torch.Tensor,
    v_cache: torch.Tensor,
    block_tables: torch.Tensor,
    req_q_start: torch.Tensor,
    req_pos_start: torch.Tensor,
    *,
    num_requests: int,
    max_context: int,
    window: int | None,
    scale: float,
    partitions: tuple[int, int] | None = None,
    host_q_lens: list[int] | None = None,
    generic: bool = False,
    sink: torch.Tensor | None = None,
    chunk: int | None = None,
    softcap: float | None = None,
    keep_first: int = 0,
) -> torch.Tensor:
    """softmax(q k^T * scale) v for every new token, keys read in place from the pages.

    q: [T, H, hd]; k_cache, v_cache: [num_blocks, KV, block_size, hd]; block_tables: [R, W]
    int32; req_q_start: [R + 1] int32 (rows of each request in q); req_pos_start: [R] int32.
    max_context: the largest position + 1 any request reaches in this step (host int).
    A query at position p sees keys j <= p of its request, and j > p - window with a window.

    `sink` (float32 [H]): a logit per query head whose exponential joins the softmax's denominator
    once; it has no key and no value and is not scaled.

    `chunk`: the sequence is cut into runs of `chunk` positions, counted from position 0, and a
    query sees only the keys of its own run (still j <= p). `softcap`: every scaled score becomes
    softcap * tanh(score / softcap) before the softmax (the sink is not capped).

    `keep_first`: the first positions of a sequence, which stay visible behind the window and outside
    the chunk. q may be [T, H, KV, hd], a vector per key head: a head's score is then the sum of the
    products with all kv heads' keys (its values are still those of its own kv head): how scores that
    are mixed across heads run, the mix being part of the queries.

    bfloat16 with head size 64 or 128 runs the tensor-core kernels (decode kernel for requests
    that bring at most 8 tokens, prefill kernel for longer portions; `host_q_lens`, the tokens
    each request brings, tells which are needed; heads with a vector per key head have kernels of
    their own); everything else, and `generic=True`, runs the
    general CUDA-core kernel.
    """
    require_cuda(q, k_cache, v_cache, block_tables, req_q_start, req_pos_start)
    KV, bs = k_cache.shape[1], k_cache.shape[2]
    parts, summed = 1, q.dim() == 4  # (with one kv head the sum has one term)
    if summed:
        parts = q.shape[2]
        if parts != KV:
            raise KernelLibraryError(f"paged_attention: queries of {parts} parts against {KV} key heads")
    T, H, hd = q.shape[0], q.shape[1], q.shape[-1]
    if not q.is_contiguous() or k_cache.shape != v_cache.shape or k_cache.shape[3] != hd:
        raise KernelLibraryError("paged_attention: q must be contiguous and the caches [blocks, KV, bs, hd]")
    if k_cache.dtype != q.dtype or v_cache.dtype != q.dtype:
        raise KernelLibraryError("paged_attention: cache and query dtypes differ")
    for t in (block_tables, req_q_start, req_pos_start):
        if t.dtype != torch.int32 or not t.is_contiguous():
            raise KernelLibraryError("paged_attention: index tensors must be contiguous int32")
    win = int(window) if window else 0
    chunk, softcap = int(chunk or 0), float(softcap or 0.0)
    out = torch.empty(T, H, hd, device=q.device, dtype=q.dtype)
    if sink is not None:
        require_cuda(sink)
        if sink.dtype != torch.float32 or sink.shape != (H,) or not sink.is_contiguous():
            raise KernelLibraryError(f"paged_attention: sink must be contiguous float32 [{H}]")
    span = min(win, chunk) if win and chunk else (win or chunk)  # a chunk bounds the keys of a row as a window does
    keep = int(keep_first) if span else 0
    if q.dtype == torch.bfloat16 and not generic and not summed and not keep and lib().asb_attention_mma_supported(hd, H // KV):
        return _paged_attention_mma(q, out, k_cache, v_cache, block_tables, req_q_start, req_pos_start,
                                    num_requests, max_context, win, scale, partitions, host_q_lens, sink, chunk, softcap, span)  # fmt: skip
    if q.dtype == torch.bfloat16 and not generic and summed and not chunk and not softcap and sink is None and lib().asb_attention_parts_supported(hd, H, KV):
        return _paged_attention_parts(q, out, k_cache, v_cache, block_tables, req_q_start, req_pos_start, num_requests, max_context,
                                      win, keep, scale, partitions, host_q_lens)  # fmt: skip
    ps, np_ = partitions or plan_partitions(T, num_requests, KV, H // KV, max_context, span)
    part_m = part_l = part_acc = None
    if np_ > 1:
        part_m = torch.empty(T * H * np_, device=q.device, dtype=torch.float32)
        part_l = torch.empty_like(part_m)
        part_acc = torch.empty(T * H * np_ * hd, device=q.device, dtype=torch.float32)
    check(lib().asb_paged_attention_parts(
        ptr(out), ptr(q), ptr(k_cache), ptr(v_cache), ptr(block_tables), ptr(req_q_start),
        ptr(req_pos_start), ptr(part_m), ptr(part_l), ptr(part_acc), ptr(sink), T, num_requests, H, KV, hd, bs,
        block_tables.shape[1], win, chunk, keep, parts, ps, np_, float(scale), softcap, dtype_code(q), stream()))  # fmt: skip
    return out


def _paged_attention_mma(q, out, k_cache, v_cache, block_tables, req_q_start, req_pos_start, num_requests,
                         max_context, win, scale, partitions, host_q_lens, sink=None, chunk=0, softcap=0.0, span=None):  # fmt: skip
    span = win if span is None else span  # what bounds the keys of a row, for the planner
    T, H, hd = q.shape
    KV, bs = k_cache.shape[1], k_cache.shape[2]
    if host_q_lens is None:
        has_short = has_long = True
        all_single = False
        short_rows = T
    else:
        has_short = any(n <= SHORT_ROWS for n in host_q_lens)
        has_long = any(n > SHORT_ROWS for n in host_q_lens)
        all_single = all(n == 1 for n in host_q_lens)
        short_rows = sum(n for n in host_q_lens if n <= SHORT_ROWS)
    if has_long and PREFILL_KERNEL == "tcgen05" and lib().asb_attention_tcgen05_supported(hd, H // KV, bs):
        from atomserve_b200.ops.linear import gemm_status

        def portions():
            check(lib().asb_prefill_attention_tcgen05_masked(
                ptr(out), ptr(q), ptr(k_cache), ptr(v_cache), ptr(block_tables), ptr(req_q_start), ptr(req_pos_start), ptr(sink),
                T, num_requests, H, KV, hd, bs, k_cache.shape[0], block_tables.shape[1], win, chunk, float(scale), softcap,
                ptr(gemm_status(q.device)), stream()))  # fmt: skip

        if not has_short:
            portions()
            return out
        # What is left for the decode kernel: the short rows, with the key partitions their number
        # and context call for (a decoding request beside a prompt portion has as long a context
        # as in a step of its own). When the caller says how many tokens each request brings, the
        # kernel starts blocks for the short rows only and the partial results hold only those
        # rows; otherwise blocks start for every row of the step and the portions' leave at once.
        ps, np_ = partitions or plan_decode_partitions(short_rows, KV, H // KV, max_context, span, hd)
        compact = short_rows if host_q_lens is not None else 0
        scratch_rows = compact or T
        if partitions is None and scratch_rows * H * np_ * (hd + 2) * 4 > MIXED_SCRATCH_BYTES:
            ps, np_ = 1 << 30, 1
        part_m = part_l = part_acc = None
        if np_ > 1:
            part_m = torch.empty(scratch_rows * H * np_, device=q.device, dtype=torch.float32)
            # (without the short rows' count the merge runs over every row of the step and leaves
            # alone those whose sums are zero: the portions' rows, stored by their own kernel)
            part_l = (torch.empty if compact else torch.zeros)(scratch_rows * H * np_, device=q.device, dtype=torch.float32)
            part_acc = torch.empty(scratch_rows * H * np_ * hd, device=q.device, dtype=torch.float32)

        def single_tokens():
            check(lib().asb_paged_attention_mma_masked(
                ptr(out), ptr(q), ptr(k_cache), ptr(v_cache), ptr(block_tables), ptr(req_q_start),
                ptr(req_pos_start), ptr(part_m), ptr(part_l), ptr(part_acc), ptr(sink), T, num_requests, H, KV, hd, bs,
                block_tables.shape[1], win, chunk, ps, np_, float(scale), softcap, 1, 0, 0, compact, stream()))  # fmt: skip
            if np_ > 1 and compact:
                check(lib().asb_attention_reduce_short(ptr(out), ptr(part_m), ptr(part_l), ptr(part_acc), ptr(req_q_start),
                                                       num_requests, SHORT_ROWS, compact, H, np_, hd, dtype_code(q), stream()))  # fmt: skip
            elif np_ > 1:
                check(lib().asb_attention_reduce(ptr(out), ptr(part_m), ptr(part_l), ptr(part_acc), T * H, np_, hd,
                                                 dtype_code(q), stream()))  # fmt: skip

        if not MIXED_OVERLAP or torch.cuda.is_current_stream_capturing():
            portions()
            single_tokens()
            return out
        # Fork: the second stream starts from what this stream has done so far (q, the cache pages,
        # the scratch), runs the single tokens, and this stream goes on only when both are done.
        # The scratch is this stream's memory; it is given back after the join, so nothing that
        # reuses it can run before the second stream has finished with it.
        main = torch.cuda.current_stream(q.device)
        side, fork, join = _side_stream(q.device)
        fork.record(main)
        portions()
        with torch.cuda.stream(side):
            side.wait_event(fork)
            single_tokens()
            join.record(side)
        main.wait_event(join)
        return out
    ps, np_ = 1 << 30, 1
    if has_short and not has_long:
        ps, np_ = partitions or plan_decode_partitions(short_rows, KV, H // KV, max_context, span, hd)
    part_m = part_l = part_acc = None
    if np_ > 1:
        part_m = torch.empty(T * H * np_, device=q.device, dtype=torch.float32)
        part_l = torch.empty_like(part_m)
        part_acc = torch.empty(T * H * np_ * hd, device=q.device, dtype=torch.float32)
    check(lib().asb_paged_attention_mma_masked(
        ptr(out), ptr(q), ptr(k_cache), ptr(v_cache), ptr(block_tables), ptr(req_q_start),
        ptr(req_pos_start), ptr(part_m), ptr(part_l), ptr(part_acc), ptr(sink), T, num_requests, H, KV, hd, bs,
        block_tables.shape[1], win, chunk, ps, np_, float(scale), softcap, int(has_short), int(has_long), int(all_single), 0,
        stream()))  # fmt: skip
    if np_ > 1:
        check(lib().asb_attention_reduce(ptr(out), ptr(part_m), ptr(part_l), ptr(part_acc), T * H, np_, hd,
                                         dtype_code(q), stream()))  # fmt: skip
    return out


@functools.lru_cache(maxsize=4096)
def plan_parts_partitions(rows: int, heads: int, kv_heads: int, max_context: int, window: int, keep: int, head_dim: int) -> tuple[int, int]:
    """(key tiles of 64 per partition, partitions) for the decode kernel of heads with a vector per
    key head, one block per (row, up to 32 heads, partition): the same weighing as
    `plan_decode_partitions`, a tile's cost being the key and value heads that the block walks."""
    per_block = lib().asb_attention_parts_heads(heads, kv_heads)
    chunks = -(-heads // per_block)
    resident = lib().asb_attention_parts_resident(head_dim, heads, kv_heads) or 148
    tiles = -(-max_context // 64)
    if window:
        tiles = min(tiles, -(-min(keep, max_context) // 64) + -(-window // 64) + 1)
    items = (kv_heads + -(-kv_heads // chunks)) / 2  # a key head and a value head count as one tile of the plain kernel
    best = None
    for parts in range(1, min(tiles, 64) + 1):
        size = -(-tiles // parts)
        parts = -(-tiles // size)
        cost = -(-rows * chunks * parts // resident) * (size * items + 3) + 0.5 * parts
        if best is None or cost < best[0]:
            best = (cost, size, parts)
    return best[1], best[2]


def _paged_attention_parts(q, out, k_cache, v_cache, block_tables, req_q_start, req_pos_start, num_requests, max_context, win, keep,
                           scale, partitions, host_q_lens):  # fmt: skip
    T, H, KV, hd = q.shape
    bs = k_cache.shape[2]
    lens = host_q_lens
    has_short = lens is None or any(n <= SHORT_ROWS for n in lens)
    has_long = lens is None or any(n > SHORT_ROWS for n in lens)
    all_single = lens is not None and all(n == 1 for n in lens)
    short_rows = T if lens is None else sum(n for n in lens if n <= SHORT_ROWS)

    def launch(decode, long, pt, np_, m, l, acc, compact):
        check(lib().asb_attention_parts(
            ptr(out), ptr(q), ptr(k_cache), ptr(v_cache), ptr(block_tables), ptr(req_q_start), ptr(req_pos_start), ptr(m), ptr(l), ptr(acc),
            T, num_requests, H, KV, hd, bs, block_tables.shape[1], win, keep, pt, np_, float(scale), int(decode), int(long),
            int(all_single), compact, stream()))  # fmt: skip

    if has_long and PREFILL_KERNEL == "tcgen05" and scale > 0 and lib().asb_attention_parts_tcgen05_supported(hd, H // KV, bs):
        from atomserve_b200.ops.linear import gemm_status

        check(lib().asb_attention_parts_tcgen05(
            ptr(out), ptr(q), ptr(k_cache), ptr(v_cache), ptr(block_tables), ptr(req_q_start), ptr(req_pos_start), T, num_requests, H, KV, hd,
            bs, k_cache.shape[0], block_tables.shape[1], win, keep, float(scale), ptr(gemm_status(q.device)), stream()))  # fmt: skip
    elif has_long:
        launch(False, True, 1, 1, None, None, None, 0)
    if has_short:
        # a step that also holds long portions starts blocks, and holds partial results, for the short rows only
        compact = short_rows if has_long and lens is not None else 0
        rows = compact or T
        pt, np_ = partitions or plan_parts_partitions(short_rows, H, KV, max_context, win, keep, hd)
        if partitions is None and (lens is None or rows * H * np_ * (hd + 2) * 4 > MIXED_SCRATCH_BYTES):
            pt, np_ = 1 << 24, 1
        m = l = acc = None
        if np_ > 1:
            m = torch.empty(rows * H * np_, device=q.device, dtype=torch.float32)
            l = torch.empty_like(m)
            acc = torch.empty(rows * H * np_ * hd, device=q.device, dtype=torch.float32)
        launch(True, False, pt, np_, m, l, acc, compact)
        if np_ > 1 and compact:
            check(lib().asb_attention_reduce_short(ptr(out), ptr(m), ptr(l), ptr(acc), ptr(req_q_start), num_requests, SHORT_ROWS, compact,
                                                   H, np_, hd, dtype_code(q), stream()))  # fmt: skip
        elif np_ > 1:
            check(lib().asb_attention_reduce(ptr(out), ptr(m), ptr(l), ptr(acc), T * H, np_, hd, dtype_code(q), stream()))
    return out
