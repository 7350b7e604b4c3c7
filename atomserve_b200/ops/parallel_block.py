"""Operations of layers whose mixer and feed-forward read the same float32 stream and are added
together, of a token embedding with a hashed table of token pairs beside it, and of a product over
two streams: the Python faces of csrc/parallel_block.cu."""

from __future__ import annotations

import torch

from atomserve_b200.ops.library import KernelLibraryError, check, dtype_code, lib, ptr, require_cuda, stream
from atomserve_b200.ops.linear import PartialSums


def _rows32(t: torch.Tensor | None, name: str, shape: tuple) -> None:
    if t is not None and (t.dtype != torch.float32 or tuple(t.shape) != shape or not t.is_contiguous()):
        raise KernelLibraryError(f"{name} must be contiguous float32 {list(shape)}, got {t.dtype} {tuple(t.shape)}")


def residual_terms_norm(x: torch.Tensor | None, terms: list[tuple[torch.Tensor | PartialSums, float]], gain1: torch.Tensor | None,
                        gain2: torch.Tensor | None, eps: float, dtype: torch.dtype, *, bias: torch.Tensor | None = None,
                        want_stream: bool = True) -> tuple[torch.Tensor | None, torch.Tensor | None, torch.Tensor | None]:  # fmt: skip
    """s = x + sum of f y over the (y, f) of `terms` (at most four) + bias, x and bias optional (float32
    [n, width]; bias [width]), and its two norms N(s) gain1, N(s) gain2 in `dtype`,
    N(s) = s / sqrt(mean(s^2) + eps). The last term may be the partial sums of a product
    (`linear_for_stream`), which the kernel then adds up itself. Returns (s or None, first norm or None,
    second norm or None)."""
    if terms and isinstance(terms[-1][0], PartialSums):
        return _with_partial_sums(x, terms[:-1], *terms[-1], gain1, gain2, eps, dtype, bias, want_stream)
    first = x if x is not None else (terms[0][0] if terms else None)
    if first is None or len(terms) > 4:
        raise KernelLibraryError(f"residual_terms_norm: {len(terms)} terms" if terms else "residual_terms_norm: nothing to add")
    require_cuda(x, bias, gain1, gain2, *(y for y, _ in terms))
    n, width = first.shape
    _rows32(x, "x", (n, width))
    for y, _ in terms:
        _rows32(y, "a term", (n, width))
    for t, name in ((bias, "bias"), (gain1, "gain1"), (gain2, "gain2")):
        _rows32(t, name, (width,))
    out32 = torch.empty(n, width, device=first.device, dtype=torch.float32) if want_stream else None
    out1 = torch.empty(n, width, device=first.device, dtype=dtype) if gain1 is not None else None
    out2 = torch.empty(n, width, device=first.device, dtype=dtype) if gain2 is not None else None
    code = dtype_code(out1 if out1 is not None else out2) if (out1 is not None or out2 is not None) else 0
    ys = [ptr(y) for y, _ in terms] + [None] * (4 - len(terms))
    fs = [float(f) for _, f in terms] + [0.0] * (4 - len(terms))
    check(lib().asb_residual_terms_norm(ptr(out32), ptr(out1), ptr(out2), ptr(x), *ys, *fs, len(terms), ptr(bias), ptr(gain1),
                                        ptr(gain2), n, width, float(eps), code, stream()))  # fmt: skip
    return out32, out1, out2


def _with_partial_sums(x, terms, product: PartialSums, factor: float, gain1, gain2, eps: float, dtype, bias, want_stream):
    n, width = product.tokens, product.columns
    if bias is not None or not want_stream or dtype != torch.bfloat16 or len(terms) > 4:
        raise KernelLibraryError("residual_terms_norm: partial sums join a stream that is kept, beside bfloat16 products, without a bias")
    require_cuda(x, gain1, gain2, *(y for y, _ in terms))
    for t in (x, *(y for y, _ in terms)):
        _rows32(t, "a term", (n, width))
    for t in (gain1, gain2):
        _rows32(t, "gain", (width,))
    device = product.workspace.device
    out32 = torch.empty(n, width, device=device, dtype=torch.float32)
    out1 = torch.empty(n, width, device=device, dtype=dtype) if gain1 is not None else None
    out2 = torch.empty(n, width, device=device, dtype=dtype) if gain2 is not None else None
    ys = [ptr(y) for y, _ in terms] + [None] * (4 - len(terms))
    fs = [float(f) for _, f in terms] + [0.0] * (4 - len(terms))
    check(lib().asb_partial_residual_terms_norm(ptr(out32), ptr(out1), ptr(out2), ptr(product.workspace), *product.layout(), float(factor),
                                                ptr(x), *ys, *fs, len(terms), ptr(gain1), ptr(gain2), n, width, float(eps), stream()))  # fmt: skip
    return out32, out1, out2


def residual_dual_norm(x: torch.Tensor | None, y1: torch.Tensor | None, y2: torch.Tensor | None, mult: float,
                       gain1: torch.Tensor | None, gain2: torch.Tensor | None, eps: float, dtype: torch.dtype, *,
                       bias: torch.Tensor | None = None,
                       want_stream: bool = True) -> tuple[torch.Tensor | None, torch.Tensor | None, torch.Tensor | None]:  # fmt: skip
    """`residual_terms_norm` of x + mult (y1 + y2) + bias, every term optional."""
    terms = [(y, mult) for y in (y1, y2) if y is not None]
    return residual_terms_norm(x, terms, gain1, gain2, eps, dtype, bias=bias, want_stream=want_stream)


def pair_embedding(ids: torch.Tensor, positions: torch.Tensor, req_q_start: torch.Tensor, state_slots: torch.Tensor,
                   last_id: torch.Tensor, table: torch.Tensor, pairs: torch.Tensor, mul_prev: int, mul_cur: int,
                   status: torch.Tensor) -> torch.Tensor:  # fmt: skip
    """float32 out[t] = table[ids[t]] + pairs[(previous id * mul_prev + ids[t] * mul_cur) mod buckets],
    `pairs` having buckets + 1 rows, the last one for a token at position 0. The id before a
    request's first token of the step is last_id[slot] - 1 (int32 per state slot), which is then
    set to the request's last id of the step plus one."""
    require_cuda(ids, positions, req_q_start, state_slots, last_id, table, pairs, status)
    for t in (ids, positions, req_q_start, state_slots, last_id):
        if t.dtype != torch.int32 or not t.is_contiguous():
            raise KernelLibraryError("pair_embedding: index tensors must be contiguous int32")
    if table.dim() != 2 or pairs.dim() != 2 or pairs.shape[1] != table.shape[1] or pairs.dtype != table.dtype or pairs.shape[0] < 2:
        raise KernelLibraryError("pair_embedding: the two tables must share width and dtype")
    if not table.is_contiguous() or not pairs.is_contiguous():
        raise KernelLibraryError("pair_embedding: tables must be contiguous")
    out = torch.empty(ids.shape[0], table.shape[1], device=table.device, dtype=torch.float32)
    check(lib().asb_pair_embedding(ptr(out), ptr(table), ptr(pairs), ptr(ids), ptr(positions), ptr(req_q_start),
                                   ptr(state_slots), ptr(last_id), ids.shape[0], state_slots.shape[0], table.shape[1],
                                   table.shape[0], pairs.shape[0] - 1, int(mul_prev), int(mul_cur), dtype_code(table),
                                   ptr(status), stream()))  # fmt: skip
    return out


def concat_cast(a: torch.Tensor, b: torch.Tensor, dtype: torch.dtype) -> torch.Tensor:
    """[a ; b] per row in `dtype`, a and b float32 [n, width]."""
    require_cuda(a, b)
    _rows32(a, "a", tuple(a.shape))
    _rows32(b, "b", tuple(a.shape))
    out = torch.empty(a.shape[0], 2 * a.shape[1], device=a.device, dtype=dtype)
    check(lib().asb_concat_cast(ptr(out), ptr(a), ptr(b), a.shape[0], a.shape[1], dtype_code(out), stream()))
    return out
