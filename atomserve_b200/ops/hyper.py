"""Several parallel residual streams per token: closing one sublayer and opening the next in one pass
(csrc/hyper_streams.cu)."""

from __future__ import annotations

import torch

from atomserve_b200.ops.experts import ExpertSums
from atomserve_b200.ops.library import KernelLibraryError, check, dtype_code, lib, ptr, require_cuda, stream
from atomserve_b200.ops.linear import PartialSums


def _vector(t: torch.Tensor | None, name: str, shape: tuple) -> None:
    if t is not None and (t.dtype != torch.float32 or tuple(t.shape) != shape or not t.is_contiguous()):
        raise KernelLibraryError(f"hyper_streams: {name} must be contiguous float32 {list(shape)}, got {t.dtype} {tuple(t.shape)}")


def hyper_streams(x: torch.Tensor, y: torch.Tensor | PartialSums | ExpertSums | None = None, *, w_out: torch.Tensor | None = None,
                  w_mix: torch.Tensor | None = None, bias: torch.Tensor | None = None, w_in: torch.Tensor | None = None,
                  gain: torch.Tensor | None = None, eps: float = 0.0, centred: bool = True, dtype: torch.dtype = torch.float32,
                  rows: torch.Tensor | None = None) -> tuple[torch.Tensor | None, torch.Tensor | None]:  # fmt: skip
    """x: float32 streams [n, S, width], rows of unit stride (an expanded [n, 1, width] serves as S
    copies). With y, the sublayer's output (float32 [n, width], a product's partial sums, or the routed
    experts' rows), the new streams x_t <- sum_s w_mix[s, t] x_s + w_out[t] (y + bias). With `gain`,
    N(sum_s w_in[s] x_s) * gain of the new streams (of x itself without y; `rows` (int32) then picks
    tokens) in `dtype`, N(u) = (u - mean) / sqrt(var + eps), or u / sqrt(mean(u^2) + eps) if not
    `centred`. Returns (the new streams or None, the normed rows or None)."""
    if x.dim() != 3 or x.dtype != torch.float32 or x.stride(2) != 1:
        raise KernelLibraryError(f"hyper_streams: x must be float32 [tokens, streams, width] with unit column stride, got {x.dtype} {tuple(x.shape)}")
    n, S, width = x.shape
    require_cuda(x, w_out, w_mix, bias, w_in, gain, rows)
    for t, name, shape in ((w_out, "w_out", (S,)), (w_mix, "w_mix", (S, S)), (w_in, "w_in", (S,)), (bias, "bias", (width,)), (gain, "gain", (width,))):
        _vector(t, name, shape)
    if (y is None) != (w_mix is None) or (y is None) != (w_out is None):
        raise KernelLibraryError("hyper_streams: a sublayer's output goes with w_out and w_mix")
    if rows is not None and (y is not None or rows.dtype != torch.int32):
        raise KernelLibraryError("hyper_streams: int32 rows are gathered where nothing is added")
    source, y_rows, pair_row, weights, top, ws, layout = 0, None, None, None, 0, None, (0, 0, 0, 0, 0)
    if isinstance(y, PartialSums):
        if (y.tokens, y.columns) != (n, width):
            raise KernelLibraryError("hyper_streams: partial sums of another shape")
        source, ws, layout = 2, y.workspace, y.layout()
    elif isinstance(y, ExpertSums):
        require_cuda(y.y, y.pair_row, y.weights)
        if y.y.dtype != torch.float32 or y.y.shape[1] != width or y.pair_row.shape[0] != n or y.weights.shape != y.pair_row.shape:
            raise KernelLibraryError("hyper_streams: the experts' rows do not match the streams")
        source, y_rows, pair_row, weights, top = 3, y.y, y.pair_row, y.weights, y.pair_row.shape[1]
    elif y is not None:
        require_cuda(y)
        _vector(y, "y", (n, width))
        source, y_rows = 1, y
    count = n if rows is None else rows.shape[0]
    out = torch.empty(n, S, width, device=x.device, dtype=torch.float32) if y is not None else None
    normed = torch.empty(count, width, device=x.device, dtype=dtype) if gain is not None else None
    check(lib().asb_hyper_streams(ptr(out), ptr(normed), ptr(x), x.stride(0), x.stride(1), ptr(rows), source, ptr(y_rows), ptr(pair_row),
                                  ptr(weights), top, ptr(ws), *layout, ptr(bias), ptr(w_out), ptr(w_mix), ptr(w_in), ptr(gain), count, S,
                                  width, float(eps), int(centred), dtype_code(normed) if normed is not None else 0, stream()))  # fmt: skip
    return out, normed
