"""The gated delta rule over per-request state (csrc/delta_rule.cu): token by token for single tokens
and short portions, in chunks for long ones."""

from __future__ import annotations

import dataclasses

import torch

from atomserve_b200.ops.library import KernelLibraryError, check, dtype_code, lib, ptr, require_cuda, stream

STEP_TOKENS = 24  # portions of at most this many tokens run token by token
WORKSPACE_BYTES = 256 << 20  # most that a pass over chunks may take; longer steps run as several passes


@dataclasses.dataclass
class DeltaPass:
    """Chunks that run at once: `row`, `length` int32 [chunks], `req` int32 [requests, 3] (request, its
    first chunk here, its chunks here)."""

    row: torch.Tensor
    length: torch.Tensor
    req: torch.Tensor


@dataclasses.dataclass
class DeltaPlan:
    """How a step's requests run: `limit` tokens up to which a request runs token by token (0: all do),
    whether any request does, and the chunks of the others, in passes."""

    limit: int
    any_step: bool
    passes: list[DeltaPass]


def cut_into_chunks(q_lens: list[int], chunk: int, limit: int, most: int) -> list[tuple[list[int], list[int], list[list[int]]]]:
    """(first rows, lengths, [request, first chunk, chunks]) per pass of at most `most` chunks, over the
    requests that bring more than `limit` tokens; a request's chunks stay in order over the passes."""
    passes: list[tuple[list[int], list[int], list[list[int]]]] = []
    row = 0
    for r, n in enumerate(q_lens):
        for at in range(0, n if n > limit else 0, chunk):
            if not passes or len(passes[-1][0]) == most:
                passes.append(([], [], []))
            rows, lens, reqs = passes[-1]
            if not reqs or reqs[-1][0] != r:
                reqs.append([r, len(rows), 0])
            reqs[-1][2] += 1
            rows.append(row + at)
            lens.append(min(chunk, n - at))
        row += n
    return passes


def plan_delta(q_lens: list[int] | None, heads: int, dim: int, vdim: int, device: torch.device) -> DeltaPlan:
    """The plan for a step whose requests bring `q_lens` tokens (unknown: all token by token)."""
    chunk = lib().asb_delta_chunk_tokens(dim)
    if not q_lens or not chunk or max(q_lens) <= STEP_TOKENS:
        return DeltaPlan(0, True, [])
    per_chunk = 4 * heads * sum(_workspace_sizes(chunk, dim, vdim))
    cuts = cut_into_chunks(q_lens, chunk, STEP_TOKENS, max(1, WORKSPACE_BYTES // per_chunk))
    flat = [v for rows, lens, reqs in cuts for part in (rows, lens, sum(reqs, [])) for v in part]
    packed = torch.tensor(flat, dtype=torch.int32).to(device, non_blocking=True)
    passes, at = [], 0
    for rows, lens, reqs in cuts:
        a, b = at + len(rows), at + 2 * len(rows)
        passes.append(DeltaPass(packed[at:a], packed[a:b], packed[b : b + 3 * len(reqs)].view(-1, 3)))
        at = b + 3 * len(reqs)
    return DeltaPlan(STEP_TOKENS, min(q_lens) <= STEP_TOKENS, passes)


def _workspace_sizes(chunk: int, dim: int, vdim: int) -> tuple[int, int, int, int, int]:
    """Floats per (chunk, head) of the five workspaces of `asb_delta_chunks`."""
    dp, vp = -(-dim // 4) * 4, -(-vdim // 32) * 32
    return dp * 2 * chunk, chunk * dp, chunk * chunk, chunk * vp, 1


def delta_rule(x: torch.Tensor, q_off: int, k_off: int, v_off: int, z: torch.Tensor, b_off: int, a_off: int, dt_bias: torch.Tensor,
               a_log: torch.Tensor, state: torch.Tensor, state_slots: torch.Tensor, req_q_start: torch.Tensor, num_requests: int, *,
               kv_heads: int, plan: DeltaPlan) -> torch.Tensor:  # fmt: skip
    """S <- g S; u = beta (v - S^T k); S <- S + k u^T; o = S^T q for every new token of every request,
    in order; the state [slots, H, D, V] (float32) is read and left updated in each request's slot.

    x [T, columns] in the compute dtype holds q and k (kv_heads * D columns from q_off and k_off) and v
    (H * V from v_off); head h reads q and k of head h // (H / kv_heads), made unit vectors, q times
    D^(-1/2). z float32 [T, columns]: H pre-activations of beta from b_off and H of the decay from a_off;
    beta = sigmoid, g = exp(-exp(a_log) softplus(z + dt_bias)). `plan`: `plan_delta` of the step. Returns
    float32 [T, H * V]."""
    require_cuda(x, z, dt_bias, a_log, state, state_slots, req_q_start)
    if x.dim() != 2 or not x.is_contiguous() or z.dim() != 2 or z.dtype != torch.float32 or not z.is_contiguous() or z.shape[0] != x.shape[0]:
        raise KernelLibraryError("delta_rule: x contiguous [T, columns], z contiguous float32 [T, columns]")
    if state.dtype != torch.float32 or state.dim() != 4 or not state.is_contiguous():
        raise KernelLibraryError("delta_rule: state must be contiguous float32 [slots, H, D, V]")
    T = x.shape[0]
    _, H, D, V = state.shape
    if kv_heads < 1 or H % kv_heads:
        raise KernelLibraryError(f"delta_rule: {H} heads are not a multiple of {kv_heads} q/k heads")
    for t, name in ((dt_bias, "dt_bias"), (a_log, "a_log")):
        if t.dtype != torch.float32 or t.shape != (H,) or not t.is_contiguous():
            raise KernelLibraryError(f"delta_rule: {name} must be contiguous float32 [{H}]")
    for t in (state_slots, req_q_start):
        if t.dtype != torch.int32 or not t.is_contiguous():
            raise KernelLibraryError("delta_rule: index tensors must be contiguous int32")
    if max(q_off, k_off) + kv_heads * D > x.shape[1] or v_off + H * V > x.shape[1] or max(b_off, a_off) + H > z.shape[1]:
        raise KernelLibraryError("delta_rule: the column ranges lie outside their tensors")
    out = torch.empty(T, H * V, device=x.device, dtype=torch.float32)
    inputs = (ptr(out), ptr(x), x.shape[1], q_off, k_off, v_off, ptr(z), z.shape[1], b_off, a_off, ptr(dt_bias), ptr(a_log), ptr(state),
              ptr(state_slots))  # fmt: skip
    sizes = (H, D, V, H // kv_heads, float(D**-0.5))
    if plan.any_step:
        check(lib().asb_delta_step(*inputs, ptr(req_q_start), num_requests, *sizes, plan.limit, dtype_code(x), stream()))
    for p in plan.passes:
        chunks = p.row.shape[0]
        space = [torch.empty(chunks * H * n, device=x.device, dtype=torch.float32)
                 for n in _workspace_sizes(lib().asb_delta_chunk_tokens(D), D, V)]  # fmt: skip
        check(lib().asb_delta_chunks(*inputs, ptr(p.row), ptr(p.length), ptr(p.req), *(ptr(s) for s in space), chunks, p.req.shape[0],
                                     *sizes, dtype_code(x), stream()))  # fmt: skip
    return out
