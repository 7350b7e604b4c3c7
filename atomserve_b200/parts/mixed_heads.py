"""Grouped-query attention whose scores are mixed across heads before the softmax, as a mixer.

q, k and v are projected with biases; q and k are RMS-normed over their whole projection (all heads
at once, one gain entry per column), then a position encoding turns them; every head's score is
score_h <- sum_g talk[h, g] score_g over all heads' scaled scores; a query sees its last `window`
positions, itself included, and the sequence's first `keep_first` ones. `value_mix`: layers may mix
their values with those of the first layer that does, v <- (1 - lambda) v + lambda v_first, of the
same token; "first" marks that layer (it keeps its values for the step, and mixes nothing), "mixed"
a later one. Heads, sizes, eps, the score scale, the window and the encoding are parameters; keys and
values may differ in size (pages and kernels run at the larger one, zeros behind the narrower).

How it runs: the mix is linear in the queries, so it moves into them. With q'[h, c] the sum of
talk[h, g] q_g over the heads g of kv head c, head h's score is the sum over c of q'[h, c] . k_c: the
kernel that prepares the queries makes q' (float32, one rounding), and the paged attention kernels
serve heads with a vector per key head. The pages hold ordinary keys and (mixed) values.
"""

from __future__ import annotations

import torch

from atomserve_b200 import ops
from atomserve_b200.parts.base import CacheView, KVCacheSpec, Mixer, PageSpec, StepContext, build_part, register_part
from atomserve_b200.parts.spec import PartSpec, TensorSpec

FIRST_VALUES = "mixed_heads.first_values"  # in a step's plans: the first value-mixing layer's values


class MixedHeadsAttention(Mixer):
    def __init__(self, hidden_size: int, prefix: str, num_heads: int, num_kv_heads: int, head_dim: int, value_dim: int,
                 scale: float, eps: float, position: PartSpec | None = None, window: int | None = None, keep_first: int = 0,
                 value_mix: str | None = None, biases: bool = True):  # fmt: skip
        if num_heads % num_kv_heads:
            raise ValueError(f"{num_heads} heads are not a multiple of {num_kv_heads} kv heads")
        if value_mix not in (None, "first", "mixed"):
            raise ValueError(f"value_mix {value_mix!r} is neither None, 'first' nor 'mixed'")
        self.hidden_size, self.prefix = hidden_size, prefix
        self.num_heads, self.num_kv_heads, self.dim, self.value_dim = num_heads, num_kv_heads, head_dim, value_dim
        self.head_dim = max(head_dim, value_dim)  # what pages and kernels run at
        self.scale, self.eps = float(scale), float(eps)
        self.window, self.keep_first = window, (int(keep_first) if window is not None else 0)
        self.value_mix, self.biases = value_mix, biases
        self.position = build_part("position", position, hidden_size) if position else None
        self.qkv_proj = self.o_proj = self.bias = self.q_gain = self.k_gain = self.talk = None
        self.lam = 0.0

    def cache_spec(self) -> PageSpec:
        return KVCacheSpec(self.num_kv_heads, self.head_dim, self.window, keep_first=self.keep_first)

    def tensor_specs(self) -> list[TensorSpec]:
        p, d, H, KV = self.prefix, self.hidden_size, self.num_heads, self.num_kv_heads
        sizes = dict(q=H * self.dim, k=KV * self.dim, v=KV * self.value_dim)
        specs = [TensorSpec(p + n, (rows, d)) for n, rows in sizes.items()]
        if self.biases:
            specs += [TensorSpec(p + n + ".b", (rows,), kind="gain", init="normal") for n, rows in sizes.items()]
        specs += [
            TensorSpec(p + "o", (d, H * self.value_dim)),
            TensorSpec(p + "q.norm", (sizes["q"],), kind="gain", init="gain"),
            TensorSpec(p + "k.norm", (sizes["k"],), kind="gain", init="gain"),
            TensorSpec(p + "talk", (H, H), kind="gain", init="identity"),
        ]
        if self.value_mix == "mixed":
            specs.append(TensorSpec(p + "vmix", (), kind="gain", init="normal"))
        return specs

    def load(self, tensors: dict[str, torch.Tensor]) -> None:
        p = self.prefix
        self.qkv_proj = torch.cat([tensors[p + n] for n in "qkv"]).contiguous()
        self.bias = torch.cat([tensors[p + n + ".b"] for n in "qkv"]).contiguous() if self.biases else None
        self.q_gain, self.k_gain, self.talk = (tensors[p + n].contiguous() for n in ("q.norm", "k.norm", "talk"))
        self.o_proj = tensors[p + "o"]
        if self.value_dim != self.head_dim:  # attention gives heads of head_dim, zeros behind the values
            o = self.o_proj.new_zeros(self.hidden_size, self.num_heads, self.head_dim)
            o[:, :, : self.value_dim] = self.o_proj.view(self.hidden_size, self.num_heads, self.value_dim)
            self.o_proj = o.view(self.hidden_size, -1).contiguous()
        self.lam = float(tensors[p + "vmix"]) if self.value_mix == "mixed" else 0.0
        if self.position is not None:
            self.position.prepare(self.o_proj.device)
            rotary = self.position.fused_rotary()
            if rotary is None or rotary.magnitude != 1.0:
                raise NotImplementedError("attention with mixed heads turns its pairs by position x frequency")

    def attend(self, h: torch.Tensor, ctx: StepContext, cache: CacheView, write_cache: bool) -> torch.Tensor:
        """The heads' outputs side by side, [T, H * head_dim]."""
        H, KV = self.num_heads, self.num_kv_heads
        if not write_cache:
            raise NotImplementedError("attention with mixed heads reads the pages it writes")
        rotary = self.position.fused_rotary() if self.position is not None else None
        proj = None
        if self.qkv_proj.shape[0] % 4 == 0:
            # with few tokens the product stays as the GEMM's partial sums and the next kernel adds them up
            proj = ops.linear_partial(h, self.qkv_proj)
        if proj is None:
            proj = ops.linear(h, self.qkv_proj)
        q, values = ops.mixed_heads_prepare(
            proj, H, KV, self.dim, self.value_dim, self.head_dim, ctx.positions, self.talk, bias=self.bias,
            q_gain=self.q_gain, k_gain=self.k_gain, eps=self.eps, inv_freq=rotary.inv_freq if rotary else None,
            rotary_dim=rotary.rotary_dim if rotary else 0, interleaved=rotary is None or rotary.pairing == "interleaved",
            v_first=ctx.plans[FIRST_VALUES] if self.value_mix == "mixed" else None, lam=self.lam,
            keep_values=self.value_mix == "first", slots=cache.slots, k_cache=cache.k, v_cache=cache.v,
        )  # fmt: skip
        if values is not None:
            ctx.plans[FIRST_VALUES] = values
        out = ops.paged_attention(
            q, cache.k, cache.v, cache.block_tables, ctx.req_q_start, ctx.req_pos_start,
            num_requests=ctx.num_requests, max_context=ctx.max_context, window=self.window, scale=self.scale,
            host_q_lens=ctx.host_q_lens or None, keep_first=self.keep_first,
        )  # fmt: skip
        return out.view(-1, H * self.head_dim)

    def forward(self, h: torch.Tensor, residual: torch.Tensor | None, ctx: StepContext,
                cache: CacheView | None, write_cache: bool = True) -> torch.Tensor:  # fmt: skip
        return ops.linear(self.attend(h, ctx, cache, write_cache), self.o_proj, residual,
                          out_dtype=torch.float32 if residual is None else None)  # fmt: skip

    def forward_for_stream(self, h: torch.Tensor, ctx: StepContext, cache: CacheView | None, write_cache: bool = True):
        """mix(h) for a block that adds it to float32 streams itself: float32, or the output
        projection's partial sums (`ops.linear_for_stream`)."""
        return ops.linear_for_stream(self.attend(h, ctx, cache, write_cache), self.o_proj)


register_part("mixer", "mixed_heads_attention", MixedHeadsAttention)
