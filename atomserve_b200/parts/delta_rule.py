"""The gated delta rule as a mixer: a matrix state per head that every token first decays, then
corrects towards its value at its key.

q, k (kv_heads x dim) and v (heads x vdim) are projections of the input, each passed through a short
causal convolution per channel and SiLU; per head q and k are made unit vectors, q times dim^(-1/2);
head h reads the q and k of head h // (heads / kv_heads). With beta = sigmoid(Wb h) and
g = exp(-exp(A) softplus(Wa h + dt_bias)), one of each per head and token,

    S <- g S;   u = beta (v - S^T k);   S <- S + k u^T;   o = S^T q          S: [dim, vdim], float32

Each head's o is divided by its root mean square, multiplied by a gain that the heads share and by
silu(Wg h), and the heads side by side are projected back. A request keeps S and the convolution's last
taps - 1 inputs in its state slot, zero at admission. The projections, the convolution and its
activation are in the compute dtype; unit norms, gates and everything in the recurrence are float32
(the gates' pre-activations are the float32 sums of their product).

Heads, sizes, taps and eps are parameters. The mixer can run beside another on one stacked product
(`input_weights` / `forward_from`).
"""

from __future__ import annotations

import torch

from atomserve_b200 import ops
from atomserve_b200.parts.base import CacheView, Mixer, StateSpec, StepContext, register_part
from atomserve_b200.parts.spec import TensorSpec


class GatedDeltaRule(Mixer):
    state_in_graphs = True  # the states are touched by this mixer's kernels alone, through ctx.state_slots
    reads_input = True  # beside its columns of a stacked product, for the gates' own product

    def __init__(self, hidden_size: int, prefix: str, heads: int, kv_heads: int, dim: int, vdim: int, conv: int, eps: float):
        if kv_heads < 1 or heads % kv_heads or conv < 1:
            raise ValueError(f"{heads} heads over {kv_heads} q/k heads, {conv} taps")
        self.hidden_size, self.prefix = hidden_size, prefix
        self.heads, self.kv_heads, self.dim, self.vdim, self.taps, self.eps = heads, kv_heads, dim, vdim, conv, float(eps)
        self.key_width, self.value_width = kv_heads * dim, heads * vdim
        self.channels = 2 * self.key_width + self.value_width  # what the convolution runs over: q, k, v
        self.in_proj = self.gate_proj = self.o_proj = self.conv_taps = None
        self.a_log = self.dt_bias = self.gain = None

    def state_specs(self) -> list[StateSpec]:
        return [StateSpec("s", (self.heads, self.dim, self.vdim), torch.float32),
                StateSpec("conv", (self.taps - 1, self.channels), torch.float32)]  # fmt: skip

    def tensor_specs(self) -> list[TensorSpec]:
        p, d, H = self.prefix, self.hidden_size, self.heads
        specs = []
        for n, width in (("q", self.key_width), ("k", self.key_width), ("v", self.value_width)):
            specs += [TensorSpec(p + n, (width, d)), TensorSpec(p + n + ".conv", (width, self.taps), kind="gain", init="gain")]
        return specs + [
            TensorSpec(p + "b", (H, d)), TensorSpec(p + "a", (H, d)),
            TensorSpec(p + "A_log", (H,), kind="gain", init="normal"), TensorSpec(p + "dt_bias", (H,), kind="gain", init="normal"),
            TensorSpec(p + "norm", (self.vdim,), kind="gain", init="gain"),
            TensorSpec(p + "g", (self.value_width, d)), TensorSpec(p + "o", (d, self.value_width)),
        ]  # fmt: skip

    def load(self, tensors: dict[str, torch.Tensor]) -> None:
        p = self.prefix
        self.in_proj = torch.cat([tensors[p + n] for n in "qkvg"]).contiguous()
        self.conv_taps = torch.cat([tensors[p + n + ".conv"] for n in "qkv"]).contiguous()
        # the two gates' rows in a product of their own, whose float32 sums are never rounded
        self.gate_proj = torch.cat([tensors[p + "b"], tensors[p + "a"]]).contiguous()
        self.a_log, self.dt_bias = tensors[p + "A_log"].contiguous(), tensors[p + "dt_bias"].contiguous()
        self.gain = tensors[p + "norm"].repeat(self.heads).contiguous()
        self.o_proj = tensors[p + "o"]

    def input_weights(self) -> torch.Tensor:
        """The stacked input projection (q, k, v, output gate), for a mixer that runs this one beside
        another and multiplies once for both."""
        return self.in_proj

    def mixed_from(self, proj: torch.Tensor, col: int, ctx: StepContext, cache: CacheView, h: torch.Tensor) -> torch.Tensor:
        """The normed, gated heads side by side, [T, heads * vdim], from a product that holds this mixer's
        projection in the columns from `col`."""
        H, kw = self.heads, self.key_width
        z = ops.linear(h, self.gate_proj, out_dtype=torch.float32)
        qkv = ops.causal_conv_silu(proj, col, self.conv_taps, cache.state["conv"], ctx.state_slots, ctx.req_q_start, ctx.num_requests,
                                   ctx.host_q_lens)  # fmt: skip
        # how long portions are cut is worked out once per step for all layers of these sizes
        key = ("delta_rule", H, self.dim, self.vdim)
        if key not in ctx.plans:
            ctx.plans[key] = ops.plan_delta(ctx.host_q_lens, H, self.dim, self.vdim, proj.device)
        o = ops.delta_rule(qkv, 0, kw, 2 * kw, z, 0, H, self.dt_bias, self.a_log, cache.state["s"], ctx.state_slots, ctx.req_q_start,
                           ctx.num_requests, kv_heads=self.kv_heads, plan=ctx.plans[key])  # fmt: skip
        gate = proj[:, col + self.channels : col + self.channels + self.value_width]
        return ops.head_norm_gate(o, gate, H, gain=self.gain, eps=self.eps, gate_activation="silu")

    def forward_from(self, proj: torch.Tensor, col: int, ctx: StepContext, cache: CacheView, h: torch.Tensor) -> torch.Tensor:
        return ops.linear(self.mixed_from(proj, col, ctx, cache, h), self.o_proj, out_dtype=torch.float32)

    def forward(self, h: torch.Tensor, residual: torch.Tensor | None, ctx: StepContext,
                cache: CacheView | None, write_cache: bool = True) -> torch.Tensor:  # fmt: skip
        # without a residual (a block that sums in float32 itself) the product stays float32
        return ops.linear(self.mixed_from(ops.linear(h, self.in_proj), 0, ctx, cache, h), self.o_proj, residual,
                          out_dtype=torch.float32 if residual is None else None)  # fmt: skip


register_part("mixer", "gated_delta_rule", GatedDeltaRule)
