"""Vilulix as a ModelSpec: a decoder over a float32 residual stream whose layers add mixer and
feed-forward side by side, x <- x + mixer(N1 x) + ff(N2 x), with RMS norms whose gains are stored
less one. Mixers: "mlstm" (a matrix memory with exponential gating), "latent_attention" (queries
through a latent of their own, keys and values from one cached latent per token with a turned key part
that all heads share, a gate per output element) and "parallel" (attention in a sliding window, q and k
normed over the whole projection before the rotation, a term exp(0) in the softmax's denominator, beside
a gated delta rule; a weighted sum of the two). The feed-forward is silu-gated, or absent. A stretch of
layers may run several times with the same weights and a cache or state of its own each time; every
pass but the first opens with x <- x + embedding. The logits are capped. Layer i's tensors are
`l<i>.norm1`, `l<i>.norm2`, `l<i>.mix.*`, `l<i>.mlp.*`; the others `embed`, `final.norm`, `head`.

What the design fixes and the configuration therefore does not carry: the norms' centre; the
rotate-half pairing of both rotations; the sink's score 0; the unit norms' 1e-6, the key-size scale of
the delta rule's queries and its silu gate; the matrix memory's query scale and floor; the untied head.
"""

from __future__ import annotations

from atomserve_b200.config.registry import register_architecture
from atomserve_b200.config.vilulix_config import VilulixConfig
from atomserve_b200.parts.spec import LayerCall, LayerSpec, ModelSpec, PartSpec

GAIN_CENTRE, SINK_SCORE, MEMORY_FLOOR = 1.0, 0.0, 1e-6
ATTENTION_NAMES = dict(q="q", k="k", v="v", o="o", q_norm="q.norm", k_norm="k.norm")


def _rotary(rot: dict | None, size: int) -> PartSpec | None:
    if rot is None or not rot["dims"]:
        return None
    return PartSpec("rotary", dict(head_dim=size, theta=rot["base"], rotary_dim=rot["dims"], pairing="half"))


def _mixer(c: VilulixConfig, layer: dict, prefix: str) -> PartSpec:
    m = layer["mixer"]
    if layer["type"] == "mlstm":
        return PartSpec("matrix_memory", dict(heads=m["heads"], dim=m["dim"], vdim=m["vdim"], gate_cap=m["gate_cap"],
                                              eps=c.norm_eps, floor=MEMORY_FLOOR), prefix)  # fmt: skip
    if layer["type"] == "latent_attention":
        position = PartSpec("rotary", dict(head_dim=m["rot_dim"], theta=m["rot"]["base"], rotary_dim=m["rot"]["dims"], pairing="half"))
        return PartSpec("latent_attention", dict(heads=m["heads"], dim=m["dim"], rot_dim=m["rot_dim"], vdim=m["vdim"],
                                                 kv_rank=m["kv_rank"], q_rank=m["q_rank"], scale=m["scale"], eps=c.norm_eps,
                                                 position=position, gated="elements"), prefix)  # fmt: skip
    left, right = m["left"], m["right"]
    mask = left.get("mask")
    return PartSpec("weighted_mixers", dict(
        left=PartSpec("gqa_attention", dict(num_heads=left["heads"], num_kv_heads=left["kv_heads"], head_dim=left["dim"],
                                            value_dim=left["vdim"], qk_norm_eps=c.norm_eps, norm_over="projection",
                                            position=_rotary(left.get("rot"), left["dim"]), scale=left["scale"],
                                            window=mask["size"] if mask else None, fixed_sink=SINK_SCORE,
                                            names=ATTENTION_NAMES), prefix + "left."),
        right=PartSpec("gated_delta_rule", dict(heads=right["heads"], kv_heads=right["kv_heads"], dim=right["dim"],
                                                vdim=right["vdim"], conv=right["conv"], eps=c.norm_eps), prefix + "right."),
        left_scale=m["left_scale"], right_scale=m["right_scale"],
    ), prefix)  # fmt: skip


def build_spec(c: VilulixConfig) -> ModelSpec:
    layers, unread = [], []
    for i, layer in enumerate(c.layers):
        p, mlp = f"l{i}.", layer.get("mlp")
        norm = dict(eps=c.norm_eps, centre=GAIN_CENTRE)
        if mlp is None:
            unread.append(p + "norm2")  # a layer without a feed-forward has no use for its norm
        layers.append(LayerSpec(
            block="parallel_residual",
            mixer=_mixer(c, layer, p + "mix."),
            feed_forward=(PartSpec("gated_mlp", dict(intermediate_size=mlp["ff"], activation="silu", biases=False), p + "mlp.")
                          if mlp is not None else PartSpec("none")),
            mixer_norm=PartSpec("rms_norm", dict(norm, tensor=p + "norm1")),
            feed_forward_norm=PartSpec("rms_norm", dict(norm, tensor=p + "norm2")) if mlp is not None else PartSpec("none"),
        ))  # fmt: skip
    schedule = [LayerCall(i, before=(0, opens) if opens is not None else None) for i, opens in c.run_order()]
    return ModelSpec(
        hidden_size=c.width,
        vocab_size=c.vocab,
        max_positions=c.max_positions,
        embedding=PartSpec("scaled_embedding", dict(vocab_size=c.vocab, tensor="embed")),
        layers=tuple(layers),
        schedule=tuple(schedule),
        final_norm=PartSpec("stream_rms_norm", dict(eps=c.norm_eps, centre=GAIN_CENTRE, tensor="final.norm")),
        head=PartSpec("lm_head", dict(vocab_size=c.vocab, tied=False, tensor="head", softcap=c.logit_softcap)),
        ignored_tensors=tuple(unread),
        stream_steps=(PartSpec("add_input"),) if any(call.before for call in schedule) else (),
    )


register_architecture(VilulixConfig.architecture, VilulixConfig, build_spec)
