"""Lidizen as a ModelSpec: a decoder over several parallel float32 residual streams. Every sublayer
reads a weighted sum of the streams through a centred norm and writes back to all of them while
they are mixed (hyper-connections). The mixer is grouped-query attention with projection biases, q
and k normed over the whole projection, neighbouring pairs of the first entries turned, scores mixed
across heads before the softmax, a sliding window that keeps the sequence's first positions, and
values mixed with those of the first layer that mixes values. The feed-forward is silu-gated with
biases, routed experts of squared-ReLU layers under a biased router, or absent. The embedding adds a
hashed table of token pairs and norms the sum; at the end the streams are added up, normed, and
multiplied with the embedding table. Layer i's tensors are `l<i>.norm1`, `l<i>.hc1.*`, `l<i>.mix.*`,
`l<i>.norm2`, `l<i>.hc2.*`, `l<i>.mlp.*`; the others `embed`, `bigram`, `embed.norm`, `final.norm`.

What the design fixes and the configuration therefore does not carry: the centred norms without a
bias; the q/k norm before the rotation and its plain gains; the pairing of neighbours; silu and the
dense layer's biases; the experts' form and their missing biases; the softmax over the chosen
logits; the tied head.
"""

from __future__ import annotations

from atomserve_b200.config.lidizen_config import LidizenConfig
from atomserve_b200.config.registry import register_architecture
from atomserve_b200.parts.spec import LayerCall, LayerSpec, ModelSpec, PartSpec


def _mixer(c: LidizenConfig, i: int, prefix: str) -> PartSpec:
    m = c.layers[i]["mixer"]
    rot, mask, position = m.get("rot"), m.get("mask"), None
    if rot is not None and rot["dims"]:
        position = PartSpec("rotary", dict(head_dim=m["dim"], theta=rot["base"], rotary_dim=rot["dims"], pairing="interleaved"))
    value_mix = None
    if m.get("v_mix"):
        value_mix = "first" if i == c.first_value_layer() else "mixed"
    return PartSpec("mixed_heads_attention", dict(
        num_heads=m["heads"], num_kv_heads=m["kv_heads"], head_dim=m["dim"], value_dim=m["vdim"], scale=m["scale"], eps=c.norm_eps,
        position=position, window=mask["size"] if mask else None, keep_first=mask.get("keep_first", 0) if mask else 0,
        value_mix=value_mix, biases=True), prefix)  # fmt: skip


def _feed_forward(mlp: dict | None, prefix: str) -> PartSpec:
    if mlp is None:
        return PartSpec("none")
    if mlp["kind"] == "dense":
        return PartSpec("gated_mlp", dict(intermediate_size=mlp["ff"], activation="silu", biases=True), prefix)
    r = mlp["router"]
    return PartSpec("routed_experts", dict(experts=r["experts"], top=r["top"], expert_ff=mlp["expert"]["ff"], score="chosen_softmax",
                                           router_bias=True, form="relu2", shared_gated=False), prefix)  # fmt: skip


def build_spec(c: LidizenConfig) -> ModelSpec:
    def connection(p: str, which: int) -> PartSpec:
        return PartSpec("hyper_connection", dict(eps=c.norm_eps, streams=c.streams, tensor=f"{p}norm{which}", hc=f"{p}hc{which}."))

    layers, unread = [], []
    for i, layer in enumerate(c.layers):
        p, mlp = f"l{i}.", layer.get("mlp")
        layers.append(LayerSpec(
            block="hyper_connections",
            mixer=_mixer(c, i, p + "mix."),
            feed_forward=_feed_forward(mlp, p + "mlp."),
            mixer_norm=connection(p, 1),
            feed_forward_norm=connection(p, 2) if mlp is not None else PartSpec("none"),
        ))  # fmt: skip
        # a checkpoint may hold what a layer has no use for: a factor for values that are not mixed,
        # the norm and connection of an absent feed-forward
        if layers[-1].mixer.params["value_mix"] != "mixed":
            unread.append(p + "mix.vmix")
        if mlp is None:
            unread += [p + n for n in ("norm2", "hc2.in", "hc2.out", "hc2.mix")]
    b = c.bigram
    return ModelSpec(
        hidden_size=c.width,
        vocab_size=c.vocab,
        max_positions=c.max_positions,
        embedding=PartSpec("pair_hash_embedding", dict(vocab_size=c.vocab, buckets=b["buckets"], mul_prev=b["mul_prev"], mul_cur=b["mul_cur"],
                                                       tensor="embed", pair_tensor="bigram", norm_eps=c.norm_eps, norm_tensor="embed.norm")),  # fmt: skip
        layers=tuple(layers),
        schedule=tuple(LayerCall(i) for i in range(len(layers))),
        final_norm=PartSpec("stream_sum_norm", dict(eps=c.norm_eps, streams=c.streams, tensor="final.norm")),
        head=PartSpec("lm_head", dict(vocab_size=c.vocab, tied=True)),
        ignored_tensors=tuple(unread),
    )


register_architecture(LidizenConfig.architecture, LidizenConfig, build_spec)
