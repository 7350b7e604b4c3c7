"""A plain, slow implementation of the Vilulix design: one function per mechanism, float64, whole
sequences at once, token by token where the design is a recurrence, no cache. It shares no code with
the package; the GPU tests compare the engine with it.

Vilulix is a decoder over a residual stream x [n, width]:

  x0 = embed[tok]
  a layer:  x <- x + mixer(N1 x) + ff(N2 x),   N an RMS norm whose gain is stored less one
  the layers of `loop` run `times` times with the same weights; every pass but the first opens with
      x <- x + x0
  mixers:   "mlstm"             a matrix memory with exponential gates
            "latent_attention"  queries and keys/values through latents of their own, one turned key
                                part for all heads, a gate per output element
            "parallel"          windowed attention whose softmax has one more term, exp(0), beside a
                                gated delta rule; a weighted sum of the two
  ff:       down(silu(gate h) * up h), or absent
  logits    c tanh(head N x / c)

`stored` is applied to what an implementation may keep in a 16-bit type; the tests use it to measure
what such rounding alone does to the logits.
"""

from __future__ import annotations

import torch

F64 = torch.float64
MEMORY_FLOOR, UNIT_EPS = 1e-6, 1e-6


def keep(t: torch.Tensor) -> torch.Tensor:
    return t


def rms_unit(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def centred_gain_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    """RMS norm whose gain is 1 + w."""
    return rms_unit(x, eps) * (1.0 + w.to(F64))


def unit_vectors(x: torch.Tensor) -> torch.Tensor:
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + UNIT_EPS)


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def turn_halves(x: torch.Tensor, base: float, dims: int, first: int = 0) -> torch.Tensor:
    """x [n, heads, dim] at positions first, first + 1, ...: entry i < dims / 2 is paired with entry
    i + dims / 2, the pair turned by position * base^(-2 i / dims); the rest passes."""
    half = dims // 2
    out = x.clone()
    p = torch.arange(first, first + x.shape[0], dtype=F64)[:, None]
    for i in range(half):
        a = p * base ** (-2.0 * i / dims)
        u, v = x[:, :, i], x[:, :, i + half]
        out[:, :, i] = u * torch.cos(a) - v * torch.sin(a)
        out[:, :, i + half] = v * torch.cos(a) + u * torch.sin(a)
    return out


def softmax_and_one(scores: torch.Tensor) -> torch.Tensor:
    """exp(s_j) / (1 + sum exp(s_j)) along the last axis."""
    top = torch.clamp(scores.max(-1, keepdim=True).values, min=0.0)
    e = torch.exp(scores - top)
    return e / (torch.exp(-top) + e.sum(-1, keepdim=True))


def attend_window(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float, window: int | None) -> torch.Tensor:
    """q [n, H, d], k [n, G, d], v [n, G, dv]: query i sees j with 0 <= i - j < window; head h reads
    key head h // (H / G); weights by `softmax_and_one`."""
    n, H, _ = q.shape
    G = k.shape[1]
    out = torch.zeros(n, H, v.shape[2], dtype=F64)
    for i in range(n):
        lo = 0 if window is None else max(0, i - window + 1)
        for h in range(H):
            g = h // (H // G)
            p = softmax_and_one((k[lo : i + 1, g] @ q[i, h]) * scale)
            out[i, h] = p @ v[lo : i + 1, g]
    return out


def window_attention(h: torch.Tensor, w: dict, m: dict, eps: float, stored=keep) -> torch.Tensor:
    """The left mixer: q and k RMS-normed over all their heads at once, then turned."""
    n, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms_unit(stored(h @ w["q"].T), eps) * w["q.norm"]
    k = rms_unit(stored(h @ w["k"].T), eps) * w["k.norm"]
    v = stored(h @ w["v"].T)
    q, k = q.view(n, H, d), k.view(n, G, d)
    rot = m.get("rot")
    if rot:
        q, k = turn_halves(q, rot["base"], rot["dims"]), turn_halves(k, rot["base"], rot["dims"])
    mask = m.get("mask")
    o = attend_window(stored(q), stored(k), v.view(n, G, dv), m["scale"], mask["size"] if mask else None)
    return stored(o.reshape(n, H * dv)) @ w["o"].T


def causal_convolution(x: torch.Tensor, taps: torch.Tensor) -> torch.Tensor:
    """x [n, C], taps [C, K], the last tap the current token's; zeros before the first."""
    n, K = x.shape[0], taps.shape[1]
    out = torch.zeros_like(x)
    for t in range(n):
        for j in range(K):
            at = t - (K - 1) + j
            if at >= 0:
                out[t] += taps[:, j] * x[at]
    return out


def delta_recurrence(q, k, v, g, beta, S=None):
    """q, k [n, H, d], v [n, H, dv], g, beta [n, H]: S <- g S; u = beta (v - S^T k); S <- S + k u^T;
    o = S^T q. Returns (o [n, H, dv], the last S [H, d, dv])."""
    n, H, d = q.shape
    S = torch.zeros(H, d, v.shape[2], dtype=F64) if S is None else S.clone()
    o = torch.zeros(n, H, v.shape[2], dtype=F64)
    for t in range(n):
        for h in range(H):
            S[h] = g[t, h] * S[h]
            u = beta[t, h] * (v[t, h] - S[h].T @ k[t, h])
            S[h] = S[h] + torch.outer(k[t, h], u)
            o[t, h] = S[h].T @ q[t, h]
    return o, S


def gated_delta_rule(h: torch.Tensor, w: dict, m: dict, eps: float, stored=keep) -> torch.Tensor:
    """The right mixer."""
    n, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    conv = {c: stored(silu(causal_convolution(stored(h @ w[c].T), w[c + ".conv"]))) for c in "qkv"}
    share = H // G
    q = unit_vectors(conv["q"].view(n, G, d)).repeat_interleave(share, 1) * d**-0.5
    k = unit_vectors(conv["k"].view(n, G, d)).repeat_interleave(share, 1)
    beta = torch.sigmoid(h @ w["b"].T)
    g = torch.exp(-torch.exp(w["A_log"]) * torch.nn.functional.softplus(h @ w["a"].T + w["dt_bias"]))
    o, _ = delta_recurrence(q, k, conv["v"].view(n, H, dv), g, beta)
    y = rms_unit(o, eps) * w["norm"] * silu(stored(h @ w["g"].T)).view(n, H, dv)
    return stored(y.reshape(n, H * dv)) @ w["o"].T


def parallel_mixer(h: torch.Tensor, w: dict, m: dict, eps: float, stored=keep) -> torch.Tensor:
    left = window_attention(h, sub(w, "left."), m["left"], eps, stored)
    return m["left_scale"] * left + m["right_scale"] * gated_delta_rule(h, sub(w, "right."), m["right"], eps, stored)


def matrix_memory(h: torch.Tensor, w: dict, m: dict, eps: float, stored=keep) -> torch.Tensor:
    n, H, d, dv, cap = h.shape[0], m["heads"], m["dim"], m["vdim"], m["gate_cap"]
    q = stored(h @ w["q"].T).view(n, H, d) * d**-0.5
    k, v = stored(h @ w["k"].T).view(n, H, d), stored(h @ w["v"].T).view(n, H, dv)
    gi = cap * torch.tanh((h @ w["i"].T + w["i.b"]) / cap)
    gf = torch.nn.functional.logsigmoid(cap * torch.tanh((h @ w["f"].T + w["f.b"]) / cap))
    o = torch.zeros(n, H, dv, dtype=F64)
    for head in range(H):
        S, norm, top = torch.zeros(d, dv, dtype=F64), torch.zeros(d, dtype=F64), torch.zeros((), dtype=F64)
        for t in range(n):
            old, top = top, torch.maximum(gf[t, head] + top, gi[t, head])
            keeps, takes = torch.exp(gf[t, head] + old - top), torch.exp(gi[t, head] - top)
            S = keeps * S + takes * torch.outer(k[t, head], v[t, head])
            norm = keeps * norm + takes * k[t, head]
            o[t, head] = (S.T @ q[t, head]) / (torch.maximum((norm @ q[t, head]).abs(), torch.exp(-top)) + MEMORY_FLOOR)
    o = rms_unit(o, eps).reshape(n, H * dv) * w["norm"]
    return stored(o * torch.sigmoid(stored(h @ w["g"].T))) @ w["o"].T


def latent_attention(h: torch.Tensor, w: dict, m: dict, eps: float, stored=keep) -> torch.Tensor:
    n, H, d, r, dv, rank = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    cq = stored(rms_unit(stored(h @ w["dq"].T), eps) * w["dq.norm"])
    q = stored(cq @ w["uq"].T).view(n, H, d + r)
    down = stored(h @ w["dkv"].T)
    c = stored(rms_unit(down[:, :rank], eps) * w["dkv.norm"])
    base, dims = m["rot"]["base"], m["rot"]["dims"]
    qr = stored(turn_halves(q[:, :, d:], base, dims))
    kr = stored(turn_halves(down[:, None, rank:], base, dims))[:, 0]
    k, v = stored(c @ w["uk"].T).view(n, H, d), stored(c @ w["uv"].T).view(n, H, dv)
    o = torch.zeros(n, H, dv, dtype=F64)
    for i in range(n):
        for head in range(H):
            s = (k[: i + 1, head] @ q[i, head, :d] + kr[: i + 1] @ qr[i, head]) * m["scale"]
            o[i, head] = torch.softmax(s, 0) @ v[: i + 1, head]
    return stored(stored(o.reshape(n, H * dv)) * torch.sigmoid(stored(h @ w["g"].T))) @ w["o"].T


def gated_mlp(h: torch.Tensor, w: dict, stored=keep) -> torch.Tensor:
    return stored(silu(stored(h @ w["gate"].T)) * stored(h @ w["up"].T)) @ w["down"].T


MIXERS = {"parallel": parallel_mixer, "mlstm": matrix_memory, "latent_attention": latent_attention}


def sub(weights: dict, prefix: str) -> dict:
    return {k[len(prefix) :]: v.to(F64) for k, v in weights.items() if k.startswith(prefix)}


def layer(x: torch.Tensor, weights: dict, i: int, cfg: dict, stored=keep) -> torch.Tensor:
    spec, eps, p = cfg["layers"][i], cfg["norm"]["eps"], f"l{i}."
    h1 = stored(centred_gain_norm(x, weights[p + "norm1"], eps))
    y = MIXERS[spec["type"]](h1, sub(weights, p + "mix."), spec["mixer"], eps, stored)
    if spec.get("mlp") is not None:
        h2 = stored(centred_gain_norm(x, weights[p + "norm2"], eps))
        y = y + gated_mlp(h2, sub(weights, p + "mlp."), stored)
    return x + y


def run_order(cfg: dict) -> list[tuple[int, bool]]:
    """(layer, whether the embedding is added before it) in the order the layers run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    order = [(i, False) for i in range(loop["start"])]
    for t in range(loop["times"]):
        order += [(i, t > 0 and i == loop["start"]) for i in range(loop["start"], loop["stop"])]
    return order + [(i, False) for i in range(loop["stop"], n)]


def forward(tokens: list[int], weights: dict, cfg: dict, streams: list | None = None, stored=keep) -> torch.Tensor:
    """float64 logits [n, vocab]; `streams`, if a list, collects x after every layer run."""
    x0 = weights["embed"][tokens].to(F64)
    x = x0
    for i, opens in run_order(cfg):
        if opens:
            x = x + x0
        x = layer(x, weights, i, cfg, stored)
        if streams is not None:
            streams.append(x)
    x = stored(centred_gain_norm(x, weights["final.norm"], cfg["norm"]["eps"]))
    c = cfg["logit_softcap"]
    return c * torch.tanh(x @ weights["head"].to(F64).T / c)


def tensor_shapes(cfg: dict) -> dict[str, tuple[int, ...]]:
    d = cfg["width"]
    shapes = {"embed": (cfg["vocab"], d), "final.norm": (d,), "head": (cfg["vocab"], d)}
    for i, spec in enumerate(cfg["layers"]):
        p, m = f"l{i}.", spec["mixer"]
        new = {"norm1": (d,)}
        if spec["type"] == "mlstm":
            H, K, V = m["heads"], m["heads"] * m["dim"], m["heads"] * m["vdim"]
            new.update({"mix.q": (K, d), "mix.k": (K, d), "mix.v": (V, d), "mix.g": (V, d), "mix.o": (d, V), "mix.norm": (V,),
                        "mix.i": (H, d), "mix.i.b": (H,), "mix.f": (H, d), "mix.f.b": (H,)})  # fmt: skip
        elif spec["type"] == "latent_attention":
            H, V = m["heads"], m["heads"] * m["vdim"]
            new.update({"mix.dq": (m["q_rank"], d), "mix.dq.norm": (m["q_rank"],), "mix.uq": (H * (m["dim"] + m["rot_dim"]), m["q_rank"]),
                        "mix.dkv": (m["kv_rank"] + m["rot_dim"], d), "mix.dkv.norm": (m["kv_rank"],),
                        "mix.uk": (H * m["dim"], m["kv_rank"]), "mix.uv": (V, m["kv_rank"]), "mix.g": (V, d), "mix.o": (d, V)})  # fmt: skip
        else:
            a, b = m["left"], m["right"]
            qw, kw = a["heads"] * a["dim"], a["kv_heads"] * a["dim"]
            new.update({"mix.left.q": (qw, d), "mix.left.k": (kw, d), "mix.left.v": (a["kv_heads"] * a["vdim"], d),
                        "mix.left.q.norm": (qw,), "mix.left.k.norm": (kw,), "mix.left.o": (d, a["heads"] * a["vdim"])})  # fmt: skip
            H, K, V = b["heads"], b["kv_heads"] * b["dim"], b["heads"] * b["vdim"]
            new.update({"mix.right." + n: s for n, s in {
                "q": (K, d), "q.conv": (K, b["conv"]), "k": (K, d), "k.conv": (K, b["conv"]), "v": (V, d), "v.conv": (V, b["conv"]),
                "b": (H, d), "a": (H, d), "A_log": (H,), "dt_bias": (H,), "norm": (b["vdim"],), "g": (V, d), "o": (d, V)}.items()})  # fmt: skip
        if spec.get("mlp") is not None:
            ff = spec["mlp"]["ff"]
            new.update({"norm2": (d,), "mlp.gate": (ff, d), "mlp.up": (ff, d), "mlp.down": (d, ff)})
        shapes.update({p + n: s for n, s in new.items()})
    return shapes


def random_checkpoint(cfg: dict, seed: int) -> dict[str, torch.Tensor]:
    """Random float32 weights whose matrices are exact in bfloat16: matrices N(0, 1 / fan_in), the
    embedding N(0, 1), the model's norms N(0, 0.2) around zero, plain gains 1 + N(0, 0.1), gate biases
    N(1, 1), convolution taps N(0, 1 / taps), A_log N(-1, 1) and dt_bias N(-1, 1) (decays from near 0
    to near 1), query and key gains of the attention times 1.5 (scores that spread)."""
    g = torch.Generator().manual_seed(seed)
    w = {}
    for name, shape in tensor_shapes(cfg).items():
        last = name.rsplit(".", 1)[-1]
        draw = torch.randn(shape, generator=g)
        if last in ("norm1", "norm2") or name == "final.norm":
            w[name] = 0.2 * draw
        elif last == "norm":
            w[name] = (1.0 + 0.1 * draw) * (1.5 if name.endswith((".q.norm", ".k.norm")) else 1.0)
        elif last == "b" and len(shape) == 1:
            w[name] = 1.0 + draw
        elif last in ("A_log", "dt_bias"):
            w[name] = draw - 1.0
        else:
            w[name] = (draw * (1.0 if name == "embed" else shape[1] ** -0.5)).bfloat16().float()
    return w


def greedy_generate(tokens: list[int], weights: dict, cfg: dict, n: int) -> list[int]:
    """The n tokens that follow when the largest logit is taken each time (the whole sequence is
    run again for every token: slow and stateless)."""
    tokens = list(tokens)
    first = len(tokens)
    for _ in range(n):
        tokens.append(int(forward(tokens, weights, cfg)[-1].argmax()))
    return tokens[first:]
