"""A plain, slow implementation of the Lidizen design: one function per mechanism, float64, whole
sequences at once, no cache. It shares no code with the package; the GPU tests compare the engine
with it.

Lidizen is a decoder over S parallel residual streams X [n, S, width]:

  x0 = N(embed[tok] + bigram[row(prev, tok)]),  X_s = x0 for every s,  N a centred norm with a gain
  a layer:  two sublayers f (mixer, feed-forward), each with vectors `in`, `out` [S] and a matrix
            `mix` [S, S]:  u = sum_s in_s X_s;  y = f(N u);  X_t <- sum_s mix[s, t] X_s + out_t y
  mixer:    grouped-query attention with projection biases; q and k RMS-normed over the whole
            projection, then turned in neighbouring pairs; every score is a learned mix of all
            heads' scores; a window that always keeps the first positions; values mixed with those
            of the first layer that mixes values
  ff:       silu-gated with biases, routed experts of squared-ReLU layers, or none
  at the end x = sum_s X_s, a centred norm, and the embedding table as the head
"""

from __future__ import annotations

import math

import torch

F64 = torch.float64


def keep(t: torch.Tensor) -> torch.Tensor:
    return t


def centred_norm(x: torch.Tensor, gain: torch.Tensor, eps: float) -> torch.Tensor:
    c = x - x.mean(-1, keepdim=True)
    return c / torch.sqrt((c * c).mean(-1, keepdim=True) + eps) * gain.to(F64)


def rms_norm(x: torch.Tensor, gain: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * gain.to(F64)


def pair_rows(tokens: list[int], buckets: int, mul_prev: int, mul_cur: int) -> list[int]:
    """Row of the pair table for each token; the table's last row for a token without a previous one."""
    return [buckets if i == 0 else (tokens[i - 1] * mul_prev + t * mul_cur) % buckets for i, t in enumerate(tokens)]


def embedding(tokens: list[int], weights: dict, cfg: dict) -> torch.Tensor:
    b = cfg["embedding"]["bigram"]
    rows = pair_rows(tokens, b["buckets"], b["mul_prev"], b["mul_cur"])
    e = weights["embed"][tokens].to(F64) + weights["bigram"][rows].to(F64)
    return centred_norm(e, weights["embed.norm"], cfg["norm"]["eps"])


def gather_streams(X: torch.Tensor, w_in: torch.Tensor) -> torch.Tensor:
    """[n, S, d] -> [n, d]: the sublayer's input."""
    u = torch.zeros(X.shape[0], X.shape[2], dtype=F64)
    for s in range(X.shape[1]):
        u = u + float(w_in[s]) * X[:, s]
    return u


def advance_streams(X: torch.Tensor, y: torch.Tensor, w_out: torch.Tensor, w_mix: torch.Tensor) -> torch.Tensor:
    """All streams at once from the old ones; `w_mix` is indexed [from, to]."""
    S = X.shape[1]
    new = []
    for t in range(S):
        x = float(w_out[t]) * y
        for s in range(S):
            x = x + float(w_mix[s, t]) * X[:, s]
        new.append(x)
    return torch.stack(new, dim=1)


def rotate_pairs(x: torch.Tensor, positions: torch.Tensor, base: float, dims: int) -> torch.Tensor:
    """x [n, heads, size]: entries 2i and 2i + 1 of the first `dims` turn by position * base^(-2i / dims)."""
    out = x.clone()
    for i in range(dims // 2):
        a = positions.to(F64) * base ** (-2.0 * i / dims)
        c, s = torch.cos(a)[:, None], torch.sin(a)[:, None]
        u, v = x[:, :, 2 * i], x[:, :, 2 * i + 1]
        out[:, :, 2 * i], out[:, :, 2 * i + 1] = u * c - v * s, v * c + u * s
    return out


def visible(n: int, mask: dict | None) -> torch.Tensor:
    """[n, n] bool: query i sees key j <= i that is less than `size` behind it or among the first
    `keep_first` positions of the sequence."""
    ok = torch.zeros(n, n, dtype=torch.bool)
    for i in range(n):
        for j in range(i + 1):
            ok[i, j] = mask is None or i - j < mask["size"] or j < mask.get("keep_first", 0)
    return ok


def mix_heads(scores: torch.Tensor, talk: torch.Tensor) -> torch.Tensor:
    """scores [H, n, n]: every head's score becomes a weighted sum of all heads' scores."""
    return torch.einsum("hg,gij->hij", talk.to(F64), scores)


def softmax_over(scores: torch.Tensor, ok: torch.Tensor) -> torch.Tensor:
    scores = scores.masked_fill(~ok, -math.inf)
    e = torch.exp(scores - scores.max(-1, keepdim=True).values)
    return e / e.sum(-1, keepdim=True)


def attention(h: torch.Tensor, w: dict, m: dict, eps: float, first_values: torch.Tensor | None = None, start: int = 0,
              stored=keep) -> tuple[torch.Tensor, torch.Tensor]:
    """(the mixer's output, its values before mixing). `first_values`: those of the first layer that
    mixes values, where this is a later one. `stored` (here and below) is applied to what an engine may
    keep in 16 bits between kernels."""
    n = h.shape[0]
    H, G, d, vd = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    project = lambda name: stored(stored(h @ w[name].to(F64).T) + w[name + ".b"].to(F64))  # noqa: E731
    q, k, v = project("q"), project("k"), project("v")
    own = v
    q, k = rms_norm(q, w["q.norm"], eps).view(n, H, d), rms_norm(k, w["k.norm"], eps).view(n, G, d)
    rot = m.get("rot")
    if rot is not None and rot["dims"]:
        pos = torch.arange(start, start + n)
        q, k = rotate_pairs(q, pos, rot["base"], rot["dims"]), rotate_pairs(k, pos, rot["base"], rot["dims"])
    q, k = stored(q), stored(k)
    if first_values is not None:
        lam = float(w["vmix"])
        v = stored((1.0 - lam) * v + lam * first_values)
    v = v.view(n, G, vd)
    share = H // G
    k, v = k.repeat_interleave(share, dim=1), v.repeat_interleave(share, dim=1)
    scores = torch.einsum("ihd,jhd->hij", q, k) * m["scale"]
    p = softmax_over(mix_heads(scores, w["talk"]), visible(n, m.get("mask")))
    o = stored(torch.einsum("hij,jhv->ihv", p, v)).reshape(n, H * vd)
    return o @ w["o"].to(F64).T, own


def dense(h: torch.Tensor, w: dict, stored=keep) -> torch.Tensor:
    gate = h @ w["gate"].to(F64).T + w["gate.b"].to(F64)
    up = h @ w["up"].to(F64).T + w["up.b"].to(F64)
    return stored(gate * torch.sigmoid(gate) * up) @ w["down"].to(F64).T + w["down.b"].to(F64)


def route(h: torch.Tensor, w: dict, top: int) -> tuple[torch.Tensor, torch.Tensor]:
    """(chosen [n, top], weights [n, top]): the largest logits, their softmax among themselves."""
    z = h @ w["router"].to(F64).T + w["router.b"].to(F64)
    best = torch.topk(z, top, dim=-1)
    return best.indices, torch.softmax(best.values, dim=-1)


def choice_margin(h: torch.Tensor, w: dict, top: int) -> torch.Tensor:
    """[n]: by how much the last chosen expert's logit leads the best one left out."""
    z = (h @ w["router"].to(F64).T + w["router.b"].to(F64)).sort(-1, descending=True).values
    if top >= z.shape[1]:
        return torch.full((h.shape[0],), math.inf, dtype=F64)
    return z[:, top - 1] - z[:, top]


def experts(h: torch.Tensor, w: dict, mlp: dict, stored=keep, margins: list | None = None) -> torch.Tensor:
    top = mlp["router"]["top"]
    chosen, weights = route(h, w, top)
    if margins is not None:
        margins.append(choice_margin(h, w, top))
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, wt in zip(chosen[t].tolist(), weights[t]):
            inner = stored(torch.relu(h[t] @ w[f"e{e}.up"].to(F64).T) ** 2)
            out[t] += wt * (inner @ w[f"e{e}.down"].to(F64).T)
    return out


def sub(weights: dict, prefix: str) -> dict:
    return {k[len(prefix) :]: v for k, v in weights.items() if k.startswith(prefix)}


def forward(tokens: list[int], weights: dict, cfg: dict, streams: list | None = None, stored=keep,
            margins: list | None = None) -> torch.Tensor:
    """float64 logits [n, vocab]; `streams`, if a list, collects the sum of the streams after every
    layer, and `margins` the routers' margins of choice per position, one entry per routed layer."""
    eps = cfg["norm"]["eps"]
    x0 = embedding(tokens, weights, cfg)
    X = torch.stack([x0] * cfg["streams"], dim=1)
    first_values = None
    for i, spec in enumerate(cfg["layers"]):
        hc1, hc2 = sub(weights, f"l{i}.hc1."), sub(weights, f"l{i}.hc2.")
        h = stored(centred_norm(gather_streams(X, hc1["in"]), weights[f"l{i}.norm1"], eps))
        mixes = bool(spec["mixer"].get("v_mix"))
        y, own = attention(h, sub(weights, f"l{i}.mix."), spec["mixer"], eps, first_values if mixes else None, stored=stored)
        if mixes and first_values is None:
            first_values = own
        X = advance_streams(X, y, hc1["out"], hc1["mix"])
        mlp = spec.get("mlp")
        if mlp is not None:
            h = stored(centred_norm(gather_streams(X, hc2["in"]), weights[f"l{i}.norm2"], eps))
            w = sub(weights, f"l{i}.mlp.")
            y = dense(h, w, stored) if mlp["kind"] == "dense" else experts(h, w, mlp, stored, margins)
            X = advance_streams(X, y, hc2["out"], hc2["mix"])
        if streams is not None:
            streams.append(X.sum(1))
    x = stored(centred_norm(X.sum(1), weights["final.norm"], eps))
    return x @ weights["embed"].to(F64).T


def tensor_shapes(cfg: dict) -> dict[str, tuple[int, ...]]:
    """Names and shapes of a checkpoint (the factor of a layer that has nothing to mix its values with aside)."""
    d, S = cfg["width"], cfg["streams"]
    shapes = {"embed": (cfg["vocab"], d), "bigram": (cfg["embedding"]["bigram"]["buckets"] + 1, d), "embed.norm": (d,)}
    mixed_before = False
    for i, spec in enumerate(cfg["layers"]):
        p, m, mlp = f"l{i}.", spec["mixer"], spec.get("mlp")
        H, G = m["heads"], m["kv_heads"]
        rows = dict(q=H * m["dim"], k=G * m["dim"], v=G * m["vdim"])
        for n, r in rows.items():
            shapes[f"{p}mix.{n}"], shapes[f"{p}mix.{n}.b"] = (r, d), (r,)
        shapes[p + "mix.q.norm"], shapes[p + "mix.k.norm"] = (rows["q"],), (rows["k"],)
        shapes[p + "mix.talk"], shapes[p + "mix.o"] = (H, H), (d, H * m["vdim"])
        if m.get("v_mix"):
            if mixed_before:
                shapes[p + "mix.vmix"] = ()
            mixed_before = True
        for q in (1, 2) if mlp is not None else (1,):
            shapes[f"{p}norm{q}"] = (d,)
            shapes[f"{p}hc{q}.in"], shapes[f"{p}hc{q}.out"], shapes[f"{p}hc{q}.mix"] = (S,), (S,), (S, S)
        if mlp is None:
            continue
        if mlp["kind"] == "dense":
            f = mlp["ff"]
            shapes.update({p + "mlp.gate": (f, d), p + "mlp.gate.b": (f,), p + "mlp.up": (f, d), p + "mlp.up.b": (f,),
                           p + "mlp.down": (d, f), p + "mlp.down.b": (d,)})  # fmt: skip
        else:
            E, f = mlp["router"]["experts"], mlp["expert"]["ff"]
            for e in range(E):
                shapes[f"{p}mlp.e{e}.up"], shapes[f"{p}mlp.e{e}.down"] = (f, d), (d, f)
            shapes[p + "mlp.router"], shapes[p + "mlp.router.b"] = (E, d), (E,)
    shapes["final.norm"] = (d,)
    return shapes


def random_checkpoint(cfg: dict, seed: int) -> dict[str, torch.Tensor]:
    """Random float32 weights whose matrices are exact in bfloat16: matrices N(0, 1 / fan_in) (the two
    embedding tables N(0, 1), routers N(0, 4 / fan_in) so that choices are seldom close), gains
    1 + N(0, 0.1), biases N(0, 0.3), the mix of heads 1 + N(0, 0.25), the streams' weights away from one
    another, the values' factor in 0.2 .. 0.7."""
    g = torch.Generator().manual_seed(seed)
    w = {}
    for name, shape in tensor_shapes(cfg).items():
        last = name.rsplit(".", 1)[-1]
        noise = torch.randn(shape, generator=g)
        if last == "vmix":
            w[name] = 0.2 + 0.5 * torch.rand(shape, generator=g)
        elif last == "talk":
            w[name] = torch.eye(shape[0]) + 0.5 * shape[0] ** -0.5 * noise
        elif ".hc" in name:
            S = shape[0]
            w[name] = {"in": 1.0 / S + 0.3 * noise, "out": 1.0 + 0.3 * noise, "mix": 0.8 * torch.eye(S) + 0.25 * noise if last == "mix" else None}[last]
        elif last == "b":
            w[name] = 0.3 * noise
        elif len(shape) == 1:
            w[name] = 1.0 + 0.1 * noise
        else:
            std = 1.0 if name in ("embed", "bigram") else (2.0 if last == "router" else 1.0) * shape[1] ** -0.5
            w[name] = (noise * std).bfloat16().float()
    return w


def greedy_generate(tokens: list[int], weights: dict, cfg: dict, n: int) -> list[int]:
    """The n tokens that follow when the largest logit is taken each time (the whole sequence is
    run again for every token: slow and stateless)."""
    tokens = list(tokens)
    first = len(tokens)
    for _ in range(n):
        tokens.append(int(forward(tokens, weights, cfg)[-1].argmax()))
    return tokens[first:]
