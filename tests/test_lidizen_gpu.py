"""The Lidizen design on the GPU against the plain implementation: each mechanism's part alone,
then whole models through the trace replayer in every way of cutting requests into steps, then
greedy generation through the engine and its scheduler."""

import math

import numpy as np
import pytest
import torch

import plain_lidizen as plain
from gefilix_helpers import check, prompts, write_folder
from helpers import mixed_trace
from test_engine_gpu import step_context
from test_tigesun_gpu import ROUNDINGS, Pages, doubles, i32, judge, paged, rounded, row_errors
from tiny_lidizen import LIDIZEN, attention

pytestmark = pytest.mark.gpu
DTYPES = [torch.float32, torch.bfloat16]
EPS = 1e-5
F64 = torch.float64


def on_device(w, dtype):
    """Matrices in the compute dtype; gains, biases and the mixing matrices float32."""
    small = ("talk", "mix", "in", "out")
    return {k: v.cuda().to(dtype if v.dim() == 2 and k.rsplit(".", 1)[-1] not in small else torch.float32) for k, v in w.items()}


# ---- each mechanism alone -------------------------------------------------------------------


def connection(d, S, centred, name, g, eps):
    from atomserve_b200.parts import PartSpec, build_part

    part = build_part("norm", PartSpec("hyper_connection", dict(eps=eps, streams=S, centred=centred, tensor=name, hc=name + ".hc.")), d)
    w = {name: 1 + 0.3 * torch.randn(d, generator=g), name + ".hc.in": torch.randn(S, generator=g), name + ".hc.out": torch.randn(S, generator=g),
         name + ".hc.mix": torch.randn(S, S, generator=g)}  # fmt: skip
    part.load({k: v.cuda() for k, v in w.items()})
    return part, w


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("d,S,centred", [(72, 1, True), (100, 3, True), (256, 2, True), (1030, 4, False), (512, 5, True), (61, 3, False), (128, 9, True)])
def test_hyper_connections_alone(dtype, d, S, centred):
    """A sublayer's input from streams that all differ, and from one row that stands for equal streams;
    the new streams with the next sublayer's input from the same kernel; the last sublayer of a model;
    a bias; the final norm over the streams' sum, on chosen rows."""
    from atomserve_b200.parts import PartSpec, build_part

    g = torch.Generator().manual_seed(d + S)
    T = 13
    one, w1 = connection(d, S, centred, "n1", g, EPS)
    two, w2 = connection(d, S, centred, "n2", g, 3 * EPS)
    for part in (one, two):
        part.bind_dtype(dtype)
    norm = plain.centred_norm if centred else plain.rms_norm
    X, y, b = torch.randn(T, S, d, generator=g), 2 * torch.randn(T, d, generator=g), torch.randn(d, generator=g)
    x0 = 1 + torch.randn(T, d, generator=g)

    def read(streams, w, name, eps):
        return norm(plain.gather_streams(streams.double(), w[name + ".hc.in"]), w[name], eps).float()

    h = one.forward(X.cuda())
    assert h.dtype == dtype
    check(h, read(X, w1, "n1", EPS), dtype, "the sublayer's input", 0.01)
    check(one.forward(x0.cuda()), read(torch.stack([x0] * S, 1), w1, "n1", EPS), dtype, "equal streams", 0.01)
    rows = i32([7, 0, 3])
    check(one.forward(X.cuda(), rows), read(X, w1, "n1", EPS)[[7, 0, 3]], dtype, "chosen rows", 0.01)
    for streams, start in ((X, X), (x0, torch.stack([x0] * S, 1))):
        for bias in (None, b):
            ref = plain.advance_streams(start.double(), y.double() + (0 if bias is None else bias.double()), w1["n1.hc.out"], w1["n1.hc.mix"])
            new, h = one.add_forward(streams.cuda(), y.cuda(), two, None if bias is None else bias.cuda())
            assert new.dtype == torch.float32 and h.dtype == dtype
            check(new.reshape(T, -1), ref.float().reshape(T, -1), torch.float32, "the new streams")
            check(h, read(ref, w2, "n2", 3 * EPS), dtype, "the next sublayer's input", 0.01)
            new, h = one.add_forward(streams.cuda(), y.cuda(), None, None if bias is None else bias.cuda())
            assert h is None
            check(new.reshape(T, -1), ref.float().reshape(T, -1), torch.float32, "the new streams, nothing follows")
    last = build_part("norm", PartSpec("stream_sum_norm", dict(eps=EPS, streams=S, centred=centred, tensor="f")), d)
    last.load({"f": w1["n1"].cuda()})
    last.bind_dtype(dtype)
    check(last.forward(X.cuda(), rows), norm(X.double().sum(1), w1["n1"], EPS).float()[[7, 0, 3]], dtype, "the streams' sum", 0.01)


def test_streams_that_read_partial_sums_and_experts_rows():
    """A product's partial sums and the routed experts' rows, added up inside the kernel, against the
    finished tensors."""
    from atomserve_b200 import ops

    g = torch.Generator().manual_seed(4)
    met = 0
    for T, d, K, S in ((1, 256, 512, 3), (5, 336, 1024, 2), (8, 2048, 2048, 4), (33, 256, 392, 6)):
        inner = torch.randn(T, K, generator=g).bfloat16().cuda()
        w = (torch.randn(d, K, generator=g) * K**-0.5).bfloat16().cuda()
        part, _ = connection(d, S, True, "n", g, EPS)
        part.bind_dtype(torch.bfloat16)
        X, b = torch.randn(T, S, d, generator=g).cuda(), torch.randn(d, generator=g).cuda()
        whole = part.add_forward(X, ops.linear(inner, w, out_dtype=torch.float32), part, b)
        y = ops.linear_for_stream(inner, w)
        met += isinstance(y, ops.PartialSums)
        fused = part.add_forward(X, y, part, b)
        assert float((whole[0] - fused[0]).abs().max() / whole[0].abs().max()) < 2e-6
        assert bool(((whole[1].float() - fused[1].float()).abs() <= 2.0**-7 * whole[1].float().abs() + 1e-6).all())
        rows, pair_row = torch.randn(3 * T, d, generator=g).cuda(), torch.randperm(3 * T, generator=g).view(T, 3).to(torch.int32).cuda()
        weights = torch.rand(T, 3, generator=g).cuda()
        whole = part.add_forward(X, ops.combine(rows, pair_row, weights), part)
        fused = part.add_forward(X, ops.ExpertSums(rows, pair_row, weights), part)
        assert torch.equal(whole[0], fused[0]) and torch.equal(whole[1], fused[1])
    assert met, "no shape ran with partial sums"


@pytest.mark.parametrize("dtype", DTYPES)
def test_normed_pair_embedding(dtype):
    from atomserve_b200.parts import CacheView, PartSpec, build_part

    g = torch.Generator().manual_seed(3)
    vocab, d, buckets = 50, 40, 13
    cfg = dict(norm=dict(eps=EPS), embedding=dict(bigram=dict(buckets=buckets, mul_prev=1000003, mul_cur=7)))
    w = {"embed": rounded(torch.randn(vocab, d, generator=g)), "bigram": rounded(torch.randn(buckets + 1, d, generator=g)),
         "embed.norm": 1 + 0.3 * torch.randn(d, generator=g)}  # fmt: skip
    part = build_part("embedding", PartSpec("pair_hash_embedding", dict(vocab_size=vocab, buckets=buckets, mul_prev=1000003, mul_cur=7, tensor="embed",
                                                                        pair_tensor="bigram", norm_eps=EPS, norm_tensor="embed.norm")), d)  # fmt: skip
    part.load(on_device(w, dtype))
    tokens = torch.randint(0, vocab, (23,), generator=g).tolist()
    ref = plain.embedding(tokens, w, cfg).float()
    view = CacheView(state=dict(last=torch.zeros(2, 1, dtype=torch.int32, device="cuda")))
    at = 0
    for n in (5, 1, 1, 2, 14):
        ctx = step_context([n], [at], [1])
        ctx.token_ids = i32(tokens[at : at + n])
        check(part.forward_step(ctx, view), ref[at : at + n], torch.float32, f"tokens {at} to {at + n}")
        at += n


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,dim,vdim,dims,interleaved,normed", [
    (6, 3, 24, 16, 8, True, True), (8, 2, 48, 64, 40, True, True), (5, 5, 10, 12, 10, True, True), (8, 1, 128, 128, 64, True, True),
    (8, 2, 64, 128, 0, True, False), (16, 2, 32, 32, 16, False, True), (32, 4, 128, 128, 64, True, True), (16, 4, 128, 96, 126, True, True), (12, 4, 16, 8, 6, False, True), (2, 2, 64, 64, 64, True, True),
])  # fmt: skip
def test_prepared_queries_keys_and_values(dtype, H, G, dim, vdim, dims, interleaved, normed):
    """Biases, the norm over the whole projection, both pairings at near and far positions, the mix of
    the heads, values mixed with an earlier layer's, zeros behind what a head holds; pages hold ones
    beforehand (a slot used again keeps nothing of its former owner), and a token without a slot stores
    nothing."""
    from atomserve_b200 import ops

    bs, hd = 4, max(dim, vdim)
    g = torch.Generator().manual_seed(H * dim + dims)
    positions = [0, 1, 2, 5, 63, 64, 1000, 4097, 30000, 7]
    T = len(positions)
    sizes = (H * dim, G * dim, G * vdim)
    q, k, v = (rounded(torch.randn(T, n, generator=g)) for n in sizes)
    bias = 0.5 * torch.randn(sum(sizes), generator=g)
    gq, gk = 1 + 0.3 * torch.randn(sizes[0], generator=g), 1 + 0.3 * torch.randn(sizes[1], generator=g)
    talk, lam, first = torch.randn(H, H, generator=g), 0.3, rounded(torch.randn(T, sizes[2], generator=g))
    bq, bk, bv = (b.double() for b in bias.split(sizes))
    pos = torch.tensor(positions)

    def turn(x):
        if interleaved or not dims:
            return plain.rotate_pairs(x, pos, 50.0, dims)
        order = [j for i in range(dims // 2) for j in (i, i + dims // 2)] + list(range(dims, dim))
        back = torch.argsort(torch.tensor(order))
        return plain.rotate_pairs(x[..., order], pos, 50.0, dims)[..., back]

    norm = (lambda x, gain: plain.rms_norm(x, gain, EPS)) if normed else (lambda x, gain: x)
    rq, rk = turn(norm(q.double() + bq, gq).view(T, H, dim)), turn(norm(k.double() + bk, gk).view(T, G, dim))
    share = H // G
    rq = torch.stack([torch.einsum("hg,tgd->thd", talk[:, c * share : (c + 1) * share].double(), rq[:, c * share : (c + 1) * share]) for c in range(G)], 2)
    own = v.double() + bv
    pages_k = torch.ones(8, G, bs, hd, device="cuda", dtype=dtype)
    pages_v = torch.ones_like(pages_k)
    slots = [21, 0, 31, 13, 14, 3, 8, 9, 18, -1]
    inv_freq = torch.tensor([50.0 ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=torch.float32).cuda() if dims else None
    common = dict(bias=bias.cuda(), q_gain=gq.cuda() if normed else None, k_gain=gk.cuda() if normed else None, eps=EPS, inv_freq=inv_freq,
                  rotary_dim=dims, interleaved=interleaved, slots=i32(slots), k_cache=pages_k, v_cache=pages_v)  # fmt: skip
    proj = torch.cat([q, k, v], 1).cuda().to(dtype)
    _, values = ops.mixed_heads_prepare(proj, H, G, dim, vdim, hd, i32(positions), talk.cuda(), keep_values=True, **common)
    tol = 0.01 if dtype == torch.bfloat16 else 1e-5
    slack = pos.double() * 2.0**-23 * 4  # float32 angles: position x frequency is off by up to 2^-24 of itself

    def close(got, ref, what):
        limit = (tol + slack[: got.shape[0]].view(-1, *[1] * (ref.dim() - 1))) * ref.abs().max()
        assert bool(((got.double().cpu() - ref).abs() <= limit).all()), what

    close(values, own, "values kept for later layers")
    out, none = ops.mixed_heads_prepare(proj, H, G, dim, vdim, hd, i32(positions), talk.cuda(), v_first=first.cuda().to(dtype), lam=lam, **common)
    assert none is None and out.shape == (T, H, G, hd)
    close(out[..., :dim], rq, "mixed queries")
    assert not out[..., dim:].any()
    real = slots[:-1]
    got_k, got_v = (p.float().cpu().permute(0, 2, 1, 3).reshape(-1, G, hd) for p in (pages_k, pages_v))
    close(got_k[real][..., :dim], rk[:-1], "keys")
    close(got_v[real][..., :vdim], ((1 - lam) * own + lam * first.double()).view(T, G, vdim)[:-1], "mixed values")
    assert not got_k[real][..., dim:].any() and not got_v[real][..., vdim:].any()
    untouched = sorted(set(range(8 * bs)) - set(real))
    assert (got_k[untouched] == 1).all() and (got_v[untouched] == 1).all()


def test_prepared_queries_from_partial_sums():
    """The stacked product left as the tensor-core GEMM's partial sums gives what the finished product
    gives, up to the rounding of the product to 16 bits."""
    from atomserve_b200 import ops

    g = torch.Generator().manual_seed(9)
    met = 0
    for T, K, H, G, dim, vdim in ((1, 512, 4, 2, 64, 64), (7, 1024, 8, 2, 128, 128), (30, 768, 4, 1, 48, 64)):
        rows = H * dim + G * (dim + vdim)
        h, w = torch.randn(T, K, generator=g).bfloat16().cuda(), (torch.randn(rows, K, generator=g) * K**-0.5).bfloat16().cuda()
        hd, talk = max(dim, vdim), torch.randn(H, H, generator=g).cuda()
        results = []
        for product in (ops.linear(h, w), ops.linear_partial(h, w)):
            met += isinstance(product, ops.PartialSums)
            if product is None:
                continue
            pages = [torch.ones(8, G, 4, hd, device="cuda", dtype=torch.bfloat16) for _ in range(2)]
            q, v = ops.mixed_heads_prepare(product, H, G, dim, vdim, hd, i32(range(T)), talk, bias=torch.ones(rows).cuda(), q_gain=torch.ones(H * dim).cuda(),
                                           k_gain=torch.ones(G * dim).cuda(), eps=EPS, inv_freq=torch.ones(dim // 2).cuda(), rotary_dim=dim,
                                           keep_values=True, slots=i32(range(T)), k_cache=pages[0], v_cache=pages[1])  # fmt: skip
            results.append([q, v, *pages])
        for a, b in zip(results[0], results[-1]):
            assert float((a.float() - b.float()).abs().max() / a.float().abs().max()) < 0.02
    assert met, "no shape ran with partial sums"


def attend(q_parts, pages, requests, lens, starts, scale, **more):
    from atomserve_b200 import ops

    ctx = step_context(lens, starts)
    q = torch.cat(q_parts).cuda().to(pages.dtype).contiguous()
    return ops.paged_attention(q, pages.pools[0], pages.pools[1], pages.table(requests), ctx.req_q_start, ctx.req_pos_start,
                               num_requests=len(lens), max_context=ctx.max_context, scale=scale, host_q_lens=lens, **more).float().cpu()  # fmt: skip


SHAPES = [(10, 3, 16, 24, 1, 1), (64, 64, 16, 64, 2, 2), (16, 16, 16, 64, 5, 1), (100, 20, 16, 128, 2, 4), (1, 1, 4, 16, 2, 1), (33, 40, 8, 128, 4, 3),
          (70, 300, 16, 64, 1, 8), (300, 5, 16, 128, 8, 2), (64, 0, 16, 128, 3, 2)]  # fmt: skip


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window,keep,bs,hd,G,share", SHAPES)
def test_one_key_stands_out_at_the_edges_of_window_and_kept_positions(dtype, window, keep, bs, hd, G, share):
    """All keys are zero but one, whose parts' products (of both signs) sum to a large score and whose
    value is e_1 in one value head: a query sees it exactly when it is less than `window` behind or among
    the first `keep` positions, so the result is known in closed form; from single tokens and from
    portions that start before the edge."""
    H, scale, T = G * share, 0.5, 700
    a = torch.linspace(-1.0, 3.0, G) if G > 1 else torch.tensor([3.0])  # the parts' queries
    b = torch.full((G,), 20.0) / a.sum() if G > 1 else torch.tensor([20.0 / 3.0])
    a, b = rounded(a), rounded(b)
    score = float((a * b).sum()) * scale
    q = torch.zeros(1, H, G, hd)
    q[:, :, :, 0] = a
    marks = sorted({0, keep - 1, keep, keep + 1, 63, 64, 65, 300, 300 + bs, T - 1} & set(range(T)))
    value_head = G - 1
    for mark in marks:
        k, v = torch.zeros(T, G, hd), torch.zeros(T, G, hd)
        k[mark, :, 0], v[mark, value_head, 1] = b, 1.0
        pages = Pages([(G, hd), (G, hd)], bs, dtype, blocks=T // bs + 5, seed=mark)
        pages.put("r", k, v)
        for p in sorted({mark, mark + 1, mark + window - 1, mark + window, mark + window + 1, T - 1} & set(range(T))):
            seen = mark <= p and (p - mark < window or mark < keep)
            total = min(p + 1, window) + min(keep, max(0, p + 1 - window))
            want = math.exp(score) / (math.exp(score) + total - 1) if seen else 0.0
            one = attend([q], pages, ["r"], [1], [p], scale, window=window, keep_first=keep)[0, :, 1]
            lo = max(0, p - 40)
            many = attend([q.expand(p + 1 - lo, H, G, hd)], pages, ["r"], [p + 1 - lo], [lo], scale, window=window, keep_first=keep)[-1, :, 1]
            for got in (one, many):
                mine = got[value_head * share : (value_head + 1) * share]
                assert np.allclose(mine, want, rtol=2e-2 if dtype == torch.bfloat16 else 2e-5, atol=1e-6), (mark, p, mine, want)
                assert not got[: value_head * share].any(), "a head read another head's values"


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("hd,bs", [(24, 16), (64, 16), (128, 16)])
def test_kept_positions_for_heads_that_are_not_mixed(dtype, hd, bs):
    """`keep_first` belongs to the attention and not to the mix: ordinary grouped-query heads have it too."""
    H, G, T, window, keep = 4, 2, 300, 20, 9
    g = torch.Generator().manual_seed(hd)
    q, k, v = rounded(2 * torch.randn(T, H, hd, generator=g)), rounded(torch.randn(T, G, hd, generator=g)), rounded(torch.randn(T, G, hd, generator=g))
    ok = plain.visible(T, dict(size=window, keep_first=keep))
    scores = torch.einsum("ihd,jhd->hij", q.double(), k.double().repeat_interleave(2, 1)) * 0.2
    ref = torch.einsum("hij,jhd->ihd", plain.softmax_over(scores, ok), v.double().repeat_interleave(2, 1)).float()
    pages = Pages([(G, hd), (G, hd)], bs, dtype, blocks=T // bs + 5)
    pages.put("r", k, v)
    got = attend([q], pages, ["r"], [T], [0], 0.2, window=window, keep_first=keep)
    check(got.reshape(T, -1), ref.reshape(T, -1), dtype, "portion")
    got = attend([q[T - 1 :]], pages, ["r"], [1], [T - 1], 0.2, window=window, keep_first=keep)
    check(got.reshape(1, -1), ref[T - 1 :].reshape(1, -1), dtype, "single token")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,hd,bs", [(8, 2, 128, 16), (12, 4, 64, 16), (16, 4, 128, 32), (32, 8, 64, 16), (40, 1, 64, 8), (6, 3, 40, 4), (16, 8, 128, 16),
                                       (34, 2, 128, 16), (3, 3, 128, 64), (10, 5, 128, 16), (32, 8, 128, 16), (16, 16, 64, 16), (8, 8, 128, 4)])  # fmt: skip
@pytest.mark.parametrize("window,keep", [(None, 0), (150, 70), (40, 3)])
def test_attention_over_parts_in_mixed_batches(dtype, H, G, hd, bs, window, keep):
    """Random queries with a vector per key head: a long portion, one that starts mid-sequence, single
    tokens with few and many keys and short portions in one step (with and without the lengths on the
    host), against a plain softmax; then the single tokens alone, cut into several partitions."""
    from atomserve_b200 import ops

    g = torch.Generator().manual_seed(H * hd)
    shapes = {"a": (200, 0), "b": (90, 333), "c": (1, 700), "d": (1, 5), "e": (3, 64), "f": (1, 127), "g": (8, 0)}
    scale = 0.5 * (hd * G) ** -0.5
    pages = Pages([(G, hd), (G, hd)], bs, dtype, blocks=1700 // bs + 8)
    qs, refs = {}, {}
    for n, (new, start) in shapes.items():
        T = start + new
        q, k, v = rounded(3 * torch.randn(new, H, G, hd, generator=g)), rounded(torch.randn(T, G, hd, generator=g)), rounded(torch.randn(T, G, hd, generator=g))
        pages.put(n, k, v)
        i, j = torch.arange(start, T)[:, None], torch.arange(T)[None, :]
        ok = (j <= i) & ((i - j < window) | (j < keep)) if window else j <= i
        p = plain.softmax_over(torch.einsum("ihcd,jcd->hij", q.double(), k.double()) * scale, ok)
        qs[n], refs[n] = q, torch.einsum("hij,jhd->ihd", p, v.double().repeat_interleave(H // G, 1)).float()
    for names in (list(shapes), ["c", "a", "d"], ["b"], ["d", "e", "g"], ["c", "d", "f"]):
        lens, starts = [shapes[n][0] for n in names], [shapes[n][1] for n in names]
        ref = torch.cat([refs[n] for n in names])
        got = attend([qs[n] for n in names], pages, names, lens, starts, scale, window=window, keep_first=keep)
        check(got.reshape(ref.shape[0], -1), ref.reshape(ref.shape[0], -1), dtype, f"requests {names}", 0.02)
        ctx = step_context(lens, starts)
        q = torch.cat([qs[n] for n in names]).cuda().to(dtype).contiguous()
        args = (q, *pages.pools, pages.table(names), ctx.req_q_start, ctx.req_pos_start)
        kw = dict(num_requests=len(lens), max_context=ctx.max_context, window=window, scale=scale, keep_first=keep)
        got = ops.paged_attention(*args, **kw)
        check(got.reshape(ref.shape[0], -1), ref.reshape(ref.shape[0], -1), dtype, f"requests {names}, lengths unknown", 0.02)
        if max(lens) == 1 and dtype == torch.bfloat16 and hd in (64, 128):
            for tiles in (1, 3):
                got = ops.paged_attention(*args, **kw, host_q_lens=lens, partitions=(tiles, -(-701 // (64 * tiles)) + 1))
                check(got.reshape(ref.shape[0], -1), ref.reshape(ref.shape[0], -1), dtype, f"partitions of {tiles} tiles", 0.02)


def mixer_weights(g, d, m):
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    cfg = dict(width=d, vocab=4, streams=1, embedding=dict(bigram=dict(buckets=1)), layers=[dict(type="attention", mixer=m, mlp=None)])
    w = {"x." + k[len("l0.mix."):]: v for k, v in plain.random_checkpoint(cfg, H * 7 + D).items() if k.startswith("l0.mix.")}
    w["x.vmix"] = torch.tensor(0.4)
    return w


def mixer_part(d, m, eps, value_mix):
    """The mixer as the model's description names it."""
    from atomserve_b200.config.registry import config_from_dict
    from atomserve_b200.parts import build_part

    cfg = dict(architecture="Lidizen", vocab=8, width=d, streams=1, norm=dict(eps=eps), embedding=dict(bigram=dict(buckets=2, mul_prev=1, mul_cur=1)),
               layers=[dict(type="attention", mixer=m, mlp=None)])  # fmt: skip
    arch, config = config_from_dict(cfg)
    spec = arch.build_spec(config).layers[0].mixer
    return build_part("mixer", type(spec)(spec.kind, dict(spec.params, value_mix=value_mix), "x."), d)


MIXERS = [
    attention(6, 3, 24, 16, 0.3, window=10, keep=3, rot=(100.0, 8)),
    attention(4, 2, 12, 40, 0.4, window=33, keep=18, rot=(30.0, 12)),
    attention(2, 1, 8, 8, 0.5, window=1, keep=1),
    attention(3, 3, 20, 24, 0.35, window=5, rot=(30.0, 20)),
    attention(8, 2, 128, 128, 0.1, window=16, keep=6, rot=(10000.0, 64)),
    attention(8, 4, 48, 64, 0.15, window=19, keep=21, rot=(500.0, 40)),
    attention(16, 4, 64, 64, 0.12, rot=(100.0, 64)),
    attention(20, 1, 128, 96, 0.1, window=12, keep=4, rot=(100.0, 128)),
    attention(8, 8, 64, 64, 0.12, window=9, keep=2, rot=(100.0, 32)),
]  # fmt: skip


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("mixes", [False, True])
@pytest.mark.parametrize("layer", MIXERS, ids=lambda m: f"{m['mixer']['heads']}x{m['mixer']['dim']}")
def test_mixer_alone(dtype, layer, mixes):
    """A sequence in two portions and then token by token through scattered pages equals the plain
    mixer on the whole sequence; then two requests in one step, one of them starting mid-sequence;
    as a layer that keeps its values and as one that mixes them with an earlier layer's."""
    from atomserve_b200.parts import CacheView
    from atomserve_b200.parts.mixed_heads import FIRST_VALUES

    d, T, bs = 72, 45, 4
    m = layer["mixer"]
    G, hd, kv = m["kv_heads"], max(m["dim"], m["vdim"]), m["kv_heads"] * m["vdim"]
    g = torch.Generator().manual_seed(m["heads"] * 7 + m["dim"])
    w = mixer_weights(g, d, m)
    part = mixer_part(d, m, EPS, "mixed" if mixes else "first")
    part.load(on_device(w, dtype))
    h, h2 = rounded(3 * torch.randn(T, d, generator=g)), rounded(3 * torch.randn(9, d, generator=g))
    f1, f2 = rounded(torch.randn(T, kv, generator=g)), rounded(torch.randn(9, kv, generator=g))
    (ref, own), (ref2, own2) = (plain.attention(x.double(), doubles(w, "x."), m, EPS, f.double() if mixes else None) for x, f in ((h, f1), (h2, f2)))
    assert part.cache_spec().tensors[0].width == hd and part.cache_spec().keep_first == (m.get("mask") or {}).get("keep_first", 0)
    view = CacheView(k=torch.ones(24, G, bs, hd, device="cuda", dtype=dtype), block_size=bs)
    view.v = torch.ones_like(view.k)
    table = torch.randperm(24, generator=g).tolist()
    mine, other = table[:12], table[12:]

    def run(x, firsts, lens, starts):
        ctx = step_context(lens, starts)
        if mixes:
            ctx.plans[FIRST_VALUES] = firsts.cuda().to(dtype).contiguous()
        y = part.forward(x.cuda().to(dtype), None, ctx, view)
        assert y.dtype == torch.float32  # what a block that sums in float32 takes
        return y, (None if mixes else ctx.plans[FIRST_VALUES])

    view.block_tables = i32([mine])
    outs, kept = [], []
    for start, n in [(0, 14), (14, 2), (16, 9)] + [(p, 1) for p in range(25, T - 6)]:
        view.slots = paged(mine, bs, range(start, start + n))
        y, v = run(h[start : start + n], f1[start : start + n], [n], [start])
        outs.append(y)
        kept.append(v)
    done = T - 6
    view.block_tables = i32([other, mine])
    view.slots = torch.cat([paged(other, bs, range(9)), paged(mine, bs, range(done, T))])
    both, v = run(torch.cat([h2, h[done:]]), torch.cat([f2, f1[done:]]), [9, 6], [0, done])
    check(torch.cat(outs + [both[9:]]), ref.float(), dtype, "portions and single tokens", 0.05)
    check(both[:9], ref2.float(), dtype, "the second request beside it", 0.05)
    if not mixes:
        check(torch.cat(kept + [v[9:]]), own.float(), dtype, "values for later layers", 0.02)
        check(v[:9], own2.float(), dtype, "the second request's values", 0.02)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("d,T,E,top,ff", [(72, 40, 5, 2, 40), (64, 9, 2, 2, 16), (100, 33, 1, 1, 12), (256, 300, 8, 3, 128), (96, 70, 7, 4, 8), (64, 5, 4, 1, 24)])
def test_squared_relu_experts_alone(dtype, d, T, E, top, ff):
    """The largest biased logits win and are weighted among themselves; a bias large enough to decide
    the choice; experts without a gate. The inputs are what the plain router separates by more than rounding."""
    from atomserve_b200.models.lidizen import _feed_forward
    from atomserve_b200.parts import build_part

    mlp = dict(kind="moe", expert=dict(ff=ff), router=dict(experts=E, top=top))
    cfg = dict(width=d, vocab=4, streams=1, embedding=dict(bigram=dict(buckets=1)), layers=[dict(mixer=dict(heads=1, kv_heads=1, dim=8, vdim=8), mlp=mlp)])
    w = {k[len("l0.mlp."):]: v for k, v in plain.random_checkpoint(cfg, seed=E).items() if k.startswith("l0.mlp.")}
    g = torch.Generator().manual_seed(d + E)
    w["router.b"] = 2 * torch.randn(E, generator=g)
    h = rounded(torch.randn(T, d, generator=g))
    clear = plain.choice_margin(h.double(), w, top) > 2e-2
    assert clear.sum() >= T // 2
    spec = _feed_forward(mlp, "x.")
    part = build_part("feed_forward", spec, d)
    part.load(on_device({"x." + k: v for k, v in w.items()}, dtype))
    assert part.sums_alone()
    got = part.forward(h.cuda().to(dtype), None, None)
    assert got.dtype == torch.float32
    ref = plain.experts(h.double(), w, mlp).float()
    check(got[clear.cuda()], ref[clear], dtype, "experts", 0.03)
    chosen, _ = plain.route(h.double(), w, top)
    without, _ = plain.route(h.double(), {**w, "router.b": torch.zeros(E)}, top)
    assert E == top or (chosen.sort(-1).values != without.sort(-1).values).any(), "the bias never changed a choice"


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("d,ff,T", [(72, 100, 9), (256, 384, 5), (256, 512, 300)])
def test_dense_feed_forward_alone(dtype, d, ff, T):
    from atomserve_b200.models.lidizen import _feed_forward
    from atomserve_b200.parts import build_part

    g = torch.Generator().manual_seed(ff)
    w = {"f." + n: rounded(torch.randn(s, generator=g) * s[1] ** -0.5) for n, s in (("gate", (ff, d)), ("up", (ff, d)), ("down", (d, ff)))}
    w.update({"f.gate.b": torch.randn(ff, generator=g), "f.up.b": torch.randn(ff, generator=g), "f.down.b": torch.randn(d, generator=g)})
    part = build_part("feed_forward", _feed_forward(dict(kind="dense", ff=ff), "f."), d)
    part.load(on_device(w, dtype))
    h = rounded(2 * torch.randn(T, d, generator=g))
    check(part.forward(h.cuda().to(dtype), None, step_context([T], [0])), plain.dense(h.double(), doubles(w, "f.")).float(), dtype, "feed-forward")


# ---- whole models through the step function -------------------------------------------------

LENGTHS = {"a": [5, 49, 130, 1, 64], "b": [33, 2, 97, 40], "c": [300, 9, 70], "d": [70, 3, 130, 20]}


def oracle(cfg, w, prompt):
    return plain.forward(prompt, w, cfg).float()


def sure_positions(cfg, w, prompt, margin):
    """[n] bool: positions at which every router's choice leads by `margin` at least. Elsewhere
    rounding may choose another expert, which is a jump and no rounding error: such positions are
    left out of a comparison (0.03 of a logit for bfloat16, 1e-4 for float32)."""
    margins = []
    plain.forward(prompt, w, cfg, margins=margins)
    return torch.stack(margins).min(0).values > margin if margins else torch.ones(len(prompt), dtype=torch.bool)


def sure_both(cfg, w, p):
    return dict(float32=sure_positions(cfg, w, p, 1e-4), bfloat16=sure_positions(cfg, w, p, 0.03))


def judged(got, ref, dtype, what, lossy, sure):
    keep = sure[dtype]
    if keep.any():
        judge(got.float().cpu()[keep], ref[keep], dtype, what, lossy[keep])


def allowance(cfg, w, prompt, ref):
    """What rounding alone does, per position: the largest error of the plain implementation itself
    over several ways of rounding to 16 bits everything an engine may keep in them."""
    return torch.stack([row_errors(plain.forward(prompt, w, cfg, stored=f), ref) for f in ROUNDINGS]).max(0).values


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    out = {}
    for name, (cfg, bs) in LIDIZEN.items():
        w = plain.random_checkpoint(cfg, seed=31)
        folder = write_folder(cfg, w, tmp_path_factory.mktemp(f"lidizen_{name}"))
        ps = prompts(cfg, LENGTHS[name], seed=8)
        refs = [oracle(cfg, w, p) for p in ps]
        sure = [sure_both(cfg, w, p) for p in ps]
        assert all(s["bfloat16"].float().mean() > 0.25 for s in sure if len(s["bfloat16"]) > 8), "too few positions are left to compare"
        out[name] = (cfg, bs, folder, w, ps, refs, [allowance(cfg, w, p, r) for p, r in zip(ps, refs)], sure)
    return out


def replayer(folder, dtype, bs, max_tokens, **more):
    from atomserve_b200.engine.replay import TraceReplayer

    return TraceReplayer(folder, dtype, max_tokens, bs, **more)


CASES = [(n, d) for n in LIDIZEN for d in ("float32", "bfloat16")]


@pytest.mark.parametrize("name,dtype", CASES)
def test_whole_then_token_by_token_then_portions(models, name, dtype):
    cfg, bs, folder, _, ps, refs, tols, sures = models[name]
    rp = replayer(folder, dtype, bs, max(-(-len(p) // 64) * 64 for p in ps))
    sizes = [2, 7, 3, 16, 2, 17, 5, 31, 2, 9, 1, 33]
    for i, (p, ref, tol, sure) in enumerate(zip(ps, refs, tols, sures)):
        n = len(p)

        def held(logits, places, what):
            judged(logits, ref[places], dtype, f"{name} request {i} {what}", tol[places], {k: v[places] for k, v in sure.items()})

        held(rp.step([dict(id=i, tokens=p, want=list(range(n)))], end=[i]), list(range(n)), "whole")
        head = max(n - 40, 0)
        if head:
            held(rp.step([dict(id=i, tokens=p[:head], want=[0, head - 1])], end=[]), [0, head - 1], "head")
        for j in range(head, n):
            held(rp.step([dict(id=i, tokens=[p[j]], want=[0])], end=[i] if j == n - 1 else []), [j], f"position {j} alone")
        at, k = 0, i
        while at < n:
            m = min(sizes[k % len(sizes)], n - at)
            k += 1
            logits = rp.step([dict(id=i, tokens=p[at : at + m], want=list(range(m)))], end=[i] if at + m == n else [])
            held(logits, list(range(at, at + m)), f"portion {at}:{at + m}")
            at += m


@pytest.mark.parametrize("name,dtype", CASES)
def test_mixed_requests_reusing_pages_and_slots(models, name, dtype):
    """Up to four live requests in four state slots, portions beside single tokens, in a pool so
    small that pages and slots freed by finished requests are taken again; every request appears
    four times, each equal to itself alone."""
    cfg, bs, folder, _, ps, refs, tols, sures = models[name]
    ps3, refs3, tols3, sures3 = ps * 4, refs * 4, tols * 4, sures * 4
    biggest = sorted((-(-len(p) // 64) * 64 for p in ps3), reverse=True)
    rp = replayer(folder, dtype, bs, sum(biggest[:4]), max_live=4)
    rng = np.random.default_rng(13)
    for entries, end in mixed_trace(ps3, rng, largest=40):
        logits = rp.step([dict(id=e["id"], tokens=e["tokens"], want=e["want"]) for e in entries], end=end)
        row = 0
        for e in entries:
            n = len(e["tokens"])
            places = list(range(e["at"], e["at"] + n))
            judged(logits[row : row + n], refs3[e["id"]][places], dtype, f"{name} request {e['id']} at {e['at']}",
                   tols3[e["id"]][places], {k: v[places] for k, v in sures3[e["id"]].items()})
            row += n
    assert sum(len(p) for p in ps3) > rp.cache.num_blocks * bs, "the pool was large enough to never reuse a page"


@pytest.fixture(scope="module")
def long_prompts(models):
    out = {}
    for name in ("a", "c"):
        cfg, w = models[name][0], models[name][3]
        p = prompts(cfg, [300], seed=12)[0]
        ref = oracle(cfg, w, p)
        out[name] = (p, ref, allowance(cfg, w, p, ref), sure_both(cfg, w, p))
    return out


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding(models, long_prompts, dtype):
    """280 tokens one by one after a short prompt, from CUDA graphs: windows move over decoded tokens,
    the kept positions stay, the last token and the first layer's values travel with their step."""
    for name in ("a", "c"):
        cfg, bs, folder, w = models[name][:4]
        p, ref, tol, sure = long_prompts[name]
        rp = replayer(folder, dtype, bs, 320)
        assert rp.runner.use_graphs
        rp.step([dict(id="x", tokens=p[:20], want=[])], end=[])
        for j in range(20, len(p)):
            logits = rp.step([dict(id="x", tokens=[p[j]], want=[0])], end=[])
            if j % 9 == 0 or j > 290:
                judged(logits, ref[j : j + 1], dtype, f"{name} decode position {j}", tol[j : j + 1], {k: v[j : j + 1] for k, v in sure.items()})
        held = rp.live["x"][0]
        windowed = [(g.spec, table) for g, table in zip(rp.cache.groups, held.block_tables) if g.spec.window]
        assert len(windowed) >= 3
        for spec, table in windowed:  # pages between the kept ones and the window have gone back to the pool
            kept = -(-spec.keep_first // bs)
            assert all(b >= 0 for b in table[:kept]) and len(table) == -(-len(p) // bs)
            assert sum(b >= 0 for b in table) <= kept + -(-spec.window // bs) + 1


def test_the_streams_after_every_layer(models):
    """The sum of the float32 streams after each layer against the plain implementation's, in float32."""
    for name in ("a", "b", "d"):
        cfg, bs, folder, w, ps = models[name][:5]
        p = ps[1]
        layers = []
        plain.forward(p, w, cfg, streams=layers)
        rp = replayer(folder, "float32", bs, 64)
        seen = []
        for block in rp.model.blocks:
            inner = block.forward_chain

            def wrapped(*a, _inner=inner, **k):
                out = _inner(*a, **k)
                assert out[0].shape[1] == cfg["streams"]
                seen.append(out[0].sum(1).double().cpu())
                return out

            block.forward_chain = wrapped
        rp.step([dict(id=0, tokens=p, want=[0])], end=[0])
        assert len(seen) == len(layers)
        for i, (got, ref) in enumerate(zip(seen, layers)):
            assert float((got - ref).abs().max() / ref.abs().max()) < 2e-5, f"{name}: streams after layer {i}"


# ---- generation through the engine -----------------------------------------------------------

GREEDY = dict(temperature=0.0, ignore_eos=True)


def engine_for(folder, dtype, bs, **kw):
    from atomserve_b200.config import EngineConfig
    from atomserve_b200.engine.engine import create_engine
    from atomserve_b200.weights import load_model

    _, _, model = load_model(folder, dtype, "cuda")
    config = EngineConfig(**{"block_size": bs, "num_blocks": 64, "max_model_len": 64 * bs, "max_num_seqs": 8,
                             "max_num_batched_tokens": 256, **kw})  # fmt: skip
    return create_engine(model, config, sampler_seed=0)


@pytest.mark.parametrize("name", ["a", "b", "d"])
def test_greedy_generation_through_the_engine(models, name):
    """The engine's own entry point and scheduler: batched, in portions under a small budget, and
    with so few pages that requests are preempted and recomputed (state slots given back and
    zeroed again); float32 tokens equal the plain implementation's."""
    from atomserve_b200.engine.sequence import SamplingParams

    cfg, bs, folder, w = models[name][:4]
    ps = prompts(cfg, [5, 17, 33], seed=3)
    expect = [plain.greedy_generate(p, w, cfg, 8) for p in ps]
    params = SamplingParams(max_tokens=8, **GREEDY)
    assert engine_for(folder, "float32", bs).generate(ps, params) == expect
    chunked = engine_for(folder, "float32", bs, max_num_batched_tokens=8, max_num_seqs=4)
    assert chunked.generate(ps, params) == expect
    assert chunked.num_steps > 8 + 3
    short = engine_for(folder, "float32", bs, num_blocks=7, max_model_len=7 * bs, enable_prefix_caching=False)
    n = bs + 8
    ps2 = prompts(cfg, [bs + 3, bs + 5, 2 * bs - 1], seed=5)
    assert short.generate(ps2, SamplingParams(max_tokens=n, **GREEDY)) == [plain.greedy_generate(p, w, cfg, n) for p in ps2]
    assert short.stats()["kv_blocks_used"] == 0


def test_greedy_generation_in_bfloat16_picks_near_best_tokens(models):
    from atomserve_b200.engine.sequence import SamplingParams

    cfg, bs, folder, w = models["c"][:4]
    ps = prompts(cfg, [40, 7, 90], seed=3)
    outs = engine_for(folder, "bfloat16", bs, max_num_batched_tokens=48).generate(ps, SamplingParams(max_tokens=12, **GREEDY))
    for p, out in zip(ps, outs):
        assert len(out) == 12
        full = list(p) + list(out)
        ref = oracle(cfg, w, full)
        sure = sure_positions(cfg, w, full, 0.03)
        spread = float((ref - ref.mean(-1, keepdim=True)).pow(2).mean().sqrt())
        for i, token in enumerate(out):
            row = ref[len(p) + i - 1]
            if sure[len(p) + i - 1]:
                assert float(row.max() - row[token]) <= 0.2 * spread, f"token {i} lies far below the best"


def test_command_line_and_random_weights(tmp_path):
    """`python -m atomserve_b200` on a Lidizen folder written by the package's own random-weights
    writer from a configuration that round-trips through config.json."""
    import json
    import subprocess
    import sys

    from atomserve_b200.config.registry import config_from_dict
    from atomserve_b200.weights.random_init import write_model_folder

    arch, config = config_from_dict(LIDIZEN["c"][0])
    folder = write_model_folder(config, 3, tmp_path / "m", "bfloat16")
    assert json.loads((folder / "config.json").read_text())["architecture"] == "Lidizen"
    done = subprocess.run([sys.executable, "-m", "atomserve_b200", str(folder), "--prompt-ids", "5,6,7", "--max-tokens", "6",
                           "--temperature", "0"], capture_output=True, text=True, timeout=600)  # fmt: skip
    assert done.returncode == 0, done.stderr[-2000:]
    assert len(json.loads(done.stdout.strip().splitlines()[-1])["output_ids"]) == 6
