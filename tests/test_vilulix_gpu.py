"""The Vilulix design on the GPU against the plain implementation: each mechanism's part alone,
then whole models through the trace replayer in every way of cutting requests into steps, then
greedy generation through the engine and its scheduler."""

import numpy as np
import pytest
import torch

import plain_vilulix as plain
from gefilix_helpers import check, prompts, write_folder
from helpers import mixed_trace
from test_engine_gpu import step_context
from test_tigesun_gpu import ROUNDINGS, Pages, doubles, i32, judge, rounded, row_errors
from tiny_vilulix import VILULIX, delta, latent, parallel, window

pytestmark = pytest.mark.gpu
DTYPES = [torch.float32, torch.bfloat16]
EPS = 1e-5
F64 = torch.float64


def on_device(w, dtype):
    """Matrices in the compute dtype, everything with one axis (and convolution taps) float32."""
    return {k: v.cuda().to(dtype if v.dim() == 2 and not k.endswith("conv") else torch.float32) for k, v in w.items()}


def paged(table, bs, positions):
    return i32([table[p // bs] * bs + p % bs for p in positions])


# ---- each mechanism alone -------------------------------------------------------------------


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("d", [72, 100, 256, 1030, 2048, 4100])
def test_sum_of_terms_and_both_norms_of_it(dtype, d):
    from atomserve_b200 import ops

    g = torch.Generator().manual_seed(d)
    x, *ys = (3 * torch.randn(9, d, generator=g) for _ in range(5))
    g1, g2, bias = 1 + 0.3 * torch.randn(d, generator=g), 1 + 0.3 * torch.randn(d, generator=g), torch.randn(d, generator=g)
    factors = [1.0, -0.7, 1.6, 0.3]
    for n, with_x, with_bias in ((0, True, False), (1, True, False), (2, False, True), (3, True, True), (4, True, False)):
        s = (x.double() if with_x else 0) + sum(f * y.double() for f, y in zip(factors[:n], ys)) + (bias.double() if with_bias else 0)
        terms = [(y.cuda(), f) for f, y in zip(factors[:n], ys)]
        out, h1, h2 = ops.residual_terms_norm(x.cuda() if with_x else None, terms, g1.cuda(), g2.cuda(), EPS, dtype,
                                              bias=bias.cuda() if with_bias else None)  # fmt: skip
        check(out, s.float(), torch.float32, f"the sum of {n} terms")
        check(h1, (plain.rms_unit(s, EPS) * g1.double()).float(), dtype, "first norm", 0.01)
        check(h2, (plain.rms_unit(s, EPS) * g2.double()).float(), dtype, "second norm", 0.01)
        if n:
            out, h1, h2 = ops.residual_terms_norm(x.cuda() if with_x else None, terms, None, None, 0.0, dtype,
                                                  bias=bias.cuda() if with_bias else None)  # fmt: skip
            assert h1 is None and h2 is None
            check(out, s.float(), torch.float32, "the sum alone")
    with pytest.raises(ops.KernelLibraryError):
        ops.residual_terms_norm(x.cuda(), [(y.cuda(), 1.0) for y in ys + ys[:1]], None, None, 0.0, dtype)


def test_sum_whose_last_term_is_a_products_partial_sums():
    """With few tokens a layer's last product stays as the GEMM's partial sums and the sum's kernel adds
    them up: the finished product as a term, up to the order in which a row's sums are formed."""
    from atomserve_b200 import ops
    from atomserve_b200.ops.linear import PartialSums

    g = torch.Generator().manual_seed(4)
    met = 0
    for T, d, K in ((1, 256, 512), (5, 336, 1024), (8, 2048, 2048), (33, 256, 392)):
        inner = torch.randn(T, K, generator=g).bfloat16().cuda()
        w = (torch.randn(d, K, generator=g) * K**-0.5).bfloat16().cuda()
        x, y1, y2 = (torch.randn(T, d, generator=g).cuda() for _ in range(3))
        g1, g2 = ((1 + 0.1 * torch.randn(d, generator=g)).cuda() for _ in range(2))
        for terms, gains in (([], (g1, g2)), ([(y1, 0.7)], (g1, None)), ([(y1, -1.5), (y2, 0.4)], (g1, g2)), ([(y1, 1.0)], (None, None))):
            whole = ops.residual_terms_norm(x, [*terms, (ops.linear(inner, w, out_dtype=torch.float32), 1.3)], *gains, EPS, torch.bfloat16)
            y = ops.linear_for_stream(inner, w)
            met += isinstance(y, PartialSums)
            fused = ops.residual_terms_norm(x, [*terms, (y, 1.3)], *gains, EPS, torch.bfloat16)
            assert float((whole[0] - fused[0]).abs().max() / whole[0].abs().max()) < 2e-6, (T, d, K)
            for a, b, gain in zip(whole[1:], fused[1:], gains):
                assert (a is None) == (b is None) == (gain is None)
                assert gain is None or bool(((a.float() - b.float()).abs() <= 2.0**-7 * a.float().abs() + 1e-30).all()), (T, d, K)
    assert met, "no shape ran with partial sums"


@pytest.mark.parametrize("dtype", DTYPES)
def test_gains_around_zero_and_the_opening_of_a_pass(dtype):
    from atomserve_b200.parts import PartSpec, build_part

    d, T = 72, 13
    g = torch.Generator().manual_seed(1)
    w = 0.3 * torch.randn(d, generator=g)
    x, x0 = torch.randn(T, d, generator=g), torch.randn(T, d, generator=g)
    norm = build_part("norm", PartSpec("stream_rms_norm", dict(eps=EPS, centre=1.0, tensor="n")), d)
    norm.load({"n": w.cuda()})
    norm.bind_dtype(dtype)
    check(norm.forward(x.cuda()), plain.centred_gain_norm(x.double(), w, EPS).float(), dtype, "the norm", 0.01)
    check(norm.forward(x.cuda(), i32([4, 0])), plain.centred_gain_norm(x.double(), w, EPS).float()[[4, 0]], dtype, "chosen rows", 0.01)
    step = build_part("stream_step", PartSpec("add_input"), d)
    step.bind_dtype(dtype)
    check(step.forward(x.cuda(), x0.cuda(), 1, None), x + x0, torch.float32, "the opening alone")

    class Opened:
        def block_norms(self):
            return norm.gain, None, EPS

    out, (h1, h2) = step.forward_then(x.cuda(), x0.cuda(), 2, None, Opened())
    assert h2 is None
    check(out, x + x0, torch.float32, "the opening")
    check(h1, plain.centred_gain_norm((x + x0).double(), w, EPS).float(), dtype, "the norm of the block it opens", 0.01)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("C,K", [(48, 4), (37, 3), (130, 1), (64, 2), (24, 9), (16, 20)])
def test_convolution_with_its_state(dtype, C, K):
    """Portions of one token, fewer than the taps, across the kernel's tile of 32 and longer than it; two
    requests in one step, slots in another order, other slots untouched."""
    from atomserve_b200 import ops

    g = torch.Generator().manual_seed(C + K)
    taps = torch.randn(C, K, generator=g)
    off, columns = 3 if C % 2 else 8, C + 16
    seqs = {n: rounded(torch.randn(k, columns, generator=g)) for n, k in (("a", 150), ("b", 41))}
    refs = {n: plain.silu(plain.causal_convolution(s[:, off : off + C].double(), taps.double())).float() for n, s in seqs.items()}
    state = torch.zeros(5, K - 1, C, device="cuda")
    at, slot = dict(a=0, b=0), dict(a=3, b=1)
    for step in ([("a", 2)], [("b", 1), ("a", 1)], [("a", 33), ("b", 2)], [("a", 1)], [("b", 32), ("a", 32)], [("a", 70)], [("b", 6), ("a", 11)]):
        lens = [n for _, n in step]
        ctx = step_context(lens, [at[r] for r, _ in step], [slot[r] for r, _ in step])
        x = torch.cat([seqs[r][at[r] : at[r] + n] for r, n in step]).cuda().to(dtype)
        out = ops.causal_conv_silu(x, off, taps.cuda(), state, ctx.state_slots, ctx.req_q_start, len(lens), lens).cpu()
        row = 0
        for r, n in step:
            check(out[row : row + n], refs[r][at[r] : at[r] + n], dtype, f"{r} at {at[r]}", 0.02)
            row, at[r] = row + n, at[r] + n
            held = seqs[r][max(at[r] - (K - 1), 0) : at[r], off : off + C]
            want = torch.cat([torch.zeros(K - 1 - held.shape[0], C), held])
            assert torch.equal(state[slot[r]].cpu(), want), (r, at[r])
    assert at == {n: len(s) for n, s in seqs.items()} and not state[[0, 2, 4]].any()


DELTA_SIZES = [(2, 1, 16, 24), (3, 3, 24, 40), (4, 2, 64, 64), (2, 1, 128, 128), (1, 1, 130, 20), (2, 1, 256, 33), (2, 2, 300, 8),
               (5, 1, 8, 3), (6, 2, 32, 96), (1, 1, 1, 1), (2, 2, 33, 130), (1, 1, 600, 36)]  # fmt: skip


def delta_inputs(g, n, H, G, D, V):
    q, k, v = (rounded(torch.randn(n, w, generator=g)) for w in (G * D, G * D, H * V))
    z = torch.randn(n, 2 * H, generator=g) * 2
    return torch.cat([q, k, v], 1), z


def delta_reference(x, z, H, G, D, V, dt_bias, a_log):
    n, share = x.shape[0], H // G
    q, k, v = (t.double() for t in x.split([G * D, G * D, H * V], 1))
    q = plain.unit_vectors(q.view(n, G, D)).repeat_interleave(share, 1) * D**-0.5
    k = plain.unit_vectors(k.view(n, G, D)).repeat_interleave(share, 1)
    g = torch.exp(-torch.exp(a_log.double()) * torch.nn.functional.softplus(z[:, H:].double() + dt_bias.double()))
    o, S = plain.delta_recurrence(q, k, v.view(n, H, V), g, torch.sigmoid(z[:, :H].double()))
    return o.reshape(n, H * V).float(), S.float()


def run_delta(x, z, state, slots, lens, H, G, D, V, dt_bias, a_log, dtype):
    from atomserve_b200 import ops

    ctx = step_context(lens, [0] * len(lens), slots)
    plan = ops.plan_delta(lens, H, D, V, torch.device("cuda"))
    return ops.delta_rule(x.cuda().to(dtype), 0, G * D, 2 * G * D, z.cuda(), 0, H, dt_bias.cuda(), a_log.cuda(), state, ctx.state_slots,
                          ctx.req_q_start, len(lens), kv_heads=G, plan=plan).cpu()  # fmt: skip


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,D,V", DELTA_SIZES)
def test_delta_rule_alone(dtype, H, G, D, V, monkeypatch):
    """Whole (in chunks), token by token, in portions on both sides of the limit between the two forms and
    of a chunk's 32 and 64 tokens, unequal requests in one step with slots in another order, and a step
    whose chunks take several passes: outputs and states against the plain recurrence, in 32 bits
    whatever the inputs' type. Decays reach from near 0 to near 1."""
    from atomserve_b200.ops import delta as delta_ops

    gen = torch.Generator().manual_seed(H * 1000 + D)
    dt_bias, a_log = torch.randn(H, generator=gen) - 1, torch.randn(H, generator=gen) - 1
    lens = (170, 33, 1)
    seqs = [delta_inputs(gen, n, H, G, D, V) for n in lens]
    refs = [delta_reference(x, z, H, G, D, V, dt_bias, a_log) for x, z in seqs]
    state = torch.zeros(6, H, D, V, device="cuda")
    args = (H, G, D, V, dt_bias, a_log, dtype)

    def held(got, ref, what):  # (the inputs are exact in 16 bits, the rest is float32)
        err = float((got.double() - ref.double()).abs().max() / ref.double().abs().max())
        assert err < 2e-5, f"{what}: {err:.3g}"

    x, z = seqs[0]
    held(run_delta(x, z, state, [2], [lens[0]], *args), refs[0][0], "whole")
    held(state[2].cpu(), refs[0][1], "the state after it")
    assert not state[[0, 1, 3, 4, 5]].any(), "a slot other than the request's was written"
    state.zero_()
    got, at = [], 0
    for n in (1, 24, 25, 2, 1, 64, 3, 50):
        got.append(run_delta(x[at : at + n], z[at : at + n], state, [4], [n], *args))
        at += n
    assert at == lens[0]
    held(torch.cat(got), refs[0][0], "in portions")
    held(state[4].cpu(), refs[0][1], "the state after portions")
    state.zero_()
    got = [run_delta(x[t : t + 1], z[t : t + 1], state, [0], [1], *args) for t in range(60)]
    held(torch.cat(got), refs[0][0][:60], "token by token")
    state.zero_()
    per_chunk = 4 * H * sum(delta_ops._workspace_sizes(64 if D <= 128 else 32, D, V))
    monkeypatch.setattr(delta_ops, "WORKSPACE_BYTES", 2 * per_chunk)
    out = run_delta(torch.cat([s[0] for s in seqs]), torch.cat([s[1] for s in seqs]), state, [5, 0, 3], list(lens), *args)
    held(out, torch.cat([r[0] for r in refs]), "three requests in one step, in several passes")
    for slot, (_, S) in zip((5, 0, 3), refs):
        held(state[slot].cpu(), S, "a state after the joint step")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("D,V", [(24, 16), (128, 64), (200, 8)])
def test_a_value_written_once_is_found_far_away(dtype, D, V):
    """Decay 1 and beta 1: a value written at key e_0 among hundreds of writes at e_1 is read back
    unchanged wherever it lies (the first token, both sides of chunk borders, the token itself), never
    before, and a second write at e_0 replaces it. From one long portion, and from single tokens behind
    a portion."""
    T, H, G = 300, 2, 1
    dt_bias, a_log = torch.full((H,), -200.0), torch.zeros(H)  # softplus(-200): no decay
    z = torch.zeros(T, 2 * H)
    z[:, :H] = 200.0  # sigmoid: 1
    probes = sorted({0, 1, 31, 32, 63, 64, 65, 127, 128, 250, T - 1})
    for mark in (0, 1, 31, 32, 63, 64, 100, 191, 192, T - 1):
        second = mark + 70 if mark + 70 < T else None
        x = torch.zeros(T, 2 * G * D + H * V)
        x[:, 0] = 1.0  # every query asks for e_0
        x[:, G * D + 1] = 1.0  # every key is e_1 ...
        values = x[:, 2 * G * D :]
        values += 0.25
        for at, value in ((mark, 2.0), (second, -3.0)):
            if at is not None:
                x[at, G * D], x[at, G * D + 1] = 1.0, 0.0  # ... but the marked ones
                values[at] = value
        state = torch.zeros(2, H, D, V, device="cuda")
        whole = run_delta(x, z, state, [1], [T], H, G, D, V, dt_bias, a_log, dtype)
        state.zero_()
        cut = 240
        head = run_delta(x[:cut], z[:cut], state, [0], [cut], H, G, D, V, dt_bias, a_log, dtype)
        tail = [run_delta(x[t : t + 1], z[t : t + 1], state, [0], [1], H, G, D, V, dt_bias, a_log, dtype) for t in range(cut, T)]
        for got in (whole, torch.cat([head, *tail])):
            for p in sorted(set(probes) | {max(mark - 1, 0), mark} | ({second - 1, second} if second else set())):
                want = 0.0 if p < mark else (-3.0 if second is not None and p >= second else 2.0)
                assert torch.allclose(got[p], torch.full((H * V,), want * D**-0.5), rtol=1e-5, atol=1e-6), (mark, p, want)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,D,V,dims,interleaved", [(6, 2, 24, 16, 12, False), (4, 4, 16, 32, 16, False), (8, 2, 64, 64, 32, False),
                                                      (4, 1, 128, 128, 128, False), (3, 3, 10, 14, 0, False), (2, 1, 32, 8, 8, True)])  # fmt: skip
def test_norm_over_the_projection_and_rotation(dtype, H, G, D, V, dims, interleaved):
    """q and k normed over all heads at once, then turned at positions near and far (float32 angles),
    zeros behind what a head holds; the columns begin inside a wider product; pages are filled with
    ones beforehand: a slot used again keeps nothing of its former owner."""
    from atomserve_b200 import ops

    bs, hd, col = 4, max(D, V), 16
    g = torch.Generator().manual_seed(D + dims)
    positions = [0, 1, 2, 7, 98, 99, 1000, 30000]
    T = len(positions)
    q, k, v = (rounded(torch.randn(T, n, generator=g) * (1 + t)) for t, n in enumerate((H * D, G * D, G * V)))
    gq, gk = 1 + 0.3 * torch.randn(H * D, generator=g), 1 + 0.3 * torch.randn(G * D, generator=g)
    inv = torch.tensor([100.0 ** (-2.0 * i / max(dims, 1)) for i in range(dims // 2)], dtype=F64)

    def turned(x, heads):
        out = x.view(T, heads, D).clone()
        for t, p in enumerate(positions):
            for i in range(dims // 2):
                a, b = (2 * i, 2 * i + 1) if interleaved else (i, i + dims // 2)
                c, s = torch.cos(p * inv[i]), torch.sin(p * inv[i])
                u, w = x.view(T, heads, D)[t, :, a], x.view(T, heads, D)[t, :, b]
                out[t, :, a], out[t, :, b] = u * c - w * s, w * c + u * s
        return out

    rq = turned(plain.rms_unit(q.double(), EPS) * gq.double(), H)
    rk = turned(plain.rms_unit(k.double(), EPS) * gk.double(), G)
    pages_k = torch.ones(8, G, bs, hd, device="cuda", dtype=dtype)
    pages_v = torch.ones_like(pages_k)
    slots = [21, 0, 31, 13, -1, 3, 8, 9]
    proj = torch.cat([torch.full((T, col), 9.0), q, k, v, torch.full((T, 8), 9.0)], 1).cuda().to(dtype)
    out = ops.projection_norm_rope_store(proj, col, H, G, D, V, hd, i32(positions), gq.cuda(), gk.cuda(), EPS,
                                         inv_freq=inv.float().cuda() if dims else None, rotary_dim=dims, interleaved=interleaved,
                                         slots=i32(slots), k_cache=pages_k, v_cache=pages_v).double().cpu()  # fmt: skip
    only = ops.projection_norm_rope_store(proj, col, H, G, D, V, hd, i32(positions), gq.cuda(), gk.cuda(), EPS,
                                          inv_freq=inv.float().cuda() if dims else None, rotary_dim=dims, interleaved=interleaved)  # fmt: skip
    assert torch.equal(only.double().cpu(), out)
    # angles are float32 by the design: position x frequency is off by up to 2^-24 of itself
    slack = ((0.03 if dtype == torch.bfloat16 else 1e-5) + torch.tensor(positions).double() * 2.0**-22)[:, None, None]
    assert bool(((out[:, :, :D] - rq).abs() <= slack * (1 + rq.abs())).all()) and not out[:, :, D:].any()
    kept = [i for i, s in enumerate(slots) if s >= 0]
    at = [slots[i] for i in kept]
    got_k = pages_k.double().cpu().permute(0, 2, 1, 3).reshape(-1, G, hd)
    got_v = pages_v.double().cpu().permute(0, 2, 1, 3).reshape(-1, G, hd)
    assert bool(((got_k[at][:, :, :D] - rk[kept]).abs() <= slack[kept] * (1 + rk[kept].abs())).all()) and not got_k[at][:, :, D:].any()
    assert torch.equal(got_v[at][:, :, :V], v.view(T, G, V)[kept].double()) and not got_v[at][:, :, V:].any()
    untouched = sorted(set(range(8 * bs)) - set(at))
    assert (got_k[untouched] == 1).all() and (got_v[untouched] == 1).all()


def attend(q_parts, pages, requests, lens, starts, scale, window, sink):
    from atomserve_b200 import ops

    ctx = step_context(lens, starts)
    q = torch.cat(q_parts).cuda().to(pages.dtype).contiguous()
    return ops.paged_attention(q, pages.pools[0], pages.pools[1], pages.table(requests), ctx.req_q_start, ctx.req_pos_start,
                               num_requests=len(lens), max_context=ctx.max_context, window=window, scale=scale,
                               host_q_lens=lens, sink=sink).float().cpu()  # fmt: skip


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("size,bs,hd", [(20, 16, 24), (7, 8, 40), (100, 16, 64), (33, 16, 128), (1, 4, 16), (290, 16, 64), (64, 16, 128)])
def test_one_key_stands_out_at_the_windows_edges(dtype, size, bs, hd):
    """All keys are zero but one whose score is large; its value is e_1, and the denominator holds one
    more term, exp(0) = 1, once whatever the number of key partitions. For a query at position p the key
    at p - size + 1 is the last one seen and the key at p - size the first one not seen."""
    H, G, scale, T = 4, 2, 0.5, 330
    sink = torch.zeros(H, device="cuda")
    q = torch.zeros(1, H, hd)
    q[:, :, 0] = 4.0  # score of the marked key: 4 * 2.5 * 0.5 = 5
    marks = {0, 1, bs - 1, bs, 2 * bs, T - size - 1, T - size, T - size + 1, T - 2, T - 1}
    for mark in sorted(m for m in marks if 0 <= m < T):
        k, v = torch.zeros(T, G, hd), torch.zeros(T, G, hd)
        k[mark, :, 0], v[mark, :, 1] = 2.5, 1.0
        pages = Pages([(G, hd), (G, hd)], bs, dtype, blocks=T // bs + 5, seed=mark)
        pages.put("r", k, v)
        for p in sorted({T - 1, mark, min(mark + size - 1, T - 1), min(mark + size, T - 1)}):
            seen = 0 <= p - mark < size
            want = np.exp(5.0) / (np.exp(5.0) + min(p + 1, size) - 1 + 1) if seen else 0.0
            one = attend([q], pages, ["r"], [1], [p], scale, size, sink)[0, :, 1].tolist()
            lo = max(0, p - 40)
            many = attend([q.expand(p + 1 - lo, H, hd)], pages, ["r"], [p + 1 - lo], [lo], scale, size, sink)[-1, :, 1].tolist()
            for got in (one, many):
                assert np.allclose(got, want, rtol=2e-2 if dtype == torch.bfloat16 else 1e-5, atol=1e-6), (mark, p, got, want)


def mixer_weights(g, d, layer):
    cfg = dict(vocab=4, width=d, layers=[dict(layer, mlp=None)])
    seed = int(torch.randint(0, 1 << 30, (1,), generator=g))
    w = plain.random_checkpoint(cfg, seed)
    return {"x." + k[len("l0.mix.") :]: v for k, v in w.items() if k.startswith("l0.mix.")}


def mixer_part(d, layer, eps):
    """The mixer as the model's description names it."""
    from atomserve_b200.config.registry import config_from_dict
    from atomserve_b200.parts import build_part
    from atomserve_b200.models.vilulix import _mixer

    cfg = dict(architecture="Vilulix", vocab=8, width=d, norm=dict(eps=eps), logit_softcap=1.0, layers=[dict(layer, mlp=None)])
    _, config = config_from_dict(cfg)
    return build_part("mixer", _mixer(config, config.layers[0], "x."), d)


MIXERS = [
    parallel(window(6, 2, 24, 16, 0.5, 20, dims=12), delta(4, 2, 16, 40, 4), (0.7, 1.6)),
    parallel(window(4, 4, 16, 32, 0.6, 7), delta(3, 3, 24, 8, 2), (1.3, 0.4)),
    parallel(window(2, 1, 32, 8, 0.3, 500, dims=0), delta(5, 1, 8, 3, 1), (1.0, 1.0)),
    parallel(window(3, 3, 40, 40, 0.35, 1, dims=8), delta(2, 1, 40, 24, 9), (2.0, 0.9)),
    parallel(window(8, 2, 64, 64, 0.2, 33, dims=32), delta(2, 2, 128, 64, 4), (-0.5, 1.0)),
    parallel(window(20, 1, 128, 128, 0.1, 25), delta(4, 1, 136, 36, 3), (1.0, 0.0)),
    parallel(window(2, 2, 16, 16, 0.5, None), delta(1, 1, 20, 20, 5), (0.0, 1.0)),
    latent(5, 24, 8, 20, 40, 28, 0.4, 1000.0),
    latent(1, 12, 20, 36, 24, 40, 0.35, 50.0),
    latent(4, 64, 32, 64, 128, 96, 0.2, 30000.0),
    latent(3, 10, 6, 14, 22, 18, 0.6, 10.0),
    latent(40, 16, 16, 8, 64, 24, 0.3, 100.0),
    latent(2, 32, 64, 1, 136, 8, 0.15, 500.0),
]  # fmt: skip


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("layer", MIXERS, ids=lambda m: f"{m['type']}-{MIXERS.index(m)}")
def test_mixer_alone(dtype, layer):
    """A sequence in two portions and then token by token through scattered pages and a state slot equals
    the plain mixer on the whole sequence; then two requests in one step, one of them mid-sequence."""
    from atomserve_b200.parts import CacheView

    d, T, bs = 72, 75, 4
    m = layer["mixer"]
    g = torch.Generator().manual_seed(MIXERS.index(layer))
    w = mixer_weights(g, d, layer)
    part = mixer_part(d, layer, EPS)
    part.load(on_device(w, dtype))
    assert sorted(s.name for s in part.tensor_specs()) == sorted(w)
    h, h2 = rounded(2 * torch.randn(T, d, generator=g)), rounded(2 * torch.randn(9, d, generator=g))
    mechanism = plain.MIXERS[layer["type"]]
    ref, ref2 = (mechanism(x.double(), doubles(w, "x."), m, EPS).float() for x in (h, h2))
    spec = part.cache_spec()
    view = CacheView(pages={t.name: torch.ones(46, t.heads, bs, t.width, device="cuda", dtype=dtype) for t in spec.tensors},
                     state={s.name: torch.zeros(3, *s.shape, device="cuda") for s in part.state_specs()}, block_size=bs)
    table = torch.randperm(46, generator=g).tolist()
    mine, other = table[:20], table[20:40]
    view.block_tables = i32([mine])
    outs = []
    for start, n in [(0, 34), (34, 2), (36, 9)] + [(p, 1) for p in range(45, T - 6)]:
        view.slots = paged(mine, bs, range(start, start + n))
        outs.append(part.forward(h[start : start + n].cuda().to(dtype), None, step_context([n], [start], [2]), view))
    done = T - 6
    view.block_tables = i32([other, mine])
    view.slots = torch.cat([paged(other, bs, range(9)), paged(mine, bs, range(done, T))])
    both = part.forward(torch.cat([h2, h[done:]]).cuda().to(dtype), None, step_context([9, 6], [0, done], [0, 2]), view)
    assert both.dtype == torch.float32  # what a block that sums in float32 takes
    check(torch.cat(outs + [both[9:]]), ref, dtype, "portions and single tokens", 0.05)
    check(both[:9], ref2, dtype, "the second request beside it", 0.05)
    assert all(not s[1].any() for s in view.state.values()), "a slot of no request was written"


# ---- whole models through the step function -------------------------------------------------

LENGTHS = {"a": [5, 49, 130, 1, 64], "b": [33, 2, 97, 40], "c": [200, 9, 70], "d": [70, 3, 130, 20], "e": [45, 2, 110]}


def oracle(cfg, w, prompt):
    return plain.forward(prompt, w, cfg).float()


def allowance(cfg, w, prompt, ref):
    """What rounding alone does, per position: the largest error of the plain implementation itself
    over several ways of rounding to 16 bits everything an engine may keep in them."""
    return torch.stack([row_errors(plain.forward(prompt, w, cfg, stored=f), ref) for f in ROUNDINGS]).max(0).values


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    out = {}
    for name, (cfg, bs) in VILULIX.items():
        w = plain.random_checkpoint(cfg, seed=31)
        folder = write_folder(cfg, w, tmp_path_factory.mktemp(f"vilulix_{name}"))
        ps = prompts(cfg, LENGTHS[name], seed=9)
        refs = [oracle(cfg, w, p) for p in ps]
        out[name] = (cfg, bs, folder, w, ps, refs, [allowance(cfg, w, p, r) for p, r in zip(ps, refs)])
    return out


def replayer(folder, dtype, bs, max_tokens, **more):
    from atomserve_b200.engine.replay import TraceReplayer

    return TraceReplayer(folder, dtype, max_tokens, bs, **more)


CASES = [(n, d) for n in VILULIX for d in ("float32", "bfloat16")]


@pytest.mark.parametrize("name,dtype", CASES)
def test_whole_then_token_by_token_then_portions(models, name, dtype):
    cfg, bs, folder, _, ps, refs, tols = models[name]
    rp = replayer(folder, dtype, bs, max(-(-len(p) // 64) * 64 for p in ps))
    sizes = [2, 7, 3, 16, 2, 17, 5, 31, 2, 9, 1, 33]
    for i, (p, ref, tol) in enumerate(zip(ps, refs, tols)):
        n = len(p)

        def held(logits, places, what):
            judge(logits, ref[places], dtype, f"{name} request {i} {what}", tol[places])

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
    cfg, bs, folder, _, ps, refs, tols = models[name]
    ps4, refs4, tols4 = ps * 4, refs * 4, tols * 4
    biggest = sorted((-(-len(p) // 64) * 64 for p in ps4), reverse=True)
    rp = replayer(folder, dtype, bs, sum(biggest[:4]), max_live=4)
    rng = np.random.default_rng(17)
    for entries, end in mixed_trace(ps4, rng, largest=60):
        logits = rp.step([dict(id=e["id"], tokens=e["tokens"], want=e["want"]) for e in entries], end=end)
        row = 0
        for e in entries:
            n = len(e["tokens"])
            places = list(range(e["at"], e["at"] + n))
            judge(logits[row : row + n], refs4[e["id"]][places], dtype, f"{name} request {e['id']} at {e['at']}", tols4[e["id"]][places])
            row += n
    assert sum(len(p) for p in ps4) > rp.cache.num_blocks * bs, "the pool was large enough to never reuse a page"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding(models, dtype):
    """280 tokens one by one after a short prompt, from CUDA graphs: the states are carried through every
    step, windows pass over decoded tokens and give their pages back."""
    for name in ("a", "c"):
        cfg, bs, folder, w = models[name][:4]
        p = prompts(cfg, [300], seed=12)[0]
        ref = oracle(cfg, w, p)
        tol = allowance(cfg, w, p, ref)
        rp = replayer(folder, dtype, bs, 320)
        assert rp.runner.use_graphs
        rp.step([dict(id="x", tokens=p[:20], want=[])], end=[])
        for j in range(20, len(p)):
            logits = rp.step([dict(id="x", tokens=[p[j]], want=[0])], end=[])
            if j % 9 == 0 or j > 290:
                judge(logits, ref[j : j + 1], dtype, f"{name} decode position {j}", tol[j : j + 1])
        held = rp.live["x"][0]
        windowed = [(g.spec.window, table) for g, table in zip(rp.cache.groups, held.block_tables) if g.spec.window]
        assert windowed, "no windowed layer kept pages of its own"
        for size, table in windowed:
            assert sum(b >= 0 for b in table) <= -(-size // bs) + 1 and len(table) == -(-len(p) // bs)


def test_the_stream_after_every_layer(models):
    """The float32 residual stream after each entry of the run order (a layer of the loop counts every
    time it runs) against the plain implementation's, in float32."""
    for name in ("a", "d", "e"):
        cfg, bs, folder, w, ps = models[name][:5]
        p = ps[2]
        layers = []
        plain.forward(p, w, cfg, streams=layers)
        rp = replayer(folder, "float32", bs, 192)
        seen = []
        for block in rp.model.blocks:
            inner = block.forward_chain

            def wrapped(*a, _inner=inner, **k):
                out = _inner(*a, **k)
                seen.append(out[0].double().cpu())
                return out

            block.forward_chain = wrapped
        rp.step([dict(id=0, tokens=p, want=[0])], end=[0])
        assert len(seen) == len(plain.run_order(cfg)) == len(layers)
        for i, (got, ref) in enumerate(zip(seen, layers)):
            assert float((got - ref).abs().max() / ref.abs().max()) < 3e-5, f"{name}: stream after layer run {i}"


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
    n = bs + 4
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
        ref = oracle(cfg, w, list(p) + list(out))
        spread = float((ref - ref.mean(-1, keepdim=True)).pow(2).mean().sqrt())
        for i, token in enumerate(out):
            row = ref[len(p) + i - 1]
            assert float(row.max() - row[token]) <= 0.15 * spread, f"token {i} lies far below the best"


def test_command_line_and_random_weights(tmp_path):
    """`python -m atomserve_b200` on a Vilulix folder written by the package's own random-weights
    writer from a configuration that round-trips through config.json."""
    import json
    import subprocess
    import sys

    from atomserve_b200.config.registry import config_from_dict
    from atomserve_b200.weights.random_init import write_model_folder

    arch, config = config_from_dict(VILULIX["b"][0])
    folder = write_model_folder(config, 3, tmp_path / "m", "bfloat16")
    assert json.loads((folder / "config.json").read_text())["architecture"] == "Vilulix"
    done = subprocess.run([sys.executable, "-m", "atomserve_b200", str(folder), "--prompt-ids", "5,6,7", "--max-tokens", "6",
                           "--temperature", "0"], capture_output=True, text=True, timeout=600)  # fmt: skip
    assert done.returncode == 0, done.stderr[-2000:]
