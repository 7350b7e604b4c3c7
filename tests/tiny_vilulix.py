"""Small Vilulix configurations for the tests. They differ from one another in every size and option:
loops over a middle stretch of the layers, over the first ones, over all of them, over one layer, run
once, and no loop; layers with and without a feed-forward; as many q/k heads as heads, fewer, one; key
sizes below, at and above a value's, and above what a chunk of 64 tokens takes; one, two, four and nine
taps; windows of one token, shorter than a page, across page borders and longer than the prompts;
rotations of a whole head, of a part of it, and none; latents smaller and larger than the heads
together; side-by-side mixers weighted below, at and above 1; caps on logits and gates that are tight
and loose; a width and a vocabulary that are no multiples of 8. Score scales are larger than
1 / sqrt(size), so that scores spread over many units and single keys matter."""


def _mlp(ff):
    return dict(kind="dense", ff=ff) if ff else None


def memory(heads, dim, vdim, cap, ff=None):
    return dict(type="mlstm", mixer=dict(heads=heads, dim=dim, vdim=vdim, gate_cap=cap), mlp=_mlp(ff))


def latent(heads, dim, rot_dim, vdim, kv_rank, q_rank, scale, base, ff=None):
    return dict(type="latent_attention", mixer=dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, kv_rank=kv_rank, q_rank=q_rank,
                                                    scale=scale, rot=dict(base=base, dims=rot_dim)), mlp=_mlp(ff))  # fmt: skip


def window(heads, kv_heads, dim, vdim, scale, size, base=100.0, dims=None):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale)
    if size:
        m["mask"] = dict(size=size)
    if dims != 0:
        m["rot"] = dict(base=base, dims=dim if dims is None else dims)
    return m


def delta(heads, kv_heads, dim, vdim, conv):
    return dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, conv=conv)


def parallel(left, right, scales, ff=None):
    return dict(type="parallel", mixer=dict(left=left, right=right, left_scale=scales[0], right_scale=scales[1]), mlp=_mlp(ff))


def _model(vocab, width, eps, cap, loop, layers):
    out = dict(architecture="Vilulix", vocab=vocab, width=width, norm=dict(eps=eps), logit_softcap=cap, layers=list(layers))
    if loop is not None:
        out["loop"] = dict(zip(("start", "stop", "times"), loop))
    return out


# a loop over the middle layers, three passes; a layer before it and one behind
VILULIX_A = _model(300, 96, 1e-5, 12.0, (1, 3, 3), [
    parallel(window(6, 2, 24, 16, 0.5, 20, base=300.0, dims=12), delta(4, 2, 16, 40, 4), (0.7, 1.6), 100),
    latent(5, 24, 8, 20, 40, 28, 0.4, 1000.0, 72),
    memory(3, 24, 40, 6.0, None),
    parallel(window(4, 4, 16, 32, 0.6, 7), delta(3, 3, 24, 8, 2), (1.3, 0.4), None),
])  # fmt: skip
BLOCK_SIZE_A = 16

# no loop; a window of one token and one longer than every prompt; no rotation; a single tap and nine
VILULIX_B = _model(257, 64, 1e-6, 40.0, None, [
    memory(1, 16, 16, 10.0, 72),
    parallel(window(2, 1, 32, 8, 0.3, 500, dims=0), delta(5, 1, 8, 3, 1), (1.0, 1.0), 40),
    latent(1, 12, 20, 36, 24, 40, 0.35, 50.0, None),
    parallel(window(3, 3, 40, 40, 0.35, 1, base=20.0, dims=8), delta(2, 1, 40, 24, 9), (2.0, 0.9), 64),
])  # fmt: skip
BLOCK_SIZE_B = 8

# sizes at which the bfloat16 products and attention run this package's tensor-core kernels; the loop runs the
# first three layers twice
VILULIX_C = _model(640, 256, 2e-6, 25.0, (0, 3, 2), [
    parallel(window(8, 2, 64, 64, 0.2, 100, base=5000.0, dims=32), delta(4, 2, 64, 128, 4), (0.8, 1.2), 384),
    latent(4, 64, 32, 64, 128, 96, 0.2, 30000.0, 256),
    memory(2, 64, 160, 8.0, 256),
    parallel(window(4, 1, 128, 128, 0.15, 33), delta(2, 2, 128, 64, 3), (1.1, 0.6), 512),
])  # fmt: skip
BLOCK_SIZE_C = 16

# a width and a vocabulary that are no multiples of 8; all layers twice
VILULIX_D = _model(131, 100, 1e-5, 8.0, (0, 2, 2), [
    latent(3, 10, 6, 14, 22, 18, 0.6, 10.0, 60),
    parallel(window(2, 2, 12, 20, 0.8, 5, dims=6), delta(1, 1, 12, 20, 5), (0.5, 2.0), None),
])  # fmt: skip
BLOCK_SIZE_D = 4

# one layer four times, then one with a long key; memories alone keep no pages of their own
VILULIX_E = _model(140, 48, 1e-5, 30.0, (0, 1, 4), [
    memory(2, 20, 12, 3.0, 56),
    parallel(window(4, 2, 8, 8, 0.9, 37, base=7.0, dims=4), delta(2, 1, 136, 36, 4), (1.0, 1.5), None),
])  # fmt: skip
BLOCK_SIZE_E = 8

VILULIX = {"a": (VILULIX_A, BLOCK_SIZE_A), "b": (VILULIX_B, BLOCK_SIZE_B), "c": (VILULIX_C, BLOCK_SIZE_C),
           "d": (VILULIX_D, BLOCK_SIZE_D), "e": (VILULIX_E, BLOCK_SIZE_E)}  # fmt: skip
