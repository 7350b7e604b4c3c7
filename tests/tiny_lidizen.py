"""Small Lidizen configurations for the tests. They differ from one another in every size and
option: one to five streams; as many kv heads as heads, fewer, one; keys wider and narrower than the
values and equal to them; rotations of a whole head, of a part of it, none; windows of one token,
shorter than a page, across page borders and longer than the prompts, without kept positions, with
fewer than a page of them, with several pages, with more than the window; no window; layers that mix
values and layers that do not, the first layer among either; dense and routed feed-forwards and layers
without one; one to four choices; biases of the router that matter; pair tables of one row and
more, with multipliers beyond the table; widths and vocabularies that are no multiples of 8. Score
scales are larger than 1 / sqrt(size) where keys are few, so that single keys matter."""


def attention(heads, kv_heads, dim, vdim, scale, window=None, keep=None, rot=None, v_mix=False, mlp=None):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, v_mix=v_mix)
    if window is not None:
        m["mask"] = dict(size=window)
        if keep is not None:
            m["mask"]["keep_first"] = keep
    if rot is not None:
        m["rot"] = dict(base=rot[0], dims=rot[1])
    return dict(type="attention", mixer=m, mlp=mlp)


def dense(ff):
    return dict(kind="dense", ff=ff)


def moe(experts, top, ff):
    return dict(kind="moe", expert=dict(ff=ff), router=dict(experts=experts, top=top))


def model(vocab, width, streams, eps, pairs, layers):
    return dict(architecture="Lidizen", vocab=vocab, width=width, streams=streams, norm=dict(eps=eps),
                embedding=dict(bigram=dict(zip(("buckets", "mul_prev", "mul_cur"), pairs))), layers=list(layers))  # fmt: skip


# sizes that only the general kernels serve
LIDIZEN_A = model(300, 96, 3, 1e-5, (61, 29, 11), [
    attention(6, 3, 24, 16, 0.3, window=10, keep=3, rot=(100.0, 8), mlp=dense(72)),
    attention(4, 2, 12, 40, 0.4, window=33, keep=18, rot=(30.0, 12), v_mix=True, mlp=moe(5, 2, 40)),
    attention(2, 1, 16, 16, 0.35, rot=(1000.0, 16)),
    attention(2, 2, 20, 40, 0.3, window=7, keep=40, v_mix=True, mlp=moe(3, 3, 24)),
])  # fmt: skip
BLOCK_SIZE_A = 16

# one stream, windows of one token and longer than every prompt, odd sizes
LIDIZEN_B = model(257, 60, 1, 1e-6, (17, 3, 1000003), [
    attention(2, 1, 10, 6, 0.5, window=1, keep=1, rot=(50.0, 4), v_mix=True, mlp=moe(2, 1, 18)),
    attention(4, 4, 12, 20, 0.4, window=500, keep=2, v_mix=False, mlp=dense(50)),
    attention(3, 1, 14, 6, 0.4, window=2, rot=(10.0, 14), v_mix=True, mlp=moe(6, 4, 10)),
])  # fmt: skip
BLOCK_SIZE_B = 8

# sizes at which the bfloat16 products and attention run this package's tensor-core kernels
LIDIZEN_C = model(704, 224, 4, 2e-6, (1009, 211, 13), [
    attention(8, 2, 128, 128, 0.12, window=90, keep=30, rot=(10000.0, 64), v_mix=True, mlp=moe(8, 3, 128)),
    attention(12, 4, 64, 32, 0.16, window=64, keep=64, rot=(500.0, 64), mlp=dense(320)),
    attention(4, 2, 96, 128, 0.13, rot=(400000.0, 32), v_mix=True, mlp=moe(6, 1, 64)),
    attention(20, 1, 64, 64, 0.15, window=17, keep=5, rot=(100.0, 48)),
])  # fmt: skip
BLOCK_SIZE_C = 16

# five streams, many kv heads, small pages; the first layer has no feed-forward
LIDIZEN_D = model(130, 100, 5, 1e-5, (1, 1, 1), [
    attention(5, 5, 10, 10, 0.6, window=5, keep=2, rot=(10.0, 10), v_mix=True),
    attention(10, 5, 8, 10, 0.5, window=12, keep=9, v_mix=True, mlp=moe(7, 4, 8)),
])  # fmt: skip
BLOCK_SIZE_D = 4

LIDIZEN = {"a": (LIDIZEN_A, BLOCK_SIZE_A), "b": (LIDIZEN_B, BLOCK_SIZE_B), "c": (LIDIZEN_C, BLOCK_SIZE_C),
           "d": (LIDIZEN_D, BLOCK_SIZE_D)}  # fmt: skip
