"""Small random models of the hybrid design for the tests: sizes that are not multiples of anything, layers that differ
from one another, loops, windows of one, one tap, one head, several experts per token, no feed-forward."""
from latent_cases import write_folder  # noqa: F401
from oracle.hybrid_lm import random_model  # noqa: F401


def attention(heads, kv_heads, dim, vdim, window, scale=None):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": dim ** -0.5 if scale is None else scale, "mask": {"size": window}}


def recurrence(width, blocks, taps):
    return {"width": width, "blocks": blocks, "conv": taps}


def parallel(left, right, left_scale, right_scale, mlp):
    return {"type": "parallel", "mixer": {"left": left, "right": right, "left_scale": left_scale, "right_scale": right_scale}, "mlp": mlp}


def delta(heads, kv_heads, dim, vdim, taps, mlp):
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": taps}, "mlp": mlp}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def routed(experts, top, ff):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def config(width, vocab, layers, loop=None, eps=1e-5):
    return {"architecture": "Dozusun", "width": width, "vocab": vocab, "norm": {"eps": eps}, "layers": layers, "loop": loop}


# odd sizes; windows of 1, 7 and 19; a loop that ends inside; no feed-forward, dense, one and three experts per token
UNEVEN = config(90, 203, [
    delta(3, 1, 11, 7, 2, routed(5, 3, 21)),
    parallel(attention(6, 2, 13, 9, 19, 0.5), recurrence(42, 3, 3), 0.7, 1.3, None),
    parallel(attention(5, 1, 20, 33, 7), recurrence(35, 5, 1), 1.1, 0.4, routed(4, 1, 13)),
    delta(4, 4, 6, 18, 5, dense(77)),
    parallel(attention(1, 1, 8, 8, 1), recurrence(17, 1, 4), 0.9, 0.8, dense(50)),
], loop={"start": 1, "stop": 4, "times": 2}, eps=1e-3)

# sizes in whole vectors, one layer after the other, sharp scores
EVEN = config(192, 500, [
    parallel(attention(8, 2, 64, 48, 70, 0.25), recurrence(256, 2, 4), 0.8, 1.2, dense(256)),
    delta(4, 2, 64, 96, 4, routed(8, 2, 64)),
    delta(2, 2, 40, 40, 3, None),
    parallel(attention(3, 3, 40, 72, 129), recurrence(96, 6, 6), 1.5, 0.5, routed(3, 3, 48)),
], eps=1e-6)

# head sizes of a large model and beyond: long keys in the scan's wide form, values wider than a tile, many heads per group,
# blocks longer than a warp's row of vectors
LARGE = config(256, 300, [
    delta(2, 1, 128, 128, 4, dense(400)),
    delta(1, 1, 300, 36, 4, None),
    parallel(attention(12, 1, 128, 128, 150), recurrence(640, 2, 4), 1.0, 1.0, routed(16, 2, 40)),
    delta(1, 1, 520, 20, 2, dense(40)),
    parallel(attention(2, 1, 200, 264, 64), recurrence(1200, 2, 4), 0.6, 1.4, dense(120)),
], loop={"start": 2, "stop": 3, "times": 3})

ALL = {"uneven": UNEVEN, "even": EVEN, "large": LARGE}
