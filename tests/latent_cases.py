"""Small random models of the latent-attention design for the tests: sizes that are not multiples of anything, layers
that differ from one another, shared caches with windows of their own, a layer without a feed-forward."""
import json
import os


def mixer(heads, dim, rot, vdim, q_rank, kv_rank, window, kv_from=None, scale=None, base=10000.0):
    m = {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "mask": {"size": window},
         "rot": {"base": base, "dims": rot}, "scale": scale if scale is not None else (dim + rot) ** -0.5}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return m


def config(width, vocab, layers, alpha=1.7, cap=11.0, eps=1e-5, scale=2.5):
    """layers: (mixer, ff or None, limit)."""
    return {"architecture": "Bikelix", "width": width, "vocab": vocab, "embedding": {"scale": scale}, "norm": {"eps": eps}, "postln_alpha": alpha,
            "logit_softcap": cap,
            "layers": [{"type": "latent_attention", "mixer": m, "mlp": None if ff is None else {"kind": "dense", "ff": ff, "limit": lim}}
                       for m, ff, lim in layers]}


# every layer different; odd sizes; windows of 1, 7, 19 and 41; two layers read earlier caches, one with a wider window
UNEVEN = config(90, 203, [
    (mixer(3, 24, 8, 40, 44, 56, 19), 130, 1.1),
    (mixer(5, 17, 6, 9, 21, 30, 7, base=500.0), 77, 0.8),
    (mixer(2, 13, 8, 33, 50, 56, 41, kv_from=0), None, None),
    (mixer(4, 20, 6, 12, 16, 30, 1, kv_from=1, base=500.0), 64, 2.5),
    (mixer(3, 24, 8, 16, 44, 24, 19), None, None),
], alpha=1.2, cap=7.0, eps=1e-3)

# sizes in whole vectors; scores far from uniform
EVEN = config(256, 500, [
    (mixer(9, 32, 16, 48, 96, 128, 70, scale=0.3), 320, 2.0),
    (mixer(9, 32, 16, 48, 96, 128, 33, kv_from=0, scale=0.25), 320, 2.0),
    (mixer(4, 64, 16, 72, 64, 80, 96), 200, 1.0),
], alpha=1.3, cap=20.0)

# the head sizes of a large model, values wider than 128 and a query wider than the tensor-core kernel stages
LARGE = config(192, 300, [
    (mixer(2, 128, 64, 128, 160, 512, 150), 256, 3.0),
    (mixer(1, 192, 32, 200, 64, 96, 64), 256, 3.0),
    (mixer(1, 700, 40, 300, 64, 96, 64), 128, 3.0),
], alpha=1.0)

ALL = {"uneven": UNEVEN, "even": EVEN, "large": LARGE}


def write_folder(path, cfg, weights):
    from llvq_b200.safetensors import write_safetensors
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    write_safetensors(os.path.join(path, "model.safetensors"), weights)
    return str(path)
