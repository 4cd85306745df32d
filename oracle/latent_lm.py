"""Plain CPU statement of the latent-attention decoder (design "Bikelix"; test infrastructure only).

One function per mechanism, whole sequences at once, no cache, every matrix product and every sum in
`dtype` (float64 unless a caller asks for less). The product path shares no code with this file. `cfg` is
the parsed config.json of a model folder, `w` a mapping from tensor name to a CPU tensor.
"""
from __future__ import annotations

import math

import torch


def root_mean_square_norm(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def plain_norm(x, w, eps):
    """RMS norm whose weight is stored as it is applied."""
    return root_mean_square_norm(x, eps) * w


def zero_centred_norm(x, w, eps):
    """RMS norm whose weight is stored around zero: the factor is 1 + w."""
    return root_mean_square_norm(x, eps) * (1.0 + w)


def rotate(x, positions, dims, base):
    """x [T, ..., n]: dimension i < dims / 2 turns with dimension i + dims / 2 by position * base^(-2 i / dims)."""
    half = dims // 2
    i = torch.arange(half, dtype=torch.float64)
    angle = positions.to(torch.float64)[:, None] * base ** (-2.0 * i / dims)
    shape = (x.shape[0],) + (1,) * (x.dim() - 2) + (half,)
    c, s = angle.cos().reshape(shape).to(x.dtype), angle.sin().reshape(shape).to(x.dtype)
    u, v, rest = x[..., :half], x[..., half:dims], x[..., dims:]
    return torch.cat([u * c - v * s, v * c + u * s, rest], dim=-1)


def window_mask(n, size):
    """visible[i, j]: a position sees itself and the size - 1 positions before it (size None: all before it)."""
    d = torch.arange(n)[:, None] - torch.arange(n)[None, :]
    return (d >= 0) if size is None else (d >= 0) & (d < size)


def softmax_with_sink(scores, visible, sink):
    """scores [H, T, T], sink [H] or None: the sink adds exp(sink_h) to the denominator and nothing to the numerator."""
    s = scores.masked_fill(~visible[None], -math.inf)
    top = s.amax(-1, keepdim=True)
    if sink is not None:
        top = torch.maximum(top, sink[:, None, None])
    e = torch.exp(s - top)
    den = e.sum(-1, keepdim=True)
    if sink is not None:
        den = den + torch.exp(sink[:, None, None] - top)
    return e / den


def latent_of(h, w, p, mx, eps, positions):
    """The two things a cache holds of a token: the normed latent [T, kv_rank] and the rotated shared key part."""
    y = h @ w[p + ".dkv"].T
    c = plain_norm(y[:, :mx["kv_rank"]], w[p + ".dkv.norm"], eps)
    return c, rotate(y[:, mx["kv_rank"]:], positions, mx["rot"]["dims"], mx["rot"]["base"])


def latent_queries(h, w, p, mx, eps, positions):
    H, dim = mx["heads"], mx["dim"]
    q = plain_norm(h @ w[p + ".dq"].T, w[p + ".dq.norm"], eps) @ w[p + ".uq"].T
    q = q.reshape(h.shape[0], H, dim + mx["rot_dim"])
    return q[..., :dim], rotate(q[..., dim:], positions, mx["rot"]["dims"], mx["rot"]["base"])


def attend(qn, qr, c, kr, uk, uv, scale, visible, sink):
    """Queries [I, H, dim] and [I, H, rot_dim], cached latents [J, kv_rank] and rotated key parts [J, rot_dim], one
    visible[i, j] per pair -> [I, H, vdim]. uk: [H dim, kv_rank], uv: [H vdim, kv_rank], both head by head."""
    H, n = qn.shape[1], c.shape[0]
    k = (c @ uk.T).reshape(n, H, -1)
    v = (c @ uv.T).reshape(n, H, -1)
    scores = (torch.einsum("ihd,jhd->hij", qn, k) + torch.einsum("ihd,jd->hij", qr, kr)) * scale
    return torch.einsum("hij,jhd->ihd", softmax_with_sink(scores, visible, sink), v)


def latent_attention(h, latents, layer, w, p, mx, eps):
    """h [T, D]; `latents` keeps every layer's (latent, rotated key part) for the layers that read them again."""
    n = h.shape[0]
    positions = torch.arange(n)
    src = mx.get("kv_from")
    if src is None:
        latents[layer] = latent_of(h, w, p, mx, eps, positions)
        src = layer
    c, kr = latents[src]
    qn, qr = latent_queries(h, w, p, mx, eps, positions)
    mask = mx.get("mask")
    y = attend(qn, qr, c, kr, w[p + ".uk"], w[p + ".uv"], mx["scale"], window_mask(n, mask["size"] if mask else None), w.get(p + ".sink"))
    return y.reshape(n, -1) @ w[p + ".o"].T


def clamped_gated_mlp(h, w, p, limit):
    g = torch.minimum(h @ w[p + ".gate"].T + w[p + ".gate.b"], torch.tensor(limit, dtype=h.dtype))
    u = torch.clamp(h @ w[p + ".up"].T + w[p + ".up.b"], -limit, limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ w[p + ".down"].T + w[p + ".down.b"]


def softcap(logits, cap):
    return logits if cap is None else cap * torch.tanh(logits / cap)


def forward(cfg, w, tokens, dtype=torch.float64, layers_out=None):
    """Logits [T, vocab] of one sequence from its first token; `layers_out` collects the stream after every layer."""
    w = {k: t.to(dtype) for k, t in w.items()}
    eps, alpha = cfg["norm"]["eps"], cfg["postln_alpha"]
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)] * cfg["embedding"]["scale"]
    latents = {}
    for i, layer in enumerate(cfg["layers"]):
        assert layer["type"] == "latent_attention"
        y = latent_attention(x, latents, i, w, f"l{i}.mix", layer["mixer"], eps)
        x = zero_centred_norm(alpha * x + y, w[f"l{i}.norm1"], eps)
        if layer.get("mlp") is not None:
            y = clamped_gated_mlp(x, w, f"l{i}.mlp", layer["mlp"]["limit"])
            x = zero_centred_norm(alpha * x + y, w[f"l{i}.norm2"], eps)
        if layers_out is not None:
            layers_out.append(x)
    x = zero_centred_norm(x, w["final.norm"], eps)
    return softcap(x @ w["embed"].T, cfg["logit_softcap"])


def random_model(cfg, seed=0, weight_scale=1.0):
    """Seeded bf16 weights of a configuration: fan-in scaled matrices, norm weights and biases away from their neutral
    values, so that leaving one out shows."""
    g = torch.Generator().manual_seed(seed)
    D = cfg["width"]
    w = {}

    def mat(name, rows, cols, gain=1.0):
        w[name] = (torch.randn(rows, cols, generator=g) * (gain * weight_scale / cols ** 0.5)).bfloat16()

    def vec(name, n, mean=0.0, std=0.3):
        w[name] = (mean + std * torch.randn(n, generator=g)).bfloat16()

    w["embed"] = (0.3 * torch.randn(cfg["vocab"], D, generator=g)).bfloat16()  # logits of a few units
    for i, layer in enumerate(cfg["layers"]):
        mx, p = layer["mixer"], f"l{i}.mix"
        H = mx["heads"]
        vec(f"l{i}.norm1", D)
        mat(p + ".dq", mx["q_rank"], D)
        vec(p + ".dq.norm", mx["q_rank"], 1.0)
        mat(p + ".uq", H * (mx["dim"] + mx["rot_dim"]), mx["q_rank"], 1.5)
        if mx.get("kv_from") is None:
            mat(p + ".dkv", mx["kv_rank"] + mx["rot_dim"], D)
            vec(p + ".dkv.norm", mx["kv_rank"], 1.0)
        mat(p + ".uk", H * mx["dim"], mx["kv_rank"], 1.5)
        mat(p + ".uv", H * mx["vdim"], mx["kv_rank"])
        vec(p + ".sink", H, 0.5, 1.0)
        mat(p + ".o", D, H * mx["vdim"], 2.0)
        if layer.get("mlp") is not None:
            ff = layer["mlp"]["ff"]
            vec(f"l{i}.norm2", D)
            mat(f"l{i}.mlp.gate", ff, D, 1.5)
            vec(f"l{i}.mlp.gate.b", ff)
            mat(f"l{i}.mlp.up", ff, D, 1.5)
            vec(f"l{i}.mlp.up.b", ff)
            mat(f"l{i}.mlp.down", D, ff, 1.5)
            vec(f"l{i}.mlp.down.b", D)
    vec("final.norm", D)
    return w
