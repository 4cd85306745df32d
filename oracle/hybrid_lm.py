"""Plain CPU statement of the hybrid decoder (design "Dozusun"; test infrastructure only): layers that mix tokens with a
gated delta rule, or with windowed attention and a gated linear recurrence side by side, and feed-forwards that are dense
or chosen by token id.

One function per mechanism, whole sequences at once, recurrences as written, every product and every sum in `dtype`
(float64 unless a caller asks for less). The product path shares no code with this file. `cfg` is the parsed
config.json of a model folder, `w` a mapping from tensor name to a CPU tensor.
"""
from __future__ import annotations

import math

import torch


# ---- norms, activations, convolution ----------------------------------------------
def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def unit_vector(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def silu(x):
    return x * torch.sigmoid(x)


def gelu_tanh(x):
    return 0.5 * x * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (x + 0.044715 * x ** 3)))


def softplus(x):
    return torch.clamp(x, min=0) + torch.log1p(torch.exp(-x.abs()))


def causal_conv(x, w):
    """x [T, C], w [C, taps]: y_t = sum_k w[:, taps - 1 - k] x_{t - k}, zeros before the first token."""
    taps = w.shape[1]
    padded = torch.cat([x.new_zeros(taps - 1, x.shape[1]), x])
    return sum(padded[k:k + x.shape[0]] * w[:, k] for k in range(taps))


# ---- gated delta rule ---------------------------------------------------------------
def delta_rule(q, k, v, beta, g, state=None):
    """q, k [T, H, dim], v [T, H, vdim], beta, g [T, H] -> o [T, H, vdim], S [H, dim, vdim]; one token after another."""
    T, H, dim = q.shape
    S = q.new_zeros(H, dim, v.shape[2]) if state is None else state.clone()
    out = []
    for t in range(T):
        S = g[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out.append(torch.einsum("hdv,hd->hv", S, q[t]))
    return torch.stack(out), S


def delta_decay(a, A_log, dt_bias):
    return torch.exp(-torch.exp(A_log) * softplus(a + dt_bias))


def gated_head_norm(o, w, gate, eps):
    """o, gate [T, H, vdim]: per-head RMS norm with one weight for all heads, times silu(gate)."""
    return rms_norm(o, w, eps) * silu(gate)


def delta_mixer(h, w, p, mx, eps):
    T, H, G, dim, vdim = h.shape[0], mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
    q, k, v = (silu(causal_conv(h @ w[f"{p}.{n}"].T, w[f"{p}.{n}.conv"])) for n in "qkv")
    q = unit_vector(q.reshape(T, G, dim)) * dim ** -0.5
    k = unit_vector(k.reshape(T, G, dim))
    q, k = (x.repeat_interleave(H // G, dim=1) for x in (q, k))
    beta = torch.sigmoid(h @ w[p + ".b"].T)
    g = delta_decay(h @ w[p + ".a"].T, w[p + ".A_log"], w[p + ".dt_bias"])
    o, _ = delta_rule(q, k, v.reshape(T, H, vdim), beta, g)
    o = gated_head_norm(o, w[p + ".norm"], (h @ w[p + ".g"].T).reshape(T, H, vdim), eps)
    return o.reshape(T, H * vdim) @ w[p + ".o"].T


# ---- windowed attention ---------------------------------------------------------------
def window_mask(n, size):
    """visible[i, j]: a position sees itself and the size - 1 positions before it (size None: all before it)."""
    d = torch.arange(n)[:, None] - torch.arange(n)[None, :]
    return (d >= 0) if size is None else (d >= 0) & (d < size)


def grouped_attention(q, k, v, scale, visible):
    """q [I, H, dim], k [J, G, dim], v [J, G, vdim], visible [I, J] -> [I, H, vdim]."""
    H, G = q.shape[1], k.shape[1]
    k, v = (x.repeat_interleave(H // G, dim=1) for x in (k, v))
    s = torch.einsum("ihd,jhd->hij", q, k) * scale
    p = torch.softmax(s.masked_fill(~visible[None], -math.inf), dim=-1)
    return torch.einsum("hij,jhd->ihd", p, v)


def attention_mixer(h, w, p, mx, eps):
    T, H, G, dim, vdim = h.shape[0], mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
    q = rms_norm((h @ w[p + ".q"].T).reshape(T, H, dim), w[p + ".q.norm"], eps)
    k = rms_norm((h @ w[p + ".k"].T).reshape(T, G, dim), w[p + ".k.norm"], eps)
    v = (h @ w[p + ".v"].T).reshape(T, G, vdim)
    mask = mx.get("mask")
    y = grouped_attention(q, k, v, mx["scale"], window_mask(T, mask["size"] if mask else None)).reshape(T, H * vdim)
    return (y * torch.sigmoid(h @ w[p + ".g"].T)) @ w[p + ".o"].T


# ---- real-gated linear recurrence -------------------------------------------------------
def block_diagonal(u, m, b):
    """u [T, width], m [blocks, n, n] as [out, in], b [blocks, n]."""
    T, (blocks, n, _) = u.shape[0], m.shape
    return (torch.einsum("tbi,boi->tbo", u.reshape(T, blocks, n), m) + b).reshape(T, blocks * n)


def linear_recurrence(a, x):
    """S_t = a_t S_{t-1} + x_t from zero; a, x [T, width]."""
    S, out = torch.zeros_like(x[0]), []
    for t in range(x.shape[0]):
        S = a[t] * S + x[t]
        out.append(S)
    return torch.stack(out)


def gated_recurrence(u, r, i, lam):
    log_a = -8.0 * r * softplus(lam)
    return linear_recurrence(torch.exp(log_a), torch.sqrt(-torch.expm1(2.0 * log_a)) * i * u)


def recurrent_mixer(h, w, p, mx):
    y = gelu_tanh(h @ w[p + ".y"].T + w[p + ".y.b"])
    u = causal_conv(h @ w[p + ".x"].T + w[p + ".x.b"], w[p + ".conv"]) + w[p + ".conv.b"]
    r = torch.sigmoid(block_diagonal(u, w[p + ".ra"], w[p + ".ra.b"]))
    i = torch.sigmoid(block_diagonal(u, w[p + ".ri"], w[p + ".ri.b"]))
    return (gated_recurrence(u, r, i, w[p + ".lam"]) * y) @ w[p + ".o"].T


def parallel_mixer(h, w, p, mx, eps):
    return mx["left_scale"] * attention_mixer(h, w, p + ".left", mx["left"], eps) + mx["right_scale"] * recurrent_mixer(h, w, p + ".right", mx["right"])


# ---- feed-forward -----------------------------------------------------------------------
def gated_mlp(h, w, p):
    return (silu(h @ w[p + ".gate"].T) * (h @ w[p + ".up"].T)) @ w[p + ".down"].T


def table_routed_mlp(h, tokens, w, p, experts):
    """The token's id names its experts; each has weight 1 / top."""
    table = w[p + ".table"][tokens].long()
    y = torch.zeros_like(h)
    for e in range(experts):
        hit = (table == e).any(1).nonzero()[:, 0]
        if len(hit):
            y[hit] += gated_mlp(h[hit], w, f"{p}.e{e}") / table.shape[1]
    return y


# ---- the model ----------------------------------------------------------------------------
def layer_runs(cfg):
    """Layer indices in the order they run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return list(range(n))
    a, b = loop["start"], loop["stop"]
    return list(range(a)) + list(range(a, b)) * loop["times"] + list(range(b, n))


def forward(cfg, w, tokens, dtype=torch.float64, layers_out=None):
    """Logits [T, vocab] of one sequence from its first token; `layers_out` collects the stream after every layer run."""
    w = {k: t if t.dtype == torch.int32 else t.to(dtype) for k, t in w.items()}
    eps = cfg["norm"]["eps"]
    tokens = torch.as_tensor(tokens, dtype=torch.long)
    x = w["embed"][tokens]
    for i in layer_runs(cfg):
        layer, p = cfg["layers"][i], f"l{i}"
        h = rms_norm(x, w[p + ".norm1"], eps)
        y = {"delta": delta_mixer, "parallel": parallel_mixer}[layer["type"]](h, w, p + ".mix", layer["mixer"], eps)
        mlp = layer.get("mlp")
        if mlp is not None:
            h = rms_norm(x, w[p + ".norm2"], eps)
            y = y + (gated_mlp(h, w, p + ".mlp") if mlp["kind"] == "dense" else
                     table_routed_mlp(h, tokens, w, p + ".mlp", mlp["router"]["experts"]))
        x = x + y
        if layers_out is not None:
            layers_out.append(x)
    return rms_norm(x, w["final.norm"], eps) @ w["head"].T

def random_model(cfg, seed=0):
    """Seeded bf16 weights (tables int32): fan-in scaled matrices, norm weights, biases and decays away from neutral
    values, so that leaving one out shows; decays slow enough that far tokens count."""
    g = torch.Generator().manual_seed(seed)
    D, w = cfg["width"], {}

    def mat(name, *shape, gain=1.0):
        w[name] = (torch.randn(*shape, generator=g) * (gain / shape[-1] ** 0.5)).bfloat16()

    def vec(name, *shape, mean=0.0, std=0.3):
        w[name] = (mean + std * torch.randn(*shape, generator=g)).bfloat16()

    mat("embed", cfg["vocab"], D, gain=D ** 0.5)
    mat("head", cfg["vocab"], D)
    vec("final.norm", D, mean=1.0)
    for i, layer in enumerate(cfg["layers"]):
        mx, p, mlp = layer["mixer"], f"l{i}.mix", layer.get("mlp")
        vec(f"l{i}.norm1", D, mean=1.0)
        if layer["type"] == "delta":
            H, G, dim, vdim, taps = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"], mx["conv"]
            for name, n in (("q", G * dim), ("k", G * dim), ("v", H * vdim)):
                mat(f"{p}.{name}", n, D)
                mat(f"{p}.{name}.conv", n, taps, gain=1.5)
            mat(p + ".b", H, D)
            mat(p + ".a", H, D)
            vec(p + ".A_log", H, mean=-2.0, std=1.0)
            vec(p + ".dt_bias", H, mean=-1.0, std=1.0)
            vec(p + ".norm", vdim, mean=1.0)
            mat(p + ".g", H * vdim, D)
            mat(p + ".o", D, H * vdim, gain=2.0)
        else:
            a, r = mx["left"], mx["right"]
            for name, n in (("q", a["heads"] * a["dim"]), ("k", a["kv_heads"] * a["dim"]), ("v", a["kv_heads"] * a["vdim"]), ("g", a["heads"] * a["vdim"])):
                mat(f"{p}.left.{name}", n, D)
            vec(p + ".left.q.norm", a["dim"], mean=1.0)
            vec(p + ".left.k.norm", a["dim"], mean=1.0)
            mat(p + ".left.o", D, a["heads"] * a["vdim"], gain=2.0)
            W, B = r["width"], r["blocks"]
            for name in ("y", "x"):
                mat(f"{p}.right.{name}", W, D)
                vec(f"{p}.right.{name}.b", W)
            mat(p + ".right.conv", W, r["conv"], gain=1.5)
            vec(p + ".right.conv.b", W)
            for name in ("ra", "ri"):
                mat(f"{p}.right.{name}", B, W // B, W // B)
                vec(f"{p}.right.{name}.b", B, W // B)
            vec(p + ".right.lam", W, mean=-4.0, std=1.5)
            mat(p + ".right.o", D, W, gain=2.0)
        if mlp is None:
            continue
        vec(f"l{i}.norm2", D, mean=1.0)
        units = [(f"l{i}.mlp", mlp["ff"])] if mlp["kind"] == "dense" else [(f"l{i}.mlp.e{e}", mlp["expert"]["ff"]) for e in range(mlp["router"]["experts"])]
        for m, ff in units:
            mat(m + ".gate", ff, D, gain=1.5)
            mat(m + ".up", ff, D, gain=1.5)
            mat(m + ".down", D, ff, gain=1.5)
        if mlp["kind"] == "moe":
            E, top = mlp["router"]["experts"], mlp["router"]["top"]
            w[f"l{i}.mlp.table"] = torch.stack([torch.randperm(E, generator=g)[:top] for _ in range(cfg["vocab"])]).int()
    return w
