"""Decoder with latent attention ("Bikelix") on dense weights, bf16 or f32.

A layer's attention caches one latent row and one rotated key part per position, shared by all heads; it sees a
sliding window, and its softmax carries a learned sink per head. A layer may read the cache of an earlier layer
instead of keeping its own. Sublayers read the residual stream as it is and every sum is normed afterwards
(x <- norm(alpha x + sublayer(x)), weights stored around zero); the feed-forward is a clamped gated unit.

Prompt portions expand keys and values (matrix products by the library, as the archive-code model's long prompts,
the rest in row kernels and one attention kernel). The token step keeps everything in the latent space:

    per layer   [dq | dkv] with the norm of the sum before it   (llvq_dn_gemv, norm or embed prologue)
                uq with the norm of the query latent            (norm prologue)
                query into the latent space; the token's cache row (llvq_dn_latent_query)
                attention over the ring, split over positions      (llvq_dn_latent_decode)
                merge, sink, value expansion                       (llvq_dn_latent_value)
                o                                               (plain)
                gate and up with the norm of the sum before it, the gated unit of their sums (norm prologue, glu epilogue)
                down                                            (plain)
    then        the last norm, and the head with the final norm, soft cap and greedy pick

The residual stream, norms, rotations, scores, softmax and the token step's activations are f32 in both element
types; in bf16 the weights, the prompt's activations and the cache are bf16.
"""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass
from typing import List, Optional, Sequence

import numpy as np

from . import _lib
from .cache import LatentRing
from .dense import DenseLM, DenseMatrix
from .registry import register

GLU_GAIN, GLU_SHIFT = 1.702, 1.0  # sigmoid(1.702 g), (u + 1)


@dataclass(frozen=True)
class LatentAttentionConfig:
    heads: int
    dim: int            # unrotated query/key dimensions per head
    rot_dim: int        # rotated ones
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    rot_base: float
    rot_dims: int
    window: Optional[int]   # positions a query sees, itself included; None: all before it
    kv_from: Optional[int] = None

    @staticmethod
    def parse(m: dict, layer: int) -> "LatentAttentionConfig":
        mask, rot = m.get("mask"), m["rot"]
        c = LatentAttentionConfig(int(m["heads"]), int(m["dim"]), int(m["rot_dim"]), int(m["vdim"]), int(m["q_rank"]), int(m["kv_rank"]),
                                  float(m["scale"]), float(rot["base"]), int(rot["dims"]),
                                  int(mask["size"]) if mask else None, None if m.get("kv_from") is None else int(m["kv_from"]))
        if min(c.heads, c.dim, c.rot_dim, c.vdim, c.q_rank, c.kv_rank) < 1 or (c.window is not None and c.window < 1):
            raise ValueError(f"layer {layer}: a size of {c} is not positive")
        if c.rot_dims % 2 or not 0 < c.rot_dims <= c.rot_dim:
            raise ValueError(f"layer {layer}: {c.rot_dims} rotated of {c.rot_dim} dimensions")
        return c


@dataclass(frozen=True)
class GatedMlpConfig:
    ff: int
    limit: float

    @staticmethod
    def parse(m: Optional[dict], layer: int) -> Optional["GatedMlpConfig"]:
        if m is None:
            return None
        if m.get("kind", "dense") != "dense":
            raise ValueError(f"layer {layer}: feed-forward of kind {m['kind']!r}; only 'dense' is known")
        return GatedMlpConfig(int(m["ff"]), float(m["limit"]))


@dataclass(frozen=True)
class LatentLayerConfig:
    attn: LatentAttentionConfig
    mlp: Optional[GatedMlpConfig]


@dataclass(frozen=True)
class LatentConfig:
    vocab: int
    width: int
    eps: float
    alpha: float                    # weight of the stream in x <- norm(alpha x + sublayer(x))
    embed_scale: float
    softcap: Optional[float]
    layers: Sequence[LatentLayerConfig]

    @staticmethod
    def parse(c: dict) -> "LatentConfig":
        layers: List[LatentLayerConfig] = []
        for i, l in enumerate(c["layers"]):
            if l["type"] != "latent_attention":
                raise ValueError(f"layer {i}: mixer {l['type']!r}; only 'latent_attention' is known")
            a = LatentAttentionConfig.parse(l["mixer"], i)
            if a.kv_from is not None:
                src = layers[a.kv_from].attn if 0 <= a.kv_from < i else None
                if src is None or src.kv_from is not None or (src.kv_rank, src.rot_dim, src.rot_base, src.rot_dims) != (
                        a.kv_rank, a.rot_dim, a.rot_base, a.rot_dims):
                    raise ValueError(f"layer {i} reads the cache of layer {a.kv_from}: it must be an earlier layer with a cache of its own "
                                     "and the same latent and rotation")
            layers.append(LatentLayerConfig(a, GatedMlpConfig.parse(l.get("mlp"), i)))
        if not layers:
            raise ValueError("a model without layers")
        cap = c.get("logit_softcap")
        return LatentConfig(int(c["vocab"]), int(c["width"]), float(c["norm"]["eps"]), float(c["postln_alpha"]),
                            float(c["embedding"]["scale"]), float(cap) if cap else None, layers)


class LatentLM(DenseLM):
    PHASES = ("embed", "projections", "latent_query", "attention", "latent_value", "norm", "head")

    def __init__(self, cfg: LatentConfig, tensor, dtype: str, capacity: int, device, prefill_chunk: int = 2048):
        """`tensor(name)` gives a weight by its name (any device)."""
        import torch
        self.cfg, self.eps, self.softcap = cfg, cfg.eps, cfg.softcap or 0.0
        self._init_dense(dtype, device, capacity, prefill_chunk)
        f32 = dict(dtype=torch.float32, device=device)

        def mat(*names, interleave: bool = False):
            return DenseMatrix([tensor(n) for n in names], self.dtype, device, interleave)

        def vec(*names, base: float = 0.0):
            return torch.cat([tensor(n).to(**f32) for n in names]) + base

        self.embed = self.head = mat("embed")
        if self.embed.w.shape[0] != cfg.vocab or self.embed.k != cfg.width:
            raise ValueError(f"embed is {tuple(tensor('embed').shape)}, config.json says {cfg.vocab} x {cfg.width}")
        self.final_norm = vec("final.norm", base=1.0)  # stored around zero
        self.layers, self.rings, tables = [], [], {}
        for i, lc in enumerate(cfg.layers):
            a, p = lc.attn, f"l{i}.mix"
            L = {"norm1": vec(f"l{i}.norm1", base=1.0), "dq_norm": vec(p + ".dq.norm"), "uq": mat(p + ".uq"), "ukv": mat(p + ".uk", p + ".uv"),
                 "sink": vec(p + ".sink"), "o": mat(p + ".o")}
            if a.kv_from is None:
                L["dq_dkv"], L["kv_norm"] = mat(p + ".dq", p + ".dkv"), vec(p + ".dkv.norm")
                readers = [i] + [k for k, o in enumerate(cfg.layers) if o.attn.kv_from == i]
                widest = max(min(cfg.layers[k].attn.window or capacity, capacity) for k in readers)
                self.rings.append(LatentRing(capacity, widest, prefill_chunk, a.kv_rank, a.rot_dim, self.dtype, device))
            else:
                L["dq_dkv"], L["kv_norm"] = mat(p + ".dq"), None
                self.rings.append(self.rings[a.kv_from])
            if lc.mlp is not None:
                m = f"l{i}.mlp"
                L.update(norm2=vec(f"l{i}.norm2", base=1.0), gate_up=mat(m + ".gate", m + ".up", interleave=True),  # (gate, up) pairs
                         gate_up_b=vec(m + ".gate.b", m + ".up.b").reshape(2, -1).t().reshape(-1).contiguous(),
                         down=mat(m + ".down"), down_b=vec(m + ".down.b"))
            self._check_layer(i, lc, L)
            if (a.rot_base, a.rot_dims) not in tables:  # angles in double, rounded once
                f = a.rot_base ** (-2.0 * np.arange(a.rot_dims // 2, dtype=np.float64) / a.rot_dims)
                ang = np.arange(capacity, dtype=np.float64)[:, None] * f[None, :]
                tables[a.rot_base, a.rot_dims] = tuple(torch.from_numpy(t(ang).astype(np.float32)).to(device) for t in (np.cos, np.sin))
            L["cos"], L["sin"] = tables[a.rot_base, a.rot_dims]
            self.layers.append(L)
        self._init_step()

    def _check_layer(self, i: int, lc: LatentLayerConfig, L: dict) -> None:
        a, D = lc.attn, self.cfg.width
        want = {"dq_dkv": (a.q_rank + (a.kv_rank + a.rot_dim if a.kv_from is None else 0), D), "uq": (a.heads * (a.dim + a.rot_dim), a.q_rank),
                "ukv": (a.heads * (a.dim + a.vdim), a.kv_rank), "o": (D, a.heads * a.vdim)}
        vecs = {"norm1": D, "dq_norm": a.q_rank, "sink": a.heads}
        if a.kv_from is None:
            vecs["kv_norm"] = a.kv_rank
        if lc.mlp is not None:
            want.update(gate_up=(2 * lc.mlp.ff, D), down=(D, lc.mlp.ff))
            vecs.update(norm2=D, gate_up_b=2 * lc.mlp.ff, down_b=D)
        for name, shape in want.items():
            if (L[name].n, L[name].k) != shape:
                raise ValueError(f"layer {i}: {name} is {(L[name].n, L[name].k)}, config.json says {shape}")
        for name, n in vecs.items():
            if L[name].numel() != n:
                raise ValueError(f"layer {i}: {name} has {L[name].numel()} values, config.json says {n}")

    # ---- the token step ----------------------------------------------------------
    def _init_step(self) -> None:
        """Fixed buffers and the launch list of one token: (phase, call) pairs over prebuilt descriptors."""
        import torch
        cfg, lib, dev = self.cfg, self.lib, self.device
        f32 = dict(dtype=torch.float32, device=dev)
        attn = [lc.attn for lc in cfg.layers]
        sms = torch.cuda.get_device_properties(dev).multi_processor_count

        def splits(a):
            heads, tile = (16, 64) if self.dtype == torch.bfloat16 else (8, 32)  # per CTA and step of the attention kernel
            groups = -(-a.heads // heads)
            return max(1, min(-(-min(a.window or self.capacity, self.capacity) // tile), 2 * sms // groups, 128))

        buf = lambda n: torch.zeros(n, **f32)
        self._stream = [buf(cfg.width), buf(cfg.width)]  # a norm reads one and stores the other
        self._x = buf(cfg.width)                         # the stream behind the last layer
        self._y = buf(max(L["dq_dkv"].n for L in self.layers))
        self._q = buf(max(L["uq"].n for L in self.layers))
        self._ctx = buf(max(L["o"].k for L in self.layers))
        self._o, self._down = buf(cfg.width), buf(cfg.width)
        self._act = buf(max([lc.mlp.ff for lc in cfg.layers if lc.mlp is not None] or [1]))
        self._qlat = buf(max(a.heads * r.ld for a, r in zip(attn, self.rings)))
        self._part = buf(max(a.heads * splits(a) * (a.kv_rank + 2) for a in attn))
        self._init_head()
        ptr = lambda t: t.data_ptr() if t is not None else None
        self._lat = []
        for a, L, r in zip(attn, self.layers, self.rings):
            self._lat.append(_lib.DenseLatent(
                dtype=self.dt, heads=a.heads, dim=a.dim, rot_dim=a.rot_dim, vdim=a.vdim, kv_rank=a.kv_rank, ldk=L["ukv"].ld, slots=r.slots,
                ld=r.ld, rot_dims=a.rot_dims, window=min(a.window or self.capacity, self.capacity), splits=splits(a), scale=a.scale,
                eps=cfg.eps, ring=ptr(r.rows), cos_t=ptr(L["cos"]), sin_t=ptr(L["sin"]), uk=L["ukv"].ptr(), uv=L["ukv"].ptr(a.heads * a.dim),
                kv_norm=ptr(L["kv_norm"]), sink=ptr(L["sink"]), qlat=ptr(self._qlat), part=ptr(self._part)))

        steps = []
        tok, pos = self._tok.data_ptr(), self._pos.data_ptr()

        def gemv(m, y, bias=None, phase="projections", **kw):
            d = _lib.DenseGemv(dtype=self.dt, n_out=m.n, k=m.k, ldw=m.ld, w=m.ptr(), bias=ptr(bias), y=ptr(y), eps=cfg.eps, **kw)
            steps.append((phase, lambda st, d=d: _lib.check_dense(lib.llvq_dn_gemv(C.byref(d), st))))

        def normed(delta, w):
            """Prologue fields of x <- norm(alpha x + delta): the stream moves to the other buffer."""
            kw = dict(prologue=_lib.DN_NORM, alpha=cfg.alpha, x=ptr(self._stream[0]), delta=ptr(delta), norm_w=ptr(w), a_out=ptr(self._stream[1]))
            self._stream.reverse()
            return kw

        pending = None  # (sublayer output, norm weight) of the sum the next projection forms
        for i, (lc, L) in enumerate(zip(cfg.layers, self.layers)):
            a, lat = lc.attn, self._lat[i]
            if pending is None:
                first = dict(prologue=_lib.DN_EMBED, scale=cfg.embed_scale, table=self.embed.ptr(), ld_table=self.embed.ld, table_rows=cfg.vocab,
                             token=tok, a_out=ptr(self._stream[0]))
            else:
                first = normed(*pending)
            gemv(L["dq_dkv"], self._y, **first)
            gemv(L["uq"], self._q, prologue=_lib.DN_NORM, alpha=1.0, x=ptr(self._y), norm_w=ptr(L["dq_norm"]))
            y_kv = self._y.data_ptr() + 4 * a.q_rank if a.kv_from is None else None
            steps.append(("latent_query", lambda st, lat=lat, y=y_kv: _lib.check_dense(lib.llvq_dn_latent_query(C.byref(lat), ptr(self._q), y, pos, st))))
            steps.append(("attention", lambda st, lat=lat: _lib.check_dense(lib.llvq_dn_latent_decode(C.byref(lat), pos, st))))
            steps.append(("latent_value", lambda st, lat=lat: _lib.check_dense(lib.llvq_dn_latent_value(C.byref(lat), ptr(self._ctx), st))))
            gemv(L["o"], self._o, prologue=_lib.DN_PLAIN, x=ptr(self._ctx))
            pending = (self._o, L["norm1"])
            if lc.mlp is not None:
                gemv(L["gate_up"], self._act, L["gate_up_b"], glu=1, limit=lc.mlp.limit, gain=GLU_GAIN, shift=GLU_SHIFT, **normed(*pending))
                gemv(L["down"], self._down, L["down_b"], prologue=_lib.DN_PLAIN, x=ptr(self._act))
                pending = (self._down, L["norm2"])
        last, (delta, w) = self._stream[0], pending
        steps.append(("norm", lambda st: _lib.check_dense(lib.llvq_dn_postnorm_rows(
            _lib.DN_F32, ptr(last), ptr(delta), None, ptr(w), cfg.alpha, cfg.eps, None, ptr(self._x), 1, cfg.width, st))))
        steps.append(("head", lambda st: self._head(self._x, st)))
        self._steps = steps

    # ---- prompt portions ---------------------------------------------------------
    def _expand(self, c, ukv, a, transposed: bool):
        """Keys and values of cached latents c [n, kv_rank]: ([n, keys | values], None), or ([n, keys], [values, n to a
        multiple of 8]) for the attention kernel that reads the values along the positions."""
        import torch
        if not transposed:
            return self._mm(c, ukv.rows(0)), None
        n, split = c.shape[0], a.heads * a.dim
        vt = torch.empty(a.heads * a.vdim, -(-n // 8) * 8, dtype=self.dtype, device=self.device)
        if n % 8:
            vt[:, n:].zero_()
        torch.mm(ukv.rows(split), c.t(), out=vt[:, :n])
        return self._mm(c, ukv.rows(0, split)), vt

    def hidden(self, tokens, pos, end: int, layers_out: Optional[list] = None):
        """tokens, pos: int64 [L], positions [end - L, end); returns the f32 stream [L, width] behind the last layer.
        `layers_out` collects a copy of the stream behind every layer."""
        import torch
        cfg, lib, st = self.cfg, self.lib, self._cuda_stream()
        n, D = tokens.numel(), cfg.width
        start = end - n
        if n > self.prefill_chunk or start < 0 or end > self.capacity:
            raise ValueError(f"a portion of {n} tokens at position {start} (at most {self.prefill_chunk}, capacity {self.capacity})")
        check = _lib.check_dense
        new = lambda *shape: torch.empty(*shape, dtype=self.dtype, device=self.device)
        x = torch.empty(n, D, dtype=torch.float32, device=self.device)
        xt = new(n, D)  # the stream in the projections' element type
        check(lib.llvq_dn_embed_rows(self.dt, self.embed.ptr(), self.embed.ld, cfg.vocab, tokens.data_ptr(), n, D, cfg.embed_scale, x.data_ptr(),
                                     xt.data_ptr(), st))

        def add_norm(y, bias, w):
            check(lib.llvq_dn_postnorm_rows(self.dt, x.data_ptr(), y.data_ptr(), bias.data_ptr() if bias is not None else None, w.data_ptr(),
                                            cfg.alpha, cfg.eps, xt.data_ptr(), x.data_ptr(), n, D, st))

        for lc, L, lat, ring in zip(cfg.layers, self.layers, self._lat, self.rings):
            a = lc.attn
            y = self._mm(xt, L["dq_dkv"].rows(0))
            cq = new(n, a.q_rank)
            check(lib.llvq_dn_latent_rows(C.byref(lat), y.data_ptr(), y.shape[1], a.q_rank, L["dq_norm"].data_ptr(), cq.data_ptr(), start, n,
                                          1 if a.kv_from is None else 0, st))
            q = self._mm(cq, L["uq"].rows(0))
            lo = max(0, start - lat.window + 1)  # the first position any query of the portion sees
            rows = ring.read(lo, end)
            kv, vt = self._expand(rows[:, :a.kv_rank], L["ukv"], a, lib.llvq_dn_latent_prefill_transposes(C.byref(lat), n))
            ctx = new(n, a.heads * a.vdim)
            check(lib.llvq_dn_latent_prefill(C.byref(lat), q.data_ptr(), kv.data_ptr(), kv.shape[1],
                                             rows.data_ptr() + a.kv_rank * rows.element_size(), ring.ld, vt.data_ptr() if vt is not None else None,
                                             vt.shape[1] if vt is not None else 0, n, end - lo, start, lo, ctx.data_ptr(), 0, st))
            add_norm(self._mm(ctx, L["o"].rows(0)), None, L["norm1"])
            if lc.mlp is not None:
                gu = self._mm(xt, L["gate_up"].rows(0))
                act = new(n, lc.mlp.ff)
                check(lib.llvq_dn_glu_rows(self.dt, gu.data_ptr(), L["gate_up_b"].data_ptr(), act.data_ptr(), n, lc.mlp.ff, lc.mlp.limit, GLU_GAIN,
                                           GLU_SHIFT, st))
                add_norm(self._mm(act, L["down"].rows(0)), L["down_b"], L["norm2"])
            if layers_out is not None:
                layers_out.append(x.clone())
        return x

    def cache_bytes(self) -> int:
        """Bytes of all rings (a shared one counts once)."""
        return sum(r.rows.numel() * r.rows.element_size() for r in {id(r): r for r in self.rings}.values())


@register("Bikelix", "folder", ("bfloat16", "float32"))
def _load_latent(config, weights, dtype, capacity, device, **options):
    import torch
    if not torch.cuda.is_available():
        raise RuntimeError("a CUDA device is needed: the library has no CPU path")
    torch.cuda.set_device(device)
    return LatentLM(LatentConfig.parse(config), weights.tensor, dtype, capacity, torch.device("cuda", device), **options)
