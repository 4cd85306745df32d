"""Hybrid decoder ("Dozusun") on dense weights, bf16 or f32.

A layer's two sublayers read the same residual stream, each through a norm of its own: x <- x + (mixer + feed-forward).
Mixers: a gated delta rule, or windowed grouped-query attention and a real-gated linear recurrence side by side.
Feed-forwards: a gated unit, a stack of them of which the token's id names some, or none. A span of layers may run several
times with the same weights; every pass has a cache and a state of its own.

Token step, per layer run:

    every projection of both sublayers, their norms in the prologue     (llvq_dn_gemv, two row sets)
    the mixer: attention and recurrence in one launch, or the delta rule (llvq_dn_mixer_token, llvq_dn_delta_token)
    every output projection and the residual sum                        (llvq_dn_gemv over activations side by side)

Prompt portions run the projections as matrix products by the library and the rest in row kernels, the attention kernels
of the latent model, and one scan per recurrence. The residual stream, norms, scores, softmax, states and all that enters
a recurrence are f32 in both element types.
"""
from __future__ import annotations

import ctypes as C
import math
from dataclasses import dataclass
from typing import List, Optional, Sequence, Union

from . import _lib
from .cache import ConvInputs, KvRing, RecurrentState, whole_vectors
from .dense import ColumnMatrix, DenseLM, DenseMatrix
from .registry import register


def _positive(layer, c, *values):
    if min(values) < 1:
        raise ValueError(f"layer {layer}: a size of {c} is not positive")


@dataclass(frozen=True)
class AttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: Optional[int]   # positions a query sees, itself included; None: all before it

    @staticmethod
    def parse(m: dict, layer: int) -> "AttentionConfig":
        mask = m.get("mask")
        c = AttentionConfig(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), float(m["scale"]), int(mask["size"]) if mask else None)
        _positive(layer, c, c.heads, c.kv_heads, c.dim, c.vdim, 1 if c.window is None else c.window)
        if c.heads % c.kv_heads:
            raise ValueError(f"layer {layer}: {c.heads} heads over {c.kv_heads} key/value heads")
        return c


@dataclass(frozen=True)
class RecurrenceConfig:
    width: int
    blocks: int
    taps: int

    @staticmethod
    def parse(m: dict, layer: int) -> "RecurrenceConfig":
        c = RecurrenceConfig(int(m["width"]), int(m["blocks"]), int(m["conv"]))
        _positive(layer, c, c.width, c.blocks, c.taps)
        if c.width % c.blocks:
            raise ValueError(f"layer {layer}: a width of {c.width} in {c.blocks} blocks")
        return c


@dataclass(frozen=True)
class ParallelConfig:
    left: AttentionConfig
    right: RecurrenceConfig
    left_scale: float
    right_scale: float

    @staticmethod
    def parse(m: dict, layer: int) -> "ParallelConfig":
        return ParallelConfig(AttentionConfig.parse(m["left"], layer), RecurrenceConfig.parse(m["right"], layer), float(m["left_scale"]), float(m["right_scale"]))


@dataclass(frozen=True)
class DeltaConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    taps: int

    @staticmethod
    def parse(m: dict, layer: int) -> "DeltaConfig":
        c = DeltaConfig(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), int(m["conv"]))
        _positive(layer, c, c.heads, c.kv_heads, c.dim, c.vdim, c.taps)
        if c.heads % c.kv_heads:
            raise ValueError(f"layer {layer}: {c.heads} heads over {c.kv_heads} key heads")
        return c

    @property
    def channels(self) -> int:
        return 2 * self.kv_heads * self.dim + self.heads * self.vdim


@dataclass(frozen=True)
class MlpConfig:
    """experts 0: one dense unit; else a stack of units of ff, `top` of them per token."""
    ff: int
    experts: int = 0
    top: int = 0

    @staticmethod
    def parse(m: Optional[dict], layer: int) -> Optional["MlpConfig"]:
        if m is None:
            return None
        if m["kind"] == "dense":
            c = MlpConfig(int(m["ff"]))
        elif m["kind"] == "moe":
            c = MlpConfig(int(m["expert"]["ff"]), int(m["router"]["experts"]), int(m["router"]["top"]))
            if not 1 <= c.top <= c.experts:
                raise ValueError(f"layer {layer}: {c.top} of {c.experts} experts")
        else:
            raise ValueError(f"layer {layer}: feed-forward of kind {m['kind']!r}; 'dense' and 'moe' are known")
        _positive(layer, c, c.ff)
        return c


_MIXERS = {"parallel": ParallelConfig, "delta": DeltaConfig}


@dataclass(frozen=True)
class HybridLayerConfig:
    mixer: Union[ParallelConfig, DeltaConfig]
    mlp: Optional[MlpConfig]


@dataclass(frozen=True)
class HybridConfig:
    vocab: int
    width: int
    eps: float
    layers: Sequence[HybridLayerConfig]
    runs: Sequence[int]     # layer indices in the order they run

    @staticmethod
    def parse(c: dict) -> "HybridConfig":
        layers: List[HybridLayerConfig] = []
        for i, l in enumerate(c["layers"]):
            if l["type"] not in _MIXERS:
                raise ValueError(f"layer {i}: mixer {l['type']!r}; {sorted(_MIXERS)} are known")
            layers.append(HybridLayerConfig(_MIXERS[l["type"]].parse(l["mixer"], i), MlpConfig.parse(l.get("mlp"), i)))
        if not layers:
            raise ValueError("a model without layers")
        return HybridConfig(int(c["vocab"]), int(c["width"]), float(c["norm"]["eps"]), layers, HybridConfig.order(len(layers), c.get("loop")))

    @staticmethod
    def order(n: int, loop: Optional[dict]) -> Sequence[int]:
        if not loop:
            return tuple(range(n))
        start, stop, times = int(loop["start"]), int(loop["stop"]), int(loop["times"])
        if not 0 <= start < stop <= n or times < 1:
            raise ValueError(f"a loop over layers {start} to {stop} of {n}, {times} times")
        return tuple(range(start)) + tuple(range(start, stop)) * times + tuple(range(stop, n))


class _Route:
    """Which rows of a portion go to which expert: rows sorted by expert, where each row's results end up."""

    def __init__(self, lib, table, experts: int, tokens, stream):
        import torch
        n, self.top = tokens.numel(), table.shape[1]
        new = lambda k: torch.empty(k, dtype=torch.int32, device=table.device)
        self.source, self.places, self.ends = new(n * self.top), new(n * self.top), new(experts)
        _lib.check_dense(lib.llvq_dn_route_rows(table.data_ptr(), table.shape[0], self.top, experts, tokens.data_ptr(), n, self.source.data_ptr(),
                                                self.places.data_ptr(), self.ends.data_ptr(), stream))
        self._host = None

    def host_ends(self) -> List[int]:
        if self._host is None:
            self._host = self.ends.tolist()
        return self._host


class HybridLM(DenseLM):
    PHASES = ("projections", "mixer", "delta", "output", "head")
    # columns one token projection takes, in bf16 as segments of a matrix each; beyond, mixer and feed-forward have one each
    JOINED_SEGMENTS, SEGMENT, JOINED_COLUMNS_F32 = 8, 2560, 40000

    def __init__(self, cfg: HybridConfig, tensor, dtype: str, capacity: int, device, prefill_chunk: int = 2048):
        """`tensor(name)` gives a weight by its name (any device)."""
        self.cfg, self.eps, self._tensor = cfg, cfg.eps, tensor
        self._init_dense(dtype, device, capacity, prefill_chunk)
        D = cfg.width
        self.embed, self.head = self._mat("embed", shape=(cfg.vocab, D)), self._mat("head", shape=(cfg.vocab, D))
        self.final_norm = self._vec("final.norm", D)
        self.layers = []
        for i, lc in enumerate(cfg.layers):
            L = {"norm1": self._vec(f"l{i}.norm1", D)}
            outs = (self._load_parallel if isinstance(lc.mixer, ParallelConfig) else self._load_delta)(f"l{i}.mix", lc.mixer, L)
            self._load_mlp(f"l{i}", lc.mlp, L, outs)
            self.layers.append(L)
        del self._tensor
        self._init_state()
        self._init_step()

    # ---- weights -------------------------------------------------------------------
    def _take(self, name: str, *shape: int):
        t = self._tensor(name)
        if tuple(t.shape) != shape:
            raise ValueError(f"{name} is {tuple(t.shape)}, config.json says {shape}")
        return t

    def _vec(self, name: str, *shape: int):
        import torch
        return self._take(name, *shape).to(dtype=torch.float32, device=self.device).contiguous()

    def _mat(self, name: str, shape):
        return DenseMatrix([self._take(name, *shape)], self.dtype, self.device)

    def _load_parallel(self, p: str, c: ParallelConfig, L: dict):
        import torch
        a, r, D = c.left, c.right, self.cfg.width
        l, n = p + ".left", r.width // r.blocks
        rows = [(l + ".q", a.heads * a.dim), (l + ".k", a.kv_heads * a.dim), (l + ".v", a.kv_heads * a.vdim), (l + ".g", a.heads * a.vdim),
                (p + ".right.y", r.width), (p + ".right.x", r.width)]
        L["in"] = DenseMatrix([self._take(name, k, D) for name, k in rows], self.dtype, self.device)
        at, L["at"] = 0, {}
        for name, k in rows:
            L["at"][name.rsplit(".", 1)[1]] = at
            at += k
        L["in_b"] = torch.zeros(L["in"].n, dtype=torch.float32, device=self.device)
        for name in ("y", "x"):
            lo = L["at"][name]
            L["in_b"][lo:lo + r.width] = self._vec(f"{p}.right.{name}.b", r.width)
        L["y_b"], L["x_b"] = (L["in_b"][L["at"][k]:L["at"][k] + r.width].clone() for k in ("y", "x"))  # vectors of their own: aligned
        L["q_norm"], L["k_norm"] = self._vec(l + ".q.norm", a.dim), self._vec(l + ".k.norm", a.dim)
        p += ".right"
        L["conv"], L["conv_b"] = self._vec(p + ".conv", r.width, r.taps), self._vec(p + ".conv.b", r.width)
        L["lam"] = torch.logaddexp(self._vec(p + ".lam", r.width).double(), torch.zeros((), dtype=torch.float64, device=self.device)).float()  # softplus
        gates = [self._take(f"{p}.{k}", r.blocks, n, n) for k in ("ra", "ri")]
        L["gates"] = torch.zeros(r.blocks, 2 * n, whole_vectors(n, self.dtype), dtype=self.dtype, device=self.device)
        for k, g in enumerate(gates):
            L["gates"][:, k * n:(k + 1) * n, :n].copy_(g)
        L["gates_b"] = torch.cat([self._vec(f"{p}.{k}.b", r.blocks, n) for k in ("ra", "ri")], dim=1).contiguous()
        return [self._take(l + ".o", D, a.heads * a.vdim), self._take(p + ".o", D, r.width)]

    def _load_delta(self, p: str, c: DeltaConfig, L: dict):
        import torch
        D, qk, v = self.cfg.width, c.kv_heads * c.dim, c.heads * c.vdim
        rows = [("q", qk), ("k", qk), ("v", v), ("g", v), ("b", c.heads), ("a", c.heads)]
        L["in"] = DenseMatrix([self._take(f"{p}.{name}", k, D) for name, k in rows], self.dtype, self.device)
        L["conv"] = torch.cat([self._vec(f"{p}.{name}.conv", k, c.taps) for name, k in rows[:3]])
        L["decay"] = self._vec(p + ".A_log", c.heads).double().exp().float()
        L["dt_bias"], L["norm"] = self._vec(p + ".dt_bias", c.heads), self._vec(p + ".norm", c.vdim)
        return [self._take(p + ".o", D, v)]

    def _load_mlp(self, p: str, c: Optional[MlpConfig], L: dict, outs) -> None:
        """The feed-forward's matrices, and the output projection of the mixer's parts (and a dense unit's, where one
        token projection takes them all)."""
        import torch
        D, m = self.cfg.width, p + ".mlp"
        L["parts"] = len(outs)
        own = sum(whole_vectors(o.shape[1], self.dtype) for o in outs)

        def joined(columns, routed):
            """Whether the mixer's columns and so many more, or `routed` matrices of so many, go into one projection."""
            if self.dtype == torch.float32:
                return own + max(routed, 1) * columns <= self.JOINED_COLUMNS_F32
            segments = -(-own // self.SEGMENT) + routed * -(-columns // self.SEGMENT) if routed else -(-(own + columns) // self.SEGMENT)
            return segments <= self.JOINED_SEGMENTS
        if c is not None:
            L["norm2"] = self._vec(p + ".norm2", D)
        if c is not None and not c.experts:
            L["gate_up"] = DenseMatrix([self._take(f"{m}.{k}", c.ff, D) for k in ("gate", "up")], self.dtype, self.device, interleave=True)
            down = self._take(m + ".down", D, c.ff)
            both = joined(whole_vectors(c.ff, self.dtype), 0)
            L["down"] = None if both else DenseMatrix([down], self.dtype, self.device)
            outs = [*outs, down] if both else outs
        elif c is not None:
            ffp = whole_vectors(c.ff, self.dtype)
            up = torch.zeros(c.experts, ffp, 2, whole_vectors(D, self.dtype), dtype=self.dtype, device=self.device)  # (gate, up) pairs
            down = torch.zeros(c.experts, D, ffp, dtype=self.dtype, device=self.device)
            for e in range(c.experts):
                up[e, :c.ff, 0, :D].copy_(self._take(f"{m}.e{e}.gate", c.ff, D))
                up[e, :c.ff, 1, :D].copy_(self._take(f"{m}.e{e}.up", c.ff, D))
                down[e, :, :c.ff].copy_(self._take(f"{m}.e{e}.down", D, c.ff))
            L["experts_up"], L["experts_down"], L["routed_apart"] = up.flatten(1, 2), down, not joined(ffp, c.top)
            L["table"] = self._take(m + ".table", self.cfg.vocab, c.top).to(dtype=torch.int32, device=self.device).contiguous()
            if int(L["table"].min()) < 0 or int(L["table"].max()) >= c.experts:
                raise ValueError(f"{m}.table names experts outside 0 .. {c.experts - 1}")
        L["out"] = ColumnMatrix(outs, self.dtype, self.device)

    # ---- what a sequence keeps -------------------------------------------------------
    def _window(self, a: AttentionConfig) -> int:
        return min(a.window or self.capacity, self.capacity)

    def _init_state(self) -> None:
        self.states = []   # one per layer run
        for i in self.cfg.runs:
            c, dev = self.cfg.layers[i].mixer, self.device
            if isinstance(c, ParallelConfig):
                self.states.append({"ring": KvRing(self.capacity, self._window(c.left), self.prefill_chunk, c.left.kv_heads, c.left.dim, c.left.vdim,
                                                   self.dtype, dev),
                                    "conv": ConvInputs(c.right.taps, c.right.width, dev), "state": RecurrentState(c.right.width, device=dev)})
            else:
                self.states.append({"conv": ConvInputs(c.taps, c.channels, dev),
                                    "state": RecurrentState(c.heads, c.dim, -(-c.vdim // 4) * 4, device=dev)})

    def cache_bytes(self) -> int:
        """Bytes of all rings, states and convolution inputs."""
        size = lambda t: t.numel() * t.element_size()
        return sum(size(s["conv"].rows) + size(s["state"].halves) + (size(s["ring"].rows) if "ring" in s else 0) for s in self.states)

    # ---- the token step ----------------------------------------------------------
    def _init_step(self) -> None:
        """Fixed buffers and the launch list of one token: (phase, call) pairs over prebuilt descriptors."""
        import torch
        cfg, lib, dev, check = self.cfg, self.lib, self.device, _lib.check_dense
        sms = torch.cuda.get_device_properties(dev).multi_processor_count
        ptr = lambda t, at=0: t.data_ptr() + at * t.element_size() if t is not None else None
        buf = lambda n, dtype=torch.float32: torch.zeros(n, dtype=dtype, device=dev)
        mixers = [lc.mixer for lc in cfg.layers]
        attn = [c.left for c in mixers if isinstance(c, ParallelConfig)]
        delta = [c for c in mixers if isinstance(c, DeltaConfig)]

        def units(a):  # groups of heads a CTA of the attention serves
            return a.kv_heads * -(-a.heads // a.kv_heads // 4)

        def splits(a):
            return max(1, min(-(-self._window(a) // 64), 2 * sms // units(a), 128))

        def act_columns(L, lc):
            down = lc.mlp.top * L["experts_down"].shape[2] if lc.mlp is not None and lc.mlp.experts else L["down"].ld if L.get("down") is not None else 0
            return L["out"].ld + down

        self._x = buf(cfg.width)
        self._y = buf(max(L["in"].n for L in self.layers))
        self._act = buf(max(act_columns(L, lc) for L, lc in zip(self.layers, cfg.layers)))
        self._part = buf(max([a.heads * splits(a) * (a.vdim + 2) for a in attn] or [1]))
        self._o = buf(max([c.heads * -(-c.vdim // 4) * 4 for c in delta] or [1]))
        self._arrived = buf(max([units(a) for a in attn] + [c.heads for c in delta]), torch.int32)
        self._init_head()
        tok, pos, steps = self._tok.data_ptr(), self._pos.data_ptr(), []

        def gemv(phase, m, **kw):
            own = dict(n_out=m.n, k=m.k, ldw=m.ld, w=m.ptr()) if m is not None else dict(n_out=cfg.width)
            d = _lib.DenseGemv(dtype=self.dt, eps=self.eps, alpha=1.0, limit=math.inf, gain=1.0, **own, **kw)
            steps.append((phase, lambda st: check(lib.llvq_dn_gemv(C.byref(d), st))))

        self._mix = []   # descriptors per layer run
        for k, (i, s) in enumerate(zip(cfg.runs, self.states)):
            L, lc = self.layers[i], cfg.layers[i]
            c, mlp = lc.mixer, lc.mlp
            out, parts = L["out"], L["parts"]
            act_at = out.at[parts] if len(out.at) > parts else out.ld  # the feed-forward's activation
            route = {}
            kw = dict(prologue=_lib.DN_NORM, norm_w=ptr(L["norm1"]), y=ptr(self._y), bias=ptr(L.get("in_b")))
            if k == 0:  # the stream starts at the token's embedding
                kw.update(table=self.embed.ptr(), ld_table=self.embed.ld, table_rows=cfg.vocab, token=tok, scale=1.0, t_out=ptr(self._x))
            else:
                kw.update(x=ptr(self._x))
            if mlp is not None:
                kw.update(norm_w2=ptr(L["norm2"]), y2=ptr(self._act, act_at), glu2=1)
                if mlp.experts:
                    route = dict(token=tok, route=ptr(L["table"]), route_rows=cfg.vocab, top=mlp.top, matrices=mlp.experts)
                    kw.update(w2=ptr(L["experts_up"]), rows2=mlp.top * L["experts_up"].shape[1], glu_scale=1.0 / mlp.top, **route)
                else:
                    kw.update(w2=L["gate_up"].ptr(), rows2=L["gate_up"].n)
            gemv("projections", L["in"], **kw)

            if isinstance(c, ParallelConfig):
                a, r, at, ring = c.left, c.right, L["at"], s["ring"]
                g = _lib.DenseGqa(dtype=self.dt, heads=a.heads, kv_heads=a.kv_heads, dim=a.dim, vdim=a.vdim, slots=ring.slots, ld=ring.ld, kd=ring.kd,
                                  vd=ring.vd, window=self._window(a), splits=splits(a), scale=a.scale, eps=self.eps, out_scale=c.left_scale,
                                  ring=ptr(ring.rows), q_norm=ptr(L["q_norm"]), k_norm=ptr(L["k_norm"]), q=ptr(self._y, at["q"]), k=ptr(self._y, at["k"]),
                                  v=ptr(self._y, at["v"]), gate=ptr(self._y, at["g"]), part=ptr(self._part), arrived=ptr(self._arrived),
                                  out=ptr(self._act, out.at[0]))
                u = _lib.DenseLru(dtype=self.dt, blocks=r.blocks, n=r.width // r.blocks, taps=r.taps, ldw=L["gates"].shape[2], out_scale=c.right_scale,
                                  conv_w=ptr(L["conv"]), conv_b=ptr(L["conv_b"]), b=ptr(L["gates_b"]), lam=ptr(L["lam"]), conv=ptr(s["conv"].rows),
                                  state=ptr(s["state"].halves), w=ptr(L["gates"]), x=ptr(self._y, at["x"]), y=ptr(self._y, at["y"]),
                                  out=ptr(self._act, out.at[1]))
                self._mix.append((g, u))
                steps.append(("mixer", lambda st, g=g, u=u: check(lib.llvq_dn_mixer_token(C.byref(g), C.byref(u), pos, st))))
            else:
                v = 2 * c.kv_heads * c.dim + c.heads * c.vdim
                d = _lib.DenseDelta(dtype=self.dt, heads=c.heads, kv_heads=c.kv_heads, dim=c.dim, vdim=c.vdim, vp=s["state"].halves.shape[3], taps=c.taps,
                                    eps=self.eps, conv_w=ptr(L["conv"]), decay=ptr(L["decay"]), dt_bias=ptr(L["dt_bias"]), norm=ptr(L["norm"]),
                                    conv=ptr(s["conv"].rows), state=ptr(s["state"].halves), x=ptr(self._y), gate=ptr(self._y, v),
                                    beta=ptr(self._y, v + c.heads * c.vdim), alpha=ptr(self._y, v + c.heads * c.vdim + c.heads), o=ptr(self._o),
                                    arrived=ptr(self._arrived), out=ptr(self._act, out.at[0]))
                self._mix.append(d)
                steps.append(("delta", lambda st, d=d: check(lib.llvq_dn_delta_token(C.byref(d), pos, st))))

            kw = dict(prologue=_lib.DN_PLAIN, y=ptr(self._x), residual=ptr(self._x))
            if route:
                down = L["experts_down"]
                route.update(w_r=ptr(down), k_r=down.shape[2], ld_r=down.shape[2])
                if L["routed_apart"]:
                    gemv("output", out, x=ptr(self._act), **kw)
                    gemv("output", None, x=ptr(self._act, act_at), **kw, **route)
                else:
                    gemv("output", out, x=ptr(self._act), **kw, **route)
            else:
                gemv("output", out, x=ptr(self._act), **kw)
                if L.get("down") is not None:
                    gemv("output", L["down"], x=ptr(self._act, act_at), **kw)
        steps.append(("head", lambda st: self._head(self._x, st)))
        self._steps = steps

    # ---- prompt portions ---------------------------------------------------------
    def _grouped(self, x, stack, route: _Route):
        """Rows of x, sorted by expert, through their expert's matrix [experts, out, in]."""
        import torch
        if self.dtype == torch.bfloat16 and not (stack.shape[1] | stack.shape[2]) & 7:
            return torch._grouped_mm(x, stack.transpose(1, 2), offs=route.ends)
        y = torch.empty(x.shape[0], stack.shape[1], dtype=x.dtype, device=x.device)
        lo = 0
        for e, hi in enumerate(route.host_ends()):
            if hi > lo:
                y[lo:hi] = self._mm(x[lo:hi], stack[e])
            lo = hi
        return y

    def _parallel_rows(self, h, L, c: ParallelConfig, s, desc, act, start: int, end: int, st) -> None:
        import torch
        a, r, n, lib, check = c.left, c.right, end - start, self.lib, _lib.check_dense
        g, u = desc
        new = lambda *shape: torch.empty(*shape, dtype=self.dtype, device=self.device)
        y = self._mm(h, L["in"].rows(0))
        ld, size = y.shape[1], y.element_size()
        at = {k: y.data_ptr() + v * size for k, v in L["at"].items()}
        to = lambda part: act.data_ptr() + L["out"].at[part] * size
        qn, ctx = new(n, a.heads * a.dim), new(n, a.heads * a.vdim)
        check(lib.llvq_dn_gqa_rows(C.byref(g), at["q"], at["k"], at["v"], ld, qn.data_ptr(), start, n, st))
        lo = max(0, start - g.window + 1)  # the first position any query of the portion sees
        rows = s["ring"].read(lo, end)
        vt = s["ring"].values_transposed(rows) if lib.llvq_dn_gqa_prefill_transposes(C.byref(g), n) else None
        check(lib.llvq_dn_gqa_prefill(C.byref(g), qn.data_ptr(), rows.data_ptr(), vt.data_ptr() if vt is not None else None,
                                      vt.shape[1] if vt is not None else 0, n, end - lo, start, lo, ctx.data_ptr(), 0, st))
        check(lib.llvq_dn_gate_rows(self.dt, ctx.data_ptr(), ctx.shape[1], at["g"], ld, to(0), act.shape[1], n, ctx.shape[1], c.left_scale, st))
        conv, ring = new(n, r.width), s["conv"].rows.data_ptr()
        check(lib.llvq_dn_conv_rows(self.dt, at["x"], ld, L["x_b"].data_ptr(), L["conv"].data_ptr(), L["conv_b"].data_ptr(), ring, conv.data_ptr(),
                                    r.width, r.taps, start, n, st))
        check(lib.llvq_dn_conv_keep(self.dt, at["x"], ld, L["x_b"].data_ptr(), ring, r.width, r.taps, start, n, st))
        k = r.width // r.blocks
        z = self._bmm(conv.view(n, r.blocks, k).transpose(0, 1), L["gates"][:, :, :k], torch.float32)
        check(lib.llvq_dn_lru_rows(C.byref(u), conv.data_ptr(), z.data_ptr(), at["y"], ld, L["y_b"].data_ptr(), to(1), act.shape[1], start, n, st))

    def _delta_rows(self, h, L, c: DeltaConfig, desc, act, start: int, end: int, st) -> None:
        import torch
        n, lib, check = end - start, self.lib, _lib.check_dense
        v = c.channels + c.heads * c.vdim
        y = self._mm(h, L["in"].rows(0, v))
        ba = self._mm(h, L["in"].rows(v), torch.float32)
        floats = C.c_size_t()
        check(lib.llvq_dn_delta_scratch(C.byref(desc), n, C.byref(floats)))
        scratch = torch.empty(floats.value, dtype=torch.float32, device=self.device)
        check(lib.llvq_dn_delta_rows(C.byref(desc), y.data_ptr(), v, ba.data_ptr(), y.data_ptr() + c.channels * y.element_size(), v, scratch.data_ptr(),
                                     act.data_ptr() + L["out"].at[0] * y.element_size(), act.shape[1], start, n, st))

    def hidden(self, tokens, pos, end: int, layers_out: Optional[list] = None):
        """tokens, pos: int64 [L], positions [end - L, end); returns the f32 stream [L, width] behind the last layer.
        `layers_out` collects a copy of the stream behind every layer run."""
        import torch
        cfg, lib, st, check = self.cfg, self.lib, self._cuda_stream(), _lib.check_dense
        n, D = tokens.numel(), cfg.width
        start = end - n
        if n > self.prefill_chunk or start < 0 or end > self.capacity:
            raise ValueError(f"a portion of {n} tokens at position {start} (at most {self.prefill_chunk}, capacity {self.capacity})")
        new = lambda *shape: torch.empty(*shape, dtype=self.dtype, device=self.device)
        ptr = lambda t: t.data_ptr() if t is not None else None
        x = torch.empty(n, D, dtype=torch.float32, device=self.device)
        check(lib.llvq_dn_embed_rows(self.dt, self.embed.ptr(), self.embed.ld, cfg.vocab, tokens.data_ptr(), n, D, 1.0, x.data_ptr(), None, st))
        y = routed = places = None  # what the stream takes up before the next norms
        top, routes = 1, {}

        def add_norms(w1=None, h1=None, w2=None, h2=None):
            check(lib.llvq_dn_add_norms_rows(self.dt, x.data_ptr(), ptr(y), ptr(routed), ptr(places), top, ptr(w1), ptr(h1), ptr(w2), ptr(h2), self.eps,
                                             n, D, st))

        for i, s, desc in zip(cfg.runs, self.states, self._mix):
            L, lc = self.layers[i], cfg.layers[i]
            mlp, out = lc.mlp, L["out"]
            h1, h2 = new(n, D), new(n, D) if mlp is not None else None
            add_norms(L["norm1"], h1, L.get("norm2"), h2)
            act = (torch.zeros if out.padded else torch.empty)(n, out.ld, dtype=self.dtype, device=self.device)
            if isinstance(lc.mixer, ParallelConfig):
                self._parallel_rows(h1, L, lc.mixer, s, desc, act, start, end, st)
            else:
                self._delta_rows(h1, L, lc.mixer, desc, act, start, end, st)
            routed = places = None
            gated = lambda gu, dst, ld, ff, scale: check(lib.llvq_dn_gated_rows(self.dt, gu.data_ptr(), None, dst, ld, gu.shape[0], ff, math.inf, 1.0, 0.0,
                                                                                scale, st))
            if mlp is not None and mlp.experts:
                if i not in routes:
                    routes[i] = _Route(lib, L["table"], mlp.experts, tokens, st)
                route, ff = routes[i], L["experts_down"].shape[2]
                gu = self._grouped(h2.index_select(0, route.source), L["experts_up"][:, :, :D], route)
                e = new(gu.shape[0], ff)
                gated(gu, e.data_ptr(), ff, ff, 1.0 / mlp.top)
                routed, places, top = self._grouped(e, L["experts_down"], route), route.places, mlp.top
            elif mlp is not None:
                gu = self._mm(h2, L["gate_up"].rows(0))
                if L["down"] is None:
                    gated(gu, act.data_ptr() + out.at[-1] * act.element_size(), out.ld, mlp.ff, 1.0)
                else:
                    e = new(n, mlp.ff)
                    gated(gu, e.data_ptr(), mlp.ff, mlp.ff, 1.0)
                    routed, places, top = self._mm(e, L["down"].rows(0)), torch.arange(n, dtype=torch.int32, device=self.device), 1
            y = self._mm(act, out.rows(0))
            if layers_out is not None:
                add_norms()
                y = routed = places = None
                layers_out.append(x.clone())
        if y is not None:
            add_norms()
        return x


@register("Dozusun", "folder", ("bfloat16", "float32"))
def _load_hybrid(config, weights, dtype, capacity, device, **options):
    import torch
    if not torch.cuda.is_available():
        raise RuntimeError("a CUDA device is needed: the library has no CPU path")
    torch.cuda.set_device(device)
    return HybridLM(HybridConfig.parse(config), weights.tensor, dtype, capacity, torch.device("cuda", device), **options)
