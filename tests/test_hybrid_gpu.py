"""Hybrid model on the GPU against the plain CPU implementation (oracle/hybrid_lm.py): every mechanism alone, then the
model: prompts, token-by-token decoding, portions, states and slots used again, window edges, greedy generation."""
import copy
import ctypes as C
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import hybrid_cases as cases
from conftest import ROOT
from dense_util import DTYPES, TYPES, P, dn, gen, lib, no_time_out, ok, rel, rnd, run, stream, tokens_of, worst_row
from oracle import hybrid_lm as plain

pytestmark = pytest.mark.gpu

TOL = {"float32": 3e-5, "bfloat16": 4e-2}   # relative l2 of logits against the float64 statement


def build(cfg, seed, dtype, capacity, chunk=2048, weights=None):
    from llvq_b200.hybrid import HybridConfig, HybridLM
    w = weights if weights is not None else cases.random_model(cfg, seed)
    return HybridLM(HybridConfig.parse(cfg), lambda n: w[n], dtype, capacity, torch.device("cuda"), prefill_chunk=chunk), w


# ---- projections over two row sets and routed stacks --------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n,k,n2,top,experts,ff", [(5, 7, 6, 1, 2, 3), (33, 90, 40, 2, 5, 21), (640, 264, 1000, 3, 4, 64), (130, 1536, 4, 20, 24, 5), (2, 2056, 600, 8, 9, 130)])
def test_second_rows_share_the_normed_stream(dtype, n, k, n2, top, experts, ff):
    from llvq_b200.dense import DenseMatrix
    _lib, L = lib()
    T = TYPES[dtype]
    w, w2, x, nw, nw2, bias = rnd(1, n, k), rnd(2, n2, k), rnd(3, k), 1 + 0.3 * rnd(4, k), 1 + 0.3 * rnd(5, k), rnd(6, n)
    m, m2 = DenseMatrix([w], T, "cuda"), DenseMatrix([w2], T, "cuda")
    xg, ng, ng2, bg = x.cuda(), nw.cuda(), nw2.cuda(), bias.cuda()
    y = torch.full((n,), 9.0, device="cuda")
    h1, h2 = (plain.rms_norm(x.double(), f.double(), 1e-3) for f in (nw, nw2))
    tol = 3e-6

    def go(y2, **kw):
        d = _lib.DenseGemv(dtype=dn(dtype), prologue=_lib.DN_NORM, n_out=n, k=k, ldw=m.ld, w=m.ptr(), y=P(y), x=P(xg), alpha=1.0, eps=1e-3,
                           norm_w=P(ng), bias=P(bg), norm_w2=P(ng2), y2=P(y2), limit=float("inf"), gain=1.0, **kw)
        ok(L.llvq_dn_gemv(C.byref(d), stream()))
        assert rel(y, w.double() @ h1 + bias.double()) < tol
        y.fill_(9.0)
        return y2

    got = go(torch.full((n2,), 9.0, device="cuda"), rows2=n2, w2=m2.ptr())
    assert rel(got, w2.double() @ h2) < tol
    s = (w2.double() @ h2).reshape(-1, 2)
    got = go(torch.full((n2 // 2,), 9.0, device="cuda"), rows2=n2, w2=m2.ptr(), glu2=1, glu_scale=0.25)
    assert rel(got, 0.25 * plain.silu(s[:, 0]) * s[:, 1]) < 1e-5
    # a stack: the token's table row names the matrices, in its order; foreign ids read row 0
    stack = rnd(7, experts, 2 * ff, k)
    sm = DenseMatrix([stack.flatten(0, 1)], T, "cuda")
    table = torch.stack([torch.randperm(experts, generator=gen(r))[:top] for r in range(4)]).int()
    tg = table.cuda()
    for tok in (2, 0, 3, 4, -1):
        t = torch.tensor([tok], device="cuda")
        got = go(torch.full((top * ff,), 9.0, device="cuda"), rows2=top * 2 * ff, w2=sm.ptr(), glu2=1, route=P(tg), route_rows=4, top=top, matrices=experts,
                 token=P(t))
        s = torch.cat([stack[int(e)].double() @ h2 for e in table[tok if 0 <= tok < 4 else 0]]).reshape(-1, 2)
        assert rel(got, plain.silu(s[:, 0]) * s[:, 1]) < 1e-5, tok
    # the stream starts at the token's embedding
    emb = rnd(8, 4, k)
    em, t, t_out = DenseMatrix([emb], T, "cuda"), torch.tensor([1], device="cuda"), torch.zeros(k, device="cuda")
    y2 = torch.full((n2,), 9.0, device="cuda")
    d = _lib.DenseGemv(dtype=dn(dtype), prologue=_lib.DN_NORM, n_out=n, k=k, ldw=m.ld, w=m.ptr(), y=P(y), alpha=1.0, eps=1e-3, norm_w=P(ng), norm_w2=P(ng2),
                       y2=P(y2), rows2=n2, w2=m2.ptr(), table=em.ptr(), ld_table=em.ld, table_rows=4, token=P(t), scale=1.0, t_out=P(t_out))
    ok(L.llvq_dn_gemv(C.byref(d), stream()))
    assert torch.equal(t_out.cpu(), emb[1])
    assert rel(y, w.double() @ plain.rms_norm(emb[1].double(), nw.double(), 1e-3)) < tol
    assert rel(y2, w2.double() @ plain.rms_norm(emb[1].double(), nw2.double(), 1e-3)) < tol
    no_time_out()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n,cols,top,experts,ff", [(5, [7, 3], 1, 2, 5), (90, [54, 42], 3, 5, 21), (256, [4096, 640], 2, 16, 768), (100, [30], 8, 9, 8), (64, [2048, 2048], 1, 3, 5000),
                                                   (40, [9000], 5, 6, 1000), (70, [15000, 2000], 2, 3, 9000)])
def test_output_projection_adds_routed_columns_to_the_stream(dtype, n, cols, top, experts, ff):
    from llvq_b200.cache import whole_vectors
    from llvq_b200.dense import ColumnMatrix
    _lib, L = lib()
    T = TYPES[dtype]
    parts = [rnd(11 + i, n, c) for i, c in enumerate(cols)]
    m, ffp = ColumnMatrix(parts, T, "cuda"), whole_vectors(ff, T)
    down = rnd(20, experts, n, ff)
    dg = torch.zeros(experts, n, ffp, dtype=T, device="cuda")
    dg[..., :ff].copy_(down)
    act, acts = torch.zeros(m.ld + top * ffp, device="cuda"), [rnd(30 + i, c) for i, c in enumerate(cols)]
    for lo, a in zip(m.at, acts):
        act[lo:lo + len(a)] = a.cuda()
    e = rnd(40, top, ff)
    for j in range(top):
        act[m.ld + j * ffp:m.ld + j * ffp + ff] = e[j].cuda()
    x = rnd(41, n)
    xg = x.cuda()
    base = x.double() + sum(p.double() @ a.double() for p, a in zip(parts, acts))
    kw = dict(dtype=dn(dtype), prologue=_lib.DN_PLAIN, n_out=n, k=m.k, ldw=m.ld, w=m.ptr(), x=P(act), eps=1.0)
    d = _lib.DenseGemv(y=P(xg), residual=P(xg), **kw)
    ok(L.llvq_dn_gemv(C.byref(d), stream()))
    assert rel(xg, base) < 3e-6
    table = torch.stack([torch.randperm(experts, generator=gen(r))[:top] for r in range(3)]).int()
    tg = table.cuda()
    for tok in (0, 2):
        xg.copy_(x)
        t = torch.tensor([tok], device="cuda")
        d = _lib.DenseGemv(y=P(xg), residual=P(xg), w_r=P(dg), k_r=ffp, ld_r=ffp, route=P(tg), route_rows=3, top=top, matrices=experts, token=P(t), **kw)
        ok(L.llvq_dn_gemv(C.byref(d), stream()))
        routed = sum(down[int(k)].double() @ e[j].double() for j, k in enumerate(table[tok]))
        assert rel(xg, base + routed) < 3e-6, tok
        xg.copy_(x)  # the routed columns alone
        d = _lib.DenseGemv(dtype=dn(dtype), prologue=_lib.DN_PLAIN, n_out=n, x=act[m.ld:].data_ptr(), y=P(xg), residual=P(xg), eps=1.0, w_r=P(dg), k_r=ffp, ld_r=ffp,
                           route=P(tg), route_rows=3, top=top, matrices=experts, token=P(t))
        ok(L.llvq_dn_gemv(C.byref(d), stream()))
        assert rel(xg, x.double() + routed) < 3e-6, tok
    no_time_out()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n", [5, 90, 256, 4100])
def test_row_kernels(dtype, n):
    _, L = lib()
    T, rows = TYPES[dtype], 7
    tol = 1e-6 if dtype == "float32" else 3e-3
    x, y, w1, w2, e = rnd(21, rows, n), rnd(22, rows, n), 1 + 0.3 * rnd(23, n), 1 + 0.3 * rnd(24, n), rnd(25, 2 * rows, n)
    places = torch.randperm(2 * rows, generator=gen(1)).int()
    xg, yg, eg, pg, w1g, w2g = x.cuda(), y.to(T).cuda(), e.to(T).cuda(), places.cuda(), w1.cuda(), w2.cuda()
    h1, h2 = torch.zeros(rows, n, dtype=T, device="cuda"), torch.zeros(rows, n, dtype=T, device="cuda")

    def go(y, e, top, w1, h1, w2, h2):
        ok(L.llvq_dn_add_norms_rows(dn(dtype), P(xg), P(y), P(e), P(pg) if e is not None else None, top, P(w1), P(h1), P(w2), P(h2), 1e-2, rows, n, stream()))
    want = x.double()
    go(None, None, 0, w1g, h1, None, None)
    assert rel(h1, plain.rms_norm(want, w1.double(), 1e-2)) < tol and torch.equal(xg.cpu(), x)
    want = want + y.double()
    go(yg, None, 0, w1g, h1, w2g, h2)
    assert rel(xg, want) < 1e-6 and rel(h1, plain.rms_norm(want, w1.double(), 1e-2)) < tol and rel(h2, plain.rms_norm(want, w2.double(), 1e-2)) < tol
    want = want + y.double() + e.double()[places.long().reshape(rows, 2)].sum(1)
    go(yg, eg, 2, None, None, None, None)
    assert rel(xg, want) < 1e-6
    gu = 2 * rnd(26, rows, 2 * n)
    gug, act = gu.to(T).cuda(), torch.full((rows, n + 8), 7.0, dtype=T, device="cuda")
    ok(L.llvq_dn_gated_rows(dn(dtype), P(gug), None, P(act), n + 8, rows, n, float("inf"), 1.0, 0.0, 0.5, stream()))
    assert rel(act[:, :n], 0.5 * plain.silu(gu.double()[:, 0::2]) * gu.double()[:, 1::2]) < tol and bool((act[:, n:] == 7.0).all())
    ok(L.llvq_dn_gate_rows(dn(dtype), P(yg), n, P(gug), 2 * n, P(act), n + 8, rows, n, 1.5, stream()))
    assert rel(act[:, :n], 1.5 * y.double() * torch.sigmoid(gu.double()[:, :n])) < tol and bool((act[:, n:] == 7.0).all())


@pytest.mark.parametrize("vocab,experts,top,n", [(3, 4, 2, 6), (50, 1, 1, 33), (200, 70, 5, 700), (90, 256, 8, 2048), (7, 9, 9, 31)])
def test_route_sorts_rows_by_expert_and_finds_them_again(vocab, experts, top, n):
    from llvq_b200.hybrid import _Route
    _, L = lib()
    table = torch.stack([torch.randperm(experts, generator=gen(r))[:top] for r in range(vocab)]).int()
    toks = torch.randint(0, vocab, (n,), generator=gen(1))
    toks[n // 2] = vocab + 5                         # an id outside the table reads its first row
    r = _Route(L, table.cuda(), experts, toks.cuda(), stream())
    named = table[torch.where(toks < vocab, toks, 0)]
    source, lo = r.source.cpu().long(), 0
    for e, hi in enumerate(r.host_ends()):
        assert source[lo:hi].tolist() == (named == e).any(1).nonzero()[:, 0].tolist()
        lo = hi
    assert lo == n * top
    places = r.places.cpu().long().reshape(n, top)
    assert torch.equal(source[places], torch.arange(n)[:, None].expand(n, top))
    expert_of = torch.searchsorted(torch.tensor(r.host_ends()), places, right=True)
    assert torch.equal(expert_of, named.long())


# ---- windowed grouped-query attention ------------------------------------------------
class Attention:
    """One layer's operands: raw queries, keys, values and output gates of n positions, and the descriptor."""

    def __init__(self, dtype, heads, kv_heads, dim, vdim, n, window, slots, seed=0, splits=3, scale=None, chunk=1):
        from llvq_b200.cache import KvRing
        _lib, _ = lib()
        self.dtype, T = dtype, TYPES[dtype]
        self.n, self.H, self.G, self.dim, self.vdim, self.window = n, heads, kv_heads, dim, vdim, window
        self.scale = dim ** -0.5 if scale is None else scale
        self.q, self.k = rnd(seed + 31, n, heads, dim), rnd(seed + 32, n, kv_heads, dim)
        self.v, self.gate = rnd(seed + 33, n, kv_heads, vdim), rnd(seed + 34, n, heads, vdim)
        self.qn, self.kn = 1 + 0.3 * rnd(seed + 35, dim), 1 + 0.3 * rnd(seed + 36, dim)
        self.qn_g, self.kn_g = self.qn.cuda(), self.kn.cuda()
        self.ring = KvRing(slots, slots, 1, kv_heads, dim, vdim, T, "cuda")
        self.part = torch.zeros(heads * splits * (vdim + 2), device="cuda")
        self.arrived = torch.zeros(kv_heads * -(-heads // kv_heads // 4), dtype=torch.int32, device="cuda")
        self.d = _lib.DenseGqa(dtype=dn(dtype), heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, slots=slots, ld=self.ring.ld, kd=self.ring.kd, vd=self.ring.vd,
                               window=window, splits=splits, scale=self.scale, eps=1e-4, out_scale=0.7, ring=P(self.ring.rows), q_norm=P(self.qn_g),
                               k_norm=P(self.kn_g), part=P(self.part), arrived=P(self.arrived))

    def want(self, gated=True):
        q, k = plain.rms_norm(self.q.double(), self.qn.double(), 1e-4), plain.rms_norm(self.k.double(), self.kn.double(), 1e-4)
        y = plain.grouped_attention(q, k, self.v.double(), self.scale, plain.window_mask(self.n, self.window))
        return 0.7 * y * torch.sigmoid(self.gate.double()) if gated else y

    def store(self, lo, hi):
        """Rows of a portion: the cache rows and the normed queries."""
        _, L = lib()
        T = TYPES[self.dtype]
        y = torch.cat([t[lo:hi].flatten(1) for t in (self.q, self.k, self.v)], dim=1).to(T).cuda()
        qn = torch.zeros(hi - lo, self.H * self.dim, dtype=T, device="cuda")
        at = [0, self.H * self.dim, (self.H + self.G) * self.dim]
        ok(L.llvq_dn_gqa_rows(C.byref(self.d), *(y.data_ptr() + a * y.element_size() for a in at), y.shape[1], P(qn), lo, hi - lo, stream()))
        return qn

    def decode(self, p):
        _, L = lib()
        q, k, v, g = (t[p].cuda().contiguous() for t in (self.q, self.k, self.v, self.gate))
        out, pos = torch.full((self.H, self.vdim), 7.0, device="cuda"), torch.tensor([p], device="cuda")
        self.d.q, self.d.k, self.d.v, self.d.gate, self.d.out = P(q), P(k), P(v), P(g), P(out)
        ok(L.llvq_dn_mixer_token(C.byref(self.d), None, P(pos), stream()))
        return out.cpu()

    def prefill(self, lo, hi, kernel=0):
        """Queries lo .. hi - 1; earlier rows are in the ring. kernel 1: the generic one, 2: not the transposed one."""
        _, L = lib()
        qn = self.store(lo, hi)
        key0 = max(0, lo - self.window + 1)
        rows = self.ring.read(key0, hi)
        vt = self.ring.values_transposed(rows) if kernel == 0 and L.llvq_dn_gqa_prefill_transposes(C.byref(self.d), hi - lo) else None
        self.transposed = vt is not None
        out = torch.full((hi - lo, self.H, self.vdim), 7.0, dtype=TYPES[self.dtype], device="cuda")
        ok(L.llvq_dn_gqa_prefill(C.byref(self.d), P(qn), P(rows), P(vt), vt.shape[1] if vt is not None else 0, hi - lo, hi - key0, lo, key0, P(out),
                                 1 if kernel == 1 else 0, stream()))
        return out.float().cpu()


HEADS = [(4, 4, 24, 40), (6, 2, 13, 9), (5, 1, 17, 33), (8, 2, 64, 48), (12, 1, 128, 128), (2, 1, 200, 264), (1, 1, 8, 8), (3, 3, 3, 2), (16, 8, 32, 184)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", HEADS, ids=str)
def test_prompt_attention(dtype, shape):
    tol = 3e-6 if dtype == "float32" else 1.2e-2
    for window in (1, 45, 64, 1000):
        a = Attention(dtype, *shape, 300, window, 300, scale=1.5 * shape[2] ** -0.5)
        want = a.want(gated=False)
        for lo, hi in ((0, 300), (0, 1), (0, 2), (37, 140), (127, 129), (299, 300), (64, 256)):
            if lo:
                a.store(0, lo)
            for kernel in (0, 1, 2) if dtype == "bfloat16" and lo == 37 else (0,):
                got = a.prefill(lo, hi, kernel)
                assert rel(got, want[lo:hi]) < tol and worst_row(got, want[lo:hi]) < 4 * tol, (window, lo, hi, kernel)
    a.prefill(0, 300)
    assert a.transposed == (dtype == "bfloat16" and not (shape[2] | shape[3]) & 7 and shape[3] <= 192)
    no_time_out()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", HEADS, ids=str)
def test_token_attention_over_the_ring(dtype, shape):
    tol = 3e-6 if dtype == "float32" else 1.5e-2  # cached keys and values are rounded once
    for window, slots, splits in ((1, 40, 1), (33, 40, 2), (64, 64, 3), (65, 70, 1), (150, 160, 3), (400, 400, 7)):
        a = Attention(dtype, *shape, 260, window, slots, splits=splits, seed=window, scale=1.5 * shape[2] ** -0.5)
        want, at = a.want(), 0
        for p in (0, 1, 2, 31, 63, 64, 65, 100, 149, 150, 159, 160, 161, 200, 259):
            while at < p:
                hi = min(p, at + slots)
                a.store(at, hi)
                at = hi
            held = a.ring.rows.clone()
            first = a.decode(p)
            assert (first - want[p]).norm() < tol * want.norm() / 260 ** 0.5, (window, slots, p)
            assert torch.equal(a.decode(p), first)           # again at the same position
            once = a.ring.rows.clone()
            a.ring.rows.copy_(held)
            a.store(p, p + 1)                                  # the row a portion stores
            assert rel(a.ring.rows, once) < (1e-6 if dtype == "float32" else 2e-3)
            at = p + 1
        assert int(a.arrived.abs().sum()) == 0


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_query_that_looks_for_one_key_finds_it_just_inside_the_window_only(dtype):
    """One key stands out for one query by tens of score units: just inside the window it takes all the weight, just
    outside it leaves no trace, whatever tile, split or portion its place falls into."""
    n, window = 330, 130
    tol = 1e-5 if dtype == "float32" else 2.5e-2  # scores of up to 40 from keys and queries of 8 bits
    for p in (129, 130, 131, 192, 255, 256, 329):
        for gap in (window - 1, window, 0, 1, 63, 64):
            if p - gap < 0:
                continue
            a = Attention(dtype, 4, 2, 40, 24, n, window, window + 70, seed=7, splits=4, scale=1.0)
            j = p - gap
            a.q[p], a.k[j] = a.k[j].repeat_interleave(2, 0), a.k[j]
            a.qn, a.kn = torch.ones(40), torch.ones(40)
            a.qn_g.fill_(1.0), a.kn_g.fill_(1.0)
            want = a.want(gated=False)
            alone = a.v[j].double().repeat_interleave(2, 0)
            assert (rel(want[p], alone) < 1e-3) == (gap < window)
            for lo in (max(0, p - 60), max(0, p - 5), p):
                a.store(max(0, lo - window - 2), lo) if lo else None
                assert rel(a.prefill(lo, min(n, p + 9))[p - lo], want[p]) < tol, (p, gap, lo)
            a.store(max(0, p - window - 2), p)
            assert rel(a.decode(p), a.want()[p]) < tol, (p, gap)


# ---- convolutions and the gated linear recurrence --------------------------------------
PORTIONS = ([200], [2], [1, 2, 3, 70, 1, 5], [64, 65, 63, 8], [33, 1])


def portions(n, sizes):
    at, k = 0, 0
    while at < n:
        m = min(sizes[min(k, len(sizes) - 1)], n - at)
        yield at, at + m
        at, k = at + m, k + 1


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("channels,taps", [(1, 1), (37, 2), (300, 4), (64, 5), (20, 9)])
def test_convolution_carries_its_inputs_over_portions(dtype, channels, taps):
    _, L = lib()
    T, n, ld = TYPES[dtype], 200, channels + 3
    x, w, b, xb = rnd(1, n, channels), rnd(2, channels, taps), rnd(3, channels), rnd(4, channels)
    want = plain.causal_conv(x.double() + xb.double(), w.double()) + b.double()
    buf = torch.full((n, ld), 50.0, dtype=T, device="cuda")
    buf[:, :channels] = x.cuda()
    wg, bg, xbg = w.cuda(), b.cuda(), xb.cuda()
    ring = torch.full((taps, channels), float("nan"), device="cuda")  # nothing ahead of the first token is read
    for sizes in PORTIONS:
        out = torch.zeros(n, channels, dtype=T, device="cuda")
        for lo, hi in portions(n, sizes):
            src = buf[lo:].data_ptr()
            ok(L.llvq_dn_conv_rows(dn(dtype), src, ld, P(xbg), P(wg), P(bg), P(ring), out[lo:].data_ptr(), channels, taps, lo, hi - lo, stream()))
            ok(L.llvq_dn_conv_keep(dn(dtype), src, ld, P(xbg), P(ring), channels, taps, lo, hi - lo, stream()))
        assert rel(out, want) < (1e-6 if dtype == "float32" else 3e-3), sizes


class Recurrence:
    """One recurrent block's operands over n tokens, and the descriptor."""

    def __init__(self, dtype, blocks, size, taps, n, seed=0, lam=-4.0):
        from llvq_b200.cache import ConvInputs, RecurrentState, whole_vectors
        _lib, _ = lib()
        T = TYPES[dtype]
        self.dtype, self.n, self.width, self.blocks, self.size = dtype, n, blocks * size, blocks, size
        W = self.width
        self.x, self.y = rnd(seed + 1, n, W), rnd(seed + 2, n, W)
        self.conv_w, self.conv_b = rnd(seed + 3, W, taps), 0.3 * rnd(seed + 4, W)
        self.ra, self.ri = ((rnd(seed + k, blocks, size, size) / size ** 0.5).bfloat16().float() for k in (5, 6))
        self.rab, self.rib, self.lam = rnd(seed + 7, blocks, size), rnd(seed + 8, blocks, size), lam + 1.5 * rnd(seed + 9, W)
        self.g = torch.zeros(blocks, 2 * size, whole_vectors(size, T), dtype=T, device="cuda")
        self.g[:, :size, :size], self.g[:, size:, :size] = self.ra.cuda(), self.ri.cuda()
        self.t = dict(conv_w=self.conv_w.cuda(), conv_b=self.conv_b.cuda(), b=torch.cat([self.rab, self.rib], 1).contiguous().cuda(),
                      lam=plain.softplus(self.lam.double()).float().cuda(), w=self.g)
        self.conv, self.state = ConvInputs(taps, W, "cuda"), RecurrentState(W, device="cuda")
        self.conv.rows.fill_(float("nan")), self.state.halves.fill_(float("nan"))  # nothing is read ahead of the first token
        self.d = _lib.DenseLru(dtype=dn(dtype), blocks=blocks, n=size, taps=taps, ldw=self.g.shape[2], out_scale=1.3, conv=P(self.conv.rows),
                               state=P(self.state.halves), **{k: P(v) for k, v in self.t.items()})

    def want(self, rounded=False):
        u = plain.causal_conv(self.x.double(), self.conv_w.double()) + self.conv_b.double()
        u = u.bfloat16().double() if rounded else u
        r, i = (torch.sigmoid(plain.block_diagonal(u, m.double(), b.double())) for m, b in ((self.ra, self.rab), (self.ri, self.rib)))
        return plain.gated_recurrence(u, r, i, self.lam.double()) * plain.gelu_tanh(self.y.double()) * 1.3

    def token(self, p):
        _, L = lib()
        x, y, out, pos = self.x[p].cuda(), self.y[p].cuda(), torch.zeros(self.width, device="cuda"), torch.tensor([p], device="cuda")
        self.d.x, self.d.y, self.d.out = P(x), P(y), P(out)
        ok(L.llvq_dn_mixer_token(None, C.byref(self.d), P(pos), stream()))
        return out.cpu()

    def rows(self, lo, hi):
        _, L = lib()
        T, n, W = TYPES[self.dtype], hi - lo, self.width
        x, y = self.x[lo:hi].to(T).cuda(), self.y[lo:hi].to(T).cuda()
        u, out = torch.zeros(n, W, dtype=T, device="cuda"), torch.zeros(n, W, dtype=T, device="cuda")
        zero = torch.zeros(W, device="cuda")
        ok(L.llvq_dn_conv_rows(self.d.dtype, P(x), W, None, self.d.conv_w, self.d.conv_b, self.d.conv, P(u), W, self.d.taps, lo, n, stream()))
        ok(L.llvq_dn_conv_keep(self.d.dtype, P(x), W, None, self.d.conv, W, self.d.taps, lo, n, stream()))
        z = torch.einsum("tbi,boi->bto", u.view(n, self.blocks, self.size).double(), self.g[..., :self.size].double()).float().contiguous()
        ok(L.llvq_dn_lru_rows(C.byref(self.d), P(u), P(z), P(y), W, P(zero), P(out), W, lo, n, stream()))
        return out.float().cpu()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("blocks,size,taps", [(1, 1, 1), (3, 14, 3), (5, 7, 2), (4, 80, 4), (2, 320, 4), (1, 700, 5)])
def test_linear_recurrence_by_token_and_by_portion(dtype, blocks, size, taps):
    n = 200
    a = Recurrence(dtype, blocks, size, taps, n)
    want, rounded = a.want(), a.want(rounded=dtype == "bfloat16")
    got = torch.stack([a.token(p) for p in range(n)])
    assert rel(got, want) < 3e-6 and worst_row(got, want) < 1e-4
    for sizes in PORTIONS:
        got = torch.cat([a.rows(lo, hi) for lo, hi in portions(n, sizes)])
        assert rel(got, rounded) < (3e-6 if dtype == "float32" else 4e-3), sizes
    # portions and tokens in turn, on the same state; a token run again at its position changes nothing
    got, at = [], 0
    for m in (70, 1, 1, 2, 1, 65, 60):
        if m == 1:
            first = a.token(at)
            assert torch.equal(a.token(at), first)
            got.append(first[None])
        else:
            got.append(a.rows(at, at + m))
        at += m
    assert at == n and rel(torch.cat(got), want) < (3e-6 if dtype == "float32" else 1e-2)


def test_a_state_that_hardly_decays_is_carried_exactly():
    """Thousands of tokens with decays of 1 - 1e-5 and below: an error in a decay would add up over all of them."""
    n = 3000
    a = Recurrence("float32", 2, 24, 2, n, seed=3, lam=-13.0)
    want = a.want()
    got = torch.cat([a.rows(lo, hi) for lo, hi in portions(n, [1500, 700, 2, 800])])
    assert rel(got[-100:], want[-100:]) < 5e-6
    for p in range(64):
        a.token(p)
    got = a.rows(64, n)
    assert rel(got[-100:], want[-100:]) < 5e-6


# ---- gated delta rule --------------------------------------------------------------------
class Delta:
    def __init__(self, dtype, heads, kv_heads, dim, vdim, taps, n, seed=0, decay=-2.0):
        from llvq_b200.cache import ConvInputs, RecurrentState
        _lib, _ = lib()
        self.dtype, self.n, self.H, self.G, self.dim, self.vdim = dtype, n, heads, kv_heads, dim, vdim
        self.ch = 2 * kv_heads * dim + heads * vdim
        self.x, self.gate = rnd(seed + 1, n, self.ch), rnd(seed + 2, n, heads, vdim)
        self.b, self.a = rnd(seed + 3, n, heads), rnd(seed + 4, n, heads)
        self.conv_w, self.A_log, self.dt, self.norm = rnd(seed + 5, self.ch, taps), decay + rnd(seed + 6, heads), rnd(seed + 7, heads), 1 + 0.3 * rnd(seed + 8, vdim)
        self.t = dict(conv_w=self.conv_w.cuda(), decay=self.A_log.double().exp().float().cuda(), dt_bias=self.dt.cuda(), norm=self.norm.cuda())
        vp = -(-vdim // 4) * 4
        self.conv, self.state = ConvInputs(taps, self.ch, "cuda"), RecurrentState(heads, dim, vp, device="cuda")
        self.conv.rows.fill_(float("nan"))
        self.state.halves[..., :vdim] = float("nan")  # nothing is read ahead of the first token
        self.o, self.arrived = torch.zeros(heads * vp, device="cuda"), torch.zeros(heads, dtype=torch.int32, device="cuda")
        self.d = _lib.DenseDelta(dtype=dn(dtype), heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, vp=vp, taps=taps, eps=1e-4, conv=P(self.conv.rows),
                                 state=P(self.state.halves), o=P(self.o), arrived=P(self.arrived), **{k: P(v) for k, v in self.t.items()})

    def want(self):
        n, H, G = self.n, self.H, self.G
        c = plain.silu(plain.causal_conv(self.x.double(), self.conv_w.double()))
        q, k, v = c.split([G * self.dim, G * self.dim, H * self.vdim], dim=1)
        q, k = plain.unit_vector(q.reshape(n, G, -1)) * self.dim ** -0.5, plain.unit_vector(k.reshape(n, G, -1))
        q, k = q.repeat_interleave(H // G, 1), k.repeat_interleave(H // G, 1)
        o, _ = plain.delta_rule(q, k, v.reshape(n, H, -1), torch.sigmoid(self.b.double()), plain.delta_decay(self.a.double(), self.A_log.double(), self.dt.double()))
        return plain.gated_head_norm(o, self.norm.double(), self.gate.double(), 1e-4)

    def token(self, p):
        _, L = lib()
        t = [v[p].cuda().contiguous() for v in (self.x, self.gate, self.b, self.a)]
        out, pos = torch.zeros(self.H, self.vdim, device="cuda"), torch.tensor([p], device="cuda")
        self.d.x, self.d.gate, self.d.beta, self.d.alpha, self.d.out = *(P(v) for v in t), P(out)
        ok(L.llvq_dn_delta_token(C.byref(self.d), P(pos), stream()))
        return out.cpu()

    def rows(self, lo, hi):
        _, L = lib()
        T, n, hv = TYPES[self.dtype], hi - lo, self.H * self.vdim
        x, gate = self.x[lo:hi].to(T).cuda(), self.gate[lo:hi].flatten(1).to(T).cuda()
        ba = torch.cat([self.b[lo:hi], self.a[lo:hi]], 1).contiguous().cuda()
        floats = C.c_size_t()
        ok(L.llvq_dn_delta_scratch(C.byref(self.d), n, C.byref(floats)))
        scratch, out = torch.zeros(floats.value, device="cuda"), torch.full((n, hv + 5), 7.0, dtype=T, device="cuda")
        ok(L.llvq_dn_delta_rows(C.byref(self.d), P(x), self.ch, P(ba), P(gate), hv, P(scratch), P(out), hv + 5, lo, n, stream()))
        assert bool((out[:, hv:] == 7.0).all())
        return out[:, :hv].float().cpu().view(n, self.H, self.vdim)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", [(1, 1, 1, 1, 1), (3, 1, 11, 7, 2), (4, 4, 6, 18, 5), (4, 2, 64, 96, 4), (2, 1, 128, 128, 4), (1, 1, 256, 33, 3), (2, 1, 300, 36, 4),
                                   (1, 1, 520, 20, 2), (1, 1, 1000, 9, 2)], ids=str)
def test_delta_rule_by_token_and_by_portion(dtype, shape):
    n = 200
    a = Delta(dtype, *shape, n)
    want = a.want()
    got = torch.stack([a.token(p) for p in range(n)])
    assert rel(got, want) < 1e-5 and worst_row(got, want) < 1e-4
    assert int(a.arrived.abs().sum()) == 0
    for sizes in PORTIONS:
        got = torch.cat([a.rows(lo, hi) for lo, hi in portions(n, sizes)])
        assert rel(got, want) < (1e-5 if dtype == "float32" else 4e-3), sizes
    got, at = [], 0
    for m in (70, 1, 1, 2, 1, 65, 60):
        if m == 1:
            first = a.token(at)
            assert torch.equal(a.token(at), first)
            got.append(first[None])
        else:
            got.append(a.rows(at, at + m))
        at += m
    assert at == n and rel(torch.cat(got), want) < (1e-5 if dtype == "float32" else 4e-3)


@pytest.mark.parametrize("dtype", DTYPES)
def test_delta_state_remembers_a_far_key(dtype):
    """Hardly any decay, and a query that equals one far key: what was written there is read back hundreds of tokens on."""
    n, far = 700, 40
    a = Delta(dtype, 2, 2, 64, 64, 1, n, seed=5, decay=-9.0)
    qk = 2 * 64
    a.conv_w[:], a.t["conv_w"][:] = 1.0, 1.0
    a.b[:] = -4.0                                    # small writes everywhere
    a.b[far] = 8.0
    a.x[-1, :qk] = a.x[far, qk:2 * qk]               # the last query is the far key
    want = a.want()
    b = copy.copy(a)
    b.x = a.x.clone()
    b.x[far, 2 * qk:] = -a.x[far, 2 * qk:]
    assert ((b.want()[-1] - want[-1]).norm() / want[-1].norm()) > 0.3  # the plain statement depends on it
    tol = 1e-4 if dtype == "float32" else 6e-3
    assert rel(a.rows(0, n)[-1], want[-1]) < tol
    got = torch.cat([a.rows(lo, hi) for lo, hi in portions(n - 1, [333, 64, 2, 300])])
    assert rel(a.token(n - 1), want[-1]) < tol and rel(got[far:], want[far:-1]) < 6e-3


# ---- the model ---------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(cases.ALL))
def test_prompts_portions_and_tokens_give_the_plain_logits(dtype, name):
    cfg = cases.ALL[name]
    m, w = build(cfg, 5, dtype, 400)
    toks = tokens_of(cfg, 210, 6)
    layers, want_layers = [], []
    want = plain.forward(cfg, w, toks, layers_out=want_layers)
    m.hidden(torch.tensor(toks, device="cuda"), m.positions[:210], end=210, layers_out=layers)
    assert len(layers) == len(want_layers) == len(m.cfg.runs)
    for i, (a, b) in enumerate(zip(layers, want_layers)):
        assert rel(a, b) < (1e-5 if dtype == "float32" else 4e-2), i
    runs = {"whole": [210], "tokens": [1], "twos": [2], "mixed": [64, 1, 3, 17, 2, 1, 1, 70, 5, 2], "then tokens": [150, 1]}
    for k, sizes in runs.items():
        y = run(m, toks, sizes)
        assert rel(y, want) < TOL[dtype], k
        worst = (y.double() - want).norm(dim=1) / want.norm(dim=1)
        assert worst.max() < 4 * TOL[dtype], (k, int(worst.argmax()))
    assert rel(run(m, toks[:40], [1], use_graph=False), want[:40]) < TOL[dtype]
    no_time_out()


@pytest.mark.parametrize("dtype", DTYPES)
def test_rings_that_wrap_and_states_used_again(dtype):
    """Portions of at most 16 tokens: the rings are a window and 15 positions long and wrap many times; further sequences
    start over in the slots and states the ones before have left. Every pass of a looped layer keeps its own."""
    m, w = build(cases.UNEVEN, 8, dtype, 900, chunk=16)
    assert [s["ring"].slots for s in m.states if "ring" in s] == [34, 22, 34, 22, 16]
    stores = [s["state"].halves.data_ptr() for s in m.states] + [s["conv"].rows.data_ptr() for s in m.states]
    assert len(set(stores)) == 2 * len(m.cfg.runs) and m.cache_bytes() > 0
    for seed, n, sizes in ((1, 300, [7, 16, 2, 1, 1, 40, 3]), (2, 95, [1]), (3, 1, [1]), (4, 140, [140]), (5, 23, [20, 2])):
        toks = tokens_of(cases.UNEVEN, n, seed)
        want = plain.forward(cases.UNEVEN, w, toks)
        y = run(m, toks, sizes)
        assert rel(y, want) < TOL[dtype], (seed, n)
        assert ((y.double() - want).norm(dim=1) / want.norm(dim=1)).max() < 4 * TOL[dtype]


def test_logits_do_not_depend_on_what_ran_before():
    m, w = build(cases.EVEN, 9, "bfloat16", 300, chunk=50)
    toks = tokens_of(cases.EVEN, 120, 1)
    first = run(m, toks, [50, 30, 1])
    run(m, tokens_of(cases.EVEN, 299, 2), [13])
    m.feed(tokens_of(cases.EVEN, 77, 3), [0])  # left without a release: generate takes the states over
    m.generate(tokens_of(cases.EVEN, 5, 4), 9, use_graph=True)
    assert torch.equal(run(m, toks, [50, 30, 1]), first)


@pytest.mark.parametrize("odd", [0, 1])
def test_the_first_replayed_step_does_not_move_the_state_twice(odd):
    """Capturing the step's graph runs it once ahead of the first replay."""
    m, w = build(cases.UNEVEN, 19, "float32", 100)
    toks = tokens_of(cases.UNEVEN, 30 + odd, 2)
    want = plain.forward(cases.UNEVEN, w, toks)
    got = torch.cat([m.feed(toks[:20 + odd], [19 + odd])] + [m.feed([t], [0]) for t in toks[20 + odd:]])
    assert rel(got, want[19 + odd:]) < TOL["float32"]


@pytest.mark.parametrize("name,layer", [("uneven", 1), ("uneven", 2), ("even", 0), ("even", 3)])
def test_every_layers_window_ends_where_it_should(name, layer):
    """One attention layer alone, its neighbours blind: a token reaches exactly window - 1 positions ahead."""
    cfg = copy.deepcopy(cases.ALL[name])
    cfg["layers"], cfg["loop"] = [cfg["layers"][layer]], None
    m_, mlp = cfg["layers"][0]["mixer"], cfg["layers"][0]["mlp"]
    m_["right_scale"] = 0.0
    size = m_["left"]["mask"]["size"]
    m, w = build(cfg, 10, "float32", 300, chunk=96)
    at = 21
    toks = tokens_of(cfg, at + size + 4, 5)
    other = list(toks)
    other[at] = (other[at] + 1) % cfg["vocab"]
    inside, outside = at + size - 1, at + size
    want = (plain.forward(cfg, w, toks) - plain.forward(cfg, w, other)).norm(dim=1)
    assert want[inside] > 1e-6 and want[outside] < 1e-12  # the plain statement has the edge there
    for sizes in ([len(toks)], [at + 1, 2], [30, 1], [1]):
        d = (run(m, toks, sizes) - run(m, other, sizes)).norm(dim=1)
        assert abs(float(d[inside]) - float(want[inside])) < 0.2 * float(want[inside]) + 1e-4, sizes
        assert float(d[outside]) == 0.0 and float(d[at - 1]) == 0.0, sizes


def test_long_decoding_stays_on_the_plain_logits():
    for dtype in DTYPES:
        m, w = build(cases.UNEVEN, 12, dtype, 700, chunk=8)
        toks = tokens_of(cases.UNEVEN, 600, 7)
        want = plain.forward(cases.UNEVEN, w, toks)
        y = run(m, toks, [5, 1])
        assert rel(y[-100:], want[-100:]) < TOL[dtype]
        assert rel(run(m, toks[:64], [1], use_graph=False), want[:64]) < TOL[dtype]


def test_output_projections_apart_where_one_would_be_too_long():
    from llvq_b200.hybrid import HybridLM
    toks = tokens_of(cases.EVEN, 90, 3)
    w = cases.random_model(cases.EVEN, 21)
    want = plain.forward(cases.EVEN, w, toks)
    held = HybridLM.JOINED_SEGMENTS, HybridLM.JOINED_COLUMNS_F32
    try:
        HybridLM.JOINED_SEGMENTS, HybridLM.JOINED_COLUMNS_F32 = 0, 0
        for dtype in DTYPES:
            m, _ = build(cases.EVEN, 21, dtype, 128, weights=w)
            assert m.layers[0]["down"] is not None and m.layers[1]["routed_apart"] and m.layers[3]["routed_apart"]
            for sizes in ([90], [1], [40, 1, 1, 2]):
                assert rel(run(m, toks, sizes), want) < TOL[dtype], sizes
    finally:
        HybridLM.JOINED_SEGMENTS, HybridLM.JOINED_COLUMNS_F32 = held


@pytest.mark.parametrize("name", list(cases.ALL))
def test_greedy_generation_through_the_entry_point(tmp_path, name):
    """The command line and load_model on a folder: the tokens are the plain statement's greedy ones (f32), the graph
    replays the eager tokens, and the bf16 model agrees with its own fed logits."""
    from llvq_b200.registry import load_model
    cfg = cases.ALL[name]
    w = cases.random_model(cfg, 14)
    path = cases.write_folder(tmp_path / name, cfg, w)
    prompt = tokens_of(cfg, 20, 8)
    seq = list(prompt)
    for _ in range(24):
        seq.append(int(plain.forward(cfg, w, seq)[-1].argmax()))
    want = seq[20:]
    assert len(set(want)) > 4
    m = load_model(path, 64, "float32", prefill_chunk=7)
    assert m.generate(prompt, 24) == want and m.generate(prompt, 24, use_graph=True) == want
    assert m.generate(prompt, 1) == want[:1] and m.generate(prompt, 0) == []
    with pytest.raises(ValueError):
        m.generate(prompt, 60)
    b = load_model(path, 64)
    assert b.dtype == torch.bfloat16
    out = b.generate(prompt, 24, use_graph=True)
    assert b.generate(prompt, 24) == out
    fed = [b.feed(prompt, [19])] + [b.feed([t], [0]) for t in out[:-1]]
    assert [int(y[0].argmax()) for y in fed] == out
    if name == "uneven":
        res = subprocess.run([sys.executable, "-m", "llvq_b200", "generate", "--model", path, "--tokens", ",".join(map(str, prompt)), "--max-new", "24",
                              "--dtype", "float32"], cwd=ROOT, capture_output=True, text=True, timeout=300)
        assert res.returncode == 0 and json.loads(res.stdout)["tokens"] == want, res.stderr
        steps = [{"step": 0, "entries": [{"id": "a", "tokens": prompt[:9], "want": [8, 1]}], "end": []},
                 {"step": 1, "entries": [{"id": "a", "tokens": prompt[9:10], "want": [0]}], "end": ["a"]},
                 {"step": 2, "entries": [{"id": "b", "tokens": prompt[:3], "want": [2]}], "end": ["b"]}]
        res = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", path, "--dtype", "float32", "--out", str(tmp_path), "--max-tokens", "32"],
                             input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=300)
        assert res.returncode == 0 and res.stdout.split() == "done 0 done 1 done 2".split(), res.stderr
        full = plain.forward(cfg, w, prompt)
        for step, rows in ((0, [8, 1]), (1, [9]), (2, [2])):
            assert rel(torch.from_numpy(np.fromfile(tmp_path / f"{step}.f32", "<f4").reshape(len(rows), -1)), full[rows]) < TOL["float32"]


def test_phases_leave_the_tokens_alone():
    _lib, L = lib()
    m, _ = build(cases.EVEN, 15, "bfloat16", 96)
    prompt = tokens_of(cases.EVEN, 12, 3)
    want = m.generate(prompt, 30, use_graph=True)
    ph = m.phase_split(reps=2)
    assert set(ph) == set(m.PHASES) | {"sum"} and all(v >= 0 for v in ph.values())
    assert m.generate(prompt, 30, use_graph=True) == want
    try:
        L.llvq_dn_set_overlap(0)
        other, _ = build(cases.EVEN, 15, "bfloat16", 96)
        assert other.generate(prompt, 30, use_graph=True) == want
    finally:
        L.llvq_dn_set_overlap(1)


def test_weights_that_do_not_fit_the_configuration_are_refused():
    w = cases.random_model(cases.UNEVEN, 1)
    for name, shape in (("l0.mix.q", (12, 90)), ("l1.mix.left.q.norm", (12,)), ("embed", (203, 91)), ("l1.mix.right.ra", (3, 14, 13)), ("l0.mlp.e4.up", (20, 90)),
                        ("l3.mix.v.conv", (72, 4)), ("l2.mix.right.o", (90, 34))):
        bad = dict(w)
        bad[name] = torch.zeros(*shape).bfloat16()
        with pytest.raises(ValueError, match="config.json says"):
            build(cases.UNEVEN, 1, "bfloat16", 16, weights=bad)
    bad = dict(w)
    bad["l0.mlp.table"] = w["l0.mlp.table"] + 3
    with pytest.raises(ValueError, match="outside"):
        build(cases.UNEVEN, 1, "bfloat16", 16, weights=bad)
    bad = dict(w)
    del bad["l4.mix.right.lam"]
    with pytest.raises(KeyError):
        build(cases.UNEVEN, 1, "bfloat16", 16, weights=bad)
