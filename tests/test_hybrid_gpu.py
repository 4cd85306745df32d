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
        assert rel(xg, base + sum(down[int(k)].double() @ e[j].double() for j, k in enumerate(table[tok]))) < 3e-6, tok
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
