"""Latent-attention model on the GPU against the plain CPU implementation (oracle/latent_lm.py): every kernel alone,
then the model: prompts, token-by-token decoding, portions, reused slots, window edges, greedy generation."""
import copy
import ctypes as C

import numpy as np
import pytest
import torch

import latent_cases as cases
from oracle import latent_lm as plain

pytestmark = pytest.mark.gpu

F64 = torch.float64
TOL = {"float32": 3e-5, "bfloat16": 4e-2}   # relative l2 of logits against the float64 statement
TYPES = {"float32": torch.float32, "bfloat16": torch.bfloat16}
DTYPES = list(TYPES)


def gen(seed):
    return torch.Generator().manual_seed(seed)


def rnd(seed, *shape, dtype="bfloat16"):
    """Values every element type holds exactly."""
    return torch.randn(*shape, generator=gen(seed)).to(TYPES[dtype]).float()


def rel(a, b):
    a, b = a.double().cpu(), b.double().cpu()
    return ((a - b).norm() / b.norm().clamp_min(1e-30)).item()


def lib():
    from llvq_b200 import _lib
    return _lib, _lib.load_dense()


def stream():
    return C.c_void_p(torch.cuda.current_stream().cuda_stream)


def P(t):
    return t.data_ptr() if t is not None else None


def padded(w, dtype):
    from llvq_b200.latent import DenseMatrix
    return DenseMatrix([w], TYPES[dtype], "cuda")


def dn(dtype):
    _lib, _ = lib()
    return {"float32": _lib.DN_F32, "bfloat16": _lib.DN_BF16}[dtype]


def build(cfg, seed, dtype, capacity, chunk=2048, weights=None):
    from llvq_b200.latent import LatentConfig, LatentLM
    w = weights if weights is not None else plain.random_model(cfg, seed)
    return LatentLM(LatentConfig.parse(cfg), lambda n: w[n], dtype, capacity, torch.device("cuda"), prefill_chunk=chunk), w


def tokens_of(cfg, n, seed):
    return torch.randint(0, cfg["vocab"], (n,), generator=gen(seed)).tolist()


def run(m, toks, sizes, use_graph=True):
    """Feed a sequence in portions of the given sizes (the last one repeats); logits of every position."""
    out, at, k = [], 0, 0
    while at < len(toks):
        n = min(sizes[min(k, len(sizes) - 1)], len(toks) - at)
        out.append(m.feed(toks[at:at + n], list(range(n)), use_graph=use_graph))
        at, k = at + n, k + 1
    m.release()
    return torch.cat(out).cpu()


# ---- one kernel at a time ----------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n,k", [(1, 1), (5, 7), (33, 40), (203, 90), (640, 264), (130, 530), (70, 1100), (1500, 2056), (1201, 1536), (3, 9000), (150, 17408),
                                 (4, 20488)])
def test_token_projection_and_its_prologues(dtype, n, k):
    _lib, L = lib()
    tol = 2e-6 if dtype == "float32" else 2e-6  # activations stay f32, so bf16 weights lose nothing either
    w, x, delta, bias, nw = rnd(1, n, k), rnd(2, k), rnd(3, k), rnd(4, n), 1 + 0.3 * rnd(5, k)
    m = padded(w, dtype)
    y, a_out = torch.full((n,), 9.0, device="cuda"), torch.zeros(k, device="cuda")
    bg = bias.cuda()
    xg, dg, nwg = x.cuda(), delta.cuda(), nw.cuda()

    def go(**kw):
        d = _lib.DenseGemv(dtype=dn(dtype), n_out=n, k=k, ldw=m.ld, w=m.ptr(), y=P(y), eps=1e-3, **kw)
        _lib.check_dense(L.llvq_dn_gemv(C.byref(d), stream()))
        return y.clone()

    W, X = w.double(), x.double()
    scale = W.norm()

    def close(got, a, b=None):
        want = W @ a + (b.double() if b is not None else 0.0)
        assert ((got.double().cpu() - want).norm() / (scale * a.norm() / k ** 0.5 + want.norm())).item() < tol

    close(go(prologue=_lib.DN_PLAIN, x=P(xg)), X)
    close(go(prologue=_lib.DN_PLAIN, x=P(xg), bias=P(bg)), X, bias)
    t = 1.7 * X + delta.double()
    close(go(prologue=_lib.DN_NORM, x=P(xg), delta=P(dg), alpha=1.7, norm_w=P(nwg), a_out=P(a_out)), plain.plain_norm(t, nw.double(), 1e-3))
    assert rel(a_out, plain.plain_norm(t, nw.double(), 1e-3)) < 1e-6 and torch.equal(xg.cpu(), x)
    close(go(prologue=_lib.DN_NORM, x=P(xg), alpha=1.0, norm_w=P(nwg)), plain.plain_norm(X, nw.double(), 1e-3))
    if n % 2 == 0:  # rows in (gate, up) pairs
        y = torch.full((n // 2,), 9.0, device="cuda")
        s = (W @ plain.plain_norm(t, nw.double(), 1e-3) + bias.double()).reshape(-1, 2)
        gate, up = s[:, 0].clamp(max=2.0), s[:, 1].clamp(-2.0, 2.0)
        pairs = go(prologue=_lib.DN_NORM, x=P(xg), delta=P(dg), alpha=1.7, norm_w=P(nwg), bias=P(bg), glu=1, limit=2.0, gain=1.3, shift=0.5)
        assert rel(pairs, gate * torch.sigmoid(1.3 * gate) * (up + 0.5)) < 1e-5
        y = torch.full((n,), 9.0, device="cuda")
    table = rnd(8, 6, k)
    tm = padded(table, dtype)
    tok = torch.tensor([4], device="cuda")
    emb = dict(prologue=_lib.DN_EMBED, table=tm.ptr(), ld_table=tm.ld, table_rows=6, token=P(tok), scale=0.6, a_out=P(a_out))
    close(go(**emb), 0.6 * table[4].double())
    assert rel(a_out, 0.6 * table[4]) < 1e-6
    tok.fill_(6)  # outside the table: row 0, not foreign memory
    close(go(**emb), 0.6 * table[0].double())
    no_time_out()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n,k", [(3, 12), (500, 90), (5000, 256), (30001, 128)])
def test_head_caps_logits_and_picks_the_lowest_best_row(dtype, n, k):
    _lib, L = lib()
    w, x, nw = rnd(11, n, k), rnd(12, k), 1 + 0.2 * rnd(13, k)
    best = n // 3
    h = plain.plain_norm(x.double(), nw.double(), 1e-5)
    w[best] = (h / h.norm() * 9).bfloat16().float()
    w[n - 1] = w[best]  # a tie
    m = padded(w, dtype)
    y, val, idx = torch.zeros(n, device="cuda"), torch.zeros(1, device="cuda"), torch.zeros(1, dtype=torch.long, device="cuda")
    scratch = torch.zeros(8192, dtype=torch.uint8, device="cuda")
    xg, nwg = x.cuda(), nw.cuda()
    for cap in (0.0, 6.0):
        d = _lib.DenseGemv(dtype=dn(dtype), prologue=_lib.DN_NORM, n_out=n, k=k, ldw=m.ld, w=m.ptr(), y=P(y), x=P(xg), alpha=1.0, norm_w=P(nwg),
                           eps=1e-5, softcap=cap)
        _lib.check_dense(L.llvq_dn_head(C.byref(d), P(scratch), P(val), P(idx), stream()))
        want = plain.softcap(w.double() @ h, cap or None)
        assert rel(y, want) < 2e-6 and int(idx) == best
        assert abs(float(val) - float(want[best])) < 1e-4


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n", [5, 90, 256, 4100])
def test_row_kernels(dtype, n):
    _lib, L = lib()
    T, rows = TYPES[dtype], 7
    tol = 1e-6 if dtype == "float32" else 3e-3  # one rounding to bf16 where the result is bf16
    x, y, w, bias = rnd(21, rows, n), rnd(22, rows, n), 1 + 0.3 * rnd(23, n), rnd(24, n)
    xg, yg, wg, bg = x.cuda(), y.to(T).cuda(), w.cuda(), bias.cuda()
    xt, out = torch.zeros(rows, n, dtype=T, device="cuda"), torch.zeros(rows, n, device="cuda")
    want = plain.plain_norm(2.5 * x.double() + y.double() + bias.double(), w.double(), 1e-2)
    _lib.check_dense(L.llvq_dn_postnorm_rows(dn(dtype), P(xg), P(yg), P(bg), P(wg), 2.5, 1e-2, P(xt), P(out), rows, n, stream()))
    assert rel(out, want) < 1e-6 and rel(xt, want) < tol
    _lib.check_dense(L.llvq_dn_postnorm_rows(dn(dtype), P(xg), None, None, P(wg), 1.0, 1e-2, P(xt), P(xg), rows, n, stream()))  # in place
    assert rel(xg, plain.plain_norm(x.double(), w.double(), 1e-2)) < 1e-6
    table = rnd(25, 11, n)
    tm, ids = padded(table, dtype), torch.tensor([3, 0, 10, 3, 11, -1, 7], device="cuda")
    _lib.check_dense(L.llvq_dn_embed_rows(dn(dtype), tm.ptr(), tm.ld, 11, P(ids), rows, n, 0.3, P(out), P(xt), stream()))
    want = 0.3 * table[torch.tensor([3, 0, 10, 3, 0, 0, 7])].double()
    assert rel(out, want) < 1e-6 and rel(xt, want) < tol
    gu, gb = 2 * rnd(26, rows, 2 * n), rnd(27, 2 * n)  # (gate, up) pairs
    gug, gbg, act = gu.to(T).cuda(), gb.cuda(), torch.zeros(rows, n, dtype=T, device="cuda")
    _lib.check_dense(L.llvq_dn_glu_rows(dn(dtype), P(gug), P(gbg), P(act), rows, n, 1.1, 1.702, 1.0, stream()))
    s = gu.double() + gb.double()
    g, u = s[:, 0::2].clamp(max=1.1), s[:, 1::2].clamp(-1.1, 1.1)
    assert rel(act, g * torch.sigmoid(1.702 * g) * (u + 1)) < tol
    v = 30 * rnd(28, 1000)
    vg = v.cuda()
    _lib.check_dense(L.llvq_dn_softcap(P(vg), 1000, 5.0, stream()))
    assert rel(vg, 5 * torch.tanh(v.double() / 5)) < 1e-6


def no_time_out():
    _lib, L = lib()
    err = C.c_int32(7)
    _lib.check_dense(L.llvq_dn_poll_error(C.byref(err)))
    assert err.value == 0


class Attention:
    """One latent-attention layer's operands: random latents, keys and queries of n positions, and the descriptor."""

    def __init__(self, dtype, heads, dim, rot, vdim, rank, n, window, slots, rot_dims=None, sink=True, seed=0, splits=3, scale=None):
        from llvq_b200.cache import LatentRing
        _lib, _ = lib()
        self.dtype, T = dtype, TYPES[dtype]
        self.n, self.H, self.dim, self.rot, self.vdim, self.rank = n, heads, dim, rot, vdim, rank
        self.window, self.rot_dims = window, rot if rot_dims is None else rot_dims
        self.scale = scale or (dim + rot) ** -0.5
        self.base = 300.0
        self.qn, self.qr = rnd(seed + 31, n, heads, dim), rnd(seed + 32, n, heads, rot)   # before rotation
        self.c = rnd(seed + 33, n, rank)
        self.kr = rnd(seed + 34, n, rot)                                                  # as cached: rotated
        self.uk = (rnd(seed + 35, heads * dim, rank) / rank ** 0.5).bfloat16().float()
        self.uv = (rnd(seed + 36, heads * vdim, rank) / rank ** 0.5).bfloat16().float()
        self.sink = rnd(seed + 37, heads) if sink else None
        half = self.rot_dims // 2
        ang = torch.arange(n, dtype=F64)[:, None] * self.base ** (-2.0 * torch.arange(half, dtype=F64) / self.rot_dims)
        self.cos, self.sin = ang.cos().float().cuda(), ang.sin().float().cuda()
        self.ring = LatentRing(slots, slots, 1, rank, rot, T, "cuda")
        assert self.ring.slots == slots
        self.ukv = padded(torch.cat([self.uk, self.uv]), dtype)
        self.sink_g = self.sink.cuda() if sink else None
        self.qlat = torch.zeros(heads * self.ring.ld, device="cuda")
        self.part = torch.zeros(heads * splits * (rank + 2), device="cuda")
        self.d = _lib.DenseLatent(dtype=dn(dtype), heads=heads, dim=dim, rot_dim=rot, vdim=vdim, kv_rank=rank, ldk=self.ukv.ld, slots=slots,
                                  ld=self.ring.ld, rot_dims=self.rot_dims, window=window, splits=splits, scale=self.scale, eps=1e-4,
                                  ring=P(self.ring.rows), cos_t=P(self.cos), sin_t=P(self.sin), uk=self.ukv.ptr(), uv=self.ukv.ptr(heads * dim),
                                  kv_norm=None, sink=P(self.sink_g), qlat=P(self.qlat), part=P(self.part))

    def store(self, lo, hi):
        for p in range(lo, hi):
            self.ring.rows[p % self.ring.slots, :self.rank + self.rot] = torch.cat([self.c[p], self.kr[p]]).cuda()

    def want(self):
        """[n, H, vdim]: every position's attention over its window."""
        qr = plain.rotate(self.qr.double(), torch.arange(self.n), self.rot_dims, self.base)
        return plain.attend(self.qn.double(), qr, self.c.double(), self.kr.double(), self.uk.double(), self.uv.double(), self.scale,
                            plain.window_mask(self.n, self.window), self.sink.double() if self.sink is not None else None)

    def decode(self, p):
        """The token at p against the ring, which must hold its row and those before it."""
        _lib, L = lib()
        q = torch.cat([self.qn[p], self.qr[p]], dim=-1).reshape(-1).cuda()
        pos, ctx = torch.tensor([p], device="cuda"), torch.zeros(self.H, self.vdim, device="cuda")
        _lib.check_dense(L.llvq_dn_latent_query(C.byref(self.d), P(q), None, P(pos), stream()))
        _lib.check_dense(L.llvq_dn_latent_decode(C.byref(self.d), P(pos), stream()))
        _lib.check_dense(L.llvq_dn_latent_value(C.byref(self.d), P(ctx), stream()))
        return ctx.cpu()

    def prefill(self, lo, hi, kernel=0, key0=None):
        """Queries lo .. hi - 1 over keys key0 (by default the first one any of them sees) .. hi - 1. kernel: 0 = the one
        the library picks, 1 = the generic one, 2 = the one for values along the keys where the library prefers them
        transposed."""
        _lib, L = lib()
        T = TYPES[self.dtype]
        key0 = max(0, lo - self.window + 1) if key0 is None else key0
        q = torch.cat([self.qn[lo:hi], self.qr[lo:hi]], dim=-1).reshape(hi - lo, -1).to(T).cuda().contiguous()
        c = self.c[key0:hi].double()
        kv = torch.cat([c @ self.uk.double().T, c @ self.uv.double().T], dim=1).to(T).cuda().contiguous()
        rows = torch.zeros(hi - key0, self.ring.ld, dtype=T, device="cuda")
        rows[:, self.rank:self.rank + self.rot] = self.kr[key0:hi].to(T).cuda()
        out = torch.full((hi - lo, self.H, self.vdim), 7.0, dtype=T, device="cuda")
        vt, split = None, self.H * self.dim
        if kernel == 0 and L.llvq_dn_latent_prefill_transposes(C.byref(self.d), hi - lo):
            vt = torch.zeros(self.H * self.vdim, -(-kv.shape[0] // 8) * 8, dtype=T, device="cuda")
            vt[:, :kv.shape[0]] = kv[:, split:].t()
            kv = kv[:, :split].contiguous()
        self.transposed = vt is not None
        _lib.check_dense(L.llvq_dn_latent_prefill(C.byref(self.d), P(q), P(kv), kv.shape[1], P(rows) + self.rank * rows.element_size(), self.ring.ld,
                                                  P(vt), vt.shape[1] if vt is not None else 0, hi - lo, hi - key0, lo, key0, P(out), 1 if kernel == 1 else 0, stream()))
        return out.float().cpu()


HEADS = [  # heads, dim, rot, vdim, kv_rank, rot_dims
    (3, 24, 8, 40, 56, None), (5, 17, 6, 9, 30, None), (9, 32, 16, 48, 128, None), (2, 128, 64, 128, 512, None), (1, 192, 32, 200, 96, None),
    (1, 700, 40, 300, 64, None), (2, 16, 12, 20, 24, 6), (17, 8, 2, 8, 8, None), (2, 3, 2, 17, 5, None),
    (2, 56, 40, 72, 24, None), (1, 8, 8, 8, 8, None), (3, 40, 8, 184, 32, 4), (1, 120, 56, 192, 16, None)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", HEADS, ids=str)
@pytest.mark.parametrize("window", [1, 45, 64, 1000])
def test_prompt_attention(dtype, shape, window):
    H, dim, rot, vdim, rank, rd = shape
    a = Attention(dtype, H, dim, rot, vdim, rank, 300, window, 300, rot_dims=rd, scale=2.0 * (dim + rot) ** -0.5)
    want = a.want()
    tol = 3e-6 if dtype == "float32" else 1.2e-2
    for lo, hi in ((0, 300), (0, 1), (0, 2), (37, 140), (127, 129), (299, 300), (64, 256)):
        got = a.prefill(lo, hi)
        assert rel(got, want[lo:hi]) < tol, (lo, hi)
        worst = (got.double() - want[lo:hi]).flatten(1).norm(dim=1) / want[lo:hi].flatten(1).norm(dim=1)
        assert worst.max() < 4 * tol, (lo, hi, int(worst.argmax()))
    if dtype == "bfloat16":
        for kernel in (1, 2):
            assert rel(a.prefill(37, 140, kernel=kernel), want[37:140]) < tol
    assert rel(a.prefill(200, 290, key0=0), want[200:290]) < tol  # keys ahead of every window are ignored
    no_time_out()


@pytest.mark.parametrize("window", [1, 64, 129, 700, 5000])
def test_prompt_attention_of_long_portions_on_the_tensor_cores(window):
    """Several query tiles of 128 and pairs of them, ragged ends, scores that grow along the keys (the running maximum is
    raised again and again, and by more than the rescaling threshold)."""
    a = Attention("bfloat16", 2, 128, 64, 128, 64, 900, window, 900, seed=2, scale=4.0 * 192 ** -0.5)
    for grow in (False, True):
        if grow:
            u = torch.randn(64, generator=gen(9))
            a.c = (a.c * 0.05 + torch.linspace(0, 3, 900)[:, None] * u / u.norm() * 2).bfloat16().float()
            k = (u.double() @ a.uk.double().T).reshape(1, 2, 128)
            a.qn = (a.qn * 0.1 + (k / k.norm(dim=-1, keepdim=True)).float() * 6).bfloat16().float()
        want = a.want()
        for lo, hi in ((0, 900), (0, 129), (100, 228), (131, 700), (640, 900), (0, 64)):
            got = a.prefill(lo, hi)
            assert a.transposed
            assert rel(got, want[lo:hi]) < 1.2e-2, (grow, lo, hi)
            worst = (got.double() - want[lo:hi]).flatten(1).norm(dim=1) / want[lo:hi].flatten(1).norm(dim=1)
            assert worst.max() < 4e-2, (grow, lo, hi, int(worst.argmax()))
    no_time_out()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", HEADS, ids=str)
def test_token_attention_over_the_ring(dtype, shape):
    H, dim, rot, vdim, rank, rd = shape
    tol = 3e-6 if dtype == "float32" else 1.2e-2
    for window, slots, splits in ((1, 40, 1), (33, 40, 2), (32, 32, 3), (150, 160, 3), (400, 400, 5)):
        a = Attention(dtype, H, dim, rot, vdim, rank, 220, window, slots, rot_dims=rd, splits=splits, seed=window, scale=2.0 * (dim + rot) ** -0.5)
        want, at = a.want(), 0
        for p in (0, 1, 2, 31, 32, 33, 63, 100, 149, 150, 159, 160, 161, 219):
            a.store(at, p + 1)
            at = p + 1
            assert rel(a.decode(p), want[p]) < tol, (window, slots, p)


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_query_that_looks_for_one_key_finds_it_just_inside_the_window_only(dtype):
    """One latent stands out for one query by tens of score units. Just inside the window it takes all the weight; just
    outside it leaves no trace, whatever tile, split or portion its place falls into."""
    n, window = 330, 130
    for p in (129, 130, 131, 192, 255, 256, 329):
        for gap in (window - 1, window, 0, 1, 63, 64):
            if p - gap < 0:
                continue
            a = Attention(dtype, 3, 24, 8, 40, 56, n, window, window + 3, seed=7, splits=4)
            j = p - gap
            a.c[j] *= 4
            k = (a.c[j].double() @ a.uk.double().T).reshape(3, 24)
            a.qn[p] = (k / k.norm(dim=1, keepdim=True) * 60 / a.scale / k.norm(dim=1, keepdim=True)).bfloat16().float()
            want = a.want()
            alone = (a.c[j].double() @ a.uv.double().T).reshape(3, 40)
            assert (rel(want[p], alone) < 1e-3) == (gap < window)
            tol = 1e-5 if dtype == "float32" else 1.2e-2
            for lo in (0, max(0, p - 5), p):
                assert rel(a.prefill(lo, min(n, p + 9))[p - lo], want[p]) < tol, (p, gap, lo)
            a.store(max(0, p - window - 2), p + 1)
            assert rel(a.decode(p), want[p]) < tol, (p, gap)


@pytest.mark.parametrize("dtype", DTYPES)
def test_sink_alone_decides_how_much_of_the_values_is_left(dtype):
    a = Attention(dtype, 3, 24, 8, 40, 56, 90, 20, 90, seed=3)
    for s in (-200.0, 0.0, 3.0, 60.0):
        a.sink = torch.tensor([s, s - 1, -s])
        a.sink_g.copy_(a.sink)
        want = a.want()
        a.store(0, 71)
        got = a.decode(70)
        full = a.prefill(0, 90)
        for h in range(3):
            scale = max(want[70, h].norm().item(), 1e-6)
            assert (got[h].double() - want[70, h]).norm().item() < (1e-5 if dtype == "float32" else 1.2e-2) * scale + 1e-9, (s, h)
            scale = max(want[:, h].norm().item(), 1e-6)
            assert (full[:, h].double() - want[:, h]).norm().item() < (1e-5 if dtype == "float32" else 1.2e-2) * scale + 1e-9, (s, h)
    b = Attention(dtype, 3, 24, 8, 40, 56, 90, 20, 90, seed=3, sink=False)
    b.store(0, 71)
    assert rel(b.decode(70), b.want()[70]) < 1.2e-2 and rel(b.prefill(0, 90), b.want()) < 1.2e-2


@pytest.mark.parametrize("dtype", DTYPES)
def test_cache_rows_from_a_portion_and_from_a_token(dtype):
    """The down projections of tokens become the same normed, rotated ring rows on both paths, and the query latent is
    normed; rows of other slots stay as they are."""
    _lib, L = lib()
    T, (qr_, rank, rot) = TYPES[dtype], (21, 30, 6)
    a = Attention(dtype, 2, 10, rot, 8, rank, 60, 9, 16)
    y, kvn, qn = rnd(51, 12, qr_ + rank + rot), 1 + 0.3 * rnd(52, rank), 1 + 0.3 * rnd(53, qr_)
    kvn_g, qn_g, yg = kvn.cuda(), qn.cuda(), y.to(T).cuda()
    a.d.kv_norm = P(kvn_g)
    cq = torch.zeros(12, qr_, dtype=T, device="cuda")
    a.ring.rows.fill_(5.0)
    pos = torch.arange(40, 52)
    want = torch.cat([plain.plain_norm(y[:, qr_:qr_ + rank].double(), kvn.double(), 1e-4),
                      plain.rotate(y[:, qr_ + rank:].double(), pos, rot, a.base)], dim=1)
    tol = 1e-6 if dtype == "float32" else 4e-3
    _lib.check_dense(L.llvq_dn_latent_rows(C.byref(a.d), P(yg), y.shape[1], qr_, P(qn_g), P(cq), 40, 12, 1, stream()))
    assert rel(cq, plain.plain_norm(y[:, :qr_].double(), qn.double(), 1e-4)) < tol
    for k in range(12):
        assert rel(a.ring.rows[(40 + k) % 16, :rank + rot], want[k]) < tol
    for s in range(52 % 16, 40 % 16):
        assert (a.ring.rows[s] == 5.0).all()
    held = a.ring.rows.clone()
    a.ring.rows.fill_(5.0)
    q, yk = torch.zeros(2 * (10 + rot), device="cuda"), y.cuda()
    for k in range(12):
        p = torch.tensor([40 + k], device="cuda")
        _lib.check_dense(L.llvq_dn_latent_query(C.byref(a.d), P(q), yk.data_ptr() + 4 * (k * y.shape[1] + qr_), P(p), stream()))
    torch.cuda.synchronize()
    assert rel(a.ring.rows, held) < (1e-7 if dtype == "float32" else 2e-3)


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
    for i, (a, b) in enumerate(zip(layers, want_layers)):
        assert rel(a, b) < (1e-5 if dtype == "float32" else 4e-2), i
    runs = {"whole": run(m, toks, [210]), "tokens": run(m, toks, [1]), "eager tokens": run(m, toks[:40], [1], use_graph=False),
            "twos": run(m, toks[:90], [2]), "mixed": run(m, toks, [64, 1, 3, 17, 2, 1, 1, 70, 5, 2]), "then tokens": run(m, toks, [150, 1])}
    for k, y in runs.items():
        ref = want[:y.shape[0]]
        assert rel(y, ref) < TOL[dtype], k
        worst = (y.double() - ref).norm(dim=1) / ref.norm(dim=1)
        assert worst.max() < 4 * TOL[dtype], (k, int(worst.argmax()))


@pytest.mark.parametrize("dtype", DTYPES)
def test_rings_that_wrap_and_slots_used_again(dtype):
    """Portions of at most 16 tokens: the rings are a window and 15 positions long and wrap many times; a second and a
    third sequence start over in slots the ones before have left."""
    m, w = build(cases.UNEVEN, 8, dtype, 900, chunk=16)
    assert [r.slots for r in m.rings] == [56, 22, 56, 22, 34]
    assert m.rings[2] is m.rings[0] and m.cache_bytes() < sum(r.rows.numel() * r.rows.element_size() for r in m.rings)
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
    m.feed(tokens_of(cases.EVEN, 77, 3), [0])  # left without a release: generate takes the cache over
    m.generate(tokens_of(cases.EVEN, 5, 4), 9, use_graph=True)
    assert torch.equal(run(m, toks, [50, 30, 1]), first)


@pytest.mark.parametrize("name,layer", [("uneven", 0), ("uneven", 1), ("uneven", 2), ("even", 0), ("even", 1), ("even", 2)])
def test_every_layers_window_ends_where_it_should(name, layer):
    """All other layers see themselves alone, so a token reaches exactly window - 1 positions ahead: changing it moves
    the logits just inside the window and leaves those just outside alone, in prompts, in portions and decoded."""
    cfg = copy.deepcopy(cases.ALL[name])
    for i, l in enumerate(cfg["layers"]):
        if i != layer:
            l["mixer"]["mask"]["size"] = 1
    size = cfg["layers"][layer]["mixer"]["mask"]["size"]
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
    """Hundreds of decoded tokens, several times around every ring, with and without the graph."""
    for dtype in DTYPES:
        m, w = build(cases.UNEVEN, 12, dtype, 700, chunk=8)
        toks = tokens_of(cases.UNEVEN, 600, 7)
        want = plain.forward(cases.UNEVEN, w, toks)
        y = run(m, toks, [5, 1])
        assert rel(y[-100:], want[-100:]) < TOL[dtype]
        assert rel(run(m, toks[:64], [1], use_graph=False), want[:64]) < TOL[dtype]


@pytest.mark.parametrize("name", list(cases.ALL))
def test_greedy_generation_through_the_entry_point(tmp_path, name):
    """The command line and load_model on a folder: the tokens are the plain statement's greedy ones (f32), the graph
    replays the eager tokens, and the bf16 model agrees with its own fed logits."""
    import json
    import os
    import subprocess
    import sys
    from conftest import ROOT
    from llvq_b200.registry import load_model
    cfg = cases.ALL[name]
    w = plain.random_model(cfg, 14)
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


def test_phases_and_overlap_leave_the_tokens_alone():
    _lib, L = lib()
    m, _ = build(cases.EVEN, 15, "bfloat16", 96)
    prompt = tokens_of(cases.EVEN, 12, 3)
    want = m.generate(prompt, 30, use_graph=True)
    ph = m.phase_split(reps=2)
    assert set(ph) == set(m.PHASES) | {"sum"} and all(v >= 0 for v in ph.values())
    assert m.generate(prompt, 30, use_graph=True) == want
    before = L.llvq_dn_launch_count()
    try:
        L.llvq_dn_set_overlap(0)
        plain_launches, _ = build(cases.EVEN, 15, "bfloat16", 96)
        assert plain_launches.generate(prompt, 30, use_graph=True) == want
    finally:
        L.llvq_dn_set_overlap(1)
    assert L.llvq_dn_launch_count() > before


def test_weights_that_do_not_fit_the_configuration_are_refused():
    w = plain.random_model(cases.UNEVEN, 1)
    for name, shape in (("l0.mix.uq", (95, 44)), ("l1.mix.sink", (4,)), ("embed", (203, 91)), ("l0.mlp.up.b", (131,))):
        bad = dict(w)
        bad[name] = torch.zeros(*shape).bfloat16()
        with pytest.raises((ValueError, RuntimeError)):
            build(cases.UNEVEN, 1, "bfloat16", 16, weights=bad)
    bad = dict(w)
    del bad["l4.mix.dkv"]
    with pytest.raises(KeyError):
        build(cases.UNEVEN, 1, "bfloat16", 16, weights=bad)
