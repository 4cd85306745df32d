"""Helpers of the GPU tests of the dense-weight models."""
import ctypes as C

import torch

F64 = torch.float64
TYPES = {"float32": torch.float32, "bfloat16": torch.bfloat16}
DTYPES = list(TYPES)


def gen(seed):
    return torch.Generator().manual_seed(seed)


def rnd(seed, *shape):
    """Values every element type holds exactly."""
    return torch.randn(*shape, generator=gen(seed)).bfloat16().float()


def rel(a, b):
    a, b = a.double().cpu(), b.double().cpu()
    return ((a - b).norm() / b.norm().clamp_min(1e-30)).item()


def worst_row(a, b):
    a, b = a.double().cpu().flatten(1), b.double().cpu().flatten(1)
    return ((a - b).norm(dim=1) / b.norm(dim=1).clamp_min(1e-30)).max().item()


def lib():
    from llvq_b200 import _lib
    return _lib, _lib.load_dense()


def stream():
    return C.c_void_p(torch.cuda.current_stream().cuda_stream)


def P(t):
    return t.data_ptr() if t is not None else None


def dn(dtype):
    _lib, _ = lib()
    return {"float32": _lib.DN_F32, "bfloat16": _lib.DN_BF16}[dtype]


def ok(status):
    _lib, _ = lib()
    _lib.check_dense(status)


def no_time_out():
    _, L = lib()
    err = C.c_int32(7)
    ok(L.llvq_dn_poll_error(C.byref(err)))
    assert err.value == 0


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
