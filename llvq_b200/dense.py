"""What the models on dense weights share (bf16 or f32, libllvq_dense.so): matrices in the kernels' layout, the products
of prompt portions by the library, the head, and the token step as a prebuilt launch list."""
from __future__ import annotations

import ctypes as C
from typing import Optional

from . import _lib
from .cache import whole_vectors
from .token_loop import TokenLoop


class DenseMatrix:
    """Row-concatenated (or row-interleaved) [out, in] matrices on the device, rows padded with zeros to whole 16-byte
    vectors."""

    def __init__(self, parts, dtype, device, interleave: bool = False):
        import torch
        self.n, self.k = sum(p.shape[0] for p in parts), parts[0].shape[1]
        self.ld = whole_vectors(self.k, dtype)
        self.w = torch.zeros(self.n, self.ld, dtype=dtype, device=device)
        if interleave:
            if len({p.shape[0] for p in parts}) != 1:
                raise ValueError(f"interleaved matrices of {[p.shape[0] for p in parts]} rows")
            for i, p in enumerate(parts):
                self.w[i::len(parts), :self.k].copy_(p)
            return
        at = 0
        for p in parts:
            self.w[at:at + p.shape[0], :self.k].copy_(p)
            at += p.shape[0]

    def rows(self, lo: int, hi: Optional[int] = None):
        """The unpadded rows as an operand of a matrix product."""
        return self.w[lo:hi, :self.k]

    def ptr(self, row: int = 0) -> int:
        return self.w.data_ptr() + row * self.ld * self.w.element_size()


class ColumnMatrix(DenseMatrix):
    """Column-concatenated [out, in] matrices, one product over activations that lie side by side: part i meets the
    columns from `at[i]` on. Every part is padded with zeros to whole 16-byte vectors, so k = ld."""

    def __init__(self, parts, dtype, device):
        import torch
        self.at, self.n = [], parts[0].shape[0]
        self.k = 0
        for p in parts:
            if p.shape[0] != self.n:
                raise ValueError(f"matrices of {[q.shape[0] for q in parts]} rows side by side")
            self.at.append(self.k)
            self.k += whole_vectors(p.shape[1], dtype)
        self.ld = self.k
        self.padded = any(whole_vectors(p.shape[1], dtype) != p.shape[1] for p in parts)
        self.w = torch.zeros(self.n, self.ld, dtype=dtype, device=device)
        for lo, p in zip(self.at, parts):
            self.w[:, lo:lo + p.shape[1]].copy_(p)


class DenseLM(TokenLoop):
    """A TokenLoop over libllvq_dense.so. A model sets `head` (DenseMatrix), `final_norm` (f32 factors as applied), `eps`,
    `softcap` (0: none) and `_steps`, the (phase, call) list of one token."""
    softcap = 0.0

    def _init_dense(self, dtype: str, device, capacity: int, prefill_chunk: int) -> None:
        import torch
        self.lib = _lib.load_dense()
        self.dtype = {"bfloat16": torch.bfloat16, "float32": torch.float32}[dtype]
        self.dt = {"bfloat16": _lib.DN_BF16, "float32": _lib.DN_F32}[dtype]
        self._init_loop(device, capacity, prefill_chunk)

    def _init_head(self) -> None:
        import torch
        dev = self.device
        self._logits = torch.zeros(self.head.n, dtype=torch.float32, device=dev)
        self._best_val, self._scratch = torch.zeros(1, dtype=torch.float32, device=dev), torch.zeros(8192, dtype=torch.uint8, device=dev)
        self._best_idx = torch.zeros(1, dtype=torch.long, device=dev)

    @staticmethod
    def _cuda_stream():
        import torch
        return C.c_void_p(torch.cuda.current_stream().cuda_stream)

    # ---- the token step ----------------------------------------------------------
    def _eager_step(self) -> None:
        st, only = self._cuda_stream(), self._only
        for phase, call in self._steps:
            if only is None or only == phase:
                call(st)
        if only is None:
            self._tok.copy_(self._best_idx)
            self._pos += 1

    def _head(self, x, st) -> None:
        """Final norm, (capped) logits and greedy pick of one f32 hidden state."""
        H = self.head
        d = _lib.DenseGemv(dtype=self.dt, prologue=_lib.DN_NORM, n_out=H.n, k=H.k, ldw=H.ld, alpha=1.0, eps=self.eps, softcap=self.softcap,
                           w=H.ptr(), y=self._logits.data_ptr(), x=x.data_ptr(), norm_w=self.final_norm.data_ptr())
        _lib.check_dense(self.lib.llvq_dn_head(C.byref(d), self._scratch.data_ptr(), self._best_val.data_ptr(), self._best_idx.data_ptr(), st))

    def step_logits(self):
        return self._logits.clone()

    def pick_last(self, x):
        self._head(x[-1:].contiguous(), self._cuda_stream())
        return self._best_idx.clone()

    # ---- prompt portions ---------------------------------------------------------
    def _product(self, fn, x, w, out_dtype=None):
        """A library product: bf16 with f32 accumulation, or true f32."""
        import torch
        m = torch.backends.cuda.matmul
        if self.dtype == torch.float32:
            held, m.allow_tf32 = m.allow_tf32, False
            try:
                return fn(x, w)
            finally:
                m.allow_tf32 = held
        return fn(x, w) if out_dtype is None else fn(x, w, out_dtype=out_dtype)

    def _mm(self, x, w, out_dtype=None):
        """x w^T."""
        import torch
        return self._product(torch.mm, x, w.t(), out_dtype)

    def _bmm(self, x, w, out_dtype=None):
        """x[b] w[b]^T."""
        import torch
        return self._product(torch.bmm, x, w.transpose(1, 2), out_dtype)

    def logits(self, x):
        import torch
        st = self._cuda_stream()
        x = x.contiguous()
        h = torch.empty(x.shape, dtype=self.dtype, device=self.device)
        _lib.check_dense(self.lib.llvq_dn_postnorm_rows(self.dt, x.data_ptr(), None, None, self.final_norm.data_ptr(), 1.0, self.eps, h.data_ptr(),
                                                        None, x.shape[0], x.shape[1], st))
        y = self._mm(h, self.head.rows(0), torch.float32)
        if self.softcap:
            _lib.check_dense(self.lib.llvq_dn_softcap(y.data_ptr(), y.numel(), self.softcap, st))
        return y
