"""What one sequence keeps from token to token: the int8 key/value cache of grouped-query attention, rings of cached rows
(latent rows, or keys and values of a window), the states of recurrent layers and the inputs of short convolutions."""
from __future__ import annotations

from typing import Optional

KV_GROUP = 64  # llvq-llm/src/kvq.rs: groups of 64 along head_dim


def kv_quantize(x):
    """[..., head_dim] f16 -> (u8 codes, f16 scale, f16 bias), groups of 64 (kvq.rs:110-165)."""
    import torch
    g = x.float().unflatten(-1, (-1, KV_GROUP))
    mn = g.amin(-1, keepdim=True)
    mx = g.amax(-1, keepdim=True)
    s = ((mx - mn) / 255.0).half()
    mn = mn.half()
    sf = s.float()
    safe = torch.where(sf > 0, sf, torch.ones_like(sf))
    t = (g - mn.float()) / safe
    # candle's round() rounds halves away from zero (kvq.rs:149-152); torch.round would round them to even
    q = torch.where(t >= 0, torch.floor(t + 0.5), -torch.floor(0.5 - t)).clamp_(0, 255)
    q = torch.where(sf > 0, q, torch.zeros_like(q)).to(torch.uint8)
    return q.flatten(-2), s.squeeze(-1), mn.squeeze(-1)


def kv_dequantize(q, s, mn):
    g = q.unflatten(-1, (-1, KV_GROUP)).float()
    return (g * s.float().unsqueeze(-1) + mn.float().unsqueeze(-1)).half().flatten(-2)


class Int8KvCache:
    """Fixed-capacity int8 KV cache of one block: [capacity, n_kv, head_dim] codes + per-group f16 scale/bias."""

    def __init__(self, capacity: int, n_kv: int, head_dim: int, device):
        import torch
        ng = head_dim // KV_GROUP
        self.q = [torch.zeros(capacity, n_kv, head_dim, dtype=torch.uint8, device=device) for _ in range(2)]
        self.s = [torch.zeros(capacity, n_kv, ng, dtype=torch.float16, device=device) for _ in range(2)]
        self.b = [torch.zeros(capacity, n_kv, ng, dtype=torch.float16, device=device) for _ in range(2)]

    def write(self, which: int, pos, x):
        """pos: int64 device tensor [L]; x: [L, n_kv, head_dim] f16."""
        q, s, b = kv_quantize(x)
        self.q[which].index_copy_(0, pos, q)
        self.s[which].index_copy_(0, pos, s)
        self.b[which].index_copy_(0, pos, b)

    def read(self, which: int, end: Optional[int] = None):
        return kv_dequantize(self.q[which][:end], self.s[which][:end], self.b[which][:end])

    def bytes_per_position(self) -> int:
        return 2 * (self.q[0][0].numel() + 2 * 2 * self.s[0][0].numel())


def whole_vectors(n: int, dtype) -> int:
    """n elements up to a whole number of 16-byte vectors."""
    vec = 16 // dtype.itemsize
    return -(-n // vec) * vec


class RowRing:
    """One row of `width` elements (and zeros to a whole vector) per position; position p sits in slot p % slots. `slots`
    covers the widest window that reads the layer and one prompt portion, so that a portion is stored whole before its
    first query looks back."""

    def __init__(self, capacity: int, window: int, portion: int, width: int, dtype, device):
        import torch
        self.slots = min(capacity, window - 1 + portion)
        self.ld = whole_vectors(width, dtype)
        self.rows = torch.zeros(self.slots, self.ld, dtype=dtype, device=device)

    def read(self, lo: int, hi: int):
        """Rows of positions [lo, hi), in order: a view, or a copy where the ring wraps between them."""
        import torch
        if not 0 <= lo < hi or hi - lo > self.slots:
            raise ValueError(f"positions [{lo}, {hi}) of a ring of {self.slots}")
        s, n = lo % self.slots, hi - lo
        if s + n <= self.slots:
            return self.rows[s:s + n]
        return torch.cat([self.rows[s:], self.rows[:s + n - self.slots]])

    def bytes_per_position(self) -> int:
        return self.ld * self.rows.element_size()


class LatentRing(RowRing):
    """Cache of one latent-attention layer: rows [latent | rotated key part], shared by all heads."""

    def __init__(self, capacity: int, window: int, portion: int, kv_rank: int, rot_dim: int, dtype, device):
        super().__init__(capacity, window, portion, kv_rank + rot_dim, dtype, device)
        self.kv_rank, self.rot_dim = kv_rank, rot_dim


class KvRing(RowRing):
    """Cache of one grouped-query layer: rows [kv_heads keys | kv_heads values], every head padded to whole vectors."""

    def __init__(self, capacity: int, window: int, portion: int, kv_heads: int, dim: int, vdim: int, dtype, device):
        self.kv_heads, self.dim, self.vdim = kv_heads, dim, vdim
        self.kd, self.vd = whole_vectors(dim, dtype), whole_vectors(vdim, dtype)
        super().__init__(capacity, window, portion, kv_heads * (self.kd + self.vd), dtype, device)

    def values_transposed(self, rows):
        """[kv_heads * vdim, positions to a multiple of 8] of rows read from the ring, zeros beyond them."""
        import torch
        n, k = rows.shape[0], self.kv_heads * self.kd
        vt = torch.empty(self.kv_heads * self.vdim, -(-n // 8) * 8, dtype=rows.dtype, device=rows.device)
        vt[:, n:].zero_()
        v = rows[:, k:k + self.kv_heads * self.vd].unflatten(1, (self.kv_heads, self.vd))[..., :self.vdim]
        vt.view(self.kv_heads, self.vdim, -1)[..., :n].copy_(v.permute(1, 2, 0))
        return vt


class RecurrentState:
    """f32 state of one recurrent layer in two halves: the state before position p is half p % 2, so a step reads one
    half and writes the other, and running it again at its position changes nothing. Nothing needs clearing: position 0
    starts from zeros whatever is stored."""

    def __init__(self, *shape: int, device):
        import torch
        self.halves = torch.zeros(2, *shape, dtype=torch.float32, device=device)


class ConvInputs:
    """The last inputs of a short causal convolution, f32: the input of position p is row p % taps."""

    def __init__(self, taps: int, channels: int, device):
        import torch
        self.rows = torch.zeros(taps, channels, dtype=torch.float32, device=device)
