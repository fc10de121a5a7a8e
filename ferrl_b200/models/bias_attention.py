"""Sliding-window attention with a learned bias per distance, whose values are the keys.

``q = W_q h + b_q`` and ``k = W_k h + b_k`` are the only projections in front of the scores; a head's output is the
softmax-weighted sum of the keys themselves.  No rotation: positions enter through the window and through a bias that is
added to the scaled score, ``rel[bucket(i - j), head]``.  The first half of the buckets hold one distance each, the
others grow geometrically up to ``bias_max``.

For the kernels the table is spread over distances once (``[heads, window]`` float32): inside a window the bias of a key
is then one load.  A token's cache entry is its key, ``kv_heads * dim`` entries, in a ring of ``window`` slots per batch
row; each cached byte is read once and serves the score and the output.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch
from torch import nn

from .. import ops
from .lora import FusedLoraLinear


@dataclass(frozen=True)
class BiasAttentionDims:
    heads: int
    kv_heads: int
    dim: int
    scale: float
    window: int                 # tokens a query sees, itself included
    buckets: int
    bias_max: int               # distance at which the last bucket starts

    def validate(self) -> None:
        for n in ("heads", "kv_heads", "dim", "window"):
            if getattr(self, n) <= 0:
                raise ValueError(f"biased attention: {n} must be > 0")
        if self.heads % self.kv_heads:
            raise ValueError("biased attention: kv_heads must divide heads")
        if self.buckets < 2 or self.bias_max <= self.buckets // 2:
            raise ValueError("biased attention: bias_max must lie beyond the first half of the buckets")

    def bucket_of(self, n: int) -> torch.Tensor:
        """Bucket of every distance ``0 .. n-1``: where the geometric buckets start is found in whole numbers."""
        half, m = self.buckets // 2, self.buckets - self.buckets // 2
        starts = []
        for k in range(1, m):
            at = max(half, int(half * (self.bias_max / half) ** (k / m)) - 2)
            while at ** m * half ** k < self.bias_max ** k * half ** m:
                at += 1
            starts.append(at)
        d = torch.arange(n)
        far = half + torch.bucketize(d, torch.tensor(starts, dtype=torch.int64), right=True)
        return torch.where(d < half, d, far)


class BiasAttention(nn.Module):
    def __init__(self, hidden: int, dims: BiasAttentionDims, lora, targets, kw: dict):
        super().__init__()
        dims.validate()
        self.dims = d = dims
        self.inp = FusedLoraLinear(hidden, [d.heads * d.dim, d.kv_heads * d.dim], ("q", "k"),
                                   (targets.attn_q, targets.attn_k or targets.attn_v), lora, bias=True, **kw)
        self.out = FusedLoraLinear(d.heads * d.dim, [hidden], ("o",), (targets.attn_o,), lora, **kw)
        rel = torch.zeros(d.buckets, d.heads, dtype=torch.float32, device=kw.get("device"))
        if kw.get("trainable_base", False):
            self.rel = nn.Parameter(rel)
        else:
            self.register_buffer("rel", rel, persistent=False)
        self.register_buffer("table", None, persistent=False)

    def projections(self):
        return (self.inp, self.out)

    def spread(self, n: int) -> torch.Tensor:
        """``[heads, n]``: the bias of the distances ``0 .. n-1``."""
        return self.rel[self.dims.bucket_of(n).to(self.rel.device)].t()

    @torch.no_grad()
    def ensure_positions(self, n: int) -> None:
        n = min(n, self.dims.window)
        if self.table is None or self.table.shape[1] < n:
            self.table = self.spread(n).contiguous()

    @torch.no_grad()
    def refresh_derived(self):
        if self.table is not None:
            self.table.copy_(self.spread(self.table.shape[1]))       # stable address for captured decode graphs

    def bias(self) -> torch.Tensor:
        if torch.is_grad_enabled() and self.rel.requires_grad:
            return self.spread(self.table.shape[1])
        return self.table

    def forward(self, h, merged: bool = False, lens=None, store=None):
        """Whole sequences ``h`` ``[B,S,hidden]``; ``store`` receives the keys ``[B,S,kv_heads*dim]``."""
        d = self.dims
        lin = (lambda m, z: m.forward_merged(z)) if merged else (lambda m, z: m(z))
        q, k = lin(self.inp, h).split([d.heads * d.dim, d.kv_heads * d.dim], dim=-1)
        if store is not None:
            store(k)
        a = ops.bias_attention(q.unflatten(-1, (d.heads, d.dim)), k.unflatten(-1, (d.kv_heads, d.dim)), self.bias(), scale=d.scale,
                               window=d.window)
        return lin(self.out, a)

    def decode(self, h, kv_len, active, state):
        """One token per row, ``h`` ``[B,hidden]``, merged weights; ``state`` is ``(ring of keys, bias table)``."""
        d = self.dims
        q, k = self.inp.forward_merged(h).split([d.heads * d.dim, d.kv_heads * d.dim], dim=-1)
        return self.out.forward_merged(ops.bias_decode(q, k, state.ring, kv_len, state.table, dim=d.dim, scale=d.scale, active=active))

    def new_state(self, batch: int, max_len: int, dtype, device) -> "KeyRing":
        self.ensure_positions(max_len)
        d = self.dims
        return KeyRing(torch.zeros(batch, min(max_len, d.window), d.kv_heads * d.dim, dtype=dtype, device=device), self.table)


@dataclass
class KeyRing:
    """Decode cache of one layer: the last ``slots`` keys of every row, slot = position mod slots."""
    ring: torch.Tensor
    table: torch.Tensor                # the layer's biases; held here so that a captured graph keeps its operand

    def fill(self, rows, lens, keys) -> None:
        from .latent import fill_cache
        fill_cache(self.ring, rows, keys, lens)

    def tensors(self):
        return [self.ring]

    def advanced(self):
        """What a decode step changes in a way that repeating the step does not."""
        return []

    def rows_read(self, nxt: torch.Tensor) -> Optional[torch.Tensor]:
        return nxt.clamp(max=self.ring.shape[1]).sum()
