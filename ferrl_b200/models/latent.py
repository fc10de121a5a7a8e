"""Latent attention: keys and values of all heads are up projections of one low-rank latent per token.

``q = W_q h`` holds, head by head, ``dim`` entries that are not rotated and ``rot`` that are.  ``W_dkv h`` gives the
latent (``rank`` entries, RMS-normed) and one rotated key part (``rot`` entries) that all heads share; the unrotated
keys are ``W_uk c`` and the values ``W_uv c``.  A token's cache entry is the row ``[c | rotated key part]``, of a width
that does not depend on the number of heads.

Two evaluation orders, one result:

* whole sequences expand the latent once (one GEMM for keys and values) and run flash attention whose score is the
  sum of two dot products;
* decoding absorbs ``W_uk`` into the query and ``W_uv`` into the output, so all heads of a row attend to the cached
  latent rows themselves: the cache is read once per row, not once per head.

Parameters of the mechanism: head count and the four sizes, the score scale, an optional sliding window (``window``
tokens including the query's own; the decode cache is then a ring of that many slots), an optional learned sink per
head (a constant term in the softmax denominator), and the rotation's base and width.
"""
from __future__ import annotations

from dataclasses import dataclass

import torch
from torch import nn

from .. import ops
from .lora import FusedLoraLinear


@dataclass(frozen=True)
class LatentDims:
    heads: int
    dim: int                    # unrotated query / key entries per head
    rot: int                    # rotated query / key entries per head
    vdim: int                   # value entries per head
    rank: int                   # latent entries
    scale: float
    window: int = 0             # 0: every earlier token is visible
    rope_base: float = 1e4
    rope_dims: int = 0          # leading entries of the rotated part that turn (0: all of it)
    sink: bool = False

    @property
    def turned(self) -> int:
        return self.rope_dims or self.rot

    def validate(self) -> None:
        for n in ("heads", "dim", "rot", "vdim", "rank"):
            if getattr(self, n) <= 0:
                raise ValueError(f"latent attention: {n} must be > 0")
        if self.turned % 2 or self.turned > self.rot:
            raise ValueError("latent attention: the rotation needs an even width within the rotated part")
        if self.window < 0:
            raise ValueError("latent attention: window must be >= 0")

    def row_width(self) -> int:
        return ops.eager.latent_row_width(self.rank, self.rot)


class LatentAttention(nn.Module):
    """The mixer without its output projection's residual.  ``extra`` further output rows may ride in the fused input
    projection (``[q | dkv | extra]``); ``split`` hands them back."""

    def __init__(self, hidden: int, dims: LatentDims, eps: float, lora, targets, kw: dict, extra: int = 0,
                 extra_name: str = "extra"):
        super().__init__()
        dims.validate()
        self.dims, self.eps = dims, eps
        d = dims
        sizes = [d.heads * (d.dim + d.rot), d.rank + d.rot] + ([extra] if extra else [])
        names = ["q", "dkv"] + ([extra_name] if extra else [])
        adapted = [targets.attn_q, targets.attn_k or targets.attn_v] + ([False] if extra else [])
        self.inp = FusedLoraLinear(hidden, sizes, names, adapted, lora, **kw)
        self.up = FusedLoraLinear(d.rank, [d.heads * d.dim, d.heads * d.vdim], ("uk", "uv"), (False, False), None, **kw)
        self.out = FusedLoraLinear(d.heads * d.vdim, [hidden], ("o",), (targets.attn_o,), lora, **kw)
        train, dev = kw.get("trainable_base", False), kw.get("device")
        reg = (lambda n, t: setattr(self, n, nn.Parameter(t))) if train else \
            (lambda n, t: self.register_buffer(n, t, persistent=False))
        reg("latent_norm", torch.ones(d.rank, dtype=torch.float32, device=dev))
        if d.sink:
            reg("sink", torch.zeros(d.heads, dtype=torch.float32, device=dev))
        else:
            self.sink = None
        # decode operands: W_uk with each head transposed (the query absorbs it), W_uv as stored
        self.register_buffer("uk_t", None, persistent=False)

    def projections(self):
        return (self.inp, self.up, self.out)

    @torch.no_grad()
    def refresh_derived(self):
        d = self.dims
        uk = self.up.weight[:d.heads * d.dim].detach().view(d.heads, d.dim, d.rank)
        new = uk.transpose(1, 2).contiguous()
        if self.uk_t is not None and self.uk_t.shape == new.shape:
            self.uk_t.copy_(new)            # stable address for captured decode graphs
        else:
            self.uk_t = new

    def uv(self) -> torch.Tensor:
        d = self.dims
        return self.up.weight[d.heads * d.dim:].view(d.heads, d.vdim, d.rank)

    def split(self, p: torch.Tensor):
        """Fused projection -> ``(q [..., H, dim+rot], dkv, extra or None)``."""
        d = self.dims
        nq, nd = d.heads * (d.dim + d.rot), d.rank + d.rot
        q = p[..., :nq].unflatten(-1, (d.heads, d.dim + d.rot))
        return q, p[..., nq:nq + nd], (p[..., nq + nd:] if p.shape[-1] > nq + nd else None)

    def forward(self, h, positions, cos, sin, merged: bool = False, store=None):
        """Whole sequences ``h`` ``[B,S,hidden]`` -> ``(output [B,S,hidden], extra rows)``; ``store`` receives the
        latent rows ``[B,S,width]``."""
        d = self.dims
        lin = (lambda m, z: m.forward_merged(z)) if merged else (lambda m, z: m(z))
        q, dkv, extra = self.split(lin(self.inp, h))
        q, lat = ops.latent_prep(q, dkv, self.latent_norm, self.eps, cos, sin, positions, dim=d.dim, rank=d.rank)
        if store is not None:
            store(lat)
        kv = lin(self.up, lat[..., :d.rank])
        a = ops.latent_attention(q, kv, lat, dim=d.dim, vdim=d.vdim, rank=d.rank, scale=d.scale, window=d.window,
                                 sink=self.sink)
        return lin(self.out, a), extra

    def decode(self, h, kv_len, count, cos, sin, cache):
        """One token per row, ``h`` ``[B,hidden]``, merged weights.  The token's latent row is written to its slot of
        ``cache`` ``[B,slots,width]`` first; ``count[b]`` slots are then occupied (0: a retired row, which attends to
        nothing)."""
        d = self.dims
        q, dkv, extra = self.split(self.inp.forward_merged(h))
        q = ops.latent_append(q, dkv, self.latent_norm, self.eps, cos, sin, kv_len, cache, dim=d.dim, rank=d.rank)
        a = ops.latent_decode(q, self.uk_t, self.uv(), cache, count, rank=d.rank, scale=d.scale, sink=self.sink)
        return self.out.forward_merged(a), extra

    def slots(self, max_len: int) -> int:
        return min(max_len, self.dims.window) if self.dims.window else max_len


@torch.no_grad()
def fill_cache(cache: torch.Tensor, rows: torch.Tensor, lat: torch.Tensor, lens: torch.Tensor) -> None:
    """Prefilled latent rows ``lat`` ``[P,L,width]`` of true lengths ``lens`` -> cache rows ``rows``.  A cache of
    ``n < L`` slots is a ring: slot ``s`` holds the row's newest token ``p`` with ``p % n == s``."""
    P, L, _ = lat.shape
    n = cache.shape[1]
    if n >= L:
        cache[rows, :L] = lat
        return
    s = torch.arange(n, device=lat.device)[None, :]
    pos = (s + n * ((lens.long()[:, None] - 1 - s).clamp(min=0) // n)).clamp(max=L - 1)
    cache[rows] = torch.gather(lat, 1, pos[:, :, None].expand(P, n, lat.shape[2]))
