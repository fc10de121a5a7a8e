"""Mamba-2 mixer: state-space duality with a scalar decay per head.

``W_in h`` is ``[z | x | B | C | dt]``.  ``x``, ``B`` and ``C`` pass one causal convolution per channel and SiLU; with
``dt = softplus(raw + bias)`` a head's state obeys

    S_t = exp(-exp(A_log) dt) S_(t-1) + dt B_t x_t^T,      y_t = S_t^T C_t + D x_t

(``B`` and ``C`` are shared by the heads of a group).  The heads' outputs are gated by ``silu(z)``, normed in
``norm_groups`` equal parts and projected back.

The three parts of the fused projection start on 16-byte boundaries: rows of zeros fill the gaps.  Whole sequences run
convolution, scan and gated norm as one kernel each; a decode step is two, convolution + state update and gated norm.
A row's decode state is the float32 matrix of every head and a ring of the last ``conv`` convolution inputs.
"""
from __future__ import annotations

from dataclasses import dataclass

import torch
from torch import nn

from .. import ops
from .lora import FusedLoraLinear


@dataclass(frozen=True)
class Mamba2Dims:
    heads: int
    vdim: int                   # columns of a head's state: its share of x
    state: int                  # rows of a head's state: entries of B and C
    groups: int                 # B and C per token
    conv: int                   # taps of the convolution
    norm_groups: int

    @property
    def inner(self) -> int:
        return self.heads * self.vdim

    @property
    def channels(self) -> int:
        return self.inner + 2 * self.groups * self.state

    def validate(self) -> None:
        for n in ("heads", "vdim", "state", "groups", "conv", "norm_groups"):
            if getattr(self, n) <= 0:
                raise ValueError(f"mamba2: {n} must be > 0")
        if self.heads % self.groups:
            raise ValueError("mamba2: groups must divide heads")
        if self.inner % self.norm_groups:
            raise ValueError("mamba2: norm_groups must divide heads * vdim")


class Mamba2(nn.Module):
    def __init__(self, hidden: int, dims: Mamba2Dims, eps: float, lora, letters: str, kw: dict):
        """``letters``: adapted projections, the hybrid families' recurrent-layer letters (q the convolution's inputs,
        z the gate, a the step sizes, o the output)."""
        super().__init__()
        dims.validate()
        self.dims, self.eps = dims, eps
        sizes, names, adapted, self.at = [], [], [], {}
        for name, n, on in (("z", dims.inner, "z" in letters), ("xbc", dims.channels, "q" in letters), ("dt", dims.heads, "a" in letters)):
            self.at[name] = (sum(sizes), n)
            sizes.append(n)
            names.append(name)
            adapted.append(on)
            if sum(sizes) % 8:
                sizes.append(8 - sum(sizes) % 8)
                names.append("pad")
                adapted.append(False)
        self.inp = FusedLoraLinear(hidden, sizes, names, adapted, lora, **kw)
        self.out = FusedLoraLinear(dims.inner, [hidden], ("o",), ("o" in letters,), lora, **kw)
        train, dev = kw.get("trainable_base", False), kw.get("device")

        def reg(n, *shape, value=0.0):
            t = torch.full(shape, value, dtype=torch.float32, device=dev)
            if train:
                setattr(self, n, nn.Parameter(t))
            else:
                self.register_buffer(n, t, persistent=False)
        reg("conv_w", dims.channels, dims.conv)
        reg("conv_b", dims.channels)
        reg("dt_bias", dims.heads)
        reg("A_log", dims.heads)
        reg("D", dims.heads, value=1.0)
        reg("norm", dims.inner, value=1.0)

    def projections(self):
        return (self.inp, self.out)

    def ensure_positions(self, n: int) -> None:
        pass

    def refresh_derived(self):
        pass

    def set_input_weight(self, w: torch.Tensor) -> None:
        """``w``: the rows ``[z | x | B | C | dt]`` without gaps."""
        d = self.dims
        full = w.new_zeros(self.inp.weight.shape)
        src = 0
        for name in ("z", "xbc", "dt"):
            at, n = self.at[name]
            full[at:at + n] = w[src:src + n]
            src += n
        if src != w.shape[0]:
            raise ValueError(f"mamba2: input projection of {w.shape[0]} rows, expected {2 * d.inner + 2 * d.groups * d.state + d.heads}")
        self.inp.set_weight(full)

    def split(self, p: torch.Tensor):
        return tuple(p[..., at:at + n] for at, n in (self.at["z"], self.at["xbc"], self.at["dt"]))

    def forward(self, h, merged: bool = False, lens=None, store=None):
        """Whole sequences ``h`` ``[B,S,hidden]`` from an empty state; tokens at or past ``lens[b]`` leave no trace in it.
        ``store`` receives the convolution inputs ``[B,S,C]`` and the final states ``[B,heads,state,vdim]``."""
        d = self.dims
        lin = (lambda m, x: m.forward_merged(x)) if merged else (lambda m, x: m(x))
        z, xbc, dt = self.split(lin(self.inp, h))
        u = ops.ssm_conv(xbc, self.conv_w, self.conv_b)
        y, S = ops.ssm_scan(u, dt, self.dt_bias, self.A_log, self.D, lens, heads=d.heads, state=d.state, groups=d.groups)
        if store is not None:
            store(xbc, S)
        return lin(self.out, ops.gated_group_norm(y, z, self.norm, d.norm_groups, self.eps))

    def decode(self, h, kv_len, active, state):
        """One token per row, ``h`` ``[B,hidden]``, merged weights; ``state`` advances in place."""
        d = self.dims
        z, xbc, dt = self.split(self.inp.forward_merged(h))
        y = ops.ssm_step(xbc, dt, self.conv_w, self.conv_b, self.dt_bias, self.A_log, self.D, state.ring, state.S, kv_len, active,
                         groups=d.groups)
        return self.out.forward_merged(ops.gated_group_norm(y, z, self.norm, d.norm_groups, self.eps))

    def new_state(self, batch: int, max_len: int, dtype, device) -> "Mamba2State":
        d = self.dims
        return Mamba2State(torch.zeros(batch, d.conv, d.channels, dtype=dtype, device=device),
                           torch.zeros(batch, d.heads, d.state, d.vdim, dtype=torch.float32, device=device))


@dataclass
class Mamba2State:
    """Decode state of one layer: convolution inputs (slot = position mod taps) and the heads' matrices."""
    ring: torch.Tensor
    S: torch.Tensor

    def fill(self, rows, lens, xbc, S) -> None:
        from .latent import fill_cache
        fill_cache(self.ring, rows, xbc, lens)
        self.S[rows] = S

    def tensors(self):
        return [self.ring, self.S]

    def advanced(self):
        return [self.S]

    def rows_read(self, nxt):
        return None
