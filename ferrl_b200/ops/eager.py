"""Plain PyTorch restatements of every hot op.

These run the CPU path (tests, the tiny smoke config) and are the numerical
oracle that each sm_100a kernel in ``csrc/`` is checked against.  Everything
accumulates in float32 and is written the obvious way on purpose.
"""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Optional

import torch
import torch.nn.functional as F


# ---------------------------------------------------------------- norms ----
def rmsnorm(x: torch.Tensor, weight: Optional[torch.Tensor], eps: float, zero_centered: bool = False):
    """``x * rsqrt(mean(x^2)+eps) * w`` computed in fp32 then cast back; with
    ``zero_centered`` the scale is ``1 + w`` (reference nn.rs:37-157)."""
    xf = x.float()
    y = xf * torch.rsqrt(xf.pow(2).mean(-1, keepdim=True) + eps)
    if weight is not None:
        w = weight.float()
        y = y * ((1.0 + w) if zero_centered else w)
    return y.to(x.dtype)


def rmsnorm_gated(x, gate, weight, eps):
    """``rmsnorm(x) * w * silu(gate)`` (reference nn.rs:169-222)."""
    xf = x.float()
    y = xf * torch.rsqrt(xf.pow(2).mean(-1, keepdim=True) + eps) * weight.float()
    return (y * F.silu(gate.float())).to(x.dtype)


def add_rmsnorm(x, residual, weight, eps, zero_centered=False):
    """Residual add fused with the following norm: returns ``(norm(h), h)`` with
    ``h = x + residual``."""
    h = x + residual
    return rmsnorm(h, weight, eps, zero_centered), h


def l2norm(x, eps: float = 1e-6):
    xf = x.float()
    return (xf * torch.rsqrt(xf.pow(2).sum(-1, keepdim=True) + eps)).to(x.dtype)


def stable_softplus(x):
    return F.softplus(x)


def layernorm(x, weight, bias, eps):
    """Layer norm in fp32 (mean and mean squared deviation, ``eps`` inside the root), float32 result."""
    xf = x.float()
    d = xf - xf.mean(-1, keepdim=True)
    y = d * torch.rsqrt(d.pow(2).mean(-1, keepdim=True) + eps)
    if weight is not None:
        y = y * weight.float()
    return y if bias is None else y + bias.float()


def post_norm(x, y, weight, bias, eps, alpha: float = 1.0, gate=None, gate_bias=None, history=None, coef=None):
    """Norm after the residual sum on a float32 stream: ``r = layernorm(alpha * x + y * sigmoid(gate + gate_bias))``.
    ``y = None`` is a plain layer norm of ``x``; without ``gate`` the branch is added as it is.  With ``history``
    ``[n, ..., W]`` (the earlier streams) and ``coef`` ``[n + 1]`` the stream that goes on is
    ``sum_j coef[j] history[j] + coef[n] r``.  Returns ``(next, r)``, both float32."""
    t = x.float()
    if y is not None:
        yf = y.float()
        if gate is not None:
            g = gate.float()
            yf = yf * torch.sigmoid(g if gate_bias is None else g + gate_bias.float())
        t = alpha * t + yf
    r = layernorm(t, weight, bias, eps)
    if history is None:
        return r, r
    nxt = coef[history.shape[0]].float() * r
    for j in range(history.shape[0]):
        nxt = nxt + coef[j].float() * history[j]
    return nxt, r


# ----------------------------------------------------------------- rope ----
def rope_tables(inv_freq: torch.Tensor, max_pos: int, device=None):
    t = torch.arange(max_pos, dtype=torch.float32, device=inv_freq.device)
    fr = torch.outer(t, inv_freq.float())
    return fr.cos().to(device), fr.sin().to(device)


def default_inv_freq(rot_dim: int, theta: float) -> torch.Tensor:
    i = torch.arange(0, rot_dim, 2, dtype=torch.float64)
    return (1.0 / (theta ** (i / rot_dim))).float()


def llama3_inv_freq(rot_dim, theta, factor, low_freq_factor, high_freq_factor, original_max_pos):
    """Llama-3 wavelength smoothing (reference llama.rs:59-88)."""
    base = default_inv_freq(rot_dim, theta)
    low_w = original_max_pos / low_freq_factor
    high_w = original_max_pos / high_freq_factor
    out = []
    for f in base.tolist():
        w = 2.0 * math.pi / f
        if w < high_w:
            out.append(f)
        elif w > low_w:
            out.append(f / factor)
        else:
            s = (original_max_pos / w - low_freq_factor) / (high_freq_factor - low_freq_factor)
            out.append((1.0 - s) * f / factor + s * f)
    return torch.tensor(out, dtype=torch.float32)


def apply_rope(x: torch.Tensor, cos: torch.Tensor, sin: torch.Tensor, positions: torch.Tensor):
    """Rotate-half RoPE on the leading ``2*cos.shape[-1]`` channels of the last
    dim. ``x`` ``[B, S, H, D]``; ``positions`` ``[B, S]`` or ``[S]`` (int64);
    tables ``[max_pos, rot/2]``.  Channels past the rotary width pass through
    (partial RoPE, reference blocks.rs:225-244)."""
    half = cos.shape[-1]
    rot = 2 * half
    if positions.dim() == 1:
        positions = positions[None, :].expand(x.shape[0], -1)
    c = cos[positions].unsqueeze(2).float()  # [B,S,1,half]
    s = sin[positions].unsqueeze(2).float()
    xr = x[..., :rot].float()
    x1, x2 = xr[..., :half], xr[..., half:]
    out = torch.cat([x1 * c - x2 * s, x2 * c + x1 * s], dim=-1).to(x.dtype)
    if rot == x.shape[-1]:
        return out
    return torch.cat([out, x[..., rot:]], dim=-1)


def qk_norm_rope(q, k, q_w, k_w, eps, cos, sin, positions, zero_centered=False):
    """Per-head RMSNorm of q and k (skipped when the weights are ``None``)
    followed by RoPE. ``q`` ``[B,S,Hq,D]``, ``k`` ``[B,S,Hkv,D]``."""
    if q_w is not None:
        q = rmsnorm(q, q_w, eps, zero_centered)
        k = rmsnorm(k, k_w, eps, zero_centered)
    return apply_rope(q, cos, sin, positions), apply_rope(k, cos, sin, positions)


# ------------------------------------------------------------ attention ----
def attention(q, k, v, *, scale: float, causal: bool = True, window: int = 0,
              q_offset: int = 0, softmax_fp32: bool = True, kv_len: Optional[torch.Tensor] = None):
    """GQA attention. ``q`` ``[B,Sq,Hq,D]``, ``k``/``v`` ``[B,Sk,Hkv,D]``.
    Query ``i`` sits at absolute position ``q_offset + i`` and sees keys
    ``j <= pos`` (causal) and ``j > pos - window`` (sliding window, ``window>0``).
    ``kv_len`` ``[B]`` masks keys at or beyond each row's cache length."""
    B, Sq, Hq, D = q.shape
    Sk, Hkv = k.shape[1], k.shape[2]
    rep = Hq // Hkv
    qf = q.permute(0, 2, 1, 3)
    kf = k.permute(0, 2, 1, 3).repeat_interleave(rep, dim=1)
    vf = v.permute(0, 2, 1, 3).repeat_interleave(rep, dim=1)
    if softmax_fp32:
        qf, kf, vf = qf.float(), kf.float(), vf.float()
    scores = torch.matmul(qf, kf.transpose(-1, -2)) * scale
    qi = torch.arange(Sq, device=q.device)[:, None] + q_offset
    kj = torch.arange(Sk, device=q.device)[None, :]
    allowed = torch.ones(Sq, Sk, dtype=torch.bool, device=q.device)
    if causal:
        allowed &= kj <= qi
    if window and window > 0:
        allowed &= kj > qi - window
    allowed = allowed[None, None]
    if kv_len is not None:
        allowed = allowed & (kj[None, None] < kv_len.view(B, 1, 1, 1))
    scores = scores.masked_fill(~allowed, float("-inf"))
    p = torch.softmax(scores.float(), dim=-1).to(vf.dtype)
    p = torch.nan_to_num(p)  # rows with no visible key
    out = torch.matmul(p, vf)
    return out.permute(0, 2, 1, 3).to(q.dtype).contiguous()


def decode_attention(q, k_cache, v_cache, kv_len, *, scale: float, window: int = 0):
    """One new token per row against a dense cache. ``q`` ``[B,Hq,D]``, caches
    ``[B,Smax,Hkv,D]``, ``kv_len`` ``[B]`` counts valid keys *including* the new
    token (already written)."""
    B, Hq, D = q.shape
    Smax = k_cache.shape[1]
    kj = torch.arange(Smax, device=q.device)[None, :]
    allowed = kj < kv_len[:, None]
    if window and window > 0:
        allowed &= kj >= (kv_len[:, None] - window)
    Hkv = k_cache.shape[2]
    rep = Hq // Hkv
    kf = k_cache.float().repeat_interleave(rep, dim=2)  # [B,S,Hq,D]
    vf = v_cache.float().repeat_interleave(rep, dim=2)
    scores = torch.einsum("bhd,bshd->bhs", q.float(), kf) * scale
    scores = scores.masked_fill(~allowed[:, None, :], float("-inf"))
    p = torch.softmax(scores, dim=-1)
    p = torch.where(allowed.any(dim=1)[:, None, None], p, torch.zeros_like(p))   # a row with no keys attends to nothing
    return torch.einsum("bhs,bshd->bhd", p, vf).to(q.dtype)


# ----------------------------------------------------- latent attention ----
def latent_row_width(rank: int, rot: int) -> int:
    """Elements of a cached latent row ``[c | rotated key part]``, padded so that rows start on 16-byte boundaries."""
    return (rank + rot + 7) // 8 * 8


def latent_prep(q, dkv, norm_w, eps, cos, sin, positions, dim: int, rank: int):
    """``q`` ``[B,S,H,dim+rot]`` and the down projection ``dkv`` ``[B,S,rank+rot]`` -> ``(q with its last rot entries
    rotated, latent rows [B,S,width])``: a row is the RMS-normed latent followed by the rotated key part that all
    heads share."""
    qr = torch.cat([q[..., :dim], apply_rope(q[..., dim:], cos, sin, positions)], dim=-1)
    c = rmsnorm(dkv[..., :rank].float(), norm_w.float(), eps).to(dkv.dtype)
    kr = apply_rope(dkv[..., None, rank:], cos, sin, positions)[..., 0, :]
    row = torch.cat([c, kr], dim=-1)
    return qr, F.pad(row, (0, latent_row_width(rank, kr.shape[-1]) - row.shape[-1]))


def _sink_softmax(scores, sink):
    """Softmax over the last axis of ``scores`` ``[B,H,...,K]`` (fp32, masked with ``-inf``); with ``sink`` ``[H]`` the
    denominator also holds ``exp(sink_h)``."""
    if sink is None:
        return torch.nan_to_num(torch.softmax(scores, dim=-1))
    s = sink.float().view(1, -1, *([1] * (scores.dim() - 2)))
    m = torch.maximum(scores.amax(-1, keepdim=True), s)
    e = torch.exp(scores - m)
    return e / (e.sum(-1, keepdim=True) + torch.exp(s - m))


def latent_attention(q, kv, lat, *, dim: int, vdim: int, rank: int, scale: float, window: int = 0, sink=None):
    """Causal latent attention over whole sequences.  ``q`` ``[B,S,H,dim+rot]``, ``kv`` ``[B,S,H*(dim+vdim)]`` (the
    unrotated keys of all heads, then the values of all heads), ``lat`` ``[B,S,width]`` whose entries
    ``rank .. rank+rot`` are the shared rotated key part.  Returns ``[B,S,H*vdim]``."""
    B, S, H, E = q.shape
    rot = E - dim
    kn = kv[..., :H * dim].reshape(B, S, H, dim).float()
    v = kv[..., H * dim:].reshape(B, S, H, vdim).float()
    kr = lat[..., rank:rank + rot].float()
    scores = (torch.einsum("bihd,bjhd->bhij", q[..., :dim].float(), kn)
              + torch.einsum("bihr,bjr->bhij", q[..., dim:].float(), kr)) * scale
    i = torch.arange(S, device=q.device)
    ok = i[None, :] <= i[:, None]
    if window and window > 0:
        ok &= i[:, None] - i[None, :] < window
    p = _sink_softmax(scores.masked_fill(~ok, float("-inf")), sink)
    return torch.einsum("bhij,bjhd->bihd", p, v).reshape(B, S, H * vdim).to(q.dtype)


def latent_decode(q, uk_t, uv, cache, count, *, rank: int, scale: float, sink=None):
    """One query per row against cached latent rows, with the key and value up projections absorbed: ``q``
    ``[B,H,dim+rot]``, ``uk_t`` ``[H,rank,dim]``, ``uv`` ``[H,vdim,rank]``, ``cache`` ``[B,slots,width]`` of which the
    first ``count[b]`` slots are occupied.  Returns ``[B,H*vdim]``."""
    B, H, E = q.shape
    dim = uk_t.shape[2]
    qa = torch.einsum("bhd,hkd->bhk", q[..., :dim].float(), uk_t.float()).to(q.dtype).float()
    c, kr = cache[..., :rank].float(), cache[..., rank:rank + E - dim].float()
    scores = (torch.einsum("bhk,bsk->bhs", qa, c) + torch.einsum("bhr,bsr->bhs", q[..., dim:].float(), kr)) * scale
    ok = torch.arange(cache.shape[1], device=q.device)[None, :] < count[:, None]
    p = _sink_softmax(scores.masked_fill(~ok[:, None, :], float("-inf")), sink)
    ctx = torch.einsum("bhs,bsk->bhk", p, c).to(q.dtype).float()
    return torch.einsum("bhk,hvk->bhv", ctx, uv.float()).reshape(B, -1).to(q.dtype)


# --------------------------------------------- distance-biased attention ----
def bias_attention(q, k, bias, *, scale: float, window: int):
    """Causal sliding-window attention whose values are the keys: ``q`` ``[B,S,H,D]``, ``k`` ``[B,S,G,D]``, ``bias``
    ``[H,n]`` added to the scaled score of every distance ``0 .. min(window, S) - 1``.  Returns ``[B,S,H*D]``."""
    B, S, H, D = q.shape
    kf = k.float().repeat_interleave(H // k.shape[2], dim=2)
    n = torch.arange(S, device=q.device)
    d = n[:, None] - n[None, :]
    ok = (d >= 0) & (d < window)
    scores = torch.einsum("bihd,bjhd->bhij", q.float(), kf) * scale + bias.float()[:, d.clamp(0, bias.shape[1] - 1)]
    p = torch.softmax(scores.masked_fill(~ok, float("-inf")), dim=-1)
    return torch.einsum("bhij,bjhd->bihd", p, kf).reshape(B, S, H * D).to(q.dtype)


def bias_decode(q, k, cache, kv_len, bias, *, dim: int, scale: float, active=None):
    """One token per row at position ``kv_len[b]``: ``q`` ``[B,H*dim]``, its own key ``k`` ``[B,G*dim]`` goes to slot
    ``kv_len[b] % slots`` of the ring ``cache`` ``[B,slots,G*dim]`` (in place).  Rows that are not ``active`` attend to
    nothing and store nothing.  Returns ``[B,H*dim]``."""
    B, slots = cache.shape[0], cache.shape[1]
    pos = kv_len.long()
    rows = torch.arange(B, device=q.device)
    cur = pos % slots
    on = torch.ones(B, dtype=torch.bool, device=q.device) if active is None else active
    cache[rows, cur] = torch.where(on[:, None], k, cache[rows, cur])
    qh, kc = q.view(B, -1, dim).float(), cache.view(B, slots, -1, dim).float()
    kc = kc.repeat_interleave(qh.shape[1] // kc.shape[2], dim=2)
    dist = (cur[:, None] - torch.arange(slots, device=q.device)[None, :]) % slots
    ok = (dist <= pos[:, None]) & on[:, None]
    scores = torch.einsum("bhd,bshd->bhs", qh, kc) * scale + bias.float()[:, dist].transpose(0, 1)
    p = torch.nan_to_num(torch.softmax(scores.masked_fill(~ok[:, None], float("-inf")), dim=-1))
    return torch.einsum("bhs,bshd->bhd", p, kc).reshape(B, -1).to(q.dtype)


# ---------------------------------------------------- hyper-connections ----
def sinusoid_table(n: int, width: int) -> torch.Tensor:
    """``[n, width]`` float32: entry ``2i`` is ``sin(p * 10000^(-2i/width))``, entry ``2i+1`` the cosine."""
    i = torch.arange((width + 1) // 2, dtype=torch.float64)
    angle = torch.arange(n, dtype=torch.float64)[:, None] * 10000.0 ** (-2.0 * i / width)
    return torch.stack([angle.sin(), angle.cos()], dim=-1).reshape(n, -1)[:, :width].float()


def hyper_mix(x, y, mix, out):
    """Streams ``x`` ``[..., s, W]`` behind a sublayer with output ``y`` ``[..., W]``: stream ``t`` becomes
    ``sum_s mix[s, t] x_s + out[t] y`` (float32)."""
    return torch.einsum("st,...sw->...tw", mix.float(), x) + out.float()[:, None] * y.float()[..., None, :]


def hyper_norm(x, y, mix, out, inp, weight, eps, scale: float = 1.0):
    """``(streams, h)``: the streams behind the sublayer that gave ``y`` (``None``: as they are), and the RMS norm
    (weight around zero, times ``scale``) of what the next sublayer reads, ``sum_s inp[s] x_s`` (``inp=None``: the
    plain sum).  Float32."""
    if y is not None:
        x = hyper_mix(x, y, mix, out)
    u = x.sum(-2) if inp is None else torch.einsum("s,...sw->...w", inp.float(), x)
    h = u * torch.rsqrt(u.pow(2).mean(-1, keepdim=True) + eps) * (1.0 + weight.float())
    return x, h if scale == 1.0 else h * scale


# ------------------------------------------------ state-space duality ----
def ssm_conv(x, w, bias):
    """Causal convolution per channel and SiLU: ``x`` ``[B,L,C]``, ``w`` ``[C,K]`` whose last column meets the current
    token, zeros before the start."""
    xf = F.pad(x.float().transpose(1, 2), (w.shape[1] - 1, 0))
    y = F.conv1d(xf, w.float().unsqueeze(1), None if bias is None else bias.float(), groups=x.shape[2])
    return F.silu(y).transpose(1, 2).to(x.dtype)


def ssm_scan(u, dt, dt_bias, A_log, D, lens, *, heads: int, state: int, groups: int, chunk: int = 64):
    """Selective scan of ``u = [x | B | C]`` ``[B,T,H*P + 2*G*N]`` with raw step sizes ``dt`` ``[B,T,H]``, in chunks whose
    products are matrices; float32 inside.  Tokens at or past ``lens[b]`` leave the state alone.  Returns ``(y [B,T,H*P],
    state [B,H,N,P])``."""
    Bn, T, _ = u.shape
    inner = u.shape[2] - 2 * groups * state
    P, rep = inner // heads, heads // groups
    uf = u.float()
    x = uf[..., :inner].reshape(Bn, T, heads, P)
    Bm = uf[..., inner:inner + groups * state].reshape(Bn, T, groups, state).repeat_interleave(rep, dim=2)
    Cm = uf[..., inner + groups * state:].reshape(Bn, T, groups, state).repeat_interleave(rep, dim=2)
    step = F.softplus(dt.float() + dt_bias.float())
    if lens is not None:
        step = step * (torch.arange(T, device=u.device)[None, :] < lens[:, None])[..., None]
    la = -torch.exp(A_log.float()) * step
    S = x.new_zeros(Bn, heads, state, P)
    ys = []
    for t0 in range(0, T, chunk):
        xc, bc, cc = x[:, t0:t0 + chunk], Bm[:, t0:t0 + chunk], Cm[:, t0:t0 + chunk]
        cum = la[:, t0:t0 + chunk].cumsum(1).transpose(1, 2)                     # [B,H,L]
        xs = (xc * step[:, t0:t0 + chunk, :, None]).transpose(1, 2)              # [B,H,L,P]
        L = cum.shape[-1]
        seg = cum[..., :, None] - cum[..., None, :]
        seg = seg.masked_fill(~torch.ones(L, L, dtype=torch.bool, device=u.device).tril(), float("-inf"))
        scores = torch.einsum("bthn,bshn->bhts", cc, bc) * torch.exp(seg)
        y = scores @ xs + torch.einsum("bthn,bhnp->bhtp", cc, S) * torch.exp(cum)[..., None]
        left = torch.exp(cum[..., -1:] - cum)
        S = S * torch.exp(cum[..., -1])[..., None, None] + torch.einsum("bshn,bhsp->bhnp", bc, xs * left[..., None])
        ys.append(y.transpose(1, 2) + D.float()[:, None] * xc)
    return torch.cat(ys, 1).reshape(Bn, T, inner).to(u.dtype), S


def ssm_step(x, dt, conv_w, conv_b, dt_bias, A_log, D, ring, S, kv_len, active, *, groups: int):
    """One token per row at position ``kv_len[b]``: convolution inputs ``x`` ``[B,C]`` against the ring of the last ``K``
    inputs ``ring`` ``[B,K,C]`` (slot = position mod K), then the state update; ``ring`` and ``S`` ``[B,H,N,P]`` change in
    place, except for rows that are not ``active``.  Returns ``y`` ``[B,H*P]``."""
    Bn, K, _ = ring.shape
    H, N, P = S.shape[1:]
    rows, pos = torch.arange(Bn, device=x.device), kv_len.long()
    on = torch.ones(Bn, dtype=torch.bool, device=x.device) if active is None else active
    ring[rows, pos % K] = torch.where(on[:, None], x, ring[rows, pos % K])
    acc = torch.zeros(x.shape, dtype=torch.float32, device=x.device) + (0.0 if conv_b is None else conv_b.float())
    for j in range(K):
        past = ring[rows, (pos - j) % K].float() * (pos >= j)[:, None]
        acc = acc + conv_w[:, K - 1 - j].float() * past
    u = F.silu(acc).to(x.dtype).float()
    inner = H * P
    xv = u[:, :inner].view(Bn, H, P)
    Bm = u[:, inner:inner + groups * N].view(Bn, groups, N).repeat_interleave(H // groups, dim=1)
    Cm = u[:, inner + groups * N:].view(Bn, groups, N).repeat_interleave(H // groups, dim=1)
    step = F.softplus(dt.float() + dt_bias.float())
    new = S * torch.exp(-torch.exp(A_log.float()) * step)[..., None, None] + (Bm * step[..., None])[..., None] * xv[:, :, None, :]
    S.copy_(torch.where(on[:, None, None, None], new, S))
    y = torch.einsum("bhnp,bhn->bhp", new, Cm) + D.float()[:, None] * xv
    return (y.reshape(Bn, inner) * on[:, None]).to(x.dtype)


def gated_group_norm(y, z, weight, groups: int, eps: float):
    """``y * silu(z)``, each of ``groups`` equal parts divided by its own root mean square, times ``weight``."""
    v = y.float() * F.silu(z.float())
    p = v.unflatten(-1, (groups, -1))
    p = p * torch.rsqrt(p.pow(2).mean(-1, keepdim=True) + eps)
    return (p.flatten(-2) * weight.float()).to(y.dtype)


# ------------------------------------------------------------ mlp / act ----
@dataclass(frozen=True)
class ClippedGlu:
    """Gated activation ``g * sigmoid(alpha g) * (u + 1)`` with ``g = min(gate, limit)``, ``u = clamp(up, +-limit)``."""
    limit: float
    alpha: float = 1.702


def swiglu(gate_up: torch.Tensor, act="silu"):
    """``act(gate) * up`` on a fused ``[..., 2F]`` tensor laid out ``[gate | up]``; ``act`` is a name or a
    ``ClippedGlu``."""
    g, u = gate_up.chunk(2, dim=-1)
    if isinstance(act, ClippedGlu):
        gf, uf = g.float().clamp(max=act.limit), u.float().clamp(-act.limit, act.limit)
        return (gf * torch.sigmoid(act.alpha * gf) * (uf + 1.0)).to(gate_up.dtype)
    if act == "silu":
        a = F.silu(g.float())
    elif act in ("gelu_pytorch_tanh", "gelu_tanh"):
        a = F.gelu(g.float(), approximate="tanh")
    elif act == "gelu":
        a = F.gelu(g.float())
    else:
        raise ValueError(f"unsupported activation {act}")
    return (a * u.float()).to(gate_up.dtype)


# ----------------------------------------------------------------- lora ----
def lora_linear(x, w, a_stack, b_stack, bias=None):
    """``y = x Wᵀ + (x Aᵀ) Bᵀ``; ``a_stack`` ``[R, in]``, ``b_stack`` ``[out, R]``
    already carry the LoRA scale (in ``b_stack``). Either may be ``None``."""
    y = F.linear(x, w, bias)
    if a_stack is not None:
        t = F.linear(x, a_stack.to(x.dtype))
        y = y + F.linear(t, b_stack.to(x.dtype))
    return y


def linear_f32(x, w):
    """``x Wᵀ`` accumulated and returned in float32 (router logits, vocabulary logits)."""
    return F.linear(x.float(), w.float())


def lora_merge(w, a_stack, b_stack):
    """``W + B A`` in fp32, cast to ``w.dtype`` (reference lora.rs:1335-1350)."""
    if a_stack is None:
        return w
    return (w.float() + b_stack.float() @ a_stack.float()).to(w.dtype)


# -------------------------------------------------------------- logprob ----
def logprob_gather(hidden, head_w, targets, temperature: float = 1.0, softcap: float = 0.0,
                   chunk: int = 128):
    """Per-token ``log_softmax(h Wᵀ / T)[target]`` without keeping ``[N, V]``
    beyond one chunk of rows (reference model.rs:523-559). ``hidden`` ``[N, H]``,
    ``targets`` ``[N]`` -> ``[N]`` float32.  ``softcap>0`` applies
    ``cap*tanh(x/cap)`` to the logits first (Gemma)."""
    outs = []
    for s in range(0, hidden.shape[0], chunk):
        h = hidden[s:s + chunk]
        logits = F.linear(h, head_w).float()
        if softcap and softcap > 0:
            logits = softcap * torch.tanh(logits / softcap)
        logits = logits / temperature
        lp = torch.log_softmax(logits, dim=-1)
        outs.append(lp.gather(-1, targets[s:s + chunk, None].long()).squeeze(-1))
    return torch.cat(outs) if outs else hidden.new_zeros(0, dtype=torch.float32)


def embedding(ids, table, scale: float = 1.0):
    e = F.embedding(ids, table)
    return e if scale == 1.0 else (e.float() * scale).to(e.dtype)


# ---------------------------------------------------------------- adamw ----
def adamw_step(params, grads, m, v, *, lr, beta1, beta2, eps, weight_decay, step, grad_scale=1.0):
    """Decoupled AdamW, epsilon outside the square root, bias correction by
    step count (reference optim.rs:257-296).  In place on lists of fp32 tensors."""
    bc1 = 1.0 - beta1 ** step
    bc2 = 1.0 - beta2 ** step
    for p, g, mi, vi in zip(params, grads, m, v):
        g = g * grad_scale if grad_scale != 1.0 else g
        if weight_decay != 0.0:
            p.mul_(1.0 - lr * weight_decay)
        mi.mul_(beta1).add_(g, alpha=1.0 - beta1)
        vi.mul_(beta2).addcmul_(g, g, value=1.0 - beta2)
        denom = (vi / bc2).sqrt_().add_(eps)
        p.addcdiv_(mi / bc1, denom, value=-lr)
