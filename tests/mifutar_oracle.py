"""Plain, slow restatement of the Mifutar decoder, one function per mechanism.

Nothing here is shared with the product path: weights are a dict of tensors under their checkpoint names, a sequence
is a 1-D list of token ids, every position is computed from scratch and the recurrence walks token by token.  ``dt`` is
the arithmetic type (float64 by default, so that the oracle's own rounding never matters)."""
import math

import torch

from galodra_oracle import read_checkpoint, silu, visible  # noqa: F401


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm(x, w, eps):
    """Weight stored around zero."""
    return rms(x, eps) * (1 + w)


def sinusoid(p, width):
    v = []
    for c in range(width):
        a = p * 10000.0 ** (-2 * (c // 2) / width)
        v.append(math.cos(a) if c % 2 else math.sin(a))
    return torch.tensor(v, dtype=torch.float64)


# ------------------------------------------------------------------------------------------------ distance-biased attention
def bucket(n, buckets, far):
    """The first half of the buckets hold one distance each, the others grow geometrically up to ``far``."""
    half = buckets // 2
    if n < half:
        return n
    # k is the largest integer with (far / half)^k <= (n / half)^(buckets - half), compared in integers
    m, k = buckets - half, 0
    while k < m and far ** (k + 1) * half ** m <= n ** m * half ** (k + 1):
        k += 1
    return min(buckets - 1, half + k)


def attend(q, k, bias_of, scale, window):
    """``q`` ``[T,H,D]``, ``k`` ``[T,G,D]``; the values are the keys.  ``bias_of(distance)`` is ``[H]``."""
    T, H, _ = q.shape
    own = [h // (H // k.shape[1]) for h in range(H)]
    rows = []
    for i in range(T):
        js = visible(i, window)
        kk = k[js][:, own]
        s = torch.einsum("hd,jhd->hj", q[i], kk) * scale + torch.stack([bias_of(i - j) for j in js], 1)
        rows.append(torch.einsum("hj,jhd->hd", torch.softmax(s, -1), kk))
    return torch.stack(rows)


def attention(h, w, p, mx):
    H, G, D = mx["heads"], mx["kv_heads"], mx["dim"]
    T = h.shape[0]
    q = (h @ w[p + "q"].T + w[p + "q.b"]).reshape(T, H, D)
    k = (h @ w[p + "k"].T + w[p + "k.b"]).reshape(T, G, D)
    rel = w[p + "rel"]
    o = attend(q, k, lambda n: rel[bucket(n, rel.shape[0], mx["bias_max"])], mx["scale"], mx["mask"]["size"])
    return o.reshape(T, H * D) @ w[p + "o"].T


# ------------------------------------------------------------------------------------------------ state-space duality
def conv(x, w, b):
    """Causal convolution per channel; the last column of ``w`` meets the current token."""
    K = w.shape[1]
    rows = []
    for t in range(x.shape[0]):
        acc = b.clone()
        for j in range(K):
            if t - (K - 1 - j) >= 0:
                acc = acc + w[:, j] * x[t - (K - 1 - j)]
        rows.append(silu(acc))
    return torch.stack(rows)


def softplus(z):
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


def scan(x, B, C, dt, A_log, D, state=None):
    """``x`` ``[T,H,P]``, ``B`` and ``C`` ``[T,G,N]``, step sizes ``dt`` ``[T,H]`` -> ``(y [T,H,P], state [H,N,P])``."""
    T, H, P = x.shape
    own = [h // (H // B.shape[1]) for h in range(H)]
    S = x.new_zeros(H, B.shape[2], P) if state is None else state
    ys = []
    for t in range(T):
        decay = torch.exp(-torch.exp(A_log) * dt[t])
        S = decay[:, None, None] * S + dt[t][:, None, None] * B[t][own][:, :, None] * x[t][:, None, :]
        ys.append(torch.einsum("hnp,hn->hp", S, C[t][own]) + D[:, None] * x[t])
    return torch.stack(ys), S


def gated_norm(y, z, w, groups, eps):
    y = y * silu(z)
    return rms(y.reshape(*y.shape[:-1], groups, -1), eps).reshape(y.shape) * w


def mamba2(h, w, p, mx, eps):
    H, P, N, G = mx["heads"], mx["vdim"], mx["state"], mx["groups"]
    T, inner = h.shape[0], H * P
    z, x, B, C, dt = torch.split(h @ w[p + "in"].T, [inner, inner, G * N, G * N, H], -1)
    u = conv(torch.cat([x, B, C], -1), w[p + "conv"], w[p + "conv.b"])
    x, B, C = torch.split(u, [inner, G * N, G * N], -1)
    y, _ = scan(x.reshape(T, H, P), B.reshape(T, G, N), C.reshape(T, G, N), softplus(dt + w[p + "dt_bias"]), w[p + "A_log"], w[p + "D"])
    return gated_norm(y.reshape(T, inner), z, w[p + "norm"], mx["norm_groups"], eps) @ w[p + "o"].T


# ------------------------------------------------------------------------------------------------ the rest of a layer
def clipped_glu(g, u, limit):
    g, u = torch.clamp(g, max=limit), torch.clamp(u, -limit, limit)
    return g / (1 + torch.exp(-1.702 * g)) * (u + 1)


def feed_forward(h, w, p, limit):
    return clipped_glu(h @ w[p + "gate"].T, h @ w[p + "up"].T, limit) @ w[p + "down"].T


def hyper(xs, w, p, sublayer):
    """``xs``: the streams, a list of ``[T, width]``."""
    u = sum(w[p + "in"][s] * x for s, x in enumerate(xs))
    y = sublayer(u)
    return [sum(w[p + "mix"][s, t] * x for s, x in enumerate(xs)) + w[p + "out"][t] * y for t in range(len(xs))]


def layer(xs, w, i, lc, cfg):
    p, eps, mx = f"l{i}.", cfg["norm"]["eps"], lc["mixer"]

    def mixer(u):
        h = norm(u, w[p + "norm1"], eps)
        return attention(h, w, p + "mix.", mx) if lc["type"] == "attention" else mamba2(h, w, p + "mix.", mx, eps)
    xs = hyper(xs, w, p + "hc1.", mixer)
    if lc["mlp"] is None:
        return xs
    return hyper(xs, w, p + "hc2.", lambda u: feed_forward(norm(u, w[p + "norm2"], eps), w, p + "mlp.", lc["mlp"]["limit"]))


def forward(tokens, weights, cfg, dt=torch.float64, layers_out=None):
    """Logits ``[T, vocab]`` of one sequence."""
    w = {k: v.to(dt) for k, v in weights.items()}
    x = w["embed"][list(tokens)] + torch.stack([sinusoid(p, cfg["width"]) for p in range(len(tokens))]).to(dt)
    xs = [x] * cfg["streams"]
    for i, lc in enumerate(cfg["layers"]):
        xs = layer(xs, w, i, lc, cfg)
        if layers_out is not None:
            layers_out.append(sum(xs))
    return norm(sum(xs), w["final.norm"], cfg["norm"]["eps"]) @ w["head"].T * cfg["logit_scale"]
