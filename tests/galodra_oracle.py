"""Plain, slow restatement of the Galodra decoder, one function per mechanism.

Nothing here is shared with the product path: weights are a dict of tensors under their checkpoint names, a sequence
is a 1-D list of token ids, every position is computed from scratch and loops are written out.  ``dt`` is the
arithmetic type (float64 by default, so that the oracle's own rounding never matters)."""
import json
import math
import struct

import torch


def read_checkpoint(folder):
    """``(config, {name: tensor})`` from ``config.json`` and a one-file safetensors container."""
    with open(f"{folder}/config.json") as f:
        cfg = json.load(f)
    with open(f"{folder}/model.safetensors", "rb") as f:
        (n,) = struct.unpack("<Q", f.read(8))
        head = json.loads(f.read(n))
        body = f.read()
    kinds = {"BF16": torch.bfloat16, "F32": torch.float32, "I32": torch.int32}
    out = {}
    for name, d in head.items():
        if name == "__metadata__":
            continue
        lo, hi = d["data_offsets"]
        out[name] = torch.frombuffer(bytearray(body[lo:hi]), dtype=kinds[d["dtype"]]).reshape(d["shape"])
    return cfg, out


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z):
    return z / (1 + torch.exp(-z))


def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def layer_norm(x, w, b, eps):
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w + b


def rotate(x, positions, dims, base):
    """Rotate-half on the first ``dims`` entries of the last axis of ``x`` ``[T, ..., D]``."""
    cols = [x[..., i] for i in range(x.shape[-1])]
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        shape = [-1] + [1] * (x.dim() - 2)
        c = torch.tensor([math.cos(p * f) for p in positions], dtype=x.dtype).view(shape)
        s = torch.tensor([math.sin(p * f) for p in positions], dtype=x.dtype).view(shape)
        u, v = x[..., i], x[..., i + dims // 2]
        cols[i], cols[i + dims // 2] = u * c - v * s, v * c + u * s
    return torch.stack(cols, -1)


def sink_softmax(scores, sink):
    """Weights over the last axis of ``scores`` ``[H, n]`` whose denominators also hold ``exp(sink[h])``."""
    m = torch.maximum(scores.max(-1).values, sink).detach()
    e = torch.exp(scores - m[:, None])
    return e / (e.sum(-1) + torch.exp(sink - m))[:, None]


def visible(i, window):
    return list(range(max(0, i - window + 1), i + 1))


def attend(qn, qr, kn, kr, v, scale, window, sink):
    """``qn`` ``[T,H,D]``, ``qr`` ``[T,H,R]``, ``kn`` ``[T,H,D]``, ``kr`` ``[T,R]``, ``v`` ``[T,H,V]`` -> ``[T,H,V]``."""
    rows = []
    for i in range(qn.shape[0]):
        js = visible(i, window)
        s = (torch.einsum("hd,jhd->hj", qn[i], kn[js]) + torch.einsum("hr,jr->hj", qr[i], kr[js])) * scale
        rows.append(torch.einsum("hj,jhv->hv", sink_softmax(s, sink), v[js]))
    return torch.stack(rows)


def latent_attention(h, w, p, mx, eps):
    """``h`` ``[T, width]``; ``p`` is the tensor prefix, ``mx`` the mixer's configuration."""
    H, D, R, V, K = mx["heads"], mx["dim"], mx["rot_dim"], mx["vdim"], mx["kv_rank"]
    T, rot = h.shape[0], mx["rot"]
    q = (h @ w[p + "q"].T).reshape(T, H, D + R)
    kv = h @ w[p + "dkv"].T
    c = rms_norm(kv[:, :K], w[p + "dkv.norm"], eps)
    kn = (c @ w[p + "uk"].T).reshape(T, H, D)
    v = (c @ w[p + "uv"].T).reshape(T, H, V)
    o = attend(q[..., :D], rotate(q[..., D:], range(T), rot["dims"], rot["base"]), kn,
               rotate(kv[:, K:], range(T), rot["dims"], rot["base"]), v, mx["scale"], mx["mask"]["size"], w[p + "sink"])
    return o.reshape(T, H * V) @ w[p + "o"].T


def dense_ff(h, w, p):
    return (gelu_tanh(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def route(h, w, p, top):
    """Per token: the chosen experts and their (not renormalised) sigmoid scores."""
    s = 1 / (1 + torch.exp(-(h @ w[p + "router"].T)))
    picks = []
    for t in range(h.shape[0]):
        order = sorted(range(s.shape[1]), key=lambda e: (-s[t, e].item(), e))[:top]
        picks.append([(e, s[t, e]) for e in order])
    return picks


def expert(h, w, p):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def moe_ff(h, w, p, top):
    rows = []
    for t, pick in enumerate(route(h, w, p, top)):
        rows.append(sum(expert(s * h[t], w, f"{p}e{e}.") for e, s in pick))
    return torch.stack(rows)


def residual_gate(h, w, name):
    return 1 / (1 + torch.exp(-(h @ w[name].T + w[name + ".b"])))


def depth_average(history, coef):
    out = torch.zeros_like(history[0])
    for j, x in enumerate(history):
        out = out + coef[j] * x
    return out


def layer(x, w, i, lc, cfg):
    p, eps, alpha = f"l{i}.", cfg["norm"]["eps"], cfg["postln_alpha"]
    y = latent_attention(x, w, p + "mix.", lc["mixer"], eps) * residual_gate(x, w, p + "rg1")
    x = layer_norm(alpha * x + y, w[p + "norm1"], w[p + "norm1.b"], eps)
    if lc["mlp"] is None:
        return x
    if lc["mlp"]["kind"] == "dense":
        y = dense_ff(x, w, p + "mlp.")
    else:
        y = moe_ff(x, w, p + "mlp.", lc["mlp"]["router"]["top"])
    y = y * residual_gate(x, w, p + "rg2")
    return layer_norm(alpha * x + y, w[p + "norm2"], w[p + "norm2.b"], eps)


def forward(tokens, weights, cfg, dt=torch.float64, layers_out=None):
    """Logits ``[T, vocab]`` of one sequence."""
    w = {k: v.to(dt) for k, v in weights.items()}
    x = w["embed"][list(tokens)]
    history = [x]
    for i, lc in enumerate(cfg["layers"]):
        history.append(layer(x, w, i, lc, cfg))
        x = depth_average(history, w[f"l{i}.dwa"])
        if layers_out is not None:
            layers_out.append(x)
    x = layer_norm(x, w["final.norm"], w["final.norm.b"], cfg["norm"]["eps"])
    return x @ w["embed"].T
