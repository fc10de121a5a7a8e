"""Small random Mifutar checkpoints for the tests: configurations and seeded weights."""
import torch

from galodra_cases import write  # noqa: F401


def attn(heads, kv, dim, window, bias_max, scale=None):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": dim, "bias_max": bias_max,
                                           "mask": {"size": window}, "scale": scale or dim ** -0.5}}


def ssm(heads, vdim, state, groups, conv, norm_groups):
    return {"type": "mamba2", "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups}}


def ff(n, limit):
    return {"kind": "dense", "ff": n, "limit": limit}


def config(vocab, width, layers, streams, eps=1e-5, logit_scale=0.5):
    return {"architecture": "Mifutar", "vocab": vocab, "width": width, "streams": streams, "norm": {"eps": eps}, "logit_scale": logit_scale,
            "layers": [dict(l, mlp=f) for l, f in layers]}


# layers that differ in all sizes, three streams, a window shorter than the exact buckets and one beyond the last
MIXED = config(89, 64, [
    (ssm(4, 24, 16, 2, 4, 2), ff(40, 0.8)),
    (attn(6, 2, 16, 7, 20), None),
    (ssm(3, 8, 40, 1, 2, 3), None),
    (attn(2, 2, 24, 33, 19, scale=0.5), ff(72, 1.5)),
], streams=3)
# nothing is a multiple of eight, one stream, one tap, one token of window
ODD = config(61, 36, [
    (ssm(5, 7, 11, 5, 1, 7), ff(27, 0.5)),
    (attn(3, 1, 9, 1, 9), ff(13, 2.0)),
    (attn(3, 3, 5, 12, 6), None),
    (ssm(2, 3, 5, 1, 6, 1), ff(9, 1.0)),
], streams=1, eps=1e-3, logit_scale=1.0)
# one head each, five streams, a window longer than the tests' sequences
ONE = config(40, 32, [(attn(1, 1, 8, 500, 100), ff(16, 1.2)), (ssm(1, 16, 8, 1, 3, 4), ff(16, 0.3))], streams=5, logit_scale=1.7)
# sizes for the tensor-core kernels
WIDE = config(160, 128, [
    (ssm(4, 64, 128, 1, 4, 4), ff(128, 1.0)),
    (attn(8, 2, 64, 70, 60), ff(64, 0.7)),
    (ssm(8, 32, 64, 4, 4, 1), ff(128, 1.3)),
    (attn(4, 1, 128, 130, 110), None),
    (ssm(2, 128, 16, 2, 3, 1), None),
], streams=2)
CASES = {"mixed": MIXED, "odd": ODD, "one": ONE, "wide": WIDE}
BUCKETS = {"mixed": 8, "odd": 6, "one": 32, "wide": 24}


def weights(cfg, seed, buckets=8):
    """bf16 tensors under their checkpoint names; spread so that attention is far from uniform, biases, decays, gates and
    stream coefficients matter, clips are reached and the streams stay of order one."""
    g = torch.Generator().manual_seed(seed)
    W, s = cfg["width"], cfg["streams"]
    out = {}

    def put(name, *shape, std=1.0, mean=0.0):
        out[name] = (torch.randn(shape, generator=g) * std + mean).to(torch.bfloat16)

    def linear(name, o, i, gain=1.0):
        put(name, o, i, std=gain * i ** -0.5)

    put("embed", cfg["vocab"], W)
    linear("head", cfg["vocab"], W, 2.0)
    put("final.norm", W, std=0.2)
    for i, l in enumerate(cfg["layers"]):
        p, m = f"l{i}.", l["mixer"]
        for q in ("1", "2") if l["mlp"] is not None else ("1",):
            put(p + f"norm{q}", W, std=0.3)
            put(p + f"hc{q}.in", s, std=0.4, mean=1.0 / s)
            put(p + f"hc{q}.out", s, std=0.4, mean=0.7)
            put(p + f"hc{q}.mix", s, s, std=0.15)
            out[p + f"hc{q}.mix"] += 0.85 * torch.eye(s, dtype=torch.bfloat16)
        if l["type"] == "attention":
            nq, nk = m["heads"] * m["dim"], m["kv_heads"] * m["dim"]
            linear(p + "mix.q", nq, W, 1.6)
            put(p + "mix.q.b", nq, std=0.5)
            linear(p + "mix.k", nk, W, 1.6)
            put(p + "mix.k.b", nk, std=0.5)
            put(p + "mix.rel", buckets, m["heads"], std=1.2)
            linear(p + "mix.o", W, nq, 2.0)
        else:
            inner, ch = m["heads"] * m["vdim"], m["heads"] * m["vdim"] + 2 * m["groups"] * m["state"]
            linear(p + "mix.in", inner + ch + m["heads"], W, 1.5)
            put(p + "mix.conv", ch, m["conv"], std=m["conv"] ** -0.5)
            put(p + "mix.conv.b", ch, std=0.3)
            put(p + "mix.dt_bias", m["heads"], std=1.0, mean=-1.0)
            put(p + "mix.A_log", m["heads"], std=1.0, mean=-0.5)
            put(p + "mix.D", m["heads"], std=0.5, mean=1.0)
            put(p + "mix.norm", inner, std=0.2, mean=1.0)
            linear(p + "mix.o", W, inner, 2.0)
        if l["mlp"] is not None:
            n = l["mlp"]["ff"]
            linear(p + "mlp.gate", n, W, 1.5)
            linear(p + "mlp.up", n, W, 1.5)
            linear(p + "mlp.down", W, n, 2.0)
    return out
