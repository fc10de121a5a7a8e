"""Small random Galodra checkpoints for the tests: configurations, seeded weights, a safetensors writer."""
import json
import struct

import torch


def mixer(heads, dim, rot, vdim, rank, window, base=1e4, turned=None, scale=None):
    return {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "mask": {"size": window},
            "rot": {"base": base, "dims": turned or rot}, "scale": scale or (dim + rot) ** -0.5}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def config(vocab, width, layers, alpha=1.5, eps=1e-5):
    return {"architecture": "Galodra", "vocab": vocab, "width": width, "norm": {"eps": eps}, "postln_alpha": alpha,
            "layers": [{"type": "latent_attention", "mixer": m, "mlp": f} for m, f in layers]}


# every kind of feed-forward, layers that differ in all sizes, several experts a token
MIXED = config(89, 64, [
    (mixer(3, 16, 8, 24, 40, window=7, base=300.0), moe(5, 2, 40)),
    (mixer(2, 24, 16, 16, 56, window=19), None),
    (mixer(5, 8, 8, 8, 16, window=1, base=50.0), dense(72)),
    (mixer(2, 16, 24, 32, 24, window=33, base=1e6, scale=0.3), moe(3, 3, 24)),
], alpha=0.7)
# nothing is a multiple of eight
ODD = config(61, 36, [
    (mixer(3, 5, 6, 7, 11, window=5, base=77.0, turned=4), dense(27)),
    (mixer(1, 9, 2, 3, 13, window=12), moe(7, 1, 17)),
], alpha=3.0, eps=1e-3)
# one layer, one head, one expert, a window longer than the tests' sequences
ONE = config(40, 32, [(mixer(1, 8, 8, 16, 8, window=500), moe(1, 1, 16))], alpha=1.0)
# sizes for the tensor-core kernels: whole 64-column atoms, more than 16 heads, wide latents
WIDE = config(160, 128, [
    (mixer(20, 64, 32, 64, 128, window=70), dense(128)),
    (mixer(4, 128, 64, 128, 192, window=130), moe(3, 3, 64)),
    (mixer(2, 96, 16, 136, 72, window=17), None),
], alpha=1.2)
CASES = {"mixed": MIXED, "odd": ODD, "one": ONE, "wide": WIDE}


def weights(cfg, seed):
    """bf16 tensors under their checkpoint names; spread so that attention is far from uniform, gates, sinks and
    depth coefficients matter and the streams stay of order one."""
    g = torch.Generator().manual_seed(seed)
    W = cfg["width"]
    out = {}

    def put(name, *shape, std=1.0, mean=0.0):
        out[name] = (torch.randn(shape, generator=g) * std + mean).to(torch.bfloat16)

    def linear(name, o, i, gain=1.0):
        put(name, o, i, std=gain * i ** -0.5)

    put("embed", cfg["vocab"], W, std=1.0)
    put("final.norm", W, std=0.1, mean=1.0)
    put("final.norm.b", W, std=0.1)
    for i, l in enumerate(cfg["layers"]):
        p, m, f = f"l{i}.", l["mixer"], l["mlp"]
        linear(p + "mix.q", m["heads"] * (m["dim"] + m["rot_dim"]), W, 2.0)
        linear(p + "mix.dkv", m["kv_rank"] + m["rot_dim"], W, 1.5)
        put(p + "mix.dkv.norm", m["kv_rank"], std=0.2, mean=1.0)
        linear(p + "mix.uk", m["heads"] * m["dim"], m["kv_rank"], 1.5)
        linear(p + "mix.uv", m["heads"] * m["vdim"], m["kv_rank"], 2.0)
        put(p + "mix.sink", m["heads"], std=1.5, mean=0.5)
        linear(p + "mix.o", W, m["heads"] * m["vdim"], 2.0)
        for n in ("1", "2") if f is not None else ("1",):
            put(p + f"norm{n}", W, std=0.2, mean=1.0)
            put(p + f"norm{n}.b", W, std=0.2)
            linear(p + f"rg{n}", W, W, 1.5)
            put(p + f"rg{n}.b", W, std=0.5)
        put(p + "dwa", i + 2, std=0.3, mean=0.2)
        if f is None:
            continue
        if f["kind"] == "dense":
            linear(p + "mlp.gate", f["ff"], W, 1.5)
            linear(p + "mlp.up", f["ff"], W, 1.5)
            linear(p + "mlp.down", W, f["ff"], 2.0)
        else:
            linear(p + "mlp.router", f["router"]["experts"], W, 2.0)
            for e in range(f["router"]["experts"]):
                linear(p + f"mlp.e{e}.gate", f["expert"]["ff"], W, 2.0)
                linear(p + f"mlp.e{e}.up", f["expert"]["ff"], W, 2.0)
                linear(p + f"mlp.e{e}.down", W, f["expert"]["ff"], 2.0)
    return out


def write(folder, cfg, tensors):
    head, blobs, at = {}, [], 0
    for name, t in tensors.items():
        raw = t.contiguous().view(torch.int16).numpy().tobytes()
        head[name] = {"dtype": "BF16", "shape": list(t.shape), "data_offsets": [at, at + len(raw)]}
        blobs.append(raw)
        at += len(raw)
    text = json.dumps(head).encode()
    with open(f"{folder}/model.safetensors", "wb") as f:
        f.write(struct.pack("<Q", len(text)) + text + b"".join(blobs))
    with open(f"{folder}/config.json", "w") as f:
        json.dump(cfg, f)
    return str(folder)
