"""The Mifutar family against its plain restatement (``mifutar_oracle.py``): every mechanism by itself, whole prompts,
decoding through rings and recurrent states, batches, reused rows, generation, scoring gradients and trace replay.  Each
case runs on the CPU path and, marked ``gpu``, through the sm_100a kernels."""
import io
import json
import math
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import mifutar_cases as K
import mifutar_oracle as O
from family_helpers import _native, adapters, feed, near, prefill_all, rand, rms_near, row_errors, tokens  # noqa: F401

CPU = "cpu"
GPU = pytest.param("cuda", marks=pytest.mark.gpu)
F32, BF16 = torch.float32, torch.bfloat16
TOL = {F32: 3e-5, BF16: 3e-2}


def close(got, want, dtype):
    """bf16 results have entries of many sizes: rows are compared by their root mean square."""
    return near(got, want, TOL[F32]) if dtype == F32 else rms_near(got, want, 1e-2)


# ------------------------------------------------------------------------------------------------ mechanisms
@pytest.mark.parametrize("half,far", [(4, 9), (8, 128), (16, 128), (16, 129), (5, 6), (1, 50), (12, 4096), (3, 81)])
def test_distance_buckets(half, far):
    """Every distance, the exact powers where a bucket starts among them; an odd number of buckets too."""
    from ferrl_b200.models.bias_attention import BiasAttentionDims
    for buckets in (2 * half, 2 * half + 1):
        n = far + 40
        got = BiasAttentionDims(1, 1, 8, 1.0, n, buckets, far).bucket_of(n).tolist()
        assert got == [O.bucket(d, buckets, far) for d in range(n)]
        assert got[far:] == [buckets - 1] * 40 and got[:half] == list(range(half))
        for d in range(half, far):              # the formula itself, wherever it is not a tie
            v = half + math.log(d / half) / math.log(far / half) * (buckets - half)
            if abs(v - round(v)) > 1e-9:
                assert got[d] == min(buckets - 1, math.floor(v))


def loud(x, gain):
    return x * (gain / x.pow(2).sum(-1, keepdim=True).sqrt())


ATT = [  # query heads, key heads, dim, window, S
    (3, 1, 16, 5, 50), (6, 2, 64, 64, 200), (4, 4, 128, 129, 300), (2, 1, 40, 1, 70), (8, 2, 72, 128, 260), (4, 2, 5, 9, 40), (2, 2, 256, 100, 140),
    (1, 1, 8, 1000, 260), (16, 1, 64, 130, 390), (5, 5, 192, 63, 129)]


@pytest.mark.parametrize("device", [CPU, GPU])
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("shape", ATT)
def test_attention_over_sequences(device, dtype, shape):
    """Random keys, plus for some queries one loud key just inside the window, a louder one just outside or the query's
    own, and a bias table in which every distance is its own."""
    from ferrl_b200 import ops
    H, G, D, W, S = shape
    B, scale = 2, D ** -0.5
    q, k, bias = rand(B, S, H, D, seed=1), rand(B, S, G, D, seed=2), rand(H, W, seed=3)
    for i in range(W, S, 7):
        q[:, i] = loud(q[:, i], 3.0)
        for g in range(G):
            k[:, i - W + 1, g] = loud(q[:, i, g * (H // G)], 2.0 / scale)
            k[:, i - W, g] = loud(q[:, i, g * (H // G)], 4.0 / scale)
    q, k = q.to(dtype), k.to(dtype)

    def want(window):
        return torch.stack([O.attend(q[b].double(), k[b].double(), lambda n: bias[:, n].double(), scale, window) for b in range(B)]).reshape(B, S, -1)
    args = q.to(device), k.to(device), bias.to(device)
    near(ops.bias_attention(*args, scale=scale, window=W), want(W), 2 * TOL[dtype])
    if device == "cuda":
        from ferrl_b200.ops import cuda as C
        near(C.bias_attention(*args, scale=scale, window=W, variant=1), want(W), 2 * TOL[dtype])
        fused = rand(B, S, (H + G) * D + 8, seed=6, dtype=dtype).cuda()          # views of a wider projection
        fused[..., :H * D], fused[..., H * D:(H + G) * D] = q.flatten(2).cuda(), k.flatten(2).cuda()
        near(ops.bias_attention(fused[..., :H * D].unflatten(-1, (H, D)), fused[..., H * D:(H + G) * D].unflatten(-1, (G, D)), args[2], scale=scale,
                                window=W), want(W), 2 * TOL[dtype])


DEC = [  # query heads, key heads, dim, slots
    (3, 1, 16, 7), (6, 2, 64, 70), (33, 1, 64, 200), (2, 2, 8, 65), (4, 2, 5, 9), (8, 2, 128, 130), (16, 4, 128, 64), (5, 1, 256, 129),
    (4, 4, 96, 300), (2, 1, 64, 1)]


@pytest.mark.parametrize("device", [CPU, GPU])
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("shape", DEC)
def test_attention_of_one_token(device, dtype, shape):
    """Positions around a tile's and the ring's edge, before and behind its first turn, a retired row, loud keys in the
    newest, the oldest and a slot that holds nothing yet; the other slots stay as they are."""
    from ferrl_b200 import ops
    H, G, D, slots = shape
    lens = sorted({c for c in (0, 1, 31, 32, 63, 64, 65, 127, 128, slots - 2, slots - 1, slots, slots + 1, 2 * slots + 3) if c >= 0})
    B, scale = len(lens) + 1, D ** -0.5
    q, k, cache, bias = rand(B, H, D, seed=1), rand(B, G, D, seed=2), rand(B, slots, G, D, seed=3), rand(H, slots, seed=4, std=1.5)
    at = lens + [5 + slots]                                    # the last row is retired
    for b, p in enumerate(at):
        for g in range(G):
            one = loud(q[b, g * (H // G)], 2.0 / scale)
            cache[b, (p + 1) % slots, g] = 1.5 * one           # the oldest key, or a slot that was never written
            if b % 2:
                k[b, g] = one
    q, k, cache = q.to(dtype), k.to(dtype), cache.to(dtype)
    want = torch.zeros(B, H, D, dtype=torch.float64)
    after = cache.clone()
    for b, p in enumerate(lens):
        after[b, p % slots] = k[b]
        n = min(p + 1, slots)
        keys = torch.stack([after[b, (p - d) % slots] for d in range(n)]).double()        # by distance
        own = [h // (H // G) for h in range(H)]
        s = torch.einsum("hd,nhd->hn", q[b].double(), keys[:, own]) * scale + bias[:, :n].double()
        want[b] = torch.einsum("hn,nhd->hd", torch.softmax(s, -1), keys[:, own])
    on = torch.tensor([True] * len(lens) + [False])
    kv = torch.tensor(at, dtype=torch.int32)
    d = lambda t: t.to(device)  # noqa: E731
    pad = rand(B, 8, seed=9, dtype=dtype)
    fused = d(torch.cat([q.flatten(1), k.flatten(1), pad], 1))
    run = [lambda *a, **kw: ops.bias_decode(*a, **kw)]
    if device == "cuda":
        from ferrl_b200.ops import cuda as C
        run.append(lambda *a, **kw: C.bias_decode(*a, variant=1, **kw))
        run += [lambda *a, n=n, **kw: C.bias_decode(*a, splits=n, **kw) for n in (1, 2, 5)]
    for fn in run:
        ring = d(cache.flatten(2).clone())
        got = fn(fused[:, :H * D], fused[:, H * D:(H + G) * D], ring, d(kv), d(bias), dim=D, scale=scale, active=d(on))
        near(got, want.flatten(1), 2 * TOL[dtype])
        assert float(got[-1].abs().max()) == 0.0 and torch.equal(ring.cpu(), after.flatten(2))
    ring = d(cache.flatten(2).clone())
    got = ops.bias_decode(fused[:-1, :H * D], fused[:-1, H * D:(H + G) * D], ring[:-1], d(kv[:-1]), d(bias), dim=D, scale=scale)
    near(got, want[:-1].flatten(1), 2 * TOL[dtype])


@pytest.mark.parametrize("device", [CPU, GPU])
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("shape", [(24, 4, 37), (64, 2, 8), (13, 1, 5), (40, 3, 9), (9, 6, 21), (136, 4, 1), (16, 8, 3)])
def test_convolution(device, dtype, shape):
    from ferrl_b200 import ops
    C, taps, L = shape
    x, w, b = rand(2, L, C + 8, seed=1, dtype=dtype), rand(C, taps, seed=2), rand(C, seed=3)
    view = x.to(device)[..., 8:]
    for bias in (b, None):
        want = torch.stack([O.conv(x[i, :, 8:].double(), w.double(), (b if bias is not None else torch.zeros(C)).double()) for i in range(2)])
        near(ops.ssm_conv(view, w.to(device), None if bias is None else b.to(device)), want, TOL[dtype])


SCAN = [  # heads, columns, state, groups, tokens
    (4, 24, 16, 2, 70), (3, 8, 40, 1, 130), (5, 7, 11, 5, 33), (2, 64, 128, 1, 300), (8, 32, 64, 4, 129), (2, 128, 16, 2, 64), (1, 16, 8, 1, 1),
    (4, 48, 32, 2, 65), (6, 64, 64, 1, 257), (2, 64, 256, 2, 140), (2, 96, 48, 1, 200), (1, 33, 130, 1, 40)]


def scan_inputs(H, P, N, G, T, dtype, B=2):
    u = rand(B, T, H * P + 2 * G * N, seed=1, dtype=dtype)
    u[..., H * P:] *= N ** -0.25
    dt = rand(B, T, H, seed=2, dtype=dtype)
    return u, dt, rand(H, seed=3) - 1.5, rand(H, seed=4), rand(H, seed=5)


def scan_want(u, dt, dtb, A, D, H, P, N, G, lens):
    ys, Ss = [], []
    for b in range(u.shape[0]):
        n = lens[b]
        x, Bm, Cm = torch.split(u[b, :n].double(), [H * P, G * N, G * N], -1)
        y, S = O.scan(x.reshape(n, H, P), Bm.reshape(n, G, N), Cm.reshape(n, G, N), O.softplus(dt[b, :n].double() + dtb.double()), A.double(), D.double())
        ys.append(y.reshape(n, H * P))
        Ss.append(S)
    return ys, torch.stack(Ss)


@pytest.mark.parametrize("device", [CPU, GPU])
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("shape", SCAN)
def test_scan(device, dtype, shape):
    """Sequences of unequal lengths: outputs of the tokens that count and the final states; a fast-forgetting and a
    slow head side by side."""
    from ferrl_b200 import ops
    H, P, N, G, T = shape
    u, dt, dtb, A, D = scan_inputs(*shape, dtype)
    A[0], A[-1] = 3.0, -4.0
    lens = [T, max(1, T - 9)]
    ys, S = scan_want(u, dt, dtb, A, D, H, P, N, G, lens)
    args = [t.to(device) for t in (u, dt, dtb, A, D)]
    run = [lambda *a, **kw: ops.ssm_scan(*a, **kw)]
    if device == "cuda":
        from ferrl_b200.ops import cuda as C
        run.append(lambda *a, **kw: C.ssm_scan(*a, variant=1, **kw))
    for fn in run:
        y, st = fn(*args, torch.tensor(lens, device=device), heads=H, state=N, groups=G)
        near(st, S, 2e-5)                       # the state is float32 whatever the inputs are
        for b, n in enumerate(lens):
            near(y[b, :n], ys[b], TOL[dtype])
        y, _ = fn(*args, None, heads=H, state=N, groups=G)
        near(y[0], ys[0], TOL[dtype])


@pytest.mark.parametrize("device", [CPU, GPU])
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("shape", SCAN)
@pytest.mark.parametrize("taps", [1, 2, 4, 7])
def test_one_token_of_the_recurrence(device, dtype, shape, taps):
    """Steps from an empty state equal the whole sequence; a retired row keeps its ring and state."""
    from ferrl_b200 import ops
    H, P, N, G, _ = shape
    T, C, B = 11, H * P + 2 * G * N, 3
    x, dt = rand(B, T, C, seed=1, dtype=dtype), rand(B, T, H, seed=2, dtype=dtype)
    w, b, dtb, A, D = rand(C, taps, seed=3), rand(C, seed=4), rand(H, seed=5) - 1, rand(H, seed=6), rand(H, seed=7)
    u = torch.stack([O.conv(x[i].double(), w.double(), b.double()) for i in range(B)])
    if dtype == BF16:
        u = u.to(BF16)
    ys, S = scan_want(u, dt, dtb, A, D, H, P, N, G, [T] * B)
    d = lambda t: t.to(device)  # noqa: E731
    ring, state = torch.full((B, taps, C), 7.0, dtype=dtype, device=device), torch.zeros(B, H, N, P, device=device)
    kv = torch.zeros(B, dtype=torch.int32, device=device)
    par = [d(t) for t in (w, b, dtb, A, D)]
    for t in range(T):
        fused = d(torch.cat([x[:, t], dt[:, t]], 1))
        on = None
        if t == 5:                               # a row sits one step out first
            on = torch.tensor([True, False, True], device=device)
            keep = ring[1].clone(), state[1].clone()
            tmp = ring.clone(), state.clone()
            y = ops.ssm_step(fused[:, :C], fused[:, C:], *par, *tmp, kv, on, groups=G)
            assert float(y[1].abs().max()) == 0.0 and torch.equal(tmp[0][1], keep[0]) and torch.equal(tmp[1][1], keep[1])
            assert not torch.equal(tmp[1][0], state[0])
        y = ops.ssm_step(fused[:, :C], fused[:, C:], *par, ring, state, kv, None, groups=G)
        kv += 1
        near(y, torch.stack([v[t] for v in ys]), 2 * TOL[dtype] if dtype == BF16 else 1e-4)
    near(state, S, 1e-4 if dtype == F32 else 3e-2)


@pytest.mark.parametrize("device", [CPU, GPU])
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("W,groups", [(96, 2), (35, 7), (1024, 1), (2048, 8), (12, 12)])
def test_gated_group_norm(device, dtype, W, groups):
    from ferrl_b200 import ops
    y, z, w = rand(9, W, seed=1, dtype=dtype), rand(9, W + 8, seed=2, dtype=dtype), rand(W, seed=3)
    want = O.gated_norm(y.double(), z[:, :W].double(), w.double(), groups, 1e-3)
    close(ops.gated_group_norm(y.to(device), z.to(device)[:, :W], w.to(device), groups, 1e-3), want, dtype)


@pytest.mark.parametrize("device", [CPU, GPU])
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("s", [1, 2, 3, 4, 5, 9])
@pytest.mark.parametrize("W", [37, 64, 2052])
def test_hyper_connections(device, dtype, s, W):
    from ferrl_b200 import ops
    T, eps = 11, 1e-3
    x, y = rand(T, s, W, seed=1), rand(T, W, seed=2, dtype=dtype)
    mix, out, inp, w = rand(s, s, seed=3), rand(s, seed=4), rand(s, seed=5), rand(W, seed=6)
    xs = [x[:, t].double() for t in range(s)]
    wd = {"h.in": torch.zeros(s), "h.mix": mix.double(), "h.out": out.double()}
    nxt = O.hyper(xs, wd, "h.", lambda u: y.double())
    d = lambda t: t.to(device)  # noqa: E731

    def check(got, streams, coef, scale=1.0):
        near(got[1], scale * O.norm(sum(c * v for c, v in zip(coef, streams)), w.double(), eps), TOL[dtype])
        assert got[1].dtype == dtype
    got = ops.hyper_norm(d(x), d(y), d(mix), d(out), d(inp), d(w), eps, dtype)
    near(got[0], torch.stack(nxt, 1), 3e-5)
    check(got, nxt, inp.double())
    got = ops.hyper_norm(d(x), None, None, None, d(inp), d(w), eps, dtype)
    assert torch.equal(got[0].cpu(), x)
    check(got, xs, inp.double())
    fresh = d(x)
    check(ops.hyper_norm(fresh, d(y), d(mix), d(out), None, d(w), eps, dtype, 0.3, False), nxt, torch.ones(s), 0.3)
    assert torch.equal(fresh.cpu(), x)


@pytest.mark.parametrize("device", [CPU, GPU])
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("W", [7, 64, 100])
def test_embedding_and_positions(device, dtype, W):
    from ferrl_b200 import ops
    table, ids = rand(20, W, seed=1, dtype=dtype), torch.tensor([[3, 19, 0, 3], [5, 5, 1, 2]])
    pe = ops.sinusoid_table(6000, W)
    x = ops.embed_streams(ids.to(device), table.to(device), pe.to(device), torch.arange(4, device=device), 3)
    want = table[ids].double() + torch.stack([O.sinusoid(p, W) for p in range(4)])
    assert x.shape == (2, 4, 3, W) and x.dtype == F32
    for s in range(3):
        near(x[:, :, s], want, 1e-6)
    kv = torch.tensor([5, 5003], dtype=torch.int32)
    x = ops.embed_streams(ids[:, 0].to(device), table.to(device), pe.to(device), kv.to(device), 2)
    near(x[:, 1], table[ids[:, 0]].double() + torch.stack([O.sinusoid(int(p), W) for p in kv]), 1e-6)


@pytest.mark.parametrize("device", [CPU, GPU])
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("F,limit,alpha", [(40, 0.8, 1.702), (13, 7.0, 1.702), (64, 0.0, 0.5)])
def test_clipped_glu(device, dtype, F, limit, alpha):
    """Values on both sides of every clip; gradients vanish beyond them."""
    from ferrl_b200 import ops
    x = rand(50, 2 * F, seed=1, std=2.0, dtype=dtype)
    act = ops.ClippedGlu(limit, alpha)
    xd = x.double().requires_grad_(True)
    g, u = torch.clamp(xd[:, :F], max=limit), torch.clamp(xd[:, F:], -limit, limit)
    want = g / (1 + torch.exp(-alpha * g)) * (u + 1)
    if alpha == 1.702:
        near(want.detach(), O.clipped_glu(x[:, :F].double(), x[:, F:].double(), limit), 1e-9)
    y = x.to(device).requires_grad_(True)
    got = ops.swiglu(y, act)
    close(got, want.detach(), dtype)
    dy = rand(50, F, seed=2)
    (got.float() * dy.to(device)).sum().backward()
    (want * dy.double()).sum().backward()
    close(y.grad, xd.grad, dtype)


@pytest.mark.gpu
@pytest.mark.parametrize("M", [1, 70, 300])
def test_clipped_glu_in_the_projection(M):
    from ferrl_b200 import ops
    from ferrl_b200.models.lora import FusedLoraLinear
    from ferrl_b200.ops import cuda as C
    x, w = rand(M, 64, seed=1, dtype=BF16), rand(2 * 80, 64, seed=2, std=0.3, dtype=BF16)
    act = ops.ClippedGlu(0.9)
    want = O.clipped_glu(x.double() @ w[:80].double().T, x.double() @ w[80:].double().T, 0.9)
    order = FusedLoraLinear.glu_row_order(80)
    near(C.gemm_glu(x.cuda(), w[order].contiguous().cuda(), act), want, 3e-2)


@pytest.mark.parametrize("device,dtype", [(CPU, F32), (CPU, BF16), pytest.param("cuda", BF16, marks=pytest.mark.gpu)])
@pytest.mark.parametrize("M,N,Kd", [(1, 40, 64), (70, 24, 64), (1100, 520, 72), (3, 17, 16), (130, 712, 256)])
def test_projection_with_bias(device, dtype, M, N, Kd):
    from ferrl_b200 import ops
    x, w, b = rand(M, Kd, seed=1, dtype=dtype), rand(N, Kd, seed=2, dtype=dtype), rand(N, seed=3, std=5.0, dtype=dtype)
    close(ops.lora_linear(x.to(device), w.to(device), None, None, bias=b.to(device)), x.double() @ w.double().T + b.double(), dtype)


# ------------------------------------------------------------------------------------------------ whole models
def load(tmp_path, name, device, dtype=F32, seed=3, lora=None, **kw):
    from ferrl_b200.models.loader import LoaderOpts, load_auto_policy
    cfg = K.CASES[name]
    w = K.weights(cfg, seed, K.BUCKETS[name])
    folder = tmp_path / name
    folder.mkdir(exist_ok=True)
    K.write(folder, cfg, w)
    model, ident = load_auto_policy(str(folder), LoaderOpts(lora=lora, dtype=dtype, device=device, **kw))
    assert ident.model_type == "Mifutar"
    model.merge_adapters()
    return cfg, w, model


MODEL_TOL = 5e-4


def model_near(got, want, dtype):
    """float32: every position.  bf16: narrow layers average little rounding away, so the bulk tightly and all loosely."""
    if dtype == F32:
        return rms_near(got, want, MODEL_TOL)
    err = row_errors(got, want)
    assert float(err.median()) < 0.03 and float(err.max()) < 0.3, (float(err.median()), float(err.max()))


@pytest.mark.parametrize("device", [CPU, GPU])
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", sorted(K.CASES))
def test_prompts_and_decoding_match_the_oracle(tmp_path, name, dtype, device):
    """A whole prompt; the same tokens one by one from the first (through every window and round every ring); and from
    a prompt cut at several places, two tokens among them."""
    cfg, w, m = load(tmp_path, name, device, dtype)
    n = 150 if name == "wide" else 60
    toks = tokens(n, cfg["vocab"], 1)
    want = O.forward(toks, w, cfg)
    model_near(prefill_all(m.new_decoder(1, n), [toks], device)[0], want, dtype)
    for cut in (1, 2, 34):
        dec = m.new_decoder(1, n)
        got = prefill_all(dec, [toks[:cut]], device) + [feed(dec, [t], device) for t in toks[cut:]]
        model_near(torch.cat(got), want, dtype)


@pytest.mark.parametrize("device", [CPU, GPU])
@pytest.mark.parametrize("name", sorted(K.CASES))
def test_layers_match_the_oracle(tmp_path, name, device):
    cfg, w, m = load(tmp_path, name, device)
    toks, layers = tokens(25, cfg["vocab"], 2), []
    O.forward(toks, w, cfg, layers_out=layers)
    x, _ = m.forward_streams(torch.tensor([toks], device=device), detached=True)
    near(x[0].sum(-2), layers[-1], 3e-4)
    rms_near(m(torch.tensor([toks], device=device))[0], O.forward(toks, w, cfg), MODEL_TOL)


@pytest.mark.parametrize("device", [CPU, GPU])
@pytest.mark.parametrize("name", ["mixed", "odd", "wide"])
def test_unequal_batches_and_reused_rows(tmp_path, name, device):
    """Prompts of unequal lengths decoded together, the shorter ones leaving early, each equal to itself alone; then
    the same decoder starts other prompts over the rows that were given back."""
    cfg, w, m = load(tmp_path, name, device)
    dec = m.new_decoder(4, 96)
    for seed, lens, ends in ((1, (1, 40, 7, 22), (9, 30, 12, 25)), (5, (33, 2, 50, 1), (20, 14, 14, 20))):
        seqs = [tokens(n + e, cfg["vocab"], seed + i) for i, (n, e) in enumerate(zip(lens, ends))]
        got = [[x] for x in prefill_all(dec, [s[:n] for s, n in zip(seqs, lens)], device)]
        for step in range(max(ends)):
            act = [step < e for e in ends]
            logits = feed(dec, [s[n + step] if a else 0 for s, n, a in zip(seqs, lens, act)], device, None if all(act) else act)
            for i, a in enumerate(act):
                if a:
                    got[i].append(logits[i:i + 1])
        assert dec.kv_len.tolist() == [n + e for n, e in zip(lens, ends)]
        for s, rows in zip(seqs, got):
            rms_near(torch.cat(rows), O.forward(s, w, cfg), MODEL_TOL)


@pytest.mark.parametrize("device", [CPU, GPU])
def test_long_decoding(tmp_path, device):
    """More than ten windows of decoded tokens; position and bias tables grow past their first size."""
    cfg, w, m = load(tmp_path, "mixed", device, max_position_embeddings=4)
    n = 380
    toks = tokens(n, cfg["vocab"], 8)
    want = O.forward(toks, w, cfg)
    dec = m.new_decoder(2, n)
    got = prefill_all(dec, [toks[:3]] * 2, device)[:1] + [feed(dec, [t, t], device)[:1] for t in toks[3:]]
    rms_near(torch.cat(got), want, MODEL_TOL)


@pytest.mark.parametrize("device", [CPU, GPU])
def test_reach_of_the_windows(tmp_path, device):
    """One attention layer with window w: a changed token moves the logits of the w - 1 positions behind it and no
    others, in a prompt and in decoding.  One recurrent layer: a token reaches every later position."""
    from ferrl_b200.models.loader import LoaderOpts, load_auto_policy
    for window in (1, 2, 31, 32, 33, None):
        cfg = K.config(50, 32, [(K.attn(2, 1, 8, window, 20) if window else K.ssm(2, 8, 8, 1, 3, 1), K.ff(16, 1.0))], 2)
        folder = tmp_path / f"w{window}"
        folder.mkdir()
        m, _ = load_auto_policy(K.write(folder, cfg, K.weights(cfg, 1)), LoaderOpts(lora=None, device=device))
        m.merge_adapters()
        a = tokens(80, 50, 4)
        b = list(a)
        b[20] = (a[20] + 1) % 50
        la, lb = (prefill_all(m.new_decoder(1, 80), [s], device)[0] for s in (a, b))
        moved = [t for t in range(80) if float((la[t] - lb[t]).abs().max()) > 1e-6]
        last = min(80, 20 + window) if window else 24
        assert (moved if window else moved[:4]) == list(range(20, last)), (window, moved)
        da, db = m.new_decoder(1, 80), m.new_decoder(1, 80)
        for d, s in ((da, a), (db, b)):
            prefill_all(d, [s[:21]], device)
        moved = [t for t in range(21, 80) if float((feed(da, [a[t]], device) - feed(db, [b[t]], device)).abs().max()) > 1e-6]
        assert (moved if window else moved[:3]) == list(range(21, last)), (window, moved)


# ------------------------------------------------------------------------------------------------ generation, scoring
def oracle_greedy(w, cfg, prompt, n):
    toks, margin = list(prompt), 1e9
    for _ in range(n):
        top = O.forward(toks, w, cfg)[-1].topk(2)
        margin = min(margin, float(top.values[0] - top.values[1]))
        toks.append(int(top.indices[0]))
    return toks[len(prompt):], margin


@pytest.mark.parametrize("device", [CPU, GPU])
@pytest.mark.parametrize("name", ["mixed", "odd"])
def test_greedy_generation_through_the_policy(tmp_path, name, device):
    """Two prompts with groups of two through ``LmPolicy``: packing, group broadcast, sampling, the graphed step."""
    from ferrl_b200.lm_policy import LmPolicy
    from ferrl_b200.policy import EvalSampling, GenConfig, validate_generated_rollout_semantics
    from ferrl_b200.sampler import GrpoSampler
    cfg, w, m = load(tmp_path, name, device)
    prompts = [tokens(13, cfg["vocab"], 1), tokens(4, cfg["vocab"], 2)]
    want = [oracle_greedy(w, cfg, p, 20) for p in prompts]
    assert all(margin > 1e-3 for _, margin in want)
    gen = GenConfig(group_size=2, max_new_tokens=20, eval_sampling=EvalSampling(1.0, 1e-9))
    pol = LmPolicy(m, GrpoSampler(5))
    for _ in range(2):                       # the second call runs on the kept decoder and graph
        for r, p, (toks, _) in zip(pol.generate_batch(prompts, gen, [0, 2]), prompts, want):
            validate_generated_rollout_semantics(r, p, gen)
            assert r.completion(0) == toks and r.completion(1) == toks
    # EOS retires a row; the others go on unchanged
    eos = want[0][0][5]
    gen = GenConfig(group_size=2, max_new_tokens=20, eos_token_id=eos, eval_sampling=EvalSampling(1.0, 1e-9))
    for r, (toks, _) in zip(LmPolicy(m, GrpoSampler(5)).generate_batch(prompts, gen, [0, 2]), want):
        stop = toks.index(eos) + 1 if eos in toks else len(toks)
        assert r.completion(0) == toks[:stop]


@pytest.mark.gpu
def test_first_graphed_step_advances_recurrent_state_once():
    """The hybrid family keeps recurrent state too: a rollout through a freshly captured graph equals the plain loop."""
    from ferrl_b200.lm_policy import LmPolicy
    from ferrl_b200.models import LoraSpec
    from ferrl_b200.models.qwen35 import Qwen35GradModel, Qwen35Spec
    from ferrl_b200.policy import EvalSampling, GenConfig
    from ferrl_b200.sampler import GrpoSampler
    m = Qwen35GradModel(Qwen35Spec(vocab_size=512, hidden_size=256, num_hidden_layers=2, num_attention_heads=2, num_key_value_heads=1, head_dim=128,
                                   intermediate_size=256, layer_types=["linear_attention"] * 2, lin_k_heads=2, lin_v_heads=2,
                                   max_position_embeddings=128), LoraSpec(8, 16.0), dtype=BF16, device="cuda")
    m.init_random(3, 0.1)
    gen = GenConfig(group_size=1, max_new_tokens=12, eval_sampling=EvalSampling(1.0, 1e-9))
    runs = []
    for graphed in (False, True):
        pol = LmPolicy(m, GrpoSampler(5))
        pol.use_cuda_graph = graphed
        runs.append(pol.generate_batch([tokens(9, 512, 1), tokens(5, 512, 2)], gen, [0, 1]))
    for a, b in zip(*runs):
        assert torch.equal(a.token_ids, b.token_ids)
        assert float((a.rollout_logprobs - b.rollout_logprobs).abs().max()) < 1e-3


def test_sampled_rows_depend_on_their_seed_only(tmp_path):
    from ferrl_b200.lm_policy import LmPolicy
    from ferrl_b200.policy import GenConfig
    from ferrl_b200.sampler import GrpoSampler
    cfg, _, m = load(tmp_path, "mixed", CPU)
    prompts = [tokens(9, cfg["vocab"], 1), tokens(5, cfg["vocab"], 2)]
    gen = GenConfig(group_size=2, max_new_tokens=8)
    both = LmPolicy(m, GrpoSampler(5)).generate_batch(prompts, gen, [0, 2])
    alone = LmPolicy(m, GrpoSampler(5)).generate_batch(prompts[1:], gen, [2])
    assert torch.equal(both[1].token_ids, alone[0].token_ids)
    assert not torch.equal(both[1].token_ids[0], both[1].token_ids[1])


@pytest.mark.parametrize("device", [CPU, GPU])
def test_generate_verb(tmp_path, device, monkeypatch, capsys):
    from ferrl_b200 import cli
    cfg, w, _ = load(tmp_path, "one", CPU)
    prompt = tokens(6, cfg["vocab"], 3)
    monkeypatch.setattr(sys, "stdin", io.StringIO(json.dumps(prompt) + "\n"))
    assert cli.main(["generate", "--model", str(tmp_path / "one"), "--dtype", "float32", "--device", device, "--greedy",
                     "--max-new-tokens", "7"]) == 0
    assert json.loads(capsys.readouterr().out) == oracle_greedy(w, cfg, prompt, 7)[0]


def adapted_names(i, l):
    """Projections of layer ``i`` that carry adapters, with the checkpoint rows behind each."""
    out = [(l.gate_up, [(f"l{i}.mlp.gate", slice(None)), (f"l{i}.mlp.up", slice(None))]), (l.down, [(f"l{i}.mlp.down", slice(None))])] if l.ff else []
    if hasattr(l.mix, "conv_w"):
        d = l.mix.dims
        cut = [slice(0, d.inner), slice(d.inner, d.inner + d.channels), slice(d.inner + d.channels, None)]
        return [(l.mix.inp, [(f"l{i}.mix.in", c) for c in cut]), (l.mix.out, [(f"l{i}.mix.o", slice(None))])] + out
    return [(l.mix.inp, [(f"l{i}.mix.q", slice(None)), (f"l{i}.mix.k", slice(None))]), (l.mix.out, [(f"l{i}.mix.o", slice(None))])] + out


@pytest.mark.parametrize("remat", [False, True])
@pytest.mark.parametrize("name", ["mixed", "odd"])
def test_scoring_gradients_match_the_oracle(tmp_path, name, remat):
    """Log-probabilities and adapter gradients of a prompt against autograd through the plain model with the adapters
    folded into its weights."""
    from ferrl_b200.models.lora import LoraSpec
    spec = LoraSpec(4, 8.0)
    cfg, w, m = load(tmp_path, name, CPU, lora=spec, remat=remat, gdn_targets="qzao")
    adapters(m)
    toks = tokens(24, cfg["vocab"], 6)
    tgt = torch.tensor([toks[8:24]])
    lp = m.token_logprobs(torch.tensor([toks[:-1]]), torch.tensor([7]), tgt)
    lp.sum().backward()
    ww = {k: v.double() for k, v in w.items()}
    pairs = []
    for i, l in enumerate(m.layers):
        for proj, parts in adapted_names(i, l):
            assert len(proj.lora_A) == len(parts)
            for a, b, (n, rows) in zip(proj.lora_A, proj.lora_B, parts):
                A, B = (t.detach().double().requires_grad_(True) for t in (a, b))
                idx = torch.arange(ww[n].shape[0])[rows]
                ww[n] = ww[n].index_add(0, idx, spec.scale * B @ A)
                pairs += [(a, A), (b, B)]
    assert len(pairs) == len(m.trainable_params())
    logits = O.forward(toks[:-1], ww, cfg)
    want = torch.log_softmax(logits, -1)[7:].gather(1, tgt[0][:, None])[:, 0]
    near(lp[0], want.detach(), 1e-4)
    want.sum().backward()
    for got, ref in pairs:
        near(got.grad, ref.grad, 5e-3)
    # merged decoding sees the same adapters
    m.merge_adapters()
    rms_near(prefill_all(m.new_decoder(1, 24), [toks[:-1]], CPU)[0], logits.detach(), MODEL_TOL)


def test_recurrent_layers_carry_adapters_only_where_asked(tmp_path):
    from ferrl_b200.models.lora import LoraSpec
    m = load(tmp_path, "mixed", CPU, lora=LoraSpec(4, 8.0))[2]
    assert m.lora_recipe() == LoraSpec(4, 8.0).recipe()
    assert [len(l.mix.inp.lora_A) for l in m.layers] == [0, 2, 0, 2]
    m = load(tmp_path, "mixed", CPU, lora=LoraSpec(4, 8.0), gdn_targets="qo")[2]
    assert m.lora_recipe().endswith("|gdn:qo") and [len(l.mix.inp.lora_A) for l in m.layers] == [1, 2, 1, 2]
    assert [len(l.mix.out.lora_A) for l in m.layers] == [1, 1, 1, 1]


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [F32, BF16])
def test_scoring_gradients_on_the_gpu(tmp_path, dtype):
    from ferrl_b200.models.lora import LoraSpec
    models = [load(tmp_path, "wide", d, t, lora=LoraSpec(8, 16.0), gdn_targets="qzao")[2] for d, t in ((CPU, F32), ("cuda", dtype))]
    grads = []
    for m, dev in zip(models, (CPU, "cuda")):
        adapters(m)
        ids = torch.tensor([tokens(40, 160, 1), tokens(40, 160, 2)])
        lp = m.token_logprobs(ids[:, :-1].to(dev), torch.tensor([9, 9], device=dev), ids[:, 10:].to(dev))
        lp.sum().backward()
        grads.append([lp.detach().cpu()] + [p.grad.detach().cpu() for p in m.trainable_params()])
    tol = 2e-3 if dtype == F32 else 0.2
    for got, ref in zip(grads[1], grads[0]):
        assert float((got - ref).norm() / ref.norm()) < tol
    with torch.no_grad():      # grad-free scoring runs the fused inference pass
        m = models[1]
        ids = torch.tensor([tokens(40, 160, 1), tokens(40, 160, 2)], device="cuda")
        lp = m.token_logprobs(ids[:, :-1], torch.tensor([9, 9], device="cuda"), ids[:, 10:])
    assert float((lp.cpu() - grads[1][0]).abs().max()) < (1e-3 if dtype == F32 else 0.15)
    m.merge_adapters()         # interleaved snapshots with the clipped GLU in the projection's epilogue
    got = prefill_all(m.new_decoder(1, 48), [tokens(40, 160, 1)], "cuda")[0]
    ref = models[0](torch.tensor([tokens(40, 160, 1)]))[0].detach()
    model_near(got, ref.double(), dtype)


def test_full_fine_tuning_reaches_every_tensor(tmp_path):
    cfg, _, m = load(tmp_path, "mixed", CPU, full_ft=True)
    ids = torch.tensor([tokens(30, cfg["vocab"], 1)])
    m.token_logprobs(ids[:, :-1], torch.tensor([3]), ids[:, 4:]).sum().backward()
    missing = [n for n, p in m.named_parameters() if p.grad is None or not bool(p.grad.abs().sum() > 0)]
    assert missing == [] and len(m.trainable_params()) == len(list(m.named_parameters()))


# ------------------------------------------------------------------------------------------------ configuration, replay
def test_configuration_is_read_and_checked(tmp_path):
    from ferrl_b200.models.loader import LoaderOpts, load_auto_policy
    from ferrl_b200.hf import model_vocab_size
    from ferrl_b200.models.mifutar import mifutar_spec
    rows = {1: 8, 3: 8}
    assert model_vocab_size(K.MIXED) == 89
    spec = mifutar_spec(K.MIXED, rows)
    assert [getattr(l.mixer, "window", None) for l in spec.layers] == [None, 7, None, 33] and spec.streams == 3 and spec.logit_scale == 0.5
    assert spec.layers[1].mlp is None and spec.layers[3].mlp.limit == 1.5 and spec.layers[3].mixer.scale == 0.5
    for change in (lambda c: c["layers"][0].update(type="other"), lambda c: c["layers"][0]["mlp"].update(kind="other"),
                   lambda c: c["layers"][0]["mixer"].update(groups=3), lambda c: c["layers"][0]["mixer"].update(norm_groups=5),
                   lambda c: c["layers"][1]["mixer"]["mask"].update(size=0), lambda c: c["layers"][1]["mixer"].update(kv_heads=4),
                   lambda c: c["layers"][1]["mixer"].update(vdim=8), lambda c: c["layers"][1]["mixer"].update(bias_max=4),
                   lambda c: c.update(streams=0)):
        bad = json.loads(json.dumps(K.MIXED))
        change(bad)
        with pytest.raises(ValueError):
            mifutar_spec(bad, rows)
    K.write(tmp_path, K.ONE, K.weights(K.ONE, 1))
    for opts in (LoaderOpts(tp=(0, 2)), LoaderOpts(ep=(0, 2))):
        with pytest.raises(ValueError):
            load_auto_policy(str(tmp_path), opts)


def test_decode_state_does_not_grow_past_the_windows(tmp_path):
    cfg, _, m = load(tmp_path, "mixed", CPU)
    small, large = m.new_decoder(2, 64), m.new_decoder(2, 4096)
    assert small.cache_bytes() == large.cache_bytes()
    assert [s.ring.shape[1] for s in large.state] == [4, 7, 2, 33]
    assert [t.dtype for s in large.state for t in s.advanced()] == [F32, F32] == [t.dtype for t in large.step_state()]
    assert int(large.kv_tokens_read()) == 2
    with pytest.raises(ValueError):
        prefill_all(small, [tokens(65, cfg["vocab"], 1)], CPU)


@pytest.mark.parametrize("device", [CPU, GPU])
def test_trace_replay(tmp_path, device):
    """Steps of a trace: a batch that starts together, goes on by one token and loses its shorter requests, a second
    batch while the first is held, wanted places in any order."""
    from ferrl_b200.trace import TraceReplay, replay_stream
    cfg, w, _ = load(tmp_path, "mixed", CPU)
    s = {r: tokens(n, cfg["vocab"], i) for i, (r, n) in enumerate((("a", 30), ("b", 12), ("c", 21)))}
    want = {r: O.forward(t, w, cfg) for r, t in s.items()}
    rep = TraceReplay.load(str(tmp_path / "mixed"), "float32", 64, device)
    steps = [([("a", 0, 25, [3, 0, 24]), ("b", 0, 10, [9])], []), ([("a", 25, 26, [0]), ("b", 10, 11, [])], []),
             ([("b", 11, 12, [0]), ("a", 26, 27, [0])], ["b"]), ([("c", 0, 20, [19])], []), ([("a", 27, 28, [0])], []),
             ([("c", 20, 21, [0])], ["c"]), ([("a", 28, 29, [])], []), ([("a", 29, 30, [0])], ["a"])]
    lines, told = [], []
    for n, (entries, end) in enumerate(steps):
        lines.append(json.dumps({"step": n, "end": end, "entries": [
            {"id": r, "tokens": s[r][lo:hi], "want": wn} for r, lo, hi, wn in entries]}))
    replay_stream(rep, lines, str(tmp_path), told.append)
    assert told == [f"done {n}" for n in range(len(steps))] and not rep.of
    for n, (entries, _) in enumerate(steps):
        ref = [want[r][lo + k] for r, lo, _, wn in entries for k in wn]
        path = tmp_path / f"{n}.f32"
        assert path.exists() == bool(ref)
        if ref:
            got = torch.from_numpy(np.fromfile(path, "<f4").reshape(len(ref), -1))
            rms_near(got, torch.stack(ref), MODEL_TOL)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_trace_run_program(tmp_path, dtype):
    cfg, w, m = load(tmp_path, "wide", "cuda", F32)
    prefill_all(m.new_decoder(1, 8), [[1, 2, 3]], "cuda")
    toks = tokens(150, cfg["vocab"], 3)
    want = O.forward(toks, w, cfg)
    steps = [{"step": 0, "entries": [{"id": "q", "tokens": toks[:140], "want": [0, 69, 139]}], "end": []}]
    steps += [{"step": i + 1, "entries": [{"id": "q", "tokens": [t], "want": [0]}], "end": []} for i, t in enumerate(toks[140:])]
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    r = subprocess.run([os.path.join(root, "bin", "trace_run"), "--model", str(tmp_path / "wide"), "--dtype", dtype, "--out",
                        str(tmp_path), "--max-tokens", "200"], input="".join(json.dumps(x) + "\n" for x in steps), text=True,
                       capture_output=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    got = torch.cat([torch.from_numpy(np.fromfile(tmp_path / f"{i}.f32", "<f4").reshape(-1, cfg["vocab"])) for i in range(11)])
    model_near(got, want[[0, 69, 139] + list(range(140, 150))], F32 if dtype == "float32" else BF16)
