"""The Galodra family against its plain restatement (``galodra_oracle.py``): every mechanism by itself, whole prompts,
decoding through the ring caches, batches, reused slots, generation, scoring gradients and trace replay.  Each case
runs on the CPU path and, marked ``gpu``, through the sm_100a kernels."""
import io
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import galodra_cases as K
import galodra_oracle as O
from family_helpers import _native, adapters, feed, near, prefill_all, rand, rms_near, row_errors, tokens  # noqa: F401

CPU = "cpu"
GPU = pytest.param("cuda", marks=pytest.mark.gpu)
F32, BF16 = torch.float32, torch.bfloat16


TOL = {F32: 3e-5, BF16: 3e-2}


# ------------------------------------------------------------------------------------------------ mechanisms
ATT = [  # heads, dim, rot, vdim, window, S
    (3, 16, 8, 24, 5, 50), (2, 64, 64, 64, 64, 200), (2, 128, 64, 128, 129, 300), (1, 40, 24, 136, 1, 70),
    (2, 192, 64, 128, 128, 200), (2, 5, 6, 7, 9, 40), (2, 72, 16, 200, 100, 140), (1, 8, 8, 8, 1000, 260)]


@pytest.mark.parametrize("device", [CPU, GPU])
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("shape", ATT)
def test_attention_over_sequences(device, dtype, shape):
    """Random keys plus, for every query, one loud key just inside the window and a louder one just outside."""
    from ferrl_b200 import ops
    H, D, R, V, W, S = shape
    B, rank = 2, 24
    scale = (D + R) ** -0.5
    q, kn, v = rand(B, S, H, D + R, seed=1), rand(B, S, H, D, seed=2), rand(B, S, H, V, seed=3)
    lat = rand(B, S, (rank + R + 7) // 8 * 8, seed=4)
    # positions agree on a code: token t carries code t mod (W + 1) in the unrotated part, queries look for the key W - 1
    # back (inside) and, more strongly, for the key W back (outside); codes need room, so only where D has it
    n = W + 1
    if n <= D and S > n:
        eye = torch.eye(n) * 4.0
        for t in range(S):
            kn[:, t, :, :n] = eye[t % n]
            q[:, t, :, :n] = (eye[(t - W + 1) % n] * 0.8 + eye[(t - W) % n] * 1.6) / scale
    sink = rand(H, seed=5, std=2.0)
    q, kn, v, lat = (x.to(dtype) for x in (q, kn, v, lat))
    want = torch.stack([O.attend(q[b, ..., :D].double(), q[b, ..., D:].double(), kn[b].double(), lat[b, :, rank:rank + R].double(),
                                 v[b].double(), scale, W, sink.double()) for b in range(B)]).reshape(B, S, H * V)
    kv = torch.cat([kn.reshape(B, S, -1), v.reshape(B, S, -1)], -1)
    args = [x.to(device) for x in (q, kv, lat)]
    got = ops.latent_attention(*args, dim=D, vdim=V, rank=rank, scale=scale, window=W, sink=sink.to(device))
    near(got, want, 2 * TOL[dtype])
    if device == "cuda":
        from ferrl_b200.ops import cuda as C
        near(C.latent_attention(*args, dim=D, vdim=V, rank=rank, scale=scale, window=W, sink=sink.cuda(), variant=1), want,
             2 * TOL[dtype])
        # no sink, no window: the same kernels as parameters of another design would use them
        free = torch.stack([O.attend(q[b, ..., :D].double(), q[b, ..., D:].double(), kn[b].double(), lat[b, :, rank:rank + R].double(),
                                     v[b].double(), scale, S + 1, torch.full((H,), -1e9, dtype=torch.float64)) for b in range(B)])
        near(C.latent_attention(*args, dim=D, vdim=V, rank=rank, scale=scale), free.reshape(B, S, H * V), 2 * TOL[dtype])


DEC = [  # heads, dim, rot, vdim, rank, slots
    (3, 16, 8, 24, 40, 7), (20, 64, 32, 64, 128, 70), (33, 32, 64, 40, 512, 200), (1, 8, 16, 8, 8, 65), (2, 5, 6, 7, 11, 9),
    (16, 24, 24, 16, 200, 130), (17, 128, 64, 128, 384, 64), (2, 16, 128, 16, 328, 129)]


@pytest.mark.parametrize("device", [CPU, GPU])
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("shape", DEC)
def test_attention_of_one_token(device, dtype, shape):
    """Absorbed decoding against expanded keys and values: every count around a key tile's edge, empty rows, a loud
    key in the last occupied slot and a louder one in the first slot that is not."""
    from ferrl_b200 import ops
    H, D, R, V, rank, slots = shape
    counts = sorted({c for c in (0, 1, 2, 63, 64, 65, slots - 1, slots) if 0 <= c <= slots})
    B, scale = len(counts), (D + R) ** -0.5
    q, uk, uv = rand(B, H, D + R, seed=1), rand(H, D, rank, seed=2, std=rank ** -0.5), rand(H, V, rank, seed=3, std=rank ** -0.5)
    cache = rand(B, slots, (rank + R + 7) // 8 * 8, seed=4)
    for b, c in enumerate(counts):
        loud = q[b, 0, D:] * (3.0 / scale / q[b, 0, D:].pow(2).sum())
        if c:
            cache[b, c - 1, rank:rank + R] = 2 * loud
        if c < slots:
            cache[b, c, rank:rank + R] = 4 * loud
    sink = rand(H, seed=5, std=2.0)
    q, uk, uv, cache = (x.to(dtype) for x in (q, uk, uv, cache))
    want = torch.zeros(B, H, V, dtype=torch.float64)
    for b, c in enumerate(counts):
        if c:
            lat, kr = cache[b, :c, :rank].double(), cache[b, :c, rank:rank + R].double()
            kn = torch.einsum("jk,hdk->jhd", lat, uk.double())
            s = (torch.einsum("hd,jhd->hj", q[b, :, :D].double(), kn) + q[b, :, D:].double() @ kr.T) * scale
            want[b] = torch.einsum("hj,jhv->hv", O.sink_softmax(s, sink.double()), torch.einsum("jk,hvk->jhv", lat, uv.double()))
    args = [x.to(device) for x in (q, uk.transpose(1, 2).contiguous(), uv, cache)] + \
        [torch.tensor(counts, dtype=torch.int32, device=device)]
    want = want.reshape(B, H * V)
    got = ops.latent_decode(*args, rank=rank, scale=scale, sink=sink.to(device))
    near(got, want, 2 * TOL[dtype])
    assert float(got[0].abs().max()) == 0.0                       # counts[0] == 0: nothing to attend to
    if device == "cuda":
        from ferrl_b200.ops import cuda as C
        for splits in (1, 2, 3):
            near(C.latent_decode(*args, rank=rank, scale=scale, sink=sink.cuda(), splits=splits), want, 2 * TOL[dtype], splits)


@pytest.mark.parametrize("device", [CPU, GPU])
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("shape", [(3, 16, 8, 40, 8), (2, 5, 6, 11, 4), (4, 64, 32, 512, 32), (1, 8, 2, 8, 2)])
def test_latent_rows_and_rotation(device, dtype, shape):
    from ferrl_b200 import ops
    H, D, R, rank, dims = shape
    B, S, base, eps = 2, 37, 300.0, 1e-3
    fused = rand(B, S, H * (D + R) + rank + R + 8, seed=1, dtype=dtype)      # as in a fused projection, with a tail
    nw = rand(rank, seed=2, std=0.3) + 1.0
    cos, sin = ops.rope_tables(ops.default_inv_freq(dims, base), 6000)
    nq = H * (D + R)
    x = fused.double()
    wq, wk = x[..., :nq].reshape(B, S, H, D + R), x[..., nq:nq + rank + R]

    def want(pos):
        wr = torch.stack([torch.cat([wq[b][..., :D], O.rotate(wq[b][..., D:], pos[b], dims, base)], -1) for b in range(B)])
        rows = torch.stack([torch.cat([O.rms_norm(wk[b][:, :rank], nw.double(), eps), O.rotate(wk[b][:, rank:], pos[b], dims, base)], -1)
                            for b in range(B)])
        return wr, rows

    def views(t):
        return t[..., :nq].unflatten(-1, (H, D + R)), t[..., nq:nq + rank + R]
    wr, rows = want([range(S)] * B)
    f = fused.to(device)
    q, lat = ops.latent_prep(*views(f), nw.to(device), eps, cos.to(device), sin.to(device), torch.arange(S, device=device), dim=D, rank=rank)
    near(q, wr, TOL[dtype] * 2)
    near(lat[..., :rank + R], rows, TOL[dtype] * 2)
    assert lat.shape[-1] % 8 == 0 and float(lat[..., rank + R:].abs().sum()) == 0.0
    # decoding: every row at a position of its own, in the ring slot of that position, nothing else touched
    kv_len = torch.tensor([5, 5003], dtype=torch.int32)
    cache = torch.full((B, 7, lat.shape[-1]), 9.0, dtype=dtype, device=device)
    f = fused[:, 0].contiguous().to(device)
    q1 = ops.latent_append(*views(f), nw.to(device), eps, cos.to(device), sin.to(device), kv_len.to(device), cache, dim=D, rank=rank)
    wr, rows = want([[int(p)] * S for p in kv_len])
    near(q1, wr[:, 0], 1e-3 if dtype == F32 else TOL[dtype] * 2)      # float32 angles at position 5003
    for b in range(B):
        slot = int(kv_len[b]) % 7
        near(cache[b, slot, :rank + R], rows[b, 0], 1e-3 if dtype == F32 else TOL[dtype] * 2)
        rest = torch.cat([cache[b, :slot], cache[b, slot + 1:]])
        assert bool((rest == 9.0).all())


@pytest.mark.parametrize("device", [CPU, GPU])
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("W", [37, 64, 1024, 2052])
def test_post_norm(device, dtype, W):
    from ferrl_b200 import ops
    T, n, eps, alpha = 11, 3, 1e-3, 0.6
    x, y, g = rand(T, W, seed=1) * 2 + 3, rand(T, W, seed=2, dtype=dtype), rand(T, W + 8, seed=3, dtype=dtype)
    gb, w, b = rand(W, seed=4), rand(W, seed=5) + 1, rand(W, seed=6)
    hist, coef = rand(n, T, W, seed=7), rand(n + 1, seed=8)
    sig = 1 / (1 + torch.exp(-(g[:, :W].double() + gb.double())))
    r = O.layer_norm(alpha * x.double() + y.double() * sig, w.double(), b.double(), eps)
    nxt = O.depth_average([h.double() for h in hist] + [r], coef.double())
    d = lambda t: t.to(device)  # noqa: E731
    cast = BF16 if dtype == BF16 else F32
    buf = torch.empty(T, W, device=device)
    gate = d(g)[:, :W]
    a, low, rr = ops.post_norm(d(x), d(y), d(w), d(b), eps, alpha, gate, d(gb), d(hist), d(coef), cast, buf)
    near(a, nxt, 3e-5)
    near(buf, r, 3e-5)
    near(rr, r, 3e-5)
    assert a.dtype == F32 and low.dtype == cast
    near(low, nxt, TOL[dtype])
    a, _, rr = ops.post_norm(d(x), d(y), d(w), d(b), eps, alpha, gate, d(gb), cast=cast)
    near(a, r, 3e-5)
    near(rr, r, 3e-5)
    near(ops.post_norm(d(x), None, d(w), d(b), eps, cast=cast)[0], O.layer_norm(x.double(), w.double(), b.double(), eps), 3e-5)
    near(ops.post_norm(d(x), d(y), d(w), None, eps, alpha, cast=cast)[0],
         O.layer_norm(alpha * x.double() + y.double(), w.double(), 0.0, eps), 3e-5)


@pytest.mark.parametrize("device", [CPU, GPU])
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("shape", [(64, 40, 5, 2), (36, 17, 7, 1), (128, 64, 6, 6), (64, 24, 33, 3)])
@pytest.mark.parametrize("T", [1, 3, 150])
def test_routed_experts(device, dtype, shape, T):
    """Sigmoid scores, the chosen ones not renormalised, multiplying the experts' inputs."""
    from ferrl_b200.models import moe as M
    H, I, E, top = shape
    x = rand(T, H, seed=1, dtype=dtype)
    w = {"router": rand(E, H, seed=2, std=2 * H ** -0.5, dtype=dtype)}
    for e in range(E):
        w.update({f"e{e}.gate": rand(I, H, seed=10 + e, std=2 * H ** -0.5, dtype=dtype),
                  f"e{e}.up": rand(I, H, seed=50 + e, std=2 * H ** -0.5, dtype=dtype),
                  f"e{e}.down": rand(H, I, seed=90 + e, std=2 * I ** -0.5, dtype=dtype)})
    want = O.moe_ff(x.double(), {k: v.double() for k, v in w.items()}, "", top)
    gu = torch.stack([torch.cat([w[f"e{e}.gate"], w[f"e{e}.up"]], 0) for e in range(E)]).to(device)
    dn = torch.stack([w[f"e{e}.down"] for e in range(E)]).to(device)
    logits = (x.double() @ w["router"].double().T).float().to(device)
    got = M.routed_experts(x.to(device), logits, gu, dn, top, score="sigmoid", renorm=False, weight_input=True)
    if dtype == F32:
        near(got, want, 3e-4)
    else:
        rms_near(got, want, 2e-2)


# ------------------------------------------------------------------------------------------------ whole models
def load(tmp_path, name, device, dtype=F32, seed=3, lora=None, **kw):
    from ferrl_b200.models.loader import LoaderOpts, load_auto_policy
    cfg = K.CASES[name]
    w = K.weights(cfg, seed)
    folder = tmp_path / name
    folder.mkdir(exist_ok=True)
    K.write(folder, cfg, w)
    model, ident = load_auto_policy(str(folder), LoaderOpts(lora=lora, dtype=dtype, device=device, **kw))
    assert ident.model_type == "Galodra"
    model.merge_adapters()
    return cfg, w, model


MODEL_TOL = 3e-4


def model_near(got, want, dtype):
    """float32: every position.  bf16: the bulk of them, since an expert chosen the other way on a close call moves its
    token's logits and a little those that attend to it."""
    if dtype == F32:
        return rms_near(got, want, MODEL_TOL)
    err = row_errors(got, want)
    assert float(err.median()) < 0.03 and float(err.quantile(0.8)) < 0.08, (float(err.median()), float(err.quantile(0.8)))


@pytest.mark.parametrize("device", [CPU, GPU])
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", sorted(K.CASES))
def test_prompts_and_decoding_match_the_oracle(tmp_path, name, dtype, device):
    """A whole prompt; the same tokens one by one from the first (through every window and round every ring); and from
    a prompt cut at several places."""
    cfg, w, m = load(tmp_path, name, device, dtype)
    n = 60
    toks = tokens(n, cfg["vocab"], 1)
    want = O.forward(toks, w, cfg)
    model_near(prefill_all(m.new_decoder(1, n), [toks], device)[0], want, dtype)
    for cut in (1, 2, 19, 34):
        dec = m.new_decoder(1, n)
        got = prefill_all(dec, [toks[:cut]], device) + [feed(dec, [t], device) for t in toks[cut:]]
        model_near(torch.cat(got), want, dtype)


def test_layers_match_the_oracle(tmp_path):
    cfg, w, m = load(tmp_path, "mixed", CPU)
    toks, layers = tokens(25, cfg["vocab"], 2), []
    O.forward(toks, w, cfg, layers_out=layers)
    x = m.forward_hidden(torch.tensor([toks]), detached=True)
    near(x[0], layers[-1], 3e-4)


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
    """More than ten windows of decoded tokens; rotation tables grow past their first size."""
    cfg, w, m = load(tmp_path, "mixed", device, max_position_embeddings=16)
    n = 380
    toks = tokens(n, cfg["vocab"], 8)
    want = O.forward(toks, w, cfg)
    dec = m.new_decoder(2, n)
    got = prefill_all(dec, [toks[:3]] * 2, device)[:1] + [feed(dec, [t, t], device)[:1] for t in toks[3:]]
    rms_near(torch.cat(got), want, MODEL_TOL)


@pytest.mark.parametrize("device", [CPU, GPU])
def test_reach_of_the_windows(tmp_path, device):
    """One layer with window w: a changed token moves the logits of the w - 1 positions behind it and no others, in a
    prompt and in decoding."""
    from ferrl_b200.models.loader import LoaderOpts, load_auto_policy
    for window in (1, 2, 31, 32, 33):
        cfg = K.config(50, 32, [(K.mixer(2, 8, 8, 8, 24, window), K.dense(16))])
        folder = tmp_path / f"w{window}"
        folder.mkdir()
        m, _ = load_auto_policy(K.write(folder, cfg, K.weights(cfg, 1)), LoaderOpts(lora=None, device=device))
        m.merge_adapters()
        a = tokens(80, 50, 4)
        b = list(a)
        b[20] = (a[20] + 1) % 50
        la, lb = (prefill_all(m.new_decoder(1, 80), [s], device)[0] for s in (a, b))
        moved = [t for t in range(80) if float((la[t] - lb[t]).abs().max()) > 1e-6]
        assert moved == list(range(20, 20 + window)), (window, moved)
        da, db = m.new_decoder(1, 80), m.new_decoder(1, 80)
        for d, s in ((da, a), (db, b)):
            prefill_all(d, [s[:21]], device)
        moved = [t for t in range(21, 80) if float((feed(da, [a[t]], device) - feed(db, [b[t]], device)).abs().max()) > 1e-6]
        assert moved == list(range(21, 20 + window)), (window, moved)


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


@pytest.mark.parametrize("remat", [False, True])
def test_scoring_gradients_match_the_oracle(tmp_path, remat):
    """Log-probabilities and adapter gradients of a prompt against autograd through the plain model with the adapters
    folded into its weights."""
    from ferrl_b200.models.lora import LoraSpec
    spec = LoraSpec(4, 8.0)
    cfg, w, m = load(tmp_path, "mixed", CPU, lora=spec, remat=remat)
    adapters(m)
    toks = tokens(24, cfg["vocab"], 6)
    tgt = torch.tensor([toks[8:24]])
    lp = m.token_logprobs(torch.tensor([toks[:-1]]), torch.tensor([7]), tgt)
    lp.sum().backward()
    ww = {k: v.double() for k, v in w.items()}
    pairs = []
    for i, l in enumerate(m.layers):
        for proj, names in ((l.mix.inp, ("mix.q", "mix.dkv")), (l.mix.out, ("mix.o",)), (l.gate_up, ("mlp.gate", "mlp.up")), (l.down, ("mlp.down",))):
            if proj is None:
                continue
            assert len(proj.lora_A) == len(names)
            for a, b, n in zip(proj.lora_A, proj.lora_B, names):
                A, B = (t.detach().double().requires_grad_(True) for t in (a, b))
                ww[f"l{i}.{n}"] = ww[f"l{i}.{n}"] + spec.scale * B @ A
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


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [F32, BF16])
def test_scoring_gradients_on_the_gpu(tmp_path, dtype):
    from ferrl_b200.models.lora import LoraSpec
    models = [load(tmp_path, "wide", d, t, lora=LoraSpec(8, 16.0))[2] for d, t in ((CPU, F32), ("cuda", dtype))]
    grads = []
    for m, dev in zip(models, (CPU, "cuda")):
        adapters(m)
        ids = torch.tensor([tokens(40, 160, 1), tokens(40, 160, 2)])
        lp = m.token_logprobs(ids[:, :-1].to(dev), torch.tensor([9, 9], device=dev), ids[:, 10:].to(dev))
        lp.sum().backward()
        grads.append([lp.detach().cpu()] + [p.grad.detach().cpu() for p in m.trainable_params()])
    tol = 2e-3 if dtype == F32 else 0.12
    for got, ref in zip(grads[1], grads[0]):
        assert float((got - ref).norm() / ref.norm()) < tol
    with torch.no_grad():      # grad-free scoring runs the fused inference pass
        m = models[1]
        ids = torch.tensor([tokens(40, 160, 1), tokens(40, 160, 2)], device="cuda")
        lp = m.token_logprobs(ids[:, :-1], torch.tensor([9, 9], device="cuda"), ids[:, 10:])
    assert float((lp.cpu() - grads[1][0]).abs().max()) < (1e-3 if dtype == F32 else 0.15)


def test_full_fine_tuning_reaches_every_tensor(tmp_path):
    cfg, _, m = load(tmp_path, "mixed", CPU, full_ft=True)
    ids = torch.tensor([tokens(30, cfg["vocab"], 1)])
    m.token_logprobs(ids[:, :-1], torch.tensor([3]), ids[:, 4:]).sum().backward()
    missing = [n for n, p in m.named_parameters() if p.grad is None or not bool(p.grad.abs().sum() > 0)]
    assert missing == [] and len(m.trainable_params()) == len(list(m.named_parameters()))


# ------------------------------------------------------------------------------------------------ configuration, replay
def test_configuration_is_read_and_checked(tmp_path):
    from ferrl_b200.models.galodra import galodra_spec
    from ferrl_b200.models.loader import LoaderOpts, load_auto_policy
    spec = galodra_spec(K.MIXED)
    assert [l.mixer.window for l in spec.layers] == [7, 19, 1, 33] and spec.layers[1].mlp is None and spec.alpha == 0.7
    assert (spec.layers[0].mlp.experts, spec.layers[0].mlp.top, spec.layers[2].mlp.experts) == (5, 2, 0)
    for change in (lambda c: c["layers"][0].update(type="other"), lambda c: c["layers"][0]["mlp"].update(kind="other"),
                   lambda c: c["layers"][0]["mlp"]["router"].update(top=6), lambda c: c["layers"][0]["mixer"]["mask"].update(size=0),
                   lambda c: c["layers"][0]["mixer"]["rot"].update(dims=9)):
        bad = json.loads(json.dumps(K.MIXED))
        change(bad)
        with pytest.raises(ValueError):
            galodra_spec(bad)
    K.write(tmp_path, K.ONE, K.weights(K.ONE, 1))
    for opts in (LoaderOpts(tp=(0, 2)), LoaderOpts(ep=(0, 2))):
        with pytest.raises(ValueError):
            load_auto_policy(str(tmp_path), opts)


def test_cache_is_a_ring_of_the_window(tmp_path):
    cfg, _, m = load(tmp_path, "mixed", CPU)
    small, large = m.new_decoder(2, 64), m.new_decoder(2, 4096)
    assert small.cache_bytes() == large.cache_bytes()
    assert [c.shape[1] for c in large.cache] == [l["mixer"]["mask"]["size"] for l in cfg["layers"]]
    assert int(large.kv_tokens_read()) >= 2
    with pytest.raises(ValueError):
        prefill_all(small, [tokens(65, cfg["vocab"], 1)], CPU)


@pytest.mark.parametrize("device", [CPU, GPU])
def test_trace_replay(tmp_path, device):
    """Steps of a trace: a batch that starts together, goes on by one token and loses its shorter requests, a second
    batch while the first is held, wanted places in any order."""
    from ferrl_b200.trace import TraceError, TraceReplay, replay_stream
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
    rep.step([{"id": "x", "tokens": [1, 2], "want": []}])
    for bad in ([{"id": "x", "tokens": [1, 2], "want": []}], [{"id": "x", "tokens": [1], "want": []}, {"id": "y", "tokens": [1], "want": []}],
                [{"id": "y", "tokens": [1], "want": [1]}], [{"id": "y", "tokens": [], "want": []}]):
        with pytest.raises(TraceError):
            rep.step(bad)
    with pytest.raises(TraceError):
        rep.step([], ["nobody"])


def test_trace_replay_of_another_family(fixtures_dir):
    """The replay is not bound to one family: a Qwen3 fixture, two requests, one of which ends early."""
    from ferrl_b200.trace import TraceReplay
    folder = os.path.join(fixtures_dir, "tiny_qwen3")
    rep = TraceReplay.load(folder, "float32", 64, CPU)
    m = rep.policy.model
    a, b = tokens(12, m.spec.vocab_size, 1), tokens(6, m.spec.vocab_size, 2)
    full = m(torch.tensor([a]))[0]
    out = rep.step([{"id": "b", "tokens": b, "want": []}, {"id": "a", "tokens": a[:9], "want": [8, 2]}], ["b"])
    near(out, full[[8, 2]].detach(), 1e-4)
    for t in range(9, 12):
        near(rep.step([{"id": "a", "tokens": [a[t]], "want": [0]}])[0], full[t].detach(), 1e-4)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_trace_run_program(tmp_path, dtype):
    cfg, w, _ = load(tmp_path, "wide", "cuda", F32)
    prefill_all(load(tmp_path, "wide", "cuda", F32)[2].new_decoder(1, 8), [[1, 2, 3]], "cuda")
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
