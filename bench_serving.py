"""Prefill and decode throughput of a serving-sized slice of a family (``python bench.py --serving``).

Each size runs the Galodra or the Mifutar family beside the existing family closest to it, at equal width, depth, head
count, feed-forward width and window, with random weights in bf16 and no adapters:

    dense-4k   8 layers, width 4096, 32 heads (latent 512, 128 + 64 score entries, values 128), window 1024, GeGLU 12288
               beside Gemma-style sliding-window layers (32 query / 16 key-value heads of 128)
    dense-1k   12 layers, width 1024, 16 heads (latent 256, 64 + 32, values 64), window 512, GeGLU 4096
               beside Gemma-style layers (16 / 8 heads of 64)
    moe-2k     8 layers, width 2048, 16 heads (latent 512, 128 + 64, values 128), window 1024, 64 experts of 768, top 8
               beside Qwen3.5-style full-attention layers (16 / 2 heads of 256) with the same experts
    hybrid-4k  8 layers, width 4096, two streams, feed-forward 12288: three Mamba-2 layers (128 heads of 64 x 128 state, 8
               groups) to one biased attention layer (32 / 8 heads of 128, window 1024), beside Qwen3.5-style layers
               (GatedDeltaNet with 64 heads of 128 x 128 state, full attention with the same heads)
    hybrid-2k  12 layers, width 2048, feed-forward 6144: 64 heads of 64 x 128, 4 groups; 16 / 4 heads of 128, beside the same
               with 32 heads of 128 x 128
    hybrid-1k  12 layers, width 1024, feed-forward 4096: 32 heads of 64 x 128, 1 group; 16 / 4 heads of 64, beside the same
               with 16 heads of 128 x 128

Prefill: 8 prompts of 2048 tokens.  Decode: 128 rows at 1024 cached tokens, one step replayed from a CUDA graph.  Times
are CUDA events over ``steps`` calls after ``warmup``; weights and caches are larger than L2.  One JSON line a model.
"""
from __future__ import annotations

import json

VOCAB = 32768
PROMPTS, PROMPT_LEN, ROWS, CONTEXT = 8, 2048, 128, 1024

SIZES = {
    "dense-4k": dict(layers=8, width=4096, heads=32, kv=16, dim=128, rot=64, vdim=128, rank=512, window=1024, ff=12288),
    "dense-1k": dict(layers=12, width=1024, heads=16, kv=8, dim=64, rot=32, vdim=64, rank=256, window=512, ff=4096),
    "moe-2k": dict(layers=8, width=2048, heads=16, kv=2, dim=128, rot=64, vdim=128, rank=512, window=1024, ff=768, experts=64, top=8),
    "hybrid-4k": dict(family="mifutar", layers=8, width=4096, heads=32, kv=8, dim=128, window=1024, ff=12288, ssm=128, groups=8),
    "hybrid-2k": dict(family="mifutar", layers=12, width=2048, heads=16, kv=4, dim=128, window=1024, ff=6144, ssm=64, groups=4),
    "hybrid-1k": dict(family="mifutar", layers=12, width=1024, heads=16, kv=4, dim=64, window=1024, ff=4096, ssm=32, groups=1),
}


def build(size: str, family: str, device):
    import torch
    s = SIZES[size]
    kw = dict(dtype=torch.bfloat16, device=device, keep_transpose=False)
    max_len = max(PROMPT_LEN, CONTEXT) + 256
    if family == "galodra":
        from ferrl_b200.models.galodra import FeedForward, GalodraGradModel, GalodraSpec, LatentDims, LayerSpec
        dims = LatentDims(s["heads"], s["dim"], s["rot"], s["vdim"], s["rank"], (s["dim"] + s["rot"]) ** -0.5, s["window"], 1e4, 0, True)
        ff = FeedForward(s["ff"], s.get("experts", 0), s.get("top", 0))
        m = GalodraGradModel(GalodraSpec(VOCAB, s["width"], [LayerSpec(dims, ff)] * s["layers"], alpha=2.0), None, **kw)
    elif family == "mifutar":
        from ferrl_b200.models.mifutar import BiasAttentionDims, ClippedFeedForward, LayerSpec, Mamba2Dims, MifutarGradModel, MifutarSpec
        ff = ClippedFeedForward(s["ff"], 7.0)
        rec = LayerSpec(Mamba2Dims(s["ssm"], 64, 128, s["groups"], 4, s["groups"]), ff)
        att = LayerSpec(BiasAttentionDims(s["heads"], s["kv"], s["dim"], s["dim"] ** -0.5, s["window"], 32, 128), ff)
        m = MifutarGradModel(MifutarSpec(VOCAB, s["width"], ([rec] * 3 + [att]) * (s["layers"] // 4), streams=2), None, **kw)
    elif "ssm" in s:
        from ferrl_b200.models.qwen35 import Qwen35GradModel, Qwen35Spec
        m = Qwen35GradModel(Qwen35Spec(VOCAB, s["width"], s["layers"], s["heads"], s["kv"], s["dim"], s["ff"],
                                       (["linear_attention"] * 3 + ["full_attention"]) * (s["layers"] // 4), max_position_embeddings=max_len,
                                       tie_word_embeddings=False, lin_k_heads=s["ssm"] // 4, lin_v_heads=s["ssm"] // 2), None, **kw)
    elif "experts" in s:
        from ferrl_b200.models.qwen35 import MoeDims, Qwen35GradModel, Qwen35Spec
        m = Qwen35GradModel(Qwen35Spec(VOCAB, s["width"], s["layers"], s["heads"], s["kv"], 256, s["ff"], ["full_attention"] * s["layers"],
                                       max_position_embeddings=max_len, moe=MoeDims(s["experts"], s["top"], s["ff"], 0)), None, **kw)
    else:
        from ferrl_b200.models.gemma4 import Gemma4GradModel, Gemma4Spec
        m = Gemma4GradModel(Gemma4Spec(VOCAB, s["width"], s["layers"], s["heads"], s["kv"], s["vdim"], s["vdim"], s["kv"], s["ff"],
                                       ["sliding_attention"] * s["layers"], s["window"], attention_k_eq_v=False, final_logit_softcapping=0.0,
                                       max_position_embeddings=max_len), None, **kw)
    m.init_random(1, 0.02)
    m.merge_adapters()
    return m


def measure(model, steps: int, warmup: int, device) -> dict:
    import torch

    def timed(fn):
        for _ in range(warmup):
            fn()
        torch.cuda.synchronize()
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record()
        for _ in range(steps):
            fn()
        b.record()
        torch.cuda.synchronize()
        return a.elapsed_time(b) / steps
    g = torch.Generator(device=device).manual_seed(0)
    ids = lambda n, L: torch.randint(0, VOCAB, (n, L), generator=g, device=device)  # noqa: E731
    with torch.no_grad():
        dec = model.new_decoder(PROMPTS, PROMPT_LEN + 128)
        prompt, lens = ids(PROMPTS, PROMPT_LEN), torch.full((PROMPTS,), PROMPT_LEN, device=device)
        pre = timed(lambda: dec.prefill(prompt, lens))
        del dec
        dec = model.new_decoder(ROWS, CONTEXT + 128)
        for r in range(0, ROWS, 16):
            dec.prefill(ids(16, CONTEXT), torch.full((16,), CONTEXT, device=device), torch.arange(r, r + 16, device=device))
        tok = ids(1, ROWS)[0]
        length = dec.kv_len.clone()

        def step():
            dec.kv_len.copy_(length)            # every step at the same context
            dec.decode(tok)
        step()
        torch.cuda.synchronize()
        graph = torch.cuda.CUDAGraph()
        with torch.cuda.graph(graph):
            step()
        one = timed(graph.replay)
        cache = dec.cache_bytes()
    return {"prefill_ms": round(pre, 3), "prefill_tok_s": round(PROMPTS * PROMPT_LEN / pre * 1e3), "decode_ms": round(one, 4),
            "decode_tok_s": round(ROWS / one * 1e3), "cache_mb": round(cache / 2 ** 20, 1)}


def main(sizes, steps: int, warmup: int, clock_sampler) -> int:
    import torch
    from ferrl_b200.ops import cuda as C
    device = torch.device("cuda", 0)
    torch.cuda.set_device(device)
    for size in sizes:
        for family in (SIZES[size].get("family", "galodra"), "closest"):
            model = build(size, family, device)
            clocks = clock_sampler(0)
            clocks.start()
            before = C.launches()
            out = measure(model, steps, warmup, device)
            print(json.dumps({"serving": size, "model": type(model).__name__, **out, "steps": steps, "warmup": warmup, "dtype": "bf16",
                              "data": "random weights and token ids", "gpu_launches": C.launches() - before, "clocks": clocks.stop()}), flush=True)
            if C.kernel_status() != 0:
                raise SystemExit(f"kernel status {C.kernel_status()}")
            del model
            torch.cuda.empty_cache()
    return 0
