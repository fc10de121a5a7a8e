"""Galodra: decoder-only language model with latent attention, gated residual branches, norms after the residual sum
and a learned average over depth; dense GeGLU or mixture-of-experts feed-forwards.

With ``X_0`` the embedding, ``x`` the stream and ``LN`` a layer norm with bias, layer ``i`` is

    x  <- LN1(a x + sigmoid(G1 x + b1) * mixer(x))
    X_(i+1) = LN2(a x + sigmoid(G2 x + b2) * ff(x))        (absent feed-forward: X_(i+1) = x)
    x  <- sum_{j <= i+1} w_ij X_j

and the logits are ``E LN(x)`` with the embedding table ``E``.  The mixer is sliding-window latent attention with a
sink per head (``models/latent.py``).  Experts are chosen by the largest sigmoid scores, which multiply the experts'
inputs.

Layout for B200: the stream, the norms, the gates' sigmoid, the router logits and the attention scores are float32;
projections read a bf16 copy of the stream that the norm kernel writes beside it.  Per layer one GEMM gives
``[q | latent and rotated key | G1 x]`` and one ``[router | G2 x]``; gate, residual sum, layer norm and depth average
are one kernel (``ops.post_norm``), which also keeps the history of streams.  Decoding caches one latent row per token
in a ring of ``window`` slots.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Mapping, Optional

import torch
from torch import nn

from .. import ops
from ..comm import Comm, SoloComm
from ..remat import remat_segment
from . import moe as M
from .latent import LatentAttention, LatentDims, fill_cache
from .lora import BaseQuantization, DenseLoraTargets, FusedLoraLinear, LoraSpec

DENSE_ACT = "gelu_pytorch_tanh"
EXPERT_ACT = "silu"


@dataclass(frozen=True)
class FeedForward:
    """``experts == 0``: one dense block of width ``ff``; otherwise ``experts`` blocks of width ``ff``, ``top`` used."""
    ff: int
    experts: int = 0
    top: int = 0


@dataclass(frozen=True)
class LayerSpec:
    mixer: LatentDims
    mlp: Optional[FeedForward]


@dataclass
class GalodraSpec:
    vocab_size: int
    hidden_size: int
    layers: list = field(default_factory=list)
    norm_eps: float = 1e-6
    alpha: float = 1.0
    max_position_embeddings: int = 4096     # rows of the rotation tables at first; they grow with the cache

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    def validate(self) -> None:
        if self.vocab_size <= 0 or self.hidden_size <= 0 or not self.layers:
            raise ValueError("galodra: vocab, width and layers must not be empty")
        for l in self.layers:
            l.mixer.validate()
            f = l.mlp
            if f is not None and (f.ff <= 0 or f.experts < 0 or (f.experts and not 0 < f.top <= f.experts)):
                raise ValueError("galodra: bad feed-forward sizes")


def galodra_spec(cfg: Mapping[str, Any]) -> GalodraSpec:
    layers = []
    for i, lc in enumerate(cfg["layers"]):
        if lc["type"] != "latent_attention":
            raise ValueError(f"galodra: layer {i} has unknown mixer type {lc['type']!r}")
        m = lc["mixer"]
        dims = LatentDims(heads=int(m["heads"]), dim=int(m["dim"]), rot=int(m["rot_dim"]), vdim=int(m["vdim"]),
                          rank=int(m["kv_rank"]), scale=float(m["scale"]), window=int(m["mask"]["size"]),
                          rope_base=float(m["rot"]["base"]), rope_dims=int(m["rot"]["dims"]), sink=True)
        if dims.window <= 0:
            raise ValueError(f"galodra: layer {i} has an empty window")
        mlp, f = None, lc.get("mlp")
        if f is not None:
            if f["kind"] == "dense":
                mlp = FeedForward(int(f["ff"]))
            elif f["kind"] == "moe":
                mlp = FeedForward(int(f["expert"]["ff"]), int(f["router"]["experts"]), int(f["router"]["top"]))
            else:
                raise ValueError(f"galodra: layer {i} has unknown feed-forward kind {f['kind']!r}")
        layers.append(LayerSpec(dims, mlp))
    spec = GalodraSpec(vocab_size=int(cfg["vocab"]), hidden_size=int(cfg["width"]), layers=layers,
                       norm_eps=float(cfg["norm"]["eps"]), alpha=float(cfg["postln_alpha"]))
    spec.validate()
    return spec


def _pad8(n: int) -> int:
    return (n + 7) // 8 * 8


class GalodraLayer(nn.Module):
    def __init__(self, spec: GalodraSpec, index: int, lora: Optional[LoraSpec], dtype, device, keep_transpose, quant,
                 trainable_base: bool = False):
        super().__init__()
        ls: LayerSpec = spec.layers[index]
        H = spec.hidden_size
        t = lora.targets if lora else DenseLoraTargets(*(False,) * 7)
        kw = dict(dtype=dtype, device=device, keep_transpose=keep_transpose, quant=quant, trainable_base=trainable_base)
        self.index, self.ff, self.eps, self.alpha, self.dtype = index, ls.mlp, spec.norm_eps, spec.alpha, dtype
        self.mix = LatentAttention(H, ls.mixer, spec.norm_eps, lora, t, kw, extra=H, extra_name="rg1")
        self.route_rows = 0
        self.gate_up = self.down = self.side = None
        reg = (lambda n, v: setattr(self, n, nn.Parameter(v))) if trainable_base else \
            (lambda n, v: self.register_buffer(n, v, persistent=False))
        full = lambda n, v: torch.full((n,), v, dtype=torch.float32, device=device)  # noqa: E731
        vectors = ["norm1", "norm1_b", "rg1_b"]
        if self.ff is not None:
            vectors += ["norm2", "norm2_b", "rg2_b"]
            if self.ff.experts:
                # router rows padded to eight so that the gate rows behind them start on a 16-byte boundary
                self.route_rows = _pad8(self.ff.experts)
                reg("experts_gate_up", torch.zeros(self.ff.experts, 2 * self.ff.ff, H, dtype=dtype, device=device))
                reg("experts_down", torch.zeros(self.ff.experts, H, self.ff.ff, dtype=dtype, device=device))
            else:
                self.gate_up = FusedLoraLinear(H, [self.ff.ff] * 2, ("gate", "up"), (t.mlp_gate, t.mlp_up), lora, **kw)
                self.gate_up.enable_glu_layout()
                self.down = FusedLoraLinear(self.ff.ff, [H], ("down",), (t.mlp_down,), lora, **kw)
            self.side = FusedLoraLinear(H, [self.route_rows, H] if self.route_rows else [H],
                                        ("router", "rg2") if self.route_rows else ("rg2",),
                                        (False,) * (2 if self.route_rows else 1), None,
                                        **dict(kw, quant=BaseQuantization.NONE))     # the router keeps its exact weights
        for n in vectors:
            reg(n, full(H, 0.0 if n.endswith("_b") else 1.0))
        coef = torch.zeros(index + 2, dtype=torch.float32, device=device)
        coef[-1] = 1.0
        reg("depth_coef", coef)

    def projections(self):
        ps = list(self.mix.projections())
        for p in (self.gate_up, self.down, self.side):
            if p is not None:
                ps.append(p)
        return ps

    def adapter_params(self):
        out = []
        for p in self.projections():
            out += p.adapter_params()
        return out

    @torch.no_grad()
    def refresh_derived(self):
        self.mix.refresh_derived()

    # ------------------------------------------------------------------ parts
    def _feed_forward(self, x16, merged):
        """``(ff(x), gate logits)`` of the stream's low-precision copy ``[..., H]``."""
        f = self.ff
        lin = (lambda m, z: m.forward_merged(z)) if merged else (lambda m, z: m(z))
        if not f.experts:
            mid = self.gate_up.forward_merged_glu(x16, DENSE_ACT) if merged else ops.swiglu(self.gate_up(x16), DENSE_ACT)
            return lin(self.down, mid), lin(self.side, x16)
        x2 = x16.reshape(-1, x16.shape[-1])
        w = self.side.weight
        if x2.shape[0] <= 256:              # decode: one launch for the router and the gate
            both = ops.linear_f32(x2, w)
            logits, gate = both[:, :f.experts], both[:, self.route_rows:]
        else:
            logits, gate = ops.linear_f32(x2, w[:f.experts]), ops.lora_linear(x2, w[self.route_rows:], None, None)
        y = M.routed_experts(x2, logits, self.experts_gate_up, self.experts_down, f.top, score="sigmoid", renorm=False,
                             weight_input=True, act=EXPERT_ACT)
        return y.view(x16.shape), gate.reshape(*x16.shape[:-1], -1)

    def _after_mixer(self, x, y, g, history=None, out=None):
        """First norm; for a layer without feed-forward also the depth average."""
        return ops.post_norm(x, y, self.norm1, self.norm1_b, self.eps, self.alpha, g, self.rg1_b, history=history,
                             coef=None if history is None else self.depth_coef, cast=self.dtype, out=out)

    def _after_ff(self, x, y, g, history, out=None):
        return ops.post_norm(x, y, self.norm2, self.norm2_b, self.eps, self.alpha, g, self.rg2_b, history=history,
                             coef=self.depth_coef, cast=self.dtype, out=out)

    # ------------------------------------------------------------------ passes
    def mixer_half(self, x, positions, cos, sin, merged=False):
        y, g = self.mix(x.to(self.dtype), positions, cos, sin, merged)
        return self._after_mixer(x, y, g)[0]

    def ff_half(self, x, merged=False):
        """``X_(i+1)`` without the depth average (training segments)."""
        y, g = self._feed_forward(x.to(self.dtype), merged)
        return ops.post_norm(x, y, self.norm2, self.norm2_b, self.eps, self.alpha, g, self.rg2_b)[0]

    def run(self, x, x16, mixed, history, out, merged):
        """Everything behind the mixer for the grad-free passes: ``mixed = (y, gate logits)``."""
        y, g = mixed
        if self.ff is None:
            return self._after_mixer(x, y, g, history, out)[:2]
        x, x16, _ = self._after_mixer(x, y, g)
        y, g = self._feed_forward(x16, merged)
        return self._after_ff(x, y, g, history, out)[:2]


class GalodraGradModel(nn.Module):
    """Policy network: grad-bearing scoring forward plus the cached decoder."""

    def __init__(self, spec: GalodraSpec, lora: Optional[LoraSpec] = None, *, dtype=torch.float32, device=None,
                 keep_transpose: Optional[bool] = None, quant: BaseQuantization = BaseQuantization.NONE,
                 remat: bool = False, full_ft: bool = False):
        super().__init__()
        spec.validate()
        self.spec, self.lora, self.remat, self.full_ft, self.dtype = spec, lora, remat, full_ft, dtype
        dev = torch.device(device) if device is not None else torch.device("cpu")
        if keep_transpose is None:
            keep_transpose = dev.type == "cuda" and not full_ft
        self.keep_transpose = keep_transpose
        emb = torch.zeros(spec.vocab_size, spec.hidden_size, dtype=dtype, device=dev)
        fn = torch.ones(spec.hidden_size, dtype=torch.float32, device=dev)
        if full_ft:
            self.embed, self.final_norm, self.final_norm_b = nn.Parameter(emb), nn.Parameter(fn), nn.Parameter(torch.zeros_like(fn))
        else:
            self.register_buffer("embed", emb, persistent=False)
            self.register_buffer("final_norm", fn, persistent=False)
            self.register_buffer("final_norm_b", torch.zeros_like(fn), persistent=False)
        self.register_buffer("head_t", None, persistent=False)
        self.layers = nn.ModuleList([GalodraLayer(spec, i, None if full_ft else lora, dtype, dev, keep_transpose, quant,
                                                  full_ft) for i in range(spec.num_hidden_layers)])
        self._tables: dict = {}
        self._positions = 0
        self.ensure_positions(spec.max_position_embeddings)

    # ------------------------------------------------------------ plumbing
    def ensure_positions(self, n: int) -> None:
        """Rotation tables for positions ``0 .. n-1`` (one pair per distinct base and width)."""
        if n <= self._positions:
            return
        self._positions = n
        self._tables = {}
        for l in self.spec.layers:
            key = (l.mixer.rope_base, l.mixer.turned)
            if key not in self._tables:
                cos, sin = ops.rope_tables(ops.default_inv_freq(key[1], key[0]), n)
                self._tables[key] = (cos.to(self.embed.device), sin.to(self.embed.device))

    def tables(self, layer: GalodraLayer):
        return self._tables[(layer.mix.dims.rope_base, layer.mix.dims.turned)]

    def _apply(self, fn, *a, **kw):
        super()._apply(fn, *a, **kw)
        n, self._positions = self._positions, 0
        self.ensure_positions(n)            # the tables live outside the buffer registry
        return self

    def head_weight(self):
        return self.embed

    @torch.no_grad()
    def refresh_head(self):
        if self.keep_transpose:
            self.head_t = self.embed.t().contiguous()

    def trainable_params(self):
        if self.full_ft:
            return [p for p in self.parameters()]
        out = []
        for l in self.layers:
            out += l.adapter_params()
        return out

    def set_adapter_enabled(self, on: bool):
        for l in self.layers:
            for p in l.projections():
                p.enabled = on

    def lora_recipe(self) -> str:
        if self.full_ft:
            return "full_ft"
        return self.lora.recipe() if self.lora else "none"

    @torch.no_grad()
    def merge_adapters(self):
        for l in self.layers:
            for p in l.projections():
                p.merge()
            l.refresh_derived()

    @torch.no_grad()
    def init_random(self, seed: int = 0, std: float = 0.02):
        g = torch.Generator().manual_seed(seed)
        dev = self.embed.device
        rnd = lambda shape: (torch.randn(shape, generator=g) * std).to(self.dtype).to(dev)  # noqa: E731
        if dev.type == "cuda":          # device-side generation for the large synthetic benchmarks
            gg = torch.Generator(device=dev).manual_seed(seed)
            rnd = lambda shape: (torch.randn(shape, generator=gg, device=dev, dtype=torch.float32) * std).to(self.dtype)  # noqa: E731
        self.embed.copy_(rnd(self.embed.shape))
        for l in self.layers:
            for p in l.projections():
                p.set_weight(rnd(p.weight.shape))
                p.init_adapters(g)
            if l.route_rows:
                for e in range(l.ff.experts):
                    l.experts_gate_up[e].copy_(rnd(l.experts_gate_up.shape[1:]))
                    l.experts_down[e].copy_(rnd(l.experts_down.shape[1:]))
            l.depth_coef.fill_(0.0)
            l.depth_coef[0] = 0.25
            l.depth_coef[-1] = 0.75
            l.refresh_derived()
        self.refresh_head()

    # ------------------------------------------------------------- forward
    def forward_hidden(self, ids, comm: Optional[Comm] = None, merged: bool = False, store=None,
                       detached: bool = False) -> torch.Tensor:
        """Final stream ``[B,S,H]`` (float32).  ``store(i, rows)`` receives every layer's latent rows (prefill)."""
        B, S = ids.shape
        self.ensure_positions(S)
        positions = torch.arange(S, device=ids.device)
        e = ops.embedding(ids, self.embed)
        if torch.is_grad_enabled() and not detached:
            return self._forward_train(e.float(), positions, merged)
        x16, x = e, e.float()
        history = torch.empty(len(self.layers) + 1, *x.shape, dtype=torch.float32, device=x.device)
        history[0].copy_(x)
        for i, layer in enumerate(self.layers):
            cos, sin = self.tables(layer)
            keep = None if store is None else (lambda rows, i=i: store(i, rows))
            mixed = layer.mix(x16, positions, cos, sin, merged, keep)
            x, x16 = layer.run(x, x16, mixed, history[:i + 1], history[i + 1], merged)
        return x

    def _forward_train(self, x, positions, merged):
        xs = [x]
        for layer in self.layers:
            cos, sin = self.tables(layer)
            params = layer.adapter_params() if not self.full_ft else list(layer.parameters())
            halves = [lambda z, l=layer, c=cos, s=sin: l.mixer_half(z, positions, c, s, merged)]
            if layer.ff is not None:
                halves.append(lambda z, l=layer: l.ff_half(z, merged))
            for half in halves:
                x = remat_segment(half, x, params) if self.remat else half(x)
            xs.append(x)
            x = layer.depth_coef[0] * xs[0]
            for j in range(1, len(xs)):
                x = x + layer.depth_coef[j] * xs[j]
        return x

    def final_hidden(self, x) -> torch.Tensor:
        """Last norm, in the compute dtype."""
        return ops.post_norm(x, None, self.final_norm, self.final_norm_b, self.spec.norm_eps, cast=self.dtype)[1]

    def logits(self, x) -> torch.Tensor:
        """Stream rows ``[N,H]`` -> float32 logits ``[N,V]``."""
        return ops.linear_f32(self.final_hidden(x), self.embed)

    def forward(self, ids, comm: Optional[Comm] = None) -> torch.Tensor:
        x = self.forward_hidden(ids, comm)
        return self.logits(x.reshape(-1, x.shape[-1])).view(*ids.shape, -1)

    def token_logprobs(self, ids, win_start, targets, temperature: float = 1.0, comm: Optional[Comm] = None):
        x = self.forward_hidden(ids, comm, detached=not torch.is_grad_enabled())
        B, L = targets.shape
        idx = (win_start.view(B, 1).long() + torch.arange(L, device=ids.device)[None, :]).clamp(max=ids.shape[1] - 1)
        xw = torch.gather(x, 1, idx[:, :, None].expand(B, L, x.shape[-1]))
        h = self.final_hidden(xw.reshape(B * L, -1))
        return ops.logprob_gather(h, self.embed, targets.reshape(-1), temperature, 0.0, head_wt=self.head_t).view(B, L)

    def new_decoder(self, batch: int, max_len: int, comm: Optional[Comm] = None) -> "GalodraCachedDecoder":
        return GalodraCachedDecoder(self, batch, max_len, comm or SoloComm())


class GalodraCachedDecoder:
    """Cached, grad-free twin over merged weights: per layer one ring of ``window`` latent rows for every batch row."""

    supports_retirement = True

    def __init__(self, model: GalodraGradModel, batch: int, max_len: int, comm: Comm):
        self.m, self.comm, self.batch, self.max_len = model, comm, batch, max_len
        model.ensure_positions(max_len)
        dev = model.embed.device
        self.slots = [l.mix.slots(max_len) for l in model.layers]
        self.cache = [torch.zeros(batch, n, l.mix.dims.row_width(), dtype=model.dtype, device=dev)
                      for l, n in zip(model.layers, self.slots)]
        self.kv_len = torch.zeros(batch, dtype=torch.int32, device=dev)

    def cache_bytes(self) -> int:
        return sum(t.numel() * t.element_size() for t in self.cache)

    @torch.no_grad()
    def prefill(self, ids, lens, rows=None, at=None):
        """Right-padded prompts ``[P,L]`` into cache rows ``rows``; logits ``[P,V]`` of the last tokens, or of the
        places ``at = (prompt indices, positions)``."""
        m = self.m
        P, L = ids.shape
        if L > self.max_len:
            raise ValueError(f"prompt of {L} tokens exceeds the cache's {self.max_len}")
        rows = torch.arange(P, device=ids.device) if rows is None else rows
        x = m.forward_hidden(ids, self.comm, merged=True, detached=True,
                             store=lambda i, lat: fill_cache(self.cache[i], rows, lat, lens))
        self.kv_len[rows] = lens.to(torch.int32)
        return m.logits(x[(torch.arange(P, device=ids.device), (lens - 1).long()) if at is None else at])

    @torch.no_grad()
    def broadcast_groups(self, group: int):
        P = self.batch // group
        src = torch.arange(P, device=self.kv_len.device).repeat_interleave(group)
        for c in self.cache:
            c.copy_(c[src])
        self.kv_len.copy_(self.kv_len[src])

    def _counts(self, active):
        """Occupied slots per row after this token, for every distinct ring size; 0 for retired rows."""
        nxt = self.kv_len + 1
        if active is not None:
            nxt = nxt * active.to(torch.int32)
        return {n: nxt.clamp(max=n) for n in set(self.slots)}

    def kv_tokens_read(self, active: Optional[torch.Tensor] = None) -> torch.Tensor:
        """Latent rows that the next ``decode`` call reads, averaged over the layers."""
        counts = self._counts(active)
        return torch.stack([counts[n].sum() for n in self.slots]).float().mean()

    @torch.no_grad()
    def decode(self, tokens, active: Optional[torch.Tensor] = None):
        """Feed one token per row; next-token logits ``[B,V]`` float32.  Rows with ``active[b]`` false stay in the
        fixed-shape batch, attend to nothing and keep their length."""
        m = self.m
        x16 = ops.embedding(tokens, m.embed)
        x = x16.float()
        history = torch.empty(len(m.layers) + 1, *x.shape, dtype=torch.float32, device=x.device)
        history[0].copy_(x)
        counts = self._counts(active)
        for i, (layer, cache) in enumerate(zip(m.layers, self.cache)):
            cos, sin = m.tables(layer)
            mixed = layer.mix.decode(x16, self.kv_len, counts[self.slots[i]], cos, sin, cache)
            x, x16 = layer.run(x, x16, mixed, history[:i + 1], history[i + 1], True)
        self.kv_len += 1 if active is None else active.to(torch.int32)
        return m.logits(x)


@torch.no_grad()
def load_galodra_weights(model: GalodraGradModel, src) -> None:
    to = lambda t: t.to(model.dtype)  # noqa: E731
    f32 = lambda n: src.get(n).float()  # noqa: E731
    cat = lambda *names: to(torch.cat([src.get(n) for n in names], 0))  # noqa: E731
    model.embed.copy_(to(src.get("embed")))
    model.final_norm.copy_(f32("final.norm"))
    model.final_norm_b.copy_(f32("final.norm.b"))
    for i, l in enumerate(model.layers):
        b = f"l{i}."
        l.mix.inp.set_weight(cat(b + "mix.q", b + "mix.dkv", b + "rg1"))
        l.mix.up.set_weight(cat(b + "mix.uk", b + "mix.uv"))
        l.mix.out.set_weight(to(src.get(b + "mix.o")))
        l.mix.latent_norm.copy_(f32(b + "mix.dkv.norm"))
        l.mix.sink.copy_(f32(b + "mix.sink"))
        l.norm1.copy_(f32(b + "norm1"))
        l.norm1_b.copy_(f32(b + "norm1.b"))
        l.rg1_b.copy_(f32(b + "rg1.b"))
        l.depth_coef.copy_(f32(b + "dwa"))
        l.refresh_derived()
        if l.ff is None:
            continue
        l.norm2.copy_(f32(b + "norm2"))
        l.norm2_b.copy_(f32(b + "norm2.b"))
        l.rg2_b.copy_(f32(b + "rg2.b"))
        rg2 = src.get(b + "rg2")
        if not l.ff.experts:
            l.gate_up.set_weight(cat(b + "mlp.gate", b + "mlp.up"))
            l.down.set_weight(to(src.get(b + "mlp.down")))
            l.side.set_weight(to(rg2))
            continue
        router = src.get(b + "mlp.router")
        pad = router.new_zeros(l.route_rows - router.shape[0], router.shape[1])
        l.side.set_weight(to(torch.cat([router, pad, rg2], 0)))
        for e in range(l.ff.experts):
            eb = f"{b}mlp.e{e}."
            l.experts_gate_up[e].copy_(cat(eb + "gate", eb + "up"))
            l.experts_down[e].copy_(to(src.get(eb + "down")))
    model.refresh_head()


def load_galodra(model_dir: str, opts):
    from .loader import TensorSource, _identity, read_config
    cfg = read_config(model_dir)
    spec = galodra_spec(cfg)
    if opts.max_position_embeddings:
        spec.max_position_embeddings = opts.max_position_embeddings
    if opts.tp is not None:
        raise ValueError("tensor parallelism is not supported for the Galodra family")
    if opts.ep is not None and opts.ep[1] > 1:
        raise ValueError("expert parallelism is not supported for the Galodra family")
    model = GalodraGradModel(spec, None if opts.full_ft else opts.lora, dtype=opts.dtype, device=opts.device,
                             quant=opts.quantization, remat=opts.remat, full_ft=opts.full_ft)
    src = TensorSource(model_dir)
    load_galodra_weights(model, src)
    g = torch.Generator().manual_seed(opts.adapter_seed)
    for l in model.layers:
        for pr in l.projections():
            pr.init_adapters(g)
    return model, _identity(model_dir, cfg, src, opts)
