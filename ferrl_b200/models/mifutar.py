"""Mifutar: decoder-only language model of Mamba-2 and distance-biased attention layers joined by hyper-connections,
with a clipped gated feed-forward and sinusoidal positions.

Every token carries ``streams`` residual streams, at first all equal to ``E[token] + sinusoid(position)``.  A sublayer
(mixer, then feed-forward where a layer has one) reads one mixture of them and writes to all:

    y = sublayer(norm(sum_s in[s] x_s)),      x_t <- sum_s mix[s, t] x_s + out[t] y

and the logits are ``scale * W_head norm(sum_s x_s)``.  The norms are RMS norms with weights around zero.  Mixers are
``models/mamba2.py`` and ``models/bias_attention.py``; the feed-forward is ``g sigmoid(1.702 g) (u + 1)`` of clipped
projections.

Layout for B200: the streams are float32 ``[..., streams, width]``; one kernel (``ops.hyper_norm``) closes a sublayer and
opens the next: it reads the streams once, writes them once and leaves the normed mixture in the compute dtype for the
projection behind it.  The output scale rides in the last norm.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Mapping, Optional, Union

import torch
from torch import nn

from .. import ops
from ..comm import Comm, SoloComm
from ..remat import remat_segment
from .bias_attention import BiasAttention, BiasAttentionDims
from .lora import BaseQuantization, DenseLoraTargets, FusedLoraLinear, LoraSpec
from .mamba2 import Mamba2, Mamba2Dims


@dataclass(frozen=True)
class ClippedFeedForward:
    ff: int
    limit: float


@dataclass(frozen=True)
class LayerSpec:
    mixer: Union[BiasAttentionDims, Mamba2Dims]
    mlp: Optional[ClippedFeedForward]


@dataclass
class MifutarSpec:
    vocab_size: int
    hidden_size: int
    layers: list = field(default_factory=list)
    streams: int = 1
    norm_eps: float = 1e-6
    logit_scale: float = 1.0
    max_position_embeddings: int = 4096     # rows of the position tables at first; they grow with the cache

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    def validate(self) -> None:
        if self.vocab_size <= 0 or self.hidden_size <= 0 or not self.layers or self.streams <= 0:
            raise ValueError("mifutar: vocab, width, streams and layers must not be empty")
        for l in self.layers:
            l.mixer.validate()
            if l.mlp is not None and (l.mlp.ff <= 0 or l.mlp.limit < 0):
                raise ValueError("mifutar: bad feed-forward sizes")


def mifutar_spec(cfg: Mapping[str, Any], bias_buckets: Mapping[int, int]) -> MifutarSpec:
    """``bias_buckets``: rows of the bias table of every attention layer (the configuration leaves them to the checkpoint)."""
    layers = []
    for i, lc in enumerate(cfg["layers"]):
        m, kind = lc["mixer"], lc["type"]
        if kind == "attention":
            if int(m.get("vdim", m["dim"])) != int(m["dim"]):
                raise ValueError(f"mifutar: layer {i}: values that are keys have the keys' size")
            dims = BiasAttentionDims(heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]), scale=float(m["scale"]),
                                     window=int(m["mask"]["size"]), buckets=int(bias_buckets[i]), bias_max=int(m["bias_max"]))
        elif kind == "mamba2":
            dims = Mamba2Dims(heads=int(m["heads"]), vdim=int(m["vdim"]), state=int(m["state"]), groups=int(m["groups"]), conv=int(m["conv"]),
                              norm_groups=int(m["norm_groups"]))
        else:
            raise ValueError(f"mifutar: layer {i} has unknown mixer type {kind!r}")
        mlp, f = None, lc.get("mlp")
        if f is not None:
            if f["kind"] != "dense":
                raise ValueError(f"mifutar: layer {i} has unknown feed-forward kind {f['kind']!r}")
            mlp = ClippedFeedForward(int(f["ff"]), float(f["limit"]))
        layers.append(LayerSpec(dims, mlp))
    spec = MifutarSpec(vocab_size=int(cfg["vocab"]), hidden_size=int(cfg["width"]), layers=layers, streams=int(cfg["streams"]),
                       norm_eps=float(cfg["norm"]["eps"]), logit_scale=float(cfg["logit_scale"]))
    spec.validate()
    return spec


class MifutarLayer(nn.Module):
    def __init__(self, spec: MifutarSpec, index: int, lora: Optional[LoraSpec], letters: str, dtype, device, keep_transpose, quant,
                 trainable_base: bool = False):
        super().__init__()
        ls: LayerSpec = spec.layers[index]
        H, s = spec.hidden_size, spec.streams
        t = lora.targets if lora else DenseLoraTargets(*(False,) * 7)
        kw = dict(dtype=dtype, device=device, keep_transpose=keep_transpose, quant=quant, trainable_base=trainable_base)
        self.ff, self.eps, self.dtype = ls.mlp, spec.norm_eps, dtype
        if isinstance(ls.mixer, Mamba2Dims):
            self.mix = Mamba2(H, ls.mixer, spec.norm_eps, lora, letters, kw)
        else:
            self.mix = BiasAttention(H, ls.mixer, lora, t, kw)
        self.gate_up = self.down = None
        if self.ff is not None:
            self.act = ops.ClippedGlu(self.ff.limit)
            self.gate_up = FusedLoraLinear(H, [self.ff.ff] * 2, ("gate", "up"), (t.mlp_gate, t.mlp_up), lora, **kw)
            self.gate_up.enable_glu_layout()
            self.down = FusedLoraLinear(self.ff.ff, [H], ("down",), (t.mlp_down,), lora, **kw)

        def reg(n, v):
            if trainable_base:
                setattr(self, n, nn.Parameter(v))
            else:
                self.register_buffer(n, v, persistent=False)
        for q in self.sublayers():
            reg(f"norm{q}", torch.zeros(H, dtype=torch.float32, device=device))
            reg(f"hc{q}_in", torch.full((s,), 1.0 / s, dtype=torch.float32, device=device))
            reg(f"hc{q}_out", torch.ones(s, dtype=torch.float32, device=device))
            reg(f"hc{q}_mix", torch.eye(s, dtype=torch.float32, device=device))

    def sublayers(self):
        return (1,) if self.ff is None else (1, 2)

    def projections(self):
        return [p for p in (*self.mix.projections(), self.gate_up, self.down) if p is not None]

    def adapter_params(self):
        out = []
        for p in self.projections():
            out += p.adapter_params()
        return out

    # ------------------------------------------------------------------ parts
    def enter(self, q: int, x, pending):
        """Close the sublayer before (``pending``: its output and coefficients) and open sublayer ``q``."""
        return ops.hyper_norm(x, *pending, getattr(self, f"hc{q}_in"), getattr(self, f"norm{q}"), self.eps, self.dtype)

    def leave(self, q: int, y):
        return y, getattr(self, f"hc{q}_mix"), getattr(self, f"hc{q}_out")

    def feed_forward(self, h, merged: bool):
        if merged:
            return self.down.forward_merged(self.gate_up.forward_merged_glu(h, self.act))
        return self.down(ops.swiglu(self.gate_up(h), self.act))

    def run(self, x, pending, mixer):
        """Grad-free: ``mixer(h)`` and the feed-forward on streams that are rewritten in place."""
        x, h = self.enter(1, x, pending)
        pending = self.leave(1, mixer(h))
        if self.ff is not None:
            x, h = self.enter(2, x, pending)
            pending = self.leave(2, self.feed_forward(h, True))
        return x, pending

    def half(self, q: int, x, merged: bool = False):
        """Sublayer ``q`` as a function of the streams (training segments)."""
        _, h = self.enter(q, x, (None, None, None))
        y = self.mix(h, merged) if q == 1 else self.feed_forward(h, merged)
        return ops.hyper_mix(x, *self.leave(q, y))


class MifutarGradModel(nn.Module):
    """Policy network: grad-bearing scoring forward plus the cached decoder."""

    def __init__(self, spec: MifutarSpec, lora: Optional[LoraSpec] = None, *, dtype=torch.float32, device=None,
                 keep_transpose: Optional[bool] = None, quant: BaseQuantization = BaseQuantization.NONE,
                 remat: bool = False, full_ft: bool = False, recurrent_targets: str = ""):
        """``recurrent_targets``: adapted projections of the Mamba-2 layers (letters of q z a o)."""
        super().__init__()
        spec.validate()
        self.spec, self.lora, self.remat, self.full_ft, self.dtype = spec, lora, remat, full_ft, dtype
        self.letters = "".join(c for c in "qzao" if lora is not None and not full_ft and c in recurrent_targets.replace("i", "qz"))
        dev = torch.device(device) if device is not None else torch.device("cpu")
        if keep_transpose is None:
            keep_transpose = dev.type == "cuda" and not full_ft
        self.keep_transpose = keep_transpose
        table = lambda: torch.zeros(spec.vocab_size, spec.hidden_size, dtype=dtype, device=dev)  # noqa: E731
        fn = torch.zeros(spec.hidden_size, dtype=torch.float32, device=dev)
        if full_ft:
            self.embed, self.final_norm, self.head = nn.Parameter(table()), nn.Parameter(fn), nn.Parameter(table())
        else:
            self.register_buffer("embed", table(), persistent=False)
            self.register_buffer("final_norm", fn, persistent=False)
            self.register_buffer("head", table(), persistent=False)
        self.register_buffer("head_t", None, persistent=False)
        self.register_buffer("pe", None, persistent=False)
        self.layers = nn.ModuleList([MifutarLayer(spec, i, None if full_ft else lora, self.letters, dtype, dev, keep_transpose, quant, full_ft)
                                     for i in range(spec.num_hidden_layers)])
        self.ensure_positions(spec.max_position_embeddings)

    # ------------------------------------------------------------ plumbing
    def ensure_positions(self, n: int) -> None:
        """Sinusoids and attention biases for positions ``0 .. n-1``."""
        if self.pe is None or self.pe.shape[0] < n:
            self.pe = ops.sinusoid_table(n, self.spec.hidden_size).to(self.embed.device)
        for l in self.layers:
            l.mix.ensure_positions(n)

    def head_weight(self):
        return self.head

    @torch.no_grad()
    def refresh_head(self):
        if self.keep_transpose:
            self.head_t = self.head.t().contiguous()

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
        if not self.lora:
            return "none"
        return self.lora.recipe() + (f"|gdn:{self.letters}" if self.letters else "")

    @torch.no_grad()
    def merge_adapters(self):
        for l in self.layers:
            for p in l.projections():
                p.merge()
            l.mix.refresh_derived()

    @torch.no_grad()
    def init_random(self, seed: int = 0, std: float = 0.02):
        g = torch.Generator().manual_seed(seed)
        dev = self.embed.device
        gg = torch.Generator(device=dev).manual_seed(seed) if dev.type == "cuda" else g   # device-side for the large synthetic benchmarks
        rnd = lambda shape, s=std: torch.randn(shape, generator=gg, device=dev, dtype=torch.float32) * s  # noqa: E731
        self.embed.copy_(rnd(self.embed.shape))
        self.head.copy_(rnd(self.head.shape))
        for l in self.layers:
            for p in l.projections():
                p.set_weight(rnd(p.weight.shape).to(self.dtype))
                p.init_adapters(g)
            if isinstance(l.mix, Mamba2):
                l.mix.conv_w.copy_(rnd(l.mix.conv_w.shape, 0.3))
                l.mix.A_log.copy_(torch.log(torch.rand(l.mix.A_log.shape, generator=g) * 15 + 1))
                l.mix.dt_bias.copy_(rnd(l.mix.dt_bias.shape, 0.5) - 3.0)
            else:
                l.mix.rel.copy_(rnd(l.mix.rel.shape, 0.5))
                l.mix.refresh_derived()
        self.refresh_head()

    # ------------------------------------------------------------- forward
    def run_layers(self, x, mixer_of):
        """Grad-free pass over all layers: streams and the last sublayer's output, still to be added."""
        pending = (None, None, None)
        for i, layer in enumerate(self.layers):
            x, pending = layer.run(x, pending, mixer_of(i, layer.mix))
        return x, pending

    def forward_streams(self, ids, comm: Optional[Comm] = None, merged: bool = False, detached: bool = False):
        """Streams behind the last layer, ``[B,S,streams,H]`` float32."""
        B, S = ids.shape
        self.ensure_positions(S)
        positions = torch.arange(S, device=ids.device)
        x = ops.embed_streams(ids, self.embed, self.pe, positions, self.spec.streams)
        if torch.is_grad_enabled() and not detached:
            for layer in self.layers:
                params = layer.adapter_params() if not self.full_ft else list(layer.parameters())
                for q in layer.sublayers():
                    fn = (lambda z, l=layer, q=q: l.half(q, z, merged))
                    x = remat_segment(fn, x, params) if self.remat else fn(x)
            return x, (None, None, None)
        with torch.no_grad():
            if merged:
                return self.run_layers(x, lambda i, mix: lambda h: mix(h, True))
            for layer in self.layers:
                pending = (None, None, None)
                for q in layer.sublayers():
                    x, h = layer.enter(q, x, pending)
                    pending = layer.leave(q, layer.mix(h) if q == 1 else layer.feed_forward(h, False))
                x = ops.hyper_mix(x, *pending)
            return x, (None, None, None)

    def final_hidden(self, x, pending=(None, None, None)):
        """Last norm of the streams' sum, times the output scale, in the compute dtype."""
        return ops.hyper_norm(x, *pending, None, self.final_norm, self.spec.norm_eps, self.dtype, self.spec.logit_scale, False)[1]

    def logits(self, x, pending=(None, None, None)) -> torch.Tensor:
        """Stream rows ``[N,streams,H]`` -> float32 logits ``[N,V]``."""
        return ops.linear_f32(self.final_hidden(x, pending), self.head)

    @staticmethod
    def pick(x, pending, at):
        """Rows ``at`` of the streams and of the pending output."""
        y, mix, out = pending
        return x[at], (None if y is None else y[at], mix, out)

    def forward(self, ids, comm: Optional[Comm] = None) -> torch.Tensor:
        x, pending = self.forward_streams(ids, comm)
        return self.logits(*self.pick(x.flatten(0, 1), (None if pending[0] is None else pending[0].flatten(0, 1), *pending[1:]),
                                      slice(None))).view(*ids.shape, -1)

    def token_logprobs(self, ids, win_start, targets, temperature: float = 1.0, comm: Optional[Comm] = None):
        x, pending = self.forward_streams(ids, comm, detached=not torch.is_grad_enabled())
        B, L = targets.shape
        idx = (win_start.view(B, 1).long() + torch.arange(L, device=ids.device)[None, :]).clamp(max=ids.shape[1] - 1)
        rows = torch.arange(B, device=ids.device)[:, None].expand(B, L)
        h = self.final_hidden(*self.pick(x, pending, (rows.reshape(-1), idx.reshape(-1))))
        return ops.logprob_gather(h, self.head, targets.reshape(-1), temperature, 0.0, head_wt=self.head_t).view(B, L)

    def new_decoder(self, batch: int, max_len: int, comm: Optional[Comm] = None) -> "MifutarCachedDecoder":
        return MifutarCachedDecoder(self, batch, max_len, comm or SoloComm())


class MifutarCachedDecoder:
    """Cached, grad-free twin over merged weights: per layer the mixer's own decode state, one row of it per batch row."""

    supports_retirement = True

    def __init__(self, model: MifutarGradModel, batch: int, max_len: int, comm: Comm):
        self.m, self.comm, self.batch, self.max_len = model, comm, batch, max_len
        model.ensure_positions(max_len)
        dev = model.embed.device
        self.pe = model.pe                      # held here so that a captured graph keeps its operand
        self.state = [l.mix.new_state(batch, max_len, model.dtype, dev) for l in model.layers]
        self.kv_len = torch.zeros(batch, dtype=torch.int32, device=dev)

    def cache_bytes(self) -> int:
        return sum(t.numel() * t.element_size() for s in self.state for t in s.tensors())

    def step_state(self):
        """Tensors that a decode step advances; a step that is taken twice has to start from a copy of them."""
        return [t for s in self.state for t in s.advanced()]

    @torch.no_grad()
    def prefill(self, ids, lens, rows=None, at=None):
        """Right-padded prompts ``[P,L]`` into state rows ``rows``; logits ``[P,V]`` of the last tokens, or of the
        places ``at = (prompt indices, positions)``."""
        m = self.m
        P, L = ids.shape
        if L > self.max_len:
            raise ValueError(f"prompt of {L} tokens exceeds the cache's {self.max_len}")
        rows = torch.arange(P, device=ids.device) if rows is None else rows
        lens = lens.long()
        x = ops.embed_streams(ids, m.embed, m.pe, torch.arange(L, device=ids.device), m.spec.streams)
        x, pending = m.run_layers(x, lambda i, mix: lambda h: mix(h, True, lens, lambda *kept: self.state[i].fill(rows, lens, *kept)))
        self.kv_len[rows] = lens.to(torch.int32)
        return m.logits(*m.pick(x, pending, (torch.arange(P, device=ids.device), lens - 1) if at is None else at))

    @torch.no_grad()
    def broadcast_groups(self, group: int):
        P = self.batch // group
        src = torch.arange(P, device=self.kv_len.device).repeat_interleave(group)
        for s in self.state:
            for t in s.tensors():
                t.copy_(t[src])
        self.kv_len.copy_(self.kv_len[src])

    def kv_tokens_read(self, active: Optional[torch.Tensor] = None) -> torch.Tensor:
        """Cached keys that the next ``decode`` call reads, averaged over the layers that keep any."""
        nxt = self.kv_len + 1
        if active is not None:
            nxt = nxt * active.to(torch.int32)
        read = [r for r in (s.rows_read(nxt) for s in self.state) if r is not None]
        return torch.stack(read).float().mean() if read else torch.zeros((), device=nxt.device)

    @torch.no_grad()
    def decode(self, tokens, active: Optional[torch.Tensor] = None):
        """Feed one token per row; next-token logits ``[B,V]`` float32.  Rows with ``active[b]`` false stay in the
        fixed-shape batch, and their state and length as they are."""
        m = self.m
        x = ops.embed_streams(tokens, m.embed, self.pe, self.kv_len, m.spec.streams)
        x, pending = m.run_layers(x, lambda i, mix: lambda h: mix.decode(h, self.kv_len, active, self.state[i]))
        self.kv_len += 1 if active is None else active.to(torch.int32)
        return m.logits(x, pending)


@torch.no_grad()
def load_mifutar_weights(model: MifutarGradModel, src) -> None:
    to = lambda t: t.to(model.dtype)  # noqa: E731
    f32 = lambda n: src.get(n).float()  # noqa: E731
    cat = lambda *names: to(torch.cat([src.get(n) for n in names], 0))  # noqa: E731
    model.embed.copy_(to(src.get("embed")))
    model.head.copy_(to(src.get("head")))
    model.final_norm.copy_(f32("final.norm"))
    for i, l in enumerate(model.layers):
        b = f"l{i}."
        for q in l.sublayers():
            getattr(l, f"norm{q}").copy_(f32(f"{b}norm{q}"))
            for n in ("in", "out", "mix"):
                getattr(l, f"hc{q}_{n}").copy_(f32(f"{b}hc{q}.{n}"))
        m = l.mix
        m.out.set_weight(to(src.get(b + "mix.o")))
        if isinstance(m, Mamba2):
            m.set_input_weight(to(src.get(b + "mix.in")))
            for n, name in (("conv_w", "conv"), ("conv_b", "conv.b"), ("dt_bias", "dt_bias"), ("A_log", "A_log"), ("D", "D"), ("norm", "norm")):
                getattr(m, n).copy_(f32(f"{b}mix.{name}"))
        else:
            m.inp.set_weight(cat(b + "mix.q", b + "mix.k"))
            m.inp.bias.copy_(cat(b + "mix.q.b", b + "mix.k.b"))
            m.rel.copy_(f32(b + "mix.rel"))
            m.refresh_derived()
        if l.ff is not None:
            l.gate_up.set_weight(cat(b + "mlp.gate", b + "mlp.up"))
            l.down.set_weight(to(src.get(b + "mlp.down")))
    model.refresh_head()


def load_mifutar(model_dir: str, opts):
    from .loader import TensorSource, _identity, read_config
    cfg = read_config(model_dir)
    src = TensorSource(model_dir)
    spec = mifutar_spec(cfg, {i: src.get(f"l{i}.mix.rel").shape[0] for i, lc in enumerate(cfg["layers"]) if lc["type"] == "attention"})
    if opts.max_position_embeddings:
        spec.max_position_embeddings = opts.max_position_embeddings
    if opts.tp is not None:
        raise ValueError("tensor parallelism is not supported for the Mifutar family")
    if opts.ep is not None and opts.ep[1] > 1:
        raise ValueError("expert parallelism is not supported for the Mifutar family")
    model = MifutarGradModel(spec, None if opts.full_ft else opts.lora, dtype=opts.dtype, device=opts.device, quant=opts.quantization,
                             remat=opts.remat, full_ft=opts.full_ft, recurrent_targets=opts.gdn_targets)
    load_mifutar_weights(model, src)
    g = torch.Generator().manual_seed(opts.adapter_seed)
    for l in model.layers:
        for pr in l.projections():
            pr.init_adapters(g)
    return model, _identity(model_dir, cfg, src, opts)
