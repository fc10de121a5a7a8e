"""Replay of a token trace: given ids go through a model step by step and chosen logits are written out.

The replay owns no forward pass.  A step of first tokens is a batch of ``LmPolicy``: its prompts are packed and
prefilled as for generation, into a decoder of the policy (``decoder_for``).  A step that goes on by one token is that
decoder's ``decode``.  Nothing is sampled.

Input, one JSON object a line::

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

``want`` lists the places among the entry's tokens whose logits are asked for, ``end`` the requests that are finished
after the step.  A step with wanted places writes ``<out>/<step>.f32``: little-endian float32 ``[wanted, vocab]`` in
the order of the entries.  After every step the line ``done <step>`` is printed.
"""
from __future__ import annotations

import json
import os
import sys
from typing import Iterable, Optional

import torch

from .lm_policy import LmPolicy
from .sampler import GrpoSampler

DTYPES = {"bfloat16": torch.bfloat16, "float32": torch.float32}


class TraceError(ValueError):
    pass


class _Batch:
    """Requests that started together: one decoder, one row each."""

    def __init__(self, dec, ids):
        self.dec = dec
        self.row = {rid: i for i, rid in enumerate(ids)}
        self.live = set(ids)


class TraceReplay:
    def __init__(self, policy: LmPolicy, max_tokens: int):
        self.policy, self.max_tokens = policy, max_tokens
        self.of: dict = {}              # request -> its batch

    @staticmethod
    def load(model_dir: str, dtype: str, max_tokens: int, device: str = "cuda") -> "TraceReplay":
        from .models.loader import LoaderOpts, load_auto_policy
        if dtype == "float32":          # float32 means float32: no reduced-precision matrix products
            torch.backends.cuda.matmul.allow_tf32 = False
            torch.backends.cudnn.allow_tf32 = False
            torch.set_float32_matmul_precision("highest")
        model, _ = load_auto_policy(model_dir, LoaderOpts(dtype=DTYPES[dtype], device=device, lora=None))
        return TraceReplay(LmPolicy(model, GrpoSampler(0)), max_tokens)

    # ------------------------------------------------------------------ steps
    @torch.no_grad()
    def step(self, entries, end=()) -> Optional[torch.Tensor]:
        """Run one step; float32 logits ``[wanted, V]`` on the host, or ``None`` when nothing is wanted."""
        for e in entries:
            n = len(e["tokens"])
            if n == 0 or any(not 0 <= w < n for w in e["want"]):
                raise TraceError(f"request {e['id']!r}: no tokens, or a wanted place outside them")
        if len({e["id"] for e in entries}) != len(entries):
            raise TraceError("a request appears twice in one step")
        known = [e["id"] in self.of for e in entries]
        if any(known) and not all(known):
            raise TraceError("a step either starts all its requests or goes on with all of them")
        out = None
        if entries:
            out = self._go_on(entries) if known[0] else self._start(entries)
        for rid in end:
            batch = self.of.pop(rid, None)
            if batch is None:
                raise TraceError(f"request {rid!r} ends but was never started")
            batch.live.discard(rid)
        if out is not None:
            out = out.float().cpu()
        if self.policy.device().type == "cuda":
            from .ops import cuda as C
            if C.kernel_status() != 0:
                raise RuntimeError("a kernel reported a bounded-wait timeout")
        return out

    def _decoder(self, batch: int, longest: int):
        dec, key = self.policy.decoder_for(batch, max(self.max_tokens, longest))
        if any(b.dec is dec for b in self.of.values()):       # still in use by requests that are not finished
            return self.policy.model.new_decoder(batch, key[1], self.policy.comm)
        return dec

    def _start(self, entries):
        prompts = [e["tokens"] for e in entries]
        self.policy.refresh_merged()
        dec = self._decoder(len(entries), max(len(p) for p in prompts))
        ids, lens = self.policy.pack_prompts(prompts)
        at = [(i, w) for i, e in enumerate(entries) for w in e["want"]]
        places = None
        if at:
            dev = ids.device
            places = (torch.tensor([a for a, _ in at], device=dev), torch.tensor([b for _, b in at], device=dev))
        logits = dec.prefill(ids, lens, at=places)
        batch = _Batch(dec, [e["id"] for e in entries])
        for e in entries:
            self.of[e["id"]] = batch
        return logits if at else None

    def _go_on(self, entries):
        batch = self.of[entries[0]["id"]]
        if any(self.of[e["id"]] is not batch for e in entries):
            raise TraceError("the requests of a step did not start together")
        if any(len(e["tokens"]) != 1 for e in entries):
            raise TraceError("a request goes on by one token")
        dec, n = batch.dec, len(batch.row)
        toks = [self.policy.pad_token_id] * n
        for e in entries:
            toks[batch.row[e["id"]]] = e["tokens"][0]
        dev = self.policy.device()
        tokens = torch.tensor(toks, dtype=torch.int64).to(dev)
        here = {e["id"] for e in entries}
        idle = [r for rid, r in batch.row.items() if rid not in here]
        if not idle:
            logits = dec.decode(tokens)
        elif getattr(dec, "supports_retirement", False):
            active = torch.ones(n, dtype=torch.bool)
            active[idle] = False
            logits = dec.decode(tokens, active.to(dev))
        else:
            if batch.live - here:
                raise TraceError("this model family cannot hold back a live request of a batch")
            dec.kv_len[torch.tensor(idle, device=dev)] = 0    # finished rows run on a pad token at position 0
            logits = dec.decode(tokens)
        want = [batch.row[e["id"]] for e in entries for _ in e["want"]]
        return logits[torch.tensor(want, device=dev)] if want else None


def replay_stream(replay: TraceReplay, lines: Iterable[str], out_dir: str, tell=None) -> None:
    tell = tell or (lambda s: print(s, flush=True))
    for line in lines:
        if not line.strip():
            continue
        d = json.loads(line)
        logits = replay.step(d["entries"], d.get("end", ()))
        if logits is not None:
            with open(os.path.join(out_dir, f"{d['step']}.f32"), "wb") as f:
                f.write(logits.contiguous().numpy().astype("<f4").tobytes())
        tell(f"done {d['step']}")


def add_arguments(p) -> None:
    p.add_argument("--model", required=True, help="folder with config.json and safetensors weights")
    p.add_argument("--dtype", required=True, choices=sorted(DTYPES))
    p.add_argument("--out", required=True, help="folder that receives <step>.f32")
    p.add_argument("--max-tokens", type=int, required=True, help="most tokens that live requests hold at any time")


def run(args) -> int:
    from . import _build
    _build.ensure()
    replay = TraceReplay.load(args.model, args.dtype, args.max_tokens)
    replay_stream(replay, sys.stdin, args.out)
    return 0


def main(argv=None) -> int:
    import argparse
    ap = argparse.ArgumentParser(prog="trace_run", description="Feed a token trace through a model and write chosen logits.")
    add_arguments(ap)
    return run(ap.parse_args(argv))


if __name__ == "__main__":
    sys.exit(main())
