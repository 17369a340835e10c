"""Token generation with layered models: request scheduling over the slots of one session, and the command line.

    python -m mdlarc_scale_b200.generation --model DIR --prompts prompts.jsonl --max-new 64

Requests wait until a slot is free; the prompts of admitted requests are prefilled in packed calls of
bounded size (long prompts in portions) between runs of graph-replayed decode steps of the sequences already
generating; a finished sequence's slot goes to the next request.  Picking the next token (argmax or
temperature / top-k sampling) happens on the device.
"""
from __future__ import annotations

import argparse
import json
import sys
from collections import deque
from dataclasses import dataclass, field

import numpy as np
import torch

from .engine import EngineBase
from .inference import DEFAULT_PREFILL_TOKENS, POLL_EVERY
from .layered import Segment


@dataclass
class Request:
    rid: int
    prompt: list[int]
    fed: int = 0                 # prompt tokens already in the cache
    slot: int = -1
    produced: int = 0            # tokens picked so far (host count; an upper bound once the end token is out)
    output: list[int] = field(default_factory=list)


class Scheduler:
    """Runs requests to completion on one session of a layered engine."""

    def __init__(self, engine: EngineBase, max_new: int, t_max: int, n_slots: int, prefill_tokens: int = DEFAULT_PREFILL_TOKENS,
                 end_token: int | None = None, temperature: float = 0.0, top_k: int | None = None, seed: int = 0,
                 want_logits: bool = False):
        self.engine, self.max_new = engine, int(max_new)
        self.end_token = -1 if end_token is None else int(end_token)
        self.session = engine.new_session(
            n_slots, t_max, self.max_new, min(prefill_tokens, n_slots * t_max), stop_on_end=True,
            want_step_logits=want_logits, temperature=temperature, top_k=top_k or 0, sample_seed=seed,
            sample_stream=np.zeros(n_slots, np.int64), end_token=self.end_token)
        self.waiting: deque[Request] = deque()
        self.filling: list[Request] = []
        self.decoding: list[Request] = []
        self.done: list[Request] = []
        self.step_logits: dict[int, torch.Tensor] = {}

    def submit(self, request: Request) -> None:
        n = len(request.prompt)
        if n == 0:
            raise ValueError("a prompt needs at least one token")
        if n + self.max_new - 1 > self.session.t_max:
            raise ValueError(f"prompt of {n} tokens plus {self.max_new} new ones exceeds the session's {self.session.t_max} positions")
        if min(request.prompt) < 0 or max(request.prompt) >= self.engine.vocab_size:
            raise ValueError("a prompt token lies outside the vocabulary")
        self.waiting.append(request)

    def _admit(self) -> None:
        while self.waiting and self.session.free_slots:
            r = self.waiting.popleft()
            r.slot = self.session.acquire()
            self.session.out_tokens[r.slot].fill_(-1)
            self.session.sample_stream[r.slot] = r.rid & 0x7FFFFFFF
            self.filling.append(r)

    def _prefill(self) -> None:
        room, call, armed = self.session.max_prefill_tokens, [], []
        for r in self.filling:
            n = min(room, len(r.prompt) - r.fed)
            if n <= 0:
                break
            last = r.fed + n == len(r.prompt)
            call.append(Segment(r.slot, r.prompt[r.fed:r.fed + n], arm=last))
            r.fed += n
            room -= n
            if last:
                armed.append(r)
        self.session.prefill_segments(call)
        for r in armed:
            self.filling.remove(r)
            r.produced = 1
            self.decoding.append(r)

    def _decode(self) -> None:
        left = min(self.max_new - r.produced for r in self.decoding)
        n = min(left, POLL_EVERY)
        if n > 0:
            self.session.decode(n)
            for r in self.decoding:
                r.produced += n
                self.session.lens[r.slot] += n

    def _retire(self) -> None:
        ended = self.session.finished() if self.end_token >= 0 else None
        for r in list(self.decoding):
            if r.produced < self.max_new and (ended is None or not ended[r.slot]):
                continue
            row = self.session.out_tokens[r.slot].cpu().tolist()
            if self.end_token in row:
                row = row[:row.index(self.end_token) + 1]
            r.output = row
            if self.session.step_logits is not None:
                self.step_logits[r.rid] = self.session.step_logits[r.slot, :len(row)].clone()
            self.decoding.remove(r)
            self.session.release(r.slot)
            self.done.append(r)

    def run(self) -> list[Request]:
        """Until every submitted request is done; returns them in submission order."""
        while self.waiting or self.filling or self.decoding:
            self._admit()
            if self.filling:
                self._prefill()
            if self.decoding:
                self._decode()
                self._retire()
        self.session.poll()      # surfaces any device-side error word
        return sorted(self.done, key=lambda r: r.rid)

    def close(self) -> None:
        self.session.close()


def generate(engine: EngineBase, prompts, max_new: int, end_token: int | None = None, temperature: float = 0.0,
             top_k: int | None = None, seed: int = 0, max_batch: int = 256,
             prefill_tokens: int = DEFAULT_PREFILL_TOKENS, return_logits: bool = False):
    """Continuations of token-id prompts: one list of generated ids per prompt, the end token (if any) included.
    Greedy unless ``temperature > 0``; a request's random stream depends on ``seed`` and its index only."""
    if max_new <= 0 or not prompts:
        return ([[] for _ in prompts], {}) if return_logits else [[] for _ in prompts]
    t_max = max(len(p) for p in prompts) + max_new
    sched = Scheduler(engine, max_new, t_max, min(len(prompts), max_batch), prefill_tokens, end_token, temperature,
                      top_k, seed, return_logits)
    try:
        for i, p in enumerate(prompts):
            sched.submit(Request(i, [int(t) for t in p]))
        out = [r.output for r in sched.run()]
        return (out, sched.step_logits) if return_logits else out
    finally:
        sched.close()


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(description="generate token ids with a model folder (config.json + model.safetensors)")
    ap.add_argument("--model", required=True)
    ap.add_argument("--prompts", default="-", help="file of JSON lists of token ids, one a line ('-': standard input)")
    ap.add_argument("--max-new", type=int, default=64)
    ap.add_argument("--end-token", type=int, default=None)
    ap.add_argument("--dtype", default="bfloat16", help="bfloat16 | bfloat16-operands | float32")
    ap.add_argument("--temperature", type=float, default=0.0)
    ap.add_argument("--top-k", type=int, default=None)
    ap.add_argument("--seed", type=int, default=0)
    ap.add_argument("--max-batch", type=int, default=256)
    args = ap.parse_args(argv)
    from .registry import load_model
    engine = load_model(args.model, "cuda:0", args.dtype)
    src = sys.stdin if args.prompts == "-" else open(args.prompts)
    prompts = [json.loads(line) for line in src if line.strip()]
    for row in generate(engine, prompts, args.max_new, args.end_token, args.temperature, args.top_k, args.seed, args.max_batch):
        print(json.dumps(row))
    return 0


if __name__ == "__main__":
    sys.exit(main())
