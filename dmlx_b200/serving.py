"""Driving a loaded model: text-free generation through the engine, and feeding given tokens step by step.

`generate` submits prompts to the engine (scheduler, page budget, samplers) and returns what it produced.
`TokenFeeder` runs batches whose tokens the caller decides: it keeps each request's slot and length, runs the
model's step on the portions it is given (portions of prompts beside single tokens, in one batch) and returns
the logits asked for.  Slots come from and go back to the pool's block manager, as the scheduler's do.
"""
from __future__ import annotations

import ctypes as C
from typing import Dict, List, Optional, Sequence, Tuple

import numpy as np

from . import _lib
from . import device as dev
from ._lib import lib
from .models import PAGE_TOKENS, LoadedModel


def pages_for(tokens: int) -> int:
    return (tokens + PAGE_TOKENS - 1) // PAGE_TOKENS


def generate(loaded: LoadedModel, prompts: Sequence[Sequence[int]], max_new_tokens: int, *, stop_tokens: Sequence[int] = (),
             temperature: float = 0.0, top_k: int = 0, top_p: float = 1.0, seed: int = 0, prefill_chunk: int = 512,
             n_pages: Optional[int] = None, prefix_sharing: bool = False) -> List[List[int]]:
    """New tokens of every prompt, all served by one engine.  temperature 0 is greedy."""
    per_seq = max(pages_for(len(p) + max_new_tokens) for p in prompts)
    if n_pages is None:
        n_pages = sum(sorted((pages_for(len(p) + max_new_tokens) for p in prompts), reverse=True)[:loaded.limits.max_seqs])
    for p in prompts:
        if any(not 0 <= int(t) < loaded.vocab for t in p):
            raise ValueError(f"a prompt holds a token outside the vocabulary of {loaded.vocab}")
    kv = loaded.new_cache(n_pages, per_seq)
    engine = dev.Engine(loaded.model, kv, min(prefill_chunk, loaded.limits.max_rows))
    engine.set_max_step_tokens(loaded.limits.max_rows)
    engine.set_prefix_sharing(prefix_sharing)
    for i, p in enumerate(prompts):
        engine.submit(i, p, max_new_tokens, stop_tokens)
        if temperature > 0:
            engine.set_sampler(i, temperature, top_k or loaded.vocab, top_p, seed + i)
    while engine.active_count():
        engine.step()
    out = []
    for i in range(len(prompts)):
        status = engine.request_status(i)
        if status != _lib.OK:
            raise _lib.B200Error(status)
        out.append(engine.result(i)[0])
    engine.close()
    kv.close()
    return out


class TokenFeeder:
    """Steps over tokens the caller gives; requests are known by names of the caller's choice."""

    def __init__(self, loaded: LoadedModel, n_pages: int, max_pages_per_seq: Optional[int] = None):
        self.loaded = loaded
        self.kv = loaded.new_cache(n_pages, max_pages_per_seq or n_pages)
        self._bm = lib.b200_sched_bm_create_with_kv(self.kv._h)
        if not self._bm:
            raise _lib.B200Error(_lib.ERR_CUDA)
        self._live: Dict[object, List[int]] = {}  # name -> [slot, tokens in the cache]

    def close(self):
        if getattr(self, "_bm", None) and lib is not None:
            lib.b200_sched_bm_destroy(self._bm)
            self._bm = None
            self.kv.close()

    def __del__(self):
        self.close()

    def length(self, name) -> int:
        return self._live[name][1] if name in self._live else 0

    def free_pages(self) -> int:
        return self.kv.free_count()

    def step(self, entries: Sequence[Tuple[object, Sequence[int], Sequence[int]]]) -> np.ndarray:
        """One batch of (name, next tokens, places among them whose logits are wanted); a new name takes a slot.
        Returns f32 logits [wanted places in order, vocab]."""
        descs, flat, want = [], [], []
        for name, tokens, places in entries:
            if len(tokens) == 0:
                continue
            if name not in self._live:
                slot = C.c_int32()
                _lib.check(lib.b200_sched_bm_park_slot(self._bm, C.byref(slot)))
                self._live[name] = [slot.value, 0]
            slot, length = self._live[name]
            if pages_for(length + len(tokens)) > self.kv.cfg.max_pages_per_seq:
                raise ValueError(f"request {name!r}: {length + len(tokens)} tokens exceed what one sequence holds")
            if any(not 0 <= p < len(tokens) for p in places):
                raise ValueError(f"request {name!r}: a wanted place lies outside its {len(tokens)} tokens")
            descs.append((slot, len(tokens), length, len(flat)))
            want += [len(flat) + int(p) for p in places]
            flat += [int(t) for t in tokens]
        if not descs:
            return np.zeros((0, self.loaded.vocab), np.float32)
        if len({d[0] for d in descs}) != len(descs):
            raise ValueError("a request stands in one step twice")
        # a step whose tokens are all the sampled rows' needs no extra logits: each request's last row is computed anyway
        ends = np.cumsum([d[1] for d in descs]) - 1
        last = {int(r): i for i, r in enumerate(ends)}
        extra = [] if all(r in last for r in want) else want
        self.loaded.model.step(self.kv, descs, flat, extra)
        for d, (name, tokens, _) in zip(descs, [e for e in entries if len(e[1])]):
            self._live[name][1] += len(tokens)
        if not want:
            return np.zeros((0, self.loaded.vocab), np.float32)
        if extra:
            return self.loaded.model.logits(len(descs), len(want))
        return self.loaded.model.logits(0, len(descs))[[last[r] for r in want]]

    def end(self, name):
        """Gives back what a finished request holds."""
        slot, _ = self._live.pop(name)
        _lib.check(lib.b200_sched_bm_unpark_slot(self._bm, slot))
