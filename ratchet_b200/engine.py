"""Serving loop over a model of ``models.REGISTRY``: sequence slots, steps over blocks of tokens, sampling, generation.

A slot owns one sequence's state tensors (and the decode step captured over them).  A new sequence takes a free slot, whose
state is reset; ending a sequence gives the slot back.  A step runs only the tokens it brings: one token goes through the fused
decode step, a block through the lazy graph in portions of at most ``portion`` tokens."""
from __future__ import annotations

from collections import deque
from dataclasses import dataclass, field
from typing import Deque, Dict, Hashable, Iterable, List, Optional, Sequence

import numpy as np

from .capi import ERR_BOUNDS, ERR_INVALID_ARG, ERR_OOM, RatchetCudaError
from .nn import SequenceState


class Sampler:
    """Greedy (temperature 0) or softmax sampling over the `top_k` highest logits (0: all)."""

    def __init__(self, temperature: float = 0.0, top_k: int = 0, seed: int = 0):
        if temperature < 0 or top_k < 0:
            raise RatchetCudaError(ERR_INVALID_ARG, "sampler: temperature and top_k must not be negative")
        self.temperature, self.top_k, self.rng = temperature, top_k, np.random.Generator(np.random.PCG64(seed))

    @property
    def greedy(self) -> bool:
        return self.temperature == 0.0

    def pick(self, logits: np.ndarray) -> int:
        if self.greedy:
            return int(np.argmax(logits))
        z = logits.astype(np.float64) / self.temperature
        if 0 < self.top_k < z.size:
            z = np.where(z >= np.partition(z, -self.top_k)[-self.top_k], z, -np.inf)
        p = np.exp(z - z.max())
        return int(self.rng.choice(z.size, p=p / p.sum()))


@dataclass
class Request:
    prompt: Sequence[int]
    max_new_tokens: int
    sampler: Sampler = field(default_factory=Sampler)
    stop: Optional[int] = None           # token id that ends the request (it is part of the output)
    output: List[int] = field(default_factory=list)


class Engine:
    def __init__(self, model, max_tokens: Optional[int] = None, slots: int = 1, portion: int = 4096):
        if slots < 1 or portion < 1:
            raise RatchetCudaError(ERR_INVALID_ARG, "engine: at least one slot and one token per portion")
        self.model, self.max_tokens, self.portion = model, max_tokens, portion
        self._free: List[SequenceState] = [model.new_state(max_tokens) for _ in range(slots)]
        self._live: Dict[Hashable, SequenceState] = {}

    # ------------------------------------------------------------------ sequences
    def begin(self, seq: Hashable) -> SequenceState:
        if seq in self._live:
            raise RatchetCudaError(ERR_INVALID_ARG, f"sequence {seq!r} is already live")
        if not self._free:
            raise RatchetCudaError(ERR_OOM, f"no free slot for sequence {seq!r} ({len(self._live)} live)")
        state = self._free.pop()
        state.reset()
        self._live[seq] = state
        return state

    def end(self, seq: Hashable) -> None:
        if seq in self._live:
            self._free.append(self._live.pop(seq))

    def position(self, seq: Hashable) -> int:
        return self._live[seq].position if seq in self._live else 0

    def _check(self, state: SequenceState, tokens: Sequence[int]) -> None:
        if len(tokens) and not (0 <= min(tokens) and max(tokens) < self.model.vocab):
            raise RatchetCudaError(ERR_BOUNDS, f"a token id lies outside the vocabulary of {self.model.vocab}")
        if self.max_tokens is not None and state.position + len(tokens) > self.max_tokens:
            raise RatchetCudaError(ERR_INVALID_ARG, f"{state.position + len(tokens)} tokens exceed the {self.max_tokens} a slot holds")

    def step(self, seq: Hashable, tokens: Sequence[int], want: Sequence[int] = ()) -> np.ndarray:
        """The next tokens of a sequence (a new one is begun); f32 logits [len(want), vocab] of the wanted places among them."""
        if len(want) and not (0 <= min(want) and max(want) < len(tokens)):
            raise RatchetCudaError(ERR_INVALID_ARG, "a wanted place lies outside the step's tokens")
        state = self._live.get(seq) or self.begin(seq)
        self._check(state, tokens)
        out = np.empty((len(want), self.model.vocab), np.float32)
        for a in range(0, len(tokens), self.portion):
            part = tokens[a:a + self.portion]
            rows = [k for k, p in enumerate(want) if a <= p < a + len(part)]
            if len(part) == 1:
                logits, _ = self.model.decode(state, int(part[0]))
                if rows:
                    out[rows] = logits.to_numpy()
            else:
                got = self.model.prefill(part, state, [want[k] - a for k in rows])
                if rows:
                    out[rows] = got
        return out

    # ------------------------------------------------------------------ generation
    def run(self, requests: Iterable[Request]) -> List[Request]:
        """Serve requests to the end, first come, first served: a request enters when a slot is free (its prompt runs at once),
        then every live sequence gets one token per round.  Greedy sequences pick on the device."""
        requests = list(requests)
        waiting: Deque[int] = deque(range(len(requests)))
        live: Dict[int, bool] = {}
        names = {k: object() for k in range(len(requests))}

        def take(k: int, token: int) -> None:
            r = requests[k]
            r.output.append(token)
            if len(r.output) >= r.max_new_tokens or token == r.stop:
                self.end(names[k])
                live.pop(k, None)
            else:
                live[k] = True

        try:
            while waiting or live:
                while waiting and self._free:
                    k = waiting.popleft()
                    r = requests[k]
                    if not len(r.prompt) or r.max_new_tokens < 1:
                        raise RatchetCudaError(ERR_INVALID_ARG, "a request needs a prompt and at least one new token")
                    take(k, r.sampler.pick(self.step(names[k], list(r.prompt), [len(r.prompt) - 1])[0]))
                for k in list(live):
                    r, state = requests[k], self._live[names[k]]
                    self._check(state, r.output[-1:])
                    logits, token = self.model.decode(state, r.output[-1])
                    take(k, int(token.to_numpy()[0]) if r.sampler.greedy else r.sampler.pick(logits.to_numpy()[0]))
        finally:
            for name in names.values():
                self.end(name)
        return requests

    def generate(self, prompt: Sequence[int], max_new_tokens: int, sampler: Optional[Sampler] = None, stop: Optional[int] = None) -> List[int]:
        return self.run([Request(prompt, max_new_tokens, sampler or Sampler(), stop)])[0].output
