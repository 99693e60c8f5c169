"""What every decoder of this package offers, whatever its model: the recorded step, and the calls that a generation loop,
the trace replay and the command line drive.

A decoder serves sequences through
    seq = decoder.open()                       a place for one sequence (its caches, states and position)
    rows = decoder.forward(seq, tokens, want)  runs the next tokens; logits of the wanted places among them
    ids = decoder.decode_greedy(seq, n)        n further tokens, arg-max fed back on the device
    decoder.close(seq)                         gives the place back
Prompts may be fed in portions of any size; decode_greedy continues from the last place whose logits were asked for.
"""
from __future__ import annotations

from dataclasses import dataclass, field

import torch


class RecordedStep:
    """A fixed sequence of launches over fixed device buffers: run eagerly, or recorded once into a CUDA graph and replayed."""

    def __init__(self, launches, device):
        self._launches, self._dev = launches, device
        self.graph = None

    def run(self) -> None:
        for f in self._launches:
            f()

    def capture(self) -> None:
        """Records the launches (call after at least one eager run; nothing is executed)."""
        torch.cuda.synchronize(self._dev)
        g = torch.cuda.CUDAGraph()
        with torch.cuda.graph(g):
            self.run()
        self.graph = g

    def replay(self, n: int = 1) -> None:
        if self.graph is None:
            raise RuntimeError("capture() first")
        for _ in range(n):
            self.graph.replay()


@dataclass
class Request:
    prompt: list
    n_new: int
    tokens: list = field(default_factory=list)  # generated


class RequestQueue:
    """First-come scheduler over a decoder: requests run one after the other, each prompt in portions of at most `portion`
    tokens (None: as the decoder cuts them), then greedy decoding; a finished request's place is reused by the next."""

    def __init__(self, decoder, portion: int | None = None):
        self.decoder, self.portion, self._waiting = decoder, portion, []

    def submit(self, prompt, n_new: int) -> Request:
        r = Request([int(t) for t in prompt], int(n_new))
        if not r.prompt or r.n_new < 0:
            raise ValueError("a request needs a prompt and a count of new tokens that is not negative")
        self._waiting.append(r)
        return r

    def run(self) -> None:
        while self._waiting:
            r = self._waiting.pop(0)
            seq = self.decoder.open()
            try:
                step = self.portion or len(r.prompt)
                for at in range(0, len(r.prompt), step):
                    part = r.prompt[at: at + step]
                    last = at + step >= len(r.prompt)
                    self.decoder.forward(seq, part, [len(part) - 1] if last else [])
                if r.n_new:
                    r.tokens = self.decoder.decode_greedy(seq, r.n_new)
            finally:
                self.decoder.close(seq)


def generate(decoder, prompt, n_new: int, portion: int | None = None) -> list:
    """Greedy continuation of one prompt."""
    q = RequestQueue(decoder, portion)
    r = q.submit(prompt, n_new)
    q.run()
    return r.tokens
