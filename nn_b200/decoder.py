"""What every cached decoder of this package shares: the decoding step replayed as a CUDA graph, and the generation loop.

A decoder serves ``batch`` sequences in lockstep.  It provides ``_forward(steps)`` -- queue one pass over ``steps`` new positions
of every sequence, whose ids lie in ``self.ids``, and leave the next token of each in ``self.ids[0:batch]`` -- and
``prefill(ids)``, which reads prompts from position 0.  Positions and sampled ids live on the device, so a recorded step serves
every position (DecodingContext.CaptureStep / ReplayStep, src/NeuralSharp/Layers/Decoding.cs:129-155).  The loop is the
reference's (CharGpt.Generate, samples/Shared/Gpt/CharGpt.cs:231-318), with its re-read of the last half of the window when a
model has a limited context.
"""
from __future__ import annotations

import ctypes as C

import numpy as np

from . import native as N


class CachedDecoder:
    def begin_decoding(self, context: int | None) -> None:
        """context: the most positions a sequence can have (None: no limit, e.g. sliding windows and recurrent states)."""
        self.context = context
        self.graph = None
        self.launches_per_step = 0

    def step(self, use_graph: bool = True) -> None:
        """One cached decoding step for every sequence; the first call records it as a CUDA graph
        (DecodingContext.CaptureStep / ReplayStep, Layers/Decoding.cs:129-155)."""
        assert self.context is None or self.length + 1 <= self.context, "context is full: re-read the window first"
        if not use_graph:
            self._forward(1)
        else:
            if self.graph is None:
                self._forward(1)               # un-captured once: sizes scratch memory, sets kernel attributes
                self.length += 1
                self.launches_per_step = self._n
                self.dev.capture_begin()
                try:
                    self._forward(1)
                except Exception:
                    N.call("ns_capture_abort", self.dev.handle)
                    raise
                self.graph = self.dev.capture_end()
                return                          # the captured pass did not execute; the un-captured one was this step
            self.dev.graph_launch(self.graph)
        self.length += 1

    def drop_graph(self) -> None:
        """Forgets the recorded step; the next one records again."""
        if self.graph is not None:
            self.dev.synchronize()
            self.dev.graph_destroy(self.graph)
            self.graph = None

    def read_ids(self) -> np.ndarray:
        return self.ids.download(count=self.batch).copy()

    def generate(self, prompt: np.ndarray, n_new: int, use_graph: bool = True, marks: dict | None = None,
                 mark_every: int = 32) -> tuple[np.ndarray, int]:
        """Decoding of n_new tokens per sequence; returns (tokens [batch, n_new], context resets).
        marks: when a dict is given, device events are recorded into it on the device's stream -- "start" (before the
        prompt is read), "prefill_end" (the first token is on the device), "steps" = [(tokens produced so far, event), ...]
        every mark_every decoding steps and after the last one -- for timing a generation from outside."""
        B, context = self.batch, self.context

        def mark(name=None, count=None):
            if marks is None:
                return
            e = self.dev.event()
            self.dev.record(e)
            if name is not None:
                marks[name] = e
            else:
                marks.setdefault("steps", []).append((count, e))

        history = [list(map(int, row)) for row in np.asarray(prompt)]
        hist_dev = self.dev.empty(B * max(n_new, 1), N.NS_I32)
        pending = 0            # tokens sampled on the device and not yet fetched
        out: list[list[int]] = [[] for _ in range(B)]
        resets = 0

        def flush():
            nonlocal pending
            if pending:
                got = hist_dev.download((pending, B), count=pending * B)
                for row in got:
                    for b in range(B):
                        history[b].append(int(row[b])); out[b].append(int(row[b]))
                pending = 0

        def keep_token():
            nonlocal pending
            N.call("ns_d2d_async", self.dev.handle, C.c_uint64(hist_dev.ptr + pending * B * 4), C.c_uint64(self.ids.ptr), C.c_uint64(B * 4))
            pending += 1

        def window(keep):
            return np.array([h[-keep:] for h in history], dtype=np.int32)

        mark("start")
        self.prefill(window(len(history[0]) if context is None else min(len(history[0]), context - 1)))
        keep_token()
        mark("prefill_end")
        produced = 1
        while produced < n_new:
            if context is not None and self.length >= context:
                flush()
                self.prefill(window(context // 2))     # window full: re-read the last half from position 0
                keep_token()
                resets += 1
                produced += 1
                continue
            self.step(use_graph)
            keep_token()
            produced += 1
            if (produced - 1) % mark_every == 0 or produced == n_new:
                mark(count=produced)
        flush()
        self.dev.synchronize()
        return np.array(out, dtype=np.int32)[:, :n_new], resets
