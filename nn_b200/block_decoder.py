"""What every decoder made of blocks (nn_b200.blocks) over a 32-bit residual stream shares: the workspace, the sequences' slots, the
head, portions of prompts, and the hooks of the generation loop.

A model class names its blocks in ``_build(weights)`` and queues a pass's embedding and layers in ``_layers(step)``, which leaves the
residual stream in the workspace's "x".  Sequences live in slots (nn_b200.state); there is no limit on a sequence's length,
because windows are rings and the other layers are recurrent.
"""
from __future__ import annotations

import ctypes as C

import numpy as np

from . import native as N
from .blocks import Product, Step, Workspace, bf16_bits, f32, pad8, rms_rows
from .decoder import CachedDecoder
from .device import Device
from .state import SequenceStates


class BlockDecoder(CachedDecoder):
    """weights: mapping of tensor name -> array, bf16 bits (uint16) or float32; any mapping works, every tensor is looked up once.
    cfg has vocab, width and eps.  dtype NS_BF16 or NS_F32.  `batch` sequences run in lockstep in generate(); `slots` (default:
    batch) sequences can be open at a time; a pass takes at most `max_prefill` tokens per sequence, longer prompts are read in
    portions."""

    LOGIT_ROWS = 64          # rows the head works on at a time
    HEAD = "head"            # the output matrix's tensor

    def __init__(self, dev: Device, cfg, weights, batch: int = 1, max_prefill: int = 512, dtype: int = N.NS_BF16, slots: int | None = None):
        self.dev, self.cfg, self.batch, self.dtype, self.max_prefill = dev, cfg, batch, dtype, max_prefill
        ws = self.ws = Workspace(dev, dtype)
        D = cfg.width
        self.states = SequenceStates(dev, slots if slots is not None else batch)
        self._blocks: list = []                              # whatever has to be closed
        self._build(weights)
        self.head = Product(ws, weights[self.HEAD])
        self.final_norm = dev.from_numpy(f32(weights["final.norm"]))
        ws.need("x", D, N.NS_F32)
        ws.need("h", pad8(D))
        rows = batch * max_prefill
        self.logit_rows = max(batch, self.LOGIT_ROWS)
        ws.allocate(max(rows, self.logit_rows), batch)
        self.states.allocate()
        self.logits_padded = dev.empty(self.logit_rows * self.head.ld, N.NS_F32)
        self.logits = self.logits_padded if self.head.ld == cfg.vocab else dev.empty(self.logit_rows * cfg.vocab, N.NS_F32)
        self.ids = dev.zeros(rows, N.NS_I32)
        self.slot_ids = dev.zeros(batch, N.NS_I32)
        self.row_map = dev.zeros(self.logit_rows, N.NS_I32)
        self._slots_now: list[int] | None = None
        self._lockstep: list[int] | None = None              # the slots generate() uses
        self.sampler = None
        self.length = 0
        self.begin_decoding(None)

    def _build(self, weights) -> None:
        raise NotImplementedError

    def _layers(self, step: Step) -> None:
        raise NotImplementedError

    def _table(self, a):
        """A matrix whose rows are looked up, on the device in the model's number format."""
        return self.dev.from_numpy((bf16_bits(a) if self.dtype == N.NS_BF16 else f32(a)).reshape(-1))

    def _embed(self, step: Step, table: int, table_ld: int, y: int, scale: float = 1.0, bigram=None, hashing: dict | None = None) -> None:
        """y = scale * table[token] (+ a row of `bigram` named by the token and the one before it)."""
        b, u, D = hashing or {"buckets": 1, "mul_prev": 0, "mul_cur": 0}, C.c_uint64, self.cfg.width
        N.call("ns_embed_ngram", self.dev.handle, u(self.ids.ptr), u(table), self.dtype, table_ld, C.c_float(scale), u(bigram.ptr if bigram else 0), D,
               b["buckets"], C.c_int64(b["mul_prev"]), C.c_int64(b["mul_cur"]), u(step.slots), u(self.states.last.ptr), step.batch, step.steps, D, self.cfg.vocab, u(y))
        step.launches += 1

    # ------------------------------------------------------------------ one pass
    def _head(self, step: Step, rows: int) -> None:
        """Logits of the `rows` rows row_map names."""
        cfg, dev, ws = self.cfg, self.dev, self.ws
        D, V = cfg.width, cfg.vocab
        rms_rows(step, dev, ws["x"], None, 0.0, 0, self.final_norm, cfg.eps, D, ws["h"], self.dtype, pad8(D), rows=rows, row_map=self.row_map.ptr)
        self.head.into(ws["h"], rows, self.logits_padded.ptr)
        step.launches += 1
        if self.logits is not self.logits_padded:
            N.call("ns_d2d_2d_async", dev.handle, C.c_uint64(self.logits.ptr), C.c_uint64(V * 4), C.c_uint64(self.logits_padded.ptr),
                   C.c_uint64(self.head.ld * 4), C.c_uint64(V * 4), C.c_uint64(rows))

    def _advance(self, step: Step) -> None:
        N.call("ns_seq_advance", self.dev.handle, C.c_uint64(self.ids.ptr), C.c_uint64(step.slots), step.batch, step.steps,
               C.c_uint64(self.states.pos.ptr), C.c_uint64(self.states.last.ptr))
        step.launches += 1

    def _step(self, batch: int, steps: int, longest: int) -> Step:
        assert batch * steps <= self.ws.rows and steps <= self.max_prefill
        return Step(batch, steps, self.slot_ids.ptr, self.states.pos.ptr, longest)

    def _use_slots(self, slots: list[int]) -> None:
        if slots != self._slots_now:
            self._put(self.slot_ids, np.asarray(slots, np.int32))
            self._slots_now = list(slots)

    def _put(self, dst, a: np.ndarray) -> None:
        a = np.ascontiguousarray(a, np.int32)
        N.call("ns_h2d", self.dev.handle, C.c_uint64(dst.ptr), a.ctypes.data_as(C.c_void_p), C.c_uint64(a.nbytes))

    # ------------------------------------------------------------------ sequences by slot
    def open_sequence(self) -> int:
        return self.states.open()

    def close_sequence(self, slot: int) -> None:
        self.states.close(slot)

    def feed(self, slots: list[int], ids: np.ndarray, want=()) -> np.ndarray:
        """The next tokens ids [len(slots), t] of the named sequences, from the cache and state their earlier tokens left.  Returns
        the logits [len(want), vocab] after the places `want` names: t-indices for one sequence, (sequence, t-index) pairs else."""
        ids = np.atleast_2d(np.asarray(ids, np.int32))
        b, t = ids.shape
        assert b == len(slots) <= self.batch
        pairs = [(0, int(p)) if np.isscalar(p) else (int(p[0]), int(p[1])) for p in want]
        out = np.empty((len(pairs), self.cfg.vocab), np.float32)
        self._use_slots(list(slots))
        for at in range(0, t, self.max_prefill):
            n = min(self.max_prefill, t - at)
            self._put(self.ids, ids[:, at:at + n])
            step = self._step(b, n, max(self.states.position[s] for s in slots) + at)
            self._layers(step)
            self._advance(step)
            here = [i for i, (_, p) in enumerate(pairs) if at <= p < at + n]
            for k in range(0, len(here), self.logit_rows):
                part = here[k:k + self.logit_rows]
                self._put(self.row_map, np.array([pairs[i][0] * n + pairs[i][1] - at for i in part]))
                self._head(step, len(part))
                out[part] = self.logits.download((len(part), self.cfg.vocab), count=len(part) * self.cfg.vocab)
        for s in slots:
            self.states.position[s] += t
        self.dev.synchronize()
        return out

    # ------------------------------------------------------------------ the generation loop's hooks (nn_b200.decoder)
    def set_sampler(self, sampler) -> None:
        """Sample with ``sampler`` (nn_b200.sampling.TokenSampler for this batch and vocabulary) instead of greedily."""
        self.sampler = sampler
        self.drop_graph()

    def _forward(self, steps: int) -> None:
        step = self._step(self.batch, steps, self.length)
        self._layers(step)
        self._advance(step)
        self._head(step, self.batch)
        h, V = self.dev.handle, self.cfg.vocab
        if self.sampler is None:
            N.call("ns_argmax_i32", h, C.c_uint64(self.logits.ptr), self.batch, V, C.c_int64(V), C.c_uint64(self.ids.ptr))
        else:
            self.sampler.Sample(self.logits, 1)
            N.call("ns_ids_from_f32", h, C.c_uint64(self.sampler.Ids.ptr), C.c_uint64(self.ids.ptr), self.batch)
        self._n = step.launches + 1

    def _last_rows(self, steps: int) -> None:
        self._put(self.row_map, np.arange(1, self.batch + 1) * steps - 1)

    def prefill(self, ids: np.ndarray) -> None:
        """ids [batch, t]: reads t positions from position 0 and leaves the next token of every sequence in ids[0:batch]."""
        ids = np.ascontiguousarray(ids, dtype=np.int32)
        b, t = ids.shape
        assert b == self.batch and t >= 1
        if self._lockstep is None:
            self._lockstep = [self.states.open() for _ in range(b)]
        else:
            self.states.rewind(*self._lockstep)
        self._use_slots(self._lockstep)
        self.length = 0
        for at in range(0, t, self.max_prefill):
            n = min(self.max_prefill, t - at)
            self._put(self.ids, ids[:, at:at + n])
            if at + n < t:
                step = self._step(b, n, at)
                self._layers(step)
                self._advance(step)
                self.length += n
            else:
                self._last_rows(n)
                self._forward(n)
        self._last_rows(1)
        self.length = t

    def read_logits(self) -> np.ndarray:
        return self.logits.download((self.batch, self.cfg.vocab), count=self.batch * self.cfg.vocab)

    def close(self) -> None:
        self.drop_graph()
        for b in self._blocks:
            b.close()
        self.head.close()
