"""Fabezen: a decoder whose layers mix a gated delta rule (one decay per head, or one per head and key channel) with latent
attention over a sliding window, in any order, with a bigram embedding and a tied output.

The model is a list of blocks (nn_b200.blocks) over a 32-bit residual stream:
    x <- x + m * mixer(rms(x));  x <- x + m * ff(rms(x))
and the row kernel that adds a block's output also normalises for the next block.  Layers may share weights; what
a sequence carries is kept per layer.  Sequences live in slots (nn_b200.state); there is no limit on a sequence's length, because windows
are rings and the other layers are recurrent.
"""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass, field

import numpy as np

from . import native as N
from .blocks import DeltaMixer, DenseGlu, LatentAttentionMixer, Product, Source, Step, Workspace, bf16_bits, f32, pad8, rms_rows
from .decoder import CachedDecoder
from .device import Device
from .state import SequenceStates

MIXERS = ("delta", "channel_delta", "latent_attention")


@dataclass
class LayerConfig:
    type: str
    mixer: dict
    mlp: dict | None
    weights_of: int | None = None


@dataclass
class FabezenConfig:
    vocab: int
    width: int
    layers: list = field(default_factory=list)
    eps: float = 1e-5
    residual_mult: float = 1.0
    embedding_scale: float = 1.0
    bigram: dict | None = None          # buckets, mul_prev, mul_cur

    @staticmethod
    def from_dict(j: dict) -> "FabezenConfig":
        layers = []
        for i, e in enumerate(j["layers"]):
            if e["type"] not in MIXERS:
                raise ValueError(f"layer {i}: unknown type {e['type']!r}")
            if e.get("mlp") is not None and e["mlp"].get("kind", "dense") != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward {e['mlp'].get('kind')!r}")
            layers.append(LayerConfig(e["type"], dict(e["mixer"]), e.get("mlp"), e.get("weights_of")))
        for i, layer in enumerate(layers):
            if layer.weights_of is not None and not 0 <= layer.weights_of < len(layers):
                raise ValueError(f"layer {i}: weights_of {layer.weights_of}")
        emb = j.get("embedding") or {}
        return FabezenConfig(vocab=int(j["vocab"]), width=int(j["width"]), layers=layers, eps=float(j["norm"]["eps"]),
                             residual_mult=float(j.get("residual_mult", 1.0)), embedding_scale=float(emb.get("scale", 1.0)), bigram=emb.get("bigram"))

    def owner(self, i: int) -> int:
        """The layer whose tensors layer i uses."""
        seen = set()
        while self.layers[i].weights_of is not None:
            if i in seen:
                raise ValueError("weights_of goes round in a circle")
            seen.add(i)
            i = self.layers[i].weights_of
        return i

    def tensor_shapes(self) -> dict:
        """name -> shape of every tensor of a weight file that the configuration fixes (low ranks are the file's own)."""
        D = self.width
        out = {"embed": (self.vocab, D), "final.norm": (D,)}
        if self.bigram is not None:
            out["bigram"] = (self.bigram["buckets"] + 1, D)
        for i, layer in enumerate(self.layers):
            if layer.weights_of is not None:
                continue
            p, m = f"l{i}.", layer.mixer
            out[p + "norm1"] = (D,)
            if layer.type == "latent_attention":
                H = m["heads"]
                t = {"dq": (m["q_rank"], D), "dq.norm": (m["q_rank"],), "uq": (H * (m["dim"] + m["rot_dim"]), m["q_rank"]),
                     "dkv": (m["kv_rank"] + m["rot_dim"], D), "dkv.norm": (m["kv_rank"],), "uk": (H * m["dim"], m["kv_rank"]),
                     "uv": (H * m["vdim"], m["kv_rank"]), "o": (D, H * m["vdim"])}
            else:
                H, qk, v = m["heads"], m["kv_heads"] * m["dim"], m["heads"] * m["vdim"]
                t = {"q": (qk, D), "k": (qk, D), "v": (v, D), "q.conv": (qk, m["conv"]), "k.conv": (qk, m["conv"]), "v.conv": (v, m["conv"]), "b": (H, D),
                     "A_log": (H,), "norm": (m["vdim"],), "o": (D, v)}
                if layer.type == "delta":
                    t.update({"a": (H, D), "dt_bias": (H,), "g": (v, D)})
                else:
                    t.update({"a1": (None, D), "a2": (H * m["dim"], None), "dt_bias": (H * m["dim"],), "g1": (None, D), "g2": (v, None)})
            out.update({p + "mix." + k: s for k, s in t.items()})
            if layer.mlp is not None:
                ff = layer.mlp["ff"]
                out.update({p + "norm2": (D,), p + "mlp.gate": (ff, D), p + "mlp.up": (ff, D), p + "mlp.down": (D, ff)})
        return out


class _LayerWeights:
    """The blocks made from one layer's tensors."""

    def __init__(self, ws: Workspace, cfg: FabezenConfig, i: int, w):
        layer, p, m, dev = cfg.layers[i], f"l{i}.", cfg.layers[i].mixer, ws.dev
        t = lambda name: w[p + "mix." + name]
        self.norm1 = dev.from_numpy(f32(w[p + "norm1"]))
        if layer.type == "latent_attention":
            names = {"dq": "dq", "dq_norm": "dq.norm", "uq": "uq", "dkv": "dkv", "dkv_norm": "dkv.norm", "uk": "uk", "uv": "uv", "o": "o"}
            self.mixer = LatentAttentionMixer(ws, m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["q_rank"], m["kv_rank"], float(m["scale"]),
                                              int(m["mask"]["size"]), m["rot"]["base"], int(m["rot"]["dims"]), cfg.eps,
                                              {k: t(n) for k, n in names.items()})
        else:
            names = {"q": "q", "k": "k", "v": "v", "b": "b", "o": "o", "q_conv": "q.conv", "k_conv": "k.conv", "v_conv": "v.conv", "A_log": "A_log",
                     "dt_bias": "dt_bias", "norm": "norm"}
            names.update({n: n for n in (("a", "g") if layer.type == "delta" else ("a1", "a2", "g1", "g2"))})
            self.mixer = DeltaMixer(ws, m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"], cfg.eps, {k: t(n) for k, n in names.items()})
        self.norm2 = self.ff = None
        if layer.mlp is not None:
            self.norm2 = dev.from_numpy(f32(w[p + "norm2"]))
            self.ff = DenseGlu(ws, w[p + "mlp.gate"], w[p + "mlp.up"], w[p + "mlp.down"])

    def close(self) -> None:
        self.mixer.close()
        if self.ff is not None:
            self.ff.close()


class Fabezen(CachedDecoder):
    """weights: mapping of tensor name -> array, bf16 bits (uint16) or float32, in the shapes of FabezenConfig.tensor_shapes; any
    mapping works, every tensor is looked up once.  dtype NS_BF16 or NS_F32.  `batch` sequences run in lockstep in generate();
    `slots` (default: batch) sequences can be open at a time; a pass takes at most `max_prefill` tokens per sequence, longer
    prompts are read in portions."""

    LOGIT_ROWS = 64          # rows the head works on at a time

    def __init__(self, dev: Device, cfg: FabezenConfig, weights, batch: int = 1, max_prefill: int = 512, dtype: int = N.NS_BF16, slots: int | None = None):
        self.dev, self.cfg, self.batch, self.dtype, self.max_prefill = dev, cfg, batch, dtype, max_prefill
        ws = self.ws = Workspace(dev, dtype)
        D = cfg.width
        self.states = SequenceStates(dev, slots if slots is not None else batch)
        self._owned = {}
        self.layers = []
        for i in range(len(cfg.layers)):
            j = cfg.owner(i)
            if j not in self._owned:
                self._owned[j] = _LayerWeights(ws, cfg, j, weights)
            lw = self._owned[j]
            self.layers.append((lw, lw.mixer.reserve(self.states, max_prefill)))
        self.head = Product(ws, weights["embed"])            # also the embedding table
        self.final_norm = dev.from_numpy(f32(weights["final.norm"]))
        self.bigram = None
        if cfg.bigram is not None:
            table = weights["bigram"]
            self.bigram = dev.from_numpy((bf16_bits(table) if dtype == N.NS_BF16 else f32(table)).reshape(-1))
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

    # ------------------------------------------------------------------ one pass
    def _layers(self, step: Step) -> None:
        """Embedding and every layer for the ids of the pass; leaves the residual stream in ``x``."""
        cfg, dev, ws = self.cfg, self.dev, self.ws
        D, x, h, m = cfg.width, ws["x"], ws["h"], cfg.residual_mult
        u = C.c_uint64
        b = cfg.bigram or {"buckets": 1, "mul_prev": 0, "mul_cur": 0}
        N.call("ns_embed_ngram", dev.handle, u(self.ids.ptr), u(self.head.w_ptr), self.dtype, self.head.k_ld, C.c_float(cfg.embedding_scale),
               u(self.bigram.ptr if self.bigram else 0), D, b["buckets"], C.c_int64(b["mul_prev"]), C.c_int64(b["mul_cur"]), u(step.slots),
               u(self.states.last.ptr), step.batch, step.steps, D, cfg.vocab, u(x))
        step.launches += 1
        source: Source | None = None
        for lw, cache in self.layers:
            rms_rows(step, dev, x, source, m, x if source else 0, lw.norm1, cfg.eps, D, h, self.dtype, pad8(D))
            source = lw.mixer.forward(h, cache, step)
            if lw.ff is not None:
                rms_rows(step, dev, x, source, m, x, lw.norm2, cfg.eps, D, h, self.dtype, pad8(D))
                source = lw.ff.forward(h, step)
        rms_rows(step, dev, x, source, m, x, None, cfg.eps, D, 0, self.dtype, 0)

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
        for lw in self._owned.values():
            lw.close()
        self.head.close()
