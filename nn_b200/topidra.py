"""Topidra: a decoder whose layers are windowed softmax attention with a sink, or linear attention with fixed decays, in any order, some
of them run several times in a row.

The model is a list of blocks (nn_b200.blocks) over a 32-bit residual stream, with a norm before and after every sublayer:
    x <- x + rms(mixer(rms(x)));  x <- x + rms(ff(rms(x)))
The row kernel that adds a sublayer's output normalises it first and normalises the sum for the next one.  Layers of a loop share
their weights from pass to pass, what a sequence carries is kept per pass, and before every pass but the first the embedding is added
to x (by the row kernel that ends the pass before).
"""
from __future__ import annotations

from dataclasses import dataclass, field

from . import native as N
from .block_decoder import BlockDecoder
from .blocks import DenseGlu, LightningMixer, Step, WindowAttentionMixer, Workspace, f32, pad8, rms_post_rows, rms_rows

MIXERS = ("attention", "lightning")


@dataclass
class LayerConfig:
    type: str
    mixer: dict
    mlp: dict | None


@dataclass
class TopidraConfig:
    vocab: int
    width: int
    layers: list = field(default_factory=list)
    eps: float = 1e-5
    loop: dict | None = None            # start, stop, times

    @staticmethod
    def from_dict(j: dict) -> "TopidraConfig":
        layers = []
        for i, e in enumerate(j["layers"]):
            if e["type"] not in MIXERS:
                raise ValueError(f"layer {i}: unknown type {e['type']!r}")
            if e.get("mlp") is not None and e["mlp"].get("kind", "dense") != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward {e['mlp'].get('kind')!r}")
            layers.append(LayerConfig(e["type"], dict(e["mixer"]), e.get("mlp")))
        if not layers:
            raise ValueError("a model without layers")
        loop = j.get("loop")
        if loop is not None:
            loop = {k: int(loop[k]) for k in ("start", "stop", "times")}
            if not 0 <= loop["start"] <= loop["stop"] <= len(layers) or loop["times"] < 1:
                raise ValueError(f"loop {loop} over {len(layers)} layers")
        return TopidraConfig(vocab=int(j["vocab"]), width=int(j["width"]), layers=layers, eps=float(j["norm"]["eps"]), loop=loop)

    def runs(self) -> list:
        """(layer, whether the embedding is added before it), in the order the layers run."""
        n = len(self.layers)
        start, stop, times = (self.loop["start"], self.loop["stop"], self.loop["times"]) if self.loop else (0, 0, 1)
        out = [(i, False) for i in range(start)]
        for t in range(times):
            out += [(i, t > 0 and i == start) for i in range(start, stop)]
        return out + [(i, False) for i in range(stop, n)]

    def tensor_shapes(self) -> dict:
        """name -> shape of every tensor of a weight file."""
        D = self.width
        out = {"embed": (self.vocab, D), "final.norm": (D,), "head": (self.vocab, D)}
        for i, layer in enumerate(self.layers):
            p, m = f"l{i}.", layer.mixer
            out.update({p + "norm1": (D,), p + "norm1b": (D,)})
            if layer.type == "attention":
                H, q, k, v = m["heads"], m["heads"] * m["dim"], m["kv_heads"] * m["dim"], m["kv_heads"] * m["vdim"]
                t = {"q": (q, D), "k": (k, D), "v": (v, D), "q.norm": (q,), "k.norm": (k,), "sink": (H,), "g": (H, D), "o": (D, H * m["vdim"])}
            else:
                qk, v = m["heads"] * m["dim"], m["heads"] * m["vdim"]
                t = {"q": (qk, D), "k": (qk, D), "v": (v, D), "g": (v, D), "norm": (v,), "o": (D, v)}
            out.update({p + "mix." + k: s for k, s in t.items()})
            if layer.mlp is not None:
                ff = layer.mlp["ff"]
                out.update({p + "norm2": (D,), p + "norm2b": (D,), p + "mlp.gate": (ff, D), p + "mlp.up": (ff, D), p + "mlp.down": (D, ff)})
        return out


class _LayerWeights:
    """The blocks made from one layer's tensors."""

    def __init__(self, ws: Workspace, cfg: TopidraConfig, i: int, w):
        layer, p, m = cfg.layers[i], f"l{i}.", cfg.layers[i].mixer
        up = lambda name: ws.dev.from_numpy(f32(w[p + name]))
        t = lambda *names: {n.replace(".", "_"): w[p + "mix." + n] for n in names}
        if layer.type == "attention":
            self.mixer = WindowAttentionMixer(ws, m["heads"], m["kv_heads"], m["dim"], m["vdim"], float(m["scale"]), int(m["mask"]["size"]), cfg.eps,
                                              t("q", "k", "v", "g", "o", "q.norm", "k.norm", "sink"))
        else:
            self.mixer = LightningMixer(ws, m["heads"], m["dim"], m["vdim"], m["decay"], cfg.eps, t("q", "k", "v", "g", "o", "norm"))
        self.norm1, self.norm1b = up("norm1"), up("norm1b")
        self.ff = None
        if layer.mlp is not None:
            self.norm2, self.norm2b = up("norm2"), up("norm2b")
            self.ff = DenseGlu(ws, w[p + "mlp.gate"], w[p + "mlp.up"], w[p + "mlp.down"], N.ACT_RELU)

    def close(self) -> None:
        self.mixer.close()
        if self.ff is not None:
            self.ff.close()


class Topidra(BlockDecoder):
    """weights in the shapes of TopidraConfig.tensor_shapes; the rest as BlockDecoder has it."""

    def _build(self, weights) -> None:
        cfg = self.cfg
        self._blocks = [_LayerWeights(self.ws, cfg, i, weights) for i in range(len(cfg.layers))]
        # (blocks, this run's cache or state, embedding added before it)
        self.layers = [(self._blocks[i], self._blocks[i].mixer.reserve(self.states, self.max_prefill), again) for i, again in cfg.runs()]
        self.table = self._table(weights["embed"])
        # x as the embedding leaves it, kept where a later pass adds it again
        self.embedded = "embedded" if any(again for _, _, again in self.layers) else "x"
        self.ws.need(self.embedded, cfg.width, N.NS_F32)

    def _layers(self, step: Step) -> None:
        """Embedding and every layer for the ids of the pass; leaves the residual stream in ``x``."""
        cfg, dev, ws = self.cfg, self.dev, self.ws
        D, eps, x, h = cfg.width, cfg.eps, ws["x"], ws["h"]
        embedded = ws[self.embedded]
        self._embed(step, self.table.ptr, D, embedded)
        rms_rows(step, dev, embedded, None, 0.0, 0, self.layers[0][0].norm1, eps, D, h, self.dtype, pad8(D))
        here = embedded                       # where the residual stream is read
        for i, (lw, cache, _) in enumerate(self.layers):
            source, post = lw.mixer.forward(h, cache, step), lw.norm1b
            if lw.ff is not None:
                rms_post_rows(step, dev, here, source, post, 0, x, lw.norm2, eps, D, h, self.dtype, pad8(D))
                here, source, post = x, lw.ff.forward(h, step), lw.norm2b
            following = self.layers[i + 1] if i + 1 < len(self.layers) else None
            rms_post_rows(step, dev, here, source, post, embedded if following and following[2] else 0, x, following[0].norm1 if following else None, eps, D, h,
                          self.dtype, pad8(D))
            here = x
